"""Model directories that describe themselves: ``config.json`` with an ``architecture`` key + ``model.safetensors``.

``load_pretrained`` picks the family by that key, builds the framework configuration and the model, and fills the
weights; ``save_pretrained`` writes the same form. Families register in ``ARCHITECTURES``. (HuggingFace directories,
recognised by ``model_type``, load through :mod:`.hf_interop` into a model built from a YAML configuration.)"""

from __future__ import annotations

import json
from pathlib import Path
from typing import Callable, Dict, Optional, Tuple

import torch

from ..config.loader import validate_config
from ..config.schema import MainConfig
from ..layers.mixer import Stored, stored
from .hf_interop import read_hf_state_dict


def _need(doc: dict, *path):
    node = doc
    for key in path:
        if not isinstance(node, dict) or key not in node:
            raise KeyError(f"config.json lacks {'.'.join(path)}")
        node = node[key]
    return node


Shapes = Optional[Dict[str, Tuple[int, ...]]]       # tensor name -> shape, where sizes are not in the document


def _stream_config(doc: dict, precision: str, **model) -> MainConfig:
    """What the documents of the residual-stream families have in common."""
    layers = _need(doc, "layers")
    c = MainConfig()
    c.model(d_model=int(_need(doc, "width")), vocab_size=int(_need(doc, "vocab")), num_layers=len(layers),
            layer_loop=doc.get("loop") or None, ln_eps=float(_need(doc, "norm", "eps")),
            embed_scale=float(_need(doc, "embedding", "scale")), precision=precision, dropout_embd=0.0, dropout_attn=0.0,
            dropout_mlp=0.0, reset_position_ids=False, reset_attention_mask=False, **model)
    c.data(task_type="synthetic", vocab_size=int(doc["vocab"]))
    c.trainer(micro_batch_size=1, train_batch_size=1, gradient_accumulation_steps=None)
    return validate_config(c)


def _stream_tensors(model) -> Dict[str, Stored]:
    """Tensor name of the checkpoint -> where the model keeps it."""
    d, v = model.model.d_model, model.vocab_size
    out = {"embed": stored(model.embedding.word_embeddings.weight.data[:v, :d]),
           "final.norm": stored(model.output_layernorm.weight.data)}
    if model.untied:
        out["head"] = stored(model.output_layer.weight.data[:d, :v].t())
    out.update(model.model.stored_tensors())
    return out


def _first_sizes(layers, attention: str = "") -> dict:
    """Head counts and sizes of the first layer that has them (informational: layers have sizes of their own)."""
    for spec in layers:
        m = spec.get("mixer") or {}
        m = m.get(attention, {}) if attention else m
        if "heads" in m:
            return dict(num_attention_heads=int(m["heads"]), num_attention_groups=int(m.get("kv_heads", m["heads"])),
                        head_dim=int(m["dim"]))
    return dict(num_attention_heads=1, num_attention_groups=1, head_dim=1)


def _first_ff(layers) -> int:
    return next((int(s["mlp"]["ff"]) for s in layers if s.get("mlp")), 0)


# --------------------------------------------------------------------------- Tetepel
def tetepel_config(doc: dict, precision: str = "bfloat16", shapes: Shapes = None) -> MainConfig:
    layers = _need(doc, "layers")
    return _stream_config(doc, precision, name="tetepel", layer_specs=list(layers), activation_type="geglu",
                          residual_streams=int(_need(doc, "streams")), norm_groups=int(_need(doc, "norm", "groups")),
                          d_ffn=_first_ff(layers), untie_embed=False, **_first_sizes(layers))


def tetepel_document(config) -> dict:
    m = config.model
    return {"architecture": "Tetepel", "embedding": {"scale": 1.0 if m.embed_scale is None else m.embed_scale},
            "layers": m.layer_specs, "loop": m.layer_loop, "norm": {"eps": m.ln_eps, "groups": m.norm_groups},
            "streams": m.residual_streams, "vocab": m.vocab_size, "width": m.d_model}


# --------------------------------------------------------------------------- Kedavik
_KEDAVIK_RANKS = {"decay_rank": "a1", "gate_rank": "g1"}      # sizes that only the tensors of the right branch tell


def kedavik_config(doc: dict, precision: str = "bfloat16", shapes: Shapes = None) -> MainConfig:
    layers = []
    for i, spec in enumerate(_need(doc, "layers")):
        spec = dict(spec)
        if spec.get("type") == "parallel":
            right = dict(_need(spec, "mixer", "right"))
            for key, tensor in _KEDAVIK_RANKS.items():
                shape = (shapes or {}).get(f"l{i}.mix.right.{tensor}")
                if shape is not None:
                    right[key] = int(shape[0])
            spec["mixer"] = {**spec["mixer"], "right": right}
        layers.append(spec)
    return _stream_config(doc, precision, name="kedavik", layer_specs=layers, activation_type="gelu", d_ffn=_first_ff(layers),
                          residual_mult=float(_need(doc, "residual_mult")), untie_embed=True, lm_head_bias=False,
                          **_first_sizes(layers, "left"))


def kedavik_document(config) -> dict:
    m = config.model
    layers = []
    for spec in m.layer_specs:
        if spec.get("type") == "parallel":
            right = {k: v for k, v in spec["mixer"]["right"].items() if k not in _KEDAVIK_RANKS}
            spec = {**spec, "mixer": {**spec["mixer"], "right": right}}
        layers.append(spec)
    return {"architecture": "Kedavik", "embedding": {"scale": 1.0 if m.embed_scale is None else m.embed_scale},
            "layers": layers, "loop": m.layer_loop, "norm": {"eps": m.ln_eps}, "residual_mult": m.residual_mult,
            "vocab": m.vocab_size, "width": m.d_model}


# "architecture" of config.json -> (configuration from document, precision and tensor shapes; document from
# configuration; places of the checkpoint's tensors in the model)
ARCHITECTURES: Dict[str, Tuple[Callable, Callable, Callable]] = {
    "Tetepel": (tetepel_config, tetepel_document, _stream_tensors),
    "Kedavik": (kedavik_config, kedavik_document, _stream_tensors),
}


# --------------------------------------------------------------------------- directories
def read_document(path) -> dict:
    p = Path(path) / "config.json"
    if not p.exists():
        raise FileNotFoundError(f"no config.json in {path}")
    doc = json.loads(p.read_text())
    name = doc.get("architecture")
    if name not in ARCHITECTURES:
        raise ValueError(f"{p}: architecture {name!r} is not known here ({', '.join(ARCHITECTURES)})")
    return doc


def load_tensors(model, tensors: Dict[str, torch.Tensor]) -> None:
    """Fill ``model`` from checkpoint tensors; every tensor must be there with its shape, and none may be left over."""
    from ..models import family_of

    want = _entry(family_of(model.config.model.name))[2](model)
    missing = sorted(set(want) - set(tensors))
    extra = sorted(set(tensors) - set(want))
    if missing or extra:
        raise KeyError(f"checkpoint does not fit the configuration: missing {missing[:4]}, unexpected {extra[:4]}")
    for name, place in want.items():
        t = tensors[name]
        if tuple(t.shape) != place.shape:
            raise ValueError(f"{name}: expected shape {place.shape}, got {tuple(t.shape)}")
        place.put(t)
    for p in model.parameters():      # the views above go through .data: tell whoever derives values from weights
        torch._C._autograd._unsafe_set_version_counter((p,), (p._version + 1,))
    model.model.refresh()


def _entry(family: str):
    for name, entry in ARCHITECTURES.items():
        if name.upper() == family:
            return entry
    raise ValueError(f"family {family} has no self-describing checkpoint form ({', '.join(ARCHITECTURES)})")


def load_pretrained(path, precision: str = "bfloat16", device=None):
    """(model in evaluation mode, configuration) of a model directory."""
    from ..models import LanguageModel

    doc = read_document(path)
    weights = read_hf_state_dict(path)
    config = ARCHITECTURES[doc["architecture"]][0](doc, precision, {k: tuple(t.shape) for k, t in weights.items()})
    model = LanguageModel(config, device=device).eval()
    load_tensors(model, weights)
    return model, config


def save_pretrained(model, config, path) -> Path:
    """Write ``config.json`` and ``model.safetensors`` (values in the model's own precision)."""
    from safetensors.torch import save_file

    from ..models import family_of

    _, document, tensors = _entry(family_of(config.model.name))
    out = Path(path)
    out.mkdir(parents=True, exist_ok=True)
    (out / "config.json").write_text(json.dumps(document(config), indent=1, sort_keys=True))
    dtype = next(model.parameters()).dtype
    save_file({k: v.value().to("cpu", dtype).contiguous() for k, v in tensors(model).items()},
              str(out / "model.safetensors"))
    return out
