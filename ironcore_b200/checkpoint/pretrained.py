"""Model directories that describe themselves: ``config.json`` with an ``architecture`` key + ``model.safetensors``.

``load_pretrained`` picks the family by that key, builds the framework configuration and the model, and fills the
weights; ``save_pretrained`` writes the same form. Families register in ``ARCHITECTURES``. (HuggingFace directories,
recognised by ``model_type``, load through :mod:`.hf_interop` into a model built from a YAML configuration.)"""

from __future__ import annotations

import json
from pathlib import Path
from typing import Callable, Dict, Tuple

import torch

from ..config.loader import validate_config
from ..config.schema import MainConfig
from ..layers.latent_attention import Stored, stored
from .hf_interop import read_hf_state_dict


def _need(doc: dict, *path):
    node = doc
    for key in path:
        if not isinstance(node, dict) or key not in node:
            raise KeyError(f"config.json lacks {'.'.join(path)}")
        node = node[key]
    return node


# --------------------------------------------------------------------------- Tetepel
def tetepel_config(doc: dict, precision: str = "bfloat16") -> MainConfig:
    layers = _need(doc, "layers")
    first = layers[0] if layers else {}
    heads = int((first.get("mixer") or {}).get("heads", 1))
    c = MainConfig()
    c.model(name="tetepel", d_model=int(_need(doc, "width")), vocab_size=int(_need(doc, "vocab")),
            num_layers=len(layers), layer_specs=list(layers), layer_loop=doc.get("loop") or None,
            residual_streams=int(_need(doc, "streams")), norm_groups=int(_need(doc, "norm", "groups")),
            ln_eps=float(_need(doc, "norm", "eps")), embed_scale=float(_need(doc, "embedding", "scale")),
            num_attention_heads=heads, num_attention_groups=heads, head_dim=int((first.get("mixer") or {}).get("dim", 1)),
            d_ffn=int((first.get("mlp") or {}).get("ff", 0)), activation_type="geglu", precision=precision,
            untie_embed=False, dropout_embd=0.0, dropout_attn=0.0, dropout_mlp=0.0, reset_position_ids=False,
            reset_attention_mask=False)
    c.data(task_type="synthetic", vocab_size=int(doc["vocab"]))
    c.trainer(micro_batch_size=1, train_batch_size=1, gradient_accumulation_steps=None)
    return validate_config(c)


def tetepel_document(config) -> dict:
    m = config.model
    return {"architecture": "Tetepel", "embedding": {"scale": 1.0 if m.embed_scale is None else m.embed_scale},
            "layers": m.layer_specs, "loop": m.layer_loop, "norm": {"eps": m.ln_eps, "groups": m.norm_groups},
            "streams": m.residual_streams, "vocab": m.vocab_size, "width": m.d_model}


def tetepel_tensors(model) -> Dict[str, Stored]:
    """Tensor name of the checkpoint -> where the model keeps it."""
    out = {"embed": stored(model.embedding.word_embeddings.weight.data[:model.vocab_size, :model.model.d_model]),
           "final.norm": stored(model.output_layernorm.weight.data)}
    for i, layer in enumerate(model.model.layers):
        out.update({f"l{i}.{name}": v for name, v in layer.stored_tensors().items()})
    return out


ARCHITECTURES: Dict[str, Tuple[Callable, Callable, Callable]] = {
    "Tetepel": (tetepel_config, tetepel_document, tetepel_tensors),
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
        place.view.copy_(t.reshape(place.view.shape))
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
    config = ARCHITECTURES[doc["architecture"]][0](doc, precision)
    model = LanguageModel(config, device=device).eval()
    load_tensors(model, read_hf_state_dict(path))
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
    save_file({k: v.view.reshape(v.shape).to("cpu", dtype).contiguous() for k, v in tensors(model).items()},
              str(out / "model.safetensors"))
    return out
