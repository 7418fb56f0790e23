"""Decoder over fp32 residual streams with a mixer per layer chosen by the configuration.

``config.model.layer_specs`` lists the layers (mixer type and sizes, feed-forward or none); ``layer_loop`` repeats a
block of layers: the passes share the weights, while each has cache rows and states to itself. Switches of the
configuration say what surrounds a sublayer: learned stream weights or a plain residual, gates, a token shift, inputs of
a loop's passes. Between sublayers everything happens in one fused boundary (:mod:`ironcore_b200.ops.streams`): the
finished sublayer's result is gated and written into the streams, the next one's input is read, normed and shifted.

There is one evaluation, :meth:`StreamModel.hidden`, over a :class:`~ironcore_b200.rl.batch.StepBatch` and a cache:
the rollout engine calls it for prompts, decoding and mixed steps, and ``LanguageModel.forward`` with a cache of the
call's own. There is no backward pass: these families are served, not trained."""

from __future__ import annotations

from typing import Dict, List, Optional, Tuple

import torch
import torch.nn as nn

from ..layers.activations import is_glu
from ..layers.gated_delta import GatedDelta, GatedDeltaSpec
from ..layers.grouped_attention import GroupedAttention, GroupedAttentionSpec
from ..layers.latent_attention import LatentAttention, LatentAttentionSpec
from ..layers.mixer import BranchMixer, CacheSpec, PackedLinear, Stored, pad_to, stored
from ..layers.selective_scan import SelectiveScan, SelectiveScanSpec
from ..layers.streams import DenseMLP, GatedStreamMLP, ResidualGate, StreamPort
from ..ops import streams as OS
from ..parallel import mesh


# Mixers by the names of the configuration: (model configuration, the layer's mixer sizes) -> module
def _latent_attention(m, mixer, **kw):
    return LatentAttention(m.d_model, LatentAttentionSpec.from_mixer(mixer), m.ln_eps, **kw)


def _selective_scan(m, mixer, **kw):
    spec = SelectiveScanSpec(inner=int(mixer["inner"]), state=int(mixer["state"]), dt_rank=int(mixer["dt_rank"]),
                             conv=int(mixer["conv"]))
    return BranchMixer(m.d_model, [("", SelectiveScan(spec, **kw), 1.0)], **kw)


def _attention_beside_delta(m, mixer, **kw):
    left, right = mixer["left"], mixer["right"]
    rot = left.get("rot") or {}
    attention = GroupedAttentionSpec(
        heads=int(left["heads"]), kv_heads=int(left["kv_heads"]), dim=int(left["dim"]), vdim=int(left["vdim"]),
        scale=float(left["scale"]), rot_dims=int(rot.get("dims", 0)), rot_base=float(rot.get("base", 10000.0)),
        chunk=int((left.get("mask") or {}).get("size") or 0))
    delta = GatedDeltaSpec(
        heads=int(right["heads"]), kv_heads=int(right["kv_heads"]), dim=int(right["dim"]), vdim=int(right["vdim"]),
        conv=int(right["conv"]), decay_rank=int(right.get("decay_rank") or right["dim"]),
        gate_rank=int(right.get("gate_rank") or right["vdim"]))
    return BranchMixer(m.d_model, [("left.", GroupedAttention(attention, **kw), mixer["left_scale"]),
                                   ("right.", GatedDelta(delta, m.ln_eps, **kw), mixer["right_scale"])], **kw)


MIXERS = {"latent_attention": _latent_attention, "mamba1": _selective_scan, "parallel": _attention_beside_delta}


def _feed_forward(m, mlp, **kw):
    if mlp.get("kind") != "dense":
        raise ValueError(f"unknown feed-forward kind {mlp.get('kind')!r} (known: dense)")
    return (GatedStreamMLP if is_glu(m.activation_type) else DenseMLP)(m.d_model, int(mlp["ff"]), m.activation_type, **kw)


def run_schedule(num_layers: int, loop: Optional[dict]) -> List[Tuple[int, Optional[int]]]:
    """(layer index, number of the loop's pass that starts right before it or None) of every run: layers
    ``start .. stop - 1`` repeat ``times`` times as a block."""
    if not loop:
        return [(i, None) for i in range(num_layers)]
    start, stop, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    if not 0 <= start <= stop <= num_layers or times < 0:
        raise ValueError(f"layer loop {loop} does not fit {num_layers} layers")
    block = [(i, t if i == start else None) for t in range(times) for i in range(start, stop)]
    return [(i, None) for i in range(start)] + block + [(i, None) for i in range(stop, num_layers)]


def run_order(num_layers: int, loop: Optional[dict]) -> List[int]:
    """Layer index of every run."""
    return [i for i, _ in run_schedule(num_layers, loop)]


class StreamLayer(nn.Module):
    def __init__(self, config, spec: dict, dtype=None, device=None):
        super().__init__()
        m = config.model
        kind = spec.get("type")
        if kind not in MIXERS:
            raise ValueError(f"unknown mixer type {kind!r} (known: {', '.join(MIXERS)})")
        kw = dict(dtype=dtype, device=device)

        def port():
            return StreamPort(m.d_model, m.residual_streams, m.norm_groups, m.ln_eps, device=device,
                              learned=m.stream_mixing, gain=m.residual_mult)

        self.mixer_port = port()
        self.mixer = MIXERS[kind](m, spec["mixer"], **kw)
        self.shift = nn.Parameter(torch.zeros(m.d_model, dtype=torch.float32, device=device)) if m.token_shift else None
        self.mixer_gate = ResidualGate(m.d_model, **kw) if m.residual_gates else None
        self.mlp_port = self.mlp = None
        if spec.get("mlp"):
            self.mlp_port, self.mlp = port(), _feed_forward(m, spec["mlp"], **kw)

    def cache_spec(self) -> CacheSpec:
        spec = self.mixer.cache_spec()
        if self.shift is not None:
            spec.states["shift"] = ((self.shift.numel(),), torch.float32)
        return spec

    def stored_tensors(self) -> Dict[str, Stored]:
        """Checkpoint name (without the layer prefix) -> where its values are."""
        out = {f"mix.{k}": v for k, v in self.mixer.stored_tensors().items()}
        if self.mixer_gate is not None:
            out.update({f"rg1{k}": v for k, v in self.mixer_gate.stored_tensors().items()})
        if self.shift is not None:
            out["shift"] = stored(self.shift.data)
        if self.mlp is not None:
            out.update(self.mlp.stored_tensors())
        for n, port in ((1, self.mixer_port), (2, self.mlp_port)):
            if port is not None:
                out[f"norm{n}"] = stored(port.norm.weight.data)
                if port.learned:
                    out.update({f"hc{n}.in": stored(port.read.data), f"hc{n}.out": stored(port.write.data),
                                f"hc{n}.mix": stored(port.mix.data)})
        return out


class StreamModel(nn.Module):
    def __init__(self, config, dtype=None, device=None):
        super().__init__()
        m = config.model
        if not m.layer_specs:
            raise ValueError("model.layer_specs is empty: this family takes its layers from the configuration")
        if mesh.get_tensor_model_parallel_world_size() > 1:
            raise ValueError("residual-stream models are not sharded: tensor_model_parallel_size must be 1")
        if m.residual_gates and not is_glu(m.activation_type):
            raise ValueError("residual gates come with the gated feed-forward: activation_type must be a gated one")
        self.config = config
        self.d_model, self.width, self.streams = m.d_model, pad_to(m.d_model, 8), int(m.residual_streams)
        self.layers = nn.ModuleList([StreamLayer(config, spec, dtype, device) for spec in m.layer_specs])
        self.schedule = run_schedule(len(self.layers), m.layer_loop)
        self.order = [i for i, _ in self.schedule]
        self.loop_step = None
        if m.layer_loop and m.loop_inputs:
            self.loop_step = nn.Parameter(torch.zeros((int(m.layer_loop["times"]), m.d_model), dtype=torch.float32,
                                                      device=device))
        self.register_buffer("sum_streams", torch.ones(self.streams, dtype=torch.float32, device=device), persistent=False)

    def stored_tensors(self) -> Dict[str, Stored]:
        """Checkpoint name -> where its values are."""
        out = {} if self.loop_step is None else {"loop.step": stored(self.loop_step.data)}
        for i, layer in enumerate(self.layers):
            out.update({f"l{i}.{name}": v for name, v in layer.stored_tensors().items()})
        return out

    def init_special(self, generator: Optional[torch.Generator] = None):
        """Values that the common initialisation does not fit: zero padding, plain residual streams, a mild shift."""
        with torch.no_grad():
            for layer in self.layers:
                if hasattr(layer.mixer, "reset"):
                    layer.mixer.reset(generator)
                places = layer.stored_tensors()
                keep = {name: p.value().clone() for name, p in places.items()}
                for mod in layer.modules():
                    if isinstance(mod, PackedLinear):
                        mod.weight.zero_()
                for name, p in places.items():
                    p.put(keep[name])
                for port in (layer.mixer_port, layer.mlp_port):
                    if port is not None:
                        port.reset()
                if layer.shift is not None:
                    layer.shift.fill_(0.25)

    def refresh(self):
        """Rebuild what is derived from weights (call after changing them under a captured decode step)."""
        for layer in self.layers:
            if hasattr(layer.mixer, "refresh"):
                layer.mixer.refresh()

    def make_cache(self, max_seqs: int, max_seq_len: int, block_size: int, num_blocks: Optional[int] = None,
                   device=None, dtype=None):
        from ..rl.kv_cache import LayerCache

        return LayerCache([self.layers[i].cache_spec() for i in self.order], max_seqs=max_seqs, max_seq_len=max_seq_len,
                          block_size=block_size, num_blocks=num_blocks, dtype=dtype, device=device)

    def hidden(self, batch, cache, table: torch.Tensor, scale: float, final_norm) -> torch.Tensor:
        """Final-normed rows ``batch.want`` (all rows when None) of the batch, [rows, width]."""
        dtype = table.dtype
        source = embedded = OS.TokenEmbed(batch.tokens, table, scale, self.streams)
        for run, (index, turn) in enumerate(self.schedule):
            layer = self.layers[index]
            shift = add = None
            if layer.shift is not None:
                state = cache.states[run]["shift"]
                # a sequence that continues with several rows reads its old state while its last row writes the new one
                prev = state.clone() if batch.kind == "extend" else state
                shift = OS.TokenShift(layer.shift, prev, state, batch.seqs, batch.positions)
            if turn is not None and self.loop_step is not None:
                add = OS.StreamAdd(self.loop_step.data[turn], embedded if turn > 0 else None)
            x, h, hs = self._boundary(source, layer.mixer_port, dtype, shift, add)
            y = layer.mixer(h if hs is None else hs, batch, cache, run)
            source = self._written(x, y, layer.mixer_port, *self._gate(layer, h))
            if layer.mlp is not None:
                x, h, _ = self._boundary(source, layer.mlp_port, dtype)
                y, gate = layer.mlp(h)
                source = self._written(x, y, layer.mlp_port, gate, None if gate is None else layer.mlp.bias)
            self._observe(source, run)
        _, h, _ = OS.boundary(source, self.sum_streams, final_norm.weight, final_norm.groups, final_norm.eps,
                              width=self.width, dtype=dtype, rows=batch.want, keep_streams=False)
        return h

    # set to a list to collect the sum of the streams after every layer run, fp32 [T, D] each
    trace: Optional[list] = None

    def _observe(self, source, run: int):
        if self.trace is not None:
            x, _, _ = OS.boundary(source, self.sum_streams, torch.ones(self.d_model, device=source.y.device), 1, 1.0,
                                  width=self.width, dtype=source.y.dtype)
            self.trace.append(x.sum(1))

    @staticmethod
    def _gate(layer, h):
        return (None, None) if layer.mixer_gate is None else (layer.mixer_gate(h), layer.mixer_gate.bias)

    @staticmethod
    def _written(x, y, port: StreamPort, gate, bias) -> OS.StreamWrite:
        return OS.StreamWrite(x, y, gate, bias, port.mix, port.write)

    def _boundary(self, source, port: StreamPort, dtype, shift=None, add=None):
        return OS.boundary(source, port.read, port.norm.weight, port.norm.groups, port.norm.eps, width=self.width,
                           dtype=dtype, shift=shift, add=add)
