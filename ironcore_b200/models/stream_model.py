"""Decoder with several residual streams per token and a mixer per layer chosen by the configuration.

``config.model.layer_specs`` lists the layers (mixer type and sizes, feed-forward or none); ``layer_loop`` repeats a
block of layers: the passes share the weights, while each has cache rows and shift states to itself.
Between sublayers everything happens in one fused boundary (:mod:`ironcore_b200.ops.streams`): the finished sublayer's
result is gated and written into the streams, the next one's input is read, normed and shifted.

There is one evaluation, :meth:`StreamModel.hidden`, over a :class:`~ironcore_b200.rl.batch.StepBatch` and a cache:
the rollout engine calls it for prompts, decoding and mixed steps, and ``LanguageModel.forward`` with a cache of the
call's own. There is no backward pass: the family is served, not trained."""

from __future__ import annotations

from typing import Dict, List, Optional

import torch
import torch.nn as nn

from ..layers.latent_attention import LatentAttention, LatentAttentionSpec, PackedLinear, Stored, pad_to, stored
from ..layers.streams import GatedStreamMLP, ResidualGate, StreamPort
from ..ops import streams as OS
from ..parallel import mesh


def _latent_attention(d_model, mixer, eps, dtype, device):
    return LatentAttention(d_model, LatentAttentionSpec.from_mixer(mixer), eps, dtype=dtype, device=device)


MIXERS = {"latent_attention": _latent_attention}
FEED_FORWARDS = {"dense": "geglu"}       # kind -> gated activation


def run_order(num_layers: int, loop: Optional[dict]) -> List[int]:
    """Layer index of every run: layers ``start .. stop - 1`` repeat ``times`` times as a block."""
    if not loop:
        return list(range(num_layers))
    start, stop, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    if not 0 <= start <= stop <= num_layers or times < 0:
        raise ValueError(f"layer loop {loop} does not fit {num_layers} layers")
    return list(range(start)) + list(range(start, stop)) * times + list(range(stop, num_layers))


class StreamLayer(nn.Module):
    def __init__(self, config, spec: dict, dtype=None, device=None):
        super().__init__()
        m = config.model
        kind = spec.get("type")
        if kind not in MIXERS:
            raise ValueError(f"unknown mixer type {kind!r} (known: {', '.join(MIXERS)})")
        ports = (m.d_model, m.residual_streams, m.norm_groups, m.ln_eps)
        self.mixer_port = StreamPort(*ports, device=device)
        self.mixer = MIXERS[kind](m.d_model, spec["mixer"], m.ln_eps, dtype, device)
        self.shift = nn.Parameter(torch.zeros(m.d_model, dtype=torch.float32, device=device))
        self.mixer_gate = ResidualGate(m.d_model, dtype=dtype, device=device)
        self.mlp_port = self.mlp = None
        mlp = spec.get("mlp")
        if mlp:
            if mlp.get("kind") not in FEED_FORWARDS:
                raise ValueError(f"unknown feed-forward kind {mlp.get('kind')!r} (known: {', '.join(FEED_FORWARDS)})")
            self.mlp_port = StreamPort(*ports, device=device)
            self.mlp = GatedStreamMLP(m.d_model, int(mlp["ff"]), FEED_FORWARDS[mlp["kind"]], dtype=dtype, device=device)

    def stored_tensors(self) -> Dict[str, Stored]:
        """Checkpoint name (without the layer prefix) -> where its values are."""
        out = {f"mix.{k}": v for k, v in self.mixer.stored_tensors().items()}
        out.update({f"rg1{k}": v for k, v in self.mixer_gate.stored_tensors().items()})
        out["shift"] = stored(self.shift.data)
        if self.mlp is not None:
            out.update(self.mlp.stored_tensors())
        for n, port in ((1, self.mixer_port), (2, self.mlp_port)):
            if port is not None:
                out.update({f"norm{n}": stored(port.norm.weight.data), f"hc{n}.in": stored(port.read.data),
                            f"hc{n}.out": stored(port.write.data), f"hc{n}.mix": stored(port.mix.data)})
        return out


class StreamModel(nn.Module):
    def __init__(self, config, dtype=None, device=None):
        super().__init__()
        m = config.model
        if not m.layer_specs:
            raise ValueError("model.layer_specs is empty: this family takes its layers from the configuration")
        if mesh.get_tensor_model_parallel_world_size() > 1:
            raise ValueError("residual-stream models are not sharded: tensor_model_parallel_size must be 1")
        self.config = config
        self.d_model, self.width, self.streams = m.d_model, pad_to(m.d_model, 8), int(m.residual_streams)
        self.layers = nn.ModuleList([StreamLayer(config, spec, dtype, device) for spec in m.layer_specs])
        self.order = run_order(len(self.layers), m.layer_loop)
        self.register_buffer("sum_streams", torch.ones(self.streams, dtype=torch.float32, device=device), persistent=False)

    @property
    def max_window(self) -> int:
        """The widest window of any layer; 0 when some layer sees everything."""
        windows = [self.layers[i].mixer.spec.window for i in self.order]
        return 0 if not windows or min(windows) <= 0 else max(windows)

    def init_special(self, generator: Optional[torch.Generator] = None):
        """Values that the common initialisation does not fit: zero padding, plain residual streams, a mild shift."""
        with torch.no_grad():
            for layer in self.layers:
                places = layer.stored_tensors()
                keep = {name: p.view.clone() for name, p in places.items()}
                for mod in layer.modules():
                    if isinstance(mod, PackedLinear):
                        mod.weight.zero_()
                for name, p in places.items():
                    p.view.copy_(keep[name])
                for port in (layer.mixer_port, layer.mlp_port):
                    if port is not None:
                        port.reset()
                layer.shift.fill_(0.25)

    def refresh(self):
        """Rebuild what is derived from weights (call after changing them under a captured decode step)."""
        for layer in self.layers:
            if hasattr(layer.mixer, "refresh"):
                layer.mixer.refresh()

    def make_cache(self, max_seqs: int, max_seq_len: int, block_size: int, num_blocks: Optional[int] = None,
                   device=None, dtype=None):
        from ..rl.kv_cache import LatentCache

        return LatentCache([self.layers[i].mixer.c_width for i in self.order], self.d_model, max_seqs=max_seqs,
                           max_seq_len=max_seq_len, block_size=block_size, num_blocks=num_blocks,
                           window=self.max_window, dtype=dtype, device=device)

    def hidden(self, batch, cache, table: torch.Tensor, scale: float, final_norm) -> torch.Tensor:
        """Final-normed rows ``batch.want`` (all rows when None) of the batch, [rows, width]."""
        dtype = table.dtype
        source = OS.TokenEmbed(batch.tokens, table, scale, self.streams)
        for run, index in enumerate(self.order):
            layer = self.layers[index]
            state = cache.shift_state[run]
            # a sequence that continues with several rows reads its old state while its last row writes the new one
            prev = state.clone() if batch.kind == "extend" else state
            shift = OS.TokenShift(layer.shift, prev, state, batch.seqs, batch.positions)
            x, h, hs = self._boundary(source, layer.mixer_port, dtype, shift)
            source = OS.StreamWrite(x, layer.mixer(hs, batch, cache, run), layer.mixer_gate(h), layer.mixer_gate.bias,
                                    layer.mixer_port.mix, layer.mixer_port.write)
            if layer.mlp is not None:
                x, h, _ = self._boundary(source, layer.mlp_port, dtype)
                y, gate = layer.mlp(h)
                source = OS.StreamWrite(x, y, gate, layer.mlp.bias, layer.mlp_port.mix, layer.mlp_port.write)
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

    def _boundary(self, source, port: StreamPort, dtype, shift=None):
        return OS.boundary(source, port.read, port.norm.weight, port.norm.groups, port.norm.eps, width=self.width,
                           dtype=dtype, shift=shift)
