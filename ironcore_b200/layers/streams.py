"""Parts of a residual-stream layer: the stream weights of a sublayer, its residual gate and the token shift.

All of them are small fp32 vectors consumed by the fused boundary (:func:`ironcore_b200.ops.streams.boundary`);
only the residual gate also owns a matrix."""

from __future__ import annotations

from typing import Dict

import torch
import torch.nn as nn

from ..ops.latent import project
from .activations import Activation
from .mixer import PackedLinear, Stored, pad_to, stored
from .norm import GroupedRMSNorm


class StreamPort(nn.Module):
    """How one sublayer reads from and writes to the streams: ``u = sum_s read[s] x_s``, then (all from the old
    values) ``x_t <- sum_s mix[s, t] x_s + write[t] y``; and the grouped norm of what it reads. The stream weights are
    parameters, or without ``learned`` constants: plain residual streams whose results count ``gain`` times."""

    def __init__(self, d_model: int, streams: int, groups: int, eps: float, device=None, learned: bool = True,
                 gain: float = 1.0):
        super().__init__()
        self.learned = learned
        kw = dict(dtype=torch.float32, device=device)
        for name, value in (("read", torch.full((streams,), 1.0 / streams, **kw)),
                            ("write", torch.full((streams,), float(gain), **kw)), ("mix", torch.eye(streams, **kw))):
            if learned:
                self.register_parameter(name, nn.Parameter(value))
            else:
                self.register_buffer(name, value, persistent=False)
        self.norm = GroupedRMSNorm(d_model, groups, eps, device=device)

    def reset(self):
        if not self.learned:
            return
        with torch.no_grad():
            self.read.fill_(1.0 / self.read.numel())
            self.write.fill_(1.0)
            self.mix.copy_(torch.eye(self.mix.shape[0]))


class ResidualGate(nn.Module):
    """Logits of the element-wise gate of a sublayer's result, ``sigmoid(W h + b)``."""

    def __init__(self, d_model: int, dtype=None, device=None):
        super().__init__()
        self.d_model = d_model
        width = pad_to(d_model, 8)
        self.proj = PackedLinear(width, width, dtype=dtype, device=device)
        self.bias = nn.Parameter(torch.zeros(d_model, dtype=torch.float32, device=device))

    def forward(self, h: torch.Tensor) -> torch.Tensor:
        return self.proj(h)

    def stored_tensors(self) -> Dict[str, Stored]:
        return {"": stored(self.proj.weight.data[:self.d_model, :self.d_model]), ".b": stored(self.bias.data)}


class DenseMLP(nn.Module):
    """down(act(up h + b)) + b, for residual streams without gates."""

    def __init__(self, d_model: int, d_ffn: int, activation: str = "gelu", dtype=None, device=None):
        super().__init__()
        self.d_model, self.d_ffn = d_model, d_ffn
        width, f_width = pad_to(d_model, 8), pad_to(d_ffn, 8)
        self.activation = Activation(activation)
        self.up_proj = PackedLinear(f_width, width, dtype=dtype, device=device, bias=True)
        self.down_proj = PackedLinear(width, f_width, dtype=dtype, device=device, bias=True)

    def forward(self, h: torch.Tensor):
        """h [T, width] -> (result [T, width], no gate)."""
        return self.down_proj(self.activation(self.up_proj(h))), None

    def stored_tensors(self) -> Dict[str, Stored]:
        d, f = self.d_model, self.d_ffn
        return {"mlp.up": stored(self.up_proj.weight.data[:f, :d]), "mlp.up.b": stored(self.up_proj.bias.data[:f]),
                "mlp.down": stored(self.down_proj.weight.data[:d, :f]), "mlp.down.b": stored(self.down_proj.bias.data[:d])}


class GatedStreamMLP(nn.Module):
    """Gated feed-forward whose first product also yields the residual-gate logits: [gate | up | gate logits]."""

    def __init__(self, d_model: int, d_ffn: int, activation: str = "geglu", dtype=None, device=None):
        super().__init__()
        self.d_model, self.d_ffn = d_model, d_ffn
        self.width, self.f_width = pad_to(d_model, 8), pad_to(d_ffn, 8)
        self.activation = Activation(activation)
        self.up_proj = PackedLinear(2 * self.f_width + self.width, self.width, dtype=dtype, device=device)
        self.down = PackedLinear(self.width, self.f_width, dtype=dtype, device=device)
        self.bias = nn.Parameter(torch.zeros(d_model, dtype=torch.float32, device=device))

    def forward(self, h: torch.Tensor):
        """h [T, width] -> (result [T, width], gate logits [T, width])."""
        z = project(h, self.up_proj.weight)
        return self.down(self.activation(z[:, :2 * self.f_width])), z[:, 2 * self.f_width:]

    def stored_tensors(self) -> Dict[str, Stored]:
        w, d, f, fw = self.up_proj.weight.data, self.d_model, self.d_ffn, self.f_width
        return {"mlp.gate": stored(w[:f, :d]), "mlp.up": stored(w[fw:fw + f, :d]),
                "mlp.down": stored(self.down.weight.data[:d, :f]), "rg2": stored(w[2 * fw:2 * fw + d, :d]),
                "rg2.b": stored(self.bias.data)}
