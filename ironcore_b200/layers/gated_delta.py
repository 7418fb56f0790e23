"""Gated delta rule branch: columns [q | k | v | beta logits | low-rank decay | low-rank output gate] of the shared input
product. Two narrow products expand decay and output gate; one kernel does the short convolutions, unit norms, decay
factors and beta, one the recurrence, one the normed and gated output. The state per sequence is the rule's matrix per head
(fp32) and the last inputs of the convolutions. Head sizes are padded to multiples of 8 with zeros."""

from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Dict, List, Optional

import torch
import torch.nn as nn

from ..ops import recurrent as OR
from .mixer import Branch, CacheSpec, PackedLinear, Store, Stored, pad_to, stored


@dataclass
class GatedDeltaSpec:
    heads: int
    kv_heads: int       # heads of q and k
    dim: int            # size of a q / k head
    vdim: int           # size of a v head
    conv: int           # taps of the short convolutions, the current token included
    decay_rank: int     # inner size of the decay's product
    gate_rank: int      # inner size of the output gate's product

    def __post_init__(self):
        if self.heads % self.kv_heads:
            raise ValueError(f"{self.heads} heads do not share {self.kv_heads} query / key heads evenly")
        if not 0 < self.dim <= OR.DELTA_MAX_DIM:
            raise ValueError(f"gated delta rule: key heads of {self.dim} (at most {OR.DELTA_MAX_DIM})")


class GatedDelta(Branch):
    def __init__(self, spec: GatedDeltaSpec, eps: float, dtype=None, device=None):
        super().__init__()
        self.spec, self.eps = spec, float(eps)
        s = spec
        self.k, self.v = pad_to(s.dim, 8), pad_to(s.vdim, 8)
        self.conv_width = 2 * s.kv_heads * self.k + s.heads * self.v
        self.b_width, self.a_rank, self.g_rank = pad_to(s.heads, 8), pad_to(s.decay_rank, 8), pad_to(s.gate_rank, 8)
        self.in_width = self.conv_width + self.b_width + self.a_rank + self.g_rank
        self.out_width = s.heads * self.v
        f32 = dict(dtype=torch.float32, device=device)
        self.decay_proj = PackedLinear(s.heads * self.k, self.a_rank, dtype=dtype, device=device)
        self.gate_proj = PackedLinear(s.heads * self.v, self.g_rank, dtype=dtype, device=device)
        self.conv_weight = nn.Parameter(torch.zeros((s.conv, self.conv_width), **f32))
        self.a_log = nn.Parameter(torch.zeros(s.heads, **f32))
        self.dt_bias = nn.Parameter(torch.zeros(s.heads * self.k, **f32))
        self.out_layernorm = nn.Parameter(torch.ones(self.v, **f32))

    def stored_tensors(self, w_in: torch.Tensor, w_out: torch.Tensor) -> Dict[str, Stored]:
        s, d = self.spec, w_in.shape[1]
        nk, nv = s.kv_heads * self.k, s.heads * self.v
        q, k, v, b, a1, g1 = w_in.split([nk, nk, nv, self.b_width, self.a_rank, self.g_rank])
        cq, ck, cv = self.conv_weight.data.split([nk, nk, nv], dim=1)

        def heads(w, n, padded, size):           # [n * padded, cols] -> the first `size` rows of every head
            return stored(w.view(n, padded, -1)[:, :size], n * size, w.shape[1])

        def taps(w, n, padded, size):            # [taps, n * padded] -> [n, size, taps]
            return stored(w.unflatten(1, (n, padded))[:, :, :size].permute(1, 2, 0), n * size, s.conv)

        return {
            "q": heads(q, s.kv_heads, self.k, s.dim), "q.conv": taps(cq, s.kv_heads, self.k, s.dim),
            "k": heads(k, s.kv_heads, self.k, s.dim), "k.conv": taps(ck, s.kv_heads, self.k, s.dim),
            "v": heads(v, s.heads, self.v, s.vdim), "v.conv": taps(cv, s.heads, self.v, s.vdim),
            "b": stored(b[:s.heads]), "A_log": stored(self.a_log.data), "norm": stored(self.out_layernorm.data[:s.vdim]),
            "a1": stored(a1[:s.decay_rank]),
            "a2": heads(self.decay_proj.weight.data[:, :s.decay_rank], s.heads, self.k, s.dim),
            "dt_bias": stored(self.dt_bias.data.view(s.heads, self.k)[:, :s.dim], s.heads * s.dim),
            "g1": stored(g1[:s.gate_rank]),
            "g2": heads(self.gate_proj.weight.data[:, :s.gate_rank], s.heads, self.v, s.vdim),
            "o": stored(w_out.unflatten(1, (s.heads, self.v))[:, :, :s.vdim], d, s.heads * s.vdim),
        }

    def native_symbols(self) -> List[str]:
        return ["icb_short_conv", "icb_delta_prepare"]

    def cache_spec(self) -> CacheSpec:
        s = self.spec
        return CacheSpec(states={"conv": ((s.conv - 1, self.conv_width), None),
                                 "rule": ((s.heads, self.v, OR.state_dim(self.k)), torch.float32)})

    def reset(self, generator: Optional[torch.Generator] = None) -> None:
        with torch.no_grad():
            self.a_log.copy_(torch.linspace(0.0, math.log(16.0), self.spec.heads))
            self.dt_bias.fill_(-4.0)
            self.conv_weight.zero_()
            self.conv_weight[-1].fill_(1.0)

    def forward(self, z, out, batch, store: Store, scale: float) -> None:
        s = self.spec
        sizes = dict(groups=s.kv_heads, heads=s.heads, dim=self.k, vdim=self.v)
        rows = OR.Rows.of(batch)
        x, beta, a1, g1 = z.split([self.conv_width, self.b_width, self.a_rank, self.g_rank], dim=1)
        x = OR.delta_prepare(x, self.conv_weight, store.states["conv"], beta[:, :s.heads],
                             self.decay_proj(a1, torch.float32), self.a_log, self.dt_bias, rows, q_scale=s.dim ** -0.5,
                             **sizes)
        o = OR.delta_rule(x, store.states["rule"], rows, **sizes)
        OR.delta_output(o, self.gate_proj(g1, torch.float32), self.out_layernorm, self.eps, scale, heads=s.heads,
                        vdim=self.v, valid=s.vdim, out=out)
