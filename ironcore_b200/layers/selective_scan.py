"""Selective-scan branch (Mamba): columns [x | z] of the shared input product; x passes a short convolution, a narrow product
makes step, B and C of it, and the scan kernel turns them into gated outputs. The state per sequence is the scan's (fp32) and
the last inputs of the convolution."""

from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional

import torch
import torch.nn as nn

from ..ops import recurrent as OR
from .mixer import Branch, CacheSpec, PackedLinear, Store, Stored, pad_to, stored


@dataclass
class SelectiveScanSpec:
    inner: int          # channels
    state: int          # states per channel
    dt_rank: int
    conv: int           # taps of the short convolution, the current token included

    def __post_init__(self):
        if min(self.inner, self.state, self.dt_rank, self.conv) < 1:
            raise ValueError(f"selective scan: sizes must be positive ({self})")
        OR.scan_lanes(self.state)      # refuses what the kernel cannot hold


class SelectiveScan(Branch):
    def __init__(self, spec: SelectiveScanSpec, dtype=None, device=None):
        super().__init__()
        self.spec = spec
        self.inner, self.rank, self.n = pad_to(spec.inner, 8), pad_to(spec.dt_rank, 8), pad_to(spec.state, 8)
        self.in_width, self.out_width = 2 * self.inner, self.inner
        f32 = dict(dtype=torch.float32, device=device)
        self.x_proj = PackedLinear(self.rank + 2 * self.n, self.inner, dtype=dtype, device=device)    # [step | B | C]
        self.dt_proj = PackedLinear(self.inner, self.rank, dtype=dtype, device=device)
        self.conv_weight = nn.Parameter(torch.zeros((spec.conv, self.inner), **f32))
        self.conv_bias = nn.Parameter(torch.zeros(self.inner, **f32))
        self.dt_bias = nn.Parameter(torch.zeros(self.inner, **f32))
        self.a_log = nn.Parameter(torch.zeros((self.inner, pad_to(spec.state, 4)), **f32))
        self.d = nn.Parameter(torch.zeros(self.inner, **f32))

    def stored_tensors(self, w_in: torch.Tensor, w_out: torch.Tensor) -> Dict[str, Stored]:
        s, x = self.spec, self.x_proj.weight.data
        d = w_in.shape[1]
        return {
            "in": stored(w_in.view(2, self.inner, d)[:, :s.inner], 2 * s.inner, d),
            "conv": stored(self.conv_weight.data[:, :s.inner].t()), "conv.b": stored(self.conv_bias.data[:s.inner]),
            "x": stored([x[lo:lo + n, :s.inner] for lo, n in ((0, s.dt_rank), (self.rank, s.state),
                                                              (self.rank + self.n, s.state))]),
            "dt": stored(self.dt_proj.weight.data[:s.inner, :s.dt_rank]), "dt.b": stored(self.dt_bias.data[:s.inner]),
            "A_log": stored(self.a_log.data[:s.inner, :s.state]), "D": stored(self.d.data[:s.inner]),
            "o": stored(w_out[:, :s.inner]),
        }

    def native_symbols(self) -> List[str]:
        return ["icb_short_conv", "icb_selective_scan"]

    def cache_spec(self) -> CacheSpec:
        return CacheSpec(states={"conv": ((self.spec.conv - 1, self.inner), None),
                                 "scan": ((self.inner, self.a_log.shape[1]), torch.float32)})

    def reset(self, generator: Optional[torch.Generator] = None) -> None:
        with torch.no_grad():
            self.a_log.copy_(torch.log(torch.arange(1, self.a_log.shape[1] + 1).float()).expand_as(self.a_log))
            self.d.fill_(1.0)
            self.dt_bias.fill_(-4.0)
            self.conv_weight.zero_()
            self.conv_weight[-1].fill_(1.0)

    def forward(self, z, out, batch, store: Store, scale: float) -> None:
        rows = OR.Rows.of(batch)
        u = OR.short_conv(z[:, :self.inner], self.conv_weight, self.conv_bias, store.states["conv"], rows)
        low = self.x_proj(u)
        dt = self.dt_proj(low[:, :self.rank], torch.float32)
        OR.selective_scan(u, dt, z[:, self.inner:], low, self.rank, self.rank + self.n, self.spec.state, self.dt_bias,
                          self.a_log, self.d, store.states["scan"], rows, out)
        if scale != 1.0:
            out.mul_(scale)

