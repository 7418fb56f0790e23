"""Recurrent mixers: short causal convolution, selective scan, gated delta rule (``csrc/short_conv.cu``,
``csrc/selective_scan.cu``, ``csrc/gated_delta.cu``) and their PyTorch restatements.

Every op takes the rows of many sequences at once (:class:`Rows`) and carries a fixed-size state per sequence slot: the
same call serves prompts, continued portions, one more token for each, and mixtures. A sequence at position 0 starts from
zeros whatever its slot holds. CUDA tensors (bf16 or fp32 activations) always take the kernels; the restatements are the
CPU path and the oracle of the GPU tests."""

from __future__ import annotations

from dataclasses import dataclass
from typing import Iterator, Optional, Tuple

import torch
import torch.nn.functional as TF

from . import native
from .native import call, dtype_code, ptr, stream_ptr

P, I, L, F = native.P, native.I, native.L, native.F
native.register("icb_short_conv", [P, L, P, P, P, P, P, P, I, P, L, I, I, I, I, P])
native.register("icb_selective_scan", [P, L, P, L, P, L, P, L, I, I, P, P, P, P, P, L, P, P, P, I, I, I, I, I, I, P])
native.register("icb_delta_prepare", [P, L, P, P, I, P, P, P, P, L, P, P, P, P, P, P, P, P, I, I, I, I, I, F, I, P])
native.register("icb_delta_rule", [P, P, P, P, P, P, P, P, P, P, P, I, I, I, I, I, I, I, P])
native.register("icb_delta_output", [P, P, L, P, F, F, P, L, I, I, I, I, I, P])

UNIT_EPS = 1e-6       # inside the root of the unit norms of the delta rule
DELTA_MAX_DIM = 256   # widest key head of the delta rule kernels
SCAN_MAX_STATE = 512  # most states per channel of the scan kernel


@dataclass
class Rows:
    """Rows of sequence slots ``seqs`` (int32 [T], a sequence's rows adjacent and in order) at ``positions`` (int32 [T]).
    ``cu`` (int32 [n + 1]) bounds them; None: every row is the only one of its sequence. ``longest``: most rows of one."""

    seqs: torch.Tensor
    positions: torch.Tensor
    cu: Optional[torch.Tensor]
    longest: int

    @staticmethod
    def of(batch) -> "Rows":
        if batch.kind == "decode":
            return Rows(batch.seqs, batch.positions, None, 1)
        return Rows(batch.seqs, batch.positions, batch.cu_seqlens, batch.max_len)

    @property
    def count(self) -> int:
        return self.seqs.numel() if self.cu is None else self.cu.numel() - 1

    def spans(self) -> Iterator[Tuple[int, int, int, bool]]:
        """(first row, end, slot, starts at position 0) of every sequence (CPU restatements)."""
        bounds = list(range(self.seqs.numel() + 1)) if self.cu is None else self.cu.tolist()
        for a, b in zip(bounds[:-1], bounds[1:]):
            if a < b:
                yield a, b, int(self.seqs[a]), int(self.positions[a]) == 0


def state_dim(dim: int) -> int:
    """Pitch of the delta rule's state along the key channels."""
    return (dim + 31) // 32 * 32 if dim <= 128 else (dim + 63) // 64 * 64


# --------------------------------------------------------------------------- short convolution
def short_conv(x: torch.Tensor, weight: torch.Tensor, bias: Optional[torch.Tensor], state: torch.Tensor, rows: Rows,
               want: bool = True) -> Optional[torch.Tensor]:
    """silu(causal convolution over time) per channel: x [T, C] (any pitch), weight fp32 [taps, C] (the last row is the
    current token's), bias fp32 [C] or None, state [slots, taps - 1, C]: the inputs that precede the rows, brought up to
    date. ``want=False``: the state only."""
    t, c = x.shape
    taps = weight.shape[0]
    if x.is_cuda:
        y = torch.empty((t, c), dtype=x.dtype, device=x.device) if want else None
        if want or rows.cu is not None:
            call("icb_short_conv", ptr(x), x.stride(0), ptr(weight), ptr(bias), ptr(state), ptr(rows.seqs),
                 ptr(rows.positions), ptr(rows.cu), rows.count, ptr(y), c, t, c, taps, dtype_code(x.dtype), stream_ptr())
        return y
    return _conv_reference(x, weight, bias, state, rows, keep=True)


def _conv_reference(x, weight, bias, state, rows, keep):
    taps = weight.shape[0]
    y = torch.empty(x.shape, dtype=x.dtype)
    for a, b, slot, fresh in rows.spans():
        past = torch.zeros_like(state[slot]) if fresh else state[slot]
        full = torch.cat([past, x[a:b]])
        out = TF.conv1d(full.float().t()[None], weight.t()[:, None], groups=x.shape[1])[0].t()
        y[a:b] = TF.silu(out if bias is None else out + bias).to(x.dtype)
        if keep and taps > 1:
            state[slot] = full[full.shape[0] - (taps - 1):].clone()
    return y


# --------------------------------------------------------------------------- selective scan
def scan_lanes(n: int) -> int:
    """States per lane of the scan kernel (a channel's states are spread over a power of two of lanes, sixteen at most):
    few idle lanes, several states per lane, since every lane also pays for the per-channel work, but not so many that the
    machine runs out of warps (measured: 8 of 16)."""
    best, cost = 0, float("inf")
    for ns in (8, 4, 12, 16, 32):
        lanes = 1
        while lanes * ns < n:
            lanes *= 2
        if lanes > 16:
            continue
        c = lanes * (ns + 3.0) + (16.0 if ns > 16 else 8.0 if ns > 8 else 0.0)
        if c < cost:
            best, cost = ns, c
    if best == 0:
        raise ValueError(f"selective scan: {n} states per channel (at most {SCAN_MAX_STATE})")
    return best


def selective_scan(u: torch.Tensor, dt: torch.Tensor, z: torch.Tensor, bc: torch.Tensor, b_col: int, c_col: int, n: int,
                   dt_bias: torch.Tensor, a_log: torch.Tensor, d: torch.Tensor, state: torch.Tensor, rows: Rows,
                   out: torch.Tensor, per_lane: Optional[int] = None) -> None:
    """out [T, C] = (sum_n S[n] C[n] + d u) silu(z) with S[n] <- exp(step A[n]) S[n] + step u B[n], step = softplus(dt +
    dt_bias), A = -exp(a_log). u, z [T, C]; dt fp32 [T, C]; bc [T, ...]: B in columns b_col .. + n, C in c_col .. + n;
    a_log [C, n rounded up to 4], state fp32 [slots, C, same]."""
    t, c = u.shape
    if u.is_cuda:
        call("icb_selective_scan", ptr(u), u.stride(0), ptr(dt), dt.stride(0), ptr(z), z.stride(0), ptr(bc), bc.stride(0),
             int(b_col), int(c_col), ptr(dt_bias), ptr(a_log), ptr(d), ptr(state), ptr(out), out.stride(0),
             ptr(rows.seqs), ptr(rows.positions), ptr(rows.cu), rows.count, rows.longest, c, int(n),
             per_lane or scan_lanes(n), dtype_code(u.dtype), stream_ptr())
        return
    a = -torch.exp(a_log[:, :n])
    step = TF.softplus(dt + dt_bias, threshold=1e9)
    uf, b, k = u.float(), bc[:, b_col:b_col + n].float(), bc[:, c_col:c_col + n].float()
    for lo, hi, slot, fresh in rows.spans():
        s = torch.zeros_like(a) if fresh else state[slot, :, :n].clone()
        for i in range(lo, hi):
            s = torch.exp(step[i][:, None] * a) * s + (step[i] * uf[i])[:, None] * b[i]
            out[i] = ((s @ k[i] + d * uf[i]) * TF.silu(z[i].float())).to(out.dtype)
        state[slot, :, :n] = s


# --------------------------------------------------------------------------- gated delta rule
@dataclass
class DeltaInputs:
    q: torch.Tensor       # fp32 [T, groups * dim], unit vectors times q_scale
    k: torch.Tensor       # fp32 [T, groups * dim], unit vectors
    qk: torch.Tensor      # fp32 [T, groups]
    decay: torch.Tensor   # fp32 [T, heads * dim]
    v: torch.Tensor       # [T, heads * vdim]
    beta: torch.Tensor    # fp32 [T, heads]


def delta_prepare(x: torch.Tensor, conv_weight: torch.Tensor, conv_state: torch.Tensor, beta_in: torch.Tensor,
                  a: torch.Tensor, a_log: torch.Tensor, dt_bias: torch.Tensor, rows: Rows, *, groups: int, heads: int,
                  dim: int, vdim: int, q_scale: float) -> DeltaInputs:
    """From projections to the recurrence's operands: x [T, 2 groups dim + heads vdim] = [q | k | v] through the short
    convolution (state as in :func:`short_conv`), unit norms of q and k per head, beta = sigmoid(beta_in), decay =
    exp(-exp(a_log) softplus(a + dt_bias)) (in the memory of ``a``, fp32 [T, heads dim])."""
    t = x.shape[0]
    f32 = dict(dtype=torch.float32, device=x.device)
    if x.is_cuda:
        o = DeltaInputs(torch.empty((t, groups * dim), **f32), torch.empty((t, groups * dim), **f32),
                        torch.empty((t, groups), **f32), a, torch.empty((t, heads * vdim), dtype=x.dtype, device=x.device),
                        torch.empty((t, heads), **f32))
        if not a.is_contiguous():
            raise ValueError("delta_prepare: the decay input must be contiguous")
        call("icb_delta_prepare", ptr(x), x.stride(0), ptr(conv_weight), ptr(conv_state), conv_weight.shape[0],
             ptr(rows.seqs), ptr(rows.positions), ptr(rows.cu), ptr(beta_in), beta_in.stride(0), ptr(a), ptr(a_log),
             ptr(dt_bias), ptr(o.q), ptr(o.k), ptr(o.qk), ptr(o.v), ptr(o.beta), t, groups, heads, dim, vdim,
             float(q_scale), dtype_code(x.dtype), stream_ptr())
        if rows.cu is not None:
            short_conv(x, conv_weight, None, conv_state, rows, want=False)
        return o
    # like the kernel, the convolved q and k go into their norms unrounded
    y = _conv_reference(x.float(), conv_weight, None, conv_state.float(), rows, keep=False)
    _conv_reference(x, conv_weight, None, conv_state, rows, keep=True)
    n = groups * dim

    def unit(m):
        m = m.view(t, groups, dim)
        return m / torch.sqrt(m.pow(2).sum(-1, keepdim=True) + UNIT_EPS)

    q, k = unit(y[:, :n]) * q_scale, unit(y[:, n:2 * n])
    rate = -torch.exp(a_log).repeat_interleave(dim)
    a.copy_(torch.exp(rate * TF.softplus(a + dt_bias, threshold=1e9)))
    return DeltaInputs(q.reshape(t, -1), k.reshape(t, -1), (q * k).sum(-1), a, y[:, 2 * n:].to(x.dtype),
                       torch.sigmoid(beta_in.float()))


def delta_rule(x: DeltaInputs, state: torch.Tensor, rows: Rows, *, groups: int, heads: int, dim: int,
               vdim: int) -> torch.Tensor:
    """Per head: S <- decay S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q. state fp32 [slots, heads, vdim,
    state_dim(dim)] (columns of S are its rows). Returns o, fp32 [T, heads * vdim]."""
    t = x.v.shape[0]
    o = torch.empty((t, heads * vdim), dtype=torch.float32, device=x.v.device)
    if x.v.is_cuda:
        call("icb_delta_rule", ptr(x.q), ptr(x.k), ptr(x.decay), ptr(x.qk), ptr(x.v), ptr(x.beta), ptr(state), ptr(o),
             ptr(rows.seqs), ptr(rows.positions), ptr(rows.cu), rows.count, rows.longest, groups, heads, dim, vdim,
             dtype_code(x.v.dtype), stream_ptr())
        return o
    per = heads // groups
    q = x.q.view(t, groups, dim).repeat_interleave(per, 1)
    k = x.k.view(t, groups, dim).repeat_interleave(per, 1)
    g, v = x.decay.view(t, heads, dim), x.v.float().view(t, heads, vdim)
    for lo, hi, slot, fresh in rows.spans():
        s = torch.zeros(heads, vdim, dim) if fresh else state[slot, :, :, :dim].clone()
        for i in range(lo, hi):
            s = s * g[i][:, None, :]
            u = x.beta[i][:, None] * (v[i] - torch.einsum("hvk,hk->hv", s, k[i]))
            s = s + u[:, :, None] * k[i][:, None, :]
            o[i] = torch.einsum("hvk,hk->hv", s, q[i]).reshape(-1)
        state[slot, :, :, :dim] = s
    return o


def delta_output(o: torch.Tensor, gate: torch.Tensor, weight: torch.Tensor, eps: float, scale: float, *, heads: int,
                 vdim: int, valid: int, out: torch.Tensor) -> None:
    """out [T, heads * vdim] = scale * sigmoid(gate) * weight * o / rms(o over the ``valid`` first values of a head; the
    others are zero). gate fp32 [T, heads * vdim], weight fp32 [vdim]."""
    t = o.shape[0]
    if o.is_cuda:
        call("icb_delta_output", ptr(o), ptr(gate), gate.stride(0), ptr(weight), float(eps), float(scale), ptr(out),
             out.stride(0), t, heads, vdim, int(valid), dtype_code(out.dtype), stream_ptr())
        return
    oh = o.view(t, heads, vdim)
    y = oh * torch.rsqrt(oh.pow(2).sum(-1, keepdim=True) / valid + eps) * weight * scale
    out.copy_((y * torch.sigmoid(gate[:, :heads * vdim].reshape(t, heads, vdim))).reshape(t, -1).to(out.dtype))
