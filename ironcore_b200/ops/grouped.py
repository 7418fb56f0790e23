"""Grouped-head attention with rotary positions over a paged cache (``csrc/grouped_attention.cu``, the flash and the paged
decode kernels) and its PyTorch restatements.

CUDA tensors (bf16 or fp32) always take the kernels; the restatements are the CPU path and the oracle of the GPU tests."""

from __future__ import annotations

from typing import Optional

import torch

from . import native
from .functional import use_native
from .native import call, dtype_code, ptr, stream_ptr

P, I, L, F = native.P, native.I, native.L, native.F
native.register("icb_rope_cache", [P, L, P, P, P, P, P, I, P, F, I, I, I, I, I, I, P])
native.register("icb_attend_rows", [P, L, P, P, P, I, I, P, P, P, P, L, I, I, I, I, I, I, I, F, I, P])


def rotary_frequencies(dims: int, base: float) -> torch.Tensor:
    """Radians per position of every rotated pair, fp64 [dims / 2]: base^(-2 i / dims)."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    return float(base) ** (-2.0 * i / dims)


def first_visible(position: torch.Tensor, window: int, chunk: int) -> torch.Tensor:
    """First position that a query at ``position`` sees: a sliding window and / or fixed chunks (0: none)."""
    lo = torch.zeros_like(position)
    if window > 0:
        lo = torch.maximum(lo, position - window + 1)
    if chunk > 0:
        lo = torch.maximum(lo, position // chunk * chunk)
    return lo


def rope_cache(z: torch.Tensor, freq: torch.Tensor, positions: torch.Tensor, *, heads: int, groups: int, kd: int, vd: int,
               k_cache: torch.Tensor, v_cache: torch.Tensor, slots: torch.Tensor, gate_scale: Optional[float] = None
               ) -> Optional[torch.Tensor]:
    """z [T, >= (heads + groups) kd + groups vd (+ heads)]: [q | k | v | gate logits]. Rotates q and k in place (pairs
    (i, i + half) of every head by ``positions * freq``), writes keys and values to cache rows ``slots`` (negative:
    skip). With ``gate_scale`` returns ``gate_scale * sigmoid(logits)``, fp32 [T, heads]."""
    t, half = z.shape[0], freq.numel()
    if z.is_cuda:
        gate = torch.empty((t, heads), dtype=torch.float32, device=z.device) if gate_scale is not None else None
        call("icb_rope_cache", ptr(z), z.stride(0), ptr(k_cache), ptr(v_cache), ptr(slots), ptr(positions), ptr(freq), half,
             ptr(gate), float(gate_scale or 0.0), t, heads, groups, kd, vd, dtype_code(z.dtype), stream_ptr())
        return gate
    angle = positions.double()[:, None] * freq
    c, s = torch.cos(angle).float()[:, None], torch.sin(angle).float()[:, None]
    qk = z[:, :(heads + groups) * kd].view(t, heads + groups, kd)
    u, v = qk[..., :half].float(), qk[..., half:2 * half].float()
    qk[..., :half], qk[..., half:2 * half] = (u * c - v * s).to(z.dtype), (v * c + u * s).to(z.dtype)
    ok = slots >= 0
    base = (heads + groups) * kd
    k_cache[slots[ok]] = z[:, heads * kd:base][ok]
    v_cache[slots[ok]] = z[:, base:base + groups * vd][ok]
    if gate_scale is None:
        return None
    return gate_scale * torch.sigmoid(z[:, base + groups * vd:base + groups * vd + heads].float())


def attend_prompts(z: torch.Tensor, *, heads: int, groups: int, hd: int, cu_seqlens: torch.Tensor, max_len: int,
                   window: int, chunk: int, scale: float, gate: Optional[torch.Tensor], out: torch.Tensor) -> None:
    """Whole prompts out of the packed projection z [q | k | v] (head size hd for all) into ``out`` [T, heads * hd]."""
    nq, nk = heads * hd, groups * hd
    q, k, v = z[:, :nq], z[:, nq:nq + nk], z[:, nq + nk:nq + 2 * nk]
    if use_native(z):
        from . import attention as attn

        attn.flash_fwd_heads(q, k, v, heads, groups, hd, cu_seqlens, max_len, scale=scale, window=window, chunk=chunk,
                             gate=gate, out=out)
        return
    per = heads // groups
    bounds = cu_seqlens.tolist()
    for a, b in zip(bounds[:-1], bounds[1:]):
        idx = torch.arange(b - a, device=z.device)
        seen = (idx[None, :] <= idx[:, None]) & (idx[None, :] >= first_visible(idx, window, chunk)[:, None])
        qh = q[a:b].float().view(-1, heads, hd)
        kh = k[a:b].float().view(-1, groups, hd).repeat_interleave(per, 1)
        vh = v[a:b].float().view(-1, groups, hd).repeat_interleave(per, 1)
        s = torch.einsum("ihd,jhd->hij", qh, kh) * scale
        o = torch.einsum("hij,jhd->ihd", torch.softmax(s.masked_fill(~seen, float("-inf")), dim=-1), vh)
        out[a:b] = (o if gate is None else o * gate[a:b, :, None]).reshape(b - a, -1).to(out.dtype)


def attend_rows(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, table: torch.Tensor, block_size: int,
                seqs: torch.Tensor, positions: torch.Tensor, *, heads: int, groups: int, kd: int, vd: int, window: int,
                chunk: int, scale: float, max_keys: int, gate: Optional[torch.Tensor], out: torch.Tensor) -> None:
    """Query rows q [T, heads * kd] against the visible cache rows (k_cache [slots, groups * kd], v_cache [slots,
    groups * vd]) of sequences ``seqs`` up to ``positions``, into ``out`` [T, heads * vd]. ``max_keys`` bounds how many
    keys a row sees. 16-bit heads of 64 or 128 run on the tensor cores."""
    t = q.shape[0]
    if q.is_cuda:
        if use_native(q) and kd == vd and kd in (64, 128) and block_size % 16 == 0:
            from .paged import mma_decode

            mma_decode(q, k_cache, v_cache, table, positions, heads, groups, kd, block_size=block_size, max_keys=max_keys,
                       scale=scale, out=out, seqs=seqs, len_bias=1, window=window, chunk=chunk, gate=gate)
            return
        call("icb_attend_rows", ptr(q), q.stride(0), ptr(k_cache), ptr(v_cache), ptr(table), table.shape[1],
             int(block_size), ptr(seqs), ptr(positions), ptr(gate), ptr(out), out.stride(0), t, heads, groups, kd, vd,
             int(window), int(chunk), float(scale), dtype_code(q.dtype), stream_ptr())
        return
    per = heads // groups
    lo = first_visible(positions, window, chunk)
    for i in range(t):
        tok = torch.arange(int(lo[i]), int(positions[i]) + 1)
        rows = table[int(seqs[i]), tok // block_size].long() * block_size + tok % block_size
        k = k_cache[rows].float().view(-1, groups, kd).repeat_interleave(per, 1)
        v = v_cache[rows].float().view(-1, groups, vd).repeat_interleave(per, 1)
        p = torch.softmax(torch.einsum("hd,jhd->hj", q[i].float().view(heads, kd), k) * scale, dim=-1)
        o = torch.einsum("hj,jhd->hd", p, v)
        out[i] = (o if gate is None else o * gate[i, :, None]).reshape(-1).to(out.dtype)
