"""Latent attention ops (``csrc/latent.cu``, the windowed flash kernel) and their PyTorch restatements.

CUDA tensors (bf16 or fp32) always take the kernels; the restatements are the CPU path and the oracle of the GPU
tests."""

from __future__ import annotations

from typing import Optional, Tuple

import torch

from . import kernels, native
from .functional import use_native
from .native import call, dtype_code, ptr, stream_ptr

P, I, L, F = native.P, native.I, native.L, native.F
native.register("icb_latent_norm", [P, L, P, P, P, I, P, P, P, P, I, I, I, I, I, F, I, P])
native.register("icb_head_product", [P, P, P, P, I, I, I, I, I, P])
native.register("icb_latent_attend", [P, P, P, P, P, P, P, I, I, I, I, I, I, F, I, I, P, L, P, I])

MMA_MAX_RANK = 512     # widest latent row of the tensor-core attention kernel


def project(x: torch.Tensor, weight: torch.Tensor, out_dtype: Optional[torch.dtype] = None,
            bias: Optional[torch.Tensor] = None, transposed: bool = False) -> torch.Tensor:
    """x [T, K] @ weight [N, K]^T (checkpoint orientation; ``transposed``: weight [K, N]) + bias -> [T, N] in
    ``out_dtype`` (default: x's)."""
    out_dtype = out_dtype or x.dtype
    if use_native(x):
        return (kernels.mm_nn if transposed else kernels.mm_nt)(x, weight, out_dtype=out_dtype, bias=bias)
    w = weight if transposed else weight.t()
    if x.dtype == torch.float32:
        tf32 = x.is_cuda and torch.backends.cuda.matmul.allow_tf32
        if tf32:
            torch.backends.cuda.matmul.allow_tf32 = False      # a 32-bit model is 32-bit, whatever training switched on
        try:
            y = x @ w
        finally:
            if tf32:
                torch.backends.cuda.matmul.allow_tf32 = True
        return y if bias is None else y + bias
    y = x.float() @ w.float()
    return (y if bias is None else y + bias.float()).to(out_dtype)


def latent_norm(z: torch.Tensor, q_weight: torch.Tensor, c_weight: torch.Tensor, heads: int, eps: float, *,
                q_width: int, c_width: int, dtype: torch.dtype, cache: Optional[torch.Tensor] = None,
                slots: Optional[torch.Tensor] = None, want_latent: bool = False
                ) -> Tuple[torch.Tensor, Optional[torch.Tensor], torch.Tensor]:
    """z [T, >= q_rank + rank + heads] fp32, columns [query latent | latent | head gates]. Returns (query latent
    [T, q_width], latent [T, c_width] or None, sigmoid of the gates fp32 [T, heads]), both latents RMS-normed; the
    latent also goes to rows ``slots`` (int64; negative: skip) of ``cache`` [rows, c_width]."""
    t, q_rank, rank = z.shape[0], q_weight.numel(), c_weight.numel()
    if z.is_cuda:
        cq = torch.empty((t, q_width), dtype=dtype, device=z.device)
        c = torch.empty((t, c_width), dtype=dtype, device=z.device) if want_latent else None
        gate = torch.empty((t, heads), dtype=torch.float32, device=z.device)
        call("icb_latent_norm", ptr(z), z.stride(0), ptr(q_weight), ptr(c_weight), ptr(cq), q_width, ptr(c), ptr(cache),
             ptr(slots), ptr(gate), t, q_rank, rank, c_width, heads, float(eps), dtype_code(dtype), stream_ptr())
        return cq, c, gate

    def norm(v, w, width):
        v = v * torch.rsqrt(v.pow(2).mean(-1, keepdim=True) + eps) * w
        return torch.nn.functional.pad(v, (0, width - v.shape[1])).to(dtype)

    cq = norm(z[:, :q_rank], q_weight, q_width)
    c = norm(z[:, q_rank:q_rank + rank], c_weight, c_width)
    gate = torch.sigmoid(z[:, q_rank + rank:q_rank + rank + heads])
    if cache is not None:
        ok = slots >= 0
        cache[slots[ok]] = c[ok]
    return cq, (c if want_latent else None), gate


def head_product(x: torch.Tensor, weight: torch.Tensor, gate: Optional[torch.Tensor] = None) -> torch.Tensor:
    """x [T, H, K], weight [H, N, K] -> [T, H, N], every head with its own matrix, times ``gate`` [T, H] if given."""
    t, h, k = x.shape
    n = weight.shape[1]
    if x.is_cuda:
        if not (x.is_contiguous() and weight.is_contiguous()):
            raise ValueError("head_product operands must be contiguous")
        out = torch.empty((t, h, n), dtype=x.dtype, device=x.device)
        call("icb_head_product", ptr(x), ptr(weight), ptr(out), ptr(gate), t, h, k, n, dtype_code(x.dtype), stream_ptr())
        return out
    y = torch.einsum("thk,hnk->thn", x.float(), weight.float())
    if gate is not None:
        y = y * gate[:, :, None]
    return y.to(x.dtype)


def _attend_splits(rows: int, heads: int, rank: int, max_keys: int, legacy: bool) -> int:
    """Ranges of keys per query row for the tensor-core kernels: as many CTAs as the machine holds at once (one per SM
    for tcgen05; two or three for mma.sync), each with at least two 128-key tiles."""
    sms = torch.cuda.get_device_properties(torch.cuda.current_device()).multi_processor_count
    groups = (heads + 31) // 32 if heads > 16 else 1
    slots = sms * ((2 if rank > 256 else 3) if legacy else 1)
    return max(1, min(slots // max(1, rows * groups), 32, max_keys // (128 if legacy else 256)))


def latent_attend(q: torch.Tensor, cache: torch.Tensor, block_table: torch.Tensor, block_size: int, seqs: torch.Tensor,
                  positions: torch.Tensor, *, window: int, scale: float, max_keys: int,
                  legacy: bool = False) -> torch.Tensor:
    """q [T, H, R] against latent cache rows [slots, R] -> [T, H, R]: softmax-weighted sum of the latents that row
    (``seqs`` int32, ``positions`` int32) sees. ``window`` <= 0: every earlier token. ``max_keys`` bounds how many
    keys any row sees. ``legacy``: mma.sync where tcgen05 would serve (CUDA, bf16)."""
    t, h, r = q.shape
    if q.is_cuda:
        out = torch.empty_like(q)
        nsplit, scratch = 1, None
        if q.dtype == torch.bfloat16 and r % 64 == 0 and r <= MMA_MAX_RANK:
            legacy = legacy or r % 128 != 0
            nsplit = _attend_splits(t, h, r, max_keys, legacy)
            if nsplit > 1:
                scratch = torch.empty(t * h * nsplit * (r + 2), dtype=torch.float32, device=q.device)
        call("icb_latent_attend", ptr(q), ptr(cache), ptr(block_table), ptr(seqs), ptr(positions), ptr(out),
             ptr(scratch), t, h, r, int(block_size), block_table.shape[1], int(window), float(scale), nsplit,
             dtype_code(q.dtype), stream_ptr(), cache.shape[0], ptr(native.status_tensor(q.device)), 1 if legacy else 0)
        return out
    out = torch.empty_like(q)
    for i in range(t):
        pos = int(positions[i])
        lo = max(0, pos - window + 1) if window > 0 else 0
        tok = torch.arange(lo, pos + 1)
        c = cache[block_table[int(seqs[i]), tok // block_size].long() * block_size + tok % block_size].float()
        p = torch.softmax(q[i].float() @ c.t() * scale, dim=-1)
        out[i] = (p @ c).to(q.dtype)
    return out


def prompt_attend(q: torch.Tensor, kv: torch.Tensor, heads: int, hd: int, cu_seqlens: torch.Tensor, max_len: int, *,
                  window: int, scale: float, gate: torch.Tensor) -> torch.Tensor:
    """Whole prompts: q [T, H * hd], kv [T, 2 * H * hd] -> gated head outputs [T, H * hd] (flash kernel on CUDA)."""
    if use_native(q):
        from . import attention as attn

        return attn.flash_fwd_window(q, kv, heads, hd, cu_seqlens, max_len, scale=scale, window=window, gate=gate)
    qh = q.float().view(-1, heads, hd)
    k, v = kv.float().view(-1, 2, heads, hd).unbind(1)
    out = torch.empty_like(qh)
    bounds = cu_seqlens.tolist()
    for a, b in zip(bounds[:-1], bounds[1:]):
        idx = torch.arange(b - a, device=q.device)
        dist = idx[:, None] - idx[None, :]
        seen = dist >= 0
        if window > 0:
            seen &= dist < window
        s = torch.einsum("ihd,jhd->hij", qh[a:b], k[a:b]) * scale
        p = torch.softmax(s.masked_fill(~seen, float("-inf")), dim=-1)
        out[a:b] = torch.einsum("hij,jhd->ihd", p, v[a:b])
    return (out * gate[:, :, None]).to(q.dtype).view(q.shape)
