"""Attention over paged K / V caches: native kernels on CUDA, PyTorch restatements elsewhere (oracle / CPU path)."""

from __future__ import annotations

from typing import Optional

import torch

from . import native
from .native import call, dtype_code, ptr, stream_ptr

P, I, L, F = native.P, native.I, native.L, native.F
native.register("icb_kv_append", [P, P, P, P, P, I, I, L, L, P])
native.register("icb_paged_decode", [P, L, P, P, P, P, P, P, I, I, I, I, I, I, F, I, P, P, I, P, I, I, I, P, L])
_SMS = None


def _decode_splits(rows: int, groups: int, max_tokens: int) -> int:
    """Context ranges per (row, kv head) for the tensor-core decode kernel: enough CTAs for two per SM, at least four
    16-token steps per range."""
    global _SMS
    if _SMS is None:
        _SMS = torch.cuda.get_device_properties(torch.cuda.current_device()).multi_processor_count
    want = -(-2 * _SMS // max(1, rows * groups))
    return max(1, min(want, 8, max(1, max_tokens // 64)))


def kv_append(k: torch.Tensor, v: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, slots: torch.Tensor):
    """k, v: [T, hkv*hd] (row views with arbitrary pitch); caches [blocks, bs, hkv, hd]; slots int64 [T]."""
    t, row = k.shape
    if k.is_cuda and k.dtype in (torch.bfloat16, torch.float16):
        call("icb_kv_append", ptr(k), ptr(v), ptr(k_cache), ptr(v_cache), ptr(slots), t, row, k.stride(0), v.stride(0),
             stream_ptr())
        return
    kc = k_cache.view(-1, row)
    vc = v_cache.view(-1, row)
    ok = slots >= 0
    kc[slots[ok]] = k[ok]
    vc[slots[ok]] = v[ok]


def paged_decode_reference(q, k_cache, v_cache, block_table, seq_lens, hq, hkv, hd, scale):
    s = q.shape[0]
    bs = k_cache.shape[1]
    out = torch.zeros((s, hq * hd), dtype=q.dtype, device=q.device)
    g = hq // hkv
    for i in range(s):
        n = int(seq_lens[i])
        if n == 0:
            continue
        pages = (n + bs - 1) // bs
        blocks = block_table[i, :pages].long()
        k = k_cache[blocks].reshape(-1, hkv, hd)[:n].float()
        v = v_cache[blocks].reshape(-1, hkv, hd)[:n].float()
        qi = q[i].view(hq, hd).float()
        k = k.repeat_interleave(g, dim=1)
        v = v.repeat_interleave(g, dim=1)
        sc = torch.einsum("hd,nhd->hn", qi, k) * scale
        p = torch.softmax(sc, dim=-1)
        out[i] = torch.einsum("hn,nhd->hd", p, v).reshape(-1).to(q.dtype)
    return out


def mma_decode(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, block_table: torch.Tensor, lens: torch.Tensor,
               hq: int, hkv: int, hd: int, *, block_size: int, max_keys: int, scale: float, out: torch.Tensor,
               seqs: Optional[torch.Tensor] = None, len_bias: int = 0, window: int = 0, chunk: int = 0,
               gate: Optional[torch.Tensor] = None) -> torch.Tensor:
    """The tensor-core kernel (16-bit, head size 64 or 128): query row i (q [T, hq*hd], any 16-byte pitch) against the
    pages of sequence ``seqs[i]`` (None: i) up to position ``lens[i] + len_bias - 1``. ``out``: [T, hq*hd], any pitch.
    ``max_keys`` bounds how many keys a row sees."""
    t = q.shape[0]
    nsplit = _decode_splits(t, hkv * ((hq // hkv + 7) // 8), max_keys)
    scratch = torch.empty(max(1, t * hq * nsplit * (hd + 2) if nsplit > 1 else 1), dtype=torch.float32, device=q.device)
    call("icb_paged_decode", ptr(q), q.stride(0), ptr(k_cache), ptr(v_cache), ptr(block_table), ptr(lens), ptr(out), None,
         t, hq, hkv, hd, int(block_size), block_table.shape[1], float(scale), dtype_code(q.dtype), stream_ptr(),
         ptr(scratch), int(nsplit), ptr(seqs), int(len_bias), int(window), int(chunk), ptr(gate), out.stride(0))
    return out


def paged_decode(q: torch.Tensor, k_cache, v_cache, block_table, seq_lens, hq: int, hkv: int, hd: int,
                 scale: Optional[float] = None) -> torch.Tensor:
    """q: [S, hq*hd] (row view, any pitch) -> [S, hq*hd]: attention of one token per sequence over its pages."""
    scale = scale if scale is not None else hd ** -0.5
    s = q.shape[0]
    if q.is_cuda and q.dtype in (torch.bfloat16, torch.float16) and hd in (64, 128):
        out = torch.empty((s, hq * hd), dtype=q.dtype, device=q.device)
        if q.stride(0) % 8 == 0 and q.data_ptr() % 16 == 0:
            # tensor-core kernel (mma.sync over the GQA group), the context split over several CTAs
            return mma_decode(q, k_cache, v_cache, block_table, seq_lens, hq, hkv, hd, block_size=k_cache.shape[1],
                              max_keys=block_table.shape[1] * k_cache.shape[1], scale=scale, out=out)
        if hq // hkv <= 8:
            call("icb_paged_decode", ptr(q), q.stride(0), ptr(k_cache), ptr(v_cache), ptr(block_table), ptr(seq_lens),
                 ptr(out), None, s, hq, hkv, hd, k_cache.shape[1], block_table.shape[1], float(scale),
                 dtype_code(q.dtype), stream_ptr(), None, 0, None, 0, 0, 0, None, 0)
            return out
    return paged_decode_reference(q, k_cache, v_cache, block_table, seq_lens, hq, hkv, hd, scale)
