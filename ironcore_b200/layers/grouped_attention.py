"""Attention branch: grouped key / value heads, (partial) rotary positions, a sliding window or fixed chunks, one output
gate per head.

Columns of the shared input product: [q | k | v | gate logits]. One kernel rotates, fills the cache and turns the logits
into factors; whole prompts then run the flash kernel on the packed columns, other rows the paged decode kernel, both
writing gated head outputs in place for the output product. In 16-bit, head sizes are padded once to the kernels' 64 or 128
(the padding is zero and changes no result)."""

from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List

import torch

from ..ops import grouped as OG
from ..ops.functional import use_native
from .mixer import Branch, CacheSpec, Store, Stored, pad_to, stored


@dataclass
class GroupedAttentionSpec:
    heads: int
    kv_heads: int
    dim: int            # query / key size of a head
    vdim: int           # value size of a head
    scale: float        # score factor
    rot_dims: int       # leading elements of a head that rotate
    rot_base: float
    window: int = 0     # visible tokens including the token itself; 0: no limit
    chunk: int = 0      # visible: the token's own chunk of this many tokens; 0: no chunks

    def __post_init__(self):
        if self.heads % self.kv_heads:
            raise ValueError(f"{self.heads} query heads do not share {self.kv_heads} key / value heads evenly")
        if self.rot_dims % 2 or self.rot_dims > self.dim:
            raise ValueError(f"rotary dimensions ({self.rot_dims}) must be even and within the head ({self.dim})")


class GroupedAttention(Branch):
    def __init__(self, spec: GroupedAttentionSpec, dtype=None, device=None):
        super().__init__()
        self.spec = s = spec
        dtype = dtype or torch.get_default_dtype()
        widest = max(s.dim, s.vdim)
        self.fast = dtype in (torch.bfloat16, torch.float16) and widest <= 128
        if self.fast:
            self.kd = self.vd = 64 if widest <= 64 else 128
        else:
            self.kd, self.vd = pad_to(s.dim, 8), pad_to(s.vdim, 8)
        self.qkv_width = (s.heads + s.kv_heads) * self.kd + s.kv_heads * self.vd
        self.in_width = self.qkv_width + pad_to(s.heads, 8)
        self.out_width = s.heads * self.vd
        self.register_buffer("freq", OG.rotary_frequencies(s.rot_dims, s.rot_base).to(device or "cpu"), persistent=False)

    def stored_tensors(self, w_in: torch.Tensor, w_out: torch.Tensor) -> Dict[str, Stored]:
        s, d = self.spec, w_in.shape[1]
        q, k, v, g, _ = w_in.split([s.heads * self.kd, s.kv_heads * self.kd, s.kv_heads * self.vd, s.heads,
                                    self.in_width - self.qkv_width - s.heads])
        return {
            "q": stored(q.view(s.heads, self.kd, d)[:, :s.dim], s.heads * s.dim, d),
            "k": stored(k.view(s.kv_heads, self.kd, d)[:, :s.dim], s.kv_heads * s.dim, d),
            "v": stored(v.view(s.kv_heads, self.vd, d)[:, :s.vdim], s.kv_heads * s.vdim, d),
            "g": stored(g),
            "o": stored(w_out.unflatten(1, (s.heads, self.vd))[:, :, :s.vdim], d, s.heads * s.vdim),
        }

    def native_symbols(self) -> List[str]:
        return ["icb_rope_cache", "icb_attend_rows"] + (["icb_flash_fwd", "icb_paged_decode"] if self.fast else [])

    def cache_spec(self) -> CacheSpec:
        s = self.spec
        return CacheSpec(rows={"k": s.kv_heads * self.kd, "v": s.kv_heads * self.vd}, window=s.window, chunk=s.chunk)

    def max_keys(self, context: int) -> int:
        """Most keys that one row sees."""
        return min([context] + [n for n in (self.spec.window, self.spec.chunk) if n > 0])

    def forward(self, z, out, batch, store: Store, scale: float) -> None:
        s = self.spec
        sizes = dict(heads=s.heads, groups=s.kv_heads)
        mask = dict(window=s.window, chunk=s.chunk, scale=s.scale)
        gate = OG.rope_cache(z, self.freq, batch.positions, kd=self.kd, vd=self.vd, k_cache=store.rows["k"],
                             v_cache=store.rows["v"], slots=batch.slots, gate_scale=scale, **sizes)
        if batch.kind == "prompt" and self.fast and (use_native(z) or not z.is_cuda):
            OG.attend_prompts(z, hd=self.kd, cu_seqlens=batch.cu_seqlens, max_len=batch.max_len, gate=gate, out=out, **sizes,
                              **mask)
        else:
            OG.attend_rows(z[:, :s.heads * self.kd], store.rows["k"], store.rows["v"], store.block_table, store.block_size,
                           batch.seqs, batch.positions, kd=self.kd, vd=self.vd, max_keys=self.max_keys(batch.max_context),
                           gate=gate, out=out, **sizes, **mask)
