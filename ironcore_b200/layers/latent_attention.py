"""Latent attention (no rotary part): queries, keys and values are expanded from low-rank latents, and a token's
normalised key/value latent is all that the cache keeps.

The mixer reads one input row ``h``. ``in_proj`` yields [query latent | latent | one gate logit per head] in one
product; both latents are RMS-normed. Two evaluations of the same attention:

* whole prompts expand keys and values from the latents of the batch and run the windowed flash kernel;
* decoding (and any other query rows) moves the per-head expansion matrices to the query and the output side and
  attends over cached latents: ``score = (K_n^T q_n) . c``, ``out = V_n sum_j p_j c_j``.

Widths are padded once, at construction: head sizes to the flash kernel's 64 or 128, latent rows to a multiple of 64,
matrix pitches to 16 bytes. The padding is zero and changes no result. ``stored_tensors`` gives the unpadded ones."""

from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List

import torch
import torch.nn as nn

from ..ops import latent as OL
from ..ops.functional import use_native
from .mixer import CacheSpec, PackedLinear, Stored, pad_to, stored


@dataclass
class LatentAttentionSpec:
    heads: int
    dim: int            # query / key size of a head
    vdim: int           # value size of a head
    q_rank: int
    kv_rank: int
    scale: float        # score factor
    window: int         # visible tokens including the token itself; 0 = all earlier tokens

    @staticmethod
    def from_mixer(mixer: dict) -> "LatentAttentionSpec":
        mask = mixer.get("mask") or {}
        return LatentAttentionSpec(heads=int(mixer["heads"]), dim=int(mixer["dim"]), vdim=int(mixer["vdim"]),
                                   q_rank=int(mixer["q_rank"]), kv_rank=int(mixer["kv_rank"]),
                                   scale=float(mixer["scale"]), window=int(mask.get("size") or 0))


class LatentAttention(nn.Module):
    def __init__(self, d_model: int, spec: LatentAttentionSpec, eps: float, dtype=None, device=None):
        super().__init__()
        self.spec, self.eps, self.d_model = spec, float(eps), d_model
        if max(spec.dim, spec.vdim) <= 128:
            self.qd = self.vd = 64 if max(spec.dim, spec.vdim) <= 64 else 128
        else:
            self.qd, self.vd = pad_to(spec.dim, 64), pad_to(spec.vdim, 64)
        self.flash = self.qd == self.vd and self.qd in (64, 128)
        self.q_width, self.c_width = pad_to(spec.q_rank, 8), pad_to(spec.kv_rank, 64)
        width = pad_to(d_model, 8)
        kw = dict(dtype=dtype, device=device)
        self.in_proj = PackedLinear(pad_to(spec.q_rank + spec.kv_rank + spec.heads, 8), width, **kw)
        self.q_up = PackedLinear(spec.heads * self.qd, self.q_width, **kw)
        self.kv_up = PackedLinear(spec.heads * (self.qd + self.vd), self.c_width, **kw)
        self.out = PackedLinear(width, spec.heads * self.vd, **kw)
        self.q_layernorm = nn.Parameter(torch.ones(spec.q_rank, dtype=torch.float32, device=device))
        self.c_layernorm = nn.Parameter(torch.ones(spec.kv_rank, dtype=torch.float32, device=device))
        self._absorb, self._absorb_of = None, None

    # ------------------------------------------------------------------ weights
    def stored_tensors(self) -> Dict[str, Stored]:
        """Checkpoint name -> where its values are."""
        s, d = self.spec, self.d_model
        w_in = self.in_proj.weight.data[:, :d]
        split = s.heads * self.qd
        kv = self.kv_up.weight.data
        return {
            "dq": stored(w_in[:s.q_rank]), "dkv": stored(w_in[s.q_rank:s.q_rank + s.kv_rank]),
            "g": stored(w_in[s.q_rank + s.kv_rank:s.q_rank + s.kv_rank + s.heads]),
            "dq.norm": stored(self.q_layernorm.data), "dkv.norm": stored(self.c_layernorm.data),
            "uq": stored(self.q_up.weight.data.view(s.heads, self.qd, -1)[:, :s.dim, :s.q_rank],
                         s.heads * s.dim, s.q_rank),
            "uk": stored(kv[:split].view(s.heads, self.qd, -1)[:, :s.dim, :s.kv_rank], s.heads * s.dim, s.kv_rank),
            "uv": stored(kv[split:].view(s.heads, self.vd, -1)[:, :s.vdim, :s.kv_rank], s.heads * s.vdim, s.kv_rank),
            "o": stored(self.out.weight.data.view(-1, s.heads, self.vd)[:d, :, :s.vdim], d, s.heads * s.vdim),
        }

    def native_symbols(self) -> List[str]:
        fast = self.out.weight.dtype in (torch.bfloat16, torch.float16)
        return ["icb_latent_norm"] + (["icb_flash_fwd"] if fast and self.flash else [])

    def cache_spec(self) -> CacheSpec:
        return CacheSpec(rows={"latent": self.c_width}, window=self.spec.window)

    def refresh(self) -> torch.Tensor:
        """[heads, c_width, qd]: the key expansion transposed for the query side, rebuilt in place (captured graphs
        keep its address) when ``kv_up`` has changed."""
        w = self.kv_up.weight
        key = (w._version, w.data_ptr())
        if self._absorb_of != key:
            fresh = w.data[:self.spec.heads * self.qd].view(self.spec.heads, self.qd, -1).transpose(1, 2)
            if self._absorb is None or self._absorb.device != w.device or self._absorb.dtype != w.dtype:
                self._absorb = fresh.contiguous()
            else:
                self._absorb.copy_(fresh)
            self._absorb_of = key
        return self._absorb

    # ------------------------------------------------------------------ compute
    def forward(self, h: torch.Tensor, batch, cache, run: int) -> torch.Tensor:
        """h [T, width] -> [T, width]; the latents of ``batch``'s tokens go to layer run ``run`` of ``cache``."""
        s = self.spec
        whole = batch.kind == "prompt" and self.flash and (use_native(h) or not h.is_cuda)
        z = self.in_proj(h, torch.float32)
        cq, c, gate = OL.latent_norm(z, self.q_layernorm, self.c_layernorm, s.heads, self.eps, q_width=self.q_width,
                                     c_width=self.c_width, dtype=h.dtype, cache=cache.rows[run]["latent"], slots=batch.slots,
                                     want_latent=whole)
        q = self.q_up(cq)
        if whole:
            ctx = OL.prompt_attend(q, self.kv_up(c), s.heads, self.qd, batch.cu_seqlens, batch.max_len,
                                   window=s.window, scale=s.scale, gate=gate)
        else:
            q = OL.head_product(q.view(-1, s.heads, self.qd), self.refresh())
            keys = min(s.window, batch.max_context) if s.window > 0 else batch.max_context
            o = OL.latent_attend(q, cache.rows[run]["latent"], cache.block_table, cache.block_size, batch.seqs,
                                 batch.positions, window=s.window, scale=s.scale, max_keys=keys)
            v_up = self.kv_up.weight.data[s.heads * self.qd:].view(s.heads, self.vd, -1)
            ctx = OL.head_product(o, v_up, gate).reshape(h.shape[0], -1)
        return self.out(ctx)
