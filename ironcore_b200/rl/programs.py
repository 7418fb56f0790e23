"""Step programs: how a model family evaluates one :class:`StepBatch` over its cache.

A program owns the choice of cache and ``logits(batch)``; sequences, pages, graphs, batching and sampling are the
engine's. ``make_program`` picks by the model's family."""

from __future__ import annotations

from typing import Optional

import torch
import torch.distributed as dist

from ..ops import functional as OF
from ..ops import kernels
from ..parallel import mesh
from . import ops as RO
from .batch import StepBatch
from .kv_cache import BlockKVCache


def _all_reduce(x, group):
    if group is not None and dist.is_initialized() and dist.get_world_size(group) > 1:
        dist.all_reduce(x, group=group)
    return x


class TransformerProgram:
    """The unified transformer on the block KV cache. Prompts run the flash attention kernel on the packed projections
    and scatter the rotated K / V rows into cache pages; all other rows append and attend over their pages. Tensor
    parallelism uses the plain (non sequence-parallel) layout, one all-reduce after each row-parallel projection."""

    def __init__(self, model, config, max_seqs: int, max_seq_len: int, block_size: Optional[int],
                 num_blocks: Optional[int]):
        self.model, self.config = model, config
        m = config.model
        block_size = block_size or config.rl.kv_block_size
        self.tp_group = mesh.get_tensor_model_parallel_group()
        self.tp = mesh.get_tensor_model_parallel_world_size()
        self.tp_rank = mesh.get_tensor_model_parallel_rank()
        self.hq = m.num_attention_heads // self.tp
        self.hkv = (m.num_attention_groups or m.num_attention_heads) // self.tp
        self.hd, self.d = m.head_dim, m.d_model
        self.layers = list(model.model.layers)
        first = next(model.parameters())
        blocks = num_blocks or max_seqs * ((max_seq_len + block_size - 1) // block_size)
        self.cache = BlockKVCache(len(self.layers), self.hkv, self.hd, blocks, block_size, max_seqs, max_seq_len,
                                  first.dtype, first.device)

    def refresh(self):
        pass

    # ------------------------------------------------------------------ building blocks
    def _embed(self, ids_2d: torch.Tensor, pos_ids: Optional[torch.Tensor] = None) -> torch.Tensor:
        emb = self.model.embedding
        w = emb.word_embeddings
        pt = emb.position_embedding.weight if emb.position_embedding is not None else None
        if self.tp > 1:
            x = OF.embedding(ids_2d, w.weight, vocab_start=w.vocab_start, pos_table=pt if self.tp_rank == 0 else None,
                             pos_ids=pos_ids)
            x = _all_reduce(x.reshape(-1, self.d).contiguous(), self.tp_group)
        else:
            x = OF.embedding(ids_2d, w.weight, pos_table=pt, pos_ids=pos_ids).reshape(-1, self.d)
        if emb.scale is not None:
            x = x * emb.scale
        return x

    def _row_parallel(self, lin, x, residual):
        if self.tp == 1:
            return OF.linear(x, lin.weight, lin.bias, residual)
        y = OF.linear(x, lin.weight, None)
        y = _all_reduce(y, self.tp_group)
        if lin.bias is not None:
            y = y + lin.bias
        return y + residual if residual is not None else y

    def _mlp(self, layer, x, residual):
        mlp = layer.mlp
        if getattr(layer, "is_moe", False):
            out, _aux = mlp(x, residual=residual)
            return out
        h = mlp.activation(OF.linear(x, mlp.up_proj.weight, mlp.up_proj.bias))
        return self._row_parallel(mlp.down_proj, h, residual)

    def _layer(self, li: int, layer, x, attend):
        n1 = layer.input_layernorm(x)
        qkv = OF.linear(n1, layer.linear_qkv.weight, layer.linear_qkv.bias)
        ctx = attend(li, layer, qkv)
        if layer.parallel_block:
            a = self._row_parallel(layer.attn_output, ctx, x)
            return self._mlp(layer, n1, a)
        res1 = n1 if layer.post_ln else x
        x = self._row_parallel(layer.attn_output, ctx, res1)
        n2 = layer.post_attn_layernorm(x)
        res2 = n2 if layer.post_ln else x
        return self._mlp(layer, n2, res2)

    def _rope_inplace(self, layer, qkv, tokens: int, seq_len: int, pos_ids):
        rot = layer.rotary_pos_emb
        if rot is None:
            return qkv
        if OF.use_native(qkv) and rot.rot_dim % 2 == 0:
            kernels.rope(qkv, qkv, nheads=self.hq + self.hkv, head_dim=self.hd, tokens=tokens, seq_len=seq_len,
                         base=rot.base, scale=rot.scaling_factor, offset=rot.offset, interleaved=rot.interleaved,
                         pos_ids=pos_ids, row_stride=qkv.stride(0), out_stride=qkv.stride(0), rot_dim=rot.rot_dim)
            return qkv
        return OF.rope_reference_packed(qkv, self.hq, self.hkv, self.hd, seq_len, rot.base, rot.scaling_factor,
                                        rot.offset, rot.interleaved, rot.rot_dim, pos_ids)

    def _head(self, x):
        x = self.model.output_layernorm(x)
        if self.model.untied:
            ol = self.model.output_layer
            return OF.linear(x, ol.weight, ol.bias)
        from ..models.language_model import linear_t

        return linear_t(x, self.model.embedding.word_embeddings.weight)

    # ------------------------------------------------------------------ one step
    def logits(self, batch: StepBatch) -> torch.Tensor:
        cache = self.cache
        t = batch.tokens.numel()
        q_cols = self.hq * self.hd
        kv_cols = self.hkv * self.hd
        prompt = batch.kind == "prompt"
        if prompt:
            seq_len = batch.max_len if batch.uniform else t
            cu = None if batch.uniform else batch.cu_seqlens
        else:
            seq_len, cu = 1, None
            tables = cache.block_table[batch.seqs.long()]
            lens = batch.positions + 1
        pos = None if prompt and batch.uniform else batch.positions

        def attend(li, layer, qkv):
            qkv = self._rope_inplace(layer, qkv, t, seq_len, pos)
            RO.kv_append(qkv[:, q_cols:q_cols + kv_cols], qkv[:, q_cols + kv_cols:], cache.k[li], cache.v[li],
                         batch.slots)
            if prompt:
                return OF.rope_attention(qkv, num_heads=self.hq, num_kv_heads=self.hkv, head_dim=self.hd,
                                         seq_len=seq_len, rope=None, causal=True, cu_seqlens=cu,
                                         fused=self.config.trainer.use_flash_attn)
            return RO.paged_decode(qkv[:, :q_cols], cache.k[li], cache.v[li], tables, lens, self.hq, self.hkv, self.hd)

        if prompt and batch.uniform:
            x = self._embed(batch.tokens.view(-1, seq_len))
        else:
            learned = self.model.embedding.position_embedding is not None
            x = self._embed(batch.tokens.view(1, -1), batch.positions.view(1, -1) if learned else None)
        for li, layer in enumerate(self.layers):
            x = self._layer(li, layer, x, attend)
        if batch.want is not None:
            if batch.want.numel() == 0:
                return torch.empty((0, self.model.padded_vocab_size // self.tp), dtype=x.dtype, device=x.device)
            x = x[batch.want.long()]
        return self._head(x)


class StreamProgram:
    """Residual-stream models: a :class:`LayerCache` of whatever the mixers keep, fp32 logits. Pages hold 64 tokens unless
    asked otherwise: a latent row is narrow, and its decode kernel copies a page with one box per 64 columns."""

    PAGE = 64

    def __init__(self, model, config, max_seqs: int, max_seq_len: int, block_size: Optional[int],
                 num_blocks: Optional[int]):
        self.model = model
        table = model.embedding.word_embeddings.weight
        self.cache = model.model.make_cache(max_seqs, max_seq_len, block_size or self.PAGE, num_blocks,
                                            device=table.device, dtype=table.dtype)

    def refresh(self):
        self.model.model.refresh()

    def logits(self, batch: StepBatch) -> torch.Tensor:
        return self.model.step_logits(batch, self.cache)


def make_program(model, config, **kw):
    from ..models.families import STREAM_FAMILIES

    return (StreamProgram if model.family in STREAM_FAMILIES else TransformerProgram)(model, config, **kw)
