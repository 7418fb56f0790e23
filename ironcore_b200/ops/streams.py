"""Residual streams: the fused sublayer boundary (``csrc/streams.cu``) and its PyTorch restatement.

A boundary writes a finished sublayer's result into the streams, reads the next sublayer's input out of them, applies
the grouped RMS norm and, where asked for, the token shift; see :func:`boundary`. CUDA tensors (bf16 or fp32
activations) always take the kernel; the restatement is the CPU path and the kernel's oracle in the GPU tests."""

from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

import torch

from . import native
from .native import call, dtype_code, ptr, stream_ptr

P, I, L, F = native.P, native.I, native.L, native.F
native.register("icb_stream_boundary", [P, P, L, L, F, P, P, P, P, L, P, L, P, P, P, P, P, P, I, F, P, P, L, P, P, P, P, P,
                                        I, I, I, I, I, P])


@dataclass
class StreamWrite:
    """What is written into the streams at a boundary: the sublayer's result ``y`` [T, >=D], optionally gated by
    ``sigmoid(gate + gate_bias)``, with the stream weights ``mix`` [S, S] ([from, to]) and ``out`` [S]. ``streams``
    are the values before it, fp32 [T, S, D]."""

    streams: torch.Tensor
    y: torch.Tensor
    gate: Optional[torch.Tensor]
    gate_bias: Optional[torch.Tensor]
    mix: torch.Tensor
    out: torch.Tensor


@dataclass
class TokenEmbed:
    """What the streams start from: row ``tokens[i]`` of ``table`` times ``scale`` in every stream."""

    tokens: torch.Tensor
    table: torch.Tensor
    scale: float
    streams: int


@dataclass
class StreamAdd:
    """What every stream gets on top where a pass of a looped block starts: ``vector`` fp32 [D] and, if given, the rows
    of ``embed``."""

    vector: torch.Tensor
    embed: Optional[TokenEmbed] = None


@dataclass
class TokenShift:
    """Blend of a row with the previous token's: ``weight`` [D]; ``prev`` / ``state`` fp32 [slots, D] are the last
    value of every sequence before / after this batch (one tensor may serve as both if no sequence has more than one
    row here); ``seqs`` / ``positions`` int32 [T]."""

    weight: torch.Tensor
    prev: torch.Tensor
    state: torch.Tensor
    seqs: torch.Tensor
    positions: torch.Tensor


def boundary(source, read: torch.Tensor, norm_weight: torch.Tensor, groups: int, eps: float, *, width: int,
             dtype: torch.dtype, shift: Optional[TokenShift] = None, rows: Optional[torch.Tensor] = None,
             keep_streams: bool = True, add: Optional[StreamAdd] = None) -> Tuple[Optional[torch.Tensor], torch.Tensor, Optional[torch.Tensor]]:
    """``source`` is a :class:`StreamWrite` or a :class:`TokenEmbed`. Returns (streams, h, shifted h): the streams
    after the write and ``add`` (None without ``keep_streams``), ``h`` [T, width] = grouped RMS norm of ``sum_s read[s] x_s`` and,
    with ``shift``, its token-shifted form. ``rows`` (int32) selects rows of the source. ``width`` >= D pads with
    zeros."""
    first = isinstance(source, TokenEmbed)
    device = source.tokens.device if first else source.streams.device
    if device.type != "cuda":
        return _boundary_reference(source, read, norm_weight, groups, eps, width, dtype, shift, rows, keep_streams, add)
    d = norm_weight.numel()
    s = source.streams if first else source.streams.shape[1]
    total = rows.numel() if rows is not None else (source.tokens.numel() if first else source.streams.shape[0])
    h = torch.empty((total, width), dtype=dtype, device=device)
    hs = torch.empty_like(h) if shift is not None else None
    x_out = torch.empty((total, s, d), dtype=torch.float32, device=device) if keep_streams else None
    embed = source if first else (add.embed if add is not None else None)
    if first and add is not None and add.embed is not None:
        raise ValueError("stream boundary: the embedding is where the streams start, it cannot be added there too")
    table = embed.table if embed is not None else None
    y = None if first else source.y
    gate = None if first else source.gate
    for t in (table, y, gate):
        if t is not None and (t.dtype != dtype or t.stride(-1) != 1):
            raise ValueError("stream boundary: table, y and gate share the activation dtype and have contiguous rows")
    call("icb_stream_boundary", ptr(embed.tokens) if embed is not None else None, ptr(table),
         table.stride(0) if table is not None else 0, table.shape[0] if table is not None else 0,
         float(embed.scale) if embed is not None else 0.0, ptr(add.vector) if add is not None else None,
         None if first else ptr(source.streams), ptr(x_out), ptr(y),
         0 if first else y.stride(0), ptr(gate), gate.stride(0) if gate is not None else 0,
         None if gate is None else ptr(source.gate_bias), None if first else ptr(source.mix),
         None if first else ptr(source.out), ptr(rows), ptr(read), ptr(norm_weight), int(groups), float(eps), ptr(h),
         ptr(hs), int(width), ptr(shift.weight) if shift else None, ptr(shift.prev) if shift else None,
         ptr(shift.state) if shift else None, ptr(shift.seqs) if shift else None,
         ptr(shift.positions) if shift else None, int(total), int(s), int(d), 0, dtype_code(dtype), stream_ptr())
    return x_out, h, hs


def grouped_rms_norm_reference(x: torch.Tensor, weight: torch.Tensor, groups: int, eps: float) -> torch.Tensor:
    parts = x.unflatten(-1, (groups, -1))
    parts = parts * torch.rsqrt(parts.pow(2).mean(-1, keepdim=True) + eps)
    return parts.flatten(-2) * weight


def _boundary_reference(source, read, norm_weight, groups, eps, width, dtype, shift, rows, keep_streams, add):
    d = norm_weight.numel()
    if isinstance(source, TokenEmbed):
        x = (source.table[source.tokens, :d].float() * source.scale).unsqueeze(1).expand(-1, source.streams, -1)
    else:
        y = source.y[:, :d].float()
        if source.gate is not None:
            y = y * torch.sigmoid(source.gate[:, :d].float() + source.gate_bias)
        x = torch.einsum("st,nsd->ntd", source.mix, source.streams) + source.out[:, None] * y[:, None]
    if add is not None:
        if add.embed is not None:
            x = x + (add.embed.table[add.embed.tokens, :d].float() * add.embed.scale).unsqueeze(1)
        x = x + add.vector
    if rows is not None:
        x = x[rows.long()]
    h = grouped_rms_norm_reference(torch.einsum("s,nsd->nd", read, x), norm_weight, groups, eps)
    hs = None
    if shift is not None:
        seqs = shift.seqs.long()
        starts = torch.ones(h.shape[0], dtype=torch.bool)
        starts[1:] = seqs[1:] != seqs[:-1]
        ends = torch.ones_like(starts)
        ends[:-1] = starts[1:]
        before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
        carried = shift.prev[seqs] * (shift.positions > 0)[:, None]
        before = torch.where(starts[:, None], carried, before)
        hs = h + (before - h) * shift.weight
        shift.state[seqs[ends]] = h[ends]

    def pad(t):
        return torch.nn.functional.pad(t, (0, width - d)).to(dtype)

    return (x.contiguous() if keep_streams else None), pad(h), (pad(hs) if hs is not None else None)
