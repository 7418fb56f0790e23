"""What a mixer keeps per layer run, and mixers made of branches that share their products.

A *branch* is one way to mix tokens (attention, a recurrence). It does not own its input and output projections: it says
how many columns it reads from the shared input product and writes for the shared output product, and where its checkpoint
tensors are inside the two weights. :class:`BranchMixer` owns those, so that several branches that read the same input cost
one product in and one product out; a branch folds its weight in the sum into what it writes."""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, List, NamedTuple, Optional, Sequence, Tuple

import torch
import torch.nn as nn

from ..ops import latent as OL


def pad_to(n: int, unit: int) -> int:
    return (n + unit - 1) // unit * unit


class Stored(NamedTuple):
    """A checkpoint tensor inside (padded, packed) parameters: views of its values, one after the other along its first
    dimension, and its stored shape."""

    views: Tuple[torch.Tensor, ...]
    shape: Tuple[int, ...]

    def put(self, t: torch.Tensor) -> None:
        for view, part in zip(self.views, t.split([v.shape[0] for v in self.views]) if len(self.views) > 1 else (t,)):
            view.copy_(part.reshape(view.shape))

    def value(self) -> torch.Tensor:
        return (self.views[0] if len(self.views) == 1 else torch.cat(self.views)).reshape(self.shape)


def stored(view, *shape: int) -> Stored:
    """``view`` a tensor, or a sequence of tensors stacked along their first dimension; ``shape`` if it is not theirs."""
    views = (view,) if isinstance(view, torch.Tensor) else tuple(view)
    return Stored(views, tuple(shape) or (sum(v.shape[0] for v in views), *views[0].shape[1:]))


class PackedLinear(nn.Module):
    """A weight in checkpoint orientation [out, in] whose rows and columns may be padded or hold several matrices."""

    def __init__(self, rows: int, cols: int, dtype=None, device=None, bias: bool = False):
        super().__init__()
        self.weight = nn.Parameter(torch.zeros((rows, cols), dtype=dtype, device=device))
        self.bias = nn.Parameter(torch.zeros(rows, dtype=dtype, device=device)) if bias else None

    def forward(self, x: torch.Tensor, out_dtype: Optional[torch.dtype] = None) -> torch.Tensor:
        return OL.project(x, self.weight, out_dtype, self.bias)


@dataclass
class CacheSpec:
    """What one layer run keeps: ``rows`` name -> width of a row per token; ``states`` name -> (shape per sequence, dtype or
    None for the activations'); and how far back its rows are read (``window`` tokens / the token's own ``chunk``, 0: to
    the first token)."""

    rows: Dict[str, int] = field(default_factory=dict)
    states: Dict[str, Tuple[Tuple[int, ...], Optional[torch.dtype]]] = field(default_factory=dict)
    window: int = 0
    chunk: int = 0

    def visible_from(self, position: int) -> Optional[int]:
        """First token whose rows a token at ``position`` reads; None without rows."""
        if not self.rows:
            return None
        lo = 0
        if self.window > 0:
            lo = max(lo, position - self.window + 1)
        if self.chunk > 0:
            lo = max(lo, position // self.chunk * self.chunk)
        return lo


class Branch(nn.Module):
    """Subclasses set ``in_width`` / ``out_width`` (multiples of 8) and implement the rest."""

    in_width: int
    out_width: int

    def stored_tensors(self, w_in: torch.Tensor, w_out: torch.Tensor) -> Dict[str, Stored]:
        """Checkpoint name -> place; ``w_in`` [in_width, D] and ``w_out`` [D, out_width] are this branch's slices."""
        raise NotImplementedError

    def cache_spec(self) -> CacheSpec:
        raise NotImplementedError

    def native_symbols(self) -> List[str]:
        """Entry points of the kernel library that it calls."""
        raise NotImplementedError

    def reset(self, generator: Optional[torch.Generator] = None) -> None:
        """Starting values that a normal distribution does not fit."""

    def forward(self, z: torch.Tensor, out: torch.Tensor, batch, store: "Store", scale: float) -> None:
        """z [T, in_width] (may be changed) -> out [T, out_width], times ``scale``."""
        raise NotImplementedError


@dataclass
class Store:
    """A branch's part of a cache at one layer run."""

    rows: Dict[str, torch.Tensor]
    states: Dict[str, torch.Tensor]
    block_table: torch.Tensor
    block_size: int


class BranchMixer(nn.Module):
    """Weighted sum of branches: ``branches`` is a list of (checkpoint prefix, branch, weight in the sum)."""

    def __init__(self, d_model: int, branches: Sequence[Tuple[str, Branch, float]], dtype=None, device=None):
        super().__init__()
        self.d_model = d_model
        width = pad_to(d_model, 8)
        self.prefixes = [p for p, _, _ in branches]
        self.branches = nn.ModuleList([b for _, b, _ in branches])
        self.scales = [float(s) for _, _, s in branches]
        kw = dict(dtype=dtype, device=device)
        self.in_proj = PackedLinear(sum(b.in_width for b in self.branches), width, **kw)
        self.out_proj = PackedLinear(width, sum(b.out_width for b in self.branches), **kw)

    def _slices(self):
        i = o = 0
        for prefix, b, s in zip(self.prefixes, self.branches, self.scales):
            yield prefix, b, s, slice(i, i + b.in_width), slice(o, o + b.out_width)
            i, o = i + b.in_width, o + b.out_width

    def stored_tensors(self) -> Dict[str, Stored]:
        out = {}
        for prefix, b, _, i, o in self._slices():
            places = b.stored_tensors(self.in_proj.weight.data[i, :self.d_model], self.out_proj.weight.data[:self.d_model, o])
            out.update({prefix + k: v for k, v in places.items()})
        return out

    def cache_spec(self) -> CacheSpec:
        spec = CacheSpec()
        for prefix, b in zip(self.prefixes, self.branches):
            part = b.cache_spec()
            spec.rows.update({prefix + k: v for k, v in part.rows.items()})
            spec.states.update({prefix + k: v for k, v in part.states.items()})
            if part.rows:
                if len(spec.rows) > len(part.rows) and (spec.window, spec.chunk) != (part.window, part.chunk):
                    spec.window = spec.chunk = 0        # rows of several reaches: keep all
                else:
                    spec.window, spec.chunk = part.window, part.chunk
        return spec

    def native_symbols(self) -> List[str]:
        return [name for b in self.branches for name in b.native_symbols()]

    def reset(self, generator: Optional[torch.Generator] = None) -> None:
        for b in self.branches:
            b.reset(generator)

    def forward(self, h: torch.Tensor, batch, cache, run: int) -> torch.Tensor:
        """h [T, width] -> [T, width]."""
        z = self.in_proj(h)
        ctx = torch.empty((h.shape[0], self.out_proj.weight.shape[1]), dtype=h.dtype, device=h.device)
        rows, states = cache.rows[run], cache.states[run]
        for prefix, b, scale, i, o in self._slices():
            store = Store({k[len(prefix):]: v for k, v in rows.items() if k.startswith(prefix)},
                          {k[len(prefix):]: v for k, v in states.items() if k.startswith(prefix)}, cache.block_table,
                          cache.block_size)
            b(z[:, i], ctx[:, o], batch, store, scale)
        return self.out_proj(ctx)
