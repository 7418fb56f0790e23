"""Rollout engine: requests, batches and sampling over a family's step program and paged cache.

One step (:meth:`RolloutEngine.step`) runs the tokens it is given, for any set of requests: whole prompts of different
lengths as one packed batch, one more token for each of several running requests, or any mixture. Requests own a cache
sequence from their first token until they are ended. A decode step over ``n`` requests runs on static buffers and is
captured in a CUDA graph the second time a batch of that size comes by (launch-bound regime: dozens of small kernels
per layer). :meth:`RolloutEngine.generate` is the sampling loop on top.
(The reference only has a cache-less sampler that re-runs the whole prefix for every token:
examples/generate_text.py:12-46.)
"""

from __future__ import annotations

from collections import OrderedDict
from typing import Dict, Hashable, List, Optional, Sequence, Tuple, Union

import torch

from ..ops import native
from ..parallel import mesh
from .batch import StepBatch
from .programs import make_program
from .sampling import sample_tokens

MAX_GRAPHS = 8          # captured decode steps kept at a time, one per batch size


class _DecodeGraph:
    """Static inputs and, once captured, the replayable step of one batch size."""

    def __init__(self, n: int, device):
        self.tokens = torch.zeros(n, dtype=torch.int64, device=device)
        self.seqs = torch.zeros(n, dtype=torch.int32, device=device)
        self.bound = None            # the sequences ``seqs`` holds
        self.graph = None
        self.logits = None
        self.launches = 0


class RolloutEngine:
    def __init__(self, model, config, max_seqs: int, max_seq_len: int, block_size: Optional[int] = None,
                 use_cuda_graph: Optional[bool] = None, num_blocks: Optional[int] = None):
        self.model, self.config = model, config
        self.tp_group = mesh.get_tensor_model_parallel_group()
        self.tp = mesh.get_tensor_model_parallel_world_size()
        self.tp_rank = mesh.get_tensor_model_parallel_rank()
        self.device = next(model.parameters()).device
        self.program = make_program(model, config, max_seqs=max_seqs, max_seq_len=max_seq_len,
                                    block_size=block_size, num_blocks=num_blocks)
        self.cache = self.program.cache
        self.max_seqs = max_seqs
        on_gpu = self.device.type == "cuda"
        self.use_graph = on_gpu if use_cuda_graph is None else (use_cuda_graph and on_gpu)
        self._graphs: "OrderedDict[int, _DecodeGraph]" = OrderedDict()
        self._requests: Dict[Hashable, int] = {}

    # ------------------------------------------------------------------ requests
    def end(self, ids) -> None:
        """Forget requests; what they hold in the cache is given back."""
        for i in ids:
            self.cache.release(self._requests.pop(i))

    @torch.no_grad()
    def step(self, entries: Sequence[Tuple[Hashable, Sequence[int], Optional[Sequence[int]]]]) -> torch.Tensor:
        """``entries``: (request id, its next tokens, places among them whose logits are wanted; None = the last).
        An unknown id starts a request. Returns logits [wanted, V_local] in entry order, in a buffer that the next
        step may overwrite."""
        vocab = self.model.vocab_size
        wants, base = [], 0
        for rid, tokens, want in entries:
            n = len(tokens)
            if n == 0:
                raise ValueError(f"request {rid!r}: a step needs at least one token")
            if min(tokens) < 0 or max(tokens) >= vocab:
                raise ValueError(f"request {rid!r}: token ids must be in [0, {vocab})")
            places = [n - 1] if want is None else list(want)
            if any(not 0 <= p < n for p in places):
                raise ValueError(f"request {rid!r}: wanted places must be in [0, {n})")
            wants += [base + p for p in places]
            base += n
        ids = [e[0] for e in entries]
        if len(set(ids)) != len(ids):
            raise ValueError("a request may appear once in a step")
        flat = [t for _, tokens, _ in entries for t in tokens]
        counts = [len(tokens) for _, tokens, _ in entries]
        fresh = []
        try:
            for i in ids:
                if i not in self._requests:
                    self._requests[i] = self.cache.acquire()
                    fresh.append(i)
            seqs = [self._requests[i] for i in ids]
            if not fresh and max(counts) == 1:
                logits = self._decode(seqs, torch.tensor(flat, dtype=torch.int64))
                return logits if wants == list(range(len(ids))) else logits[wants]
            return self._rows(seqs, counts, torch.tensor(flat, dtype=torch.int64), wants)
        except Exception:
            self.end(fresh)
            raise

    # ------------------------------------------------------------------ batches
    def _make_room(self, seqs: List[int], counts: List[int]):
        cache = self.cache
        for s in seqs:
            cache.drop_before(s, cache.visible_from(cache.length(s)))
        cache.reserve_many((s, cache.length(s) + n) for s, n in zip(seqs, counts))

    def _rows(self, seqs: List[int], counts: List[int], tokens: torch.Tensor, want: Optional[List[int]]) -> torch.Tensor:
        """Prompts and everything else that is not one token for each of several running requests."""
        cache, dev = self.cache, self.device
        self._make_room(seqs, counts)
        starts = [cache.length(s) for s in seqs]
        n = torch.tensor(counts)
        row_seq = torch.tensor(seqs).repeat_interleave(n)
        offset = torch.tensor(starts) - torch.cat([torch.zeros(1, dtype=torch.int64), n.cumsum(0)[:-1]])
        row_pos = torch.arange(int(n.sum())) + offset.repeat_interleave(n)
        cu = torch.cat([torch.zeros(1, dtype=torch.int64), n.cumsum(0)]).to(torch.int32)
        seq_dev, pos_dev = row_seq.to(dev, torch.int32), row_pos.to(dev, torch.int32)
        batch = StepBatch(kind="prompt" if not any(starts) else "extend", tokens=tokens.to(dev), seqs=seq_dev,
                          positions=pos_dev, slots=cache.slots_for(seq_dev, pos_dev), max_len=max(counts),
                          max_context=max(s + c for s, c in zip(starts, counts)), cu_seqlens=cu.to(dev),
                          uniform=len(set(counts)) == 1,
                          want=None if want is None else torch.tensor(want, dtype=torch.int32, device=dev))
        logits = self.program.logits(batch)
        cache.seq_lens[torch.tensor(seqs, device=dev)] = torch.tensor([s + c for s, c in zip(starts, counts)],
                                                                      dtype=torch.int32, device=dev)
        for s, start, c in zip(seqs, starts, counts):
            cache.advance(s, start + c)
        return logits

    def _decode_body(self, tokens: torch.Tensor, seqs: torch.Tensor) -> torch.Tensor:
        cache = self.cache
        index = seqs.long()
        pos = cache.seq_lens[index]
        batch = StepBatch(kind="decode", tokens=tokens, seqs=seqs, positions=pos, slots=cache.slots_for(index, pos),
                          max_len=1, max_context=cache.max_seq_len)
        logits = self.program.logits(batch)
        cache.seq_lens[index] = pos + 1
        return logits

    def _decode(self, seqs: List[int], tokens: torch.Tensor) -> torch.Tensor:
        """One more token for every sequence; the logits may be a static buffer that the next call overwrites."""
        n = len(seqs)
        self._make_room(seqs, [1] * n)
        for s in seqs:
            self.cache.advance(s, self.cache.length(s) + 1)
        g = self._graphs.get(n)
        if g is None:
            g = self._graphs[n] = _DecodeGraph(n, self.device)
            while len(self._graphs) > MAX_GRAPHS:
                self._drop_graph(next(iter(self._graphs)))
        self._graphs.move_to_end(n)
        if g.bound != seqs:
            g.seqs.copy_(torch.tensor(seqs, dtype=torch.int32))
            warm, g.bound = g.bound is not None, list(seqs)
        else:
            warm = True
        g.tokens.copy_(tokens)
        if not self.use_graph or not warm:
            return self._decode_body(g.tokens, g.seqs)
        if g.graph is None:
            # an eager step of this size has run before: lazily set kernel attributes and derived weights are in place
            torch.cuda.synchronize()
            before = native.launches()
            g.graph = torch.cuda.CUDAGraph()
            with torch.cuda.graph(g.graph):
                g.logits = self._decode_body(g.tokens, g.seqs)
            g.launches = native.launches() - before
            native.add_launches(-g.launches)
        g.graph.replay()
        native.add_launches(g.launches)
        return g.logits

    def _drop_graph(self, n: int):
        g = self._graphs.pop(n)
        if g.graph is not None:
            torch.cuda.synchronize()

    def release_graph(self):
        """Drop the captured decode steps (and their static buffers); later decode steps capture again."""
        if any(g.graph is not None for g in self._graphs.values()):
            torch.cuda.synchronize()
        self._graphs.clear()
        import gc

        gc.collect()

    # ------------------------------------------------------------------ generation
    def _sample(self, logits, temperature, top_k, top_p, generator):
        vocab_local = self.model.padded_vocab_size // self.tp
        start = self.tp_rank * vocab_local
        valid = max(0, min(vocab_local, self.model.vocab_size - start))
        return sample_tokens(logits, temperature, top_k, top_p, generator, vocab_start=start, vocab_valid=valid,
                             group=self.tp_group if self.tp > 1 else None)

    @torch.no_grad()
    def generate(self, prompts: Union[torch.Tensor, Sequence[Sequence[int]]],
                 max_new_tokens: Union[int, Sequence[int]], temperature: float = 1.0, top_k: int = 0,
                 top_p: float = 1.0, generator: Optional[torch.Generator] = None,
                 stop_token: Optional[int] = None):
        """Sample continuations of a batch of prompts.

        ``prompts`` [S, P]: returns (tokens [S, P + N] including the prompt, log-probs of the N sampled tokens
        [S, N]). A list of token lists may be unequal, with one ``max_new_tokens`` or one per prompt and an optional
        ``stop_token``; it runs in waves of up to ``max_seqs`` prompts whose requests leave the batch as they finish,
        and returns (list of sampled tokens, list of their log-probs)."""
        was_training = self.model.training
        self.model.eval()
        self.program.refresh()
        try:
            if isinstance(prompts, torch.Tensor):
                if stop_token is not None or not isinstance(max_new_tokens, int):
                    raise ValueError("stop_token and per-prompt lengths need a list of prompts")
                return self._generate_uniform(prompts, max_new_tokens, temperature, top_k, top_p, generator)
            limits = [max_new_tokens] * len(prompts) if isinstance(max_new_tokens, int) else list(max_new_tokens)
            out, logps = [], []
            for lo in range(0, len(prompts), self.max_seqs):
                t, lp = self._generate_wave(prompts[lo:lo + self.max_seqs], limits[lo:lo + self.max_seqs], temperature,
                                            top_k, top_p, generator, stop_token)
                out += t
                logps += lp
            return out, logps
        finally:
            if was_training:
                self.model.train()

    def _acquire(self, n: int) -> List[int]:
        return [self.cache.acquire() for _ in range(n)]

    def _generate_uniform(self, prompts, max_new_tokens, temperature, top_k, top_p, generator):
        s, p = prompts.shape
        out = torch.empty((s, p + max_new_tokens), dtype=torch.int64, device=self.device)
        out[:, :p] = prompts.to(self.device)
        logps = torch.empty((s, max_new_tokens), dtype=torch.float32, device=self.device)
        if max_new_tokens == 0:
            return out, logps
        seqs = self._acquire(s)
        try:
            logits = self._rows(seqs, [p] * s, out[:, :p].reshape(-1), [(i + 1) * p - 1 for i in range(s)])
            for i in range(max_new_tokens):
                tok, lp = self._sample(logits, temperature, top_k, top_p, generator)
                out[:, p + i] = tok
                logps[:, i] = lp
                if i + 1 < max_new_tokens:
                    logits = self._decode(seqs, tok)
        finally:
            for q in reversed(seqs):
                self.cache.release(q)
        return out, logps

    def _generate_wave(self, prompts, limits, temperature, top_k, top_p, generator, stop_token):
        n = len(prompts)
        tokens: List[List[int]] = [[] for _ in range(n)]
        logps: List[List[float]] = [[] for _ in range(n)]
        live = [i for i in range(n) if limits[i] > 0]
        if not live:
            return tokens, logps
        logits = self.step([(("wave", i), prompts[i], None) for i in live])
        while live:
            tok, lp = self._sample(logits, temperature, top_k, top_p, generator)
            done = []
            for i, t, p in zip(live, tok.tolist(), lp.tolist()):
                tokens[i].append(t)
                logps[i].append(p)
                if len(tokens[i]) >= limits[i] or t == stop_token:
                    done.append(i)
            self.end([("wave", i) for i in done])
            live = [i for i in live if i not in done]
            if live:
                logits = self.step([(("wave", i), [tokens[i][-1]], None) for i in live])
        return tokens, logps
