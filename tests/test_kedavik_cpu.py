"""The Kedavik family (selective scan, chunked rotary attention beside a gated delta rule, looped layers) on CPU against the
plain restatement: every mechanism alone, then the model through the rollout engine in every way a sequence can be cut and
batched."""

import json
import os
import subprocess
import sys

import pytest
import torch

import gated_state_oracle as oracle
import kedavik_cases as K

CASES = K.cases()
TIGHT = 3e-5      # fp32 against the 64-bit restatement
F64 = torch.float64


def _rand(*shape, seed=0, scale=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale


def _rows(*spans):
    """Rows of (slot, first position, count) spans."""
    from ironcore_b200.ops.recurrent import Rows

    seqs = torch.cat([torch.full((n,), s, dtype=torch.int32) for s, _, n in spans])
    pos = torch.cat([torch.arange(p, p + n, dtype=torch.int32) for _, p, n in spans])
    cu = torch.tensor([0] + list(torch.tensor([n for _, _, n in spans]).cumsum(0)), dtype=torch.int32)
    return Rows(seqs, pos, cu, max(n for _, _, n in spans))


def _decode_rows(*pairs):
    from ironcore_b200.ops.recurrent import Rows

    return Rows(torch.tensor([s for s, _ in pairs], dtype=torch.int32), torch.tensor([p for _, p in pairs], dtype=torch.int32),
                None, 1)


# ------------------------------------------------------------------ mechanisms
@pytest.mark.parametrize("taps", [1, 2, 4, 7])
def test_short_convolution_over_portions_and_slots(taps):
    from ironcore_b200.ops import recurrent as OR

    c, n = 8, 13
    x, y, w, b = _rand(n, c), _rand(n, c, seed=1), _rand(taps, c, seed=2), _rand(c, seed=3)
    want = oracle.causal_conv(x.double(), w.t().double(), b.double())
    other = oracle.causal_conv(y.double(), w.t().double(), b.double())
    for cuts in ([13], [2] * 7, [1] * 13, [5, 1, 7]):
        state = torch.full((3, taps - 1, c), 7.0)            # leftovers of whoever had the slot before
        got, got2, lo = [], [], 0
        for k in cuts:
            k = min(k, n - lo)
            if k == 0:
                continue
            rows = _rows((2, lo, k), (0, lo, k)) if k > 1 else _decode_rows((2, lo), (0, lo))
            out = OR.short_conv(torch.cat([x[lo:lo + k], y[lo:lo + k]]), w, b, state, rows)
            got.append(out[:k])
            got2.append(out[k:])
            lo += k
        assert torch.allclose(torch.cat(got).double(), want, atol=1e-5), cuts
        assert torch.allclose(torch.cat(got2).double(), other, atol=1e-5), cuts
        assert bool((state[1] == 7.0).all())


@pytest.mark.parametrize("n", [1, 6, 16])
def test_selective_scan_carries_its_state(n):
    from ironcore_b200.ops import recurrent as OR

    c, t = 16, 11
    u, z, dt = _rand(t, c), _rand(t, c, seed=1), _rand(t, c, seed=2)
    bias, a_log, d = _rand(c, seed=3), _rand(c, (n + 3) // 4 * 4, seed=4), _rand(c, seed=5)
    width = (n + 7) // 8 * 8
    bc = _rand(t, 8 + 2 * width, seed=6)
    step = oracle.softplus(dt.double() + bias.double())
    y = oracle.selective_scan(u.double(), step, -torch.exp(a_log[:, :n].double()), bc[:, 8:8 + n].double(),
                              bc[:, 8 + width:8 + width + n].double(), d.double())
    want = y * oracle.silu(z.double())
    for cuts in ([11], [2, 9], [1] * 11):
        state = torch.full((2, *a_log.shape), 3.0)
        out, lo = torch.empty(t, c), 0
        for k in cuts:
            rows = _rows((1, lo, k)) if k > 1 else _decode_rows((1, lo))
            s = slice(lo, lo + k)
            OR.selective_scan(u[s], dt[s], z[s], bc[s], 8, 8 + width, n, bias, a_log, d, state, rows, out[s])
            lo += k
        assert torch.allclose(out.double(), want, atol=1e-4), cuts


@pytest.mark.parametrize("heads,groups,dim,vdim", [(1, 1, 8, 8), (4, 2, 16, 24), (3, 3, 24, 8)])
def test_gated_delta_rule_carries_its_state(heads, groups, dim, vdim):
    from ironcore_b200.ops import recurrent as OR

    t, taps, per = 10, 3, heads // groups
    conv = 2 * groups * dim + heads * vdim
    x, cw = _rand(t, conv), _rand(taps, conv, seed=1)
    b, a = _rand(t, heads, seed=2), _rand(t, heads * dim, seed=3)
    a_log, dt_bias = _rand(heads, seed=4) * 0.3, _rand(heads * dim, seed=5) - 1
    gate, w = _rand(t, heads * vdim, seed=6), _rand(vdim, seed=7)
    mixed = oracle.causal_conv(x.double(), cw.t().double())
    q, k, v = mixed.split([groups * dim, groups * dim, heads * vdim], dim=1)
    want = []
    for h in range(heads):
        g = h // per
        qh = torch.stack([oracle.unit(r) * dim ** -0.5 for r in q[:, g * dim:(g + 1) * dim]])
        kh = torch.stack([oracle.unit(r) for r in k[:, g * dim:(g + 1) * dim]])
        decay = torch.stack([oracle.channel_decay(a[i].double().view(heads, dim), a_log.double(),
                                                  dt_bias.double().view(heads, dim))[h] for i in range(t)])
        o = oracle.delta_rule(qh, kh, v[:, h * vdim:(h + 1) * vdim], torch.sigmoid(b[:, h].double()), decay)
        want.append(torch.stack([oracle.rms_norm(r, w.double(), 1e-3) for r in o])
                    * torch.sigmoid(gate[:, h * vdim:(h + 1) * vdim].double()) * 0.7)
    want = torch.cat(want, 1)
    sizes = dict(groups=groups, heads=heads, dim=dim, vdim=vdim)
    for cuts in ([10], [2, 2, 6], [1] * 10):
        conv_state = torch.full((2, taps - 1, conv), 5.0)
        state = torch.full((2, heads, vdim, OR.state_dim(dim)), 4.0)
        got, lo = [], 0
        for n in cuts:
            rows = _rows((1, lo, n)) if n > 1 else _decode_rows((1, lo))
            s = slice(lo, lo + n)
            ins = OR.delta_prepare(x[s], cw, conv_state, b[s], a[s].clone(), a_log, dt_bias, rows, q_scale=dim ** -0.5, **sizes)
            o = OR.delta_rule(ins, state, rows, **sizes)
            out = torch.empty(n, heads * vdim)
            OR.delta_output(o, gate[s], w, 1e-3, 0.7, heads=heads, vdim=vdim, valid=vdim, out=out)
            got.append(out)
            lo += n
        assert torch.allclose(torch.cat(got).double(), want, atol=2e-4), cuts


@pytest.mark.parametrize("dims", [2, 6, 8])
def test_partial_rotary_and_cache_rows(dims):
    from ironcore_b200.ops import grouped as OG

    t, heads, groups, kd, vd = 4, 4, 2, 8, 16
    z = _rand(t, (heads + groups) * kd + groups * vd + 8)
    before = z.clone()
    pos = torch.tensor([0, 3, 70, 4001], dtype=torch.int32)
    slots = torch.tensor([5, -1, 0, 2])
    kc, vc = torch.zeros(6, groups * kd), torch.zeros(6, groups * vd)
    gate = OG.rope_cache(z, OG.rotary_frequencies(dims, 300.0), pos, heads=heads, groups=groups, kd=kd, vd=vd, k_cache=kc,
                         v_cache=vc, slots=slots, gate_scale=0.6)
    for i in range(t):
        for h in range(heads + groups):
            want = oracle.rotate(before[i, h * kd:(h + 1) * kd].double(), int(pos[i]), dims, 300.0)
            assert torch.allclose(z[i, h * kd:(h + 1) * kd].double(), want, atol=1e-5)
        if slots[i] >= 0:
            assert torch.equal(kc[slots[i]], z[i, heads * kd:(heads + groups) * kd])
            assert torch.equal(vc[slots[i]], before[i, (heads + groups) * kd:(heads + groups) * kd + groups * vd])
    assert torch.equal(kc[[1, 3, 4]], torch.zeros(3, groups * kd))
    off = (heads + groups) * kd + groups * vd
    assert torch.allclose(gate, 0.6 * torch.sigmoid(before[:, off:off + heads]))


@pytest.mark.parametrize("chunk", [1, 4, 16, 17, 0])
def test_chunk_edges_of_the_cached_attention(chunk):
    """One key stands out at a time: it decides the result exactly while the chunk holds it, at page borders too."""
    from ironcore_b200.ops import grouped as OG

    bs, n, r = 16, 40, 8
    table = torch.tensor([[2, 0, 1]], dtype=torch.int32)          # pages out of order
    for pos in (0, 3, 4, 15, 16, 17, 33, 34, 39):
        lo = pos // chunk * chunk if chunk else 0
        for j in {0, max(0, lo - 1), lo, max(0, pos - 1), pos}:
            kc, vc = torch.zeros(3 * bs, r), torch.zeros(3 * bs, r)
            rows = [int(table[0, t // bs]) * bs + t % bs for t in range(n)]
            kc[rows] = _rand(n, r, seed=3) * 0.1
            kc[rows[j]] = torch.eye(r)[0] * 5
            vc[rows[j]] = 1.0
            out = torch.empty(1, r)
            OG.attend_rows(torch.eye(r)[:1] * 8, kc, vc, table, bs, torch.zeros(1, dtype=torch.int32),
                           torch.tensor([pos], dtype=torch.int32), heads=1, groups=1, kd=r, vd=r, window=0, chunk=chunk,
                           scale=1.0, max_keys=n, gate=None, out=out)
            assert (float(out[0, 0]) > 0.9) == oracle.visible(pos, j, chunk or None), (chunk, pos, j)


def test_windows_and_chunks_compose_and_bound_the_cache():
    from ironcore_b200.layers.mixer import CacheSpec
    from ironcore_b200.ops import grouped as OG
    from ironcore_b200.rl.kv_cache import LayerCache

    pos = torch.arange(20)
    assert OG.first_visible(pos, 0, 0).tolist() == [0] * 20
    assert OG.first_visible(pos, 3, 0).tolist() == [max(0, p - 2) for p in range(20)]
    assert OG.first_visible(pos, 3, 5).tolist() == [max(0, p - 2, p // 5 * 5) for p in range(20)]
    kv = {"k": 8}
    for specs, want in (([CacheSpec(kv, chunk=5)], 10), ([CacheSpec(kv, chunk=5), CacheSpec(kv, window=9)], 4),
                        ([CacheSpec(kv, chunk=5), CacheSpec(kv)], 0), ([CacheSpec({}, {"s": ((2,), None)})], 12)):
        assert LayerCache(specs, max_seqs=1, max_seq_len=32, device="cpu").visible_from(12) == want
    cache = LayerCache([CacheSpec(kv, {"s": ((3, 2), torch.float32)})], max_seqs=2, max_seq_len=32, device="cpu")
    assert cache.bytes_per_token() == 16 and cache.bytes_per_sequence() == 24


def test_boundary_adds_what_a_pass_brings():
    from ironcore_b200.ops import streams as OS

    n, d = 4, 6
    x, y, table, step, w = _rand(n, 1, d), _rand(n, d, seed=1), _rand(9, d, seed=2), _rand(d, seed=3), _rand(d, seed=4)
    ids = torch.tensor([3, 8, 0, 3])
    embed = OS.TokenEmbed(ids, table, 1.5, 1)
    write = OS.StreamWrite(x, y, None, None, torch.ones(1, 1), torch.tensor([0.6]))
    for add, extra in ((None, 0.0), (OS.StreamAdd(step), step.double()),
                       (OS.StreamAdd(step, embed), step.double() + 1.5 * table[ids].double())):
        new, h, _ = OS.boundary(write, torch.ones(1), w, 1, 1e-3, width=8, dtype=torch.float32, add=add)
        want = x[:, 0].double() + 0.6 * y.double() + extra
        assert torch.allclose(new[:, 0].double(), want, atol=1e-5)
        for i in range(n):
            assert torch.allclose(h[i, :d].double(), oracle.rms_norm(want[i], w.double(), 1e-3), atol=1e-5)
    first, _, _ = OS.boundary(embed, torch.ones(1), w, 1, 1e-3, width=8, dtype=torch.float32, add=OS.StreamAdd(step))
    assert torch.allclose(first[:, 0], table[ids] * 1.5 + step, atol=1e-6)


@pytest.mark.parametrize("case", ["mixed_layers", "one_group"])
def test_mixers_alone(case):
    from ironcore_b200.rl.batch import StepBatch

    cfg = CASES[case]
    w = K.weights(cfg)
    model, _ = K.build(cfg, w)
    n, d = 21, cfg["width"]
    h = _rand(n, d)
    for i, spec in enumerate(cfg["layers"]):
        mix = {k[len(f"l{i}.mix."):]: v.double() for k, v in w.items() if k.startswith(f"l{i}.mix.")}
        want = oracle.mixer(h.double(), mix, spec, cfg["norm"]["eps"])
        run = model.model.order.index(i)
        for kind in ("prompt", "extend"):
            cache = model.model.make_cache(1, n, 16, device="cpu", dtype=torch.float32)
            cache.reserve(0, n)
            seqs, pos = torch.zeros(n, dtype=torch.int32), torch.arange(n, dtype=torch.int32)
            x = torch.nn.functional.pad(h, (0, model.model.width - d))
            batch = StepBatch(kind, torch.zeros(n, dtype=torch.int64), seqs, pos, cache.slots_for(seqs, pos), n, n,
                              torch.tensor([0, n], dtype=torch.int32), True)
            got = model.model.layers[i].mixer(x, batch, cache, run)[:, :d]
            assert K.error(got, want) < TIGHT, (i, kind)


def test_feed_forward_alone():
    cfg = CASES["mixed_layers"]
    w = K.weights(cfg)
    model, _ = K.build(cfg, w)
    h = _rand(5, cfg["width"])
    with torch.no_grad():
        y, gate = model.model.layers[2].mlp(torch.nn.functional.pad(h, (0, model.model.width - cfg["width"])))
    mw = {k[7:]: v.double() for k, v in w.items() if k.startswith("l2.mlp.")}
    assert gate is None
    for i in range(5):
        assert torch.allclose(y[i, :cfg["width"]].double(), oracle.dense_mlp(h[i].double(), mw), atol=1e-5)


def test_schedule_of_layer_runs_and_passes():
    from ironcore_b200.models.stream_model import run_schedule

    for n, loop in ((3, None), (4, {"start": 1, "stop": 3, "times": 2}), (4, {"start": 0, "stop": 4, "times": 3}),
                    (3, {"start": 2, "stop": 3, "times": 1}), (3, {"start": 1, "stop": 1, "times": 5})):
        assert run_schedule(n, loop) == oracle.layer_runs({"layers": [0] * n, "loop": loop})


def test_an_oracle_with_a_planted_mistake_is_far_away():
    """The weights show what they should: each mistake, planted in the restatement, moves the logits well beyond the
    tolerance of every comparison here."""
    cfg = CASES["mixed_layers"]
    w, toks = K.weights(cfg), K.tokens(cfg, 30)
    want = K.reference(cfg, w, toks)

    def changed(**patch):
        keep = {k: getattr(oracle, k) for k in patch}
        try:
            for k, v in patch.items():
                setattr(oracle, k, v)
            return K.error(K.reference(cfg, w, toks), want)
        finally:
            for k, v in keep.items():
                setattr(oracle, k, v)

    visible, conv, rule, rotate = oracle.visible, oracle.causal_conv, oracle.delta_rule, oracle.rotate
    scan, before, decay = oracle.selective_scan, oracle.before_pass, oracle.channel_decay

    def restarted(f, parts):
        """f over a sequence whose state is lost after 17 tokens."""
        return lambda *a: torch.cat([f(*(x[lo:hi] if i in parts else x for i, x in enumerate(a))) for lo, hi in ((0, 17), (17, None))])

    def late_write(q, k, v, beta, g):          # reads out before the token's own write
        state, out = torch.zeros(q.shape[1], v.shape[1], dtype=F64), []
        for t in range(q.shape[0]):
            state = g[t][:, None] * state
            out.append(state.t() @ q[t])
            state = state + torch.outer(k[t], beta[t] * (v[t] - state.t() @ k[t]))
        return torch.stack(out)

    assert changed(visible=lambda i, j, n: visible(i, j, n and n + 1)) > 0.02
    assert changed(visible=lambda i, j, n: visible(i + 1, j + 1, n)) > 0.02
    assert changed(visible=lambda i, j, n: j <= i) > 0.02
    assert changed(causal_conv=restarted(conv, (0,))) > 0.02
    assert changed(selective_scan=restarted(scan, (0, 1, 3, 4))) > 0.02
    assert changed(delta_rule=restarted(rule, (0, 1, 2, 3, 4))) > 0.02
    assert changed(delta_rule=late_write) > 0.02
    assert changed(channel_decay=lambda a, b, c: decay(a, b, c).mean(1, keepdim=True).expand_as(a)) > 0.005
    assert changed(rotate=lambda x, p, n, b: rotate(x, p, x.numel() // 2 * 2, b)) > 0.02
    assert changed(rotate=lambda x, p, n, b: x) > 0.02
    assert changed(before_pass=lambda x, e, s, t: x + s[t]) > 0.02
    assert changed(before_pass=lambda x, e, s, t: x + e + s[t]) > 0.02
    assert changed(before_pass=lambda x, e, s, t: x if t == 0 else x + e) > 0.02
    assert changed(gelu_erf=lambda z: torch.nn.functional.silu(z)) > 0.02


# ------------------------------------------------------------------ the model through the engine
@pytest.mark.parametrize("case", list(CASES))
def test_prompt_decode_and_portions_agree_with_the_restatement(case):
    cfg = CASES[case]
    w, toks = K.weights(cfg), K.tokens(CASES[case], 37)
    want = K.reference(cfg, w, toks)
    model, c = K.build(cfg, w)
    eng = K.engine(model, c)
    for cuts in ([37], [1], [2], [5], [16, 1, 16, 4], [30, 1]):
        assert K.error(K.feed(eng, cfg, toks, cuts), want) < TIGHT, cuts
    # the model's own forward (a cache for the call)
    with torch.no_grad():
        got = model(torch.tensor([toks]))[0, :, :cfg["vocab"]]
    assert K.error(got, want) < TIGHT


def test_residual_stream_after_every_layer_run():
    cfg = CASES["mixed_layers"]
    w, toks = K.weights(cfg), K.tokens(cfg, 9)
    trace = []
    oracle.forward(cfg, w, toks, trace)
    model, c = K.build(cfg, w)
    model.model.trace = []
    K.engine(model, c).step([("a", toks, None)])
    assert len(trace) == len(model.model.trace) == 8
    for got, want in zip(model.model.trace, trace):
        assert torch.allclose(got.double(), want, atol=1e-4 * float(want.abs().max()))


@pytest.mark.parametrize("chunk", [8, 13, 16])
def test_the_first_and_the_next_to_first_key_of_a_chunk(chunk):
    """A token asks for its own earlier appearance with a score that drowns all others; the appearance lies at the edges of
    chunks and pages, in prompts and in decoding."""
    cfg = K.config([K.pair(dim=16, vdim=8, rot=2, base=1e6, chunk=chunk, ff=None)], vocab=97)
    w = K.standout_weights(cfg)
    n = 3 * chunk
    model, c = K.build(cfg, w)
    eng = K.engine(model, c)
    for ask, key in ((2 * chunk - 1, chunk), (2 * chunk - 1, chunk - 1), (2 * chunk, chunk), (2 * chunk + 1, 2 * chunk),
                     (2 * chunk, 2 * chunk - 1), (n - 1, 2 * chunk)):
        toks = list(range(n))
        toks[key] = toks[ask] = 96
        want = K.reference(cfg, w, toks)
        without = list(toks)
        without[key] = 95
        far = K.error(K.reference(cfg, w, without)[ask:ask + 1], want[ask:ask + 1])
        if oracle.visible(ask, key, chunk):
            assert far > 0.02                       # (the recurrence beside it sees across chunks)
        for cuts in ([n], [ask, 1], [2], [key + 1, 1]):
            assert K.error(K.feed(eng, cfg, toks, cuts), want) < TIGHT, (ask, key, cuts)


def test_unequal_batches_against_each_alone():
    """Prompts of different lengths start together; the shorter ones leave, others take their slots and pages."""
    cfg = CASES["mixed_layers"]
    w = K.weights(cfg)
    model, c = K.build(cfg, w)
    eng = K.engine(model, c, max_seqs=3, num_blocks=9)
    v = cfg["vocab"]
    reqs = {"a": K.tokens(cfg, 1, 2), "b": K.tokens(cfg, 34, 3), "c": K.tokens(cfg, 17, 4), "d": K.tokens(cfg, 33, 5),
            "e": K.tokens(cfg, 20, 6)}
    want = {k: K.reference(cfg, w, t) for k, t in reqs.items()}
    got = {k: [] for k in reqs}
    at = {k: 0 for k in reqs}

    def step(**counts):
        entries = [(k, reqs[k][at[k]:at[k] + n], list(range(n))) for k, n in counts.items()]
        rows = eng.step(entries)[:, :v]
        lo = 0
        for k, n in counts.items():
            got[k].append(rows[lo:lo + n].clone())
            at[k] += n
            lo += n
        eng.end([k for k in counts if at[k] == len(reqs[k])])

    step(a=1, b=20, c=15)
    step(b=1, c=1)
    step(c=1, b=1)              # another order
    step(b=1, d=16)             # a prompt joins a running request
    step(e=3, d=1, b=2)         # portions, a decode row and a prompt in one batch
    for _ in range(9):
        step(b=1, d=1, e=1)
    step(d=7, e=8)
    assert at == {k: len(t) for k, t in reqs.items()}
    for k in reqs:
        assert K.error(torch.cat(got[k]), want[k]) < TIGHT, k
    assert eng.cache.free_blocks == 9 and len(eng.cache._idle) == 3


def test_long_decoding_gives_pages_back():
    """With chunks everywhere, a sequence runs far past what the pool could hold; nothing of it is seen again, while the
    states go on. Slots and pages serve the next request."""
    cfg = K.config([K.pair(chunk=18), K.mamba(), K.pair(heads=2, kv=1, chunk=7, ff=None)], loop={"start": 0, "stop": 2, "times": 2})
    w, toks = K.weights(cfg), K.tokens(cfg, 150)
    model, c = K.build(cfg, w)
    eng = K.engine(model, c, max_seqs=2, max_seq_len=256, num_blocks=5)
    assert K.error(K.feed(eng, cfg, toks, [20, 1]), K.reference(cfg, w, toks)) < TIGHT
    other = K.tokens(cfg, 60, 9)
    assert K.error(K.feed(eng, cfg, other, [60, 1]), K.reference(cfg, w, other)) < TIGHT
    assert eng.cache.free_blocks == 5


# ------------------------------------------------------------------ generation
def _greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(oracle.forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]


def test_greedy_generation_through_the_engine():
    cfg = K.config([K.mamba(), K.pair(chunk=5)], width=24, loop={"start": 0, "stop": 2, "times": 2})
    w = K.weights(cfg)
    model, c = K.build(cfg, w)
    prompts = [K.tokens(cfg, n, n) for n in (7, 1, 18, 4)]
    limits = [6, 9, 3, 0]
    want = [_greedy(cfg, w, p, n) for p, n in zip(prompts, limits)]
    eng = K.engine(model, c, max_seqs=2)              # two waves
    got, logps = eng.generate(prompts, limits, temperature=0.0)
    assert got == want and [len(x) for x in logps] == limits
    same = torch.tensor([K.tokens(cfg, 6, 31), K.tokens(cfg, 6, 32)])
    out, _ = eng.generate(same, 5, temperature=0.0)
    assert out[:, 6:].tolist() == [_greedy(cfg, w, p, 5) for p in same.tolist()]


# ------------------------------------------------------------------ files, registry, programs
def test_model_directory_round_trip(tmp_path):
    from safetensors.torch import load_file, save_file

    from ironcore_b200.checkpoint.pretrained import load_pretrained, save_pretrained

    cfg = CASES["mixed_layers"]
    w = K.weights(cfg)
    model, c = K.build(cfg, w, precision="bfloat16")
    save_pretrained(model, c, tmp_path)
    back = load_file(str(tmp_path / "model.safetensors"))
    assert set(back) == set(w)
    for k in w:
        assert back[k].shape == w[k].shape and torch.equal(back[k].bfloat16(), w[k]), k
    assert json.loads((tmp_path / "config.json").read_text()) == json.loads(json.dumps(cfg))
    again, _ = load_pretrained(tmp_path, precision="float32")
    toks = K.tokens(cfg, 12)
    with torch.no_grad():
        got = again(torch.tensor([toks]))[0, :, :cfg["vocab"]]
    assert K.error(got, K.reference(cfg, w, toks)) < TIGHT
    for name, change in (("l0.mix.D", None), ("loop.step", None), ("l1.mix.right.a2", lambda t: t[1:])):
        bad = dict(w)
        if change is None:
            del bad[name]
        else:
            bad[name] = change(bad[name]).contiguous()
        save_file(bad, str(tmp_path / "model.safetensors"))
        with pytest.raises((KeyError, ValueError)):
            load_pretrained(tmp_path)


def test_registry_and_yaml(tmp_path):
    import yaml

    from ironcore_b200.config import apply_yaml, default_config, validate_config
    from ironcore_b200.models import LanguageModel, get_model_provider_func
    from ironcore_b200.parallel import mesh

    mesh.destroy_model_parallel()
    doc = {"model": {"name": "kedavik", "d_model": 30, "vocab_size": 53, "layer_specs": [K.mamba(), K.pair()], "untie_embed": True,
                     "layer_loop": {"start": 0, "stop": 1, "times": 2}, "residual_mult": 0.5, "precision": "float32",
                     "num_attention_heads": 1},
           "data": {"task_type": "synthetic", "vocab_size": 53}, "trainer": {"micro_batch_size": 1, "train_batch_size": 1}}
    path = tmp_path / "k.yaml"
    path.write_text(yaml.safe_dump(doc))
    c = apply_yaml(default_config(), path)
    validate_config(c)
    assert get_model_provider_func(c).__name__ == "StreamModel"
    model = LanguageModel(c)
    assert model.model.schedule == [(0, 0), (0, 1), (1, None)]
    with pytest.raises(NotImplementedError):
        model.train()(torch.tensor([[1, 2]]))
    with torch.no_grad():
        assert torch.isfinite(model.eval()(torch.tensor([[1, 2, 3]]))).all()
        assert float(model(torch.tensor([[1, 2, 3]]), labels=torch.tensor([[2, 3, 4]]))) > 0
    for key, value in (("kv_heads", 3), ("dim", 3)):
        bad = K.pair()
        bad["mixer"]["left"][key] = value
        c.model.layer_specs[1] = bad
        with pytest.raises(ValueError):
            LanguageModel(c)


def _save(tmp_path, cfg, w):
    from safetensors.torch import save_file

    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_file(w, str(tmp_path / "model.safetensors"))


REPO = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def test_replaying_a_trace(tmp_path):
    import numpy as np

    cfg = CASES["mixed_layers"]
    w = K.weights(cfg)
    _save(tmp_path, cfg, w)
    a, b = K.tokens(cfg, 20, 1), K.tokens(cfg, 6, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:18], "want": [3, 17]}, {"id": "b", "tokens": b[:5], "want": []}],
              "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[5:], "want": [0]}, {"id": "a", "tokens": a[18:19], "want": [0]}],
              "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[19:], "want": []}], "end": ["a"]}]
    r = subprocess.run([os.path.join(REPO, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out",
                        str(tmp_path / "out"), "--max-tokens", "64"], input="".join(json.dumps(s) + "\n" for s in steps),
                       capture_output=True, text=True, timeout=300, env={**os.environ, "CUDA_VISIBLE_DEVICES": ""})
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    ra, rb = K.reference(cfg, w, a), K.reference(cfg, w, b)
    for n, want in ((0, ra[[3, 17]]), (1, torch.stack([rb[5], ra[18]]))):
        got = torch.from_numpy(np.fromfile(tmp_path / "out" / f"{n}.f32", dtype="<f4")).view(-1, cfg["vocab"])
        assert K.error(got, want) < TIGHT


def test_rollout_command_on_a_model_directory(tmp_path):
    cfg = CASES["recurrent_only"]
    w = K.weights(cfg)
    _save(tmp_path, cfg, w)
    p = K.tokens(cfg, 5)
    r = subprocess.run([sys.executable, "-m", "ironcore_b200", "rollout", "--model", str(tmp_path), "--dtype", "float32",
                        "--prompt-ids", ",".join(map(str, p)), "--prompt-ids", str(p[0]), "--max-new-tokens", "4"],
                       capture_output=True, text=True, timeout=300, cwd=REPO, env={**os.environ, "CUDA_VISIBLE_DEVICES": ""})
    assert r.returncode == 0, r.stderr
    got = [[int(t) for t in line.split(",")] for line in r.stdout.split()]
    assert got == [_greedy(cfg, w, p, 4), _greedy(cfg, w, p[:1], 4)]


def test_entry_points_of_the_kernels_exist():
    from ironcore_b200.ops import build, native

    where = build.exported_symbols()
    for case in ("mixed_layers", "aligned"):
        for precision in ("float32", "bfloat16"):
            model, _ = K.build(CASES[case], K.weights(CASES[case]), precision)
            names = model.native_symbols()
            assert set(names) <= set(where), set(names) - set(where)
            assert ("icb_gemm" in names) == (precision == "bfloat16")
    assert not [n for n in native._SIGNATURES if n not in where]
