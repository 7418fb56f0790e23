"""The Kedavik family's kernels on the GPU against their PyTorch restatements, and the model on the rollout engine (eager and
captured decode steps, bf16 and fp32) against the plain restatement."""

import pytest
import torch

import gated_state_oracle as oracle
import kedavik_cases as K

pytestmark = pytest.mark.gpu
CASES = K.cases()
BF, F32 = torch.bfloat16, torch.float32


def _rand(*shape, seed=0, dtype=F32, scale=1.0):
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale).to(dtype)


def _close(got, want, dtype, loose=1.0):
    got, want = got.float().cpu(), want.float()
    if want.numel() == 0:
        assert got.shape == want.shape
        return
    tol = (2e-5 if dtype == F32 else 1.2e-2) * loose
    err, most = float((got - want).abs().max()), max(1.0, float(want.abs().max()))
    assert err <= tol * most          # (a NaN fails)


def _rows(dev, spans, decode=False):
    """Rows of (slot, first position, count) spans."""
    from ironcore_b200.ops.recurrent import Rows

    seqs = torch.cat([torch.full((n,), s, dtype=torch.int32) for s, _, n in spans]).to(dev)
    pos = torch.cat([torch.arange(p, p + n, dtype=torch.int32) for _, p, n in spans]).to(dev)
    if decode:
        return Rows(seqs, pos, None, 1)
    cu = torch.tensor([0] + list(torch.tensor([n for _, _, n in spans]).cumsum(0)), dtype=torch.int32).to(dev)
    return Rows(seqs, pos, cu, max(n for _, _, n in spans))


# prompts, continued portions and single rows; slots out of order
MIXTURE = [(3, 0, 37), (0, 5, 1), (5, 0, 1), (1, 2, 2), (4, 17, 70), (2, 1, 16)]
ONE_EACH = [(3, 9, 1), (0, 0, 1), (5, 1, 1), (1, 2, 1)]


def _spans(many):
    return [(s, p, n * many) for s, p, n in MIXTURE]


def _conv_state(spans, taps, channels, dtype, seed):
    """Carried inputs of six slots; a sequence that has seen fewer tokens than there are entries has zeros in front."""
    state = _rand(6, taps - 1, channels, seed=seed, dtype=dtype)
    for slot, pos, _ in spans:
        if pos:
            state[slot, :max(0, taps - 1 - pos)] = 0
    return state


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("channels,taps,many", [(8, 1, 1), (24, 2, 1), (72, 4, 9), (2048, 4, 3), (40, 7, 2)])
def test_short_conv_kernel(dtype, channels, taps, many):
    from ironcore_b200.ops import recurrent as OR

    for spans, decode in ((_spans(many), False), (ONE_EACH, True)):
        t = sum(n for _, _, n in spans)
        x, w, b = _rand(t, channels + 16, dtype=dtype), _rand(taps, channels, seed=1), _rand(channels, seed=2)
        state = _conv_state(spans, taps, channels, dtype, 3)

        def run(dev):
            s = state.clone().to(dev)
            return [OR.short_conv(x.to(dev)[:, 8:8 + channels], w.to(dev), b.to(dev), s, _rows(dev, spans, decode)), s]

        for g, r in zip(run("cuda"), run("cpu")):
            _close(g, r, dtype)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("channels,n,per_lane", [(8, 1, None), (40, 5, None), (264, 16, None), (264, 16, 4), (264, 16, 16), (72, 24, 12),
                                                 (136, 33, None), (24, 130, None), (16, 500, None)])
def test_selective_scan_kernel(dtype, channels, n, per_lane):
    from ironcore_b200.ops import recurrent as OR

    width, npad = (n + 7) // 8 * 8, (n + 3) // 4 * 4
    for spans, decode in ((MIXTURE, False), (ONE_EACH, True)):
        t = sum(c for _, _, c in spans)
        u, z, dt = _rand(t, channels, dtype=dtype), _rand(t, channels + 8, seed=1, dtype=dtype), _rand(t, channels, seed=2)
        bc = _rand(t, 16 + 2 * width, seed=3, dtype=dtype, scale=n ** -0.5)
        bias, a_log, d = _rand(channels, seed=4) - 2, _rand(channels, npad, seed=5) - 1, _rand(channels, seed=6)
        state = _rand(6, channels, npad, seed=7)

        def run(dev):
            s, out = state.clone().to(dev), torch.full((t, channels + 8), 9.0, dtype=dtype, device=dev)
            OR.selective_scan(u.to(dev), dt.to(dev), z.to(dev)[:, 8:], bc.to(dev), 16, 16 + width, n, bias.to(dev), a_log.to(dev),
                              d.to(dev), s, _rows(dev, spans, decode), out[:, :channels], per_lane)
            return out, s[..., :n]

        (go, gs), (wo, ws) = run("cuda"), run("cpu")
        _close(go, wo, dtype)
        _close(gs, ws, F32, 3.0)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("heads,groups,dim,vdim,taps", [(1, 1, 8, 8, 1), (4, 2, 24, 40, 4), (6, 3, 64, 64, 4), (2, 1, 96, 128, 3),
                                                        (3, 3, 128, 72, 4), (2, 2, 200, 24, 4), (20, 5, 16, 16, 2)])
def test_gated_delta_kernels(dtype, heads, groups, dim, vdim, taps):
    from ironcore_b200.ops import recurrent as OR

    conv, sizes = 2 * groups * dim + heads * vdim, dict(groups=groups, heads=heads, dim=dim, vdim=vdim)
    valid = vdim - 3
    for spans, decode in ((MIXTURE, False), (_spans(3), False), (ONE_EACH, True)):      # few rows, and enough for two launches
        t = sum(c for _, _, c in spans)
        x, beta = _rand(t, conv + 8, dtype=dtype), _rand(t, heads, seed=1, dtype=dtype)
        cw, a = _rand(taps, conv, seed=2), _rand(t, heads * dim, seed=3)
        a_log, dt_bias = _rand(heads, seed=4, scale=0.3), _rand(heads * dim, seed=5) - 3
        cs, state = _conv_state(spans, taps, conv, dtype, 6), _rand(6, heads, vdim, OR.state_dim(dim), seed=7)
        state[..., dim:] = 0
        gate, w = _rand(t, heads * vdim, seed=8), _rand(vdim, seed=9)

        def run(dev):
            s, c, rows = state.clone().to(dev), cs.clone().to(dev), _rows(dev, spans, decode)
            ins = OR.delta_prepare(x.to(dev)[:, 8:], cw.to(dev), c, beta.to(dev), a.clone().to(dev), a_log.to(dev), dt_bias.to(dev),
                                   rows, q_scale=dim ** -0.5, **sizes)
            o = OR.delta_rule(ins, s, rows, **sizes)
            o2 = o.view(t, heads, vdim).clone()
            o2[..., valid:] = 0
            out = torch.empty(t, heads * vdim + 8, dtype=dtype, device=dev)[:, 8:]
            OR.delta_output(o2.view(t, -1), gate.to(dev), w.to(dev), 1e-4, 0.8, heads=heads, vdim=vdim, valid=valid, out=out)
            return [ins.q, ins.k, ins.qk, ins.decay, ins.beta, s, o, ins.v, out, c]

        for i, (g, r) in enumerate(zip(run("cuda"), run("cpu"))):
            # a value rounded to bf16 on either side of a tie moves the recurrence by a few units of that rounding
            _close(g, r, F32 if i < 5 else dtype, 3.0)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("heads,groups,kd,vd,half", [(4, 2, 64, 64, 32), (3, 1, 128, 128, 24), (5, 5, 16, 40, 3), (2, 2, 144, 8, 0)])
def test_rope_cache_kernel(dtype, heads, groups, kd, vd, half):
    from ironcore_b200.ops import grouped as OG

    t, cols = 37, (heads + groups) * kd + groups * vd
    z = _rand(t, cols + 16, dtype=dtype)
    pos = torch.arange(t, dtype=torch.int32) * 1371
    slots = torch.randperm(t + 5, generator=torch.Generator().manual_seed(0))[:t]
    slots[3] = -1
    freq = OG.rotary_frequencies(2 * half, 5000.0) if half else torch.zeros(0, dtype=torch.float64)

    def run(dev):
        zz = z.clone().to(dev)
        kc, vc = (torch.full((t + 5, groups * n), 7.0, dtype=dtype, device=dev) for n in (kd, vd))
        gate = OG.rope_cache(zz, freq.to(dev), pos.to(dev), heads=heads, groups=groups, kd=kd, vd=vd, k_cache=kc, v_cache=vc,
                             slots=slots.to(dev), gate_scale=0.5)
        return [zz, kc, vc, gate]

    for i, (g, r) in enumerate(zip(run("cuda"), run("cpu"))):
        _close(g, r, F32 if i == 3 else dtype)


@pytest.mark.parametrize("dtype,kd,vd", [(BF, 64, 64), (BF, 128, 128), (BF, 24, 40), (BF, 144, 264), (F32, 64, 64), (F32, 96, 200)])
@pytest.mark.parametrize("heads,groups,window,chunk", [(1, 1, 0, 1), (6, 2, 0, 33), (20, 1, 0, 64), (9, 1, 40, 0), (12, 4, 17, 130)])
def test_attend_rows_kernels(dtype, kd, vd, heads, groups, window, chunk):
    """Random keys with one standout per row at the edges of what it sees, positions around page and chunk borders."""
    from ironcore_b200.ops import grouped as OG

    bs, pages, n_seq = {6: (48, 10, 3), 20: (64, 8, 3)}.get(heads, (16, 30, 3))
    positions = [0, 1, 15, 16, 32, 33, 63, 64, 65, 127, 130, 259, 260, 470]
    g = torch.Generator().manual_seed(1)
    table = torch.randperm(n_seq * pages, generator=g).to(torch.int32).view(n_seq, pages)
    kc, vc = (_rand(n_seq * pages * bs, groups * n, seed=s, dtype=dtype, scale=0.5) for s, n in ((2, kd), (3, vd)))
    rows = [(s, p) for s in range(n_seq) for p in positions]
    q = _rand(len(rows), heads, kd, seed=4, scale=0.3)
    for i, (s, p) in enumerate(rows):       # the key just inside or just outside, or the first one, stands out
        lo = int(OG.first_visible(torch.tensor(p), window, chunk))
        j = [lo, max(0, lo - 1), 0][i % 3]
        c = kc[int(table[s, j // bs]) * bs + j % bs].float().view(groups, kd).repeat_interleave(heads // groups, 0)
        q[i] += c / c.norm(dim=-1, keepdim=True) * 4
    q = q.to(dtype).view(len(rows), -1)
    seqs = torch.tensor([r[0] for r in rows], dtype=torch.int32)
    pos = torch.tensor([r[1] for r in rows], dtype=torch.int32)
    gate = torch.rand(len(rows), heads, generator=g)
    kw = dict(heads=heads, groups=groups, kd=kd, vd=vd, window=window, chunk=chunk, scale=0.7)

    def run(dev, keys, gated):
        out = torch.zeros(len(rows), heads * vd + 8, dtype=dtype, device=dev)
        qq = torch.nn.functional.pad(q, (8, 0)).to(dev)[:, 8:]
        OG.attend_rows(qq, kc.to(dev), vc.to(dev), table.to(dev), bs, seqs.to(dev), pos.to(dev), max_keys=keys,
                       gate=gate.to(dev) if gated else None, out=out[:, 8:], **kw)
        return out

    for gated in (True, False):
        want = run("cpu", 471, gated)
        for keys in (1 << 20, 100):             # many ranges, and one piece
            _close(run("cuda", keys, gated), want, dtype)


@pytest.mark.parametrize("hd,heads,groups", [(64, 4, 2), (128, 3, 1)])
@pytest.mark.parametrize("chunk", [1, 2, 63, 64, 65, 129, 200, 1000])
def test_chunked_flash_kernel(hd, heads, groups, chunk):
    """Unequal prompts; scores peak at the chunks' edges, and rows whose first key tile holds nothing visible have very
    negative scores (they must not drown). The output goes to a column slice."""
    from ironcore_b200.ops import grouped as OG

    lens = [1, 70, 300, 129, 513]
    t, nq, nk = sum(lens), heads * hd, groups * hd
    cu = torch.tensor([0] + list(torch.tensor(lens).cumsum(0)), dtype=torch.int32)
    z = _rand(t, nq + 2 * nk + 8, scale=0.5)
    k = z[:, nq:nq + nk].bfloat16().float().view(t, groups, hd).repeat_interleave(heads // groups, 1).reshape(t, nq)
    for a, b in zip(cu[:-1].tolist(), cu[1:].tolist()):
        for i in range(a, b):
            lo = a + (i - a) // chunk * chunk
            j = [lo, max(a, lo - 1), a][i % 3]
            z[i, :nq] += k[j] * (-6.0 if i % 7 == 0 else 2.0)
    z = z.bfloat16()
    gate = torch.rand(t, heads, generator=torch.Generator().manual_seed(3))

    def run(dev):
        out = torch.zeros(t, nq + 16, dtype=BF, device=dev)
        OG.attend_prompts(z.to(dev), heads=heads, groups=groups, hd=hd, cu_seqlens=cu.to(dev), max_len=513, window=0, chunk=chunk,
                          scale=0.5, gate=gate.to(dev), out=out[:, 8:8 + nq])
        return out

    _close(run("cuda"), run("cpu"), BF)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("streams,width", [(1, 64), (1, 33), (2, 30)])
def test_boundary_kernel_with_what_a_pass_brings(dtype, streams, width):
    from ironcore_b200.ops import streams as OS

    rows, pitch = 300, (width + 7) // 8 * 8
    x, y, table = _rand(rows, streams, width), _rand(rows, pitch, seed=1, dtype=dtype), _rand(19, pitch, seed=2, dtype=dtype)
    step, w = _rand(width, seed=3), _rand(width, seed=4)
    ids = torch.randint(0, 19, (rows,), generator=torch.Generator().manual_seed(0))

    def run(dev):
        embed = OS.TokenEmbed(ids.to(dev), table.to(dev), 1.5, streams)
        src = OS.StreamWrite(x.to(dev), y.to(dev), None, None, torch.eye(streams, device=dev), torch.full((streams,), 0.6, device=dev))
        read = torch.ones(streams, device=dev)
        out = []
        for source, add in ((src, OS.StreamAdd(step.to(dev))), (src, OS.StreamAdd(step.to(dev), embed)),
                            (embed, OS.StreamAdd(step.to(dev)))):
            out += OS.boundary(source, read, w.to(dev), 1, 1e-4, width=pitch, dtype=dtype, add=add)[:2]
        return out

    for i, (g, r) in enumerate(zip(run("cuda"), run("cpu"))):
        _close(g, r, dtype if i % 2 else F32)


# ------------------------------------------------------------------ the model
LIMIT = {"float32": 5e-5, "bfloat16": 0.15}


@pytest.mark.parametrize("precision", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", list(CASES))
def test_model_on_the_engine(case, precision):
    """bf16 rounding is large on these sharp little models, so the bf16 weights are milder."""
    cfg = CASES[case]
    w, toks = K.weights(cfg, peak=3.0 if precision == "float32" else 1.0), K.tokens(cfg, 50)
    want = K.reference(cfg, w, toks)
    model, c = K.build(cfg, w, precision, device="cuda")
    graph, eager = K.engine(model, c), K.engine(model, c, use_cuda_graph=False)
    for eng, cuts in ((graph, [50]), (graph, [20, 1]), (graph, [1]), (eager, [33, 1]), (eager, [2]), (graph, [7, 1, 1, 1, 16])):
        got = K.feed(eng, cfg, toks, cuts)
        assert K.error(got, want) < LIMIT[precision], (cuts, K.error(got, want))


def test_a_thousand_tokens_in_fp32():
    """Slow decays: what a state adds up over many steps stays at rounding."""
    cfg = K.config([K.mamba(inner=16, state=16), K.pair(heads=2, kv=1, chunk=50, d_heads=1, d_kv=1, ff=None)], width=16)
    w, toks = K.weights(cfg), K.tokens(cfg, 1000)
    w["l0.mix.A_log"] -= 4
    w["l0.mix.dt.b"] -= 2
    w["l1.mix.right.dt_bias"] -= 4
    model, c = K.build(cfg, w, "float32", device="cuda")
    eng = K.engine(model, c, max_seqs=2, max_seq_len=1024)
    want = K.reference(cfg, w, toks)
    for cuts in ([1000], [900, 1], [333]):
        assert K.error(K.feed(eng, cfg, toks, cuts), want) < LIMIT["float32"], cuts


def test_bf16_error_is_rounding():
    """On a model without sharp scores the bf16 path stays within a few per cent at every position."""
    cfg = K.config([K.mamba(inner=128, state=16, dt_rank=8), K.pair(heads=4, kv=2, dim=64, vdim=64, rot=64, scale=0.125, chunk=40,
                                                                    d_heads=2, d_kv=2, d_dim=64, d_vdim=64, ff=96)],
                   width=128, vocab=256)
    w, toks = K.weights(cfg, peak=0.5), K.tokens(cfg, 100)
    want = K.reference(cfg, w, toks)
    model, c = K.build(cfg, w, "bfloat16", device="cuda")
    eng = K.engine(model, c)
    for cuts in ([100], [60, 1], [33]):
        assert K.error(K.feed(eng, cfg, toks, cuts), want) < 0.05, cuts


@pytest.mark.parametrize("precision", ["float32", "bfloat16"])
def test_unequal_batches_slots_and_pages(precision):
    cfg = CASES["mixed_layers"]
    w = K.weights(cfg, peak=3.0 if precision == "float32" else 1.0)
    model, c = K.build(cfg, w, precision, device="cuda")
    eng = K.engine(model, c, max_seqs=3, num_blocks=12)
    lens = {"a": 1, "b": 40, "c": 17, "d": 33, "e": 48}
    reqs = {k: K.tokens(cfg, n, n) for k, n in lens.items()}
    got, at = {k: [] for k in reqs}, {k: 0 for k in reqs}

    def step(**counts):
        rows = eng.step([(k, reqs[k][at[k]:at[k] + n], list(range(n))) for k, n in counts.items()])[:, :cfg["vocab"]].cpu()
        lo = 0
        for k, n in counts.items():
            got[k].append(rows[lo:lo + n].clone())
            at[k], lo = at[k] + n, lo + n
        eng.end([k for k in counts if at[k] == len(reqs[k])])

    step(a=1, b=30, c=15)
    step(b=1, c=1)
    step(c=1, b=1)
    step(b=1, d=20)
    for _ in range(4):
        step(b=1, d=1)
    step(e=30, d=2, b=1)
    step(e=16, d=7, b=2)
    step(e=1)
    step(e=1)
    assert at == lens
    for k in reqs:
        assert K.error(torch.cat(got[k]), K.reference(cfg, w, reqs[k])) < LIMIT[precision], k
    assert eng.cache.free_blocks == 12


@pytest.mark.parametrize("precision", ["float32", "bfloat16"])
def test_standout_keys_at_the_edges_of_chunks(precision):
    cfg = K.config([K.pair(dim=64, vdim=32, rot=2, base=1e6, chunk=24, ff=None)], vocab=97)
    w = K.standout_weights(cfg)
    model, c = K.build(cfg, w, precision, device="cuda")
    eng = K.engine(model, c)
    for ask, key in ((47, 24), (47, 23), (48, 24), (49, 48), (48, 47), (71, 48)):
        toks = list(range(72))
        toks[key] = toks[ask] = 96
        want = K.reference(cfg, w, toks)
        for cuts in ([72], [ask, 1], [5]):
            assert K.error(K.feed(eng, cfg, toks, cuts), want) < LIMIT[precision], (ask, key, cuts)


def test_long_decoding_with_pages_given_back():
    cfg = K.config([K.pair(chunk=18), K.mamba(), K.pair(heads=2, kv=1, chunk=7, ff=None)], loop={"start": 0, "stop": 2, "times": 2})
    w, toks = K.weights(cfg), K.tokens(cfg, 150)
    model, c = K.build(cfg, w, "float32", device="cuda")
    eng = K.engine(model, c, max_seqs=2, max_seq_len=256, num_blocks=5)
    assert K.error(K.feed(eng, cfg, toks, [20, 1]), K.reference(cfg, w, toks)) < LIMIT["float32"]


def test_greedy_generation_on_the_gpu():
    cfg = K.config([K.mamba(), K.pair(chunk=5)], width=24, loop={"start": 0, "stop": 2, "times": 2})
    w = K.weights(cfg)
    model, c = K.build(cfg, w, "float32", device="cuda")
    prompts = [K.tokens(cfg, n, n) for n in (7, 1, 18)]
    want = []
    for p, n in zip(prompts, (6, 9, 3)):
        toks = list(p)
        for _ in range(n):
            toks.append(int(oracle.forward(cfg, w, toks)[-1].argmax()))
        want.append(toks[len(p):])
    eng = K.engine(model, c)
    assert eng.generate(prompts, [6, 9, 3], temperature=0.0)[0] == want
    out, logp = eng.generate(torch.tensor([K.tokens(cfg, 6, 1)]), 3, temperature=1.0)      # the sampling kernel
    assert int(out.max()) < cfg["vocab"] and bool((logp <= 0).all())


def test_weights_changed_under_a_captured_step():
    from ironcore_b200.checkpoint.pretrained import load_tensors

    cfg = CASES["aligned"]
    w, other = K.weights(cfg, 0), K.weights(cfg, 5)
    model, c = K.build(cfg, w, "float32", device="cuda")
    eng, toks = K.engine(model, c), K.tokens(cfg, 30)
    K.feed(eng, cfg, toks, [10, 1])
    load_tensors(model, other)
    assert K.error(K.feed(eng, cfg, toks, [10, 1]), K.reference(cfg, other, toks)) < LIMIT["float32"]
