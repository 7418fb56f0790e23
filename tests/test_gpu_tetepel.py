"""The Tetepel family's kernels on the GPU against their PyTorch restatements, and the model on the rollout engine
(eager and captured decode steps, bf16 and fp32) against the plain restatement."""

import pytest
import torch

import stream_latent_oracle as oracle
import tetepel_cases as T

pytestmark = pytest.mark.gpu
CASES = T.cases()
BF, F32 = torch.bfloat16, torch.float32


def _rand(*shape, seed=0, dtype=F32, scale=1.0):
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale).to(dtype)


def _close(got, want, dtype):
    got, want = got.float().cpu(), want.float()
    tol = 2e-5 if dtype == F32 else 1.2e-2
    assert torch.isfinite(got).all()
    assert float((got - want).abs().max()) <= tol * max(1.0, float(want.abs().max())), float((got - want).abs().max())


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("streams,width,groups,rows", [(1, 64, 1, 5), (2, 30, 3, 40), (3, 192, 6, 700), (4, 4096, 8, 33),
                                                       (4, 2048, 32, 1100), (6, 40, 5, 17), (3, 33, 11, 900)])
def test_boundary_kernel(dtype, streams, width, groups, rows):
    from ironcore_b200.ops import streams as OS

    pitch = (width + 7) // 8 * 8
    x, y, gate = _rand(rows, streams, width), _rand(rows, pitch, seed=1, dtype=dtype), _rand(rows, pitch + 8, seed=2, dtype=dtype)
    small = [_rand(width, seed=3), _rand(streams, streams, seed=4), _rand(streams, seed=5), _rand(streams, seed=6),
             _rand(width, seed=7), _rand(width, seed=8)]
    n_seq = min(5, rows)
    cuts = torch.linspace(0, rows, n_seq + 1).long()
    seqs = torch.cat([torch.full((int(b - a),), (3 * i) % n_seq if n_seq == 5 else i, dtype=torch.int32)
                      for i, (a, b) in enumerate(zip(cuts[:-1], cuts[1:]))])
    pos = torch.cat([torch.arange(int(b - a), dtype=torch.int32) + (7 if i % 2 else 0)
                     for i, (a, b) in enumerate(zip(cuts[:-1], cuts[1:]))])
    prev = _rand(n_seq, width, seed=9)

    def run(dev):
        bias, mix, out, read, w, shift = (t.to(dev) for t in small)
        state = torch.full((n_seq, width), 5.0, device=dev)
        src = OS.StreamWrite(x.to(dev), y.to(dev), gate.to(dev)[:, 8:], bias, mix, out)
        sh = OS.TokenShift(shift, prev.to(dev), state, seqs.to(dev), pos.to(dev))
        a = OS.boundary(src, read, w, groups, 1e-4, width=pitch, dtype=dtype, shift=sh)
        b = OS.boundary(src, read, w, groups, 1e-4, width=pitch, dtype=dtype)
        idx = torch.tensor([rows - 1, 0, rows // 2], dtype=torch.int32, device=dev)
        c = OS.boundary(src, read, w, groups, 1e-4, width=pitch, dtype=dtype, rows=idx, keep_streams=False)
        plain = OS.StreamWrite(x.to(dev), y.to(dev), None, None, mix, out)
        d = OS.boundary(plain, read, w, groups, 1e-4, width=pitch, dtype=dtype)
        return [*a, state, b[0], b[1], c[1], d[0], d[1]]

    got, want = run("cuda"), run("cpu")
    for i, (g, r) in enumerate(zip(got, want)):
        _close(g, r, F32 if i in (0, 3, 4, 7) else dtype)
    assert torch.equal(got[1][:, width:], torch.zeros_like(got[1][:, width:]))
    assert torch.equal(got[1], got[5]) and torch.equal(got[6], got[5][[rows - 1, 0, rows // 2]])


@pytest.mark.parametrize("dtype", [BF, F32])
def test_boundary_kernel_from_the_embedding(dtype):
    from ironcore_b200.ops import streams as OS

    table, ids = _rand(19, 72, dtype=dtype), torch.tensor([3, 18, 0, 3, 7, 7, 1] * 60)
    seqs = torch.arange(60, dtype=torch.int32).repeat_interleave(7)
    pos = torch.arange(7, dtype=torch.int32).repeat(60)

    def run(dev):
        state = torch.zeros(60, 70, device=dev)
        sh = OS.TokenShift(_rand(70, seed=1).to(dev), state, state, seqs.to(dev), pos.to(dev))
        out = OS.boundary(OS.TokenEmbed(ids.to(dev), table.to(dev), 1.5, 3), _rand(3, seed=2).to(dev), _rand(70, seed=3).to(dev),
                          2, 1e-4, width=72, dtype=dtype, shift=sh)
        return [*out, state]

    for i, (g, r) in enumerate(zip(run("cuda"), run("cpu"))):
        _close(g, r, F32 if i in (0, 3) else dtype)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("rows,q_rank,rank,heads", [(3, 80, 24, 5), (1300, 64, 128, 6), (70, 11, 9, 3), (1500, 13, 33, 1)])
def test_latent_norm_kernel(dtype, rows, q_rank, rank, heads):
    from ironcore_b200.ops import latent as OL

    ldz, qw, cw = (q_rank + rank + heads + 7) // 8 * 8, (q_rank + 7) // 8 * 8, (rank + 63) // 64 * 64
    z, wq, wc = _rand(rows, ldz, scale=0.1), _rand(q_rank, seed=1), _rand(rank, seed=2)
    slots = torch.randperm(rows + 9, generator=torch.Generator().manual_seed(0))[:rows]
    slots[1] = -1

    def run(dev):
        cache = torch.full((rows + 9, cw), 7.0, dtype=dtype, device=dev)
        out = OL.latent_norm(z.to(dev), wq.to(dev), wc.to(dev), heads, 1e-3, q_width=qw, c_width=cw, dtype=dtype,
                             cache=cache, slots=slots.to(dev), want_latent=True)
        return [*out, cache]

    for i, (g, r) in enumerate(zip(run("cuda"), run("cpu"))):
        _close(g, r, F32 if i == 2 else dtype)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("rows,heads,k,n", [(1, 3, 64, 64), (17, 2, 128, 192), (33, 5, 64, 512), (150, 4, 512, 128),
                                            (9, 2, 576, 80), (70, 3, 96, 16)])
def test_head_product_kernel(dtype, rows, heads, k, n):
    from ironcore_b200.ops import latent as OL

    x, w, g = _rand(rows, heads, k, dtype=dtype), _rand(heads, n, k, seed=1, dtype=dtype, scale=k ** -0.5), _rand(rows, heads, seed=2)
    for gate in (None, g):
        got = OL.head_product(x.cuda(), w.cuda(), None if gate is None else gate.cuda())
        _close(got, OL.head_product(x, w, gate), dtype)


@pytest.mark.parametrize("dtype,rank", [(BF, 64), (BF, 128), (BF, 192), (BF, 256), (BF, 320), (BF, 384), (BF, 448), (BF, 512), (BF, 576), (F32, 64),
                                        (F32, 192)])
@pytest.mark.parametrize("heads,window", [(1, 1), (6, 33), (16, 64), (17, 130), (40, 0)])
def test_latent_attend_kernel(dtype, rank, heads, window):
    """Random keys with one standout per row at the edges of the window, positions around page and tile borders."""
    from ironcore_b200.ops import latent as OL
    from ironcore_b200.ops import native

    bs, pages, n_seq = {17: (48, 10, 3), 16: (64, 8, 3), 40: (128, 4, 3)}.get(heads, (16, 30, 3))
    positions = [0, 1, 15, 16, 31, 32, 33, 63, 64, 127, 130, 299, 470]
    g = torch.Generator().manual_seed(1)
    table = torch.randperm(n_seq * pages, generator=g).to(torch.int32).view(n_seq, pages)
    cache = _rand(n_seq * pages * bs, rank, dtype=dtype, scale=0.5)
    rows = [(s, p) for s in range(n_seq) for p in positions]
    q = _rand(len(rows), heads, rank, seed=2, scale=0.3)
    for i, (s, p) in enumerate(rows):       # the key just inside or just outside, or the first one, stands out
        reach = window or p + 1
        j = [max(0, p - reach + 1), max(0, p - reach), 0][i % 3]
        c = cache[int(table[s, j // bs]) * bs + j % bs].float()
        q[i] += c / c.norm() * 3
    q = q.to(dtype)
    seqs = torch.tensor([r[0] for r in rows], dtype=torch.int32)
    pos = torch.tensor([r[1] for r in rows], dtype=torch.int32)
    want = OL.latent_attend(q, cache, table, bs, seqs, pos, window=window, scale=0.7, max_keys=471)
    for keys, legacy in ((1 << 20, False), (100, False), (1 << 20, True), (100, True)):   # many ranges, and one piece
        got = OL.latent_attend(q.cuda(), cache.cuda(), table.cuda(), bs, seqs.cuda(), pos.cuda(), window=window, scale=0.7,
                               max_keys=keys, legacy=legacy)
        _close(got, want, dtype)
    native.check_status()


def test_latent_attend_splits_leave_empty_ranges():
    """More ranges than tiles: the empty ones contribute nothing."""
    from ironcore_b200.ops import latent as OL

    for rank in (64, 128):
        cache, q = _rand(64, rank, dtype=BF), _rand(2, 4, rank, seed=1, dtype=BF)
        table = torch.arange(4, dtype=torch.int32).view(1, 4)
        seqs, pos = torch.zeros(2, dtype=torch.int32), torch.tensor([0, 40], dtype=torch.int32)
        want = OL.latent_attend(q, cache, table, 16, seqs, pos, window=0, scale=0.3, max_keys=64)
        got = OL.latent_attend(q.cuda(), cache.cuda(), table.cuda(), 16, seqs.cuda(), pos.cuda(), window=0, scale=0.3,
                               max_keys=4096)
        _close(got, want, BF)


@pytest.mark.parametrize("hd", [64, 128])
@pytest.mark.parametrize("window", [1, 2, 63, 64, 65, 129, 200, 0])
def test_windowed_flash_kernel(hd, window):
    """Unequal prompts; scores peak at the window's edges, and rows whose first key tile holds nothing visible have very
    negative scores (they must not drown)."""
    from ironcore_b200.ops import latent as OL

    heads, lens = 3, [1, 70, 300, 129, 513]
    t = sum(lens)
    cu = torch.tensor([0] + list(torch.tensor(lens).cumsum(0)), dtype=torch.int32)
    kv = _rand(t, 2 * heads * hd, dtype=BF, scale=0.5)
    q = _rand(t, heads * hd, seed=1, scale=0.5)
    k = kv[:, :heads * hd].float()
    for a, b in zip(cu[:-1].tolist(), cu[1:].tolist()):
        for i in range(a, b):
            reach = window or i - a + 1
            j = [max(a, i - reach + 1), max(a, i - reach), a][i % 3]
            q[i] += k[j] * (-6.0 if i % 7 == 0 else 2.0)
    q = q.to(BF)
    gate = torch.rand(t, heads, generator=torch.Generator().manual_seed(3))
    want = OL.prompt_attend(q, kv, heads, hd, cu, 513, window=window, scale=0.5, gate=gate)
    got = OL.prompt_attend(q.cuda(), kv.cuda(), heads, hd, cu.cuda(), 513, window=window, scale=0.5, gate=gate.cuda())
    _close(got, want, BF)
    low = kv.clone()
    low[:, :heads * hd] = _rand(1, heads * hd, seed=4, dtype=BF)          # all scores of a row alike, far below zero
    ql = (-low[:, :heads * hd].float() * 4).to(BF)
    want = OL.prompt_attend(ql, low, heads, hd, cu, 513, window=window, scale=1.0, gate=gate)
    got = OL.prompt_attend(ql.cuda(), low.cuda(), heads, hd, cu.cuda(), 513, window=window, scale=1.0, gate=gate.cuda())
    _close(got, want, BF)


def test_gated_activation_reads_column_slices():
    from ironcore_b200.ops import kernels, reference

    x = _rand(37, 2 * 48 + 16, dtype=BF)
    got = kernels.glu_fwd(x.cuda()[:, :96], "geglu")
    _close(got, reference.glu_reference(x[:, :96].float(), "geglu"), BF)


# ------------------------------------------------------------------ the model
LIMIT = {"float32": 5e-5, "bfloat16": 0.15}


@pytest.mark.parametrize("precision", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", list(CASES))
def test_model_on_the_engine(case, precision):
    """bf16 rounding is large on these sharp little models, so there the schedules are also compared with each other."""
    cfg = CASES[case]
    w, toks = T.weights(cfg, peak=3.0 if precision == "float32" else 1.0), T.tokens(cfg, 50)
    want = T.reference(cfg, w, toks)
    model, c = T.build(cfg, w, precision, device="cuda")
    graph, eager = T.engine(model, c), T.engine(model, c, use_cuda_graph=False)
    for eng, cuts in ((graph, [50]), (graph, [20, 1]), (graph, [1]), (eager, [33, 1]), (eager, [2]), (graph, [7, 1, 1, 1, 16])):
        got = T.feed(eng, cfg, toks, cuts)
        assert T.error(got, want) < LIMIT[precision], (cuts, T.error(got, want))


def test_fp32_models_ignore_the_tf32_switch():
    cfg = CASES["aligned"]
    w, toks = T.weights(cfg), T.tokens(cfg, 20)
    model, c = T.build(cfg, w, "float32", device="cuda")
    before = torch.backends.cuda.matmul.allow_tf32
    try:
        torch.backends.cuda.matmul.allow_tf32 = True
        got = T.feed(T.engine(model, c), cfg, toks, [15, 1])
        assert torch.backends.cuda.matmul.allow_tf32
    finally:
        torch.backends.cuda.matmul.allow_tf32 = before
    assert T.error(got, T.reference(cfg, w, toks)) < LIMIT["float32"]


def test_bf16_error_is_rounding():
    """On a model without sharp scores the bf16 path stays within a few per cent at every position."""
    cfg = T.config([T.layer(heads=4, dim=64, vdim=64, q_rank=48, kv_rank=64, window=40, scale=0.125, ff=96)] * 2, width=128,
                   groups=4, streams=4, vocab=256)
    w, toks = T.weights(cfg, peak=0.5), T.tokens(cfg, 100)
    want = T.reference(cfg, w, toks)
    model, c = T.build(cfg, w, "bfloat16", device="cuda")
    eng = T.engine(model, c)
    for cuts in ([100], [60, 1], [33]):
        assert T.error(T.feed(eng, cfg, toks, cuts), want) < 0.04, cuts


@pytest.mark.parametrize("precision", ["float32", "bfloat16"])
def test_unequal_batches_slots_and_pages(precision):
    cfg = CASES["mixed_layers"]
    w = T.weights(cfg, peak=3.0 if precision == "float32" else 1.0)
    model, c = T.build(cfg, w, precision, device="cuda")
    eng = T.engine(model, c, max_seqs=3, num_blocks=12)
    lens = {"a": 1, "b": 40, "c": 17, "d": 33, "e": 48}
    reqs = {k: T.tokens(cfg, n, n) for k, n in lens.items()}
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
        assert T.error(torch.cat(got[k]), T.reference(cfg, w, reqs[k])) < LIMIT[precision], k
    assert eng.cache.free_blocks == 12


def test_long_decoding_with_pages_given_back():
    cfg = T.config([T.layer(window=18), T.layer(heads=2, window=7)], streams=2, loop={"start": 0, "stop": 2, "times": 2})
    w, toks = T.weights(cfg), T.tokens(cfg, 150)
    model, c = T.build(cfg, w, "float32", device="cuda")
    eng = T.engine(model, c, max_seqs=2, max_seq_len=256, num_blocks=5)
    assert T.error(T.feed(eng, cfg, toks, [20, 1]), T.reference(cfg, w, toks)) < LIMIT["float32"]


def test_greedy_generation_on_the_gpu():
    cfg = T.config([T.layer(window=5), T.layer(heads=2, window=11, ff=None)], streams=3, width=24)
    w = T.weights(cfg)
    model, c = T.build(cfg, w, "float32", device="cuda")
    prompts = [T.tokens(cfg, n, n) for n in (7, 1, 18)]
    want = []
    for p, n in zip(prompts, (6, 9, 3)):
        toks = list(p)
        for _ in range(n):
            toks.append(int(oracle.forward(cfg, w, toks)[-1].argmax()))
        want.append(toks[len(p):])
    eng = T.engine(model, c)
    assert eng.generate(prompts, [6, 9, 3], temperature=0.0)[0] == want
    out, logp = eng.generate(torch.tensor([T.tokens(cfg, 6, 1)]), 3, temperature=1.0)      # the sampling kernel
    assert int(out.max()) < cfg["vocab"] and bool((logp <= 0).all())


def test_weights_changed_under_a_captured_step():
    cfg = CASES["aligned"]
    w, other = T.weights(cfg, 0), T.weights(cfg, 5)
    from ironcore_b200.checkpoint.pretrained import load_tensors

    model, c = T.build(cfg, w, "float32", device="cuda")
    eng, toks = T.engine(model, c), T.tokens(cfg, 30)
    T.feed(eng, cfg, toks, [10, 1])
    load_tensors(model, other)
    assert T.error(T.feed(eng, cfg, toks, [10, 1]), T.reference(cfg, other, toks)) < LIMIT["float32"]


def test_unequal_prompts_on_the_llama_family():
    """Packed prompts and mixed steps of the engine on the transformer's own kernels."""
    from helpers import tiny_config
    from ironcore_b200.config import validate_config
    from ironcore_b200.models import LanguageModel
    from ironcore_b200.parallel import mesh
    from ironcore_b200.rl import RolloutEngine

    mesh.destroy_model_parallel()
    cfg = tiny_config("llama", d_model=256, d_ffn=512, num_attention_heads=4, head_dim=64, max_seq_len=128, precision="bf16")
    validate_config(cfg)
    model = LanguageModel(cfg, device="cuda").eval()
    eng = RolloutEngine(model, cfg, max_seqs=3, max_seq_len=128)
    g = torch.Generator().manual_seed(0)
    prompts = [torch.randint(0, 512, (n,), generator=g).tolist() for n in (5, 70, 33)]
    rows = eng.step([(i, p[:-3], list(range(len(p) - 3))) for i, p in enumerate(prompts)]).float().cpu()
    tail = [eng.step([(i, p[len(p) - 3 + k:len(p) - 2 + k], [0]) for i, p in enumerate(prompts)]).float().cpu().clone()
            for k in range(2)]
    last = eng.step([(0, prompts[0][-1:], [0]), (1, prompts[1][-1:], [0])]).float().cpu()
    lo = 0
    for i, p in enumerate(prompts):
        with torch.no_grad():
            want = model(torch.tensor([p]))[0].float().cpu()
        n = len(p) - 3
        assert (rows[lo:lo + n] - want[:n]).abs().max() < 0.03 * want.abs().max()
        lo += n
        for k in range(2):
            assert (tail[k][i] - want[n + k]).abs().max() < 0.03 * want.abs().max()
        if i < 2:
            assert (last[i] - want[-1]).abs().max() < 0.03 * want.abs().max()
