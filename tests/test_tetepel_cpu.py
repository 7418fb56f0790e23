"""The Tetepel family (residual streams, latent attention) on CPU against the plain restatement: every mechanism alone,
then the model through the rollout engine in every way a sequence can be cut and batched."""

import json
import os
import subprocess
import sys

import pytest
import torch

import stream_latent_oracle as oracle
import tetepel_cases as T

CASES = T.cases()
TIGHT = 2e-5      # fp32 against the 64-bit restatement


# ------------------------------------------------------------------ mechanisms
def _rand(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed))


@pytest.mark.parametrize("groups,width", [(1, 7), (3, 12), (4, 40)])
def test_grouped_norm(groups, width):
    from ironcore_b200.ops.streams import grouped_rms_norm_reference

    x, w = _rand(5, width) * 0.01, _rand(width, seed=1)      # small values: eps inside the root counts
    want = torch.stack([oracle.grouped_rms_norm(r.double(), w.double(), groups, 1e-4) for r in x])
    assert torch.allclose(grouped_rms_norm_reference(x, w, groups, 1e-4).double(), want, atol=1e-6)


@pytest.mark.parametrize("streams", [1, 3])
def test_boundary_writes_then_reads(streams):
    """Write (all streams from the old values), gate, read and norm in one call; the mix is indexed [from, to]."""
    from ironcore_b200.ops import streams as OS

    n, d = 4, 6
    x, y, gate = _rand(n, streams, d), _rand(n, d, seed=1), _rand(n, d, seed=2)
    bias, mix, out, read = _rand(d, seed=3), _rand(streams, streams, seed=4), _rand(streams, seed=5), _rand(streams, seed=6)
    w = _rand(d, seed=7)
    new, h, _ = OS.boundary(OS.StreamWrite(x, y, gate, bias, mix, out), read, w, 2, 1e-3, width=8, dtype=torch.float32)
    for i in range(n):
        yi = y[i].double() * torch.sigmoid(gate[i].double() + bias.double())
        xs = oracle.write_streams(x[i].double(), mix.double(), out.double(), yi)
        assert torch.allclose(new[i].double(), xs, atol=1e-5)
        hi = oracle.grouped_rms_norm(oracle.read_streams(xs, read.double()), w.double(), 2, 1e-3)
        assert torch.allclose(h[i, :d].double(), hi, atol=1e-5)
    assert torch.equal(h[:, d:], torch.zeros(n, 2))
    rows = torch.tensor([2, 0], dtype=torch.int32)
    _, sel, _ = OS.boundary(OS.StreamWrite(x, y, gate, bias, mix, out), read, w, 2, 1e-3, width=8, dtype=torch.float32,
                            rows=rows, keep_streams=False)
    assert torch.equal(sel, h[[2, 0]])


def test_token_shift_over_sequences_and_portions():
    from ironcore_b200.ops import streams as OS

    d, n = 6, 7
    table, w, shift = _rand(11, d), torch.ones(d), _rand(d, seed=1)
    ids = torch.tensor([3, 5, 1, 9, 10, 0, 4])
    hs = [oracle.grouped_rms_norm(table[t].double() * 2, w.double(), 1, 1e-3) for t in ids.tolist()]
    want = torch.stack(oracle.token_shift(hs, shift.double()))
    state = torch.full((3, d), 9.0)          # leftovers of whoever had the slot before

    def run(lo, hi, seq):
        batch = OS.TokenShift(shift, state.clone(), state, torch.full((hi - lo,), seq, dtype=torch.int32),
                              torch.arange(lo, hi, dtype=torch.int32))
        return OS.boundary(OS.TokenEmbed(ids[lo:hi], table, 2.0, 2), torch.tensor([0.25, 0.75]), w, 1, 1e-3, width=d,
                           dtype=torch.float32, shift=batch)[2].double()

    got = torch.cat([run(0, 2, 1), run(2, 3, 1), run(3, n, 1)])
    assert torch.allclose(got, want, atol=1e-5)
    # two sequences side by side do not see each other
    batch = OS.TokenShift(shift, state, state, torch.tensor([0, 0, 0, 2, 2, 2, 2], dtype=torch.int32),
                          torch.tensor([0, 1, 2, 0, 1, 2, 3], dtype=torch.int32))
    both = OS.boundary(OS.TokenEmbed(ids, table, 2.0, 2), torch.tensor([0.25, 0.75]), w, 1, 1e-3, width=d,
                       dtype=torch.float32, shift=batch)[2].double()
    want2 = torch.stack(oracle.token_shift(hs[:3], shift.double()) + oracle.token_shift(hs[3:], shift.double()))
    assert torch.allclose(both, want2, atol=1e-5)


@pytest.mark.parametrize("window", [1, 4, 16, 17, 0])
def test_window_edges_of_the_cached_attention(window):
    """One key stands out at a time: it decides the result exactly while the window holds it, at page borders too."""
    from ironcore_b200.ops import latent as OL

    bs, n, r = 16, 40, 8
    table = torch.tensor([[2, 0, 1]], dtype=torch.int32)          # pages out of order
    for pos in (0, 15, 16, 31, 32, 39):
        for j in {0, max(0, pos - window), min(n - 1, max(0, pos - window + 1)), max(0, pos - 1), pos, 16 if pos >= 16 else 0}:
            cache = torch.zeros(3 * bs, r)
            rows = [int(table[0, t // bs]) * bs + t % bs for t in range(n)]
            cache[rows] = _rand(n, r, seed=3) * 0.1
            cache[rows[j]] = torch.eye(r)[0] * 5
            out = OL.latent_attend(torch.eye(r)[:1].view(1, 1, r) * 8, cache, table, bs, torch.zeros(1, dtype=torch.int32),
                                   torch.tensor([pos], dtype=torch.int32), window=window, scale=1.0, max_keys=n)
            seen = oracle.visible(pos, j, window or None)
            assert (float(out[0, 0, 0]) > 4.9) == seen, (window, pos, j)


@pytest.mark.parametrize("case", ["mixed_layers", "one_stream"])
def test_attention_layer_alone(case):
    from ironcore_b200.rl.batch import StepBatch

    cfg = CASES[case]
    w = T.weights(cfg)
    model, _ = T.build(cfg, w)
    n, d = 21, cfg["width"]
    h = _rand(n, d)
    for i, spec in enumerate(cfg["layers"]):
        mix = {k[len(f"l{i}.mix."):]: v.double() for k, v in w.items() if k.startswith(f"l{i}.mix.")}
        want = torch.stack(oracle.latent_attention(list(h.double()), mix, spec["mixer"], cfg["norm"]["eps"]))
        cache = model.model.make_cache(1, n, 16, device="cpu", dtype=torch.float32)
        cache.reserve(0, n)
        seqs, pos = torch.zeros(n, dtype=torch.int32), torch.arange(n, dtype=torch.int32)
        x = torch.nn.functional.pad(h, (0, model.model.width - d))
        for kind in ("prompt", "extend"):
            batch = StepBatch(kind, torch.zeros(n, dtype=torch.int64), seqs, pos, cache.slots_for(seqs, pos), n, n,
                              torch.tensor([0, n], dtype=torch.int32), True)
            got = model.model.layers[i].mixer(x, batch, cache, model.model.order.index(i))[:, :d]
            assert T.error(got, want) < TIGHT, (i, kind)


def test_feed_forward_and_residual_gate_alone():
    cfg = CASES["mixed_layers"]
    w = T.weights(cfg)
    model, _ = T.build(cfg, w)
    h = _rand(5, cfg["width"])
    x = torch.nn.functional.pad(h, (0, model.model.width - cfg["width"]))
    lw = {k[3:]: v.double() for k, v in w.items() if k.startswith("l1.")}
    layer = model.model.layers[1]
    with torch.no_grad():
        y, gate = layer.mlp(x)
        gate1 = layer.mixer_gate(x)
    for i in range(5):
        hi = h[i].double()
        yi = oracle.dense_mlp(hi, {k[4:]: v for k, v in lw.items() if k.startswith("mlp.")})
        assert torch.allclose(y[i, :cfg["width"]].double(), yi, atol=1e-5)
        got = y[i, :cfg["width"]].double() * torch.sigmoid(gate[i, :cfg["width"]].double() + layer.mlp.bias.double())
        assert torch.allclose(got, oracle.residual_gate(yi, hi, lw["rg2"], lw["rg2.b"]), atol=1e-5)
        got = yi * torch.sigmoid(gate1[i, :cfg["width"]].double() + layer.mixer_gate.bias.double())
        assert torch.allclose(got, oracle.residual_gate(yi, hi, lw["rg1"], lw["rg1.b"]), atol=1e-5)


def test_order_of_layer_runs():
    from ironcore_b200.models.stream_model import run_order

    for n, loop in ((3, None), (4, {"start": 1, "stop": 3, "times": 2}), (4, {"start": 0, "stop": 4, "times": 3}),
                    (3, {"start": 2, "stop": 3, "times": 1}), (3, {"start": 1, "stop": 1, "times": 5})):
        assert run_order(n, loop) == oracle.layer_order({"layers": [0] * n, "loop": loop})
    with pytest.raises(ValueError):
        run_order(2, {"start": 1, "stop": 3, "times": 1})


def test_an_oracle_with_a_planted_mistake_is_far_away():
    """The weights show what they should: each mistake, planted in the restatement, moves the logits well beyond the
    tolerance of every comparison here."""
    cfg = CASES["mixed_layers"]
    w, toks = T.weights(cfg), T.tokens(cfg, 30)
    want = T.reference(cfg, w, toks)

    def changed(**patch):
        keep = {k: getattr(oracle, k) for k in patch}
        try:
            for k, v in patch.items():
                setattr(oracle, k, v)
            return T.error(T.reference(cfg, w, toks), want)
        finally:
            for k, v in keep.items():
                setattr(oracle, k, v)

    visible, shift, write = oracle.visible, oracle.token_shift, oracle.write_streams
    assert changed(visible=lambda i, j, n: visible(i, j, n and n + 1)) > 0.02
    assert changed(visible=lambda i, j, n: visible(i, j, n and n - 1)) > 0.02
    assert changed(token_shift=lambda hs, s: shift(hs[:1], s) + [h.clone() for h in hs[1:]]) > 0.02
    assert changed(write_streams=lambda x, m, o, y: write(x, m.t(), o, y)) > 0.02
    assert changed(residual_gate=lambda y, h, a, b: y * torch.sigmoid(a @ h)) > 0.02
    assert changed(grouped_rms_norm=lambda x, a, g, e: oracle.rms_norm(x, a, e)) > 0.02


# ------------------------------------------------------------------ the model through the engine
@pytest.mark.parametrize("case", list(CASES))
def test_prompt_decode_and_portions_agree_with_the_restatement(case):
    cfg = CASES[case]
    w, toks = T.weights(cfg), T.tokens(CASES[case], 37)
    want = T.reference(cfg, w, toks)
    model, c = T.build(cfg, w)
    eng = T.engine(model, c)
    for cuts in ([37], [1], [2], [5], [16, 1, 16, 4], [30, 1]):
        assert T.error(T.feed(eng, cfg, toks, cuts), want) < TIGHT, cuts
    # the model's own forward (a cache for the call)
    with torch.no_grad():
        got = model(torch.tensor([toks]))[0, :, :cfg["vocab"]]
    assert T.error(got, want) < TIGHT


def test_residual_streams_after_every_layer_run():
    cfg = CASES["mixed_layers"]
    w, toks = T.weights(cfg), T.tokens(cfg, 9)
    trace = []
    oracle.forward(cfg, w, toks, trace)
    model, c = T.build(cfg, w)
    model.model.trace = []
    T.engine(model, c).step([("a", toks, None)])
    assert len(trace) == len(model.model.trace) == 5
    for got, want in zip(model.model.trace, trace):
        assert torch.allclose(got.double(), want, atol=1e-4 * float(want.abs().max()))


def test_unequal_batches_against_each_alone():
    """Prompts of different lengths start together; the shorter ones leave, others take their slots and pages."""
    cfg = CASES["mixed_layers"]
    w = T.weights(cfg)
    model, c = T.build(cfg, w)
    eng = T.engine(model, c, max_seqs=3, num_blocks=9)
    v = cfg["vocab"]
    reqs = {"a": T.tokens(cfg, 1, 2), "b": T.tokens(cfg, 34, 3), "c": T.tokens(cfg, 17, 4), "d": T.tokens(cfg, 33, 5),
            "e": T.tokens(cfg, 20, 6)}
    want = {k: T.reference(cfg, w, t) for k, t in reqs.items()}
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
        assert T.error(torch.cat(got[k]), want[k]) < TIGHT, k
    assert eng.cache.free_blocks == 9 and len(eng.cache._idle) == 3


def test_long_decoding_gives_pages_back():
    """With a window everywhere, a sequence runs far past what the pool could hold; nothing of it is seen again."""
    cfg = T.config([T.layer(window=18), T.layer(heads=2, window=7)], streams=2, loop={"start": 0, "stop": 2, "times": 2})
    w, toks = T.weights(cfg), T.tokens(cfg, 150)
    want = T.reference(cfg, w, toks)
    model, c = T.build(cfg, w)
    eng = T.engine(model, c, max_seqs=2, max_seq_len=256, num_blocks=5)
    assert T.error(T.feed(eng, cfg, toks, [20, 1]), want) < TIGHT
    other = T.tokens(cfg, 60, 9)
    assert T.error(T.feed(eng, cfg, other, [60, 1]), T.reference(cfg, w, other)) < TIGHT
    assert eng.cache.free_blocks == 5
    # without a window on one layer nothing is given back
    free = CASES["mixed_layers"]
    model, c = T.build(free, T.weights(free))
    eng = T.engine(model, c, max_seqs=1, num_blocks=2)
    with pytest.raises(RuntimeError, match="out of blocks"):
        T.feed(eng, free, T.tokens(free, 40), [20, 1])


def test_requests_are_checked():
    cfg = CASES["aligned"]
    model, c = T.build(cfg, T.weights(cfg))
    eng = T.engine(model, c, max_seqs=1)
    for bad in ([("a", [], None)], [("a", [cfg["vocab"]], None)], [("a", [-1], None)], [("a", [1], [1])],
                [("a", [1], None), ("a", [2], None)]):
        with pytest.raises(ValueError):
            eng.step(bad)
    with pytest.raises(RuntimeError):
        eng.step([("a", [1], None), ("b", [1], None)])
    with pytest.raises(RuntimeError, match="max_seq_len"):
        eng.step([("c", [1] * 200, None)])
    assert eng.step([("d", [1, 2], [])]).shape[0] == 0


# ------------------------------------------------------------------ generation
def _greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(oracle.forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]


def test_greedy_generation_through_the_engine():
    cfg = T.config([T.layer(window=5), T.layer(heads=2, window=11, ff=None)], streams=3, width=24)
    w = T.weights(cfg)
    model, c = T.build(cfg, w)
    prompts = [T.tokens(cfg, n, n) for n in (7, 1, 18, 4)]
    limits = [6, 9, 3, 0]
    want = [_greedy(cfg, w, p, n) for p, n in zip(prompts, limits)]
    eng = T.engine(model, c, max_seqs=2)              # two waves
    got, logps = eng.generate(prompts, limits, temperature=0.0)
    assert got == want and [len(x) for x in logps] == limits
    full = torch.log_softmax(oracle.forward(cfg, w, prompts[0] + want[0]), -1)
    assert abs(logps[0][2] - float(full[len(prompts[0]) + 1, want[0][2]])) < 1e-4
    stop = want[1][3]
    cut = want[1].index(stop) + 1
    assert eng.generate([prompts[1]], 9, temperature=0.0, stop_token=stop)[0] == [want[1][:cut]]
    same = torch.tensor([T.tokens(cfg, 6, 31), T.tokens(cfg, 6, 32)])
    out, _ = eng.generate(same, 5, temperature=0.0)
    assert out[:, 6:].tolist() == [_greedy(cfg, w, p, 5) for p in same.tolist()]


def test_unequal_prompts_on_the_transformer_families():
    """The engine's packed prompts, mixed steps and early leavers serve the existing families the same way."""
    from helpers import tiny_config
    from ironcore_b200.config import validate_config
    from ironcore_b200.models import LanguageModel
    from ironcore_b200.parallel import mesh
    from ironcore_b200.rl import RolloutEngine

    for family in ("llama", "gpt2"):
        mesh.destroy_model_parallel()
        cfg = tiny_config(family, max_seq_len=64, max_position_embeddings=64)
        cfg.trainer.use_flash_attn = False
        validate_config(cfg)
        torch.manual_seed(0)
        model = LanguageModel(cfg).eval()
        eng = RolloutEngine(model, cfg, max_seqs=3, max_seq_len=64)
        g = torch.Generator().manual_seed(0)
        prompts = [torch.randint(0, 512, (n,), generator=g).tolist() for n in (5, 19, 1)]
        out, _ = eng.generate(prompts, [4, 7, 2], temperature=0.0)
        for p, n, t in zip(prompts, (4, 7, 2), out):
            cur = list(p)
            for _ in range(n):
                with torch.no_grad():
                    cur.append(int(model(torch.tensor([cur]))[0, -1, :512].argmax()))
            assert cur[len(p):] == t, family
        toks = prompts[1]
        with torch.no_grad():
            want = model(torch.tensor([toks]))[0, :, :512]
        rows = [eng.step([("x", toks[lo:lo + 4], list(range(len(toks[lo:lo + 4]))))])[:, :512] for lo in range(0, 19, 4)]
        eng.end(["x"])
        assert torch.allclose(torch.cat(rows), want, atol=1e-4)


# ------------------------------------------------------------------ files, registry, programs
def test_model_directory_round_trip(tmp_path):
    from safetensors.torch import load_file, save_file

    from ironcore_b200.checkpoint.pretrained import load_pretrained, save_pretrained

    cfg = CASES["mixed_layers"]
    w = T.weights(cfg)
    model, c = T.build(cfg, w, precision="bfloat16")
    save_pretrained(model, c, tmp_path)
    back = load_file(str(tmp_path / "model.safetensors"))
    assert set(back) == set(w)
    for k in w:
        assert back[k].shape == w[k].shape and torch.equal(back[k], w[k]), k
    assert json.loads((tmp_path / "config.json").read_text()) == json.loads(json.dumps(cfg))
    again, _ = load_pretrained(tmp_path, precision="float32")
    toks = T.tokens(cfg, 12)
    with torch.no_grad():
        got = again(torch.tensor([toks]))[0, :, :cfg["vocab"]]
    assert T.error(got, T.reference(cfg, w, toks)) < TIGHT
    for name, change in (("l0.shift", None), ("l0.mix.uk", lambda t: t[1:])):
        bad = dict(w)
        if change is None:
            del bad[name]
        else:
            bad[name] = change(bad[name]).contiguous()
        save_file(bad, str(tmp_path / "model.safetensors"))
        with pytest.raises((KeyError, ValueError)):
            load_pretrained(tmp_path)
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "nothing"}))
    with pytest.raises(ValueError, match="not known"):
        load_pretrained(tmp_path)


def test_registry_and_yaml(tmp_path):
    import yaml

    from ironcore_b200.config import apply_yaml, default_config, validate_config
    from ironcore_b200.models import LanguageModel, get_model_provider_func
    from ironcore_b200.parallel import mesh

    mesh.destroy_model_parallel()
    doc = {"model": {"name": "tetepel", "d_model": 30, "vocab_size": 53, "layer_specs": [T.layer(), T.layer(ff=None)],
                     "layer_loop": {"start": 0, "stop": 1, "times": 2}, "residual_streams": 2, "norm_groups": 3,
                     "precision": "float32", "num_attention_heads": 1},
           "data": {"task_type": "synthetic", "vocab_size": 53}, "trainer": {"micro_batch_size": 1, "train_batch_size": 1}}
    path = tmp_path / "t.yaml"
    path.write_text(yaml.safe_dump(doc))
    c = apply_yaml(default_config(), path)
    validate_config(c)
    assert len(c.model.layer_specs) == 2
    assert get_model_provider_func(c).__name__ == "StreamModel"
    model = LanguageModel(c)
    assert model.model.order == [0, 0, 1]
    with pytest.raises(NotImplementedError):
        model.train()(torch.tensor([[1, 2]]))
    with torch.no_grad():
        assert torch.isfinite(model.eval()(torch.tensor([[1, 2, 3]]))).all()
        assert float(model(torch.tensor([[1, 2, 3]]), labels=torch.tensor([[2, 3, 4]]))) > 0
    c.model.layer_specs[0]["type"] = "unheard_of"
    with pytest.raises(ValueError, match="unknown mixer"):
        LanguageModel(c)


def _save(tmp_path, cfg, w):
    from safetensors.torch import save_file

    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_file(w, str(tmp_path / "model.safetensors"))


REPO = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def test_replaying_a_trace(tmp_path):
    import numpy as np

    cfg = CASES["five_streams"]
    w = T.weights(cfg)
    _save(tmp_path, cfg, w)
    a, b = T.tokens(cfg, 20, 1), T.tokens(cfg, 6, 2)
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
    ra, rb = T.reference(cfg, w, a), T.reference(cfg, w, b)
    for n, want in ((0, ra[[3, 17]]), (1, torch.stack([rb[5], ra[18]]))):
        got = torch.from_numpy(np.fromfile(tmp_path / "out" / f"{n}.f32", dtype="<f4")).view(-1, cfg["vocab"])
        assert T.error(got, want) < TIGHT
    assert not (tmp_path / "out" / "2.f32").exists()


def test_rollout_command_on_a_model_directory(tmp_path):
    cfg = CASES["one_stream"]
    w = T.weights(cfg)
    _save(tmp_path, cfg, w)
    p = T.tokens(cfg, 5)
    r = subprocess.run([sys.executable, "-m", "ironcore_b200", "rollout", "--model", str(tmp_path), "--dtype", "float32",
                        "--prompt-ids", ",".join(map(str, p)), "--prompt-ids", str(p[0]), "--max-new-tokens", "4"],
                       capture_output=True, text=True, timeout=300, cwd=REPO, env={**os.environ, "CUDA_VISIBLE_DEVICES": ""})
    assert r.returncode == 0, r.stderr
    got = [[int(t) for t in line.split(",")] for line in r.stdout.split()]
    assert got == [_greedy(cfg, w, p, 4), _greedy(cfg, w, p[:1], 4)]


def test_kernel_units_cover_every_entry_point():
    from ironcore_b200.ops import build, native

    where = build.exported_symbols()
    import ironcore_b200.ops.latent  # noqa: F401
    import ironcore_b200.ops.streams  # noqa: F401

    missing = [n for n in native._SIGNATURES if n not in where]
    assert not missing, missing
    assert build.unit_path("latent") != build.unit_path("streams")
