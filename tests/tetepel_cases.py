"""Small configurations and random weights of the Tetepel family for the tests."""

import torch

import stream_latent_oracle as oracle


def layer(heads=3, dim=12, vdim=10, q_rank=14, kv_rank=9, window=6, scale=0.9, ff=22):
    return {"type": "latent_attention", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
                      "mask": None if window is None else {"size": window}}}


def config(layers, width=30, vocab=53, streams=2, groups=3, loop=None, eps=3e-4, embed=2.5):
    return {"architecture": "Tetepel", "embedding": {"scale": embed}, "layers": layers, "loop": loop,
            "norm": {"eps": eps, "groups": groups}, "streams": streams, "vocab": vocab, "width": width}


def cases():
    """Name -> configuration: no two layers of a model need to have anything in common, and each case has sizes that
    others make equal, one, odd or aligned."""
    return {
        "mixed_layers": config([layer(), layer(heads=2, dim=7, vdim=15, q_rank=9, kv_rank=20, window=3, ff=17),
                                layer(heads=1, window=None, ff=None)], loop={"start": 1, "stop": 3, "times": 2}),
        "one_stream": config([layer(window=1), layer(heads=4, kv_rank=70, window=17)], streams=1, groups=1, width=33),
        "five_streams": config([layer(window=16), layer(ff=None, window=5)], streams=5, groups=5, width=40, vocab=64,
                               loop={"start": 0, "stop": 1, "times": 3}),
        "aligned": config([layer(heads=4, dim=64, vdim=64, q_rank=32, kv_rank=64, window=21, scale=0.125, ff=64)],
                          width=96, groups=12, streams=4, vocab=128, loop={"start": 0, "stop": 1, "times": 1}),
        "wide_heads": config([layer(heads=18, dim=100, vdim=72, q_rank=24, kv_rank=130, window=9, scale=0.1)], width=56,
                             groups=2, streams=3),
        "beyond_the_fast_kernels": config([layer(heads=2, dim=140, vdim=40, q_rank=200, kv_rank=530, window=11, scale=0.08)],
                                          width=64, groups=2, streams=2),
    }


def weights(cfg, seed=0, peak=3.0):
    """Random bf16-representable weights. ``peak`` widens the spread of the attention scores, so that single keys
    dominate and a missing or surplus key changes the result; stream weights, shifts and gates are far from neutral."""
    g = torch.Generator().manual_seed(seed)

    def rnd(*shape, std=1.0, mean=0.0):
        return (torch.randn(*shape, generator=g) * std + mean).bfloat16()

    def lin(out, cols, gain=1.0):
        return rnd(out, cols, std=gain * cols ** -0.5)

    d, s = cfg["width"], cfg["streams"]
    w = {"embed": rnd(cfg["vocab"], d), "final.norm": rnd(d, std=0.2, mean=1.0)}
    for i, spec in enumerate(cfg["layers"]):
        m, p = spec["mixer"], f"l{i}."
        h = m["heads"]
        sharp = (peak / (m["scale"] * m["dim"] ** 0.5)) ** 0.5
        w.update({p + "norm1": rnd(d, std=0.2, mean=1.0), p + "mix.dq": lin(m["q_rank"], d),
                  p + "mix.dq.norm": rnd(m["q_rank"], std=0.2, mean=1.0), p + "mix.uq": lin(h * m["dim"], m["q_rank"], sharp),
                  p + "mix.dkv": lin(m["kv_rank"], d), p + "mix.dkv.norm": rnd(m["kv_rank"], std=0.2, mean=1.0),
                  p + "mix.uk": lin(h * m["dim"], m["kv_rank"], sharp), p + "mix.uv": lin(h * m["vdim"], m["kv_rank"]),
                  p + "mix.g": lin(h, d, 2.0), p + "mix.o": lin(d, h * m["vdim"], 2.0), p + "shift": rnd(d, std=0.3, mean=0.4),
                  p + "rg1": lin(d, d, 2.0), p + "rg1.b": rnd(d)})
        subs = [1]
        if spec["mlp"]:
            f = spec["mlp"]["ff"]
            subs.append(2)
            w.update({p + "norm2": rnd(d, std=0.2, mean=1.0), p + "mlp.gate": lin(f, d, 1.5), p + "mlp.up": lin(f, d, 1.5),
                      p + "mlp.down": lin(d, f, 2.0), p + "rg2": lin(d, d, 2.0), p + "rg2.b": rnd(d)})
        for q in subs:
            w.update({f"{p}hc{q}.in": rnd(s, std=0.4, mean=0.6), f"{p}hc{q}.out": rnd(s, std=0.4, mean=0.8),
                      f"{p}hc{q}.mix": (torch.eye(s) * 0.8 + 0.3 * torch.randn(s, s, generator=g)).bfloat16()})
    return w


def tokens(cfg, n, seed=1):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def build(cfg, w, precision="float32", device=None):
    from ironcore_b200.checkpoint.pretrained import load_tensors, tetepel_config
    from ironcore_b200.models import LanguageModel
    from ironcore_b200.parallel import mesh

    mesh.destroy_model_parallel()
    c = tetepel_config(cfg, precision)
    model = LanguageModel(c, device=device).eval()
    load_tensors(model, w)
    return model, c


def engine(model, c, **kw):
    from ironcore_b200.rl import RolloutEngine

    kw.setdefault("max_seqs", 4)
    kw.setdefault("max_seq_len", 128)
    kw.setdefault("block_size", 16)
    return RolloutEngine(model, c, **kw)


def feed(eng, cfg, toks, cuts, rid="r"):
    """Logits of every token of one request that is run in portions of the given sizes (the last repeats)."""
    rows, lo, i = [], 0, 0
    while lo < len(toks):
        n = min(cuts[min(i, len(cuts) - 1)], len(toks) - lo)
        rows.append(eng.step([(rid, toks[lo:lo + n], list(range(n)))])[:, :cfg["vocab"]].float().cpu().clone())
        lo, i = lo + n, i + 1
    eng.end([rid])
    return torch.cat(rows)


def error(got, want):
    """Worst row: rms of the difference (mean taken off) over the rms of the expected logits."""
    d = got.double() - want.double()
    d = d - d.mean(-1, keepdim=True)
    return float((d.pow(2).mean(-1).sqrt() / want.double().pow(2).mean().sqrt()).max())


def reference(cfg, w, toks):
    return oracle.forward(cfg, w, toks)
