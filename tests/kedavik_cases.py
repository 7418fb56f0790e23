"""Small configurations and random weights of the Kedavik family for the tests."""

import math

import torch

import gated_state_oracle as oracle
from tetepel_cases import engine, error, feed, tokens  # noqa: F401


def mamba(inner=20, state=6, dt_rank=3, conv=4, ff=None):
    return {"type": "mamba1", "mixer": {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def pair(heads=4, kv=2, dim=12, vdim=10, rot=8, base=500.0, scale=0.4, chunk=7, d_heads=4, d_kv=2, d_dim=10, d_vdim=6, conv=4,
         left=0.7, right=1.2, ff=22):
    return {"type": "parallel", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
            "mixer": {"left": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": chunk},
                               "rot": {"dims": rot, "base": base}}, "left_scale": left,
                      "right": {"heads": d_heads, "kv_heads": d_kv, "dim": d_dim, "vdim": d_vdim, "conv": conv},
                      "right_scale": right}}


def config(layers, width=30, vocab=53, loop=None, eps=3e-4, embed=2.5, mult=0.8):
    return {"architecture": "Kedavik", "embedding": {"scale": embed}, "layers": layers, "loop": loop, "norm": {"eps": eps},
            "residual_mult": mult, "vocab": vocab, "width": width}


def cases():
    """Name -> configuration: no two layers of a model need to have anything in common, and each case has sizes that others
    make equal, one, odd or aligned."""
    return {
        "mixed_layers": config([mamba(), pair(), mamba(inner=9, state=5, dt_rank=9, conv=2, ff=17),
                                pair(heads=3, kv=3, dim=6, vdim=15, rot=6, chunk=16, d_heads=2, d_kv=2, d_dim=7, d_vdim=9, conv=3,
                                     ff=None)], loop={"start": 1, "stop": 3, "times": 3}),
        "all_ones": config([mamba(inner=1, state=1, dt_rank=1, conv=1),
                            pair(heads=1, kv=1, dim=2, vdim=1, rot=2, chunk=1, d_heads=1, d_kv=1, d_dim=1, d_vdim=1, conv=1, left=1.0,
                                 right=1.0, ff=1)], width=9, mult=1.0, embed=1.0, loop={"start": 0, "stop": 2, "times": 1}),
        "one_group": config([pair(heads=20, kv=1, dim=64, vdim=40, rot=16, scale=0.2, chunk=33, d_heads=6, d_kv=1, d_dim=16,
                                  d_vdim=24, conv=5), mamba(inner=40, state=33, dt_rank=16)], width=48, vocab=64),
        "aligned": config([mamba(inner=128, state=16, dt_rank=8), pair(heads=4, kv=2, dim=64, vdim=64, rot=64, scale=0.125, chunk=24,
                                                                       d_heads=2, d_kv=2, d_dim=64, d_vdim=128, ff=64)],
                          width=96, vocab=128, loop={"start": 0, "stop": 2, "times": 2}),
        "wide_heads": config([pair(heads=2, kv=2, dim=128, vdim=100, rot=32, scale=0.1, chunk=19, d_heads=4, d_kv=4, d_dim=96,
                                   d_vdim=40, conv=4)], width=56),
        "beyond_the_fast_kernels": config([pair(heads=2, kv=1, dim=140, vdim=40, rot=140, scale=0.09, chunk=11, d_heads=1, d_kv=1,
                                                d_dim=200, d_vdim=20, conv=6), mamba(inner=30, state=130, dt_rank=30, conv=9)],
                                          width=64, loop={"start": 1, "stop": 2, "times": 2}),
        "recurrent_only": config([mamba(), mamba(inner=24, state=16, ff=40)], loop={"start": 0, "stop": 1, "times": 2}),
    }


def ranks(i):
    """Inner sizes of layer i's low-rank decay and output gate: only the tensors tell."""
    return 5 + 3 * i, 9 + i


def weights(cfg, seed=0, peak=3.0):
    """Random bf16-representable weights. ``peak`` widens the spread of the attention scores, so that single keys dominate
    and a missing or surplus key changes the result; decays are slow, so that states reach far back."""
    g = torch.Generator().manual_seed(seed)

    def rnd(*shape, std=1.0, mean=0.0):
        return (torch.randn(*shape, generator=g) * std + mean).bfloat16()

    def lin(out, cols, gain=1.0):
        return rnd(out, cols, std=gain * cols ** -0.5)

    d = cfg["width"]
    w = {"embed": rnd(cfg["vocab"], d), "head": lin(cfg["vocab"], d), "final.norm": rnd(d, std=0.2, mean=1.0)}
    if cfg["loop"]:
        w["loop.step"] = rnd(cfg["loop"]["times"], d, std=0.8)
    for i, spec in enumerate(cfg["layers"]):
        m, p = spec["mixer"], f"l{i}."
        w[p + "norm1"] = rnd(d, std=0.2, mean=1.0)
        if spec["type"] == "mamba1":
            c, n, r, k = m["inner"], m["state"], m["dt_rank"], m["conv"]
            w.update({p + "mix.in": lin(2 * c, d, 1.5), p + "mix.conv": rnd(c, k, std=k ** -0.5), p + "mix.conv.b": rnd(c, std=0.3),
                      p + "mix.x": lin(r + 2 * n, c, 1.5), p + "mix.dt": lin(c, r), p + "mix.dt.b": rnd(c, mean=-2.0),
                      p + "mix.A_log": rnd(c, n, std=0.7, mean=-1.0), p + "mix.D": rnd(c), p + "mix.o": lin(d, c, 2.0)})
        else:
            a, b = m["left"], m["right"]
            sharp = (peak / (a["scale"] * a["dim"] ** 0.5)) ** 0.5
            h, gk, e = a["heads"], a["kv_heads"], b["heads"]
            qk, vv, ra, rg = b["kv_heads"] * b["dim"], e * b["vdim"], *ranks(i)
            w.update({p + "mix.left.q": lin(h * a["dim"], d, sharp), p + "mix.left.k": lin(gk * a["dim"], d, sharp),
                      p + "mix.left.v": lin(gk * a["vdim"], d, 1.5), p + "mix.left.g": lin(h, d, 2.0),
                      p + "mix.left.o": lin(d, h * a["vdim"], 2.0)})
            r = p + "mix.right."
            for name, rows in (("q", qk), ("k", qk), ("v", vv)):
                w[r + name] = lin(rows, d, 1.5)
                w[r + name + ".conv"] = rnd(rows, b["conv"], std=b["conv"] ** -0.5)
            w.update({r + "b": lin(e, d, 2.0), r + "A_log": rnd(e, std=0.5), r + "norm": rnd(b["vdim"], std=0.2, mean=1.0),
                      r + "a1": lin(ra, d), r + "a2": lin(e * b["dim"], ra), r + "dt_bias": rnd(e * b["dim"], mean=-3.0),
                      r + "g1": lin(rg, d), r + "g2": lin(vv, rg, 2.0), r + "o": lin(d, vv, 2.0)})
        if spec["mlp"]:
            f = spec["mlp"]["ff"]
            w.update({p + "norm2": rnd(d, std=0.2, mean=1.0), p + "mlp.up": lin(f, d, 1.5), p + "mlp.up.b": rnd(f, std=0.5),
                      p + "mlp.down": lin(d, f, 2.0), p + "mlp.down.b": rnd(d, std=0.5)})
    return w


def build(cfg, w, precision="float32", device=None):
    from ironcore_b200.checkpoint.pretrained import kedavik_config, load_tensors
    from ironcore_b200.models import LanguageModel
    from ironcore_b200.parallel import mesh

    mesh.destroy_model_parallel()
    c = kedavik_config(cfg, precision, {k: tuple(t.shape) for k, t in w.items()})
    model = LanguageModel(c, device=device).eval()
    load_tensors(model, w)
    return model, c


def reference(cfg, w, toks):
    return oracle.forward(cfg, w, toks)


def standout_weights(cfg, seed=0):
    """Weights under which a query finds the keys of its own token: every layer's query and key of a head are the same
    projection of the embedding, widened until the best score holds all the weight; rotations are left to the small
    frequencies (a test sets ``rot`` to 0 or 2 dimensions)."""
    w = weights(cfg, seed)
    for i, spec in enumerate(cfg["layers"]):
        if spec["type"] != "parallel":
            continue
        a = spec["mixer"]["left"]
        p = f"l{i}.mix.left."
        k = w[p + "k"].float().view(a["kv_heads"], a["dim"], -1)
        q = k.repeat_interleave(a["heads"] // a["kv_heads"], 0) * (12.0 / (a["scale"] * math.sqrt(a["dim"])))
        w[p + "q"] = q.reshape(-1, q.shape[-1]).bfloat16()
    return w
