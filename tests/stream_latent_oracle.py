"""Plain restatement of the stream-residual latent-attention design (Tetepel), one function per mechanism.

Written for reading, not for speed: loops over tokens, heads, groups and streams, 64-bit floats, no cache (every
function sees the whole sequence). It shares nothing with the package; the tests compare the package with it.

A model is ``(cfg, w)``: ``cfg`` the dictionary of a config.json, ``w`` a dictionary name -> tensor."""

import math

import torch

F64 = torch.float64


def grouped_rms_norm(x, weight, groups, eps):
    """x [D]: every one of ``groups`` consecutive equal parts over its own root mean square, times weight."""
    parts = []
    for part in x.chunk(groups):
        parts.append(part / math.sqrt(float((part * part).mean()) + eps))
    return torch.cat(parts) * weight


def rms_norm(x, weight, eps):
    return x / math.sqrt(float((x * x).mean()) + eps) * weight


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def token_shift(hs, shift):
    """hs: list of [D] over positions; blends every element with the previous position's by ``shift``."""
    out, prev = [], torch.zeros_like(hs[0])
    for h in hs:
        out.append(h + (prev - h) * shift)
        prev = h
    return out


def read_streams(streams, w_in):
    """streams [S, D] -> weighted sum [D]."""
    u = torch.zeros_like(streams[0])
    for s in range(streams.shape[0]):
        u = u + w_in[s] * streams[s]
    return u


def write_streams(streams, mix, out, y):
    """Every new stream t: sum over the old streams s of mix[s, t] times stream s, plus out[t] y."""
    new = []
    for t in range(streams.shape[0]):
        acc = out[t] * y
        for s in range(streams.shape[0]):
            acc = acc + mix[s, t] * streams[s]
        new.append(acc)
    return torch.stack(new)


def residual_gate(y, h, w, b):
    return y * torch.sigmoid(w @ h + b)


def visible(i, j, window):
    return j <= i and (window is None or i - j < window)


def latent_attention(hs, w, mixer, eps):
    """hs: list of [D]; w: the mixer's tensors by short name. Returns the list of outputs [D]."""
    heads, dim, vdim = mixer["heads"], mixer["dim"], mixer["vdim"]
    window = (mixer.get("mask") or {}).get("size")
    qs, ks, vs, gates = [], [], [], []
    for h in hs:
        cq = rms_norm(w["dq"] @ h, w["dq.norm"], eps)
        c = rms_norm(w["dkv"] @ h, w["dkv.norm"], eps)
        qs.append((w["uq"] @ cq).view(heads, dim))
        ks.append((w["uk"] @ c).view(heads, dim))
        vs.append((w["uv"] @ c).view(heads, vdim))
        gates.append(torch.sigmoid(w["g"] @ h))
    outs = []
    for i in range(len(hs)):
        seen = [j for j in range(len(hs)) if visible(i, j, window)]
        per_head = []
        for n in range(heads):
            k = torch.stack([ks[j][n] for j in seen])
            v = torch.stack([vs[j][n] for j in seen])
            p = torch.softmax((k @ qs[i][n]) * mixer["scale"], dim=0)
            per_head.append((p @ v) * gates[i][n])
        outs.append(w["o"] @ torch.cat(per_head))
    return outs


def dense_mlp(h, w):
    return w["down"] @ (gelu_tanh(w["gate"] @ h) * (w["up"] @ h))


def layer_order(cfg):
    """Indices of the layers in the order they run (a looped block repeats with the same weights)."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


def _group(w, prefix):
    return {k[len(prefix):]: t.to(F64) for k, t in w.items() if k.startswith(prefix)}


def run_layer(streams, cfg, w, i):
    """streams: list over positions of [S, D]."""
    spec, lw = cfg["layers"][i], _group(w, f"l{i}.")
    groups, eps = cfg["norm"]["groups"], cfg["norm"]["eps"]
    hs = [grouped_rms_norm(read_streams(x, lw["hc1.in"]), lw["norm1"], groups, eps) for x in streams]
    ys = latent_attention(token_shift(hs, lw["shift"]), _group(lw, "mix."), spec["mixer"], eps)
    ys = [residual_gate(y, h, lw["rg1"], lw["rg1.b"]) for y, h in zip(ys, hs)]
    streams = [write_streams(x, lw["hc1.mix"], lw["hc1.out"], y) for x, y in zip(streams, ys)]
    if spec.get("mlp"):
        hs = [grouped_rms_norm(read_streams(x, lw["hc2.in"]), lw["norm2"], groups, eps) for x in streams]
        ys = [residual_gate(dense_mlp(h, _group(lw, "mlp.")), h, lw["rg2"], lw["rg2.b"]) for h in hs]
        streams = [write_streams(x, lw["hc2.mix"], lw["hc2.out"], y) for x, y in zip(streams, ys)]
    return streams


def forward(cfg, w, tokens, trace=None):
    """Logits [len(tokens), vocab]; ``trace`` (a list) receives the stream sums [len(tokens), D] after every run."""
    table = w["embed"].to(F64)
    s = cfg["streams"]
    streams = [(table[t] * cfg["embedding"]["scale"]).expand(s, -1).clone() for t in tokens]
    for i in layer_order(cfg):
        streams = run_layer(streams, cfg, w, i)
        if trace is not None:
            trace.append(torch.stack([x.sum(0) for x in streams]))
    rows = []
    for x in streams:
        y = grouped_rms_norm(x.sum(0), w["final.norm"].to(F64), cfg["norm"]["groups"], cfg["norm"]["eps"])
        rows.append(table @ y)
    return torch.stack(rows)
