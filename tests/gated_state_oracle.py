"""Plain restatement of the Kedavik design (selective scan, chunked rotary attention beside a gated delta rule, looped
layers over one residual stream), one function per mechanism.

Written for reading, not for speed: loops over tokens and heads, 64-bit floats, no cache (every function sees the whole
sequence). It shares nothing with the package; the tests compare the package with it.

A model is ``(cfg, w)``: ``cfg`` the dictionary of a config.json, ``w`` a dictionary name -> tensor."""

import math

import torch

F64 = torch.float64
UNIT_EPS = 1e-6


def root_mean_square(x, eps):
    return torch.sqrt((x * x).mean() + eps)


def rms_norm(x, weight, eps):
    return x / root_mean_square(x, eps) * weight


def silu(x):
    return x / (1.0 + torch.exp(-x))


def softplus(x):
    return torch.clamp(x, min=0) + torch.log1p(torch.exp(-x.abs()))


def gelu_erf(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def causal_conv(xs, taps, bias=None):
    """xs [T, C], taps [C, K]: out[t, c] = sum_j taps[c, j] xs[t - (K - 1) + j, c] (+ bias), then silu."""
    n, width = xs.shape[0], taps.shape[1]
    out = torch.zeros_like(xs)
    for t in range(n):
        for j in range(width):
            s = t - (width - 1) + j
            if s >= 0:
                out[t] += taps[:, j] * xs[s]
        if bias is not None:
            out[t] += bias
    return silu(out)


def unit(x):
    return x / torch.sqrt((x * x).sum() + UNIT_EPS)


def rotate(x, position, dims, base):
    """x [dim]: the first ``dims`` elements rotate in pairs (i, i + dims / 2); the rest stay."""
    out = x.clone()
    half = dims // 2
    for i in range(half):
        a = position * base ** (-2.0 * i / dims)
        u, v = x[i], x[i + half]
        out[i] = u * math.cos(a) - v * math.sin(a)
        out[i + half] = v * math.cos(a) + u * math.sin(a)
    return out


def visible(i, j, chunk):
    return j <= i and (chunk is None or i // chunk == j // chunk)


def selective_scan(x, dt, a, b, c, d):
    """x, dt [T, C], a [C, N], b, c [T, N], d [C] -> [T, C]."""
    state = torch.zeros_like(a)
    out = []
    for t in range(x.shape[0]):
        state = torch.exp(dt[t][:, None] * a) * state + (dt[t] * x[t])[:, None] * b[t][None, :]
        out.append(state @ c[t] + d * x[t])
    return torch.stack(out)


def mamba(hs, w, m):
    """hs [T, D] -> [T, D]."""
    inner, rank, n = m["inner"], m["dt_rank"], m["state"]
    xz = hs @ w["in"].t()
    x = causal_conv(xz[:, :inner], w["conv"], w["conv.b"])
    low = x @ w["x"].t()
    dt = softplus(low[:, :rank] @ w["dt"].t() + w["dt.b"])
    y = selective_scan(x, dt, -torch.exp(w["A_log"]), low[:, rank:rank + n], low[:, rank + n:], w["D"])
    return (y * silu(xz[:, inner:])) @ w["o"].t()


def attention(hs, w, m):
    """Grouped heads, rotary positions, chunks, one gate per head. hs [T, D] -> [T, D]."""
    heads, groups, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    chunk = (m.get("mask") or {}).get("size")
    n = hs.shape[0]
    q = (hs @ w["q"].t()).view(n, heads, dim)
    k = (hs @ w["k"].t()).view(n, groups, dim)
    v = (hs @ w["v"].t()).view(n, groups, vdim)
    gate = torch.sigmoid(hs @ w["g"].t())
    rot = m["rot"]
    q = torch.stack([torch.stack([rotate(q[t, h], t, rot["dims"], rot["base"]) for h in range(heads)]) for t in range(n)])
    k = torch.stack([torch.stack([rotate(k[t, g], t, rot["dims"], rot["base"]) for g in range(groups)]) for t in range(n)])
    rows = []
    for i in range(n):
        seen = [j for j in range(n) if visible(i, j, chunk)]
        per_head = []
        for h in range(heads):
            g = h // (heads // groups)
            p = torch.softmax((k[seen, g] @ q[i, h]) * m["scale"], dim=0)
            per_head.append((p @ v[seen, g]) * gate[i, h])
        rows.append(torch.cat(per_head))
    return torch.stack(rows) @ w["o"].t()


def delta_rule(q, k, v, beta, decay):
    """One head: q, k, decay [T, dim], v [T, vdim], beta [T] -> [T, vdim]."""
    state = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype)
    out = []
    for t in range(q.shape[0]):
        state = decay[t][:, None] * state
        u = beta[t] * (v[t] - state.t() @ k[t])
        state = state + torch.outer(k[t], u)
        out.append(state.t() @ q[t])
    return torch.stack(out)


def channel_decay(a, a_log, dt_bias):
    """a, dt_bias [heads, dim], a_log [heads] -> decay factors in (0, 1)."""
    return torch.exp(-torch.exp(a_log)[:, None] * softplus(a + dt_bias))


def gated_delta(hs, w, m, eps):
    """hs [T, D] -> [T, D]."""
    heads, groups, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    n = hs.shape[0]
    q = causal_conv(hs @ w["q"].t(), w["q.conv"]).view(n, groups, dim)
    k = causal_conv(hs @ w["k"].t(), w["k.conv"]).view(n, groups, dim)
    v = causal_conv(hs @ w["v"].t(), w["v.conv"]).view(n, heads, vdim)
    beta = torch.sigmoid(hs @ w["b"].t())
    a = ((hs @ w["a1"].t()) @ w["a2"].t()).view(n, heads, dim)
    gate = torch.sigmoid((hs @ w["g1"].t()) @ w["g2"].t()).view(n, heads, vdim)
    decay = torch.stack([channel_decay(a[t], w["A_log"], w["dt_bias"].view(heads, dim)) for t in range(n)])
    outs = []
    for h in range(heads):
        g = h // (heads // groups)
        qu = torch.stack([unit(q[t, g]) * dim ** -0.5 for t in range(n)])
        ku = torch.stack([unit(k[t, g]) for t in range(n)])
        o = delta_rule(qu, ku, v[:, h], beta[:, h], decay[:, h])
        outs.append(torch.stack([rms_norm(o[t], w["norm"], eps) * gate[t, h] for t in range(n)]))
    return torch.cat(outs, dim=1) @ w["o"].t()


def parallel(hs, w, m, eps):
    left = attention(hs, _group(w, "left."), m["left"])
    right = gated_delta(hs, _group(w, "right."), m["right"], eps)
    return m["left_scale"] * left + m["right_scale"] * right


def mixer(hs, w, spec, eps):
    if spec["type"] == "mamba1":
        return mamba(hs, w, spec["mixer"])
    return parallel(hs, w, spec["mixer"], eps)


def dense_mlp(h, w):
    return w["down"] @ gelu_erf(w["up"] @ h + w["up.b"]) + w["down.b"]


def layer_runs(cfg):
    """(layer, pass of the loop that starts right before it or None) in the order the layers run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    runs = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        runs += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return runs + [(i, None) for i in range(loop["stop"], n)]


def before_pass(x, embedded, step, t):
    return x + step[t] if t == 0 else x + embedded + step[t]


def _group(w, prefix):
    return {k[len(prefix):]: t.to(F64) for k, t in w.items() if k.startswith(prefix)}


def run_layer(x, cfg, w, i):
    """x [T, D]."""
    spec, lw = cfg["layers"][i], _group(w, f"l{i}.")
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    hs = torch.stack([rms_norm(r, lw["norm1"], eps) for r in x])
    x = x + m * mixer(hs, _group(lw, "mix."), spec, eps)
    if spec.get("mlp"):
        mw = _group(lw, "mlp.")
        x = x + m * torch.stack([dense_mlp(rms_norm(r, lw["norm2"], eps), mw) for r in x])
    return x


def forward(cfg, w, tokens, trace=None):
    """Logits [len(tokens), vocab]; ``trace`` (a list) receives the residual stream [len(tokens), D] after every run."""
    embedded = w["embed"].to(F64)[torch.tensor(tokens)] * cfg["embedding"]["scale"]
    x = embedded
    for i, t in layer_runs(cfg):
        if t is not None:
            x = before_pass(x, embedded, w["loop.step"].to(F64), t)
        x = run_layer(x, cfg, w, i)
        if trace is not None:
            trace.append(x)
    rows = torch.stack([rms_norm(r, w["final.norm"].to(F64), cfg["norm"]["eps"]) for r in x])
    return rows @ w["head"].to(F64).t()
