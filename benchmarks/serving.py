"""Serving throughput of a residual-stream family (Tetepel, Kedavik) beside the Llama-style transformer of equal size, and
its kernels beside the like kernels of that model.

``python bench.py --workload serving [--family tetepel|kedavik] [--size 2k|4k] [--kernels-only]``; one JSON line per
measurement. Random weights
and tokens. Model numbers go through ``RolloutEngine.generate``: prefill is a generation of one token, a decode step is
the difference between a long and a one-token generation over the number of extra steps, both timed with CUDA events
after warm-up (the weights of the timed layers exceed the 126 MB L2). Kernel numbers rotate over copies of the inputs
that exceed L2 twice over; bytes and FLOPs are the algorithmic ones."""

from __future__ import annotations

import json

import torch

HBM_GBS, BF16_TFLOPS = 6559.7, 1670.1      # measured on this pool: copy bandwidth, burst GEMM rate
SMS, SM_GHZ = 148, 1.965                    # nominal: 128 fp32 multiply-adds and 16 special functions per SM and clock
FP32_TFMA, SPECIAL_T = SMS * SM_GHZ * 0.128, SMS * SM_GHZ * 0.016

SIZES = {
    "4k": dict(width=4096, heads=32, head=128, q_rank=1536, kv_rank=512, ff=11008, streams=4, groups=8, window=2048,
               vocab=32000, layers=4, prompt=4096, seqs=4, decode_seqs=64, decode_prompt=2048),
    "2k": dict(width=2048, heads=16, head=128, q_rank=768, kv_rank=256, ff=5632, streams=2, groups=4, window=1024,
               vocab=32000, layers=8, prompt=4096, seqs=8, decode_seqs=128, decode_prompt=1024),
}


# Kedavik beside the transformer of the same width, heads and depth: selective-scan layers (inner = 2 width) without
# feed-forward alternate with layers of attention (a quarter of the key / value heads) beside the delta rule
KEDAVIK_SIZES = {
    "4k": dict(width=4096, heads=32, kv=8, head=128, chunk=2048, d_heads=32, d_head=128, inner=8192, state=16, dt_rank=256,
               conv=4, rank=128, ff=11008, vocab=32000, layers=4, prompt=4096, seqs=4, decode_seqs=64, decode_prompt=2000),
    "2k": dict(width=2048, heads=16, kv=4, head=128, chunk=1024, d_heads=16, d_head=128, inner=4096, state=16, dt_rank=128,
               conv=4, rank=128, ff=5632, vocab=32000, layers=8, prompt=4096, seqs=8, decode_seqs=128, decode_prompt=1000),
}


def _kedavik_model(z):
    from ironcore_b200.checkpoint.pretrained import kedavik_config
    from ironcore_b200.models import LanguageModel

    scan = {"type": "mamba1", "mlp": None,
            "mixer": {"inner": z["inner"], "state": z["state"], "dt_rank": z["dt_rank"], "conv": z["conv"]}}
    pair = {"type": "parallel", "mlp": {"kind": "dense", "ff": z["ff"]},
            "mixer": {"left": {"heads": z["heads"], "kv_heads": z["kv"], "dim": z["head"], "vdim": z["head"],
                               "scale": z["head"] ** -0.5, "mask": {"size": z["chunk"]},
                               "rot": {"dims": z["head"], "base": 10000.0}}, "left_scale": 0.7,
                      "right": {"heads": z["d_heads"], "kv_heads": z["d_heads"], "dim": z["d_head"], "vdim": z["d_head"],
                                "conv": z["conv"], "decay_rank": z["rank"], "gate_rank": z["rank"]}, "right_scale": 0.7}}
    cfg = kedavik_config({"embedding": {"scale": 8.0}, "layers": [scan, pair] * (z["layers"] // 2), "loop": None,
                          "norm": {"eps": 1e-5}, "residual_mult": 0.7, "vocab": z["vocab"], "width": z["width"]})
    return LanguageModel(cfg, device="cuda").eval(), cfg


def _stream_model(z):
    from ironcore_b200.checkpoint.pretrained import tetepel_config
    from ironcore_b200.models import LanguageModel

    layer = {"type": "latent_attention", "mlp": {"kind": "dense", "ff": z["ff"]},
             "mixer": {"heads": z["heads"], "dim": z["head"], "vdim": z["head"], "q_rank": z["q_rank"],
                       "kv_rank": z["kv_rank"], "scale": z["head"] ** -0.5, "mask": {"size": z["window"]}}}
    cfg = tetepel_config({"embedding": {"scale": 8.0}, "layers": [layer] * z["layers"], "loop": None,
                          "norm": {"eps": 1e-5, "groups": z["groups"]}, "streams": z["streams"], "vocab": z["vocab"],
                          "width": z["width"]})
    return LanguageModel(cfg, device="cuda").eval(), cfg


def _llama_model(z):
    from ironcore_b200.config import default_config, validate_config
    from ironcore_b200.models import LanguageModel

    c = default_config()
    c.model(name="llama", num_layers=z["layers"], d_model=z["width"], num_attention_heads=z["heads"],
            num_attention_groups=z["heads"], head_dim=z["head"], d_ffn=z["ff"], max_seq_len=8192, ln_type="rmsnorm",
            activation_type="swiglu", no_bias=True, untie_embed=False, precision="bf16", dropout_embd=0.0,
            dropout_attn=0.0, dropout_mlp=0.0, vocab_size=z["vocab"], reset_position_ids=False,
            reset_attention_mask=False, positional_embedding={"type": "rope"})
    c.data(task_type="synthetic", vocab_size=z["vocab"])
    c.trainer(micro_batch_size=1, train_batch_size=1, gradient_accumulation_steps=None)
    validate_config(c)
    return LanguageModel(c, device="cuda").eval(), c


def _timed(fn, repeat: int = 3) -> float:
    """Median device milliseconds of fn()."""
    times = []
    for _ in range(repeat):
        s, e = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        s.record()
        fn()
        e.record()
        torch.cuda.synchronize()
        times.append(s.elapsed_time(e))
    return sorted(times)[len(times) // 2]


def bench_models(family: str, size: str, steps: int, warmup: int, report) -> None:
    from ironcore_b200.ops import native
    from ironcore_b200.rl import RolloutEngine

    z = (SIZES if family == "tetepel" else KEDAVIK_SIZES)[size]
    for label, build in ((family, _stream_model if family == "tetepel" else _kedavik_model), ("llama", _llama_model)):
        model, cfg = build(z)
        params = sum(p.numel() for p in model.parameters())
        gen = torch.Generator().manual_seed(3)
        native.reset_launches()

        def prompts(n, p):
            return torch.randint(0, z["vocab"], (n, p), generator=gen)

        engine = RolloutEngine(model, cfg, max_seqs=z["seqs"], max_seq_len=z["prompt"] + 16)
        batch = prompts(z["seqs"], z["prompt"])
        for _ in range(max(3, warmup)):
            engine.generate(batch, 1, temperature=0.0)
        ms = _timed(lambda: engine.generate(batch, 1, temperature=0.0))
        tokens = z["seqs"] * z["prompt"]
        report({"workload": "prefill", "size": size, "model": label, "params": params, "seqs": z["seqs"],
                "prompt": z["prompt"], "ms": ms, "tokens_per_s": tokens / ms * 1e3})
        del engine
        engine = RolloutEngine(model, cfg, max_seqs=z["decode_seqs"], max_seq_len=z["decode_prompt"] + steps + 16)
        batch = prompts(z["decode_seqs"], z["decode_prompt"])
        for _ in range(2):
            engine.generate(batch, 4, temperature=0.0)
        short = _timed(lambda: engine.generate(batch, 1, temperature=0.0))
        long = _timed(lambda: engine.generate(batch, 1 + steps, temperature=0.0))
        ms = (long - short) / steps
        native.check_status()
        report({"workload": "decode", "size": size, "model": label, "seqs": z["decode_seqs"],
                "context": z["decode_prompt"], "ms_per_step": ms, "tokens_per_s": z["decode_seqs"] / ms * 1e3,
                "cache_bytes_per_token": engine.cache.bytes_per_token(),
                "state_bytes_per_sequence": getattr(engine.cache, "bytes_per_sequence", int)(),
                "gpu_launches": native.launches()})
        engine.release_graph()
        del engine, model
        torch.cuda.empty_cache()


def _time_rotating(make, nbytes: int) -> float:
    """Milliseconds per call of the callables that ``make()`` returns, each over inputs of its own (``nbytes`` large):
    as many copies as it takes to exceed L2 twice over, called in turn from one captured graph (as a decode step does),
    so that no launch gap is timed and no input is in cache."""
    calls = [make() for _ in range(max(2, min(64, -(-300 * 2 ** 20 // max(nbytes, 1)))))]
    for fn in calls[:2]:
        fn()
    torch.cuda.synchronize()
    rounds = max(1, 16 // len(calls))
    graph = torch.cuda.CUDAGraph()
    with torch.cuda.graph(graph):
        for _ in range(rounds):
            for fn in calls:
                fn()
    for _ in range(3):
        graph.replay()
    return _timed(graph.replay, 5) / (rounds * len(calls))


def _rand(*shape, dtype=torch.bfloat16, scale=1.0):
    return (torch.randn(*shape, device="cuda") * scale).to(dtype)


def _emitter(size, report):
    def emit(kernel, make, *, nbytes=None, flops=None, fma=None, special=None, **extra):
        ms = _time_rotating(make, nbytes or 2 ** 31)
        rec = {"kernel": kernel, "size": size, "us": ms * 1e3, **extra}
        if nbytes is not None:
            rec.update(gbs=nbytes / ms / 1e6, of_measured_hbm=nbytes / ms / 1e6 / HBM_GBS)
        if flops is not None:
            rec.update(tflops=flops / ms / 1e9, of_measured_gemm=flops / ms / 1e9 / BF16_TFLOPS)
        if fma is not None:
            rec.update(of_nominal_fp32=fma / ms / 1e9 / FP32_TFMA)
        if special is not None:
            rec.update(of_nominal_special=special / ms / 1e9 / SPECIAL_T)
        report(rec)
        torch.cuda.empty_cache()

    return emit


def bench_kedavik_kernels(size: str, report) -> None:
    from ironcore_b200.ops import attention, grouped, kernels, latent, recurrent, streams
    from ironcore_b200.rl import ops as RO

    z = KEDAVIK_SIZES[size]
    dev, bf, f32, rand, emit = "cuda", torch.bfloat16, dict(dtype=torch.float32), _rand, _emitter(size, report)
    d, ff, taps, n, inner = (z[k] for k in ("width", "ff", "conv", "state", "inner"))
    h, g, hd, e, k = (z[x] for x in ("heads", "kv", "head", "d_heads", "d_head"))
    lh = h
    for t in (z["seqs"] * z["prompt"], z["decode_seqs"]):
        few = t == z["decode_seqs"]
        n_seq = t if few else z["seqs"]
        seqs = torch.arange(n_seq, dtype=torch.int32, device=dev).repeat_interleave(t // n_seq)
        pos = torch.arange(t // n_seq, dtype=torch.int32, device=dev).repeat(n_seq) + (z["decode_prompt"] - 1 if few else 0)
        cu = None if few else torch.arange(0, t + 1, t // n_seq, dtype=torch.int32, device=dev)
        rows = recurrent.Rows(seqs, pos, cu, t // n_seq)
        one, nw, nwb = torch.ones(1, device=dev), rand(d, **f32), rand(d)
        mix = torch.ones(1, 1, device=dev)
        step, table, ids = rand(d, **f32), rand(z["vocab"], d), torch.randint(0, z["vocab"], (t,), device=dev)

        # ---- boundary beside residual + RMSNorm
        def boundary(add):
            src = streams.StreamWrite(rand(t, 1, d, **f32), rand(t, d), None, None, mix, one)
            extra = streams.StreamAdd(step, streams.TokenEmbed(ids, table, 8.0, 1)) if add else None
            return lambda: streams.boundary(src, one, nw, 1, 1e-5, width=d, dtype=bf, add=extra)

        def norm():
            x, y = rand(t, d), rand(t, d)
            return lambda: kernels.norm_fwd(x, nwb, None, 1e-5, True, residual=y)

        emit("stream_boundary", lambda: boundary(False), nbytes=t * d * 12, rows=t)
        emit("stream_boundary + pass inputs", lambda: boundary(True), nbytes=t * d * 14, rows=t)
        emit("norm_fwd+residual (llama)", norm, nbytes=t * d * 8, rows=t)

        # ---- activations
        def act():
            x = rand(t, ff)
            return lambda: kernels.act_fwd(x, "gelu")

        def glu():
            x = rand(t, 2 * ff)
            return lambda: kernels.glu_fwd(x, "swiglu")

        emit("gelu", act, nbytes=t * ff * 4, rows=t)
        emit("glu swiglu (llama)", glu, nbytes=t * ff * 6, rows=t)

        # ---- selective scan
        cw, cb = rand(taps, inner, **f32), rand(inner, **f32)

        def conv():
            x, state = rand(t, 2 * inner), rand(n_seq, taps - 1, inner)
            return lambda: recurrent.short_conv(x[:, :inner], cw, cb, state, rows)

        dtb, al, dd = rand(inner, **f32) - 4, rand(inner, (n + 3) // 4 * 4, **f32), rand(inner, **f32)
        rank = z["dt_rank"]

        def scan():
            u, zz, raw, bc = rand(t, inner), rand(t, 2 * inner), rand(t, inner, **f32), rand(t, rank + 2 * n)
            state, out = torch.zeros(n_seq, inner, n, device=dev), torch.empty(t, inner, dtype=bf, device=dev)
            return lambda: recurrent.selective_scan(u, raw, zz[:, inner:], bc, rank, rank + n, n, dtb, al, dd, state, rows, out)

        emit("short_conv", conv, nbytes=inner * (t * 4 + n_seq * (taps - 1) * (4 if few else 2)), rows=t)
        emit("selective_scan", scan, nbytes=t * (inner * 10 + 4 * n) + n_seq * inner * n * (8 if few else 4),
             special=t * inner * n, fma=4 * t * inner * n, rows=t)

        # ---- gated delta rule
        c = 3 * e * k
        dcw, dal, ddt, ow = rand(taps, c, **f32), torch.zeros(e, device=dev), rand(e * k, **f32) - 4, rand(k, **f32)
        sizes = dict(groups=e, heads=e, dim=k, vdim=k)

        def prepared():
            x, a, b = rand(t, c + 8), rand(t, e * k, **f32), rand(t, (e + 7) // 8 * 8)
            state = rand(n_seq, taps - 1, c)
            return lambda: recurrent.delta_prepare(x[:, :c], dcw, state, b[:, :e], a, dal, ddt, rows, q_scale=k ** -0.5, **sizes)

        def rule():
            ins = recurrent.DeltaInputs(*(torch.nn.functional.normalize(rand(t, e, k, **f32), dim=-1).view(t, -1) for _ in range(2)),
                                        rand(t, e, **f32), torch.rand(t, e * k, device=dev) * 0.1 + 0.9, rand(t, e * k),
                                        torch.rand(t, e, device=dev))
            state = torch.zeros(n_seq, e, k, recurrent.state_dim(k), device=dev)
            return lambda: recurrent.delta_rule(ins, state, rows, **sizes)

        def output():
            o, gt, y = rand(t, e * k, **f32), rand(t, e * k, **f32), torch.empty(t, e * k, dtype=bf, device=dev)
            return lambda: recurrent.delta_output(o, gt, ow, 1e-5, 0.7, heads=e, vdim=k, valid=k, out=y)

        emit("delta_prepare", prepared, nbytes=t * e * k * (6 + 8 + 8 + 2) + n_seq * (taps - 1) * c * (4 if few else 2), rows=t)
        emit("delta_rule", rule, nbytes=t * e * k * 18 + n_seq * e * k * k * (8 if few else 4), fma=4 * t * e * k * k, rows=t)
        emit("delta_output", output, nbytes=t * e * k * 10, rows=t)

        # ---- rotary + cache rows beside the transformer's two kernels
        def rope(heads, groups, fused):
            cols = (heads + 2 * groups) * hd
            x = rand(t, cols + heads)
            kc, vc = rand(t, groups * hd), rand(t, groups * hd)
            slots, freq = torch.randperm(t, device=dev), grouped.rotary_frequencies(hd, 1e4).to(dev)
            nq, nk = heads * hd, groups * hd

            def two():
                kernels.rope(x, x, nheads=heads + groups, head_dim=hd, tokens=t, seq_len=1, base=1e4, interleaved=False,
                             pos_ids=pos, row_stride=x.stride(0), out_stride=x.stride(0))
                RO.kv_append(x[:, nq:nq + nk], x[:, nq + nk:nq + 2 * nk], kc, vc, slots)

            return two if not fused else lambda: grouped.rope_cache(x, freq, pos, heads=heads, groups=groups, kd=hd, vd=hd,
                                                                     k_cache=kc, v_cache=vc, slots=slots, gate_scale=0.7)

        emit("rope_cache", lambda: rope(h, g, True), nbytes=t * hd * ((h + g) * 4 + g * 2 + g * 4) + t * h * 6, rows=t)
        emit("rope + kv_append (llama)", lambda: rope(lh, lh, False), nbytes=t * hd * (2 * lh * 4 + lh * 4 + lh * 4), rows=t)

        # ---- narrow products beside a wide one
        def gemm(kk, nn, dt=bf):
            x, m = rand(t, kk), rand(nn, kk)
            return lambda: latent.project(x, m, dt)

        for label, kk, nn, dt in (("scan x", inner, rank + 2 * n, bf), ("scan step", rank, inner, torch.float32),
                                  ("decay", z["rank"], e * k, torch.float32), ("q of llama", d, d, bf)):
            emit(f"gemm {label}", lambda: gemm(kk, nn, dt), nbytes=2 * (t * kk + nn * kk) + t * nn * dt.itemsize,
                 flops=2.0 * t * kk * nn, rows=t, k=kk, n=nn)
    # ---- prompt attention
    m, p, chunk = z["seqs"], z["prompt"], z["chunk"]
    cu = torch.arange(0, (m + 1) * p, p, dtype=torch.int32, device=dev)

    def chunked():
        x, gt, y = rand(m * p, (h + 2 * g) * hd + h), torch.rand(m * p, h, device=dev), torch.empty(m * p, 2 * h * hd, dtype=bf, device=dev)
        return lambda: grouped.attend_prompts(x, heads=h, groups=g, hd=hd, cu_seqlens=cu, max_len=p, window=0, chunk=chunk,
                                              scale=hd ** -0.5, gate=gt, out=y[:, :h * hd])

    def causal():
        qkv = rand(m * p, 3 * lh * hd)
        return lambda: attention.flash_fwd(qkv, lh, lh, hd, p)

    emit("flash chunked + gate", chunked, flops=4.0 * m * sum(i % chunk + 1 for i in range(p)) * h * hd, seqs=m, prompt=p, chunk=chunk)
    emit("flash causal (llama)", causal, flops=4.0 * m * p * (p + 1) / 2 * lh * hd, seqs=m, prompt=p)
    # ---- decode attention
    b, ctx = z["decode_seqs"], z["decode_prompt"]
    seqs = torch.arange(b, dtype=torch.int32, device=dev)
    pos = torch.full((b,), ctx - 1, dtype=torch.int32, device=dev)

    def paged(heads, groups, chunked):
        bs = 64 if chunked else 16
        table = torch.randperm(b * ((ctx + bs - 1) // bs), device=dev).to(torch.int32).view(b, -1)
        q, kc, vc = rand(b, heads * hd), rand(table.numel(), bs, groups, hd), rand(table.numel(), bs, groups, hd)
        out, gt = torch.empty(b, heads * hd, dtype=bf, device=dev), torch.rand(b, heads, device=dev)
        if not chunked:
            return lambda: RO.paged_decode(q, kc, vc, table, pos + 1, heads, groups, hd)
        return lambda: grouped.attend_rows(q, kc, vc, table, bs, seqs, pos, heads=heads, groups=groups, kd=hd, vd=hd, window=0,
                                           chunk=chunk, scale=hd ** -0.5, max_keys=min(chunk, ctx), gate=gt, out=out)

    seen = (ctx - 1) % chunk + 1
    emit("paged decode, chunk", lambda: paged(h, g, True), nbytes=b * seen * g * hd * 4, seqs=b, keys=seen, kv_heads=g)
    for groups in (lh, max(1, lh // 4)):
        emit(f"paged decode (llama, {groups} kv heads)", lambda: paged(lh, groups, False), nbytes=b * ctx * groups * hd * 4, seqs=b,
             keys=ctx)


def bench_stream_kernels(size: str, report) -> None:
    from ironcore_b200.ops import attention, kernels, latent, streams
    from ironcore_b200.rl import ops as RO

    z = SIZES[size]
    dev, bf, f32, rand, emit = "cuda", torch.bfloat16, dict(dtype=torch.float32), _rand, _emitter(size, report)
    d, h, hd, r, ff, s, w = (z[k] for k in ("width", "heads", "head", "kv_rank", "ff", "streams", "window"))

    for t in (z["seqs"] * z["prompt"], z["decode_seqs"]):
        few = t == z["decode_seqs"]
        # ---- sublayer boundary beside residual + RMSNorm
        mix, out, read = rand(s, s, **f32), rand(s, **f32), rand(s, **f32)
        nw, gb, sw, nwb = rand(d, **f32), rand(d, **f32), rand(d, **f32), rand(d)
        n_seq = t if few else z["seqs"]
        seqs = torch.arange(n_seq, dtype=torch.int32, device=dev).repeat_interleave(t // n_seq)
        pos = torch.arange(t // n_seq, dtype=torch.int32, device=dev).repeat(n_seq)

        def boundary(shifted):
            src = streams.StreamWrite(rand(t, s, d, **f32), rand(t, d), rand(t, d), gb, mix, out)
            state = torch.zeros(n_seq, d, device=dev)
            shift = streams.TokenShift(sw, state, state, seqs, pos) if shifted else None
            return lambda: streams.boundary(src, read, nw, z["groups"], 1e-5, width=d, dtype=bf, shift=shift)

        def norm():
            x, y = rand(t, d), rand(t, d)
            return lambda: kernels.norm_fwd(x, nwb, None, 1e-5, True, residual=y)

        base = t * d * (2 * s * 4 + 2 + 2 + 2)
        emit("stream_boundary", lambda: boundary(False), nbytes=base, rows=t, streams=s)
        emit("stream_boundary+shift", lambda: boundary(True), nbytes=base + t * d * 2, rows=t, streams=s)
        emit("norm_fwd+residual (llama)", norm, nbytes=t * d * 8, rows=t)
        # ---- latents, gated activation
        zc = z["q_rank"] + r + h
        qn, cn = rand(z["q_rank"], **f32), rand(r, **f32)
        slots = torch.arange(t, device=dev)

        def norms():
            zin, cache = rand(t, (zc + 7) // 8 * 8, **f32), torch.zeros(t, r, dtype=bf, device=dev)
            return lambda: latent.latent_norm(zin, qn, cn, h, 1e-5, q_width=z["q_rank"], c_width=r, dtype=bf, cache=cache,
                                              slots=slots, want_latent=not few)

        def glu(name, cols):
            up = rand(t, cols)
            return lambda: kernels.glu_fwd(up[:, :2 * ff], name)

        emit("latent_norm", norms, nbytes=t * (zc * 4 + z["q_rank"] * 2 + r * 2 * (1 if few else 2) + h * 4), rows=t)
        emit("glu geglu, strided", lambda: glu("geglu", 2 * ff + d), nbytes=t * ff * 6, rows=t)
        emit("glu swiglu (llama)", lambda: glu("swiglu", 2 * ff), nbytes=t * ff * 6, rows=t)
    # ---- prompt attention: windowed and gated beside causal
    n, p = z["seqs"], z["prompt"]
    cu = torch.arange(0, (n + 1) * p, p, dtype=torch.int32, device=dev)

    def windowed():
        q, kv, g = rand(n * p, h * hd), rand(n * p, 2 * h * hd), torch.rand(n * p, h, device=dev)
        return lambda: attention.flash_fwd_window(q, kv, h, hd, cu, p, scale=hd ** -0.5, window=w, gate=g)

    def causal():
        qkv = rand(n * p, 3 * h * hd)
        return lambda: attention.flash_fwd(qkv, h, h, hd, p)

    emit("flash window+gate", windowed, flops=4.0 * n * sum(min(i + 1, w) for i in range(p)) * h * hd, seqs=n, prompt=p,
         window=w)
    emit("flash causal (llama)", causal, flops=4.0 * n * p * (p + 1) / 2 * h * hd, seqs=n, prompt=p)
    # ---- decode attention: latent beside paged K / V
    b, ctx = z["decode_seqs"], max(w, z["decode_prompt"])
    seqs = torch.arange(b, dtype=torch.int32, device=dev)
    pos = torch.full((b,), ctx - 1, dtype=torch.int32, device=dev)
    lens = pos + 1
    seen = min(w, ctx)

    def tables(bs):
        return torch.randperm(b * ((ctx + bs - 1) // bs), device=dev).to(torch.int32).view(b, -1)

    def latents(bs, legacy=False):
        table, q = tables(bs), rand(b, h, r, scale=0.1)
        lat = rand(table.numel() * bs, r)
        return lambda: latent.latent_attend(q, lat, table, bs, seqs, pos, window=w, scale=hd ** -0.5, max_keys=seen,
                                            legacy=legacy)

    def paged(hkv):
        table, q = tables(16), rand(b, h * hd)
        kc, vc = rand(table.numel(), 16, hkv, hd), rand(table.numel(), 16, hkv, hd)
        return lambda: RO.paged_decode(q, kc, vc, table, lens, h, hkv, hd)

    work = dict(nbytes=b * (seen * r * 2 + 2 * h * r * 2), flops=4.0 * b * h * seen * r, seqs=b, keys=seen)
    emit("latent_attend, pages of 64", lambda: latents(64), **work)
    emit("latent_attend, pages of 16", lambda: latents(16), **work)
    emit("latent_attend, mma.sync", lambda: latents(64, True), **work)
    for hkv in (h, max(1, h // 8)):
        emit(f"paged_decode (llama, {hkv} kv heads)", lambda: paged(hkv), nbytes=b * ctx * hkv * hd * 4,
             flops=4.0 * b * h * ctx * hd, seqs=b, keys=ctx)

    def product(k, n_out, gated):
        x, m, g = rand(b, h, k), rand(h, n_out, k), (torch.rand(b, h, device=dev) if gated else None)
        return lambda: latent.head_product(x, m, g)

    def gemm(k, n_out):
        x, m = rand(b, k), rand(n_out, k)
        return lambda: kernels.mm_nt(x, m)

    emit("head_product, query side", lambda: product(hd, r, False), nbytes=2 * h * (r * hd + b * (hd + r)), seqs=b)
    emit("head_product, output side", lambda: product(r, hd, True), nbytes=2 * h * (r * hd + b * (hd + r)), seqs=b)
    for label, k, n_out in (("o proj", d, h * hd), ("as many weights as a head product", r, h * hd)):
        emit(f"decode gemm (llama, {label})", lambda: gemm(k, n_out), nbytes=2 * (n_out * k + b * (k + n_out)), seqs=b)


def run(args) -> int:
    from bench import ClockSampler

    torch.cuda.set_device(0)
    sampler = ClockSampler(0)
    sampler.start()

    def report(rec):
        print(json.dumps(rec), flush=True)

    for size in ([args.size] if args.size else list(SIZES)):
        (bench_stream_kernels if args.family == "tetepel" else bench_kedavik_kernels)(size, report)
        if not args.kernels_only:
            bench_models(args.family, size, max(args.steps, 128), args.warmup, report)
    report({"workload": "serving", "family": args.family, "data": "synthetic", "dtype": "bf16", "clocks": sampler.stop(),
            "l2": "kernel inputs rotate over copies that exceed it twice; model weights exceed it"})
    return 0
