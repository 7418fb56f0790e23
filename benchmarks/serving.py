"""Serving throughput of the residual-stream family (Tetepel) beside the Llama-style transformer of equal size, and
its kernels beside the like kernels of that model.

``python bench.py --workload serving [--size 2k|4k] [--kernels-only]``; one JSON line per measurement. Random weights
and tokens. Model numbers go through ``RolloutEngine.generate``: prefill is a generation of one token, a decode step is
the difference between a long and a one-token generation over the number of extra steps, both timed with CUDA events
after warm-up (the weights of the timed layers exceed the 126 MB L2). Kernel numbers flush L2 between launches; bytes
and FLOPs are the algorithmic ones."""

from __future__ import annotations

import json

import torch

HBM_GBS, BF16_TFLOPS = 6559.7, 1670.1      # measured on this pool: copy bandwidth, burst GEMM rate

SIZES = {
    "4k": dict(width=4096, heads=32, head=128, q_rank=1536, kv_rank=512, ff=11008, streams=4, groups=8, window=2048,
               vocab=32000, layers=4, prompt=4096, seqs=4, decode_seqs=64, decode_prompt=2048),
    "2k": dict(width=2048, heads=16, head=128, q_rank=768, kv_rank=256, ff=5632, streams=2, groups=4, window=1024,
               vocab=32000, layers=8, prompt=4096, seqs=8, decode_seqs=128, decode_prompt=1024),
}


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


def bench_models(size: str, steps: int, warmup: int, report) -> None:
    from ironcore_b200.ops import native
    from ironcore_b200.rl import RolloutEngine

    z = SIZES[size]
    for label, build in (("tetepel", _stream_model), ("llama", _llama_model)):
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
                "cache_bytes_per_token": engine.cache.bytes_per_token(), "gpu_launches": native.launches()})
        engine.release_graph()
        del engine, model
        torch.cuda.empty_cache()


def bench_stream_kernels(size: str, report) -> None:
    from ironcore_b200.ops import attention, kernels, latent, streams
    from ironcore_b200.rl import ops as RO

    from .kernels import _flush_buffer, time_cuda

    z = SIZES[size]
    dev, bf = "cuda", torch.bfloat16
    flush = _flush_buffer()
    d, h, hd, r, ff, s = z["width"], z["heads"], z["head"], z["kv_rank"], z["ff"], z["streams"]
    w = z["window"]

    def rand(*shape, dtype=bf, scale=1.0):
        return (torch.randn(*shape, device=dev) * scale).to(dtype)

    def emit(kernel, fn, *, nbytes=None, flops=None, **extra):
        ms = time_cuda(fn, flush=flush)
        rec = {"kernel": kernel, "size": size, "us": ms * 1e3, **extra}
        if nbytes is not None:
            rec.update(gbs=nbytes / ms / 1e6, of_measured_hbm=nbytes / ms / 1e6 / HBM_GBS)
        if flops is not None:
            rec.update(tflops=flops / ms / 1e9, of_measured_gemm=flops / ms / 1e9 / BF16_TFLOPS)
        report(rec)

    # ---- sublayer boundary beside residual + RMSNorm
    for t in (z["seqs"] * z["prompt"], z["decode_seqs"]):
        x = rand(t, s, d, dtype=torch.float32)
        y, gate = rand(t, d), rand(t, d)
        f32 = dict(dtype=torch.float32)
        mix, out, read = rand(s, s, **f32), rand(s, **f32), rand(s, **f32)
        nw, gb, sw = rand(d, **f32), rand(d, **f32), rand(d, **f32)
        n_seq = z["seqs"] if t > z["decode_seqs"] else t
        seqs = torch.arange(n_seq, dtype=torch.int32, device=dev).repeat_interleave(t // n_seq)
        pos = torch.arange(t // n_seq, dtype=torch.int32, device=dev).repeat(n_seq)
        state = torch.zeros(n_seq, d, device=dev)
        src = streams.StreamWrite(x, y, gate, gb, mix, out)
        shift = streams.TokenShift(sw, state, state, seqs, pos)
        base = t * d * (2 * s * 4 + 2 + 2 + 2)
        emit("stream_boundary", lambda: streams.boundary(src, read, nw, z["groups"], 1e-5, width=d, dtype=bf),
             nbytes=base, rows=t, streams=s)
        emit("stream_boundary+shift",
             lambda: streams.boundary(src, read, nw, z["groups"], 1e-5, width=d, dtype=bf, shift=shift),
             nbytes=base + t * d * 2, rows=t, streams=s)
        nwb = rand(d)
        emit("norm_fwd+residual (llama)", lambda: kernels.norm_fwd(y, nwb, None, 1e-5, True, residual=gate),
             nbytes=t * d * 8, rows=t)
        zc = z["q_rank"] + r + h
        zin = rand(t, (zc + 7) // 8 * 8, **f32)
        qn, cn = rand(z["q_rank"], **f32), rand(r, **f32)
        cache = torch.zeros(t, r, dtype=bf, device=dev)
        slots = torch.arange(t, device=dev)
        emit("latent_norm", lambda: latent.latent_norm(zin, qn, cn, h, 1e-5, q_width=z["q_rank"], c_width=r, dtype=bf,
                                                       cache=cache, slots=slots, want_latent=t > 256),
             nbytes=t * (zc * 4 + z["q_rank"] * 2 + r * 2 * (2 if t > 256 else 1) + h * 4), rows=t)
        up = rand(t, 2 * ff + d)
        emit("glu geglu (strided)", lambda: kernels.glu_fwd(up[:, :2 * ff], "geglu"), nbytes=t * ff * 6, rows=t)
        up2 = up[:, :2 * ff].contiguous()
        emit("glu swiglu (llama)", lambda: kernels.glu_fwd(up2, "swiglu"), nbytes=t * ff * 6, rows=t)
        del x, y, gate, up, up2, zin, src, cache
        torch.cuda.empty_cache()
    # ---- prompt attention: windowed and gated beside causal
    n, p = z["seqs"], z["prompt"]
    q, kv, g = rand(n * p, h * hd), rand(n * p, 2 * h * hd), torch.rand(n * p, h, device=dev)
    cu = torch.arange(0, (n + 1) * p, p, dtype=torch.int32, device=dev)
    pairs = n * sum(min(i + 1, w) for i in range(p))
    emit("flash window+gate", lambda: attention.flash_fwd_window(q, kv, h, hd, cu, p, scale=hd ** -0.5, window=w, gate=g),
         flops=4.0 * pairs * h * hd, seqs=n, prompt=p, window=w)
    qkv = torch.cat([q, kv], dim=1)
    emit("flash causal (llama)", lambda: attention.flash_fwd(qkv, h, h, hd, p), flops=4.0 * n * p * (p + 1) / 2 * h * hd,
         seqs=n, prompt=p)
    del q, kv, qkv
    # ---- decode attention: latent beside paged K / V
    b, ctx, bs = z["decode_seqs"], max(w, z["decode_prompt"]), 16
    blocks = b * ((ctx + bs - 1) // bs)
    table = torch.randperm(blocks, device=dev).to(torch.int32).view(b, -1)
    seqs = torch.arange(b, dtype=torch.int32, device=dev)
    pos = torch.full((b,), ctx - 1, dtype=torch.int32, device=dev)
    lat = rand(blocks * bs, r)
    qa = rand(b, h, r, scale=0.1)
    seen = min(w, ctx)
    emit("latent_attend", lambda: latent.latent_attend(qa, lat, table, bs, seqs, pos, window=w, scale=hd ** -0.5,
                                                       max_keys=seen),
         nbytes=b * (seen * r * 2 + 2 * h * r * 2), flops=4.0 * b * h * seen * r, seqs=b, keys=seen)
    uk = rand(h, r, hd)
    qh, oc, uv, gt = rand(b, h, hd), rand(b, h, r), rand(h, hd, r), torch.rand(b, h, device=dev)
    emit("head_product (query side)", lambda: latent.head_product(qh, uk), nbytes=2 * (uk.numel() + b * h * (hd + r)), seqs=b)
    emit("head_product (output side)", lambda: latent.head_product(oc, uv, gt),
         nbytes=2 * (uv.numel() + b * h * (hd + r)), seqs=b)
    wq = rand(h * hd, d)
    xq = rand(b, d)
    emit("decode gemm (llama, o proj)", lambda: kernels.mm_nt(xq, wq), nbytes=2 * (wq.numel() + b * (d + h * hd)), seqs=b)
    for hkv in (h, max(1, h // 8)):
        kc, vc = rand(blocks, bs, hkv, hd), rand(blocks, bs, hkv, hd)
        qd = rand(b, h * hd)
        lens = pos + 1
        emit(f"paged_decode (llama, {hkv} kv heads)", lambda: RO.paged_decode(qd, kc, vc, table, lens, h, hkv, hd),
             nbytes=b * ctx * hkv * hd * 4, flops=4.0 * b * h * ctx * hd, seqs=b, keys=ctx)
        del kc, vc


def run(args) -> int:
    from bench import ClockSampler

    torch.cuda.set_device(0)
    sampler = ClockSampler(0)
    sampler.start()

    def report(rec):
        print(json.dumps(rec), flush=True)

    for size in ([args.size] if args.size else list(SIZES)):
        bench_stream_kernels(size, report)
        if not args.kernels_only:
            bench_models(size, max(args.steps, 32), args.warmup, report)
    report({"workload": "serving", "data": "synthetic", "dtype": "bf16", "clocks": sampler.stop(),
            "l2": "flushed between kernel launches; model weights exceed it"})
    return 0
