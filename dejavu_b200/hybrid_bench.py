"""Prefill and decode throughput of the Ninolorn design beside the dense OPT decoder at equal width and weight count,
and every kernel of both with its fraction of the measured roofline (bench.py --hybrid).

Random weights, random prompt tokens. Throughput is timed with CUDA events around whole steps: prompt passes run
eagerly, decode steps are replays of the captured graph. Kernels are timed alone, as graphs of launches that rotate
over buffers larger than L2.
"""
from __future__ import annotations

import statistics

import torch

from . import _lib, ops
from .generation import allocate_kv_cache, InferenceParams, step, update_graph_cache
from .gpt import GPTLMHeadModel, apply_sparsity_knobs, opt_config
from .ninolorn import NinolornForCausalLM

# width, layers: (OPT heads, OPT ffn) and the hybrid's head sizes; weights per layer are about equal
SIZES = {
    "1b": dict(width=2048, layers=12, opt=(32, 8192), heads=16, kv=4, gla=8, ff=5632),
    "7b": dict(width=4096, layers=8, opt=(32, 16384), heads=32, kv=8, gla=16, ff=11008),
    "30b": dict(width=7168, layers=4, opt=(56, 28672), heads=56, kv=8, gla=28, ff=19456),
}
VOCAB, WINDOW, STREAMS = 50272, 1024, 4


def hybrid_config(size: dict) -> dict:
    rot = {"base": 500000.0, "dims": 128, "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}
    mlp = {"kind": "dense", "ff": size["ff"], "limit": 7.0}
    att = {"type": "attention", "mlp": mlp,
           "mixer": {"heads": size["heads"], "kv_heads": size["kv"], "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                     "mask": {"size": WINDOW}, "rot": rot}}
    gla = {"type": "gla", "mlp": mlp, "mixer": {"heads": size["gla"], "dim": 128, "vdim": 256, "tau": 16.0}}
    return {"architecture": "Ninolorn", "vocab": VOCAB, "width": size["width"], "streams": STREAMS,
            "layers": [gla, att] * (size["layers"] // 2), "loop": None, "norm": {"eps": 1e-6}, "logit_softcap": 30.0}


def opt_model(size: dict, max_len: int, dev):
    heads, ffn = size["opt"]
    cfg = opt_config("opt-125m", n_layer=size["layers"], n_embd=size["width"], hidden_size=size["width"], n_head=heads,
                     n_inner=ffn, vocab_size=VOCAB, max_position_embeddings=max_len, n_positions=max_len)
    apply_sparsity_knobs(cfg, ffn, heads, heads, 1)
    return GPTLMHeadModel(cfg, device=dev, dtype=torch.float16).eval().init_random(0), cfg


def time_prefill(model, n: int, B: int, reps: int, dev) -> float:
    """ms of one prompt pass of B sequences of n tokens (logits of the last token)."""
    ids = torch.randint(0, VOCAB, (B, n), device=dev)
    ip = InferenceParams(max_sequence_len=n, max_batch_size=B, key_value_memory_dict=allocate_kv_cache(model, B, n, dev))
    times = []
    for i in range(3 + reps):
        ip.sequence_len_offset = 0
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        e0.record()
        step(model, ip, ids, logit_rows=[n - 1])
        e1.record()
        torch.cuda.synchronize()
        if i >= 3:
            times.append(e0.elapsed_time(e1))
    return statistics.median(times)


def time_decode(model, prompt: int, B: int, steps: int, dev) -> float:
    """ms of one captured decode step of B sequences behind a prompt."""
    with torch.inference_mode():
        cache = update_graph_cache(model, None, B, prompt, prompt + steps + 32, greedy_feedback=True, vocab_size=VOCAB)
        ip = cache.inference_params
        ip.sequence_len_offset = 0
        logits = step(model, ip, torch.randint(0, VOCAB, (B, prompt), device=dev), logit_rows=[prompt - 1])[:, -1]
        cache.input_ids.copy_(logits.argmax(-1, keepdim=True))
        cache.position_ids.fill_(prompt)
        for _ in range(8):
            cache.graph.replay()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        e0.record()
        for _ in range(steps):
            cache.graph.replay()
        e1.record()
        torch.cuda.synchronize()
        ms = e0.elapsed_time(e1) / steps
        del cache
    return ms


def kernel_table(hyb, opt, opt_cfg, size, n, kernel_timing, gbs, tflops, dev) -> dict:
    """us and fraction of roofline (the slower of bytes / bandwidth and flops / tensor peak) of each kernel alone."""
    out = {}
    g = torch.Generator(device=dev).manual_seed(1)

    def rec(name, us, nbytes, flops=0.0):
        ideal = max(nbytes / gbs / 1e3, flops / tflops / 1e6)
        out[name] = {"us": round(us, 2), "bytes": int(nbytes), "gflop": round(flops / 1e9, 3), "frac": round(ideal / us, 3)}

    def rand(*s, dtype=torch.bfloat16):
        return torch.randn(*s, device=dev, generator=g, dtype=torch.float32).to(dtype)

    gl = [l for l in hyb.layers if hasattr(l.mixer, "a2")]
    at = [l for l in hyb.layers if not hasattr(l.mixer, "a2")]
    D, S = size["width"], STREAMS
    H, G, dk, dv, W = size["heads"], size["kv"], 128, 128, WINDOW
    GH, gk, gv = size["gla"], 128, 256
    x, xh = rand(1, D), rand(1, D, dtype=torch.float16)
    copies = 1 + int(2.6e8 / (D * 3 * D * 2)) // len(at)  # enough distinct weights to stay out of L2

    def gemv(name, lin, x, **kw):
        ws = [l.weight for l in lin]
        ws = ws + [w.detach().clone() for w in ws for _ in range(copies)]
        us = kernel_timing([lambda w=w: ops.linear_gemv(x, w, **kw) for w in ws])
        M, N = ws[0].shape
        rec(name, us, M * N * 2 + N * 2 + M * 2)

    gemv("decode.qkv", [l.mixer.qkv for l in at], x)
    gemv("decode.gla_proj", [l.mixer.proj for l in gl], x)
    gemv("decode.o", [l.mixer.o for l in at], rand(1, H * dv), out_dtype=torch.float32)
    gemv("decode.gate_up", [l.mlp.gate_up for l in hyb.layers], x, activation="clamped_glu", param=7.0)
    gemv("decode.down", [l.mlp.down for l in hyb.layers], rand(1, size["ff"]), out_dtype=torch.float32)

    def opt_gemv(name, ws, x, fn=ops.dense_gemv, **kw):
        ws = ws + [w.detach().clone() for w in ws for _ in range(copies)]
        us = kernel_timing([lambda w=w: fn(x, w, **kw) for w in ws])
        rec(name, us, ws[0].numel() * 2)

    ol = list(opt.transformer.layers)
    opt_gemv("opt.decode.qkv", [l.mixer.Wqkv.weight for l in ol], xh)
    opt_gemv("opt.decode.o", [l.mixer.out_proj.weight for l in ol], xh)
    opt_gemv("opt.decode.fc1", [l.mlp.fc1.weight for l in ol], xh, activation="relu")
    opt_gemv("opt.decode.fc2", [l.mlp.fc2.weight_t for l in ol], rand(1, opt_cfg.n_inner, dtype=torch.float16),
             fn=ops.dense_transposed_gemv)

    # residual boundary: decode and prompt rows
    hc = hyb.layers[0].hc1
    norm = ol[0].norm1
    for rows, tag in ((1, "decode"), (n, "prefill")):
        k = 2 + int(2.6e8 / (rows * S * D * 4)) if rows > 1 else 8
        xs, ys = [rand(rows, S, D, dtype=torch.float32) for _ in range(k)], [rand(rows, D, dtype=torch.float32) for _ in range(k)]
        us = kernel_timing([lambda a=a, b=b: ops.hyper_step(a, b, hc.mix, hc.w_out, hc.w_in, hyb.layers[0].norm1, 1e-6,
                                                            torch.bfloat16, x_out=a) for a, b in zip(xs, ys)])
        rec(f"{tag}.hyper_step", us, rows * D * (8 * S + 4 + 2))
        del xs, ys
        hs = [rand(rows, D, dtype=torch.float16) for _ in range(2 * k)]
        if rows == 1:
            us = kernel_timing([lambda a=a, b=b: ops.add_layernorm(a, b, norm.weight, norm.bias, 1e-5)
                                for a, b in zip(hs[::2], hs[1::2])])
        else:
            us = kernel_timing([lambda a=a, b=b: norm(a + b) for a, b in zip(hs[::2], hs[1::2])])
        rec(f"opt.{tag}.add_norm", us, rows * D * 2 * 4)
        del hs

    # decode attention: the window (or the state) against OPT's cache of as many tokens
    k = 2 + int(2.6e8 / (G * W * (dk + dv) * 2))
    m = at[0].mixer
    pos = torch.full((1,), 5 * W + 3, dtype=torch.int64, device=dev)
    rings = [(rand(1, G, W, dk), rand(1, G, W, dv)) for _ in range(k)]
    row = rand(1, (H + G) * dk + G * dv)
    us = kernel_timing([lambda c=c: ops.window_attention_decode(row, *c, m.sink, m.rotary.freqs, m.rotary.amp, pos, H, W,
                                                                m.scale) for c in rings])
    rec("decode.window_attn", us, G * W * (dk + dv) * 2)
    st = [rand(1, GH, gk, gv, dtype=torch.float32) for _ in range(2 + int(2.6e8 / (GH * gk * gv * 4)))]
    mg = gl[0].mixer
    prow = rand(1, mg.proj.weight.shape[0])
    gla_args = (mg.a2, mg.a2_bias, mg.tau, mg.norm, mg.eps, mg.scale)
    us = kernel_timing([lambda s=s: ops.gated_linear_attention(prow, *gla_args, s, pos, 1) for s in st])
    rec("decode.gla", us, 2 * GH * gk * gv * 4 + mg.a2.numel() * 4)
    oh, od = opt_cfg.n_head, opt_cfg.hidden_size // opt_cfg.n_head
    kv = [(rand(1, oh, od // 8, W, 8, dtype=torch.float16), rand(1, oh, W, od, dtype=torch.float16))
          for _ in range(2 + int(2.6e8 / (oh * W * od * 4)))]
    q = rand(1, oh, od, dtype=torch.float16)
    us = kernel_timing([lambda c=c: ops.decode_attention(q, c[0], c[1], None, W, od ** -0.5) for c in kv])
    rec("opt.decode.attn", us, 2 * oh * W * od * 2)
    del rings, st, kv

    # prompt attention
    p0 = torch.zeros(1, dtype=torch.int64, device=dev)
    ring = (rand(1, G, W, dk), rand(1, G, W, dv))
    rows = [rand(n, (H + G) * dk + G * dv) for _ in range(3)]
    pairs = sum(min(i + 1, W) for i in range(n))
    us = kernel_timing([lambda r=r: ops.window_attention(r, *ring, m.sink, p0, n, H, W, m.scale) for r in rows])
    rec("prefill.window_attn", us, n * ((H + G) * dk + G * dv + H * dv) * 2, 2.0 * pairs * H * (dk + dv))
    us = kernel_timing([lambda r=r: ops.rotary_(r, m.rotary.freqs, m.rotary.amp, p0, n, H + G, dk) for r in rows])
    rec("prefill.rotary", us, n * (H + G) * dk * 4)
    rows = [rand(n, mg.proj.weight.shape[0]) for _ in range(3)]
    state = rand(1, GH, gk, gv, dtype=torch.float32)
    us = kernel_timing([lambda r=r: ops.gated_linear_attention(r, *gla_args, state, p0, n) for r in rows])
    # flops of the recurrence itself: state update and read-out
    rec("prefill.gla", us, n * GH * (2 * gk + 3 * gv) * 2, 4.0 * n * GH * gk * gv)
    rows = [rand(n, 2 * size["ff"]) for _ in range(3)]
    us = kernel_timing([lambda r=r: ops.glu(r, "clamped_glu", 7.0) for r in rows])
    rec("prefill.clamped_glu", us, n * size["ff"] * 6)
    import torch.nn.functional as F

    qkv = [rand(3, 1, oh, n, od, dtype=torch.float16) for _ in range(3)]
    us = kernel_timing([lambda t=t: F.scaled_dot_product_attention(t[0], t[1], t[2], is_causal=True) for t in qkv])
    rec("opt.prefill.sdpa", us, 4 * n * oh * od * 2, 2.0 * n * (n + 1) / 2 * oh * od * 2)
    rows = [rand(n, opt_cfg.n_inner, dtype=torch.float16) for _ in range(3)]
    us = kernel_timing([lambda r=r: F.relu(r) for r in rows])
    rec("opt.prefill.relu", us, n * opt_cfg.n_inner * 4)
    xs, w = rand(n, D), hyb.layers[0].mlp.gate_up.weight
    us = kernel_timing([lambda: torch.mm(xs, w.t())])
    rec("prefill.gate_up_gemm", us, 0, 2.0 * n * w.numel())
    return out


def run(names, kernel_timing, gbs: float, tflops: float, prompt: int = 4096, steps: int = 64, kernels: bool = True) -> dict:
    dev = torch.device("cuda", 0)
    out = {}
    for name in names:
        size = SIZES[name]
        hyb = NinolornForCausalLM(hybrid_config(size), device=dev).eval().init_random(0)
        opt, cfg = opt_model(size, prompt + steps + 64, dev)
        res = {"width": size["width"], "layers": size["layers"], "prompt": prompt,
               "hybrid_params": sum(p.numel() for p in hyb.parameters()), "opt_params": sum(p.numel() for p in opt.parameters())}
        with torch.inference_mode():
            for tag, model in (("hybrid", hyb), ("opt_dense", opt)):
                ms = time_prefill(model, prompt, 1, 5, dev)
                res[tag] = {"prefill_tokens_per_s": round(prompt / ms * 1e3), "prefill_ms": round(ms, 3)}
                for B in (1, 8):
                    ms = time_decode(model, min(prompt, 1024), B, steps, dev)
                    res[tag][f"decode_b{B}"] = {"ms_per_step": round(ms, 4), "tokens_per_s": round(B / ms * 1e3)}
            if kernels:
                res["kernels"] = kernel_table(hyb, opt, cfg, size, prompt, kernel_timing, gbs, tflops, dev)
        out[name] = res
        del hyb, opt
        torch.cuda.empty_cache()
    return out
