"""Prefill and decode throughput of the Tifosun design beside the Ninolorn one (the closest other model: a recurrent state
and a windowed attention in turn) at equal width, layers and weights per token, and every kernel of both with its fraction
of the measured roofline (bench.py --routed).

Random weights, random prompt tokens; timing as in hybrid_bench.
"""
from __future__ import annotations

import torch

from . import ops
from .hybrid_bench import SIZES, VOCAB, WINDOW, hybrid_config, time_decode, time_prefill
from .ninolorn import NinolornForCausalLM
from .tifosun import TifosunForCausalLM

EXPERTS, TOP, DIM, ROT, VDIM, RANK = 8, 2, 128, 64, 128, 512


def expert_ff(size: dict) -> int:
    """Two experts and a shared one of this size have about the weights of the other design's feed-forward."""
    return size["ff"] // (TOP + 1) // 64 * 64


def routed_config(size: dict) -> dict:
    ff = expert_ff(size)
    moe = {"kind": "moe", "router": {"experts": EXPERTS, "top": TOP}, "expert": {"ff": ff}, "shared": {"ff": ff}}
    memory = {"type": "mlstm", "mixer": {"heads": size["gla"], "dim": 128, "vdim": 256, "gate_cap": 15.0}}
    latent = {"type": "latent_attention", "mlp": moe,
              "mixer": {"heads": size["heads"], "dim": DIM, "rot_dim": ROT, "vdim": VDIM, "kv_rank": RANK,
                        "scale": (DIM + ROT) ** -0.5, "mask": {"size": WINDOW}, "rot": {"base": 10000.0, "dims": ROT}}}
    first = {**memory, "type": "mlstm_2", "mlp": {"kind": "dense", "ff": size["ff"]}}
    layers = [first, latent] + [{**memory, "mlp": moe}, latent] * (size["layers"] // 2 - 1)
    return {"architecture": "Tifosun", "vocab": VOCAB, "width": size["width"], "layers": layers, "norm": {"eps": 1e-6}}


def active_params(model) -> int:
    """Weights that one token uses."""
    n = sum(p.numel() for p in model.parameters()) - model.embed.numel()
    for layer in model.layers:
        if hasattr(layer.mlp, "router"):
            n -= (layer.mlp.gate_up.numel() + layer.mlp.down.numel()) * (EXPERTS - TOP) // EXPERTS
    return n


def kernel_table(rt, nl, size, n, kernel_timing, gbs, tflops, dev) -> dict:
    """us and fraction of roofline (the slower of bytes / bandwidth and flops / tensor peak) of each kernel alone. Names of
    the Ninolorn model's like kernels start with 'like.'."""
    out = {}
    g = torch.Generator(device=dev).manual_seed(1)

    def rec(name, us, nbytes, flops=0.0):
        ideal = max(nbytes / gbs / 1e3, flops / tflops / 1e6)
        out[name] = {"us": round(us, 2), "bytes": int(nbytes), "gflop": round(flops / 1e9, 3), "frac": round(ideal / us, 3)}

    def rand(*s, dtype=torch.bfloat16):
        return torch.randn(*s, device=dev, generator=g, dtype=torch.float32).to(dtype)

    def spread(nbytes):  # how many buffers of this size lie beyond L2
        return 2 + int(2.6e8 / nbytes)

    D, ff = size["width"], expert_ff(size)
    mem = [l for l in rt.layers if hasattr(l.mixer, "f_bias")]
    lat = [l for l in rt.layers if hasattr(l.mixer, "ukv")]
    moe = [l.mlp for l in rt.layers if hasattr(l.mlp, "router")]
    gla = [l for l in nl.layers if hasattr(l.mixer, "a2")]
    att = [l for l in nl.layers if not hasattr(l.mixer, "a2")]
    x = rand(1, D)

    def gemv(name, ws, x, out_bytes=2, **kw):
        ws = ws + [w.detach().clone() for w in ws for _ in range(int(2.6e8 / (len(ws) * ws[0].numel() * 2)))]
        us = kernel_timing([lambda w=w: ops.linear_gemv(x, w, **kw) for w in ws])
        M, N = ws[0].shape
        rec(name, us, M * N * 2 + N * 2 + M * out_bytes)

    f32 = torch.float32
    gemv("decode.mlstm_proj", [l.mixer.proj.weight for l in mem], x, 4, out_dtype=f32)
    gemv("decode.latent_proj", [l.mixer.proj.weight for l in lat], x)
    gemv("decode.o", [l.mixer.o.weight for l in lat], rand(1, size["heads"] * VDIM), 4, out_dtype=f32)
    gemv("decode.router", [m.router.weight for m in moe], x, 4, out_dtype=f32)
    gemv("decode.dense_gate_up", [rt.layers[0].mlp.gate_up.weight], x, activation="silu_glu")
    gemv("like.decode.gla_proj", [l.mixer.proj.weight for l in gla], x)
    gemv("like.decode.qkv", [l.mixer.qkv.weight for l in att], x)
    gemv("like.decode.o", [l.mixer.o.weight for l in att], rand(1, size["heads"] * 128), 4, out_dtype=f32)
    gemv("like.decode.gate_up", [l.mlp.gate_up.weight for l in nl.layers], x, activation="clamped_glu", param=7.0)
    gemv("like.decode.down", [l.mlp.down.weight for l in nl.layers], rand(1, size["ff"]), 4, out_dtype=f32)

    # routed feed-forward of one token: two experts and the shared one, logits that change from launch to launch
    zs = [rand(1, EXPERTS, dtype=f32) for _ in range(max(8, 2 * len(moe)))]
    pairs = [(moe[i % len(moe)], z) for i, z in enumerate(zs)]
    act = (torch.empty(1, TOP + 1, ff, dtype=torch.bfloat16, device=dev), torch.zeros(1, TOP, dtype=torch.int32, device=dev))
    for stage, name in ((1, "decode.moe_up"), (2, "decode.moe_down")):
        us = kernel_timing([lambda m=m, z=z: ops.moe_decode(x, z, m.gate_up, m.down, TOP, m.shared.gate_up.weight,
                                                            m.shared.down.weight, stages=stage, scratch=act) for m, z in pairs])
        rec(name, us, (TOP + 1) * ff * D * (4 if stage == 1 else 2))

    x8 = rand(8, D)
    pairs = [(moe[i % len(moe)], rand(8, EXPERTS, dtype=f32)) for i in range(max(8, 2 * len(moe)))]
    act = (torch.empty(8, TOP + 1, ff, dtype=torch.bfloat16, device=dev), torch.zeros(8, TOP, dtype=torch.int32, device=dev))
    used = sum(len(set(z.topk(TOP).indices.flatten().tolist())) for _, z in pairs) / len(pairs)
    for stage, name in ((1, "decode.moe_up, 8 seq"), (2, "decode.moe_down, 8 seq")):
        us = kernel_timing([lambda m=m, z=z: ops.moe_decode(x8, z, m.gate_up, m.down, TOP, m.shared.gate_up.weight,
                                                            m.shared.down.weight, stages=stage, scratch=act) for m, z in pairs])
        rec(name, us, (used + 1) * ff * D * (4 if stage == 1 else 2))
    gemv("like.decode.gate_up, 8 seq", [l.mlp.gate_up.weight for l in nl.layers], x8, activation="clamped_glu", param=7.0)
    gemv("like.decode.down, 8 seq", [l.mlp.down.weight for l in nl.layers], rand(8, size["ff"]), 4, out_dtype=f32)

    # residual boundary: decode and prompt rows; the routed layer's prompt boundary also adds the experts' rows
    n1, n2 = rt.layers[0].norm1, rt.layers[0].norm1b
    hc = nl.layers[0].hc1
    for rows, tag in ((1, "decode"), (n, "prefill")):
        k = spread(rows * D * 8) if rows > 1 else 8
        xs, ys = [rand(rows, D, dtype=f32) for _ in range(k)], [rand(rows, D, dtype=f32) for _ in range(k)]
        us = kernel_timing([lambda a=a, b=b: ops.residual_step(a, b, n2, n1, 1e-6, torch.bfloat16, base=1.0, x_out=a)
                            for a, b in zip(xs, ys)])
        rec(f"{tag}.residual_step", us, rows * D * (4 + 4 + 4 + 2))
        if rows > 1:
            parts = rand(rows * TOP, D)
            places = torch.randperm(rows * TOP, device=dev, generator=g).int().view(rows, TOP)
            us = kernel_timing([lambda a=a, b=b: ops.residual_step(a, b, n2, n1, 1e-6, torch.bfloat16, base=1.0, x_out=a,
                                                                   parts=parts, part_rows=places) for a, b in zip(xs, ys)])
            rec(f"{tag}.residual_step_experts", us, rows * D * (4 + 4 + 4 + 2 + 2 * TOP))
            del parts
        del xs, ys
        k = spread(rows * 16 * D) if rows > 1 else 8
        xs, ys = [rand(rows, 4, D, dtype=f32) for _ in range(k)], [rand(rows, D, dtype=f32) for _ in range(k)]
        us = kernel_timing([lambda a=a, b=b: ops.hyper_step(a, b, hc.mix, hc.w_out, hc.w_in, nl.layers[0].norm1, 1e-6,
                                                            torch.bfloat16, x_out=a) for a, b in zip(xs, ys)])
        rec(f"like.{tag}.hyper_step", us, rows * D * (32 + 4 + 2))
        del xs, ys

    # decode mixers
    H, G, W, GH = size["heads"], size["kv"], WINDOW, size["gla"]
    pos = torch.full((1,), 5 * W + 3, dtype=torch.int64, device=dev)
    m = mem[0].mixer
    st = [ops.mlstm_state(1, GH, 128, 256, dev) for _ in range(spread(GH * 128 * 256 * 4))]
    prow = rand(1, m.proj.weight.shape[0], dtype=f32)
    margs = (m.i_bias, m.f_bias, m.gate_cap, m.norm, m.eps, m.scale)
    us = kernel_timing([lambda s=s: ops.mlstm(prow, prow[:, m.main:], *margs, s, pos, 1, 128, 256, torch.bfloat16) for s in st])
    rec("decode.mlstm", us, 2 * st[0].numel() * 4)
    gm = gla[0].mixer
    gst = [rand(1, GH, 128, 256, dtype=f32) for _ in st]
    grow, gargs = rand(1, gm.proj.weight.shape[0]), (gm.a2, gm.a2_bias, gm.tau, gm.norm, gm.eps, gm.scale)
    us = kernel_timing([lambda s=s: ops.gated_linear_attention(grow, *gargs, s, pos, 1) for s in gst])
    rec("like.decode.gla", us, 2 * gst[0].numel() * 4 + gm.a2.numel() * 4)
    del st, gst
    m = lat[0].mixer
    width = RANK + ROT
    rings = [rand(1, W, width) for _ in range(spread(W * width * 2))]
    row, gate = rand(1, m.proj.weight.shape[0]), rand(1, H * VDIM)
    ukvs = [l.mixer.ukv.weight for l in lat]
    ukvs = ukvs + [w.detach().clone() for w in ukvs for _ in range(int(2.6e8 / (len(ukvs) * ukvs[0].numel())))]
    scr = (torch.zeros(1, H, width, dtype=torch.bfloat16, device=dev), torch.zeros(H * 64 * (RANK + 2), device=dev))
    for stage, name, nbytes, over in ((1, "decode.latent_query", H * DIM * RANK * 2, ukvs), (4, "decode.latent_out", H * VDIM * RANK * 2, ukvs),
                                      (2, "decode.latent_attend", W * width * 2, rings)):
        us = kernel_timing([lambda o=o: ops.latent_attention_decode(
            row, (o if stage != 2 else ukvs[0])[:H * DIM], (o if stage != 2 else ukvs[0])[H * DIM:], m.norm, m.eps, m.rotary.freqs,
            o if stage == 2 else rings[0], gate, pos, H, W, m.scale, stages=stage, scratch=scr) for o in over])
        rec(name, us, nbytes, 2.0 * H * W * (width + RANK) if stage == 2 else 0.0)
    wm = att[0].mixer
    rg = [(rand(1, G, W, 128), rand(1, G, W, 128)) for _ in range(spread(G * W * 512))]
    wrow = rand(1, (H + 2 * G) * 128)
    us = kernel_timing([lambda c=c: ops.window_attention_decode(wrow, *c, wm.sink, wm.rotary.freqs, wm.rotary.amp, pos, H, W,
                                                                wm.scale) for c in rg])
    rec("like.decode.window_attn", us, G * W * 512)
    del rings, rg, ukvs

    # prompt mixers
    p0 = torch.zeros(1, dtype=torch.int64, device=dev)
    m = mem[0].mixer
    rows, gates = [rand(n, m.main) for _ in range(3)], rand(n, 2 * GH, dtype=f32)
    state = ops.mlstm_state(1, GH, 128, 256, dev)
    us = kernel_timing([lambda r=r: ops.mlstm(r, gates, *margs, state, p0, n, 128, 256, torch.bfloat16) for r in rows])
    rec("prefill.mlstm", us, n * GH * (2 * 128 + 3 * 256) * 2, 4.0 * n * GH * 128 * 256)
    rows = [rand(n, gm.proj.weight.shape[0]) for _ in range(3)]
    gstate = rand(1, GH, 128, 256, dtype=f32)
    us = kernel_timing([lambda r=r: ops.gated_linear_attention(r, *gargs, gstate, p0, n) for r in rows])
    rec("like.prefill.gla", us, n * GH * (2 * 128 + 3 * 256) * 2, 4.0 * n * GH * 128 * 256)
    m = lat[0].mixer
    pairs_seen = sum(min(i + 1, W) for i in range(n))
    a, b = m.sizes[0], m.sizes[0] + m.sizes[1]
    rows, kv, ring = [rand(n, m.proj.weight.shape[0]) for _ in range(3)], rand(n, H * (DIM + VDIM)), rand(1, W, width)
    lrows = rand(n, width)
    us = kernel_timing([lambda r=r: ops.latent_attention(r[:, :a], kv, lrows[:, RANK:], r[:, b:b + H * VDIM], p0, n, 0, H, DIM, ROT,
                                                         W, m.scale) for r in rows])
    rec("prefill.latent_attn", us, n * (H * (DIM + ROT) + H * (DIM + VDIM) + 2 * H * VDIM + ROT) * 2, 2.0 * pairs_seen * H * (DIM + ROT + VDIM))
    us = kernel_timing([lambda r=r: ops.latent_rows(r[:, a:b], ring, m.norm, m.eps, m.rotary.freqs, p0, n, 0, RANK, store=True) for r in rows])
    rec("prefill.latent_rows", us, (2 * n + W) * width * 2)
    us = kernel_timing([lambda r=r: ops.rotary_(r[:, DIM:], m.rotary.freqs, 1.0, p0, n, H, DIM + ROT, interleaved=True) for r in rows])
    rec("prefill.rotary", us, n * H * ROT * 4)
    us = kernel_timing([lambda: torch.mm(lrows[:, :RANK], m.ukv.weight.t())])
    rec("prefill.kv_gemm (vendor)", us, n * (RANK + H * (DIM + VDIM)) * 2, 2.0 * n * m.ukv.weight.numel())
    rows = [rand(n, (H + 2 * G) * 128) for _ in range(3)]
    rg = (rand(1, G, W, 128), rand(1, G, W, 128))
    us = kernel_timing([lambda r=r: ops.window_attention(r, *rg, wm.sink, p0, n, H, W, wm.scale) for r in rows])
    rec("like.prefill.window_attn", us, n * (2 * H + 2 * G) * 128 * 2, 2.0 * pairs_seen * H * 256)
    us = kernel_timing([lambda r=r: ops.rotary_(r, wm.rotary.freqs, wm.rotary.amp, p0, n, H + G, 128) for r in rows])
    rec("like.prefill.rotary", us, n * (H + G) * 128 * 4)
    del rows, rg, kv

    # prompt feed-forward
    h = rand(n, D)
    z = [rand(n, EXPERTS, dtype=f32) for _ in range(2)]
    us = kernel_timing([lambda z=z: ops.moe_route(h, z, TOP) for z in z])
    rec("prefill.moe_route", us, n * D * 2 * (1 + TOP) + n * EXPERTS * 4)
    us = kernel_timing([lambda m=m: m.router(h, f32) for m in moe])
    rec("prefill.router_gemm (vendor)", us, n * D * 2 + n * EXPERTS * 4)
    xs, ws, offsets, _ = ops.moe_route(h, z[0], TOP)
    us = kernel_timing([lambda m=m: ops.moe_grouped(xs, m.gate_up, offsets, ws, glu=True) for m in moe])
    rec("prefill.moe_up", us, 0, 2.0 * n * TOP * 2 * ff * D)
    ax = rand(n * TOP, ff)
    us = kernel_timing([lambda m=m: ops.moe_grouped(ax, m.down, offsets) for m in moe])
    rec("prefill.moe_down", us, 0, 2.0 * n * TOP * ff * D)
    w = rt.layers[0].mlp
    us = kernel_timing([lambda: torch.mm(h, w.gate_up.weight.t())])
    rec("like.prefill.gate_up_gemm (vendor)", us, 0, 2.0 * n * w.gate_up.weight.numel())
    ax = rand(n, size["ff"])
    us = kernel_timing([lambda: torch.mm(ax, w.down.weight.t(), out_dtype=f32)])
    rec("like.prefill.down_gemm (vendor)", us, 0, 2.0 * n * w.down.weight.numel())
    rows = [rand(n, 2 * ff) for _ in range(spread(n * ff * 4))]
    us = kernel_timing([lambda r=r: ops.glu(r, "silu_glu") for r in rows])
    rec("prefill.silu_glu", us, n * ff * 6)
    rows = [rand(n, 2 * size["ff"]) for _ in range(3)]
    us = kernel_timing([lambda r=r: ops.glu(r, "clamped_glu", 7.0) for r in rows])
    rec("like.prefill.clamped_glu", us, n * size["ff"] * 6)
    return out


def run(names, kernel_timing, gbs: float, tflops: float, prompt: int = 4096, steps: int = 64, kernels: bool = True) -> dict:
    dev = torch.device("cuda", 0)
    out = {}
    for name in names:
        size = SIZES[name]
        rt = TifosunForCausalLM(routed_config(size), device=dev).eval().init_random(0)
        nl = NinolornForCausalLM(hybrid_config(size), device=dev).eval().init_random(0)
        res = {"width": size["width"], "layers": size["layers"], "prompt": prompt,
               "routed_params": sum(p.numel() for p in rt.parameters()), "routed_active": active_params(rt),
               "ninolorn_active": sum(p.numel() for p in nl.parameters()) - nl.embed.numel()}
        with torch.inference_mode():
            for tag, model in (("routed", rt), ("ninolorn", nl)):
                ms = time_prefill(model, prompt, 1, 5, dev)
                res[tag] = {"prefill_tokens_per_s": round(prompt / ms * 1e3), "prefill_ms": round(ms, 3)}
                for B in (1, 8):
                    ms = time_decode(model, min(prompt, 1024), B, steps, dev)
                    res[tag][f"decode_b{B}"] = {"ms_per_step": round(ms, 4), "tokens_per_s": round(B / ms * 1e3)}
            if kernels:
                res["kernels"] = kernel_table(rt, nl, size, prompt, kernel_timing, gbs, tflops, dev)
        out[name] = res
        del rt, nl
        torch.cuda.empty_cache()
    return out
