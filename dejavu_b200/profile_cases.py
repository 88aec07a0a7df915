"""Small single-kernel cases for profiler captures and the phase trace of the one-pass MLP kernel.

    python -m dejavu_b200.profile_cases <case>
        case: qkv | out_proj | attn | topk | exchange | ring | fc1 | fc2 | fc1_b16 | fc2_b16 | ring_trace
              hybrid_window | hybrid_gla | hybrid_decode   (shapes of the 7b size of bench.py --hybrid)
              routed_memory | routed_experts | routed_latent | routed_decode   (the same of bench.py --routed)

Every case launches ONE kind of kernel a dozen times at the per-rank shapes of an OPT-175B layer under 8-way
tensor parallelism (d 12288, 12 local heads of which 4 are active, 512 of 6144 ffn rows), rotating several weight
buffers so that a launch never finds its rows in L2, and holds well under 3 GB on the device: small enough for a
multi-pass `ncu` capture of one kernel (`-k regex:<kernel> -s <skip> -c 3`) to end by itself in seconds.
`ring_trace` needs a library built with the phase stamps (DJV_NVCC_FLAGS=-DDJV_RING_TRACE python -m
dejavu_b200.build --force) and prints, per phase of the one-pass kernel, when the blocks reached it.
"""

import ctypes as C
import sys

import numpy as np
import torch

from . import _lib, ops


def main(case: str) -> None:
    dev = torch.device("cuda:0")
    g = torch.Generator(device=dev).manual_seed(0)
    def rnd(*shape, std=0.02): return (torch.randn(*shape, device=dev, generator=g) * std).half()
    d, n, hd, a = 12288, 12, 128, 4   # OPT-175B TP8 shard
    NB, REP = 6, 2
    if case == "qkv":
        Ws = [rnd(3, n, hd, d) for _ in range(NB)]; b = rnd(3, n, hd); x = rnd(1, d, std=1.0)
        heads = torch.tensor([1, 4, 7, 10], dtype=torch.int32, device=dev); bidx = torch.zeros(a, 1, dtype=torch.int32, device=dev)
        for _ in range(REP):
            for W in Ws: ops.qkv_proj_sparse(x, W, heads, bidx, b)
    elif case == "out_proj":
        Ws = [rnd(d, n, hd) for _ in range(NB)]; b = rnd(d); ctx = rnd(1, n, hd, std=1.0)
        heads = torch.tensor([1, 4, 7, 10], dtype=torch.int32, device=dev)
        for _ in range(REP):
            for W in Ws: ops.out_proj_sparse(ctx, W, heads, b)
    elif case == "attn":
        S = 2048
        caches = [(rnd(1, n, hd // 8, S, 8, std=1.0), rnd(1, n, S, hd, std=1.0)) for _ in range(10)]
        q = rnd(1, n, hd, std=1.0); heads = torch.tensor([1, 4, 7, 10], dtype=torch.int32, device=dev)
        for _ in range(REP):
            for k, v in caches: ops.decode_attention(q, k, v, heads, 2000, hd ** -0.5)
    elif case == "topk":
        for nn, kk in ((6144, 512), (36864, 4096)):
            sc = rnd(nn, std=1.0)
            for _ in range(3): ops.topk_indices(sc, kk, torch.int32)
    elif case == "exchange":
        from .comm import TensorParallelComm
        comm = TensorParallelComm(None, dev, max_bytes=d * 2)
        x = rnd(1, d, std=1.0); r = rnd(1, d, std=1.0); gm = torch.ones(d, device=dev).half(); bt = torch.zeros(d, device=dev).half()
        for _ in range(6): comm.allreduce_add_layernorm(x, r, gm, bt, 1e-5)
        comm.end_step()
    elif case in ("ring", "fc1", "fc2", "ring_trace"):
        Z, K = 6144, 512
        W1 = [rnd(Z, d) for _ in range(NB)]; W2 = [rnd(Z, d) for _ in range(NB)]
        b1 = rnd(Z); b2 = rnd(d); x = rnd(1, d, std=1.0); h = torch.relu(rnd(1, K, std=1.0))
        idxs = [torch.randperm(Z, device=dev, generator=g)[:K].int() for _ in range(NB)]
        for _ in range(REP):
            for i in range(NB):
                if case in ("ring", "ring_trace"): ops.mlp_sparse(x, W1[i], W2[i], idxs[i], b1, b2, fused=True)
                elif case == "fc1": ops.gather_gemv(x, W1[i], idxs[i], b1, "relu")
                else: ops.gather_transposed_gemv(h, W2[i], idxs[i], b2)
    elif case in ("fc1_b16", "fc2_b16"):  # the tensor-core kernels: 16 activation rows, 4096 of 6144 rows
        Z, K, Bt = 6144, 4096, 16
        Ws = [rnd(Z, d) for _ in range(4)]; b1 = rnd(Z); b2 = rnd(d)
        x = rnd(Bt, d, std=1.0); h = torch.relu(rnd(Bt, K, std=1.0))
        idxs = [torch.randperm(Z, device=dev, generator=g)[:K].int() for _ in range(4)]
        for _ in range(REP):
            for i in range(4):
                if case == "fc1_b16": ops.gather_gemv(x, Ws[i], idxs[i], b1, "relu")
                else: ops.gather_transposed_gemv(h, Ws[i], idxs[i], b2)
    elif case in ("hybrid_window", "hybrid_gla", "hybrid_decode"):
        H, G, dk, dv, W, GH, gk, gv, rank, n = 32, 8, 128, 128, 1024, 16, 128, 256, 16, 4096
        def bf(*shape): return torch.randn(*shape, device=dev, generator=g).bfloat16()
        def f32(*shape): return torch.randn(*shape, device=dev, generator=g)
        gla = (f32(GH * gk, rank) * 0.1, torch.ones(GH * gk, device=dev), 16.0, torch.ones(gv, device=dev), 1e-6, gk ** -0.5)
        pos = torch.zeros(1, dtype=torch.int64, device=dev)
        sink = torch.ones(H, device=dev)
        if case == "hybrid_window":
            rows = [bf(n, (H + G) * dk + G * dv) for _ in range(3)]
            ring = (bf(1, G, W, dk), bf(1, G, W, dv))
            for r in rows * 2: ops.window_attention(r, *ring, sink, pos, n, H, W, dk ** -0.5)
        elif case == "hybrid_gla":
            rows, st = [bf(n, 2 * GH * (gk + gv) + rank) for _ in range(2)], f32(1, GH, gk, gv)
            for r in rows * 2: ops.gated_linear_attention(r, *gla, st, pos, n)
        else:
            far = pos + 5000
            row, prow = bf(1, (H + G) * dk + G * dv), bf(1, 2 * GH * (gk + gv) + rank)
            rings = [(bf(1, G, W, dk), bf(1, G, W, dv)) for _ in range(40)]
            states = [f32(1, GH, gk, gv) for _ in range(70)]
            freqs = torch.rand(dk // 2, device=dev)
            for r in rings: ops.window_attention_decode(row, *r, sink, freqs, 1.0, far, H, W, dk ** -0.5)
            for s in states: ops.gated_linear_attention(prow, *gla, s, far, 1)
    elif case in ("routed_memory", "routed_experts", "routed_latent", "routed_decode"):
        from .routed_bench import DIM, RANK, ROT, VDIM
        H, W, GH, gk, gv, n, D, E, ff, top = 32, 1024, 16, 128, 256, 4096, 4096, 8, 3648, 2
        def bf(*shape): return torch.randn(*shape, device=dev, generator=g).bfloat16()
        def f32(*shape): return torch.randn(*shape, device=dev, generator=g)
        pos, far = torch.zeros(1, dtype=torch.int64, device=dev), torch.full((1,), 5000, dtype=torch.int64, device=dev)
        mem = (torch.zeros(GH, device=dev), torch.full((GH,), 3.0, device=dev), 15.0, torch.ones(GH * gv, device=dev), 1e-6, gk ** -0.5)
        main, width, norm, freqs = 2 * GH * (gk + gv), RANK + ROT, torch.ones(RANK, device=dev), torch.rand(ROT // 2, device=dev)
        if case == "routed_memory":
            rows, gates, st = [bf(n, main) for _ in range(2)], f32(n, 2 * GH), ops.mlstm_state(1, GH, gk, gv, dev)
            for r in rows * 2: ops.mlstm(r, gates, *mem, st, pos, n, gk, gv, torch.bfloat16)
        elif case == "routed_experts":
            x, z, w = bf(n, D), f32(n, E), [bf(E, 2 * ff, D) for _ in range(2)]
            for wi in w * 2:
                xs, ws, off, _ = ops.moe_route(x, z, top)
                ops.moe_grouped(xs, wi, off, ws, glu=True)
        elif case == "routed_latent":
            q, kv, tail, gate = bf(n, H * (DIM + ROT)), bf(n, H * (DIM + VDIM)), bf(n, ROT), bf(n, H * VDIM)
            for _ in range(4): ops.latent_attention(q, kv, tail, gate, pos, n, 0, H, DIM, ROT, W, (DIM + ROT) ** -0.5)
        else:
            proj, uk, uv, gate = bf(1, H * (DIM + ROT) + width), bf(H * DIM, RANK), bf(H * VDIM, RANK), bf(1, H * VDIM)
            for r in [bf(1, W, width) for _ in range(8)]:
                ops.latent_attention_decode(proj, uk, uv, norm, 1e-6, freqs, r, gate, far, H, W, (DIM + ROT) ** -0.5)
            prow = f32(1, main + 2 * GH)
            for _ in range(4): ops.mlstm(prow, prow[:, main:], *mem, ops.mlstm_state(1, GH, gk, gv, dev), far, 1, gk, gv, torch.bfloat16)
    torch.cuda.synchronize()
    if case == "ring_trace":
        lib = _lib.load()
        if not hasattr(lib, "djv_mlp_ring_trace"):
            sys.exit("this library was built without -DDJV_RING_TRACE")
        lib.djv_mlp_ring_trace.restype, lib.djv_mlp_ring_trace.argtypes = C.c_int, [C.c_void_p]
        buf = np.zeros((512, 12), dtype=np.uint64)
        assert lib.djv_mlp_ring_trace(buf.ctypes.data) == 0
        t = buf[:120].astype(np.float64)  # 15 clusters of 8 blocks
        names = ["start", "first copies issued", "wait on predecessor done", "input rows ready", "first product done",
                 "cluster barrier", "activations ready", "second product done", "partial sums written", "ticket taken",
                 "result stored (last block of a segment)"]
        print("phase: microseconds after the first block's start, min / median / max over blocks (last launch)")
        for i, nm in enumerate(names):
            col = t[:, i][t[:, i] > t[:, 0].min()] if i else t[:, 0]
            if len(col):
                print(f"  {nm:42s} {(col.min() - t[:, 0].min()) / 1e3:6.2f} {(np.median(col) - t[:, 0].min()) / 1e3:6.2f} "
                      f"{(col.max() - t[:, 0].min()) / 1e3:6.2f}")
    print("ok", case)


if __name__ == "__main__":
    main(sys.argv[1])
