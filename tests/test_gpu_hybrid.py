"""Hybrid decoders on the GPU against the plain CPU oracle: every mechanism alone, then whole models (prompts, portions,
decoding, batches, reused slots, generation, command line)."""
import json
import math
import subprocess
import sys
from pathlib import Path

import pytest
import torch

sys.path.insert(0, str(Path(__file__).parent))
import hybrid_cases as H
from oracle import hybrid_oracle as O

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parents[1]
DTYPES = [torch.float32, torch.bfloat16]
TOL = {torch.float32: 2e-5, torch.bfloat16: 2e-2}  # relative to the scale of what is compared


@pytest.fixture(scope="module", autouse=True)
def hybrid_lib():
    assert torch.cuda.is_available(), "GPU tests need a CUDA device"
    from dejavu_b200 import _lib

    _lib.load_hybrid()


def gen(seed):
    return torch.Generator().manual_seed(seed)


def rnd(g, *shape, dtype=torch.float32, scale=1.0):
    """Random values that the element type holds exactly, in double."""
    return (torch.randn(*shape, generator=g) * scale).to(dtype).double()


def dev(t, dtype=torch.float32):
    return t.to(dtype).cuda().contiguous()


def close(got, want, dtype, tol=None):
    got, want = got.double().cpu(), want.double()
    assert got.shape == want.shape
    scale = float(want.abs().max()) + 1e-30
    err = float((got - want).abs().max()) / scale
    assert err < (tol or TOL[dtype]), err


# ---- mechanisms ----------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("S,D,n", [(1, 64, 3), (2, 100, 5), (3, 257, 2), (4, 4096, 3), (5, 36, 40), (8, 520, 2)])
def test_hyper_step(dtype, S, D, n):
    from dejavu_b200 import ops

    g = gen(S * D)
    x, y, mix = rnd(g, n, S, D), rnd(g, n, D), rnd(g, S, S)
    w_out, w_in, gamma = rnd(g, S), rnd(g, S), rnd(g, D)
    new = O.stream_update(x, y, mix, w_out)
    want = O.rms_norm(O.stream_in(new, w_in), gamma, 1e-3)
    xd = dev(x)
    h = ops.hyper_step(xd, dev(y), dev(mix), dev(w_out), dev(w_in), dev(gamma), 1e-3, dtype, x_out=xd)
    close(xd, new, torch.float32, 1e-6)
    close(h, want, dtype, 1e-5 if dtype == torch.float32 else 5e-3)
    rows = torch.tensor([n - 1, 0], dtype=torch.int32)
    h = ops.hyper_step(dev(x), None, None, None, None, dev(gamma), 1e-3, dtype, rows=rows.cuda())
    close(h, O.rms_norm(x.sum(1), gamma, 1e-3)[rows.long()], dtype, 1e-5 if dtype == torch.float32 else 5e-3)
    # all streams start as the embedding: without and with an update, ids out of range do not leave the table
    table, ids = rnd(g, 7, D, dtype=dtype), torch.tensor(([3, 6, 0, 5] * n)[:n])
    e = table[ids][:, None].repeat(1, S, 1)
    kw = dict(ids=ids.cuda(), embed=dev(table, dtype), streams=S)
    h = ops.hyper_step(None, None, None, None, dev(w_in), dev(gamma), 1e-3, dtype, **kw)
    close(h, O.rms_norm(O.stream_in(e, w_in), gamma, 1e-3), dtype, 1e-4 if dtype == torch.float32 else 5e-3)
    out = torch.empty(n, S, D, device="cuda")
    ops.hyper_step(None, dev(y), dev(mix), dev(w_out), None, None, 1e-3, dtype, x_out=out, **kw)
    close(out, O.stream_update(e, y, mix, w_out), torch.float32, 1e-6)
    kw["ids"] = torch.full((n,), 99).cuda()
    ops.hyper_step(None, None, None, None, None, None, 1e-3, dtype, x_out=out, **kw)
    close(out, table[6].expand(n, S, D), torch.float32, 1e-6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("B", [1, 2, 3, 4, 5, 8, 13, 32])
@pytest.mark.parametrize("N,M", [(64, 40), (1000, 34), (2048, 3000), (50, 22)])
def test_linear_gemv(dtype, B, N, M):
    from dejavu_b200 import ops

    g = gen(B * N)
    x, w = rnd(g, B, N, dtype=dtype), rnd(g, M, N, dtype=dtype, scale=N ** -0.5)
    xd, wd = dev(x, dtype), dev(w, dtype)
    y = x @ w.T
    close(ops.linear_gemv(xd, wd, torch.float32), y, torch.float32, 1e-5)
    close(ops.linear_gemv(xd, wd), y, dtype, 1e-5 if dtype == torch.float32 else 5e-3)
    close(ops.linear_gemv(xd, wd, torch.float32, "softcap", 1.5), O.softcap(y, 1.5), torch.float32, 1e-5)
    want = O.clamped_glu(y[:, 0::2], y[:, 1::2], 0.8)
    close(ops.linear_gemv(xd, wd, None, "clamped_glu", 0.8), want, dtype, 1e-5 if dtype == torch.float32 else 5e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("R,F", [(1, 3), (5, 33), (70, 128)])
def test_elementwise(dtype, R, F):
    from dejavu_b200 import ops

    gu = rnd(gen(F), R, 2 * F, dtype=dtype, scale=2.0)
    close(ops.glu(dev(gu, dtype), "clamped_glu", 0.7), O.clamped_glu(gu[:, 0::2], gu[:, 1::2], 0.7), dtype, 1e-6 if dtype == torch.float32 else 5e-3)
    y = rnd(gen(R), R, F, scale=10.0)
    close(ops.softcap_(dev(y), 6.0), O.softcap(y, 6.0), torch.float32, 1e-6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rot,dim,heads", [({"base": 1000.0, "dims": 32, "scaling": H.YARN}, 48, 5), ({"base": 5e4, "dims": 6}, 7, 2),
                                           ({"base": 1e6, "dims": 128, "scaling": {**H.YARN, "factor": 8.0}}, 128, 12)])
def test_rotary(dtype, rot, dim, heads):
    from dejavu_b200 import ops
    from dejavu_b200.mixers import RotaryTable

    n, starts = 9, [0, 3000]
    x = rnd(gen(dim), 2 * n, heads * dim + 5, dtype=dtype)
    xd, t = dev(x, dtype), RotaryTable(rot, "cuda")
    ops.rotary_(xd, t.freqs, t.amp, torch.tensor(starts).cuda(), n, heads, dim)
    want = x.clone()
    for b, s in enumerate(starts):
        r = x[b * n:(b + 1) * n, :heads * dim].reshape(n, heads, dim)
        want[b * n:(b + 1) * n, :heads * dim] = O.rotate(r, s + torch.arange(n), rot).reshape(n, -1)
    close(xd, want, dtype, 1e-4 if dtype == torch.float32 else 5e-3)


# heads, kv heads, dk, dv, window: groups of 1 to 16, sizes that are and are not multiples of 8 / 16 / 64
WINDOWS = [(4, 2, 64, 64, 45), (3, 3, 18, 10, 3), (8, 1, 128, 64, 150), (6, 2, 48, 96, 64), (16, 1, 32, 40, 7), (4, 4, 128, 128, 300),
           (5, 1, 80, 256, 33), (2, 1, 256, 80, 129), (2, 2, 64, 130, 20), (12, 4, 96, 192, 64), (1, 1, 16, 16, 1), (4, 2, 160, 64, 70), (2, 1, 192, 128, 140)]


def spiky(g, n, heads, kv, dk, dv, dtype, window):
    """Queries and keys of which some stand out, so that a far key (also one just inside or just outside the window)
    takes or would take most of the weight of its query."""
    q, k, v = rnd(g, n, heads, dk, dtype=dtype), rnd(g, n, kv, dk, dtype=dtype), rnd(g, n, kv, dv, dtype=dtype)
    for i in range(0, n, 5):
        for back in (window - 1, window, window // 2):
            if 0 <= i - back and (i + back) % 3:
                h = (i // 5) % heads
                u = q[i, h] / q[i, h].norm()
                k[i - back, h // (heads // kv)] = (u * 4 * dk ** 0.5).to(dtype).double()
    return q, k, v


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv,dk,dv,window", WINDOWS)
def test_window_attention_portions_and_decoding(dtype, heads, kv, dk, dv, window):
    """Prompt portions of many sizes, then token by token, against one pass over everything; two sequences at different
    positions in one call; a cache that another sequence used before."""
    from dejavu_b200 import ops

    n = 2 * window + 45 if window > 20 else 70
    g = gen(heads * dk + dv)
    scale, sink = dk ** -0.5, rnd(g, heads) + 1.0
    seqs = [spiky(g, n, heads, kv, dk, dv, dtype, window) for _ in range(2)]
    want = [O.window_attention(q, k, v, scale, window, sink).reshape(n, -1) for q, k, v in seqs]
    packed = [torch.cat([t.reshape(n, -1) for t in s], 1) for s in seqs]
    cap = min(window, n)
    rings = [torch.full((2, kv, cap, d), 7.0, dtype=dtype, device="cuda") for d in (dk, dv)]  # stale content
    lag = 6  # sequence 1 runs that many tokens behind
    got = [[], []]

    def call(at, m):
        rows = torch.cat([packed[b][a:a + m] for b, a in enumerate(at)])
        # (wider rows than the heads need: the stride is not the width)
        buf = torch.zeros(rows.shape[0], rows.shape[1] + 8, dtype=dtype, device="cuda")
        buf[:, :rows.shape[1]] = dev(rows, dtype)
        pos = torch.tensor(at).cuda()
        if m == 1:
            out = ops.window_attention_decode(buf, *rings, dev(sink), None, 1.0, pos, heads, window, scale)
        else:
            out = ops.window_attention(buf, *rings, dev(sink), pos, m, heads, window, scale)
        for b in range(2):
            got[b].append(out[b * m:(b + 1) * m].cpu())

    # sequence 1 first runs alone to nowhere: both start at 0, sequence 1 repeats its first tokens after the lag
    at = [0, 0]
    call(at, lag)
    got[1].clear()
    at = [lag, 0]
    for m in (2, 3, 1, 16, 2, 17, 1, 5):
        call(at, m)
        at = [a + m for a in at]
    rest = n - 8 - at[0]
    if rest > 1:
        call(at, rest)
        at = [a + rest for a in at]
    while at[0] < n:
        call(at, 1)
        at = [a + 1 for a in at]
    from dejavu_b200 import _lib

    assert _lib.load_hybrid().djv_window_timeouts() == 0
    for b in range(2):
        res = torch.cat(got[b])
        close(res, want[b][:res.shape[0]], dtype, 1e-5 if dtype == torch.float32 else 1e-2)


@pytest.mark.parametrize("dtype", DTYPES)
def test_window_attention_without_sink_or_window(dtype):
    from dejavu_b200 import ops

    n, heads, kv, dk, dv = 90, 4, 2, 32, 32
    q, k, v = spiky(gen(3), n, heads, kv, dk, dv, dtype, n)
    want = O.window_attention(q, k, v, 0.2, None, None).reshape(n, -1)
    rows = dev(torch.cat([t.reshape(n, -1) for t in (q, k, v)], 1), dtype)
    rings = [torch.zeros(1, kv, n, d, dtype=dtype, device="cuda") for d in (dk, dv)]
    at, out = 0, []
    for m in (50, 1, 1, 38):
        fn = ops.window_attention_decode if m == 1 else None
        pos = torch.tensor([at]).cuda()
        if m == 1:
            out.append(fn(rows[at:at + 1], *rings, None, None, 1.0, pos, heads, 2 ** 30, 0.2))
        else:
            out.append(ops.window_attention(rows[at:at + m], *rings, None, pos, m, heads, 2 ** 30, 0.2))
        at += m
    close(torch.cat(out), want, dtype, 1e-5 if dtype == torch.float32 else 1e-2)


@pytest.mark.parametrize("dtype", DTYPES)
def test_decode_kernel_rotates_and_stores(dtype):
    from dejavu_b200 import ops
    from dejavu_b200.mixers import RotaryTable

    heads, kv, dk, dv, window, n = 6, 2, 40, 24, 12, 30
    rot = {"base": 500.0, "dims": 32, "scaling": H.YARN}
    g = gen(11)
    q, k, v = (rnd(g, n, h, d, dtype=dtype) for h, d in ((heads, dk), (kv, dk), (kv, dv)))
    pos = torch.arange(n)
    want = O.window_attention(O.rotate(q, pos, rot), O.rotate(k, pos, rot), v, 0.15, window, None).reshape(n, -1)
    t = RotaryTable(rot, "cuda")
    rings = [torch.zeros(1, kv, window, d, dtype=dtype, device="cuda") for d in (dk, dv)]
    rows = dev(torch.cat([x.reshape(n, -1) for x in (q, k, v)], 1), dtype)
    out = [ops.window_attention_decode(rows[i:i + 1], *rings, None, t.freqs, t.amp, torch.tensor([i]).cuda(), heads, window, 0.15)
           for i in range(n)]
    close(torch.cat(out), want, dtype, 2e-5 if dtype == torch.float32 else 1e-2)
    close(rings[1][0, :, (n - 1) % window], v[n - 1], dtype, 1e-9)


GLAS = [(2, 64, 64, 16, 16.0), (3, 40, 24, 9, 8.0), (2, 20, 36, 3, 1.0), (1, 128, 128, 16, 16.0), (2, 128, 256, 5, 4.0), (1, 16, 8, 2, 0.3),
        (3, 48, 80, 12, 12.0), (1, 256, 64, 1, 30.0), (2, 33, 17, 4, 2.0), (2, 64, 96, 7, 0.5), (1, 256, 256, 16, 8.0), (2, 32, 200, 40, 0.2)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("aligned", [True, False])
@pytest.mark.parametrize("heads,dk,dv,rank,tau", GLAS)
def test_gated_linear_attention_portions_and_decoding(dtype, aligned, heads, dk, dv, rank, tau):
    """Portions of many sizes and single tokens in turn, from a state that another sequence left, against the token by
    token recurrence; two sequences per call; a key far back stands out."""
    from dejavu_b200 import ops

    n = 230
    g = gen(dk * dv)
    q, k, v, gate = (rnd(g, 2, n, heads, d, dtype=dtype) for d in (dk, dk, dv, dv))
    v[:, 3] *= 64  # (a power of two: still representable)
    low = rnd(g, 2, n, rank, dtype=dtype)
    a2, bias, norm = rnd(g, heads * dk, rank), 2.0 + 2.0 * rnd(g, heads * dk), 1 + 0.3 * rnd(g, dv)
    eps, scale = 1e-5, dk ** -0.5
    want, states = [], []
    for b in range(2):
        eye = torch.eye(rank, dtype=torch.float64)
        alpha = O.gla_decay(low[b], eye, a2, bias, tau, heads)
        o, S = O.gla_recurrence(q[b] * scale, k[b], v[b], alpha)
        want.append((O.rms_norm(o, norm, eps) * O.silu(gate[b])).reshape(n, -1))
        states.append(S)
    rows = [torch.cat([q[b].reshape(n, -1), k[b].reshape(n, -1), v[b].reshape(n, -1), gate[b].reshape(n, -1), low[b]], 1) for b in range(2)]
    state = torch.full((2, heads, dk, dv), 5.0, device="cuda")
    args = [dev(t) for t in (a2, bias)]
    got, at = [[], []], 0
    sizes = [2, 3, 1, 64, 1, 1, 63, 5, 16, 1]
    for m in sizes + [n - sum(sizes) - 4, 1, 1, 1, 1]:
        width = rows[0].shape[1]
        # rows that 16-byte copies can read (the tensor-core chunk kernels), or not (the general ones)
        buf = torch.zeros(2 * m, (width + 15) // 8 * 8 if aligned else (width | 1) + 2, dtype=dtype, device="cuda")
        buf[:, :width] = dev(torch.cat([r[at:at + m] for r in rows]), dtype)
        out = ops.gated_linear_attention(buf, *args, tau, dev(norm), eps, scale, state, torch.tensor([at, at]).cuda(), m)
        for b in range(2):
            got[b].append(out[b * m:(b + 1) * m].cpu())
        at += m
    for b in range(2):
        close(torch.cat(got[b]), want[b], dtype, 3e-5 if dtype == torch.float32 else 1e-2)
        close(state[b], states[b], torch.float32, 2e-5)


# ---- whole models --------------------------------------------------------------------------------------------------

_models: dict = {}


def model_of(case, dtype):
    from dejavu_b200.ninolorn import NinolornForCausalLM

    if (case, dtype) not in _models:
        cfg, rank = H.CASES[case]
        W = H.weights(cfg, rank)
        m = NinolornForCausalLM(cfg, {k: tuple(v.shape) for k, v in W.items()}, device="cuda", dtype=dtype).load_tensors(W)
        _models[case, dtype] = (cfg, W, m)
    return _models[case, dtype]


_expected: dict = {}


def expected(case, seed, n):
    cfg, W = model_of(case, torch.float32)[:2]
    key = (case, seed, n)
    if key not in _expected:
        ids = H.tokens(cfg, n, seed)
        _expected[key] = (ids, *O.forward(cfg, W, ids, return_layers=True))
    return _expected[key]


MODEL_TOL = {torch.float32: 5e-5, torch.bfloat16: 0.1}


def pool_for(model, n=400):
    from dejavu_b200.generation import SequencePool

    return SequencePool(model, n, torch.device("cuda"))


@pytest.mark.parametrize("case", H.CASES)
def test_layers_in_fp32(case):
    cfg, W, m = model_of(case, torch.float32)
    ids, logits, trail = expected(case, 0, 50)
    got = []
    with torch.inference_mode():
        out = m(torch.tensor([ids]).cuda(), collect=got).logits[0]
    assert len(got) == len(trail)
    for r, (a, b) in enumerate(zip(got, trail)):
        close(a, b, torch.float32, 3e-5)
    assert float(H.error(out, logits).max()) < MODEL_TOL[torch.float32]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", H.CASES)
@pytest.mark.parametrize("schedule", [[230], [1] * 40 + [190], [2] * 5 + [3, 64, 1, 1, 16, 17, 5, 1, 100, 2], [199] + [1] * 31])
def test_prompt_portions_and_decoding(case, dtype, schedule):
    """The same logits however the sequence is cut, in a slot that another request has used."""
    cfg, W, m = model_of(case, dtype)
    n = 230
    ids, logits, _ = expected(case, 1, n)
    pool = pool_for(m)
    pool.run("before", H.tokens(cfg, 120, 9))
    pool.end("before")
    at, got = 0, []
    for k in schedule + ([n - sum(schedule)] if sum(schedule) < n else []):
        got.append(pool.run("r", ids[at:at + k], range(k)))
        at += k
    assert at == n and len(pool.free) == 0
    err = H.error(torch.cat(got), logits)
    assert float(err.max()) < MODEL_TOL[dtype], (float(err.max()), int(err.argmax()))


@pytest.mark.parametrize("dtype", DTYPES)
def test_interleaved_requests_of_unequal_length(dtype):
    cfg, W, m = model_of("mixed", dtype)
    lengths = {"a": 90, "b": 33, "c": 61, "d": 7}
    want = {r: expected("mixed", i + 2, n) for i, (r, n) in enumerate(lengths.items())}
    pool, at, got = pool_for(m), dict.fromkeys(lengths, 0), {r: [] for r in lengths}
    cuts, turn = [5, 1, 2, 9, 1, 20], 0
    while any(at[r] < n for r, n in lengths.items()):
        for r, n in lengths.items():
            k = min(cuts[turn % len(cuts)], n - at[r])
            turn += 1
            if k == 0:
                continue
            got[r].append(pool.run(r, want[r][0][at[r]:at[r] + k], range(k)))
            at[r] += k
            if at[r] == n:
                pool.end(r)
    assert len(pool.free) == 4 and not pool.live
    for r in lengths:
        assert float(H.error(torch.cat(got[r]), want[r][1]).max()) < MODEL_TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("B", [2, 6, 40])
def test_batches_in_lockstep(dtype, B):
    """A batch gives every sequence the logits it has alone: prompt and decoding (40: more rows than a GEMV call takes)."""
    from dejavu_b200.generation import InferenceParams, allocate_kv_cache, step

    cfg, W, m = model_of("mixed", dtype)
    n = 60
    seqs = [expected("mixed", 20 + b % 6, n) for b in range(B)]
    ids = torch.tensor([s[0] for s in seqs]).cuda()
    ip = InferenceParams(max_sequence_len=n, max_batch_size=B, key_value_memory_dict=allocate_kv_cache(m, B, n, "cuda"))
    got = [step(m, ip, ids[:, :30]), step(m, ip, ids[:, 30:47])] + [step(m, ip, ids[:, t:t + 1]) for t in range(47, n)]
    got = torch.cat(got, 1)
    for b in range(B):
        assert float(H.error(got[b], seqs[b][1]).max()) < MODEL_TOL[dtype]


def test_long_decoding():
    """Token by token from the second on, far past every window and chunk, in fp32."""
    cfg, W, m = model_of("mixed", torch.float32)
    ids, logits, _ = expected("mixed", 5, 300)
    pool = pool_for(m)
    got = torch.cat([pool.run("r", [t], [0]) for t in ids])
    assert float(H.error(got, logits).max()) < MODEL_TOL[torch.float32]


def greedy(cfg, W, ids, new):
    ids = list(ids)
    for _ in range(new):
        ids.append(int(O.forward(cfg, W, ids)[-1].argmax()))
    return ids


@pytest.mark.parametrize("cg", [False, True])
@pytest.mark.parametrize("chunk", [None, 7])
def test_greedy_generation(cg, chunk):
    cfg, W, m = model_of("mixed", torch.float32)
    prompts = [H.tokens(cfg, 19, s) for s in (31, 32)]
    want = [greedy(cfg, W, p, 14) for p in prompts]
    out = m.generate(torch.tensor(prompts).cuda(), max_length=33, cg=cg, vocab_size=cfg["vocab"], prompt_chunk=chunk,
                     return_dict_in_generate=True, output_scores=True)
    assert out.sequences.tolist() == want
    assert len(out.scores) == 14
    # the captured step and its caches serve the next call as well
    assert m.generate(torch.tensor(prompts[::-1]).cuda(), max_length=33, cg=cg).tolist() == want[::-1]
    m._decoding_cache = None


def test_graph_step_is_the_eager_step():
    cfg, W, m = model_of("wide", torch.bfloat16)
    ids = torch.tensor([H.tokens(cfg, 30, 3)]).cuda()
    kw = dict(max_length=60, return_dict_in_generate=True, output_scores=True)
    a, b = m.generate(ids, cg=False, **kw), m.generate(ids, cg=True, **kw)
    m._decoding_cache = None
    assert torch.equal(a.sequences, b.sequences)
    assert all(torch.equal(x, y) for x, y in zip(a.scores, b.scores))


def test_command_lines(tmp_path):
    """Greedy generation and trace replay as a user runs them, from a model folder."""
    cfg, W, _ = model_of("odd", torch.float32)
    H.save(tmp_path, cfg, W)
    prompt = H.tokens(cfg, 12, 40)
    want = greedy(cfg, W, prompt, 8)[12:]
    r = subprocess.run([sys.executable, "-m", "dejavu_b200", "generate", "--model", str(tmp_path), "--tokens", ",".join(map(str, prompt)),
                        "--max-new-tokens", "8", "--dtype", "float32", "--cuda-graph"], cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [int(t) for t in r.stdout.strip().splitlines()[-1].split(",")] == want
    ids, logits, _ = expected("odd", 6, 25)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": ids[:10], "want": [0, 9]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": ids[10:12], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": ids[12:], "want": [12, 3]}], "end": ["x"]},
             {"step": 3, "entries": [{"id": "y", "tokens": ids[:1], "want": [0]}], "end": ["y"]}]
    r = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path),
                        "--max-tokens", "25"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {k}" for k in range(4)]
    for k, rows in ((0, [0, 9]), (2, [24, 15]), (3, [0])):
        data = torch.frombuffer(bytearray((tmp_path / f"{k}.f32").read_bytes()), dtype=torch.float32).view(len(rows), -1)
        assert float(H.error(data, logits[rows]).max()) < 1e-4
    assert not (tmp_path / "1.f32").exists()
