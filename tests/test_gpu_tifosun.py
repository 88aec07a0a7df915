"""Tifosun on the GPU against the plain CPU oracle: every mechanism alone, then whole models (prompts, portions, decoding,
batches, reused slots, generation, command line)."""
import json
import subprocess
import sys
from pathlib import Path

import pytest
import torch

sys.path.insert(0, str(Path(__file__).parent))
import hybrid_cases as H
import tifosun_cases as C
from oracle import tifosun_oracle as O

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parents[1]
DTYPES = [torch.float32, torch.bfloat16]


@pytest.fixture(scope="module", autouse=True)
def routed_lib():
    assert torch.cuda.is_available(), "GPU tests need a CUDA device"
    from dejavu_b200 import _lib

    lib = _lib.load_routed()
    yield lib
    assert lib.djv_window_timeouts() == lib.djv_mlstm_timeouts() == lib.djv_moe_timeouts() == 0


def gen(seed):
    return torch.Generator().manual_seed(seed)


def rnd(g, *shape, dtype=torch.float32, scale=1.0):
    """Random values that the element type holds exactly, in double."""
    return (torch.randn(*shape, generator=g) * scale).to(dtype).double()


def dev(t, dtype=torch.float32):
    return t.to(dtype).cuda().contiguous()


def close(got, want, dtype, f32, b16):
    got, want = got.double().cpu(), want.double()
    assert got.shape == want.shape
    scale = float(want.abs().max()) + 1e-30
    err = float((got - want).abs().max()) / scale
    assert err < (f32 if dtype == torch.float32 else b16), err


# ---- mechanisms ----------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D,n,k", [(64, 3, 0), (100, 5, 2), (257, 2, 1), (4096, 3, 3), (36, 400, 1), (1032, 7, 0), (7168, 2, 2), (12288, 2, 1)])
def test_residual_step(dtype, D, n, k):
    from dejavu_b200 import ops

    g = gen(D)
    x, y, gy, gh = rnd(g, n, D), rnd(g, n, D), rnd(g, D, scale=0.3), rnd(g, D, scale=0.3)
    parts = rnd(g, n + 4, D, dtype=dtype)
    places = torch.randint(0, n + 4, (n, max(k, 1)), generator=g, dtype=torch.int32)
    s = y + (parts[places.long()].sum(1) if k else 0)
    kw = dict(parts=dev(parts, dtype), part_rows=places.cuda()) if k else {}
    eps = 0.2  # (large: it shows)
    new = x + O.norm_around_zero(s, gy, eps)
    xd = dev(x)
    h = ops.residual_step(xd, dev(y), dev(gy), dev(gh), eps, dtype, base=1.0, x_out=xd, **kw)
    close(xd, new, torch.float32, 2e-6, 0)
    close(h, O.norm_around_zero(new, gh, eps), dtype, 1e-5, 5e-3)
    # plain sum, plain weight, selected rows
    rows = torch.tensor([n - 1, 0], dtype=torch.int32)
    h = ops.residual_step(dev(x), dev(y), None, dev(gh), eps, dtype, rows=rows.cuda(), **kw)
    close(h, (O.unit_rms(x + s, eps) * gh)[rows.long()], dtype, 1e-5, 5e-3)
    if k:  # parts alone
        out = torch.empty(n, D, device="cuda")
        ops.residual_step(dev(x), None, dev(gy), None, eps, dtype, base=1.0, x_out=out, **kw)
        close(out, x + O.norm_around_zero(s - y, gy, eps), torch.float32, 2e-6, 0)
    # from the embedding; ids out of range do not leave the table
    table, ids = rnd(g, 7, D, dtype=dtype), torch.tensor(([3, 6, 0, 5] * n)[:n])
    out = torch.empty(n, D, device="cuda")
    ops.residual_step(None, dev(y), dev(gy), None, eps, dtype, base=1.0, x_out=out, ids=ids.cuda(), embed=dev(table, dtype))
    close(out, table[ids] + O.norm_around_zero(y, gy, eps), torch.float32, 2e-6, 0)
    h = ops.residual_step(None, None, None, dev(gh), eps, dtype, base=1.0, ids=torch.full((n,), 99).cuda(), embed=dev(table, dtype))
    close(h, O.norm_around_zero(table[6], gh, eps).expand(n, D), dtype, 1e-5, 5e-3)
    assert ops.residual_step(dev(x), None, None, dev(gh), eps, dtype, rows=rows[:0].cuda()).shape == (0, D)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("B", [1, 3, 4, 5, 13, 32])
@pytest.mark.parametrize("N,M", [(64, 40), (1000, 34), (50, 22)])
def test_silu_gated_unit(dtype, B, N, M):
    from dejavu_b200 import ops

    g = gen(B * N)
    x, w = rnd(g, B, N, dtype=dtype), rnd(g, M, N, dtype=dtype, scale=N ** -0.5)
    y = x @ w.T
    close(ops.linear_gemv(dev(x, dtype), dev(w, dtype), None, "silu_glu"), O.silu(y[:, 0::2]) * y[:, 1::2], dtype, 1e-5, 5e-3)
    gu = rnd(g, B, M, dtype=dtype)
    close(ops.glu(dev(gu, dtype), "silu_glu"), O.silu(gu[:, 0::2]) * gu[:, 1::2], dtype, 1e-6, 5e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("base,dims,offset,heads", [(1000.0, 32, 16, 5), (5e4, 6, 1, 2), (1e6, 64, 128, 3), (70.0, 2, 0, 4)])
def test_rotary_of_neighbours(dtype, base, dims, offset, heads):
    from dejavu_b200 import ops
    from dejavu_b200.mixers import RotaryTable

    n, starts, dim = 9, [0, 3000], offset + dims
    x = rnd(gen(dim), 2 * n, heads * dim + 8, dtype=dtype)
    xd, t = dev(x, dtype), RotaryTable({"base": base, "dims": dims}, "cuda")
    ops.rotary_(xd[:, offset:], t.freqs, t.amp, torch.tensor(starts).cuda(), n, heads, dim, interleaved=True)
    want = x.clone()
    for b, s in enumerate(starts):
        r = want[b * n:(b + 1) * n, :heads * dim].view(n, heads, dim)
        r[..., offset:] = O.rotate_pairs(r[..., offset:].clone(), s + torch.arange(n), base)
    close(xd, want, dtype, 2e-4, 5e-3)


# heads, dk, dv, cap, forget bias, input bias: strong and weak forgetting, input gates that stay shut (the floor of the
# denominator decides) and ones near the cap (the constant beside it shows)
MEMORIES = [(2, 64, 64, 6.0, 2.0, 0.0), (3, 40, 24, 15.5, -1.0, 1.0), (2, 20, 36, 3.0, 0.0, -2.5), (1, 128, 128, 14.0, 4.0, 30.0),
            (2, 128, 256, 8.0, 3.0, -6.0), (1, 16, 8, 30.0, -20.0, 3.0), (3, 48, 80, 9.0, 6.0, 0.0), (1, 256, 64, 14.5, 1.0, 9.0),
            (2, 33, 17, 4.0, 1.0, 1.0), (1, 256, 256, 11.0, 2.0, -1.0), (1, 32, 200, 5.0, 5.0, 2.0), (1, 112, 384, 7.0, 3.0, 0.0),
            (2, 8, 16, 2.0, 0.5, 0.5), (1, 64, 512, 13.0, 3.0, 4.0)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("aligned", [True, False])
@pytest.mark.parametrize("heads,dk,dv,cap,fb,ib", MEMORIES)
def test_matrix_memory_portions_and_decoding(dtype, aligned, heads, dk, dv, cap, fb, ib):
    """Portions of many sizes and single tokens in turn, from a state that another sequence left, against the token by
    token recurrence; two sequences per call; a token far back stands out. The norm's constant is large, so that what
    divides the output shows."""
    from dejavu_b200 import ops

    n, eps, scale = 420, 0.05, dk ** -0.5
    g = gen(dk * dv)
    q, k, v, gate = (rnd(g, 2, n, heads, d, dtype=dtype) for d in (dk, dk, dv, dv))
    v[:, 3] *= 64  # (a power of two: still representable)
    zi, zf = rnd(g, 2, n, heads, scale=2.0), rnd(g, 2, n, heads, scale=2.0)
    bi, bf, norm = ib + rnd(g, heads), fb + rnd(g, heads), (1 + 0.3 * rnd(g, heads * dv)).float().double()
    bi, bf = bi.float().double(), bf.float().double()
    want, states = [], []
    for b in range(2):
        o, s = O.mlstm_recurrence(q[b] * scale, k[b], v[b], *O.mlstm_gates(zi[b], zf[b], bi, bf, cap))
        want.append(O.unit_rms(o, eps).reshape(n, -1) * norm * O.sigmoid(gate[b].reshape(n, -1)))
        states.append(torch.cat([s[0].reshape(heads, -1), s[1], s[2][:, None]], 1))
    rows = [torch.cat([t[b].reshape(n, -1) for t in (q, k, v, gate)], 1) for b in range(2)]
    gates = [torch.cat([zi[b], zf[b]], 1) for b in range(2)]
    state = torch.full_like(ops.mlstm_state(2, heads, dk, dv, "cuda"), 5.0)
    got, at = [[], []], 0
    sizes = [2, 3, 1, 64, 1, 1, 63, 5, 16, 1, 129, 2]
    width = rows[0].shape[1]
    for m in sizes + [n - sum(sizes) - 4, 1, 1, 1, 1]:
        # rows that 16-byte copies can read (the tensor-core chunk kernels), or not (the general ones)
        t = torch.float32 if m == 1 else dtype
        buf = torch.zeros(2 * m, (width + 15) // 8 * 8 if aligned else (width | 1) + 2, dtype=t, device="cuda")
        buf[:, :width] = dev(torch.cat([r[at:at + m] for r in rows]), t)
        out = ops.mlstm(buf, dev(torch.cat([x[at:at + m] for x in gates])), dev(bi), dev(bf), cap, dev(norm), eps, scale, state,
                        torch.tensor([at, at]).cuda(), m, dk, dv, dtype)
        for b in range(2):
            got[b].append(out[b * m:(b + 1) * m].cpu())
        at += m
    for b in range(2):
        close(torch.cat(got[b]), want[b], dtype, 1e-4, 1e-2)
        close(state[b, :, :dk * dv + dk + 1], states[b], torch.float32, 1e-4, 0)


def latent_mixer(heads, dim, rot, dv, rank, window, scale, width, dtype, seed, base=4000.0):
    from dejavu_b200.mixers import LatentAttention

    g = gen(seed)
    W = {"q": rnd(g, heads * (dim + rot), width, dtype=dtype, scale=width ** -0.5), "dkv": rnd(g, rank + rot, width, dtype=dtype, scale=width ** -0.5),
         "uk": rnd(g, heads * dim, rank, dtype=dtype, scale=rank ** -0.5), "uv": rnd(g, heads * dv, rank, dtype=dtype, scale=rank ** -0.5),
         "g": rnd(g, heads * dv, width, dtype=dtype, scale=width ** -0.5), "o": rnd(g, width, heads * dv, dtype=dtype, scale=(heads * dv) ** -0.5),
         "dkv.norm": (1 + 0.3 * rnd(g, rank)).float().double()}
    for h in range(heads):  # equal rotated parts of queries and keys: an activation's own like stands out
        W["q"][h * (dim + rot) + dim:(h + 1) * (dim + rot)] = W["dkv"][rank:]
    rotary = {"base": base, "dims": rot}
    m = LatentAttention(width, heads, dim, rot, dv, rank, scale, window, rotary, 1e-5, "cuda", dtype)
    for name, t in m.checkpoint_slots().items():
        t.copy_(W[name])
    m.zero_padding()
    mx = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": dv, "kv_rank": rank, "scale": scale, "rot": rotary,
          "mask": None if window is None else {"size": window}}
    return m, mx, W


def spiky(g, n, width, window, dtype):
    """Activations of which some repeat earlier ones, twice as large: their keys take most of the weight of the later query,
    or would, when they are just outside its window."""
    h = rnd(g, n, width, dtype=dtype)
    for i in range(0, n, 5):
        for back in (window - 1, window, window // 2):
            if 0 <= i - back and (i + back) % 3:
                h[i] = h[i - back] / 2
    return h


# heads, dim, rot, dv, rank, window
LATENTS = [(4, 32, 16, 32, 64, 45), (3, 9, 6, 10, 21, 3), (8, 64, 32, 64, 128, 150), (2, 128, 64, 128, 256, 64), (16, 16, 16, 24, 40, 7),
           (5, 48, 8, 80, 512, 130), (1, 16, 2, 16, 16, 1), (20, 24, 40, 16, 72, 33), (2, 64, 128, 96, 96, 100), (33, 8, 8, 8, 576, 20), (2, 40, 24, 256, 320, 70)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,rot,dv,rank,window", LATENTS)
def test_latent_attention_portions_and_decoding(dtype, heads, dim, rot, dv, rank, window):
    """Prompt portions of many sizes, then token by token, against one pass over everything; two sequences at different
    positions in one call; a cache that another sequence used before."""
    n, width = (2 * window + 45 if window > 20 else 70), 96
    m, mx, W = latent_mixer(heads, dim, rot, dv, rank, window, 0.5 * (dim + rot) ** -0.5, width, dtype, rank + dv)
    seqs = [spiky(gen(b), n, width, window, dtype) for b in range(2)]
    want = [O.latent_attention_mixer(h, W, "", mx, 1e-5) for h in seqs]
    cache = (torch.full((2, min(window, n), rank + rot), 7.0, dtype=dtype, device="cuda"),)  # stale content
    got = [[], []]

    def call(at, k):
        h = dev(torch.cat([seqs[b][a:a + k] for b, a in enumerate(at)]), dtype)
        out = m(h, cache, torch.tensor(at).cuda(), k, max(at))
        for b in range(2):
            got[b].append(out[b * k:(b + 1) * k].cpu())

    # sequence 1 runs 6 tokens behind: it repeats its first tokens
    call([0, 0], 6)
    got[1].clear()
    at = [6, 0]
    for k in (2, 3, 1, 16, 2, 17, 1, 5):
        call(at, k)
        at = [a + k for a in at]
    rest = n - 8 - at[0]
    if rest > 1:
        call(at, rest)
        at = [a + rest for a in at]
    while at[0] < n:
        call(at, 1)
        at = [a + 1 for a in at]
    for b in range(2):
        res = torch.cat(got[b])
        close(res, want[b][:res.shape[0]], dtype, 5e-5, 2e-2)


@pytest.mark.parametrize("dtype", DTYPES)
def test_latent_attention_without_a_window(dtype):
    n, width = 330, 64
    m, mx, W = latent_mixer(3, 32, 16, 48, 64, None, 0.2, width, dtype, 1)
    h = spiky(gen(9), n, width, 300, dtype)
    want = O.latent_attention_mixer(h, W, "", mx, 1e-5)
    cache, at, out = m.new_cache(1, n, "cuda", dtype), 0, []
    for k in (150, 1, 1, 138, 1, 39):
        out.append(m(dev(h[at:at + k], dtype), cache, torch.tensor([at]).cuda(), k, at))
        at += k
    close(torch.cat(out), want, dtype, 5e-5, 2e-2)


@pytest.mark.parametrize("dtype", DTYPES)
def test_latent_decode_of_many_sequences(dtype):
    """Sequences of one batch at unequal positions give what each gives alone."""
    B, width, window = 7, 64, 40
    m, mx, W = latent_mixer(6, 32, 16, 32, 96, window, 0.3, width, dtype, 2)
    lengths = [1, 5, 39, 40, 41, 77, 120]
    seqs = [spiky(gen(20 + b), n, width, window, dtype) for b, n in enumerate(lengths)]
    cache = m.new_cache(B, 200, "cuda", dtype)
    for b, n in enumerate(lengths):
        if n > 1:
            m(dev(seqs[b][:-1], dtype), tuple(c[b:b + 1] for c in cache), torch.tensor([0]).cuda(), n - 1, 0)
    out = m(dev(torch.stack([s[-1] for s in seqs]), dtype), cache, torch.tensor([n - 1 for n in lengths]).cuda(), 1, 0)
    want = torch.stack([O.latent_attention_mixer(s, W, "", mx, 1e-5)[-1] for s in seqs])
    close(out, want, dtype, 5e-5, 2e-2)


# width, ff, experts, top, shared ff
MIXTURES = [(64, 32, 6, 2, 48), (100, 30, 5, 3, 14), (128, 24, 40, 4, None), (256, 200, 4, 1, 40), (72, 136, 9, 9, 8), (40, 8, 1, 1, None),
            (320, 264, 3, 2, 264), (64, 64, 300, 8, None)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,ff,experts,top,shared", MIXTURES)
@pytest.mark.parametrize("rows", [1, 3, 5, 32, 33, 130, 700])
def test_mixture_of_experts(dtype, width, ff, experts, top, shared, rows):
    from dejavu_b200 import ops
    from dejavu_b200.mixers import MixtureOfExperts, SplitSum

    g = gen(width + ff)
    m = MixtureOfExperts(width, ff, experts, top, shared, "cuda", dtype)
    W = {}
    for name, t in m.checkpoint_slots().items():
        W[name] = rnd(g, *t.shape, dtype=dtype, scale=(4.0 if name == "router" else 1.5) * t.shape[1] ** -0.5)
        t.copy_(W[name])
    h = rnd(gen(rows), rows, width, dtype=dtype)
    if experts > 3:
        h[: rows // 2] = h[0] + 0.01 * h[: rows // 2].to(dtype).double()  # most tokens to a few experts, some get none
        h = h.to(dtype).double()
    mlp = {"router": {"top": top}, "shared": None if shared is None else {"ff": shared}}
    want = O.mixture(h, W, "", mlp)
    # (tokens whose last chosen and first left out score are as good as equal prove nothing)
    z = torch.sort(h @ W["router"].T, dim=1, descending=True).values
    sure = torch.ones(rows, dtype=torch.bool) if top == experts else z[:, top - 1] - z[:, top] > 1e-4
    for n in {1, rows}:
        y = m(dev(h, dtype), n)
        if isinstance(y, SplitSum):
            zero = torch.zeros(rows, width, device="cuda")
            out = torch.empty(rows, width, device="cuda")
            ops.residual_step(zero, y.y, None, None, 0.0, dtype, x_out=out, parts=y.parts, part_rows=y.places)
            assert sorted(y.places.flatten().tolist()) == list(range(rows * top))
            y = out
        close(y[sure.cuda()], want[sure], dtype, 2e-5, 2e-2)


# ---- whole models --------------------------------------------------------------------------------------------------

_models: dict = {}


def model_of(case, dtype):
    from dejavu_b200.tifosun import TifosunForCausalLM

    if (case, dtype) not in _models:
        cfg, sharp = C.CASES[case], 1.0
        if dtype == torch.bfloat16:
            cfg, sharp = C.calm(cfg), 0.6
        W = C.weights(cfg, sharp=sharp)
        _models[case, dtype] = (cfg, W, TifosunForCausalLM(cfg, device="cuda", dtype=dtype).load_tensors(W))
    return _models[case, dtype]


_expected: dict = {}


def expected(case, seed, n, dtype=torch.float32):
    cfg, W = model_of(case, dtype)[:2]
    key = (case, seed, n, dtype)
    if key not in _expected:
        ids = H.tokens(cfg, n, seed)
        _expected[key] = (ids, *O.forward(cfg, W, ids, return_layers=True))
    return _expected[key]


def check(got, want, dtype):
    """(A head whose output nearly cancels is scaled up by its norm, rounding with it: a few positions may be further off.)"""
    err = H.error(got, want)
    most, nearly_all = (1e-3, 3e-5) if dtype == torch.float32 else (0.25, 0.08)
    assert float(err.max()) < most and float(err.quantile(0.95)) < nearly_all, (float(err.quantile(0.95)), float(err.max()), int(err.argmax()))


def pool_for(model, n=400):
    from dejavu_b200.generation import SequencePool

    return SequencePool(model, n, torch.device("cuda"))


@pytest.mark.parametrize("case", C.CASES)
def test_layers_in_fp32(case):
    cfg, W, m = model_of(case, torch.float32)
    ids, logits, trail = expected(case, 0, 50)
    got = []
    with torch.inference_mode():
        out = m(torch.tensor([ids]).cuda(), collect=got).logits[0]
    assert len(got) == len(trail)
    for a, b in zip(got, trail):
        close(a, b, torch.float32, 5e-5, 0)
    check(out, logits, torch.float32)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", C.CASES)
@pytest.mark.parametrize("schedule", [[230], [1] * 40 + [190], [2] * 5 + [3, 64, 1, 1, 16, 17, 5, 1, 100, 2], [199] + [1] * 31, [37] * 5])
def test_prompt_portions_and_decoding(case, dtype, schedule):
    """The same logits however the sequence is cut, in a slot that another request has used."""
    cfg, W, m = model_of(case, dtype)
    n = 230
    ids, logits, _ = expected(case, 1, n, dtype)
    pool = pool_for(m)
    pool.run("before", H.tokens(cfg, 120, 9))
    pool.end("before")
    at, got = 0, []
    for k in schedule + ([n - sum(schedule)] if sum(schedule) < n else []):
        got.append(pool.run("r", ids[at:at + k], range(k)))
        at += k
    assert at == n and len(pool.free) == 0
    check(torch.cat(got), logits, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_interleaved_requests_of_unequal_length(dtype):
    cfg, W, m = model_of("mixed", dtype)
    lengths = {"a": 90, "b": 33, "c": 61, "d": 7}
    want = {r: expected("mixed", i + 2, n, dtype) for i, (r, n) in enumerate(lengths.items())}
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
    check(torch.cat([torch.cat(got[r]) for r in lengths]), torch.cat([want[r][1] for r in lengths]), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("B", [2, 6, 40])
def test_batches_in_lockstep(dtype, B):
    """A batch gives every sequence the logits it has alone: prompt and decoding (40: more rows than a GEMV call takes)."""
    from dejavu_b200.generation import InferenceParams, allocate_kv_cache, step

    cfg, W, m = model_of("mixed", dtype)
    n = 60
    seqs = [expected("mixed", 20 + b % 6, n, dtype) for b in range(B)]
    ids = torch.tensor([s[0] for s in seqs]).cuda()
    ip = InferenceParams(max_sequence_len=n, max_batch_size=B, key_value_memory_dict=allocate_kv_cache(m, B, n, "cuda"))
    got = [step(m, ip, ids[:, :30]), step(m, ip, ids[:, 30:47])] + [step(m, ip, ids[:, t:t + 1]) for t in range(47, n)]
    got = torch.cat(got, 1)
    for b in range(B):
        check(got[b], seqs[b][1], dtype)


def test_long_decoding():
    """Token by token from the second on, far past every window and chunk, in fp32."""
    cfg, W, m = model_of("mixed", torch.float32)
    ids, logits, _ = expected("mixed", 5, 300)
    pool = pool_for(m)
    check(torch.cat([pool.run("r", [t], [0]) for t in ids]), logits, torch.float32)


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


@pytest.mark.parametrize("B", [1, 6])
def test_graph_step_is_the_eager_step(B):
    cfg, W, m = model_of("wide", torch.bfloat16)
    ids = torch.tensor([H.tokens(cfg, 30, s) for s in range(B)]).cuda()
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
