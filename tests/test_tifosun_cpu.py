"""Tifosun without a GPU: configuration, registry, weight files, command line, argument checks, and the oracle itself (that
its mechanisms equal other ways to write them, and that the test weights make mistakes visible)."""
import ctypes
import math
import subprocess
import sys
from pathlib import Path

import pytest
import torch

sys.path.insert(0, str(Path(__file__).parent))
import hybrid_cases as H
import tifosun_cases as C
from oracle import tifosun_oracle as O

ROOT = Path(__file__).resolve().parents[1]


# ---- weight files and registry -----------------------------------------------------------------------------------

@pytest.mark.parametrize("case", C.CASES)
def test_registry_builds_and_fills_the_model(tmp_path, case):
    from dejavu_b200 import registry

    cfg = C.CASES[case]
    W = C.weights(cfg)
    H.save(tmp_path, cfg, W)
    model = registry.load_model(str(tmp_path), torch.float32, "cpu")
    assert type(model).__name__ == "TifosunForCausalLM" and model.runs == list(range(len(cfg["layers"])))
    slots = model.checkpoint_slots()
    assert set(slots) == set(W)
    for name, t in W.items():
        assert torch.equal(slots[name].double(), t), name
    for layer in model.layers:  # fused rows that are only there for alignment are zeros
        m = layer.mixer
        assert not m.proj.weight[sum(m.sizes):getattr(m, "main", None)].any()
    assert registry.load_model(str(tmp_path), None, "cpu").embed.dtype == torch.bfloat16
    assert registry.entry_for(cfg).library == "routed"
    with pytest.raises(ValueError, match="not torch.float16"):
        registry.load_model(str(tmp_path), torch.float16, "cpu")


def test_registry_errors(tmp_path):
    from dejavu_b200 import registry

    cfg = C.CASES["odd"]
    W = C.weights(cfg)
    for bad, msg in (({k: v for k, v in W.items() if k != "l0.mlp.e2.up"}, "missing \\['l0.mlp.e2.up'\\]"),
                     ({**W, "l1.mix.extra": torch.zeros(2)}, "unknown"),
                     ({**W, "l1.norm2b": torch.zeros(3)}, "l1.norm2b: shape")):
        H.save(tmp_path, cfg, bad)
        with pytest.raises(ValueError, match=msg):
            registry.load_model(str(tmp_path), torch.float32, "cpu")


def test_config_is_checked():
    from dejavu_b200.tifosun import TifosunForCausalLM, parse_config

    cfg = C.CASES["odd"]
    assert parse_config(cfg).eps == 1e-3
    first, second = cfg["layers"]
    for bad in ({**first, "type": "other"}, {**first, "mlp": {"kind": "other"}}):
        with pytest.raises(ValueError):
            parse_config({**cfg, "layers": [bad, second]})
    with pytest.raises(ValueError, match="rotary dims"):
        TifosunForCausalLM({**cfg, "layers": [{**second, "mixer": {**second["mixer"], "rot": {"base": 9.0, "dims": 4}}}]}, device="cpu")
    with pytest.raises(ValueError, match="experts"):
        TifosunForCausalLM({**cfg, "layers": [{**first, "mlp": C.moe(3, 4, 8)}]}, device="cpu")


def test_caches_hold_the_window_and_the_state():
    from dejavu_b200 import build
    from dejavu_b200.tifosun import TifosunForCausalLM

    build.build(libs=("routed",))
    m = TifosunForCausalLM(C.CASES["mixed"], device="cpu", dtype=torch.float32)
    caches = m.allocate_cache(2, 1000, "cpu")
    assert caches[1][0].shape == (2, 19, 56 + 16) and caches[3][0].shape == (2, 5, 24 + 8)
    assert m.allocate_cache(1, 11, "cpu")[1][0].shape == (1, 11, 72)
    assert caches[0][0].shape[:2] == (2, 3) and caches[0][0].shape[2] >= 40 * 24 + 40 + 1 and caches[0][0].dtype == torch.float32


def test_random_initialisation():
    from dejavu_b200.tifosun import TifosunForCausalLM

    slots = TifosunForCausalLM(C.CASES["odd"], device="cpu").init_random(3).checkpoint_slots()
    for name, t in slots.items():
        if name.endswith(("mix.norm", "dkv.norm")):
            assert bool((t == 1).all()), name
        elif "norm" in name or name.endswith("i.b"):
            assert not t.any(), name
        elif name.endswith("f.b"):
            assert bool((t == 3).all())
        else:
            assert 0.01 < float(t.float().std()) < 0.03, name


def test_command_refuses_other_types(tmp_path):
    cfg = C.CASES["odd"]
    H.save(tmp_path, cfg, C.weights(cfg))
    r = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(tmp_path), "--dtype", "float16", "--out", str(tmp_path),
                        "--max-tokens", "8"], capture_output=True, text=True, stdin=subprocess.DEVNULL)
    assert r.returncode == 3


def test_kernels_check_their_arguments_on_the_host():
    from dejavu_b200 import _lib, build

    build.build(libs=("routed",))
    lib = _lib.load_routed()
    before, p, BF = lib.djv_launch_count(), ctypes.c_void_p(0x1000), _lib.DTYPE_BF16
    bad = _lib.ERR_INVALID
    step = (BF, p, p, p, p)
    assert lib.djv_residual_step(*step, p, None, 0, p, p, 1.0, 1e-5, None, None, None, 1, 64, 0, None) == bad
    assert lib.djv_residual_step(BF, p, p, None, p, None, None, 0, p, p, 1.0, 1e-5, None, None, None, 1, 64, 0, None) == bad
    assert lib.djv_residual_step(*step, None, None, 0, p, p, 1.0, 1e-5, None, None, None, 1, 50000, 0, None) == bad
    assert lib.djv_dense_gemv(BF, BF, p, p, p, 1, 64, 7, 64, _lib.ACT["silu_glu"], 0.0, None) == bad
    assert lib.djv_glu(BF, p, p, 4, 8, _lib.ACT["relu"], 0.0, None) == bad
    gates = (p, 4, p, p)
    assert lib.djv_mlstm_prefill(BF, p, p, 200, *gates, 0.0, p, 1e-5, 1.0, p, p, 1, 4, 2, 16, 16, p, 1 << 30, None) == bad
    assert lib.djv_mlstm_prefill(BF, p, p, 100, *gates, 5.0, p, 1e-5, 1.0, p, p, 1, 4, 2, 16, 16, p, 1 << 30, None) == bad
    assert lib.djv_mlstm_prefill(BF, p, p, 200, *gates, 5.0, p, 1e-5, 1.0, p, p, 1, 4, 2, 16, 16, p, 16, None) == _lib.ERR_SCRATCH
    assert lib.djv_mlstm_decode(BF, p, p, 200, p, 3, p, p, 5.0, p, 1e-5, 1.0, p, p, 1, 2, 16, 16, None) == bad
    assert lib.djv_latent_rows(BF, p, p, 20, p, p, 1e-5, p, p, 1, 4, 0, 16, 8, 8, 0, None) == bad
    assert lib.djv_latent_rows(BF, p, p, 24, p, p, 1e-5, p, p, 1, 4, 9, 16, 8, 8, 0, None) == bad
    assert lib.djv_latent_attn(BF, p, p, 47, p, 64, p, 8, None, 0, p, 1, 4, 0, 2, 16, 8, 16, 8, 1.0, None) == bad
    assert lib.djv_latent_decode(BF, p, p, p, 1 << 20, p, 60, p, p, p, 1e-5, p, p, None, 0, p, 1, 2, 16, 8, 16, 16, 8, 8, 1.0, 7, None) == bad
    assert lib.djv_latent_decode(BF, p, p, p, 16, p, 72, p, p, p, 1e-5, p, p, None, 0, p, 1, 2, 16, 8, 16, 16, 8, 8, 1.0, 7, None) == _lib.ERR_SCRATCH
    assert lib.djv_moe_route(BF, p, p, p, p, p, p, p, p, p, 4, 3, 4, 64, None) == bad
    assert lib.djv_moe_grouped(BF, p, p, p, None, p, 4, 3, 7, 64, 1, None) == bad
    assert lib.djv_moe_decode(BF, p, p, p, p, p, p, p, p, None, None, 1, 4, 1, 64, 32, 16, 32, 3, None) == bad
    assert lib.djv_launch_count() == before


# ---- the oracle ----------------------------------------------------------------------------------------------------

def gen(seed):
    return torch.Generator().manual_seed(seed)


def rand(g, *shape):
    return torch.randn(*shape, generator=g, dtype=torch.float64)


def test_oracle_memory_equals_its_sum():
    """Without the running maximum: o = sum_s D(t, s) (q.k_s) v_s over max(|sum_s D(t, s) q.k_s|, 1), D the product of the
    gates; the constant beside the maximum is seen through e^m."""
    g = gen(3)
    n, heads, dk, dv = 14, 2, 6, 5
    q, k, v = rand(g, n, heads, dk), rand(g, n, heads, dk), rand(g, n, heads, dv)
    i, f = O.mlstm_gates(2 * rand(g, n, heads), rand(g, n, heads), rand(g, heads), rand(g, heads), 4.0)
    assert float(i.abs().max()) < 4.0 and float(f.max()) < 0.0
    got, state = O.mlstm_recurrence(q, k, v, i, f)
    m = torch.zeros(heads, dtype=torch.float64)
    for t in range(n):
        m = torch.maximum(f[t] + m, i[t])
        for h in range(heads):
            d = torch.stack([torch.exp(i[s, h] + f[s + 1:t + 1, h].sum()) for s in range(t + 1)])
            a = d * (k[:t + 1, h] @ q[t, h])
            den = max(abs(float(a.sum())), 1.0) + 1e-6 * math.exp(float(m[h]))
            assert torch.allclose(got[t, h], (a @ v[:t + 1, h]) / den)
    a, s = O.mlstm_recurrence(q[:5], k[:5], v[:5], i[:5], f[:5])
    b, s = O.mlstm_recurrence(q[5:], k[5:], v[5:], i[5:], f[5:], s)
    assert torch.allclose(torch.cat([a, b]), got) and all(torch.allclose(x, y) for x, y in zip(s, state))


def test_oracle_attention_equals_a_dense_mask():
    g = gen(1)
    n, heads, dk, dv, w = 23, 3, 8, 6, 7
    q, k, v = rand(g, n, heads, dk), rand(g, n, heads, dk), rand(g, n, heads, dv)
    got = O.window_softmax_attention(q, k, v, 0.3, w)
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    for h in range(heads):
        s = (q[:, h] @ k[:, h].T * 0.3).masked_fill((j > i) | (i - j >= w), -math.inf)
        assert torch.allclose(got[:, h], torch.softmax(s, 1) @ v[:, h])


def test_oracle_rotation_is_a_complex_product():
    g = gen(4)
    x, pos = rand(g, 5, 3, 8), torch.tensor([0, 1, 7, 100, 1000])
    f = 300.0 ** (-torch.arange(0, 8, 2, dtype=torch.float64) / 8)
    want = torch.view_as_complex(x.reshape(5, 3, 4, 2)) * torch.polar(torch.ones(5, 1, 4, dtype=torch.float64), (pos[:, None] * f)[:, None])
    assert torch.allclose(O.rotate_pairs(x, pos, 300.0), torch.view_as_real(want).reshape(5, 3, 8))
    assert torch.allclose(O.rotate_pairs(x[:, 0], pos, 300.0), torch.view_as_real(want).reshape(5, 3, 8)[:, 0])


def test_oracle_latent_keys_work_on_the_query_as_well():
    """Scores from expanded keys equal scores of queries taken through the key projection, against the latents."""
    g = gen(5)
    n, heads, dim, rank = 6, 3, 4, 7
    c, uk, q = rand(g, n, rank), rand(g, heads * dim, rank), rand(g, heads, dim)
    k, _ = O.latent_keys_values(c, rand(g, n, 2), uk, rand(g, heads, rank), heads)
    for h in range(heads):
        assert torch.allclose(k[:, h, :dim] @ q[h], c @ (uk[h * dim:(h + 1) * dim].T @ q[h]))


def test_oracle_mixture():
    mlp, cfg = C.moe(5, 2, 6, 3), C.config(10, 8, [C.memory(1, 4, 4, 2.0, C.moe(5, 2, 6, 3))])
    W = C.weights(cfg, 1)
    h = rand(gen(6), 9, 8)
    y = O.mixture(h, W, "l0.mlp.", mlp)
    s = torch.sigmoid(h @ W["l0.mlp.router"].T)
    for t in range(9):
        want = O.gated_unit(h[t], W, "l0.mlp.shared.")
        for e in s[t].topk(2).indices.tolist():
            want = want + O.gated_unit(s[t, e] * h[t], W, f"l0.mlp.e{e}.")
        assert torch.allclose(y[t], want)


def _state_lost(f):
    def wrong(q, k, v, i, fg):
        return torch.cat([f(q[:20], k[:20], v[:20], i[:20], fg[:20])[0], f(q[20:], k[20:], v[20:], i[20:], fg[20:])[0]]), None

    return wrong


def _maximum_lost(f):
    def wrong(q, k, v, i, fg):
        o, (S, N, m) = f(q[:20], k[:20], v[:20], i[:20], fg[:20])
        return torch.cat([o, f(q[20:], k[20:], v[20:], i[20:], fg[20:], (S, N, 0 * m))[0]]), None

    return wrong


def _normaliser_lost(f):
    def wrong(q, k, v, i, fg):
        o, (S, N, m) = f(q[:20], k[:20], v[:20], i[:20], fg[:20])
        return torch.cat([o, f(q[20:], k[20:], v[20:], i[20:], fg[20:], (S, 0 * N, m))[0]]), None

    return wrong


MISTAKES = {
    "window one longer": ("window_softmax_attention", lambda f: lambda q, k, v, s, w: f(q, k, v, s, w + 1)),
    "window one shorter": ("window_softmax_attention", lambda f: lambda q, k, v, s, w: f(q, k, v, s, w - 1)),
    "another scale": ("window_softmax_attention", lambda f: lambda q, k, v, s, w: f(q, k, v, s * 1.2, w)),
    "pairs half a head apart": ("rotate_pairs", lambda f: lambda x, p, b: torch.cat([(y := f(torch.stack(
        [x[..., :x.shape[-1] // 2], x[..., x.shape[-1] // 2:]], -1).flatten(-2), p, b))[..., 0::2], y[..., 1::2]], -1)),
    "another base": ("rotate_pairs", lambda f: lambda x, p, b: f(x, p, b * 1.5)),
    "latents not normed": ("latent_rows", lambda f: lambda d, w, r, b, e, p: (d[:, :r] * w, f(d, w, r, b, e, p)[1])),
    "key part normed": ("latent_rows", lambda f: lambda d, w, r, b, e, p: (f(d, w, r, b, e, p)[0], O.unit_rms(f(d, w, r, b, e, p)[1], e))),
    "state lost once": ("mlstm_recurrence", _state_lost),
    "normaliser lost once": ("mlstm_recurrence", _normaliser_lost),
    "maximum lost once": ("mlstm_recurrence", _maximum_lost),
    "gates not capped": ("capped", lambda f: lambda x, c: x),
    "another cap": ("capped", lambda f: lambda x, c: f(x, c * 1.3)),
    "weights around one": ("norm_around_zero", lambda f: lambda x, w, e: f(x, w - 1, e)),
    "weight on the output": ("mixture", lambda f: lambda h, W, p, mlp: sum(
        ((w := O.route(h @ W[p + "router"].T, mlp["router"]["top"]))[1][:, k:k + 1] * torch.stack(
            [O.gated_unit(h[t], W, f"{p}e{int(w[0][t, k])}.") for t in range(h.shape[0])]) for k in range(mlp["router"]["top"])),
        O.gated_unit(h, W, p + "shared.") if mlp["shared"] else 0)),
    "weights renormalised": ("route", lambda f: lambda z, top: (f(z, top)[0], f(z, top)[1] / f(z, top)[1].sum(1, keepdim=True))),
    "the last expert left out": ("route", lambda f: lambda z, top: f(z, max(top - 1, 1))),
}


@pytest.mark.parametrize("name", MISTAKES)
def test_test_weights_show_mistakes(monkeypatch, name):
    """A model with one mistake planted in it differs by far more than the tolerances of the GPU tests. (What divides a
    memory's output by a common factor shows only through the constant in the norm behind it: a large one.)"""
    cfg = {**C.CASES["mixed"], "norm": {"eps": 0.5}} if name in ("normaliser lost once", "maximum lost once") else C.CASES["mixed"]
    W = C.weights(cfg)
    ids = H.tokens(cfg, 45, 0)
    want = O.forward(cfg, W, ids)
    fn, wrong = MISTAKES[name]
    monkeypatch.setattr(O, fn, wrong(getattr(O, fn)))
    assert float(H.error(O.forward(cfg, W, ids), want).max()) > 0.03
