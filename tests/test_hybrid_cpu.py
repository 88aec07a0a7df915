"""Hybrid decoders without a GPU: configuration, registry, weight files, request pool, command line, and the oracle
itself (that its two forms of each mechanism agree, and that the test weights make mistakes visible)."""
import json
import math
import subprocess
import sys
from pathlib import Path
from types import SimpleNamespace

import pytest
import torch

sys.path.insert(0, str(Path(__file__).parent))
import hybrid_cases as H
from oracle import hybrid_oracle as O

ROOT = Path(__file__).resolve().parents[1]


# ---- weight files and registry ----------------------------------------------------------------------------------

def test_safetensors_reader(tmp_path):
    from dejavu_b200.checkpoint import read_safetensors

    a, b = torch.randn(3, 5).to(torch.bfloat16), torch.arange(6, dtype=torch.int32).view(2, 3)
    blobs = [a.view(torch.uint8).numpy().tobytes(), b.numpy().tobytes()]
    header = {"__metadata__": {"x": "y"},
              "a": {"dtype": "BF16", "shape": [3, 5], "data_offsets": [0, 30]},
              "b": {"dtype": "I32", "shape": [2, 3], "data_offsets": [30, 54]},
              "e": {"dtype": "F32", "shape": [0, 4], "data_offsets": [54, 54]}}
    h = json.dumps(header).encode()
    f = tmp_path / "m.safetensors"
    f.write_bytes(len(h).to_bytes(8, "little") + h + b"".join(blobs))
    got = read_safetensors(str(f))
    assert torch.equal(got["a"], a) and torch.equal(got["b"], b) and got["e"].shape == (0, 4)
    f.write_bytes(len(h).to_bytes(8, "little") + h + blobs[0])
    with pytest.raises(ValueError):
        read_safetensors(str(f))


@pytest.mark.parametrize("case", H.CASES)
def test_registry_builds_and_fills_the_model(tmp_path, case):
    from dejavu_b200 import registry

    cfg, rank = H.CASES[case]
    W = H.weights(cfg, rank)
    H.save(tmp_path, cfg, W)
    model = registry.load_model(str(tmp_path), torch.float32, "cpu")
    assert type(model).__name__ == "NinolornForCausalLM" and model.runs == O.layer_order(cfg)
    slots = model.checkpoint_slots()
    assert set(slots) == set(W)
    for name, t in W.items():
        assert torch.equal(slots[name].double(), t), name
    for layer in model.layers:  # the fused decay rows end in zeros
        if hasattr(layer.mixer, "a2"):
            assert layer.mixer.rank == rank and not layer.mixer.proj.weight[sum(layer.mixer.sizes):].any()
    assert registry.load_model(str(tmp_path), None, "cpu").embed.dtype == torch.bfloat16
    with pytest.raises(ValueError, match="not torch.float16"):
        registry.load_model(str(tmp_path), torch.float16, "cpu")


def test_registry_errors(tmp_path):
    from dejavu_b200 import registry

    cfg, rank = H.CASES["odd"]
    W = H.weights(cfg, rank)
    for bad, msg in (({k: v for k, v in W.items() if k != "head"}, "missing \\['head'\\]"),
                     ({**W, "l0.mix.extra": torch.zeros(2)}, "unknown"),
                     ({**W, "final.norm": torch.zeros(3)}, "final.norm: shape")):
        H.save(tmp_path, cfg, bad)
        with pytest.raises(ValueError, match=msg):
            registry.load_model(str(tmp_path), torch.float32, "cpu")
    H.save(tmp_path, {**cfg, "architecture": "Unheard"}, W)
    with pytest.raises(ValueError, match="unknown architecture"):
        registry.load_model(str(tmp_path), torch.float32, "cpu")


def test_config_is_checked():
    from dejavu_b200.ninolorn import parse_config

    cfg, _ = H.CASES["odd"]
    assert parse_config(cfg).loop == (0, 0, 1)
    for bad in ({**cfg, "loop": {"start": 1, "stop": 5, "times": 2}}, {**cfg, "loop": {"start": 0, "stop": 1, "times": 0}},
                {**cfg, "layers": [{**cfg["layers"][0], "type": "other"}]},
                {**cfg, "layers": [{**cfg["layers"][0], "mlp": {"kind": "other"}}]}):
        with pytest.raises(ValueError):
            parse_config(bad)


def test_registry_serves_opt_folders():
    from dejavu_b200 import registry

    raw = {"architectures": ["OPTForCausalLM"], "hidden_size": 64, "num_hidden_layers": 2, "num_attention_heads": 4,
           "ffn_dim": 128, "vocab_size": 96, "max_position_embeddings": 40, "activation_function": "relu"}
    cfg = registry.opt_config_from_json(raw)
    assert (cfg.n_layer, cfg.n_embd, cfg.n_head, cfg.n_inner, cfg.vocab_size) == (2, 64, 4, 128, 96)
    assert not cfg.mlp_sparse and not cfg.att_sparse
    from transformers import OPTConfig, OPTForCausalLM

    torch.manual_seed(0)
    hf = OPTForCausalLM(OPTConfig(**{k: v for k, v in raw.items() if k != "architectures"}, word_embed_proj_dim=64))
    sd = {k: v for k, v in hf.state_dict().items()}
    model = registry.entry_for(raw).build(raw, sd, "cpu", torch.float16)
    w = model.transformer.layers[1].mlp.fc1.weight
    assert torch.equal(w, sd["model.decoder.layers.1.fc1.weight"].half())


@pytest.mark.parametrize("rot", [{"base": 1000.0, "dims": 48, "scaling": H.YARN}, {"base": 5e5, "dims": 6, "scaling": None},
                                 {"base": 250.0, "dims": 64, "scaling": {"factor": 3.0, "original": 8, "fast": 64.0, "slow": 2.0}},
                                 {"base": 3.0, "dims": 16, "scaling": {"factor": 2.0, "original": 100000, "fast": 4.0, "slow": 4.0}}])
def test_rotary_table(rot):
    from dejavu_b200.mixers import RotaryTable

    t = RotaryTable(rot)
    freqs, amp = O.rotary_frequencies(rot)
    assert t.amp == pytest.approx(amp) and torch.allclose(t.freqs.double(), torch.tensor(freqs, dtype=torch.float64), rtol=1e-6)


# ---- request pool, with a model that only records ------------------------------------------------------------------

class Recorder:
    takes_portions = selects_logit_rows = True

    def __init__(self):
        self.config = SimpleNamespace(vocab_size=50)
        self.caches = 0

    def allocate_cache(self, batch, max_len, device):
        self.caches += 1
        return {"id": self.caches, "seen": []}

    def __call__(self, ids, position_ids=None, inference_params=None, logit_rows=None):
        c = inference_params.key_value_memory_dict
        p = inference_params.sequence_len_offset
        if position_ids is not None:
            assert int(position_ids[0, 0]) == p
        if p == 0:
            c["seen"] = []
        c["seen"] += ids[0].tolist()
        assert len(c["seen"]) == p + ids.size(1)
        return SimpleNamespace(logits=torch.tensor([[[float(c["seen"][p + r])] for r in logit_rows]]))


def test_pool_keeps_requests_apart_and_reuses_slots():
    from dejavu_b200.generation import SequencePool

    m = Recorder()
    pool = SequencePool(m, 8, "cpu")
    assert pool.run("a", [1, 2, 3], [0, 2]).flatten().tolist() == [1, 3]
    assert pool.run("b", [9], [0]).flatten().tolist() == [9]
    assert pool.run("a", [4], [0]).flatten().tolist() == [4]
    assert pool.live["a"].key_value_memory_dict["seen"] == [1, 2, 3, 4] and pool.live["b"].key_value_memory_dict["seen"] == [9]
    pool.end("a")
    pool.run("c", [7, 8], [])
    assert pool.live["c"].key_value_memory_dict["id"] == 1 and m.caches == 2
    assert pool.live["c"].key_value_memory_dict["seen"] == [7, 8]
    for tokens, rows in (([50], []), ([-1], []), ([], []), ([1], [1])):
        with pytest.raises(ValueError):
            pool.run("b", tokens, rows)
    with pytest.raises(ValueError, match="exceed the cache"):
        pool.run("b", list(range(8)), [])
    m.takes_portions = False
    with pytest.raises(ValueError, match="one piece"):
        pool.run("b", [1, 2], [])


def test_commands_explain_themselves(tmp_path):
    for cmd in ([str(ROOT / "bin" / "trace_run"), "--help"], [sys.executable, "-m", "dejavu_b200", "generate", "--help"],
                [sys.executable, "-m", "dejavu_b200", "trace", "--help"]):
        r = subprocess.run(cmd, cwd=ROOT, capture_output=True, text=True)
        assert r.returncode == 0 and "--model" in r.stdout
    cfg, rank = H.CASES["odd"]
    H.save(tmp_path, cfg, H.weights(cfg, rank))
    r = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(tmp_path), "--dtype", "float16", "--out",
                        str(tmp_path), "--max-tokens", "8"], capture_output=True, text=True, stdin=subprocess.DEVNULL)
    assert r.returncode == 3


def test_kernels_check_their_arguments_on_the_host():
    import ctypes

    from dejavu_b200 import _lib, build

    build.build()
    lib = _lib.load_hybrid()
    before = lib.djv_launch_count()
    p = ctypes.c_void_p(0x1000)
    BF = _lib.DTYPE_BF16
    assert lib.djv_hyper_step(BF, p, p, p, None, None, None, None, p, 1e-5, None, None, None, 1, 9, 64, 0, None) == _lib.ERR_INVALID
    assert lib.djv_hyper_step(BF, p, None, None, None, None, None, None, p, 1e-5, None, None, None, 1, 2, 64, 0, None) == _lib.ERR_INVALID
    assert lib.djv_dense_gemv(0, 0, p, p, p, 1, 64, 8, 64, 0, 0.0, None) == _lib.ERR_INVALID
    assert lib.djv_dense_gemv(BF, BF, p, p, p, 33, 64, 8, 64, 0, 0.0, None) == _lib.ERR_INVALID
    assert lib.djv_dense_gemv(BF, BF, p, p, p, 1, 64, 7, 64, 6, 1.0, None) == _lib.ERR_INVALID
    assert lib.djv_window_attn(BF, p, p, 400, p, p, None, p, 1, 4, 5, 2, 32, 32, 8, 8, 1.0, None) == _lib.ERR_INVALID
    assert lib.djv_window_attn(BF, p, p, 100, p, p, None, p, 1, 4, 4, 2, 32, 32, 8, 8, 1.0, None) == _lib.ERR_INVALID
    assert lib.djv_gla_prefill(BF, p, p, 1000, p, p, 8, 0.1, p, 1e-5, 1.0, p, p, 1, 4, 2, 32, 32, p, 16, None) == _lib.ERR_SCRATCH
    assert lib.djv_gla_decode(BF, p, p, 10, p, p, 8, 0.1, p, 1e-5, 1.0, p, p, 1, 2, 32, 32, None) == _lib.ERR_INVALID
    assert lib.djv_launch_count() == before


# ---- the oracle ----------------------------------------------------------------------------------------------------

def test_oracle_attention_equals_a_dense_mask():
    g = torch.Generator().manual_seed(1)
    n, heads, kv, dk, dv, w = 23, 4, 2, 8, 6, 7
    q, k, v = (torch.randn(n, h, d, generator=g, dtype=torch.float64) for h, d in ((heads, dk), (kv, dk), (kv, dv)))
    sink = torch.randn(heads, generator=g, dtype=torch.float64)
    got = O.window_attention(q, k, v, 0.3, w, sink)
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    for h in range(heads):
        s = (q[:, h] @ k[:, h // 2].T * 0.3).masked_fill((j > i) | (i - j >= w), -math.inf)
        p = torch.softmax(torch.cat([s, sink[h].expand(n, 1)], 1), 1)[:, :n]
        assert torch.allclose(got[:, h], p @ v[:, h // 2])


def test_oracle_recurrence_equals_its_sum():
    g = torch.Generator().manual_seed(2)
    n, heads, dk, dv = 11, 2, 5, 4
    q, k, v = (torch.randn(n, heads, d, generator=g, dtype=torch.float64) for d in (dk, dk, dv))
    alpha = torch.rand(n, heads, dk, generator=g, dtype=torch.float64)
    got, S = O.gla_recurrence(q, k, v, alpha)
    for t in range(n):
        want = sum((q[t] * k[s] * alpha[s + 1:t + 1].prod(0)).sum(-1, keepdim=True) * v[s] for s in range(t + 1))
        assert torch.allclose(got[t], want)
    a, Sa = O.gla_recurrence(q[:4], k[:4], v[:4], alpha[:4])
    b, Sb = O.gla_recurrence(q[4:], k[4:], v[4:], alpha[4:], Sa)
    assert torch.allclose(torch.cat([a, b]), got) and torch.allclose(S, Sb)


def test_oracle_streams():
    x = torch.tensor([[[1.0, 2.0], [10.0, 20.0]]], dtype=torch.float64)
    y = torch.tensor([[100.0, 200.0]], dtype=torch.float64)
    mix = torch.tensor([[1.0, 2.0], [3.0, 4.0]], dtype=torch.float64)
    new = O.stream_update(x, y, mix, torch.tensor([0.5, 0.25], dtype=torch.float64))
    assert new.tolist() == [[[1 + 30 + 50.0, 2 + 60 + 100.0], [2 + 40 + 25.0, 4 + 80 + 50.0]]]
    assert O.stream_in(x, torch.tensor([2.0, -1.0], dtype=torch.float64)).tolist() == [[-8.0, -16.0]]


MISTAKES = {
    "window one longer": ("window_attention", lambda f: lambda q, k, v, s, w, z: f(q, k, v, s, w + 1, z)),
    "window one shorter": ("window_attention", lambda f: lambda q, k, v, s, w, z: f(q, k, v, s, w - 1, z)),
    "no sink": ("window_attention", lambda f: lambda q, k, v, s, w, z: f(q, k, v, s, w, None)),
    "no scaling of the positions": ("rotate", lambda f: lambda x, p, r: f(x, p, {**r, "scaling": None})),
    "positions one off": ("rotary_frequencies", lambda f: lambda r: ([v * 1.05 for v in f(r)[0]], f(r)[1])),
    "mix transposed": ("stream_update", lambda f: lambda x, y, m, o: f(x, y, m.T, o)),
    "decays of another temperature": ("gla_decay", lambda f: lambda h, a1, a2, b, tau, n: f(h, a1, a2, b, tau * 1.2, n)),
    "no clamp": ("clamped_glu", lambda f: lambda g, u, lim: f(g, u, 1e9)),
    "state lost once": ("gla_recurrence", lambda f: lambda q, k, v, a: (torch.cat([f(q[:20], k[:20], v[:20], a[:20])[0],
                                                                                   f(q[20:], k[20:], v[20:], a[20:])[0]]), None)),
    "loop run once": ("layer_order", lambda f: lambda cfg: f({**cfg, "loop": None})),
}


@pytest.mark.parametrize("name", MISTAKES)
def test_test_weights_show_mistakes(monkeypatch, name):
    """A model with one mistake planted in it differs by far more than the tolerances of the GPU tests."""
    cfg, rank = H.CASES["mixed"]
    W = H.weights(cfg, rank)
    ids = H.tokens(cfg, 40, 0)
    want = O.forward(cfg, W, ids)
    fn, wrong = MISTAKES[name]
    monkeypatch.setattr(O, fn, wrong(getattr(O, fn)))
    assert float(H.error(O.forward(cfg, W, ids), want).max()) > 0.03
