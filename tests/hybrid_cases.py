"""Small Ninolorn configurations and random weights shared by the hybrid decoders' tests."""
import json
import math

import torch


def attention(heads, kv_heads, dim, vdim, window, dims=None, scaling=None, scale=None, base=1000.0, mlp=None):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
                      "scale": dim ** -0.5 if scale is None else scale, "mask": {"size": window},
                      "rot": {"base": base, "dims": dims or dim, "scaling": scaling}}}


def gla(heads, dim, vdim, tau, mlp=None):
    return {"type": "gla", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}}


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def config(vocab, width, streams, layers, loop=None, eps=1e-5, cap=9.0):
    return {"architecture": "Ninolorn", "vocab": vocab, "width": width, "streams": streams, "layers": layers,
            "loop": loop, "norm": {"eps": eps}, "logit_softcap": cap}


YARN = {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 0.5}

CASES = {
    # partial rotation, one kv head, a layer of each kind with and without a feed-forward, a loop over both kinds
    "mixed": (config(211, 176, 2, [attention(4, 1, 48, 32, 17, dims=32, scaling=YARN, scale=0.21, mlp=dense(120, 0.9)),
                                   gla(3, 40, 24, 8.0, mlp=dense(72, 2.5)),
                                   attention(2, 2, 64, 96, 5, scaling={**YARN, "factor": 1.5}),
                                   gla(2, 16, 48, 2.0)],
                     loop={"start": 1, "stop": 3, "times": 2}), 9),
    # no multiple of 8 anywhere, one stream, decays that forget within a token
    "odd": (config(97, 100, 1, [gla(2, 20, 36, 1.0, mlp=dense(50, 1.1)), attention(3, 3, 18, 10, 3, dims=6)], eps=1e-3,
                   cap=4.0), 3),
    # many query heads per kv head, a window longer than one tile of the decode kernel, five streams
    "wide": (config(130, 128, 5, [attention(8, 1, 128, 64, 150, dims=64, scaling=YARN, mlp=dense(64, 0.7)),
                                  gla(2, 64, 128, 16.0),
                                  attention(12, 2, 32, 32, 64, scale=0.3)],
                    loop={"start": 0, "stop": 1, "times": 3}), 16),
}


def shapes(cfg, rank):
    D, S = cfg["width"], cfg["streams"]
    out = {"embed": (cfg["vocab"], D), "final.norm": (D,), "head": (cfg["vocab"], D)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        H, dk, dv = m["heads"], m["dim"], m["vdim"]
        G = m.get("kv_heads", H)
        out.update({p + "mix.q": (H * dk, D), p + "mix.k": (G * dk, D), p + "mix.v": (G * dv, D), p + "mix.o": (D, H * dv)})
        if layer["type"] == "gla":
            out.update({p + "mix.g": (H * dv, D), p + "mix.norm": (dv,), p + "mix.a1": (rank, D),
                        p + "mix.a2": (H * dk, rank), p + "mix.a2.b": (H * dk,)})
        else:
            out[p + "mix.sink"] = (H,)
        subs = "1"
        if layer["mlp"]:
            ff = layer["mlp"]["ff"]
            out.update({p + "mlp.gate": (ff, D), p + "mlp.up": (ff, D), p + "mlp.down": (D, ff)})
            subs = "12"
        for q in subs:
            out.update({f"{p}norm{q}": (D,), f"{p}hc{q}.in": (S,), f"{p}hc{q}.out": (S,), f"{p}hc{q}.mix": (S, S)})
    return out


def weights(cfg, rank, seed=0):
    """bf16-representable random weights (kept in float64): matrices that keep activations near 1, norms around 1, mixes
    near a permuted identity so that the streams differ and [from, to] is not symmetric, sinks that matter."""
    g = torch.Generator().manual_seed(seed)
    W = {}
    for name, shape in shapes(cfg, rank).items():
        t = torch.randn(shape, generator=g, dtype=torch.float64)
        leaf = name.rsplit(".", 1)[-1]
        if leaf == "embed" or len(shape) == 1 and "norm" in leaf:
            t = t if leaf == "embed" else 1 + 0.3 * t
        elif leaf in ("in", "out"):
            t = (1.0 / cfg["streams"] if leaf == "in" else 1.0) * (1 + 0.4 * t)
        elif leaf == "mix":
            t = torch.eye(cfg["streams"], dtype=torch.float64) + 0.3 * t
        elif leaf == "sink":
            t = 1.0 + t
        elif leaf == "b":
            t = 1.5 * t
        elif leaf in ("q", "k"):
            t = t * 1.6 / math.sqrt(shape[1])  # peaked scores
        elif leaf in ("gate", "up"):
            t = t * 2.0 / math.sqrt(shape[1])  # both sides of the clamp
        else:
            t = t / math.sqrt(shape[1])
        W[name] = t.to(torch.bfloat16).double()
    return W


def save(folder, cfg, W):
    """config.json + model.safetensors (bf16) of a model."""
    (folder / "config.json").write_text(json.dumps(cfg))
    header, blobs, at = {}, [], 0
    for name, t in W.items():
        b = t.to(torch.bfloat16).contiguous().view(torch.uint8).numpy().tobytes()
        header[name] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [at, at + len(b)]}
        blobs.append(b)
        at += len(b)
    h = json.dumps(header).encode()
    (folder / "model.safetensors").write_bytes(len(h).to_bytes(8, "little") + h + b"".join(blobs))


def tokens(cfg, n, seed):
    g = torch.Generator().manual_seed(1000 + seed)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()


def error(got, want):
    """Root-mean-square difference of each row's logits (their mean taken off) over the scale of all rows."""
    got, want = got.double().cpu(), want.double()
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    return (d.pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt())
