"""Small Tifosun configurations and random weights shared by its tests."""
import math

import torch


def memory(heads, dim, vdim, cap, mlp=None, kind="mlstm"):
    return {"type": kind, "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}


def latent(heads, dim, rot, vdim, rank, window, scale, base=2000.0, mlp=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": scale,
                      "mask": {"size": window}, "rot": {"base": base, "dims": rot}}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=None):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff},
            "shared": None if shared is None else {"ff": shared}}


def config(vocab, width, layers, eps=1e-5):
    return {"architecture": "Tifosun", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}}


CASES = {
    # every kind of layer, with each feed-forward and without one; head sizes that are and are not multiples of 16
    "mixed": config(203, 144, [memory(3, 40, 24, 7.0, dense(88)), latent(5, 24, 16, 40, 56, 19, 0.4, mlp=moe(6, 2, 32, 48)),
                               memory(2, 64, 96, 20.0, moe(5, 1, 40), kind="mlstm_2"), latent(2, 32, 8, 16, 24, 5, 0.3),
                               memory(1, 16, 16, 3.0)]),
    # no multiple of 8 anywhere
    "odd": config(97, 100, [memory(3, 18, 10, 5.0, moe(5, 3, 30, 14)), latent(3, 9, 6, 10, 21, 7, 0.5, base=50.0, mlp=dense(50))],
                  eps=1e-3),
    # head sizes of larger models, a window longer than one tile of the kernels, many experts
    "wide": config(130, 128, [memory(2, 128, 256, 12.5, moe(40, 4, 24)), latent(4, 128, 64, 128, 192, 150, 0.11, base=3e4, mlp=moe(16, 4, 64, 104)),
                              memory(3, 80, 136, 9.0, dense(72), kind="mlstm_2"), latent(18, 16, 32, 24, 128, 70, 0.2, mlp=None)], eps=1e-6),
}


def shapes(cfg):
    D = cfg["width"]
    out = {"embed": (cfg["vocab"], D), "final.norm": (D,), "head": (cfg["vocab"], D)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        H, dk, dv = m["heads"], m["dim"], m["vdim"]
        out.update({p + "mix.g": (H * dv, D), p + "mix.o": (D, H * dv)})
        if layer["type"] == "latent_attention":
            rank, rot = m["kv_rank"], m["rot_dim"]
            out.update({p + "mix.q": (H * (dk + rot), D), p + "mix.dkv": (rank + rot, D), p + "mix.dkv.norm": (rank,),
                        p + "mix.uk": (H * dk, rank), p + "mix.uv": (H * dv, rank)})
        else:
            out.update({p + "mix.q": (H * dk, D), p + "mix.k": (H * dk, D), p + "mix.v": (H * dv, D), p + "mix.norm": (H * dv,),
                        p + "mix.i": (H, D), p + "mix.i.b": (H,), p + "mix.f": (H, D), p + "mix.f.b": (H,)})
        mlp, norms = layer["mlp"], ["norm1", "norm1b"]
        if mlp:
            norms += ["norm2", "norm2b"]
            units = {"": mlp.get("ff")}
            if mlp["kind"] == "moe":
                out[p + "mlp.router"] = (mlp["router"]["experts"], D)
                units = {f"e{e}.": mlp["expert"]["ff"] for e in range(mlp["router"]["experts"])}
                if mlp["shared"]:
                    units["shared."] = mlp["shared"]["ff"]
            for u, ff in units.items():
                out.update({f"{p}mlp.{u}gate": (ff, D), f"{p}mlp.{u}up": (ff, D), f"{p}mlp.{u}down": (D, ff)})
        out.update({p + q: (D,) for q in norms})
    return out


def calm(cfg):
    """The same design without a choice between experts: with 16-bit activations a close call goes either way, and one
    token's other expert changes every later token."""
    def mlp(m):
        if not m or m["kind"] == "dense":
            return m
        n = min(m["router"]["experts"], 4)
        return {**m, "router": {"experts": n, "top": n}}

    return {**cfg, "layers": [{**layer, "mlp": mlp(layer["mlp"])} for layer in cfg["layers"]]}


def weights(cfg, seed=0, sharp=1.0):
    """bf16-representable random weights (kept in float64): matrices that keep activations near 1, peaked scores (less so
    with a smaller `sharp`), gates that open and close, memories that keep, a router whose scores are far apart."""
    g = torch.Generator().manual_seed(seed)
    W = {}
    for name, shape in shapes(cfg).items():
        t = torch.randn(shape, generator=g, dtype=torch.float64)
        leaf = name.rsplit(".", 1)[-1]
        if name.endswith(("mix.norm", "dkv.norm")):
            t = 1 + 0.3 * t
        elif "norm" in leaf:
            t = 0.3 * t
        elif leaf == "b":
            t = (1.5 if ".f." in name else -0.5) + t
        elif leaf in ("q", "k", "uk", "dkv", "gate", "up"):
            t = t * 1.8 * sharp / math.sqrt(shape[1])
        elif leaf in ("i", "f", "router"):
            t = t * 2.5 * sharp / math.sqrt(shape[1])
        elif leaf != "embed":
            t = t / math.sqrt(shape[1])
        W[name] = t.to(torch.bfloat16).double()
    return W
