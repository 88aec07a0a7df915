"""Tifosun: a decoder whose layers mix matrix memories (mLSTM) and windowed latent attention, with a norm before and after
every sublayer and dense or routed feed-forwards.

config.json keys: vocab, width, norm.eps, layers[] with
  type 'mlstm', 'mlstm_2':    mixer {heads, dim, vdim, gate_cap}
  type 'latent_attention':    mixer {heads, dim, rot_dim, vdim, kv_rank, scale, mask {size}, rot {base, dims}}
  mlp: null, {kind 'dense', ff} or {kind 'moe', router {experts, top}, expert {ff}, shared {ff} or null}
Tensors are named embed, head, final.norm and l<i>.{norm1, norm1b, norm2, norm2b, mix.*, mlp.*}.
"""
from __future__ import annotations

from types import SimpleNamespace

import torch
import torch.nn as nn

from . import _lib, ops
from .hybrid import HybridDecoder
from .mixers import GatedMLP, LatentAttention, MatrixMemory, MixtureOfExperts, SplitSum, _empty

ARCHITECTURE = "Tifosun"
MEMORIES = ("mlstm", "mlstm_2")


def parse_config(raw: dict) -> SimpleNamespace:
    """config.json -> namespace, with what the code relies on checked."""
    cfg = SimpleNamespace(vocab_size=int(raw["vocab"]), hidden_size=int(raw["width"]), eps=float(raw["norm"]["eps"]),
                          layers=raw["layers"])
    for i, layer in enumerate(cfg.layers):
        if layer["type"] not in (*MEMORIES, "latent_attention"):
            raise ValueError(f"layer {i}: unknown mixer {layer['type']!r}")
        mlp = layer.get("mlp")
        if mlp is not None and mlp["kind"] not in ("dense", "moe"):
            raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
    return cfg


class TifosunLayer(nn.Module):
    """A mixer and, unless the layer has none, a feed-forward, each between two norms (weights stored around zero)."""

    def __init__(self, cfg, spec: dict, device=None, dtype=None):
        super().__init__()
        D, mx, f = cfg.hidden_size, spec["mixer"], {"device": device, "dtype": dtype}
        if spec["type"] in MEMORIES:
            self.mixer = MatrixMemory(D, mx["heads"], mx["dim"], mx["vdim"], mx["gate_cap"], cfg.eps, **f)
        else:
            mask = mx.get("mask")
            self.mixer = LatentAttention(D, mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"], mx["kv_rank"], mx["scale"],
                                         None if mask is None else int(mask["size"]), mx["rot"], cfg.eps, **f)
        mlp = spec.get("mlp")
        if mlp is None:
            self.mlp = None
        elif mlp["kind"] == "dense":
            self.mlp = GatedMLP(D, mlp["ff"], "silu_glu", **f)
        else:
            shared = mlp.get("shared")
            self.mlp = MixtureOfExperts(D, mlp["expert"]["ff"], mlp["router"]["experts"], mlp["router"]["top"],
                                        shared["ff"] if shared else None, **f)
        for q in ("norm1", "norm1b") + (("norm2", "norm2b") if self.mlp is not None else ()):
            setattr(self, q, _empty(D, device=device, dtype=torch.float32))

    def checkpoint_slots(self):
        """(tensor name below the layer, destination) of every tensor of the layer."""
        out = {f"mix.{k}": v for k, v in self.mixer.checkpoint_slots().items()}
        out.update({"norm1": self.norm1, "norm1b": self.norm1b})
        if self.mlp is not None:
            out.update({f"mlp.{k}": v for k, v in self.mlp.checkpoint_slots().items()})
            out.update({"norm2": self.norm2, "norm2b": self.norm2b})
        return out


class TifosunForCausalLM(HybridDecoder):
    load_kernels = staticmethod(_lib.load_routed)

    def __init__(self, config: dict, device=None, dtype=torch.bfloat16):
        """`config` is the parsed config.json."""
        cfg = parse_config(config)
        super().__init__(cfg, device, dtype)
        self.layers.extend(TifosunLayer(cfg, spec, device, dtype) for spec in cfg.layers)
        self.runs = list(range(len(cfg.layers)))

    def init_constant(self, name: str):
        """Norms 1 (stored as 0 where the weight is a distance from 1), neutral input gates, forget gates that keep."""
        if name.endswith(("mix.norm", "dkv.norm")):
            return 1.0
        if "norm" in name.rsplit(".", 1)[-1] or name.endswith(".i.b"):
            return 0.0
        return 3.0 if name.endswith(".f.b") else None

    def hidden(self, ids, caches, pos, n, past, rows, collect):
        eps = self.config.eps
        first = {"ids": ids, "embed": self.embed}
        x = None  # the residual; while None it is the embedding
        new_x = torch.empty(ids.numel(), self.config.hidden_size, dtype=torch.float32, device=ids.device)
        out, post = None, None  # the last sublayer's output and the weight of its norm

        def boundary(gamma, rows=None, keep=True):
            """The residual after the last sublayer, and the normed input of the next one."""
            nonlocal x
            y, parts, places = out if isinstance(out, SplitSum) else (out, None, None)
            store = new_x if keep and out is not None else None
            h = ops.residual_step(x, y, post, gamma, eps, self.dtype, base=1.0, x_out=store, parts=parts, part_rows=places,
                                  rows=rows, **({} if x is not None else first))
            if store is not None:
                x = store
            return h

        for r, i in enumerate(self.runs):
            layer = self.layers[i]
            out, post = layer.mixer(boundary(layer.norm1), caches[r], pos, n, past), layer.norm1b
            if layer.mlp is not None:
                out, post = layer.mlp(boundary(layer.norm2), n), layer.norm2b
            if collect is not None:
                boundary(None)
                out, post = None, None
                collect.append(x.clone())
        return boundary(self.final_norm, rows, keep=False)
