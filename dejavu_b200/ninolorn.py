"""Ninolorn: a decoder whose layers mix gated linear attention and sliding-window attention over hyper-connected
residual streams, with a range of layers that may run several times.

config.json keys: vocab, width, streams, norm.eps, logit_softcap, loop {start, stop, times}, layers[] with
  type 'gla':        mixer {heads, dim, vdim, tau}
  type 'attention':  mixer {heads, kv_heads, dim, vdim, scale, mask {size}, rot {base, dims, scaling}}
  mlp: null or {kind 'dense', ff, limit}
Tensors are named embed, head, final.norm and l<i>.{norm1, norm2, mix.*, mlp.*, hc1.*, hc2.*}.
"""
from __future__ import annotations

from types import SimpleNamespace
from typing import Optional

import torch
import torch.nn as nn

from . import _lib, ops
from .hybrid import HybridDecoder
from .mixers import GatedLinearAttention, GatedMLP, HyperConnection, WindowAttention, _empty

ARCHITECTURE = "Ninolorn"


def parse_config(raw: dict) -> SimpleNamespace:
    """config.json -> namespace, with what the code relies on checked."""
    loop = raw.get("loop") or {"start": 0, "stop": 0, "times": 1}
    cfg = SimpleNamespace(vocab_size=int(raw["vocab"]), hidden_size=int(raw["width"]), streams=int(raw["streams"]),
                          eps=float(raw["norm"]["eps"]), softcap=raw.get("logit_softcap"), layers=raw["layers"],
                          loop=(int(loop["start"]), int(loop["stop"]), int(loop["times"])))
    start, stop, times = cfg.loop
    if not (0 <= start <= stop <= len(cfg.layers) and times >= 1):
        raise ValueError(f"loop {cfg.loop} over {len(cfg.layers)} layers")
    for i, layer in enumerate(cfg.layers):
        if layer["type"] not in ("gla", "attention"):
            raise ValueError(f"layer {i}: unknown mixer {layer['type']!r}")
        mlp = layer.get("mlp")
        if mlp is not None and mlp["kind"] != "dense":
            raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
    return cfg


class HybridLayer(nn.Module):
    """A mixer and, unless the layer has none, a feed-forward, each behind its norm and its hyper-connection."""

    def __init__(self, cfg, spec: dict, rank: int, sink: bool, device=None, dtype=None):
        super().__init__()
        D, mx = cfg.hidden_size, spec["mixer"]
        if spec["type"] == "gla":
            self.mixer = GatedLinearAttention(D, mx["heads"], mx["dim"], mx["vdim"], rank, mx["tau"], cfg.eps, device,
                                              dtype)
        else:
            mask = mx.get("mask")
            self.mixer = WindowAttention(D, mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"], mx["scale"],
                                         None if mask is None else int(mask["size"]), mx.get("rot"), sink, device,
                                         dtype)
        self.norm1, self.hc1 = _empty(D, device=device, dtype=torch.float32), HyperConnection(cfg.streams, device)
        mlp = spec.get("mlp")
        self.mlp = None if mlp is None else GatedMLP(D, mlp["ff"], "clamped_glu", mlp["limit"], device, dtype)
        if self.mlp is not None:
            self.norm2, self.hc2 = _empty(D, device=device, dtype=torch.float32), HyperConnection(cfg.streams, device)

    def checkpoint_slots(self):
        """(tensor name below the layer, destination) of every tensor of the layer."""
        m = self.mixer
        if isinstance(m, GatedLinearAttention):
            parts = dict(zip(("q", "k", "v", "g", "a1"), m.proj.weight[:sum(m.sizes)].split(m.sizes)))
            parts.update({"a2": m.a2, "a2.b": m.a2_bias, "norm": m.norm})
        else:
            parts = dict(zip(("q", "k", "v"), m.qkv.weight.split(m.sizes)))
            if m.sink is not None:
                parts["sink"] = m.sink
        parts["o"] = m.o.weight
        out = {f"mix.{k}": v for k, v in parts.items()}
        if self.mlp is not None:
            out.update({f"mlp.{k}": v for k, v in self.mlp.checkpoint_slots().items()})
        for q in ("1", "2") if self.mlp is not None else ("1",):
            hc = getattr(self, "hc" + q)
            out.update({"norm" + q: getattr(self, "norm" + q), f"hc{q}.in": hc.w_in, f"hc{q}.out": hc.w_out,
                        f"hc{q}.mix": hc.mix})
        return out


class NinolornForCausalLM(HybridDecoder):
    """The residual is `streams` parallel streams; `collect` receives their sum."""

    def __init__(self, config: dict, tensor_shapes: Optional[dict] = None, gla_rank: int = 16, device=None,
                 dtype=torch.bfloat16):
        """`config` is the parsed config.json. The rank of the decay projection and the presence of sinks follow
        `tensor_shapes` (name -> shape) when given, else `gla_rank` and True."""
        cfg = parse_config(config)
        super().__init__(cfg, device, dtype)
        for i, spec in enumerate(cfg.layers):
            rank, sink = gla_rank, True
            if tensor_shapes is not None:
                rank = tensor_shapes.get(f"l{i}.mix.a1", (gla_rank,))[0]
                sink = f"l{i}.mix.sink" in tensor_shapes
            self.layers.append(HybridLayer(cfg, spec, rank, sink, device=device, dtype=dtype))
        start, stop, times = cfg.loop
        self.runs = [*range(start), *(list(range(start, stop)) * times), *range(stop, len(cfg.layers))]

    def init_constant(self, name: str):
        """Norms 1, streams that pass through (identity mix, mean in, unit out), mild decays."""
        leaf, S = name.rsplit(".", 1)[-1], self.config.streams
        if "norm" in leaf or leaf == "out":
            return 1.0
        if leaf == "in":
            return 1.0 / S
        if name.endswith((".hc1.mix", ".hc2.mix")):
            return torch.eye(S)
        return 1.0 if leaf in ("sink", "b") else None

    def hidden(self, ids, caches, pos, n, past, rows, collect):
        cfg, dev = self.config, ids.device
        S, eps = cfg.streams, cfg.eps
        first = {"ids": ids, "embed": self.embed, "streams": S}
        x = None  # the streams; while None they are all the embedding
        new_x = torch.empty(ids.numel(), S, cfg.hidden_size, dtype=torch.float32, device=dev)
        y, hc = None, None  # the last sublayer's output and its hyper-connection

        def boundary(w_in, gamma, rows=None, keep=True):
            """Streams after the last sublayer, and the normed input of the next one."""
            nonlocal x
            store = new_x if keep and y is not None else None
            h = ops.hyper_step(x, y, None if hc is None else hc.mix, None if hc is None else hc.w_out, w_in, gamma, eps,
                               self.dtype, x_out=store, rows=rows, **({} if x is not None else first))
            if store is not None:
                x = store
            return h

        for r, i in enumerate(self.runs):
            layer = self.layers[i]
            h = boundary(layer.hc1.w_in, layer.norm1)
            y, hc = layer.mixer(h, caches[r], pos, n, past), layer.hc1
            if layer.mlp is not None:
                h = boundary(layer.hc2.w_in, layer.norm2)
                y, hc = layer.mlp(h, n), layer.hc2
            if collect is not None:
                boundary(None, None)
                y = None
                collect.append(x.sum(dim=1))
        return boundary(None, self.final_norm, rows, keep=False)

    def head(self, h, decode: bool):
        cap = self.config.softcap
        if decode and h.shape[0] <= _lib.MAX_BATCH:
            return self.lm_head.decode(h, torch.float32, "softcap" if cap else "id", cap or 0.0)
        logits = self.lm_head(h, torch.float32)
        return ops.softcap_(logits, cap) if cap else logits
