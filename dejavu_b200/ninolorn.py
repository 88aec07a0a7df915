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

from . import ops
from .generation import GenerationMixin, InferenceParams
from .gpt import CausalLMOutput, _randn_big, _stable_hash
from .mixers import ClampedGatedMLP, GatedLinearAttention, HyperConnection, Linear, WindowAttention, _empty

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
        self.mlp = None if mlp is None else ClampedGatedMLP(D, mlp["ff"], mlp["limit"], device, dtype)
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
            gu = self.mlp.gate_up.weight.view(self.mlp.ff, 2, -1)
            out.update({"mlp.gate": gu[:, 0], "mlp.up": gu[:, 1], "mlp.down": self.mlp.down.weight})
        for q in ("1", "2") if self.mlp is not None else ("1",):
            hc = getattr(self, "hc" + q)
            out.update({"norm" + q: getattr(self, "norm" + q), f"hc{q}.in": hc.w_in, f"hc{q}.out": hc.w_out,
                        f"hc{q}.mix": hc.mix})
        return out


class NinolornForCausalLM(nn.Module, GenerationMixin):
    """Same calls as the other models: forward(input_ids, position_ids, inference_params).logits, generate(...)."""

    selects_logit_rows = True  # forward(logit_rows=...) computes logits at those tokens only
    takes_portions = True      # a prompt may arrive in portions of any size

    def __init__(self, config: dict, tensor_shapes: Optional[dict] = None, gla_rank: int = 16, device=None,
                 dtype=torch.bfloat16):
        """`config` is the parsed config.json. The rank of the decay projection and the presence of sinks follow
        `tensor_shapes` (name -> shape) when given, else `gla_rank` and True."""
        super().__init__()
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"this model runs in bfloat16 or float32, not {dtype}")
        self.config = cfg = parse_config(config)
        self.dtype = dtype
        f = {"device": device, "dtype": dtype}
        self.embed = _empty(cfg.vocab_size, cfg.hidden_size, **f)
        self.layers = nn.ModuleList()
        for i, spec in enumerate(cfg.layers):
            rank, sink = gla_rank, True
            if tensor_shapes is not None:
                rank = tensor_shapes.get(f"l{i}.mix.a1", (gla_rank,))[0]
                sink = f"l{i}.mix.sink" in tensor_shapes
            self.layers.append(HybridLayer(cfg, spec, rank, sink, **f))
        self.final_norm = _empty(cfg.hidden_size, device=device, dtype=torch.float32)
        self.lm_head = Linear(cfg.hidden_size, cfg.vocab_size, **f)
        start, stop, times = cfg.loop
        # layer number of every layer run; each run has a cache of its own
        self.runs = [*range(start), *(list(range(start, stop)) * times), *range(stop, len(cfg.layers))]
        # bf16 products accumulate in fp32 to the end, fp32 products are true fp32
        torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False
        if dtype == torch.float32:
            torch.backends.cuda.matmul.allow_tf32 = False

    # ---- weights ------------------------------------------------------------------------------------------
    def checkpoint_slots(self) -> dict:
        """Checkpoint tensor name -> the parameter (or slice of a fused one) that holds it."""
        out = {"embed": self.embed, "final.norm": self.final_norm, "head": self.lm_head.weight}
        for i, layer in enumerate(self.layers):
            out.update({f"l{i}.{k}": v for k, v in layer.checkpoint_slots().items()})
        return out

    def _zero_padding(self):
        for layer in self.layers:
            if isinstance(layer.mixer, GatedLinearAttention):
                layer.mixer.proj.weight[sum(layer.mixer.sizes):].zero_()

    @torch.no_grad()
    def load_tensors(self, tensors: dict):
        """Fills the model from checkpoint tensors; a missing, unknown or misshapen one is an error."""
        slots = self.checkpoint_slots()
        missing, unknown = sorted(set(slots) - set(tensors)), sorted(set(tensors) - set(slots))
        if missing or unknown:
            raise ValueError(f"checkpoint does not fit the configuration: missing {missing}, unknown {unknown}")
        for name, dst in slots.items():
            src = tensors[name]
            if tuple(src.shape) != tuple(dst.shape):
                raise ValueError(f"{name}: shape {tuple(src.shape)}, expected {tuple(dst.shape)}")
            dst.copy_(src)
        self._zero_padding()
        return self

    @torch.no_grad()
    def init_random(self, seed: int = 0, std: float = 0.02):
        """Random weights from seeds derived from tensor names: N(0, std) matrices, norms 1, streams that pass
        through (identity mix, mean in, unit out), mild decays."""
        gen = torch.Generator(device=self.embed.device)
        S = self.config.streams
        for name, dst in self.checkpoint_slots().items():
            leaf = name.rsplit(".", 1)[-1]
            if "norm" in leaf or leaf == "out":
                dst.fill_(1.0)
            elif leaf == "in":
                dst.fill_(1.0 / S)
            elif name.endswith((".hc1.mix", ".hc2.mix")):
                dst.copy_(torch.eye(S))
            elif leaf in ("sink", "b"):
                dst.fill_(1.0)
            else:
                gen.manual_seed((seed * 1000003 + _stable_hash(name)) % (2 ** 63))
                dst.copy_(_randn_big(tuple(dst.shape), gen, dst.device, std, dst.dtype))
        self._zero_padding()
        return self

    # ---- caches -------------------------------------------------------------------------------------------
    def allocate_cache(self, batch_size: int, max_seqlen: int, device) -> dict:
        """Per layer run: the window's K/V rings or the recurrent state. Nothing needs clearing between requests: a
        sequence that starts at position 0 reads neither."""
        return {r: self.layers[i].mixer.new_cache(batch_size, max_seqlen, device, self.dtype)
                for r, i in enumerate(self.runs)}

    def reset_decode_state(self, prompt_len: int, device, max_seqlen: int, batch: int = 1):
        """All decode state is in the caches and in the positions."""

    # ---- forward ------------------------------------------------------------------------------------------
    def forward(self, input_ids, position_ids=None, inference_params=None, logit_rows=None, collect=None):
        """input_ids (B, n): the next n tokens of every sequence; the caches of `inference_params` hold what came
        before. position_ids (B, n) or (B, 1): only the first column is read; without it the position is the caches'
        offset. logit_rows: places among the n tokens whose logits are wanted (default all). collect: a list that
        receives the sum of the streams after every layer run (for inspection). -> logits (B, len(logit_rows), vocab)
        fp32."""
        cfg = self.config
        B, n = input_ids.shape
        dev = input_ids.device
        if inference_params is None:
            inference_params = InferenceParams(max_sequence_len=n, max_batch_size=B,
                                               key_value_memory_dict=self.allocate_cache(B, n, dev))
        if position_ids is None:
            pos = torch.full((B,), inference_params.sequence_len_offset, dtype=torch.int64, device=dev)
        else:
            pos = position_ids[:, 0].contiguous()
        caches = inference_params.key_value_memory_dict
        ids = input_ids.reshape(-1).contiguous()
        S, eps = cfg.streams, cfg.eps
        first = {"ids": ids, "embed": self.embed, "streams": S}
        x = None  # the streams; while None they are all the embedding
        new_x = torch.empty(B * n, S, cfg.hidden_size, dtype=torch.float32, device=dev)
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
            y, hc = layer.mixer(h, caches[r], pos, n), layer.hc1
            if layer.mlp is not None:
                h = boundary(layer.hc2.w_in, layer.norm2)
                y, hc = layer.mlp(h, n), layer.hc2
            if collect is not None:
                boundary(None, None)
                y = None
                collect.append(x.sum(dim=1))
        if logit_rows is None or list(logit_rows) == list(range(n)):
            rows, R = None, n
        else:
            R = len(logit_rows)
            rows = torch.tensor([b * n + t for b in range(B) for t in logit_rows], dtype=torch.int32, device=dev)
        if R == 0:
            return CausalLMOutput(logits=torch.empty(B, 0, cfg.vocab_size, device=dev))
        h = boundary(None, self.final_norm, rows, keep=False)
        if n == 1 and B <= 32:
            logits = self.lm_head.decode(h, torch.float32, "softcap" if cfg.softcap else "id", cfg.softcap or 0.0)
        else:
            logits = self.lm_head(h, torch.float32)
            if cfg.softcap:
                ops.softcap_(logits, cfg.softcap)
        return CausalLMOutput(logits=logits.view(B, R, cfg.vocab_size))
