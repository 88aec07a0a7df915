"""Building blocks of hybrid decoders: linear layers, rotary positions, sliding-window attention with sinks, windowed
latent attention, gated linear attention, matrix memories (mLSTM), gated MLPs, mixtures of experts, hyper-connected
residual streams. bf16 (activations and products, fp32 where a comment says so) or fp32 throughout.

Each block takes its sizes and constants as arguments and works on rows (B * n, features), B sequences of n new tokens
each, with their first positions in a device tensor `pos` (B,). n == 1 is a decode step and runs the fused decode
kernels; larger n is a portion of a prompt. A mixer owns no state: `new_cache` says what a sequence needs, the forward
call gets it back. `past`, where a mixer takes it, is a bound the host knows on every sequence's position.
"""
from __future__ import annotations

import math
from typing import NamedTuple, Optional

import torch
import torch.nn as nn

from . import _lib, ops


def _empty(*shape, device=None, dtype=None):
    return nn.Parameter(torch.empty(*shape, device=device, dtype=dtype), requires_grad=False)


class Linear(nn.Module):
    """Weight (out, in). Decode rows go through the library's GEMV kernels, with an epilogue where the caller asks for
    one; longer inputs through the vendor's matrix product (bf16 products accumulate and, where asked, return fp32)."""

    def __init__(self, in_features: int, out_features: int, device=None, dtype=None):
        super().__init__()
        self.weight = _empty(out_features, in_features, device=device, dtype=dtype)

    def decode(self, x, out_dtype=None, activation="id", param=0.0):
        return ops.linear_gemv(x, self.weight, out_dtype, activation, param)

    def forward(self, x, out_dtype=None):
        if out_dtype in (None, x.dtype):
            return torch.mm(x, self.weight.t())
        return torch.mm(x, self.weight.t(), out_dtype=out_dtype)

    def part(self, x, first: int, last: int, out_dtype=None):
        """Rows first .. last - 1 of the weight only."""
        w = self.weight[first:last].t()
        return torch.mm(x, w) if out_dtype in (None, x.dtype) else torch.mm(x, w, out_dtype=out_dtype)

    def rows(self, x, decode: bool, out_dtype=None):
        if decode and x.shape[0] <= _lib.MAX_BATCH:
            return self.decode(x, out_dtype)
        return self(x, out_dtype)


class RotaryTable(nn.Module):
    """Frequencies of the rotated pairs and the factor on cos and sin. `rot` has 'base', 'dims' and optionally
    'scaling' (YaRN: factor, original, fast, slow): frequencies of pairs that turn less than `slow` times within the
    original length are divided by the factor, those that turn more than `fast` times are kept, with a linear ramp over
    the pair number between the two."""

    def __init__(self, rot: dict, device=None):
        super().__init__()
        dims, base = int(rot["dims"]), float(rot["base"])
        if dims < 2 or dims % 2:
            raise ValueError(f"rotary dims must be even and positive, got {dims}")
        self.dims = dims
        freqs = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
        self.amp = 1.0
        scaling = rot.get("scaling")
        if scaling:
            factor, original = float(scaling["factor"]), float(scaling["original"])

            def pair_at(turns):
                return dims * math.log(original / (turns * 2 * math.pi)) / (2 * math.log(base))

            first = max(math.floor(pair_at(float(scaling["fast"]))), 0)
            last = min(math.ceil(pair_at(float(scaling["slow"]))), dims - 1)
            width = max(last - first, 0.001)
            for i, f in enumerate(freqs):
                ramp = min(1.0, max(0.0, (i - first) / width))
                freqs[i] = f / factor * ramp + f * (1.0 - ramp)
            self.amp = 0.1 * math.log(factor) + 1.0
        self.register_buffer("freqs", torch.tensor(freqs, dtype=torch.float32, device=device), persistent=False)


class WindowAttention(nn.Module):
    """Causal attention over the last `window` tokens (None: all) with grouped key/value heads, rotary positions and an
    optional learned sink per head. Scores, softmax and the sink are fp32."""

    def __init__(self, width: int, heads: int, kv_heads: int, dim: int, vdim: int, scale: float,
                 window: Optional[int] = None, rot: Optional[dict] = None, sink: bool = True, device=None, dtype=None):
        super().__init__()
        if heads % kv_heads:
            raise ValueError(f"{heads} query heads over {kv_heads} key/value heads")
        self.heads, self.kv_heads, self.dim, self.vdim = heads, kv_heads, dim, vdim
        self.scale, self.window = float(scale), window
        self.sizes = (heads * dim, kv_heads * dim, kv_heads * vdim)  # rows of q, k, v in the fused weight
        self.qkv = Linear(width, sum(self.sizes), device, dtype)
        self.o = Linear(heads * vdim, width, device, dtype)
        self.sink = _empty(heads, device=device, dtype=torch.float32) if sink else None
        self.rotary = RotaryTable(rot, device) if rot else None
        if self.rotary is not None and self.rotary.dims > dim:
            raise ValueError(f"{self.rotary.dims} rotary dims in heads of {dim}")

    def new_cache(self, batch: int, max_seqlen: int, device, dtype):
        """Rings of the window's length: (K, V), (batch, kv_heads, tokens, dim)."""
        cap = max_seqlen if self.window is None else min(self.window, max_seqlen)
        return (torch.zeros(batch, self.kv_heads, cap, self.dim, device=device, dtype=dtype),
                torch.zeros(batch, self.kv_heads, cap, self.vdim, device=device, dtype=dtype))

    def forward(self, h, cache, pos, n: int, past: int = 0):
        k_ring, v_ring = cache
        qkv = self.qkv.rows(h, n == 1)
        rot = self.rotary
        window = self.window if self.window is not None else 2 ** 30
        if n == 1:
            ctx = ops.window_attention_decode(qkv, k_ring, v_ring, self.sink, None if rot is None else rot.freqs,
                                              1.0 if rot is None else rot.amp, pos, self.heads, window, self.scale)
        else:
            if rot is not None:
                ops.rotary_(qkv, rot.freqs, rot.amp, pos, n, self.heads + self.kv_heads, self.dim)
            ctx = ops.window_attention(qkv, k_ring, v_ring, self.sink, pos, n, self.heads, window, self.scale)
        return self.o.rows(ctx, n == 1, torch.float32)


class GatedLinearAttention(nn.Module):
    """Linear attention with a decay per key channel from a low-rank projection, per-head RMS norm and a silu gate. The
    state, the decays and everything they are made of besides the projections are fp32."""

    def __init__(self, width: int, heads: int, dim: int, vdim: int, rank: int, tau: float, eps: float, device=None,
                 dtype=None):
        super().__init__()
        self.heads, self.dim, self.vdim, self.rank = heads, dim, vdim, rank
        self.tau, self.eps = float(tau), float(eps)
        self.scale = dim ** -0.5
        self.sizes = (heads * dim, heads * dim, heads * vdim, heads * vdim, rank)  # q, k, v, gate, decay input
        # rows are padded so that every row of the product starts on a 16-byte boundary
        self.proj = Linear(width, -(-sum(self.sizes) // 8) * 8, device, dtype)
        self.a2 = _empty(heads * dim, rank, device=device, dtype=torch.float32)
        self.a2_bias = _empty(heads * dim, device=device, dtype=torch.float32)
        self.norm = _empty(vdim, device=device, dtype=torch.float32)
        self.o = Linear(heads * vdim, width, device, dtype)

    def zero_padding(self):
        self.proj.weight[sum(self.sizes):].zero_()

    def new_cache(self, batch: int, max_seqlen: int, device, dtype):
        """The recurrent state, fp32, whatever the model's type."""
        return (torch.zeros(batch, self.heads, self.dim, self.vdim, device=device, dtype=torch.float32),)

    def forward(self, h, cache, pos, n: int, past: int = 0):
        proj = self.proj.rows(h, n == 1)
        ctx = ops.gated_linear_attention(proj, self.a2, self.a2_bias, self.tau, self.norm, self.eps, self.scale,
                                         cache[0], pos, n)
        return self.o.rows(ctx, n == 1, torch.float32)


class MatrixMemory(nn.Module):
    """mLSTM: a (dim, vdim) state per head with scalar exponential gates, kept in range by a running maximum, a normaliser
    beside it, per-head RMS norm and a sigmoid gate. The state, the gates (from their projections on) and everything made
    of them are fp32."""

    def __init__(self, width: int, heads: int, dim: int, vdim: int, gate_cap: float, eps: float, device=None, dtype=None):
        super().__init__()
        self.heads, self.dim, self.vdim = heads, dim, vdim
        self.gate_cap, self.eps, self.scale = float(gate_cap), float(eps), dim ** -0.5
        self.sizes = (heads * dim, heads * dim, heads * vdim, heads * vdim)  # q, k, v, output gate
        # rows are padded so that every row of the product starts on a 16-byte boundary; the gates' rows come after them
        self.main = -(-sum(self.sizes) // 8) * 8
        self.proj = Linear(width, self.main + 2 * heads, device, dtype)
        f32 = {"device": device, "dtype": torch.float32}
        self.i_bias, self.f_bias, self.norm = _empty(heads, **f32), _empty(heads, **f32), _empty(heads * vdim, **f32)
        self.o = Linear(heads * vdim, width, device, dtype)

    def zero_padding(self):
        self.proj.weight[sum(self.sizes):self.main].zero_()

    def checkpoint_slots(self):
        w, m, H = self.proj.weight, self.main, self.heads
        return {**dict(zip("qkvg", w[:sum(self.sizes)].split(self.sizes))), "i": w[m:m + H], "f": w[m + H:],
                "i.b": self.i_bias, "f.b": self.f_bias, "norm": self.norm, "o": self.o.weight}

    def new_cache(self, batch: int, max_seqlen: int, device, dtype):
        """The recurrent state, fp32, whatever the model's type."""
        return (ops.mlstm_state(batch, self.heads, self.dim, self.vdim, device),)

    def forward(self, h, cache, pos, n: int, past: int = 0):
        if n == 1:  # one product for all projections, in fp32
            proj = self.proj.rows(h, True, torch.float32)
            gates = proj[:, self.main:]
        else:
            proj = self.proj.part(h, 0, self.main)
            gates = self.proj.part(h, self.main, self.main + 2 * self.heads, torch.float32)
        ctx = ops.mlstm(proj, gates, self.i_bias, self.f_bias, self.gate_cap, self.norm, self.eps, self.scale, cache[0],
                        pos, n, self.dim, self.vdim, h.dtype)
        return self.o.rows(ctx, n == 1, torch.float32)


class LatentAttention(nn.Module):
    """Causal attention over the last `window` tokens (None: all) whose keys and values are projections of one latent per
    token, with a rotated key part that all heads share and a sigmoid gate on the output. Only latents and rotated parts
    are cached. A prompt portion expands the latents in sight into keys and values; a decode step works on the latents
    themselves. Scores and softmax are fp32."""

    def __init__(self, width: int, heads: int, dim: int, rot_dim: int, vdim: int, rank: int, scale: float,
                 window: Optional[int], rot: dict, eps: float, device=None, dtype=None):
        super().__init__()
        self.heads, self.dim, self.rot_dim, self.vdim, self.rank = heads, dim, rot_dim, vdim, rank
        self.scale, self.window, self.eps = float(scale), window, float(eps)
        self.sizes = (heads * (dim + rot_dim), rank + rot_dim, heads * vdim)  # q, latent and key part, output gate
        self.proj = Linear(width, -(-sum(self.sizes) // 8) * 8, device, dtype)
        self.norm = _empty(rank, device=device, dtype=torch.float32)
        self.ukv = Linear(rank, heads * (dim + vdim), device, dtype)
        self.o = Linear(heads * vdim, width, device, dtype)
        self.rotary = RotaryTable(rot, device)
        if self.rotary.dims != rot_dim:
            raise ValueError(f"{self.rotary.dims} rotary dims in a rotated part of {rot_dim}")

    def zero_padding(self):
        self.proj.weight[sum(self.sizes):].zero_()

    def checkpoint_slots(self):
        q, d, g = self.proj.weight[:sum(self.sizes)].split(self.sizes)
        uk, uv = self.ukv.weight.split((self.heads * self.dim, self.heads * self.vdim))
        return {"q": q, "dkv": d, "g": g, "dkv.norm": self.norm, "uk": uk, "uv": uv, "o": self.o.weight}

    def new_cache(self, batch: int, max_seqlen: int, device, dtype):
        """A ring of the window's length: (batch, tokens, latent | rotated key part)."""
        cap = max_seqlen if self.window is None else min(self.window, max_seqlen)
        return (torch.zeros(batch, cap, self.rank + self.rot_dim, device=device, dtype=dtype),)

    def forward(self, h, cache, pos, n: int, past: int = 0):
        ring, = cache
        H, dim, rot, rank = self.heads, self.dim, self.rot_dim, self.rank
        window = self.window if self.window is not None else 2 ** 30
        proj = self.proj.rows(h, n == 1)
        a, b = self.sizes[0], self.sizes[0] + self.sizes[1]
        gate = proj[:, b:b + self.sizes[2]]
        if n == 1:
            uk, uv = self.ukv.weight[:H * dim], self.ukv.weight[H * dim:]
            ctx = ops.latent_attention_decode(proj, uk, uv, self.norm, self.eps, self.rotary.freqs, ring, gate, pos, H,
                                              window, self.scale)
            return self.o.rows(ctx, True, torch.float32)
        past = min(past, window - 1, ring.shape[1])
        ops.rotary_(proj[:, dim:], self.rotary.freqs, self.rotary.amp, pos, n, H, dim + rot, interleaved=True)
        rows = ops.latent_rows(proj[:, a:b], ring, self.norm, self.eps, self.rotary.freqs, pos, n, past, rank, store=past == 0)
        kv = self.ukv(rows[:, :rank])
        ctx = ops.latent_attention(proj[:, :a], kv, rows[:, rank:], gate, pos, n, past, H, dim, rot, window, self.scale)
        if past:
            ops.latent_store(rows, ring, self.norm, self.rotary.freqs, pos, n, past, rank)
        return self.o(ctx, torch.float32)


class GatedMLP(nn.Module):
    """down(unit(gate, up)); the unit is "silu_glu" (silu(gate) * up) or "clamped_glu" (min(gate, limit) * sigmoid(1.702 .) *
    (clamp(up, limit) + 1)). Gate and up rows are interleaved in one weight, so that a decode row's two products meet in one
    warp."""

    def __init__(self, width: int, ff: int, activation: str, limit: float = 0.0, device=None, dtype=None):
        super().__init__()
        self.ff, self.activation, self.limit = ff, activation, float(limit)
        self.gate_up = Linear(width, 2 * ff, device, dtype)
        self.down = Linear(ff, width, device, dtype)

    def checkpoint_slots(self):
        gu = self.gate_up.weight.view(self.ff, 2, -1)
        return {"gate": gu[:, 0], "up": gu[:, 1], "down": self.down.weight}

    def forward(self, h, n: int):
        if n == 1 and h.shape[0] <= _lib.MAX_BATCH:
            a = self.gate_up.decode(h, activation=self.activation, param=self.limit)
        else:
            a = ops.glu(self.gate_up(h), self.activation, self.limit)
        return self.down.rows(a, n == 1, torch.float32)


class SplitSum(NamedTuple):
    """A sublayer's output that the next boundary adds up: y (rows, width) fp32 or None, plus, for every row, the rows
    `places` (rows, k) of `parts`."""

    y: Optional[torch.Tensor]
    parts: torch.Tensor
    places: torch.Tensor


class MixtureOfExperts(nn.Module):
    """Every token goes through the `top` experts (silu gated units) with the largest scores sigmoid(router logits); the
    scores multiply the experts' inputs and are not renormalised. A shared expert of its own size, if any, takes every
    token. Router logits and scores are fp32.

    A prompt portion is sorted by expert and runs as grouped products (SplitSum); a decode step reads the chosen experts'
    weights only."""

    def __init__(self, width: int, ff: int, experts: int, top: int, shared_ff: Optional[int] = None, device=None, dtype=None):
        super().__init__()
        if not 1 <= top <= experts:
            raise ValueError(f"{top} of {experts} experts")
        self.ff, self.experts, self.top = ff, experts, top
        self.router = Linear(width, experts, device, dtype)
        self.gate_up = _empty(experts, 2 * ff, width, device=device, dtype=dtype)
        self.down = _empty(experts, width, ff, device=device, dtype=dtype)
        self.shared = GatedMLP(width, shared_ff, "silu_glu", device=device, dtype=dtype) if shared_ff else None

    def checkpoint_slots(self):
        out = {"router": self.router.weight}
        gu = self.gate_up.view(self.experts, self.ff, 2, -1)
        for e in range(self.experts):
            out.update({f"e{e}.gate": gu[e, :, 0], f"e{e}.up": gu[e, :, 1], f"e{e}.down": self.down[e]})
        if self.shared is not None:
            out.update({f"shared.{k}": v for k, v in self.shared.checkpoint_slots().items()})
        return out

    def forward(self, h, n: int):
        z = self.router.rows(h, n == 1, torch.float32)
        if n == 1 and h.shape[0] <= _lib.MAX_BATCH:
            if self.shared is None:
                return ops.moe_decode(h, z, self.gate_up, self.down, self.top)
            return ops.moe_decode(h, z, self.gate_up, self.down, self.top, self.shared.gate_up.weight, self.shared.down.weight)
        xs, ws, offsets, places = ops.moe_route(h, z, self.top)
        a = ops.moe_grouped(xs, self.gate_up, offsets, ws, glu=True)
        return SplitSum(None if self.shared is None else self.shared(h, n), ops.moe_grouped(a, self.down, offsets), places)


class HyperConnection(nn.Module):
    """Coefficients of one sublayer over S residual streams: `w_in` (S) mixes them into the sublayer's input, `mix`
    (S from, S to) and `w_out` (S) make the new streams from the old ones and the output. The arithmetic (fp32) is one
    kernel per boundary, shared with the norm of the sublayer that follows: ops.hyper_step."""

    def __init__(self, streams: int, device=None):
        super().__init__()
        f32 = {"device": device, "dtype": torch.float32}
        self.w_in, self.w_out, self.mix = _empty(streams, **f32), _empty(streams, **f32), _empty(streams, streams, **f32)
