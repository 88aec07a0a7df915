"""Building blocks of hybrid decoders: linear layers, rotary positions, sliding-window attention with sinks, gated
linear attention, clamped gated MLP, hyper-connected residual streams. bf16 (activations and products, fp32 where a
comment says so) or fp32 throughout.

Each block takes its sizes and constants as arguments and works on rows (B * n, features), B sequences of n new tokens
each, with their first positions in a device tensor `pos` (B,). n == 1 is a decode step and runs the fused decode
kernels; larger n is a portion of a prompt. A mixer owns no state: `new_cache` says what a sequence needs, the forward
call gets it back.
"""
from __future__ import annotations

import math
from typing import Optional

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

    def forward(self, h, cache, pos, n: int):
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

    def new_cache(self, batch: int, max_seqlen: int, device, dtype):
        """The recurrent state, fp32, whatever the model's type."""
        return (torch.zeros(batch, self.heads, self.dim, self.vdim, device=device, dtype=torch.float32),)

    def forward(self, h, cache, pos, n: int):
        proj = self.proj.rows(h, n == 1)
        ctx = ops.gated_linear_attention(proj, self.a2, self.a2_bias, self.tau, self.norm, self.eps, self.scale,
                                         cache[0], pos, n)
        return self.o.rows(ctx, n == 1, torch.float32)


class ClampedGatedMLP(nn.Module):
    """down(min(gate, limit) * sigmoid(1.702 .) * (clamp(up, limit) + 1)); gate and up rows are interleaved in one
    weight, so that a decode row's two products meet in one warp."""

    def __init__(self, width: int, ff: int, limit: float, device=None, dtype=None):
        super().__init__()
        self.ff, self.limit = ff, float(limit)
        self.gate_up = Linear(width, 2 * ff, device, dtype)
        self.down = Linear(ff, width, device, dtype)

    def forward(self, h, n: int):
        if n == 1 and h.shape[0] <= _lib.MAX_BATCH:
            a = self.gate_up.decode(h, activation="clamped_glu", param=self.limit)
        else:
            a = ops.clamped_glu(self.gate_up(h), self.limit)
        return self.down.rows(a, n == 1, torch.float32)


class HyperConnection(nn.Module):
    """Coefficients of one sublayer over S residual streams: `w_in` (S) mixes them into the sublayer's input, `mix`
    (S from, S to) and `w_out` (S) make the new streams from the old ones and the output. The arithmetic (fp32) is one
    kernel per boundary, shared with the norm of the sublayer that follows: ops.hyper_step."""

    def __init__(self, streams: int, device=None):
        super().__init__()
        f32 = {"device": device, "dtype": torch.float32}
        self.w_in, self.w_out, self.mix = _empty(streams, **f32), _empty(streams, **f32), _empty(streams, streams, **f32)
