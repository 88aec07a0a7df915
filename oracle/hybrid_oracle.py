"""Plain, slow CPU implementation of the Ninolorn decoder: gated linear attention and sliding-window attention
layers over hyper-connected residual streams. One function per mechanism, written token by token where the
mechanism is a recurrence; test infrastructure only, it shares no code with the package.

`cfg` is the parsed config.json, `W` a dict name -> tensor with the checkpoint's tensor names. The arithmetic runs in
the dtype of the tensors given (double for the tightest comparison).
"""
from __future__ import annotations

import math

import torch


# ---- small mechanisms ---------------------------------------------------------------------------------------

def rms_norm(x, w, eps):
    """x / sqrt(mean(x^2) + eps) * w over the last dimension."""
    ms = (x * x).mean(dim=-1, keepdim=True)
    return x / torch.sqrt(ms + eps) * w


def silu(x):
    return x / (1 + torch.exp(-x))


def clamped_glu(gate, up, limit):
    """Gate cut from above, up cut on both sides; g * sigmoid(1.702 g) * (u + 1)."""
    g = torch.minimum(gate, torch.full_like(gate, limit))
    u = torch.maximum(torch.minimum(up, torch.full_like(up, limit)), torch.full_like(up, -limit))
    return g / (1 + torch.exp(-1.702 * g)) * (u + 1)


def softcap(x, cap):
    return cap * torch.tanh(x / cap)


def stream_in(x, w_in):
    """Hyper-connection input: x (n, s, d), w_in (s,) -> (n, d)."""
    n, s, d = x.shape
    u = torch.zeros(n, d, dtype=x.dtype)
    for j in range(s):
        u = u + w_in[j] * x[:, j]
    return u


def stream_update(x, y, mix, w_out):
    """Hyper-connection update, from the old streams: new_t = sum_s mix[s, t] x_s + w_out[t] y."""
    n, s, d = x.shape
    new = torch.zeros_like(x)
    for t in range(s):
        acc = w_out[t] * y
        for j in range(s):
            acc = acc + mix[j, t] * x[:, j]
        new[:, t] = acc
    return new


# ---- positions ----------------------------------------------------------------------------------------------

def rotary_frequencies(rot):
    """(frequencies of the dims/2 pairs, factor on cos and sin); YaRN when rot has a 'scaling' entry."""
    dims, base = int(rot["dims"]), float(rot["base"])
    freqs = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return freqs, 1.0

    def dim_of(turns):
        return dims * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

    lo = max(math.floor(dim_of(sc["fast"])), 0)
    hi = min(math.ceil(dim_of(sc["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freqs):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / sc["factor"] * r + f * (1 - r))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x, positions, rot):
    """x (n, heads, dim) with dimension i paired with i + dims/2; dimensions from dims on pass."""
    if not rot:
        return x
    freqs, amp = rotary_frequencies(rot)
    half = len(freqs)
    a = positions.to(torch.float64)[:, None] * torch.tensor(freqs, dtype=torch.float64)[None, :]
    c, s = (a.cos() * amp).to(x.dtype)[:, None, :], (a.sin() * amp).to(x.dtype)[:, None, :]
    u, v = x[..., :half], x[..., half:2 * half]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * half:]], dim=-1)


# ---- mixers -------------------------------------------------------------------------------------------------

def window_attention(q, k, v, scale, window, sink):
    """q (n, H, dk), k (n, G, dk), v (n, G, dv), all positions 0..n-1; one query at a time. `window` None: all."""
    n, H, _ = q.shape
    G, dv = k.shape[1], v.shape[2]
    out = torch.zeros(n, H, dv, dtype=q.dtype)
    for i in range(n):
        j0 = 0 if window is None else max(0, i - window + 1)
        for h in range(H):
            g = h // (H // G)
            s = (k[j0:i + 1, g] @ q[i, h]) * scale
            m = s.max() if sink is None else torch.maximum(s.max(), sink[h])
            e = torch.exp(s - m)
            den = e.sum() + (0 if sink is None else torch.exp(sink[h] - m))
            out[i, h] = (e / den) @ v[j0:i + 1, g]
    return out


def gla_recurrence(q, k, v, alpha, state=None):
    """q, k, alpha (n, H, dk), v (n, H, dv): S <- diag(alpha) S + k v^T, o = S^T q. Returns (o, state)."""
    n, H, dk = q.shape
    dv = v.shape[2]
    S = torch.zeros(H, dk, dv, dtype=q.dtype) if state is None else state.clone()
    out = torch.zeros(n, H, dv, dtype=q.dtype)
    for t in range(n):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(dim=1)
    return out, S


def gla_decay(h, a1, a2, b, tau, heads):
    """Per-key-channel decay sigmoid(z)^(1/tau) of a low-rank z."""
    z = (h @ a1.T) @ a2.T + b
    return torch.exp(-torch.log1p(torch.exp(-z)) / tau).reshape(h.shape[0], heads, -1)


def gla_mixer(h, W, p, mx, eps):
    H, dk, dv = mx["heads"], mx["dim"], mx["vdim"]
    n = h.shape[0]
    q = (h @ W[p + "q"].T * dk ** -0.5).reshape(n, H, dk)
    k = (h @ W[p + "k"].T).reshape(n, H, dk)
    v = (h @ W[p + "v"].T).reshape(n, H, dv)
    alpha = gla_decay(h, W[p + "a1"], W[p + "a2"], W[p + "a2.b"], mx["tau"], H)
    o, _ = gla_recurrence(q, k, v, alpha)
    o = rms_norm(o, W[p + "norm"], eps).reshape(n, H * dv)
    return (o * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


def attention_mixer(h, W, p, mx):
    H, G, dk, dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    n = h.shape[0]
    pos = torch.arange(n)
    q = rotate((h @ W[p + "q"].T).reshape(n, H, dk), pos, mx.get("rot"))
    k = rotate((h @ W[p + "k"].T).reshape(n, G, dk), pos, mx.get("rot"))
    v = (h @ W[p + "v"].T).reshape(n, G, dv)
    window = (mx.get("mask") or {}).get("size")
    o = window_attention(q, k, v, mx["scale"], window, W.get(p + "sink"))
    return o.reshape(n, H * dv) @ W[p + "o"].T


def feed_forward(h, W, p, mlp):
    return clamped_glu(h @ W[p + "gate"].T, h @ W[p + "up"].T, mlp["limit"]) @ W[p + "down"].T


# ---- the model ----------------------------------------------------------------------------------------------

def layer_order(cfg):
    n = len(cfg["layers"])
    loop = cfg.get("loop") or {"start": 0, "stop": 0, "times": 1}
    body = list(range(loop["start"], loop["stop"]))
    return list(range(loop["start"])) + body * loop["times"] + list(range(loop["stop"], n))


def forward(cfg, W, tokens, return_layers=False):
    """Logits (n, vocab) of one sequence from position 0; with return_layers also the sum of the streams after every
    layer run (runs, n, width)."""
    eps = cfg["norm"]["eps"]
    e = W["embed"][torch.as_tensor(tokens)]
    x = e[:, None, :].repeat(1, cfg["streams"], 1)
    trail = []
    for i in layer_order(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        h = rms_norm(stream_in(x, W[p + "hc1.in"]), W[p + "norm1"], eps)
        if layer["type"] == "gla":
            y = gla_mixer(h, W, p + "mix.", layer["mixer"], eps)
        else:
            y = attention_mixer(h, W, p + "mix.", layer["mixer"])
        x = stream_update(x, y, W[p + "hc1.mix"], W[p + "hc1.out"])
        if layer["mlp"] is not None:
            h = rms_norm(stream_in(x, W[p + "hc2.in"]), W[p + "norm2"], eps)
            y = feed_forward(h, W, p + "mlp.", layer["mlp"])
            x = stream_update(x, y, W[p + "hc2.mix"], W[p + "hc2.out"])
        trail.append(x.sum(dim=1))
    h = rms_norm(x.sum(dim=1), W["final.norm"], eps)
    logits = softcap(h @ W["head"].T, cfg["logit_softcap"])
    return (logits, torch.stack(trail)) if return_layers else logits
