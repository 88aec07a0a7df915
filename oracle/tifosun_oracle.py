"""Plain, slow CPU implementation of the Tifosun decoder: mLSTM and windowed latent-attention layers, norms on both sides
of every sublayer, dense and routed feed-forwards. One function per mechanism, the recurrence written token by token;
test infrastructure only, it shares no code with the package.

`cfg` is the parsed config.json, `W` a dict name -> tensor with the checkpoint's tensor names. The arithmetic runs in
the dtype of the tensors given (double for the tightest comparison).
"""
from __future__ import annotations

import torch


# ---- small mechanisms ---------------------------------------------------------------------------------------

def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def norm_around_zero(x, w, eps):
    """RMS norm whose stored weight is the distance from 1."""
    return unit_rms(x, eps) * (1 + w)


def sigmoid(x):
    return 1 / (1 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def log_sigmoid(x):
    return torch.clamp(x, max=0) - torch.log1p(torch.exp(-x.abs()))


def capped(x, cap):
    return cap * torch.tanh(x / cap)


def rotate_pairs(x, positions, base):
    """x (n, ..., dims): dimensions 2i and 2i + 1 turn by position * base^(-2i / dims)."""
    dims = x.shape[-1]
    f = torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
    a = positions.to(torch.float64)[:, None] * f[None, :]
    a = a.reshape(a.shape[0], *([1] * (x.dim() - 2)), dims // 2)
    c, s = a.cos().to(x.dtype), a.sin().to(x.dtype)
    out = x.clone()
    out[..., 0::2] = x[..., 0::2] * c - x[..., 1::2] * s
    out[..., 1::2] = x[..., 1::2] * c + x[..., 0::2] * s
    return out


# ---- matrix memory --------------------------------------------------------------------------------------------

def mlstm_gates(zi, zf, bi, bf, cap):
    """(log input gate, log forget gate) from the projections and their biases."""
    return capped(zi + bi, cap), log_sigmoid(capped(zf + bf, cap))


def mlstm_recurrence(q, k, v, i, f, state=None):
    """q, k (n, H, dk), v (n, H, dv), log gates i, f (n, H). Returns (o (n, H, dv), (S, n, m))."""
    n, H, dk = q.shape
    dv = v.shape[2]
    if state is None:
        S, N, m = (torch.zeros(*s, dtype=q.dtype) for s in ((H, dk, dv), (H, dk), (H,)))
    else:
        S, N, m = (s.clone() for s in state)
    out = torch.zeros(n, H, dv, dtype=q.dtype)
    for t in range(n):
        new_m = torch.maximum(f[t] + m, i[t])
        keep, add = torch.exp(f[t] + m - new_m), torch.exp(i[t] - new_m)
        m = new_m
        S = keep[:, None, None] * S + add[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        N = keep[:, None] * N + add[:, None] * k[t]
        top = (S * q[t][:, :, None]).sum(dim=1)
        low = torch.maximum((N * q[t]).sum(dim=1).abs(), torch.exp(-m)) + 1e-6
        out[t] = top / low[:, None]
    return out, (S, N, m)


def mlstm_mixer(h, W, p, mx, eps):
    H, dk, dv = mx["heads"], mx["dim"], mx["vdim"]
    n = h.shape[0]
    q = (h @ W[p + "q"].T).reshape(n, H, dk) * dk ** -0.5
    k = (h @ W[p + "k"].T).reshape(n, H, dk)
    v = (h @ W[p + "v"].T).reshape(n, H, dv)
    i, f = mlstm_gates(h @ W[p + "i"].T, h @ W[p + "f"].T, W[p + "i.b"], W[p + "f.b"], mx["gate_cap"])
    o, _ = mlstm_recurrence(q, k, v, i, f)
    o = unit_rms(o, eps).reshape(n, H * dv) * W[p + "norm"]
    return (o * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


# ---- latent attention -----------------------------------------------------------------------------------------

def window_softmax_attention(q, k, v, scale, window):
    """q, k (n, H, dk), v (n, H, dv), positions 0..n-1, one query at a time; `window` None: all tokens before."""
    n, H, _ = q.shape
    out = torch.zeros(n, H, v.shape[2], dtype=q.dtype)
    for i in range(n):
        j0 = 0 if window is None else max(0, i - window + 1)
        for h in range(H):
            s = (k[j0:i + 1, h] @ q[i, h]) * scale
            e = torch.exp(s - s.max())
            out[i, h] = (e / e.sum()) @ v[j0:i + 1, h]
    return out


def latent_rows(d, norm, rank, base, eps, positions):
    """Rows of the down-projection -> (normed latents, rotated key part shared by the heads)."""
    return unit_rms(d[:, :rank], eps) * norm, rotate_pairs(d[:, rank:], positions, base)


def latent_keys_values(c, kr, uk, uv, heads):
    """Latents and the shared key part -> keys (n, H, dim + rot), values (n, H, dv)."""
    n = c.shape[0]
    k = (c @ uk.T).reshape(n, heads, -1)
    v = (c @ uv.T).reshape(n, heads, -1)
    return torch.cat([k, kr[:, None].expand(n, heads, kr.shape[1])], dim=-1), v


def latent_attention_mixer(h, W, p, mx, eps):
    H, dim, rot, rank = mx["heads"], mx["dim"], mx["rot_dim"], mx["kv_rank"]
    n = h.shape[0]
    pos = torch.arange(n)
    base = mx["rot"]["base"]
    q = (h @ W[p + "q"].T).reshape(n, H, dim + rot)
    q = torch.cat([q[..., :dim], rotate_pairs(q[..., dim:], pos, base)], dim=-1)
    c, kr = latent_rows(h @ W[p + "dkv"].T, W[p + "dkv.norm"], rank, base, eps, pos)
    k, v = latent_keys_values(c, kr, W[p + "uk"], W[p + "uv"], H)
    o = window_softmax_attention(q, k, v, mx["scale"], (mx.get("mask") or {}).get("size"))
    return (o.reshape(n, -1) * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


# ---- feed-forwards --------------------------------------------------------------------------------------------

def gated_unit(h, W, p):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def route(z, top):
    """Router logits (n, E) -> (chosen experts (n, top), their weights)."""
    s = sigmoid(z)
    idx = torch.sort(s, dim=1, descending=True, stable=True).indices[:, :top]
    return idx, s.gather(1, idx)


def mixture(h, W, p, mlp):
    idx, w = route(h @ W[p + "router"].T, mlp["router"]["top"])
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, we in zip(idx[t].tolist(), w[t]):
            y[t] += gated_unit(we * h[t:t + 1], W, f"{p}e{e}.")[0]
    if mlp.get("shared"):
        y = y + gated_unit(h, W, p + "shared.")
    return y


def feed_forward(h, W, p, mlp):
    return gated_unit(h, W, p) if mlp["kind"] == "dense" else mixture(h, W, p, mlp)


# ---- the model ------------------------------------------------------------------------------------------------

def forward(cfg, W, tokens, return_layers=False):
    """Logits (n, vocab) of one sequence from position 0; with return_layers also the residual after every layer
    (layers, n, width)."""
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens)]
    trail = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        mixer = latent_attention_mixer if layer["type"] == "latent_attention" else mlstm_mixer
        y = mixer(norm_around_zero(x, W[p + "norm1"], eps), W, p + "mix.", layer["mixer"], eps)
        x = x + norm_around_zero(y, W[p + "norm1b"], eps)
        if layer.get("mlp") is not None:
            y = feed_forward(norm_around_zero(x, W[p + "norm2"], eps), W, p + "mlp.", layer["mlp"])
            x = x + norm_around_zero(y, W[p + "norm2b"], eps)
        trail.append(x)
    logits = norm_around_zero(x, W["final.norm"], eps) @ W["head"].T
    return (logits, torch.stack(trail)) if return_layers else logits
