"""Plain, slow restatement of the layer-list models (Mefipel), one numpy function per mechanism.

The tests compare the layered engine with it; it shares nothing with the product: it reads the same
config.json keys and tensor names, works in numpy at the precision of ``dt`` (float64 by default) and
handles one sequence, token positions 0 .. n-1, with no cache, no chunks and no batching.
"""
from __future__ import annotations

import math

import numpy as np


# ---- elementwise pieces ----------------------------------------------------------------------------
def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rms_norm(x, w, eps):
    """Rows of x over the root of their mean square (eps inside the root), times w."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


# ---- rotation --------------------------------------------------------------------------------------
def rotation_frequencies(rot):
    """Angles per position of every pair, and the factor of cos and sin."""
    dims, base = rot["dims"], float(rot["base"])
    freq = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)])
    sc = rot.get("scaling")
    if not sc:
        return freq, 1.0
    factor, original = float(sc["factor"]), float(sc["original"])

    def turns(t):
        return dims * math.log(original / (2.0 * math.pi * t)) / (2.0 * math.log(base))

    lo = max(math.floor(turns(sc["fast"])), 0)
    hi = min(math.ceil(turns(sc["slow"])), dims - 1)
    out = np.empty_like(freq)
    for i in range(dims // 2):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out[i] = freq[i] / factor * ramp + freq[i] * (1.0 - ramp)
    return out, 0.1 * math.log(factor) + 1.0


def rotate(x, positions, rot):
    """Rotate-half on the first rot.dims entries of the last axis; x is [tokens, ..., size]."""
    freq, mul = rotation_frequencies(rot)
    half = rot["dims"] // 2
    ang = np.asarray(positions, np.float64)[:, None] * freq[None, :]
    cos, sin = np.cos(ang) * mul, np.sin(ang) * mul
    shape = (x.shape[0],) + (1,) * (x.ndim - 2) + (half,)
    cos, sin = cos.reshape(shape), sin.reshape(shape)
    u, v = x[..., :half], x[..., half:2 * half]
    out = np.array(x)
    out[..., :half] = u * cos - v * sin
    out[..., half:2 * half] = v * cos + u * sin
    return out


# ---- mixers ----------------------------------------------------------------------------------------
def lightning(h, w, mx, eps):
    """Linear attention with one decay per head, token by token."""
    T, H, D, V = h.shape[0], mx["heads"], mx["dim"], mx["vdim"]
    q = silu(h @ w["q"].T).reshape(T, H, D)
    k = silu(h @ w["k"].T).reshape(T, H, D)
    v = silu(h @ w["v"].T).reshape(T, H, V)
    S = np.zeros((H, D, V), h.dtype)
    decay = np.asarray(mx["decay"], h.dtype)[:, None, None]
    o = np.empty((T, H, V), h.dtype)
    for t in range(T):
        S = decay * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hdv,hd->hv", S, q[t])
    o = rms_norm(o.reshape(T, H * V), w["norm"], eps) * sigmoid(h @ w["g"].T)
    return o @ w["o"].T


def window_visible(i, j, size):
    return 0 <= i - j and (size is None or i - j < size)


def latent_attention(h, w, mx, eps):
    """Attention whose keys and values are expanded from one latent per token."""
    T, H, D, R, V = h.shape[0], mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"]
    pos = np.arange(T)
    q = rms_norm(h @ w["dq"].T, w["dq.norm"], eps) @ w["uq"].T
    q = q.reshape(T, H, D + R)
    q_rot = rotate(q[..., D:], pos, mx["rot"])
    down = h @ w["dkv"].T
    c = rms_norm(down[:, :mx["kv_rank"]], w["dkv.norm"], eps)
    k_rot = rotate(down[:, mx["kv_rank"]:], pos, mx["rot"])
    k = (c @ w["uk"].T).reshape(T, H, D)
    v = (c @ w["uv"].T).reshape(T, H, V)
    size = mx.get("mask", {}).get("size") if mx.get("mask") else None
    o = np.zeros((T, H, V), h.dtype)
    for i in range(T):
        lo = 0 if size is None else max(0, i - size + 1)
        s = np.einsum("hd,jhd->hj", q[i, :, :D], k[lo:i + 1]) + q_rot[i] @ k_rot[lo:i + 1].T
        s = s * mx["scale"]
        p = np.exp(s - s.max(axis=1, keepdims=True))
        p /= p.sum(axis=1, keepdims=True)
        o[i] = np.einsum("hj,jhv->hv", p, v[lo:i + 1])
    o = o.reshape(T, H * V) * sigmoid(h @ w["g"].T)
    return o @ w["o"].T


MIXERS = {"lightning": lightning, "latent_attention": latent_attention}


def dense_ff(h, w):
    return gelu_tanh(h @ w["up"].T + w["up.b"]) @ w["down"].T + w["down.b"]


# ---- the model -------------------------------------------------------------------------------------
def _sub(weights, prefix):
    n = len(prefix)
    return {k[n:]: v for k, v in weights.items() if k.startswith(prefix)}


def forward(cfg, weights, tokens, dt=np.float64, layers_out=None):
    """Logits [tokens, vocab] of one sequence; ``layers_out`` (a list) receives the residual after every layer."""
    weights = {k: np.asarray(v, dt) for k, v in weights.items()}
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    x = weights["embed"][np.asarray(tokens)]
    for i, ly in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = rms_norm(x, weights[p + "norm1"], eps)
        y = MIXERS[ly["type"]](h, _sub(weights, p + "mix."), ly["mixer"], eps)
        if ly.get("mlp"):
            y = y + dense_ff(h, _sub(weights, p + "mlp."))
        x = x + m * y
        if layers_out is not None:
            layers_out.append(x)
    return rms_norm(x, weights["final.norm"], eps) @ weights["head"].T * cfg["logit_scale"]
