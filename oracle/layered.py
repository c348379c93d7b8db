"""Plain, slow restatement of the layer-list models (Mefipel, Tozarax), one numpy function per mechanism.

The tests compare the layered engine with it; it shares nothing with the product: it reads the same
config.json keys and tensor names, works in numpy at the precision of ``dt`` (float64 by default) and
handles one sequence, token positions 0 .. n-1, with no cache, no chunks and no batching.
"""
from __future__ import annotations

import math

import numpy as np


# What a 16-bit run keeps of an activation; `forward(rounding=...)` sets it to see how far rounding alone goes.
def _exact(x):
    return x


_keep = _exact


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


def attention(h, w, mx, eps):
    """Grouped softmax attention without rotation; a window counts the token itself."""
    T, H, G, D, V = h.shape[0], mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    q = _keep(h @ w["q"].T).reshape(T, H, D)
    k = _keep(h @ w["k"].T).reshape(T, G, D)
    v = _keep(h @ w["v"].T).reshape(T, G, V)
    size = (mx.get("mask") or {}).get("size")
    out = np.zeros((T, H, V), h.dtype)
    for n in range(H):
        g = n // (H // G)
        for i in range(T):
            lo = min(j for j in range(i + 1) if window_visible(i, j, size))
            s = k[lo:i + 1, g] @ q[i, n] * mx["scale"]
            p = np.exp(s - s.max())
            out[i, n] = (p / p.sum()) @ v[lo:i + 1, g]
    return _keep(_keep(out.reshape(T, H * V)) @ w["o"].T)


def causal_conv(x, w):
    """Per channel: w's last column meets the current token, zeros before the first."""
    T, taps = x.shape[0], w.shape[1]
    y = np.zeros_like(x)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += w[:, j] * x[:T - back]
    return y


def softplus(z):
    return np.logaddexp(0.0, z)


def unit(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def gated_delta(h, w, mx, eps):
    """Delta rule with one decay and one step size per head and token, token by token."""
    T, H, G, D, V = h.shape[0], mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    short = lambda n: _keep(silu(causal_conv(_keep(h @ w[n].T), w[n + ".conv"])))  # noqa: E731
    q = unit(short("q").reshape(T, G, D)) * D ** -0.5
    k = unit(short("k").reshape(T, G, D))
    v = short("v").reshape(T, H, V)
    beta = sigmoid(h @ w["b"].T)
    decay = np.exp(-np.exp(w["A_log"]) * softplus(h @ w["a"].T + w["dt_bias"]))
    o = np.empty((T, H, V), h.dtype)
    for n in range(H):
        g, S = n // (H // G), np.zeros((D, V), h.dtype)
        for t in range(T):
            S = S * decay[t, n]
            u = beta[t, n] * (v[t, n] - k[t, g] @ S)
            S = S + np.outer(k[t, g], u)
            o[t, n] = q[t, g] @ S
    o = rms_norm(o, w["norm"], eps) * _keep(silu(h @ w["g"].T)).reshape(T, H, V)
    return _keep(_keep(o.reshape(T, H * V)) @ w["o"].T)


def parallel(h, w, mx, eps):
    """Two mixers on the same input; each result normed over the width, then their mean."""
    left = attention(h, _sub(w, "left."), mx["left"], eps)
    right = gated_delta(h, _sub(w, "right."), mx["right"], eps)
    return 0.5 * (rms_norm(left, w["left.out"], eps) + rms_norm(right, w["right.out"], eps))


MIXERS = {"lightning": lightning, "latent_attention": latent_attention, "attention": attention, "gated_delta": gated_delta,
          "parallel": parallel}


def dense_ff(h, w):
    return gelu_tanh(h @ w["up"].T + w["up.b"]) @ w["down"].T + w["down.b"]


def route(z, correction, top, groups):
    """Chosen experts of one token (best first) and their weights."""
    s = sigmoid(z)
    choice = s + correction
    if groups:
        per = len(z) // groups["count"]
        score = [sum(sorted(choice[g * per:(g + 1) * per])[-2:]) for g in range(groups["count"])]
        keep = sorted(range(groups["count"]), key=lambda g: (-score[g], g))[:groups["keep"]]
        choice = np.array([c if e // per in keep else -np.inf for e, c in enumerate(choice)])
    best = sorted(range(len(z)), key=lambda e: (-choice[e], e))[:top]
    return best, s[best]


def moe_ff(h, w, mlp):
    """Sigmoid router with a correction that takes part in the choice only; experts with a squared relu."""
    r, y = mlp["router"], np.zeros_like(h)
    z = h @ w["router"].T
    for t in range(h.shape[0]):
        for e, weight in zip(*route(z[t], w["correction"], r["top"], r.get("groups"))):
            y[t] += weight * _keep(w[f"e{e}.down"] @ _keep(np.maximum(w[f"e{e}.up"] @ h[t], 0.0) ** 2))
    return y


# ---- a layer with sublayers one after the other -------------------------------------------------------
def sublayer(x, w, p, n, eps, offset, f):
    """x plus the result of f on the norm; n is "1" (mixer) or "2" (feed-forward).  With a convolution f reads the
    norm plus its convolution, with a gate the result is multiplied by it."""
    h = _keep(rms_norm(x, offset + w[p + "norm" + n], eps))
    y = f(_keep(h + causal_conv(h, w[p + "canon" + n])) if p + "canon" + n in w else h)
    if p + "rg" + n in w:
        y = y * _keep(sigmoid(h @ w[p + "rg" + n].T + w[p + "rg" + n + ".b"]))
    return x + y


def depth_average(w, history):
    return sum(a * x for a, x in zip(w, history))


def forward_sequential(cfg, weights, tokens, layers_out=None):
    eps, offset = cfg["norm"]["eps"], cfg.get("norm_offset", 1.0)
    x = weights["embed"][np.asarray(tokens)]
    if "pos" in weights:
        x = x + weights["pos"][:len(tokens)]
    history = [x]
    for i, ly in enumerate(cfg["layers"]):
        p, mlp = f"l{i}.", ly.get("mlp")
        x = sublayer(x, weights, p, "1", eps, offset, lambda h: MIXERS[ly["type"]](h, _sub(weights, p + "mix."), ly["mixer"], eps))
        if mlp:
            ff = (lambda h: dense_ff(h, _sub(weights, p + "mlp."))) if mlp["kind"] == "dense" else (lambda h: moe_ff(h, _sub(weights, p + "mlp."), mlp))
            x = sublayer(x, weights, p, "2", eps, offset, ff)
        history.append(x)
        if p + "dwa" in weights:
            x = depth_average(weights[p + "dwa"], history)
        if layers_out is not None:
            layers_out.append(x)
    return _keep(rms_norm(x, offset + weights["final.norm"], eps)) @ weights["head"].T


# ---- the model -------------------------------------------------------------------------------------
def _sub(weights, prefix):
    n = len(prefix)
    return {k[n:]: v for k, v in weights.items() if k.startswith(prefix)}


def forward(cfg, weights, tokens, dt=np.float64, layers_out=None, rounding=_exact):
    """Logits [tokens, vocab] of one sequence; ``layers_out`` (a list) receives the residual after every layer.
    ``rounding`` is applied to the activations between linears (sequential layers only)."""
    global _keep
    _keep = rounding
    weights = {k: np.asarray(v, dt) for k, v in weights.items()}
    if cfg["architecture"] != "Mefipel":
        return forward_sequential(cfg, weights, tokens, layers_out)
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
