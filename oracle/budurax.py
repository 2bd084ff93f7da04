"""Plain float64 model of a Budurax decoder: one function per mechanism, whole sequences, no caches.

It is what the tests compare the GPU library with.  It shares no code with the library: numpy only, token by token where the
mechanism is a recurrence, key by key masks where it is attention.  Weights come as a dict name -> array, the configuration as
the dict of config.json.
"""
from __future__ import annotations

import math

import numpy as np


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def sigmoid(z):
    e = np.exp(-np.abs(z))
    return np.where(z >= 0, 1.0 / (1.0 + e), e / (1.0 + e))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def layer_norm(x, weight, bias, eps):
    centred = x - x.mean(-1, keepdims=True)
    return centred / np.sqrt((centred ** 2).mean(-1, keepdims=True) + eps) * weight + bias


def rms_norm(x, weight, eps, parts=1):
    """Each of `parts` equal pieces of the last axis is divided by its own root mean square."""
    pieces = x.reshape(*x.shape[:-1], parts, -1)
    pieces = pieces / np.sqrt((pieces ** 2).mean(-1, keepdims=True) + eps)
    return pieces.reshape(x.shape) * weight


def token_shift(h, mix):
    before = np.concatenate([np.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * mix


def causal_conv(u, taps, bias):
    """u [T, channels], taps [channels, n]: the last column multiplies the current token."""
    n = taps.shape[1]
    out = np.zeros_like(u) + bias
    for t in range(len(u)):
        for k in range(n):
            s = t - (n - 1 - k)
            if s >= 0:
                out[t] += taps[:, k] * u[s]
    return out


def mamba2_recurrence(x, B, C, dt, decay, D):
    """x [T, heads, vdim], B / C [T, groups, state], dt / decay [T, heads], D [heads] -> y [T, heads, vdim]."""
    T, heads, vdim = x.shape
    groups, state = B.shape[1:]
    per = heads // groups
    S = np.zeros((heads, state, vdim))
    y = np.zeros_like(x)
    for t in range(T):
        for h in range(heads):
            g = h // per
            S[h] = decay[t, h] * S[h] + dt[t, h] * np.outer(B[t, g], x[t, h])
            y[t, h] = C[t, g] @ S[h] + D[h] * x[t, h]
    return y


def mamba2(h, w, p, m, eps):
    """Mixer input h [T, width]; w weights, p tensor prefix, m the mixer's sizes."""
    heads, vdim, state, groups = m["heads"], m["vdim"], m["state"], m["groups"]
    inner, bc = heads * vdim, groups * state
    u = h @ w[p + "in"].T
    z, xbc, dt = u[:, :inner], u[:, inner:2 * inner + 2 * bc], u[:, 2 * inner + 2 * bc:]
    xbc = silu(causal_conv(xbc, w[p + "conv"], w[p + "conv.b"]))
    x = xbc[:, :inner].reshape(-1, heads, vdim)
    B = xbc[:, inner:inner + bc].reshape(-1, groups, state)
    C = xbc[:, inner + bc:].reshape(-1, groups, state)
    dt = softplus(dt + w[p + "dt_bias"])
    decay = np.exp(-np.exp(w[p + "A_log"]) * dt)
    y = mamba2_recurrence(x, B, C, dt, decay, w[p + "D"]).reshape(-1, inner)
    y = rms_norm(y * silu(z), w[p + "norm"], eps, m["norm_groups"])
    return y @ w[p + "o"].T


def rotary_frequencies(rot):
    dims, base = rot["dims"], float(rot["base"])
    i = np.arange(dims // 2)
    f = base ** (-2.0 * i / dims)
    s = rot.get("scaling")
    if not s:
        return f, 1.0

    def turn(t):
        return dims * math.log(s["original"] / (2.0 * math.pi * t)) / (2.0 * math.log(base))
    lo = max(math.floor(turn(s["fast"])), 0)
    hi = min(math.ceil(turn(s["slow"])), dims - 1)
    ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / s["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(s["factor"]) + 1.0


def rotate(x, rot):
    """x [T, ..., at least rot.dims]: pairs (i, i + dims / 2) turned by position times frequency."""
    freq, gain = rotary_frequencies(rot)
    half = rot["dims"] // 2
    angle = np.arange(len(x))[:, None] * freq
    shape = (len(x),) + (1,) * (x.ndim - 2) + (half,)
    c, s = np.cos(angle).reshape(shape) * gain, np.sin(angle).reshape(shape) * gain
    u, v, rest = x[..., :half], x[..., half:2 * half], x[..., 2 * half:]
    return np.concatenate([u * c - v * s, v * c + u * s, rest], -1)


def causal_softmax_attention(q, k, v, scale):
    """q / k [T, d], v [T, e]: ordinary softmax over the keys up to the query's own position."""
    s = (q @ k.T) * scale
    s = np.where(np.tril(np.ones_like(s)) > 0, s, -np.inf)
    p = np.exp(s - s.max(-1, keepdims=True))
    return (p / p.sum(-1, keepdims=True)) @ v


def latent_keys(h, w, p, m, eps):
    down = h @ w[p + "dkv"].T
    c = rms_norm(down[:, :m["kv_rank"]], w[p + "dkv.norm"], eps)
    return c, rotate(down[:, m["kv_rank"]:], m["rot"])


def latent_attention(h, w, p, m, c, k_rot):
    H, d, r, e = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    q = (h @ w[p + "q"].T).reshape(-1, H, d + r)
    q_rot = rotate(q[..., d:], m["rot"])
    k = (c @ w[p + "uk"].T).reshape(-1, H, d)
    v = (c @ w[p + "uv"].T).reshape(-1, H, e)
    out = np.zeros((len(h), H, e))
    for n in range(H):
        out[:, n] = causal_softmax_attention(np.concatenate([q[:, n, :d], q_rot[:, n]], -1), np.concatenate([k[:, n], k_rot], -1), v[:, n], m["scale"])
    out = out.reshape(len(h), H * e) * sigmoid(h @ w[p + "g"].T)
    return out @ w[p + "o"].T


def dense_mlp(h, w, p):
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def token_side_input(x, rows, w, p, eps):
    y = (gelu_tanh(x @ w[p + "gate"].T) * rows) @ w[p + "proj"].T
    return rms_norm(y, w[p + "norm"], eps)


def depth_average(states, coefficients):
    return sum(a * x for a, x in zip(coefficients, states))


def forward(config, w, tokens, layers_out=None):
    """tokens [T] -> logits [T, vocab]; layers_out (a list) receives the residual stream after every layer."""
    w = {k: np.asarray(v, np.float64) for k, v in w.items()}
    tokens = np.asarray(tokens)
    eps = config["norm"]["eps"]

    def norm(x, name):
        return layer_norm(x, w[name], w[name + ".b"], eps)
    side = config["token_side"]["dim"]
    x = w["embed"][tokens]
    states, shared = [x], {}
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = token_shift(norm(x, p + "norm1"), w[p + "shift"])
        if layer["type"] == "mamba2":
            y = mamba2(h, w, p + "mix.", m, eps)
        else:
            src = m.get("kv_from")
            shared[i] = shared[src] if src is not None else latent_keys(h, w, p + "mix.", m, eps)
            y = latent_attention(h, w, p + "mix.", m, *shared[i])
        x = x + norm(y, p + "norm1b")
        if layer["mlp"] is not None:
            x = x + norm(dense_mlp(norm(x, p + "norm2"), w, p + "mlp."), p + "norm2b")
        x = x + token_side_input(x, w["side.embed"][tokens][:, i * side:(i + 1) * side], w, p + "side.", eps)
        states.append(x)
        x = depth_average(states, w[p + "dwa"])
        if layers_out is not None:
            layers_out.append(x)
    return norm(x, "final.norm") @ w["head"].T
