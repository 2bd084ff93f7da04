"""Plain float64 model of a Lutelorn decoder: one function per mechanism, whole sequences, no caches.

It is what the tests compare the GPU library with.  It shares no code with the library: numpy only, token by token where the
mechanism is a recurrence, a full matrix of scores where it is attention.  Weights come as a dict name -> array, the
configuration as the dict of config.json.
"""
from __future__ import annotations

import numpy as np

from .budurax import rms_norm, sigmoid, silu


def offset_norm(x, weight, eps):
    """Root-mean-square norm whose weight is stored as its distance from one."""
    return rms_norm(x, 1.0 + weight, eps)


def bigram_rows(tokens, buckets, mul_prev, mul_cur):
    """Row of the pair table for every token; the sequence's first token has the row after the hashed ones."""
    rows = [buckets]
    for before, now in zip(tokens[:-1], tokens[1:]):
        rows.append((int(before) * mul_prev + int(now) * mul_cur) % buckets)
    return np.array(rows)


def embedding(tokens, w, e):
    x = w["embed"][tokens] * e["scale"]
    if "bigram" not in e:
        return x
    b = e["bigram"]
    return x + w["bigram"][bigram_rows(tokens, b["buckets"], b["mul_prev"], b["mul_cur"])]


def previous(h):
    return np.concatenate([np.zeros_like(h[:1]), h[:-1]])


def decayed_outer_products(q, k, v, decay):
    """q / k [T, heads, d], v [T, heads, e], decay [heads]: S <- decay S + k v^T, then o = S^T q."""
    S = np.zeros((k.shape[1], k.shape[2], v.shape[2]))
    out = np.zeros_like(v)
    for t in range(len(q)):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hde,hd->he", S, q[t])
    return out


def lightning(h, w, p, m, eps):
    H, d, e = m["heads"], m["dim"], m["vdim"]
    q, k, v = (silu(h @ w[p + n].T).reshape(-1, H, size) for n, size in (("q", d), ("k", d), ("v", e)))
    o = decayed_outer_products(q, k, v, np.asarray(m["decay"], np.float64)).reshape(-1, H * e)
    return (rms_norm(o, w[p + "norm"], eps) * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def rotate_neighbours(x, rot):
    """x [T, heads, dim]: dimensions (2i, 2i + 1) of the first rot.dims turn by position * base^(-2i / dims)."""
    n, base = rot["dims"], float(rot["base"])
    out = x.copy()
    for i in range(n // 2):
        a = (np.arange(len(x)) * base ** (-2.0 * i / n))[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a)
    return out


def capped_attention(q, k, v, scale, cap):
    """q / k [T, d], v [T, e]: softmax over the keys up to the query's own of cap tanh(score / cap); no cap: of the scores."""
    s = (q @ k.T) * scale
    if cap is not None:
        s = cap * np.tanh(s / cap)
    s = np.where(np.tril(np.ones_like(s)) > 0, s, -np.inf)
    p = np.exp(s - s.max(-1, keepdims=True))
    return (p / p.sum(-1, keepdims=True)) @ v


def mixed_values(v, first, share):
    return (1.0 - share) * v + share * first


def attention(h, w, p, m, first_values):
    """-> (output, this layer's own values [T, kv_heads, vdim] before any mixing)."""
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = ((h @ w[p + n].T + w[p + n + ".b"]).reshape(-1, heads, size) for n, heads, size in (("q", H, d), ("k", G, d), ("v", G, e)))
    own = v
    if "rot" in m:
        q, k = rotate_neighbours(q, m["rot"]), rotate_neighbours(k, m["rot"])
    if m.get("v_mix") and first_values is not None:
        v = mixed_values(v, first_values, float(np.asarray(w[p + "vmix"]).reshape(())))
    out = np.stack([capped_attention(q[:, n], k[:, n // (H // G)], v[:, n // (H // G)], m["scale"], m.get("softcap")) for n in range(H)], 1)
    return (out.reshape(len(h), H * e) * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T, own


def bonus_recurrence(r, k, v, decay, u):
    """r / k / decay [T, heads, d], v [T, heads, e], u [heads, d]: o = (S + diag(u) k v^T)^T r, then S <- diag(decay) S + k v^T."""
    S = np.zeros((k.shape[1], k.shape[2], v.shape[2]))
    out = np.zeros_like(v)
    for t in range(len(r)):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hde,hd->he", S + u[:, :, None] * kv, r[t])
        S = decay[t][:, :, None] * S + kv
    return out


def wkv(h, w, p, m, eps):
    H, d = m["heads"], m["dim"]
    before = previous(h)
    mix = {n: h + (before - h) * w[p + "mu." + n] for n in "rkvgw"}
    r, k, v = ((mix[n] @ w[p + n].T).reshape(-1, H, d) for n in "rkv")
    decay = np.exp(-np.exp(np.tanh(mix["w"] @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"])).reshape(-1, H, d)
    o = bonus_recurrence(r, k, v, decay, w[p + "u"]).reshape(-1, H * d)
    return (rms_norm(o, w[p + "norm"], eps, H) * silu(mix["g"] @ w[p + "g"].T)) @ w[p + "o"].T


def dense_mlp(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def forward(config, w, tokens, layers_out=None):
    """tokens [T] -> logits [T, vocab]; layers_out (a list) receives the residual stream after every layer."""
    w = {k: np.asarray(v, np.float64) for k, v in w.items()}
    tokens = np.asarray(tokens)
    eps, m = config["norm"]["eps"], config["residual_mult"]
    x = embedding(tokens, w, config["embedding"])
    first_values = None
    for i, layer in enumerate(config["layers"]):
        p, mix = f"l{i}.", layer["mixer"]
        h = offset_norm(x, w[p + "norm1"], eps)
        if layer["type"] == "lightning":
            y = lightning(h, w, p + "mix.", mix, eps)
        elif layer["type"] == "wkv":
            y = wkv(h, w, p + "mix.", mix, eps)
        else:
            y, own = attention(h, w, p + "mix.", mix, first_values)
            if mix.get("v_mix") and first_values is None:
                first_values = own
        x = x + m * y
        if layer["mlp"] is not None:
            x = x + m * dense_mlp(offset_norm(x, w[p + "norm2"], eps), w, p + "mlp.")
        if layers_out is not None:
            layers_out.append(x)
    return offset_norm(x, w["final.norm"], eps) @ w["head"].T
