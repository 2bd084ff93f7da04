"""Small random Budurax and Lutelorn models for the tests: configuration, weights, the folder that the library loads, and how a loaded
model is fed."""
import json
import os
import struct

import numpy as np


def bf16(a):
    """Values that bf16 holds exactly (rounded to nearest even), as float32."""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32).astype(np.uint64)
    return (((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint32) << 16).view(np.float32).reshape(np.shape(a))


def mamba(heads=4, vdim=16, state=16, groups=2, conv=4, norm_groups=2, ff=96):
    return dict(type="mamba2", mixer=dict(heads=heads, vdim=vdim, state=state, groups=groups, conv=conv, norm_groups=norm_groups),
                mlp=None if ff is None else dict(kind="dense", ff=ff))


def latent(heads=3, dim=16, rot_dim=16, vdim=24, kv_rank=40, scale=0.2, base=10000.0, scaling=None, kv_from=None, ff=96):
    rot = dict(base=base, dims=rot_dim)
    if scaling:
        rot["scaling"] = scaling
    mixer = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, scale=scale, rot=rot)
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return dict(type="latent_attention", mixer=mixer, mlp=None if ff is None else dict(kind="dense", ff=ff))


YARN = dict(factor=4.0, original=64, fast=16.0, slow=2.0)


def config(layers, width=72, vocab=101, side=16, eps=1e-5):
    return dict(architecture="Budurax", width=width, vocab=vocab, norm=dict(eps=eps), token_side=dict(dim=side), layers=layers)


def attention(heads=4, kv_heads=2, dim=24, vdim=20, scale=0.25, softcap=8.0, base=10000.0, rot=16, v_mix=True, ff=96):
    mixer = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, v_mix=v_mix)
    if softcap:
        mixer["softcap"] = softcap
    if rot:
        mixer["rot"] = dict(base=base, dims=rot)
    return dict(type="attention", mixer=mixer, mlp=None if ff is None else dict(kind="dense", ff=ff))


def lightning(heads=3, dim=16, vdim=24, decay=None, ff=96):
    decay = [0.4, 0.93, 0.998, 0.8, 1.0][:heads] if decay is None else decay
    return dict(type="lightning", mixer=dict(heads=heads, dim=dim, vdim=vdim, decay=decay), mlp=None if ff is None else dict(kind="dense", ff=ff))


def wkv(heads=3, dim=24, rank=10, ff=96):
    """rank is no part of the configuration: the weights' shapes give it."""
    return dict(type="wkv", mixer=dict(heads=heads, dim=dim), mlp=None if ff is None else dict(kind="dense", ff=ff), rank=rank)


def lutelorn(layers, width=72, vocab=101, eps=1e-5, scale=0.7, residual_mult=0.4, bigram=(61, 29, 13)):
    embedding = dict(scale=scale)
    if bigram:
        embedding["bigram"] = dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))
    return dict(architecture="Lutelorn", width=width, vocab=vocab, norm=dict(eps=eps), embedding=embedding, residual_mult=residual_mult, layers=layers)


def lutelorn_weights(c, seed=0):
    rng = np.random.default_rng(seed)
    W, V = c["width"], c["vocab"]
    w = {}

    def lin(name, out, inp, gain=1.0):
        w[name] = gain * rng.standard_normal((out, inp)) / np.sqrt(inp)

    w["embed"] = rng.standard_normal((V, W))
    if "bigram" in c["embedding"]:
        w["bigram"] = rng.standard_normal((c["embedding"]["bigram"]["buckets"] + 1, W))
    for i, l in enumerate(c["layers"]):
        p, m = f"l{i}.", l["mixer"]
        w[p + "norm1"] = 0.3 * rng.standard_normal(W)
        if l["type"] == "attention":
            H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for n, size in (("q", H * d), ("k", G * d), ("v", G * e)):
                lin(p + "mix." + n, size, W, 1.5 if n != "v" else 1.0)
                w[p + "mix." + n + ".b"] = 0.5 * rng.standard_normal(size)
            lin(p + "mix.g", H * e, W)
            lin(p + "mix.o", W, H * e)
            if m["v_mix"]:
                w[p + "mix.vmix"] = np.float32(0.35 + 0.1 * (i % 3))
        elif l["type"] == "lightning":
            H, d, e = m["heads"], m["dim"], m["vdim"]
            for n, size in (("q", H * d), ("k", H * d), ("v", H * e), ("g", H * e)):
                lin(p + "mix." + n, size, W, 1.5)
            w[p + "mix.norm"] = 1.0 + 0.2 * rng.standard_normal(H * e)
            lin(p + "mix.o", W, H * e)
        else:
            n, rank = m["heads"] * m["dim"], l["rank"]
            for x in "rkvg":
                lin(p + "mix." + x, n, W)
            lin(p + "mix.w1", rank, W)
            lin(p + "mix.w2", n, rank)
            w[p + "mix.w0"] = rng.uniform(-6.0, 0.5, n)
            w[p + "mix.u"] = rng.standard_normal((m["heads"], m["dim"]))
            w[p + "mix.norm"] = 1.0 + 0.2 * rng.standard_normal(n)
            for x in "rkvgw":
                w[p + "mix.mu." + x] = rng.uniform(0.0, 1.0, W)
            lin(p + "mix.o", W, n)
        if l["mlp"] is not None:
            w[p + "norm2"] = 0.3 * rng.standard_normal(W)
            ff = l["mlp"]["ff"]
            lin(p + "mlp.gate", ff, W)
            lin(p + "mlp.up", ff, W)
            lin(p + "mlp.down", W, ff)
    w["final.norm"] = 0.3 * rng.standard_normal(W)
    lin("head", V, W)
    return {k: bf16(v) for k, v in w.items()}


def weights(c, seed=0):
    """Random weights, every parameter away from its neutral value, rounded to bf16."""
    if c["architecture"] == "Lutelorn":
        return lutelorn_weights(c, seed)
    rng = np.random.default_rng(seed)
    W, V, side = c["width"], c["vocab"], c["token_side"]["dim"]
    w = {}

    def lin(name, out, inp, gain=1.0):
        w[name] = gain * rng.standard_normal((out, inp)) / np.sqrt(inp)

    def norm(name):
        w[name] = 1.0 + 0.2 * rng.standard_normal(W)
        w[name + ".b"] = 0.1 * rng.standard_normal(W)

    w["embed"] = rng.standard_normal((V, W))
    w["side.embed"] = rng.standard_normal((V, len(c["layers"]) * side))
    for i, l in enumerate(c["layers"]):
        p, m = f"l{i}.", l["mixer"]
        for n in ("norm1", "norm1b"):
            norm(p + n)
        w[p + "shift"] = rng.uniform(0.0, 1.0, W)
        w[p + "dwa"] = rng.uniform(-0.4, 0.4, i + 2)
        w[p + "dwa"][-1] += 1.0
        if l["type"] == "mamba2":
            inner, bc = m["heads"] * m["vdim"], m["groups"] * m["state"]
            lin(p + "mix.in", 2 * inner + 2 * bc + m["heads"], W)
            w[p + "mix.conv"] = rng.standard_normal((inner + 2 * bc, m["conv"])) * 0.6
            w[p + "mix.conv.b"] = 0.2 * rng.standard_normal(inner + 2 * bc)
            w[p + "mix.dt_bias"] = rng.uniform(-3.0, 0.0, m["heads"])
            w[p + "mix.A_log"] = rng.uniform(-2.0, 1.0, m["heads"])
            w[p + "mix.D"] = rng.standard_normal(m["heads"])
            w[p + "mix.norm"] = 1.0 + 0.2 * rng.standard_normal(inner)
            lin(p + "mix.o", W, inner)
        else:
            H, d, r, e, k = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            lin(p + "mix.q", H * (d + r), W)
            if "kv_from" not in m:
                lin(p + "mix.dkv", k + r, W)
                w[p + "mix.dkv.norm"] = 1.0 + 0.2 * rng.standard_normal(k)
            lin(p + "mix.uk", H * d, k)
            lin(p + "mix.uv", H * e, k)
            lin(p + "mix.g", H * e, W)
            lin(p + "mix.o", W, H * e)
        if l["mlp"] is not None:
            ff = l["mlp"]["ff"]
            for n in ("norm2", "norm2b"):
                norm(p + n)
            lin(p + "mlp.gate", ff, W)
            lin(p + "mlp.up", ff, W)
            lin(p + "mlp.down", W, ff)
        lin(p + "side.gate", side, W)
        lin(p + "side.proj", W, side)
        w[p + "side.norm"] = 0.5 * rng.standard_normal(W)
    norm("final.norm")
    lin("head", V, W)
    return {k: bf16(v) for k, v in w.items()}


def save(folder, c, w, dtype="BF16"):
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(dict(c, layers=[{k: v for k, v in l.items() if k != "rank"} for l in c["layers"]]), f)
    header, blobs, at = {}, [], 0
    for name, a in w.items():
        a = np.ascontiguousarray(a, np.float32)
        data = (a.view(np.uint32) >> 16).astype(np.uint16).tobytes() if dtype == "BF16" else a.tobytes()
        header[name] = dict(dtype=dtype, shape=list(np.shape(w[name])), data_offsets=[at, at + len(data)])
        blobs.append(data)
        at += len(data)
    text = json.dumps(header).encode()
    text += b" " * (-len(text) % 8)
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(text)) + text + b"".join(blobs))
    return str(folder)


def load(tmp_path, c, w, dtype):
    from gpt_b200 import serving
    return serving.load_model(save(tmp_path / "model", c, w), dtype)


def portions(model, seq, tokens, cuts):
    """Logits of all rows, the tokens fed in portions of the given sizes (the last size repeats)."""
    out, at, i = [], 0, 0
    while at < len(tokens):
        n = min(cuts[min(i, len(cuts) - 1)], len(tokens) - at)
        out.append(model.step([(seq, tokens[at:at + n])], range(n)))
        at += n
        i += 1
    return np.concatenate(out)


def whole(model, tokens, cuts=(1 << 20,), max_len=None):
    seq = model.open(max_len or len(tokens))
    try:
        return portions(model, seq, tokens, cuts)
    finally:
        model.close(seq)


def row_errors(got, want):
    """Per row: root mean square difference, relative to the root mean square of all expected logits."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    return np.sqrt(((got - want) ** 2).mean(-1)) / np.sqrt((want ** 2).mean())


def error(got, want):
    return float(row_errors(got, want).max())


def close(got, want, tol):
    """All but 2 % of the rows (but not the only one) within tol, all within 3 tol: rounding is amplified a few times at single rows,
    whichever form of a layer runs (the same rows in all of them); a fault moves a row by ten times that."""
    e = np.sort(row_errors(got, want))
    return bool(np.isfinite(got).all() and e[min(len(e) - 1, int(0.98 * len(e)))] <= tol and e[-1] <= 3 * tol)
