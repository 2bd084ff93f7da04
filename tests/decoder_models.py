"""Small random Budurax models for the tests: configuration, weights, the folder that the library loads."""
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


def weights(c, seed=0):
    """Random weights, every parameter away from its neutral value, rounded to bf16."""
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
        json.dump(c, f)
    header, blobs, at = {}, [], 0
    for name, a in w.items():
        a = np.ascontiguousarray(a, np.float32)
        data = (a.view(np.uint32) >> 16).astype(np.uint16).tobytes() if dtype == "BF16" else a.tobytes()
        header[name] = dict(dtype=dtype, shape=list(a.shape), data_offsets=[at, at + len(data)])
        blobs.append(data)
        at += len(data)
    text = json.dumps(header).encode()
    text += b" " * (-len(text) % 8)
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(text)) + text + b"".join(blobs))
    return str(folder)


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
