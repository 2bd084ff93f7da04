"""Lutelorn models on the GPU against the plain float64 model of the same equations (oracle/lutelorn.py)."""
import numpy as np
import pytest

import decoder_models as dm
from decoder_models import load, whole
from oracle import lutelorn
from oracle.budurax import silu

pytestmark = pytest.mark.gpu

TOL = {"float32": 2e-5, "bfloat16": 3e-2}
DTYPES = ["float32", "bfloat16"]
PROMPT = (1 << 20,)

MIXED = [dm.attention(), dm.wkv(ff=None), dm.lightning(), dm.attention(heads=6, kv_heads=2, dim=16, vdim=20, softcap=5.0, rot=16, base=500.0, ff=40),
         dm.wkv(heads=2, dim=16, rank=5), dm.lightning(heads=2, dim=24, vdim=16, ff=None), dm.attention(heads=2, kv_heads=1, vdim=8, v_mix=False, rot=6, ff=None)]

# each mechanism and size in a model of its own: (layers, overrides of the weights, other configuration)
CASES = {
    "attention": ([dm.attention(v_mix=False, ff=None)], {}, {}),
    "attention_all_dimensions_rotated": ([dm.attention(rot=24)], {}, {}),
    "attention_not_rotated": ([dm.attention(rot=None)], {}, {}),
    "attention_uncapped": ([dm.attention(softcap=None, scale=0.4)], {}, {}),
    "attention_tight_cap": ([dm.attention(softcap=1.5, scale=2.0)], {}, {}),
    "attention_heads_of_their_own": ([dm.attention(heads=3, kv_heads=3, dim=8, vdim=8, rot=2)], {}, {}),
    "attention_one_key_head": ([dm.attention(heads=5, kv_heads=1, dim=16, vdim=32)], {}, {}),
    "attention_many_query_heads": ([dm.attention(heads=40, kv_heads=2, dim=8, vdim=8, rot=4)], {}, {}),
    "attention_odd_sizes": ([dm.attention(heads=3, kv_heads=1, dim=7, vdim=5, rot=4, ff=33)], {}, dict(width=37, vocab=53)),
    "attention_wide_values": ([dm.attention(heads=2, kv_heads=1, dim=40, vdim=200, rot=8)], {}, {}),
    "attention_wide_heads": ([dm.attention(heads=2, kv_heads=2, dim=256, vdim=112, rot=64, scale=0.08)], {}, {}),
    "attention_no_biases": ([dm.attention()], {"mix.q.b": 0.0, "mix.k.b": 0.0, "mix.v.b": 0.0}, {}),
    "attention_key_bias": ([dm.attention()], {"mix.k.b": 3.0}, {}),
    "value_mix": ([dm.attention(), dm.attention(heads=2), dm.attention(heads=6)], {}, {}),
    "value_mix_of_the_first": ([dm.attention(), dm.attention()], {"mix.vmix": 1.0}, {}),
    "value_mix_starts_late": ([dm.attention(v_mix=False, vdim=8), dm.lightning(), dm.attention(), dm.attention(v_mix=False, vdim=32), dm.attention()], {}, {}),
    "lightning": ([dm.lightning(ff=None)], {}, {}),
    "lightning_extreme_decays": ([dm.lightning(heads=4, decay=[0.0, 1.0, 0.999, 1e-30])], {}, {}),
    "lightning_odd_sizes": ([dm.lightning(heads=3, dim=7, vdim=5, ff=17)], {}, dict(width=41, vocab=67)),
    "lightning_narrow_values": ([dm.lightning(heads=5, dim=40, vdim=8)], {}, {}),
    "lightning_large_heads": ([dm.lightning(heads=2, dim=128, vdim=72)], {}, {}),
    "lightning_heads_beyond_the_chunks": ([dm.lightning(heads=2, dim=136, vdim=40)], {}, {}),
    "wkv": ([dm.wkv(ff=None)], {}, {}),
    "wkv_one_head_rank_one": ([dm.wkv(heads=1, dim=16, rank=1)], {}, {}),
    "wkv_odd_sizes": ([dm.wkv(heads=3, dim=7, rank=3, ff=33)], {}, dict(width=37, vocab=53)),
    "wkv_head_64": ([dm.wkv(heads=2, dim=64, rank=16)], {}, {}),
    "wkv_head_100": ([dm.wkv(heads=2, dim=100, rank=40)], {}, {}),
    "wkv_head_128": ([dm.wkv(heads=3, dim=128, rank=24)], {}, {}),
    "wkv_heads_beyond_the_chunks": ([dm.wkv(heads=1, dim=136, rank=9)], {}, {}),
    "wkv_strong_decays": ([dm.wkv()], {"mix.w0": 4.0}, {}),
    "wkv_strongest_decays": ([dm.wkv()], {"mix.w0": 80.0}, {}),
    "wkv_weak_decays": ([dm.wkv()], {"mix.w0": -9.0}, {}),
    "wkv_decay_follows_the_token": ([dm.wkv()], {"mix.w2": "x4"}, {}),
    "wkv_no_bonus": ([dm.wkv()], {"mix.u": 0.0}, {}),
    "wkv_previous_token_only": ([dm.wkv()], {"mix.mu.r": 1.0, "mix.mu.k": 1.0, "mix.mu.v": 1.0, "mix.mu.g": 1.0, "mix.mu.w": 1.0}, {}),
    "wkv_this_token_only": ([dm.wkv()], {"mix.mu.r": 0.0, "mix.mu.k": 0.0, "mix.mu.v": 0.0, "mix.mu.g": 0.0, "mix.mu.w": 0.0}, {}),
    "no_feed_forward": ([dm.attention(ff=None), dm.wkv(ff=None), dm.lightning(ff=None)], {}, {}),
    "no_pair_embedding": ([dm.wkv(), dm.attention()], {}, dict(bigram=None)),
    "pair_embedding_large_multipliers": ([dm.lightning()], {}, dict(bigram=(97, 2147483647, 2000000011), scale=1.0)),
    "pair_embedding_one_bucket": ([dm.lightning()], {}, dict(bigram=(1, 3, 5))),
    "whole_residual": ([dm.attention(), dm.wkv(), dm.lightning()], {}, dict(residual_mult=1.0)),
    "large_eps": ([dm.attention(), dm.wkv(), dm.lightning()], {}, dict(eps=0.5)),
    "mixed": (MIXED, {}, {}),
    "wide": ([dm.wkv(heads=6, dim=64, rank=24, ff=640), dm.attention(heads=8, kv_heads=2, dim=64, vdim=64, rot=32, ff=None), dm.lightning(heads=4, dim=64, vdim=64, ff=None)], {},
             dict(width=520, vocab=600)),
}


def build(layers, overrides, other, seed=1):
    c = dm.lutelorn(layers, **other)
    w = dm.weights(c, seed)
    for key, value in overrides.items():
        for name in w:
            if name.split(".", 1)[-1] == key:
                w[name] = w[name] * float(value[1:]) if isinstance(value, str) else np.full_like(w[name], value)
    return c, w


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CASES))
def test_mechanism_prompt_and_portions(tmp_path, name, dtype):
    c, w = build(*CASES[name])
    tokens = np.random.default_rng(7).integers(0, c["vocab"], 70)
    want = lutelorn.forward(c, w, tokens)
    model = load(tmp_path, c, w, dtype)
    for cuts in (PROMPT, (50, 1), (2, 3, 2), (33, 9, 2)):
        got = whole(model, tokens, cuts)
        assert np.isfinite(got).all()
        assert dm.close(got, want, TOL[dtype]), (name, cuts, dm.error(got, want))
    model.close_model()


@pytest.mark.parametrize("dtype", DTYPES)
def test_prompt_against_decoding_and_portions_of_many_sizes(tmp_path, dtype):
    """300 tokens: longer than any tile, chunk or group of rows of the kernels; the same logits however the prompt is cut."""
    c, w = build(MIXED, {}, {}, 3)
    tokens = np.random.default_rng(8).integers(0, c["vocab"], 300)
    want = lutelorn.forward(c, w, tokens)
    model = load(tmp_path, c, w, dtype)
    for cuts in (PROMPT, (1,), (2,), (15, 16, 17, 2), (17, 64, 5), (63, 65, 2), (128, 129, 8, 9), (256, 3)):
        got = whole(model, tokens, cuts)
        assert dm.close(got, want, TOL[dtype]), (cuts, dm.error(got, want))
    model.set_option("pass_rows", 70)             # the step itself works in passes
    assert dm.close(whole(model, tokens), want, TOL[dtype])
    model.set_option("pass_rows", 4096)
    for option in ("segment_tokens", "wkv_segment_tokens"):
        model.set_option(option, 64)              # segments of a few chunks side by side
    for cuts in (PROMPT, (130, 100, 70)):
        assert dm.close(whole(model, tokens, cuts), want, TOL[dtype]), cuts
    model.set_option("wkv_segment_tokens", 16)
    assert dm.close(whole(model, tokens), want, TOL[dtype])
    model.set_option("pair", 1)                   # every product of more than eight rows on CTA pairs
    assert dm.close(whole(model, tokens), want, TOL[dtype])
    model.set_option("pair", 0)
    for option in ("expand_rows", "chunk_rows"):
        model.set_option(option, 0x7fffffff)      # the forms for a few rows, for any number of rows
    assert dm.close(whole(model, tokens), want, TOL[dtype])
    model.close_model()


@pytest.mark.parametrize("dtype", DTYPES)
def test_wide_layers_on_every_product_kernel(tmp_path, dtype):
    c, w = build(*CASES["wide"])
    tokens = np.random.default_rng(21).integers(0, c["vocab"], 330)
    want = lutelorn.forward(c, w, tokens)
    model = load(tmp_path, c, w, dtype)
    for option, value in (("pair", 0), ("pair", 1), ("pair", -1), ("stream_k", 1), ("tile_n", 128)):
        model.set_option("pair", 0)
        model.set_option(option, value)
        for cuts in (PROMPT, (200, 33, 90, 5, 1)):
            assert dm.close(whole(model, tokens, cuts), want, TOL[dtype]), (option, value, cuts)
    model.close_model()


def test_long_decoding(tmp_path):
    c, w = build(MIXED, {}, {}, 4)
    tokens = np.random.default_rng(9).integers(0, c["vocab"], 700)
    want = lutelorn.forward(c, w, tokens)
    for dtype in DTYPES:
        model = load(tmp_path, c, w, dtype)
        assert dm.close(whole(model, tokens, (4, 1)), want, TOL[dtype]), dtype
        model.close_model()


def far_key_model(distance):
    """One attention layer whose query at the last token (token 1) is made to match the key of one earlier token (token 0, `distance`
    back): nearly all of its weight lies there, up to the cap.  Only a few weak dimensions are rotated."""
    c = dm.lutelorn([dm.attention(heads=4, kv_heads=2, dim=32, vdim=16, scale=1.0, softcap=40.0, rot=8, v_mix=False, ff=None)], width=64, vocab=97, bigram=None, residual_mult=1.0)
    w = dm.weights(c, 5)
    w["l0.mix.q"] *= 0.2
    w["l0.mix.q.b"] *= 0.0
    h = lutelorn.offset_norm(w["embed"] * 0.7, w["l0.norm1"], 1e-5)
    keys = (h[0] @ w["l0.mix.k"].T + w["l0.mix.k.b"]).reshape(2, 32)
    for n in range(4):
        key = np.concatenate([np.zeros(8), keys[n // 2][8:]])
        w["l0.mix.q"][n * 32:(n + 1) * 32] += 30.0 * np.outer(key / (key @ key), h[1] / (h[1] @ h[1]))
    w["l0.mix.q"] = dm.bf16(w["l0.mix.q"])
    tokens = np.random.default_rng(distance).integers(2, 97, 3 + distance)
    tokens[2], tokens[-1] = 0, 1
    return c, w, tokens


@pytest.mark.parametrize("distance", [1, 2, 15, 16, 17, 31, 32, 63, 64, 65, 127, 128, 129, 500, 1030])
def test_far_key(tmp_path, distance):
    c, w, tokens = far_key_model(distance)
    want = lutelorn.forward(c, w, tokens)
    without = tokens.copy()
    without[2] = 50
    assert dm.error(lutelorn.forward(c, w, without)[-1:], want[-1:]) > 0.2       # the last row does depend on that one token
    for dtype in DTYPES:
        model = load(tmp_path, c, w, dtype)
        n = len(tokens)
        for cuts in (PROMPT, (n - 1, 1), (3, 1 << 20), (max(n - 2, 1), 2)):
            assert dm.close(whole(model, tokens, cuts)[-1:], want[-1:], TOL[dtype]), (dtype, cuts)
        model.close_model()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["lightning", "wkv"])
def test_state_over_a_long_silence(tmp_path, kind, dtype):
    """Slow decays: what the first tokens wrote into a recurrent state must still be there hundreds of tokens later, across portions."""
    layer = dm.lightning(decay=[0.9995, 1.0, 0.9999]) if kind == "lightning" else dm.wkv()
    c, w = build([layer], {"mix.w0": -9.0}, dict(bigram=None), 6)
    rng = np.random.default_rng(10)
    tokens = rng.integers(0, c["vocab"], 420)
    other = tokens.copy()
    other[:20] = rng.integers(0, c["vocab"], 20)
    want = lutelorn.forward(c, w, tokens)
    assert dm.error(lutelorn.forward(c, w, other)[-1:], want[-1:]) > 3 * TOL["float32"]
    model = load(tmp_path, c, w, dtype)
    model.set_option("wkv_segment_tokens", 64)
    model.set_option("segment_tokens", 64)
    for cuts in (PROMPT, (64, 64, 64, 1), (100, 7)):
        assert dm.close(whole(model, tokens, cuts), want, TOL[dtype]), cuts
    model.close_model()


@pytest.mark.parametrize("dtype", DTYPES)
def test_one_token_remembered_by_a_state(tmp_path, dtype):
    """A recurrent layer whose state holds the key of one token only: every other token's key is (nearly) zero, and the reading token
    asks for it from the other side of chunks, segments and portions."""
    c, w = build([dm.lightning(heads=2, dim=16, vdim=16, decay=[1.0, 0.999], ff=None)], {}, dict(bigram=None, width=64, residual_mult=1.0), 8)
    h = lutelorn.offset_norm(w["embed"] * 0.7, w["l0.norm1"], 1e-5)
    # keys: silu of -20 for all tokens but token 0
    away = np.linalg.lstsq(h, np.where(np.arange(len(h)) == 0, 6.0, -20.0), rcond=None)[0]
    w["l0.mix.k"] = dm.bf16(np.tile(away, (32, 1)) * np.linspace(0.8, 1.2, 32)[:, None])
    key = silu(h @ w["l0.mix.k"].T.astype(np.float64))
    tokens = np.random.default_rng(3).integers(1, 101, 200)
    quiet = np.argsort(np.abs(key).max(1))[:30]
    tokens = quiet[tokens % 30]
    tokens[5] = 0
    want = lutelorn.forward(c, w, tokens)
    without = tokens.copy()
    without[5] = quiet[0]
    assert dm.error(lutelorn.forward(c, w, without)[-1:], want[-1:]) > 0.05
    model = load(tmp_path, c, w, dtype)
    model.set_option("segment_tokens", 64)
    for cuts in (PROMPT, (5, 1), (6, 1 << 20), (64, 64, 64, 2), (3, 2, 1)):
        assert dm.close(whole(model, tokens, cuts), want, TOL[dtype]), cuts
    model.close_model()


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens(tmp_path, dtype):
    c, w = build(MIXED, {}, {}, 11)
    w["bigram"] = w["bigram"] * 4.0               # the first token's row, then the pairs', stand out
    model = load(tmp_path, c, w, dtype)
    for n in (1, 2, 3, 4, 5, 18):
        tokens = np.random.default_rng(n).integers(0, c["vocab"], n)
        want = lutelorn.forward(c, w, tokens)
        assert dm.close(whole(model, tokens), want, TOL[dtype])
        assert dm.close(whole(model, tokens, (1,)), want, TOL[dtype])
        assert dm.close(whole(model, tokens, (1, 2)), want, TOL[dtype])
    model.close_model()


@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_requests_in_one_step_and_reused_slots(tmp_path, dtype):
    c, w = build(MIXED, {}, {}, 12)
    rng = np.random.default_rng(13)
    model = load(tmp_path, c, w, dtype)
    model.set_option("wkv_segment_tokens", 16)
    texts = [rng.integers(0, c["vocab"], n) for n in (70, 1, 9, 200, 33)]
    want = [lutelorn.forward(c, w, t) for t in texts]
    first = whole(model, texts[3], (150, 1), 200)        # leaves a used slot behind
    assert dm.close(first, want[3], TOL[dtype])
    for _ in range(2):                                   # the second time in used slots
        seqs = [model.open(len(t)) for t in texts]
        got, at = [[] for _ in texts], [0] * len(texts)
        while any(a < len(t) for a, t in zip(at, texts)):
            entries, owners = [], []
            for i, t in enumerate(texts):
                n = min(int(rng.integers(1, 60)), len(t) - at[i])
                if n:
                    entries.append((seqs[i], t[at[i]:at[i] + n]))
                    owners += [i] * n
                    at[i] += n
            rows = model.step(entries, range(len(owners)))
            for o, r in zip(owners, rows):
                got[o].append(r)
            for i, t in enumerate(texts):                # a finished request's slot goes to a new one at once
                if at[i] == len(t) and seqs[i] is not None:
                    assert model.length(seqs[i]) == len(t)
                    model.close(seqs[i])
                    seqs[i] = None
        for g, x in zip(got, want):
            assert dm.close(np.stack(g), x, TOL[dtype])
    assert dm.close(whole(model, texts[0]), want[0], TOL[dtype])
    model.close_model()


@pytest.mark.parametrize("dtype", DTYPES)
def test_requests_that_decode_together(tmp_path, dtype):
    """2 to 12 requests of unequal length, one token each per step: both product kernels for a few rows, and beyond."""
    c, w = build(MIXED, {}, {}, 15)
    rng = np.random.default_rng(16)
    model = load(tmp_path, c, w, dtype)
    for batch in (2, 8, 12):
        texts = [rng.integers(0, c["vocab"], n) for n in rng.integers(6, 150, batch)]
        want = [lutelorn.forward(c, w, t)[-5:] for t in texts]
        seqs = [model.open(len(t)) for t in texts]
        for s, t in zip(seqs, texts):
            model.step([(s, t[:-5])], [])
        got = np.stack([model.step([(s, t[k:k + 1] if k < -1 else t[k:]) for s, t in zip(seqs, texts)], range(batch)) for k in range(-5, 0)], 1)
        for g, x in zip(got, want):
            assert dm.close(g, x, TOL[dtype]), batch
        for s in seqs:
            model.close(s)
    model.close_model()


def test_float32_weights_and_wanted_rows(tmp_path):
    c, w = build(MIXED, {}, {}, 14)
    tokens = np.random.default_rng(15).integers(0, c["vocab"], 90)
    want = lutelorn.forward(c, w, tokens)
    from gpt_b200 import serving
    model = serving.load_model(dm.save(tmp_path / "f32", c, w, "F32"), "float32")
    seq = model.open(90)
    rows = [0, 1, 5, 6, 7, 50, 89, 20]
    model.set_option("pass_rows", 32)
    assert dm.close(model.step([(seq, tokens)], rows), want[rows], TOL["float32"])
    model.close_model()


def test_weights_that_do_not_fit_are_refused(tmp_path):
    from gpt_b200 import GptB200Error
    c, w = build(MIXED, {}, {}, 16)
    for name, value in (("l1.mix.w2", w["l1.mix.w2"][:, :-1]), ("bigram", w["bigram"][:-1]), ("l1.mix.mu.w", None), ("l0.mix.q.b", None), ("l1.mix.w1", w["l1.mix.w1"][0])):
        broken = dict(w)
        if value is None:
            del broken[name]
        else:
            broken[name] = value
        with pytest.raises(GptB200Error, match=name.replace("w1", "w[12]")):
            load(tmp_path, c, broken, "bfloat16")


def greedy(c, w, prompt, n):
    tokens, margins = list(prompt), []
    for _ in range(n):
        lg = lutelorn.forward(c, w, tokens)[-1]
        top = np.sort(lg)[-2:]
        margins.append(top[1] - top[0])
        tokens.append(int(np.argmax(lg)))
    return tokens[len(prompt):], min(margins)


def test_greedy_generation_through_the_scheduler(tmp_path):
    from gpt_b200 import serving
    c, w = build(MIXED, {}, {}, 17)
    w["head"] = w["head"] * 4
    rng = np.random.default_rng(18)
    prompts = [list(map(int, rng.integers(0, c["vocab"], n))) for n in (5, 1, 40, 23)]
    want = [greedy(c, w, p, 24) for p in prompts]
    assert min(m for _, m in want) > 1e-3                # no near-ties that fp32 rounding could turn over
    model = load(tmp_path, c, w, "float32")
    for options in (dict(), dict(max_sequences=2, step_tokens=16, burst=4), dict(max_sequences=1, burst=1)):
        assert serving.generate(model, prompts, 24, **options) == [t for t, _ in want], options
    model.close_model()


def test_generation_loop_equals_single_steps(tmp_path):
    """The graph-replayed loop (tokens sampled on the device) and one step at a time give the same tokens."""
    c, w = build(MIXED, {}, {}, 19)
    prompts = [np.random.default_rng(20 + i).integers(0, c["vocab"], n) for i, n in enumerate((6, 31))]
    for dtype in DTYPES:
        model = load(tmp_path, c, w, dtype)

        def start():
            seqs = [model.open(120) for _ in prompts]
            lg = model.step([(s, p) for s, p in zip(seqs, prompts)], [len(prompts[0]) - 1, len(prompts[0]) + len(prompts[1]) - 1])
            return seqs, [int(t) for t in lg.argmax(-1)]
        seqs, first = start()
        loop = model.generate(seqs, first, 50)
        loop = np.concatenate([loop, model.generate(seqs, loop[-1], 13)])      # the loop goes on where it stopped
        assert [model.length(s) for s in seqs] == [len(p) + 63 for p in prompts]
        for s in seqs:
            model.close(s)
        seqs, tok = start()
        for i in range(63):
            tok = [int(t) for t in model.step([(s, [t]) for s, t in zip(seqs, tok)], [0, 1]).argmax(-1)]
            assert tok == list(loop[i]), (dtype, i)
        model.close_model()


def test_trace_runner_replays_a_model(tmp_path):
    import json
    import os
    import subprocess
    import sys
    from conftest import ROOT
    c, w = build(MIXED, {}, {}, 23)
    folder = dm.save(tmp_path / "model", c, w)
    tokens = [int(t) for t in np.random.default_rng(24).integers(0, c["vocab"], 40)]
    want = lutelorn.forward(c, w, tokens)
    steps = [dict(step=0, entries=[dict(id="a", tokens=tokens[:30], want=[0, 29])], end=[]), dict(step=1, entries=[dict(id="a", tokens=tokens[30:32], want=[])], end=[]),
             dict(step=2, entries=[dict(id="a", tokens=tokens[32:], want=[0, 7])], end=["a"])]
    out = tmp_path / "out"
    out.mkdir()
    res = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", "float32", "--out", str(out), "--max-tokens", "40"],
                         input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert res.returncode == 0, res.stderr[-2000:]
    assert res.stdout.split("\n")[:3] == ["done 0", "done 1", "done 2"]
    got = np.concatenate([np.fromfile(out / f"{i}.f32", "<f4").reshape(2, -1) for i in (0, 2)])
    assert dm.close(got, want[[0, 29, 32, 39]], TOL["float32"])
