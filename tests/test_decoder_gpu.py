"""Decoder models on the GPU against the plain float64 model of the same equations (oracle/budurax.py)."""
import numpy as np
import pytest

import decoder_models as dm
from decoder_models import load, whole
from oracle import budurax

pytestmark = pytest.mark.gpu

TOL = {"float32": 2e-5, "bfloat16": 3e-2}
DTYPES = ["float32", "bfloat16"]

MIXED = dm.config([dm.mamba(), dm.latent(scaling=dm.YARN), dm.mamba(heads=6, vdim=8, state=24, groups=3, conv=2, norm_groups=4, ff=None),
                   dm.latent(heads=5, dim=8, rot_dim=16, vdim=16, kv_rank=40, scaling=dm.YARN, kv_from=1, ff=40)])

# each mechanism and size in a model of its own: (layers, overrides of the weights, other configuration)
ZERO_SIDE = {"side.norm": 0.0}
CASES = {
    "mamba": ([dm.mamba(ff=None)], {}, {}),
    "mamba_one_group_one_tap": ([dm.mamba(heads=3, vdim=24, state=8, groups=1, conv=1, norm_groups=1)], {}, {}),
    "mamba_groups_equal_heads": ([dm.mamba(heads=4, vdim=32, state=40, groups=4, conv=6, norm_groups=4)], {}, {}),
    "mamba_odd_sizes": ([dm.mamba(heads=2, vdim=7, state=5, groups=2, conv=3, norm_groups=2, ff=33)], {}, dict(width=37, vocab=53, side=5)),
    "mamba_wide_head": ([dm.mamba(heads=2, vdim=64, state=128, groups=1, conv=4, norm_groups=1)], {}, {}),
    "latent": ([dm.latent(ff=None)], {}, {}),
    "latent_yarn": ([dm.latent(scaling=dict(factor=8.0, original=32, fast=4.0, slow=1.0))], {}, {}),
    "latent_peaked": ([dm.latent(scale=2.0)], {}, {}),
    "latent_odd_sizes": ([dm.latent(heads=1, dim=5, rot_dim=6, vdim=3, kv_rank=11, ff=17)], {}, dict(width=41, vocab=67, side=3)),
    "latent_wide": ([dm.latent(heads=2, dim=64, rot_dim=32, vdim=72, kv_rank=200)], {}, {}),
    "latent_shared_keys": ([dm.latent(), dm.mamba(), dm.latent(heads=2, vdim=8, dim=24, kv_from=0), dm.latent(heads=4, kv_from=0)], {}, {}),
    "no_feed_forward": ([dm.mamba(ff=None), dm.latent(ff=None)], {}, {}),
    "token_shift_only": ([dm.mamba(), dm.latent()], {"shift": 1.0}, {}),
    "no_token_shift": ([dm.mamba(), dm.latent()], {"shift": 0.0}, {}),
    "depth_average_of_embedding": ([dm.mamba(), dm.latent(), dm.mamba()], {"dwa": "first"}, {}),
    "token_side_strong": ([dm.mamba(), dm.latent()], {"side.norm": 3.0}, {}),
    "large_eps": ([dm.mamba(), dm.latent()], {}, dict(eps=0.5)),
    "mixed": (MIXED["layers"], {}, {}),
}


def build(layers, overrides, other, seed=1):
    c = dm.config(layers, **other)
    w = dm.weights(c, seed)
    for key, value in overrides.items():
        for name in w:
            if name.split(".", 1)[-1] == key:
                w[name] = np.eye(1, len(w[name]))[0].astype(np.float32) if isinstance(value, str) else np.full_like(w[name], value)
    return c, w


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CASES))
def test_mechanism_prompt_and_portions(tmp_path, name, dtype):
    c, w = build(*CASES[name])
    tokens = np.random.default_rng(7).integers(0, c["vocab"], 45)
    want = budurax.forward(c, w, tokens)
    model = load(tmp_path, c, w, dtype)
    for cuts in ((1 << 20,), (30, 1), (2, 3, 2)):
        got = whole(model, tokens, cuts)
        assert np.isfinite(got).all()
        assert dm.close(got, want, TOL[dtype]), (name, cuts)
    model.close_model()


@pytest.mark.parametrize("dtype", DTYPES)
def test_prompt_against_decoding_and_portions_of_many_sizes(tmp_path, dtype):
    """300 tokens: longer than any tile, chunk or group of rows of the kernels; the same logits however the prompt is cut."""
    c, w = build(MIXED["layers"], {}, {}, 3)
    tokens = np.random.default_rng(8).integers(0, c["vocab"], 300)
    want = budurax.forward(c, w, tokens)
    model = load(tmp_path, c, w, dtype)
    base = whole(model, tokens)
    assert dm.close(base, want, TOL[dtype])
    for cuts in ((1,), (2,), (17, 64, 5), (63, 65, 2), (128, 129, 8, 9), (256, 3)):
        got = whole(model, tokens, cuts)
        assert dm.close(got, want, TOL[dtype]), cuts
    model.set_option("pass_rows", 70)      # the step itself works in passes
    assert dm.close(whole(model, tokens), want, TOL[dtype])
    model.set_option("pass_rows", 4096)
    model.set_option("segment_tokens", 64)  # segments of one chunk side by side
    for cuts in ((1 << 20,), (130, 100, 70)):
        assert dm.close(whole(model, tokens, cuts), want, TOL[dtype]), cuts
    model.close_model()


@pytest.mark.parametrize("layers", [
    [dm.latent(heads=2, dim=128, rot_dim=64, vdim=128, kv_rank=96)], [dm.latent(heads=1, dim=192, rot_dim=64, vdim=80, kv_rank=520)], [dm.latent(heads=2, dim=48, vdim=136, kv_rank=72)],
    [dm.latent(heads=18, dim=8, rot_dim=8, vdim=8, kv_rank=24)], [dm.mamba(heads=2, vdim=64, state=128, groups=1, norm_groups=1), dm.mamba(heads=2, vdim=40, state=136, groups=2, norm_groups=1)],
], ids=["deep heads", "one stage", "wide values", "many heads", "large states"])
def test_large_heads_and_states(tmp_path, layers):
    """Sizes that take other rings, fragments and fallbacks of the kernels, over several key blocks and chunks."""
    c, w = build(layers, {}, {}, 24)   # weights without rows that bf16 rounding alone moves far (single heads that nearly cancel before a norm)
    tokens = np.random.default_rng(22).integers(0, c["vocab"], 330)
    want = budurax.forward(c, w, tokens)
    for dtype in DTYPES:
        model = load(tmp_path, c, w, dtype)
        for cuts in ((1 << 20,), (200, 33, 90, 5, 1)):
            assert dm.close(whole(model, tokens, cuts), want, TOL[dtype]), (dtype, cuts)
        model.close_model()


def test_long_decoding(tmp_path):
    c, w = build(MIXED["layers"], {}, {}, 4)
    tokens = np.random.default_rng(9).integers(0, c["vocab"], 700)
    want = budurax.forward(c, w, tokens)
    model = load(tmp_path, c, w, "float32")
    assert dm.close(whole(model, tokens, (4, 1)), want, TOL["float32"])
    model.close_model()
    model = load(tmp_path, c, w, "bfloat16")
    assert dm.close(whole(model, tokens, (4, 1)), want, TOL["bfloat16"])
    model.close_model()


def far_key_model(distance):
    """One attention layer whose query at the last token (token 1) is made to match the key of one earlier token (token 0, `distance`
    back): nearly all of its weight lies there.  The embedding dominates the position through a small rotated part."""
    c = dm.config([dm.latent(heads=2, dim=32, rot_dim=8, vdim=16, kv_rank=32, scale=1.0, ff=None)], width=64, vocab=97)
    w = dm.weights(c, 5)
    w["l0.shift"][:] = 0
    w["l0.mix.q"] *= 0.2
    h = budurax.layer_norm(w["embed"], w["l0.norm1"], w["l0.norm1.b"], 1e-5)
    latent = budurax.rms_norm(h @ w["l0.mix.dkv"].T[:, :32], w["l0.mix.dkv.norm"], 1e-5)
    for n in range(2):
        key = w["l0.mix.uk"].reshape(2, 32, 32)[n] @ latent[0]
        rows = slice(n * 40, n * 40 + 32)
        w["l0.mix.q"][rows] += 14.0 * np.outer(key / (key @ key), h[1] / (h[1] @ h[1]))
    w["l0.mix.q"] = dm.bf16(w["l0.mix.q"])
    rng = np.random.default_rng(distance)
    tokens = rng.integers(2, 97, 3 + distance)
    tokens[2], tokens[-1] = 0, 1
    return c, w, tokens


@pytest.mark.parametrize("distance", [1, 2, 15, 16, 31, 32, 63, 64, 65, 127, 128, 129, 500, 1030])
def test_far_key(tmp_path, distance):
    c, w, tokens = far_key_model(distance)
    want = budurax.forward(c, w, tokens)
    without = tokens.copy()
    without[2] = 50
    assert dm.error(budurax.forward(c, w, without)[-1:], want[-1:]) > 0.2       # the last row does depend on that one token
    for dtype in DTYPES:
        model = load(tmp_path, c, w, dtype)
        n = len(tokens)
        for cuts in ((1 << 20,), (n - 1, 1), (3, 1 << 20), (max(n - 2, 1), 2)):
            assert dm.close(whole(model, tokens, cuts)[-1:], want[-1:], TOL[dtype]), (dtype, cuts)
        model.close_model()


@pytest.mark.parametrize("dtype", DTYPES)
def test_state_over_a_long_silence(tmp_path, dtype):
    """Slow decays: what one token wrote into the recurrent state must still be there hundreds of tokens later, across portions."""
    c, w = build([dm.mamba(conv=3)], {"mix.dt_bias": -4.0, "mix.A_log": -6.0}, {}, 6)
    rng = np.random.default_rng(10)
    tokens = rng.integers(0, c["vocab"], 420)
    other = tokens.copy()
    other[:20] = rng.integers(0, c["vocab"], 20)
    want = budurax.forward(c, w, tokens)
    assert dm.error(budurax.forward(c, w, other)[-1:], want[-1:]) > 3 * TOL["float32"]
    model = load(tmp_path, c, w, dtype)
    for cuts in ((1 << 20,), (64, 64, 64, 1), (100, 7)):
        assert dm.close(whole(model, tokens, cuts), want, TOL[dtype]), cuts
    model.close_model()


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens(tmp_path, dtype):
    c, w = build(MIXED["layers"], {}, {}, 11)
    model = load(tmp_path, c, w, dtype)
    for n in (1, 2, 3, 4, 5):
        tokens = np.random.default_rng(n).integers(0, c["vocab"], n)
        want = budurax.forward(c, w, tokens)
        assert dm.close(whole(model, tokens), want, TOL[dtype])
        assert dm.close(whole(model, tokens, (1,)), want, TOL[dtype])
    model.close_model()


@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_requests_in_one_step_and_reused_slots(tmp_path, dtype):
    c, w = build(MIXED["layers"], {}, {}, 12)
    rng = np.random.default_rng(13)
    model = load(tmp_path, c, w, dtype)
    texts = [rng.integers(0, c["vocab"], n) for n in (70, 1, 9, 200, 33)]
    want = [budurax.forward(c, w, t) for t in texts]
    first = whole(model, texts[3], (150, 1), 200)        # leaves a used slot behind
    assert dm.close(first, want[3], TOL[dtype])
    seqs = [model.open(len(t)) for t in texts]
    got, at = [[] for _ in texts], [0] * len(texts)
    while any(a < len(t) for a, t in zip(at, texts)):
        entries, owners = [], []
        for i, t in enumerate(texts):
            n = min(int(rng.integers(1, 40)), len(t) - at[i])
            if n:
                entries.append((seqs[i], t[at[i]:at[i] + n]))
                owners += [i] * n
                at[i] += n
        rows = model.step(entries, range(len(owners)))
        for o, r in zip(owners, rows):
            got[o].append(r)
        for i, t in enumerate(texts):                    # a finished request's slot goes to a new one at once
            if at[i] == len(t) and seqs[i] is not None:
                assert model.length(seqs[i]) == len(t)
                model.close(seqs[i])
                seqs[i] = None
    for g, x in zip(got, want):
        assert dm.close(np.stack(g), x, TOL[dtype])
    assert dm.close(whole(model, texts[0]), want[0], TOL[dtype])
    model.close_model()


def test_float32_weights_and_wanted_rows(tmp_path):
    c, w = build(MIXED["layers"], {}, {}, 14)
    tokens = np.random.default_rng(15).integers(0, c["vocab"], 90)
    want = budurax.forward(c, w, tokens)
    from gpt_b200 import serving
    model = serving.load_model(dm.save(tmp_path / "f32", c, w, "F32"), "float32")
    seq = model.open(90)
    rows = [0, 1, 5, 6, 7, 50, 89, 20]
    model.set_option("pass_rows", 32)
    assert dm.close(model.step([(seq, tokens)], rows), want[rows], TOL["float32"])
    model.close_model()


def test_errors_leave_the_model_usable(tmp_path):
    from gpt_b200 import GptB200Error
    c, w = build(MIXED["layers"], {}, {}, 16)
    model = load(tmp_path, c, w, "bfloat16")
    seq = model.open(8)
    with pytest.raises(GptB200Error):
        model.step([(seq, [1] * 9)], [0])                # more than the slot holds
    with pytest.raises(GptB200Error):
        model.step([(seq, [c["vocab"]])], [0])           # not a token
    with pytest.raises(GptB200Error):
        model.step([(seq + 1, [1])], [0])                # not open
    with pytest.raises(GptB200Error):
        model.step([(seq, [1]), (seq, [2])], [0])        # twice
    with pytest.raises(GptB200Error):
        model.generate([seq], [1], 9)
    tokens = np.arange(8) % c["vocab"]
    assert dm.close(model.step([(seq, tokens)], range(8)), budurax.forward(c, w, tokens), TOL["bfloat16"])
    model.close(seq)
    with pytest.raises(GptB200Error):
        model.step([(seq, [1])], [0])
    model.close_model()
    broken = dict(w)
    del broken["l1.mix.uk"]
    with pytest.raises(GptB200Error, match="l1.mix.uk"):
        load(tmp_path, c, broken, "bfloat16")


def greedy(c, w, prompt, n):
    tokens = list(prompt)
    margins = []
    for _ in range(n):
        lg = budurax.forward(c, w, tokens)[-1]
        top = np.sort(lg)[-2:]
        margins.append(top[1] - top[0])
        tokens.append(int(np.argmax(lg)))
    return tokens[len(prompt):], min(margins)


def test_greedy_generation_through_the_scheduler(tmp_path):
    from gpt_b200 import serving
    c, w = build(MIXED["layers"], {}, {}, 17)
    w["head"] *= 4
    rng = np.random.default_rng(18)
    prompts = [list(map(int, rng.integers(0, c["vocab"], n))) for n in (5, 1, 40, 23)]
    want = [greedy(c, w, p, 24) for p in prompts]
    assert min(m for _, m in want) > 1e-3                # no near-ties that fp32 rounding could turn over
    model = load(tmp_path, c, w, "float32")
    for options in (dict(), dict(max_sequences=2, step_tokens=16, burst=4), dict(max_sequences=1, burst=1)):
        assert serving.generate(model, prompts, 24, **options) == [t for t, _ in want], options
    model.close_model()


def test_generation_loop_equals_single_steps(tmp_path):
    """The graph-replayed loop (tokens sampled on the device) and one step at a time give the same tokens; sampling follows its seed."""
    c, w = build(MIXED["layers"], {}, {}, 19)
    prompts = [np.random.default_rng(20 + i).integers(0, c["vocab"], n) for i, n in enumerate((6, 31))]
    for dtype in DTYPES:
        model = load(tmp_path, c, w, dtype)

        def start():
            seqs = [model.open(80) for _ in prompts]
            lg = model.step([(s, p) for s, p in zip(seqs, prompts)], [len(prompts[0]) - 1, len(prompts[0]) + len(prompts[1]) - 1])
            return seqs, [int(t) for t in lg.argmax(-1)]
        seqs, first = start()
        loop = np.concatenate([model.generate(seqs, first, 20), ])
        loop = np.concatenate([loop, model.generate(seqs, loop[-1], 13)])      # the loop goes on where it stopped
        assert [model.length(s) for s in seqs] == [len(p) + 33 for p in prompts]
        for s in seqs:
            model.close(s)
        seqs, tok = start()
        for i in range(33):
            tok = [int(t) for t in model.step([(s, [t]) for s, t in zip(seqs, tok)], [0, 1]).argmax(-1)]
            assert tok == list(loop[i]), (dtype, i)
        for s in seqs:
            model.close(s)
        draws = []
        for seed in (1, 1, 2):
            seqs, first = start()
            draws.append(model.generate(seqs, first, 16, temperature=1.5, seed=seed).tolist())
            for s in seqs:
                model.close(s)
        assert draws[0] == draws[1] != draws[2]
        model.close_model()


def test_sampling_follows_the_softmax():
    import ctypes
    import torch
    import gpt_b200
    from gpt_b200 import decoder
    lib, be = decoder.load_library(), gpt_b200.Backend(0, torch.cuda.current_stream().cuda_stream)
    probs = torch.tensor([0.5, 0.25, 0.125, 0.0625, 0.0625], dtype=torch.float64)
    rows = 40000
    logits = torch.full((rows, 8), 1e9, device="cuda")                       # the padding columns are not tokens
    logits[:, :5] = (1.7 * probs.log()).float()
    out = torch.empty(rows, dtype=torch.int32, device="cuda")
    assert lib.gptb200_sample_rows(be.handle, ctypes.c_void_p(out.data_ptr()), ctypes.c_void_p(logits.data_ptr()), rows, 5, 8, 1.7, 3, 0) == 0
    be.synchronize()
    got = torch.bincount(out.long().cpu(), minlength=5).double() / rows
    assert (got - probs).abs().max() < 0.012
    logits[:, 3] = 7.0
    logits[:, 4] = 7.0
    assert lib.gptb200_sample_rows(be.handle, ctypes.c_void_p(out.data_ptr()), ctypes.c_void_p(logits.data_ptr()), rows, 5, 8, 0.0, 3, 0) == 0
    be.synchronize()
    assert (out == 3).all()                                                  # the first of equals
    be.close()



def test_gpt2_is_served_by_the_same_entry_points(tmp_path):
    """The GPT-2 model through the registry, the scheduler and the trace surface: the same tokens as recomputing the prefix."""
    import json
    import torch
    import gpt_b200
    from gpt_b200 import serving
    cfg = dict(max_seq_len=64, vocab_size=97, vocab_size_padded=128, num_layers=2, num_heads=2, d_model=64, d_ffn=128)
    m = gpt_b200.Model(cfg, use_grad=False, seed=5)
    m.init(0.0, 0.3)
    (tmp_path / "gpt2").mkdir()
    m.save_checkpoint(str(tmp_path / "gpt2" / "model.bin"))
    (tmp_path / "gpt2" / "config.json").write_text(json.dumps(dict(architecture="GPT2", **cfg)))
    prompt = [3, 50, 7, 96, 11]
    tokens = list(prompt)
    for _ in range(12):
        m.set_size(1, len(tokens))
        m.forward(torch.tensor(tokens, dtype=torch.int32, device="cuda"))
        m.synchronize()

        class _Raw:
            __cuda_array_interface__ = dict(shape=(len(tokens), 128), typestr="<f4", data=(m.logits_ptr, False), version=3, strides=None)
        tokens.append(int(torch.as_tensor(_Raw(), device="cuda")[-1, :97].argmax()))
    m.close()
    model = serving.load_model(str(tmp_path / "gpt2"), "float32")
    assert serving.generate(model, [prompt, prompt], 12) == [tokens[5:]] * 2
    model.close_model()
