"""CPU checks around Lutelorn models: what the configuration reader accepts and refuses, and the float64 model that the GPU tests compare
with."""
import copy
import json

import numpy as np
import pytest

import decoder_models as dm
from oracle import lutelorn


@pytest.fixture(scope="module")
def decoder(built_library):
    from gpt_b200 import decoder as d
    return d


def text(c, **dump):
    return json.dumps(dict(c, layers=[{k: v for k, v in l.items() if k != "rank"} for l in c["layers"]]), **dump)


GOOD = dm.lutelorn([dm.attention(), dm.wkv(ff=None), dm.lightning(), dm.attention(heads=2)])


def test_configuration_is_read(decoder):
    assert decoder.check_config(text(GOOD)) == ""
    assert decoder.check_config(text(GOOD, indent=1)) == ""
    for layers in ([dm.wkv()], [dm.lightning(heads=1, decay=[1])], [dm.attention(softcap=None, rot=None, v_mix=False)], [dm.mamba(), dm.latent(), dm.attention()]):
        assert decoder.check_config(text(dm.lutelorn(layers))) == ""
    assert decoder.check_config(text(dm.lutelorn([dm.wkv()], bigram=None))) == ""
    assert decoder.check_config(text(dm.config([dm.attention(), dm.lightning()]))) == ""       # the layer kinds with another architecture's norms


@pytest.mark.parametrize("path,value,reason", [
    (["embedding"], {}, "scale"),
    (["embedding", "bigram", "buckets"], 0, "buckets"),
    (["embedding", "bigram", "mul_prev"], -1, "mul_prev"),
    (["embedding", "bigram", "mul_cur"], 1.5, "mul_cur"),
    (["residual_mult"], None, "residual_mult"),
    (["norm"], {}, "eps"),
    (["layers", 0, "mixer", "kv_heads"], 3, "kv_heads"),
    (["layers", 0, "mixer", "softcap"], -2.0, "softcap"),
    (["layers", 0, "mixer", "rot", "dims"], 26, "rotated"),
    (["layers", 0, "mixer", "rot", "dims"], 5, "rotary"),
    (["layers", 0, "mixer", "v_mix"], 1, "v_mix"),
    (["layers", 3, "mixer", "vdim"], 24, "v_mix"),
    (["layers", 1, "mixer", "dim"], 0, "dim"),
    (["layers", 2, "mixer", "decay"], [0.5], "decay"),
    (["layers", 2, "mixer", "decay"], [0.5, 1.5, 0.1], "decay"),
    (["layers", 2, "mixer", "decay"], [0.5, "x", 0.1], "decay"),
    (["layers", 1, "type"], "rwkv", "layer 1"),
    (["layers", 2, "mlp", "kind"], "experts", "experts"),
])
def test_configurations_that_do_not_fit_are_refused_with_a_reason(decoder, path, value, reason):
    c = copy.deepcopy(GOOD)
    at = c
    for k in path[:-1]:
        at = at[k]
    at[path[-1]] = value
    assert reason in decoder.check_config(text(c))


def test_wkv_needs_its_architecture(decoder):
    assert "wkv" in decoder.check_config(text(dm.config([dm.wkv()])))


# ---- the float64 model itself
def test_recurrences_against_their_closed_forms():
    rng = np.random.default_rng(0)
    T, H, d, e = 11, 2, 3, 4
    q, k, v = rng.standard_normal((T, H, d)), rng.standard_normal((T, H, d)), rng.standard_normal((T, H, e))
    decay, w, u = rng.uniform(0.2, 1, H), rng.uniform(0.2, 1, (T, H, d)), rng.standard_normal((H, d))
    a, b = lutelorn.decayed_outer_products(q, k, v, decay), lutelorn.bonus_recurrence(q, k, v, w, u)
    for t in range(T):
        for h in range(H):
            np.testing.assert_allclose(a[t, h], sum(decay[h] ** (t - s) * (q[t, h] @ k[s, h]) * v[s, h] for s in range(t + 1)), rtol=1e-10)
            want = (q[t, h] * u[h]) @ k[t, h] * v[t, h]
            for s in range(t):
                want = want + (q[t, h] * np.prod(w[s + 1:t, h], axis=0)) @ k[s, h] * v[s, h]
            np.testing.assert_allclose(b[t, h], want, rtol=1e-10)


def test_rotation_turns_neighbours_and_depends_on_distance_only():
    rng = np.random.default_rng(1)
    rot = dict(dims=6, base=50.0)
    q, k = np.tile(rng.standard_normal(8), (20, 1, 1)), np.tile(rng.standard_normal(8), (20, 1, 1))
    s = lutelorn.rotate_neighbours(q, rot)[:, 0] @ lutelorn.rotate_neighbours(k, rot)[:, 0].T
    for d in range(5):
        np.testing.assert_allclose(np.diagonal(s, -d), s[d, 0], rtol=1e-9)
    x = np.zeros((3, 1, 8))
    x[:, 0, 2] = 1.0
    y = lutelorn.rotate_neighbours(x, rot)
    a = 2 * 50.0 ** (-2 / 6)
    np.testing.assert_allclose(y[2, 0], [0, 0, np.cos(a), np.sin(a), 0, 0, 0, 0], atol=1e-15)


def test_pair_rows_cap_and_norm_by_hand():
    assert list(lutelorn.bigram_rows([3, 5, 2], 7, 10, 4)) == [7, (30 + 20) % 7, (50 + 8) % 7]
    np.testing.assert_allclose(lutelorn.offset_norm(np.array([3.0, 4.0]), np.array([0.0, 1.0]), 0.0), np.array([3.0, 8.0]) / np.sqrt(12.5))
    q, k, v = np.array([[0.0], [100.0]]), np.array([[1.0], [-1.0]]), np.array([[1.0], [0.0]])
    np.testing.assert_allclose(lutelorn.capped_attention(q, k, v, 1.0, 2.0)[1], np.exp(2.0) / (np.exp(2.0) + np.exp(-2.0)))
    np.testing.assert_allclose(lutelorn.mixed_values(4.0, 8.0, 0.25), 5.0)


@pytest.mark.parametrize("name,change", [
    ("pair", lambda w: w["bigram"][:-1].fill(0)), ("first pair", lambda w: w["bigram"][-1].fill(0)), ("q bias", lambda w: w["l0.mix.q.b"].fill(0)),
    ("v bias", lambda w: w["l0.mix.v.b"].fill(0)), ("attention gate", lambda w: w["l0.mix.g"].fill(0)), ("value share", lambda w: w["l3.mix.vmix"].fill(0)),
    ("bonus", lambda w: w["l1.mix.u"].fill(0)), ("decay map", lambda w: w["l1.mix.w2"].fill(0)), ("decay offset", lambda w: w["l1.mix.w0"].fill(-2)),
    ("shares of the previous token", lambda w: [w["l1.mix.mu." + x].fill(0) for x in "rkvgw"]), ("head norm", lambda w: w["l1.mix.norm"].fill(1)),
    ("lightning gate", lambda w: w["l2.mix.g"].fill(0)), ("norm weight", lambda w: w["l2.norm1"].fill(0)),
])
def test_test_weights_make_every_mechanism_show(name, change):
    """Leaving a mechanism out changes the logits by more than the tolerance of the GPU tests in 32 bit allows by far."""
    w = dm.weights(GOOD, 2)
    tokens = np.random.default_rng(3).integers(0, GOOD["vocab"], 12)
    want = lutelorn.forward(GOOD, w, tokens)
    broken = {k: v.copy() for k, v in w.items()}
    change(broken)
    assert dm.error(lutelorn.forward(GOOD, broken, tokens), want) > 0.01
