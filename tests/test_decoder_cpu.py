"""CPU checks of the decoder models' host side: configuration reader, rotation frequencies, registry, scheduler, trace runner -- and
of the float64 model that the GPU tests compare with."""
import copy
import importlib.machinery
import importlib.util
import io
import json
import os

import numpy as np
import pytest

import decoder_models as dm
from conftest import ROOT
from oracle import budurax


@pytest.fixture(scope="module")
def decoder(built_library):
    from gpt_b200 import decoder as d
    return d


GOOD = dm.config([dm.mamba(), dm.latent(scaling=dm.YARN), dm.mamba(ff=None), dm.latent(heads=2, scaling=dm.YARN, kv_from=1)])


def test_configuration_is_read(decoder):
    assert decoder.check_config(json.dumps(GOOD)) == ""
    assert decoder.check_config(json.dumps(GOOD, indent=3)) == ""


@pytest.mark.parametrize("path,value,reason", [
    (["architecture"], "Nothing", "unknown architecture"),
    (["width"], None, "width"),
    (["width"], 0, "width"),
    (["vocab"], 10.5, "vocab"),
    (["norm"], {}, "eps"),
    (["token_side"], {}, "dim"),
    (["layers"], [], "layers"),
    (["layers", 0, "type"], "window", "layer 0"),
    (["layers", 0, "mixer", "groups"], 3, "groups"),
    (["layers", 0, "mixer", "norm_groups"], 7, "norm_groups"),
    (["layers", 1, "mixer", "scale"], "x", "scale"),
    (["layers", 1, "mixer", "rot", "dims"], 15, "rotary"),
    (["layers", 1, "mixer", "rot", "scaling", "factor"], 0, "rotary scaling"),
    (["layers", 3, "mixer", "kv_from"], 3, "kv_from"),
    (["layers", 3, "mixer", "kv_from"], 0, "kv_from"),
    (["layers", 3, "mixer", "kv_rank"], 48, "kv_from"),
    (["layers", 0, "mlp", "kind"], "experts", "experts"),
])
def test_configurations_that_do_not_fit_are_refused_with_a_reason(decoder, path, value, reason):
    c = copy.deepcopy(GOOD)
    at = c
    for k in path[:-1]:
        at = at[k]
    at[path[-1]] = value
    assert reason in decoder.check_config(json.dumps(c))


def test_text_that_is_not_json_is_refused(decoder):
    for text in ("", "{", "[1, 2", '{"a" 1}', "{} x", '{"a": "b}', "[" * 100):
        assert decoder.check_config(text) != ""


@pytest.mark.parametrize("rot", [
    dict(dims=16, base=10000.0), dict(dims=2, base=100.0), dict(dims=64, base=1e6, scaling=dict(factor=40.0, original=4096, fast=32.0, slow=1.0)),
    dict(dims=10, base=500.0, scaling=dict(factor=1.5, original=100, fast=8.0, slow=8.0)), dict(dims=32, base=1e4, scaling=dict(factor=4.0, original=8, fast=32.0, slow=1.0)),
])
def test_rotation_frequencies(decoder, rot):
    f, gain = decoder.rotary_frequencies(rot)
    rf, rgain = budurax.rotary_frequencies(rot)
    np.testing.assert_allclose(f, rf, rtol=1e-14)
    assert gain == pytest.approx(rgain, rel=1e-14)


def test_registry_names_are_architectures_of_the_library(decoder, tmp_path):
    from gpt_b200 import serving
    assert set(serving.REGISTRY) == {"Budurax", "Lutelorn", "GPT2"}
    (tmp_path / "config.json").write_text('{"architecture": "Other"}')
    with pytest.raises(ValueError, match="Other"):
        serving.load_model(str(tmp_path))


def test_no_device_is_an_error_not_a_fallback(decoder, tmp_path):
    import torch
    if torch.cuda.is_available():
        pytest.skip("a GPU is present")
    import gpt_b200
    from gpt_b200 import serving
    folder = dm.save(tmp_path / "m", GOOD, dm.weights(GOOD))
    with pytest.raises(gpt_b200.GptB200Error) as e:
        serving.load_model(folder)
    assert e.value.status == 3


# ---- the float64 model itself
def test_recurrence_against_its_closed_form():
    """y_t = sum over s <= t of (product of the decays after s) dt_s (C_t . B_s) x_s + D x_t."""
    rng = np.random.default_rng(0)
    T, H, P, G, N = 12, 4, 3, 2, 5
    x, B, C = rng.standard_normal((T, H, P)), rng.standard_normal((T, G, N)), rng.standard_normal((T, G, N))
    dt, decay, D = rng.uniform(0.1, 1, (T, H)), rng.uniform(0.3, 1, (T, H)), rng.standard_normal(H)
    y = budurax.mamba2_recurrence(x, B, C, dt, decay, D)
    for t in range(T):
        for h in range(H):
            g = h // (H // G)
            want = D[h] * x[t, h]
            for s in range(t + 1):
                want = want + np.prod(decay[s + 1:t + 1, h]) * dt[s, h] * (C[t, g] @ B[s, g]) * x[s, h]
            np.testing.assert_allclose(y[t, h], want, rtol=1e-10)


def test_rotation_depends_on_distance_only():
    rng = np.random.default_rng(1)
    rot = dict(dims=8, base=50.0, scaling=dict(factor=2.0, original=16, fast=4.0, slow=1.0))
    q, k = np.tile(rng.standard_normal(8), (20, 1)), np.tile(rng.standard_normal(8), (20, 1))
    s = budurax.rotate(q, rot) @ budurax.rotate(k, rot).T
    for d in range(5):
        np.testing.assert_allclose(np.diagonal(s, -d), s[d, 0], rtol=1e-9)


def test_conv_shift_and_norms_by_hand():
    u, taps = np.arange(10.0).reshape(5, 2), np.array([[1.0, 2.0], [0.0, 3.0]])
    np.testing.assert_allclose(budurax.causal_conv(u, taps, np.array([0.5, 0.0]))[2], [0.5 + 1 * 2 + 2 * 4, 15.0])
    np.testing.assert_allclose(budurax.token_shift(u, np.array([1.0, 0.5]))[:2], [[0.0, 0.5], [0.0, 2.0]])
    np.testing.assert_allclose(budurax.rms_norm(np.array([3.0, 3.0, 0.0, 2.0]), 1.0, 0.0, parts=2), [1.0, 1.0, 0.0, np.sqrt(2.0)])
    np.testing.assert_allclose(budurax.layer_norm(np.array([1.0, 3.0]), 2.0, 1.0, 0.0), [-1.0, 3.0])


@pytest.mark.parametrize("name,change", [
    ("shift", lambda w: w["l0.shift"].fill(0)), ("side", lambda w: w["l0.side.norm"].fill(0)), ("dwa", lambda w: w["l2.dwa"].__setitem__(slice(0, 3), 0)),
    ("skip", lambda w: w["l0.mix.D"].fill(0)), ("gate", lambda w: w["l1.mix.g"].fill(0)), ("conv bias", lambda w: w["l0.mix.conv.b"].fill(0)),
    ("norm bias", lambda w: w["final.norm.b"].fill(0)), ("first tap", lambda w: w["l0.mix.conv"][:, 0].fill(0)),
])
def test_test_weights_make_every_mechanism_show(name, change):
    """Leaving a mechanism out changes the logits by far more than the tolerances of the GPU tests."""
    w = dm.weights(GOOD, 2)
    tokens = np.random.default_rng(3).integers(0, GOOD["vocab"], 12)
    want = budurax.forward(GOOD, w, tokens)
    broken = {k: v.copy() for k, v in w.items()}
    change(broken)
    assert dm.error(budurax.forward(GOOD, broken, tokens), want) > 0.04


# ---- scheduler and trace runner over a stand-in model
class CountingModel:
    """Next token = (sum of all tokens so far) mod vocab; records what it was given."""
    batched, vocab = True, 31

    def __init__(self):
        self.live, self.next, self.steps, self.most = {}, 0, [], 0

    def open(self, max_len):
        self.next += 1
        self.live[self.next] = [max_len, []]
        self.most = max(self.most, len(self.live))
        return self.next

    def close(self, seq):
        del self.live[seq]

    def length(self, seq):
        return len(self.live[seq][1])

    def step(self, entries, want):
        self.steps.append([len(t) for _, t in entries])
        rows = []
        for s, t in entries:
            assert len(t) and self.length(s) + len(t) <= self.live[s][0]
            for x in t:
                self.live[s][1].append(int(x))
                rows.append(np.eye(self.vocab, dtype=np.float32)[sum(self.live[s][1]) % self.vocab])
        return np.stack([rows[w] for w in want]) if len(want) else np.empty((0, self.vocab), np.float32)

    def generate(self, seqs, first, steps, temperature=0.0, seed=0):
        out = np.empty((steps, len(seqs)), np.int32)
        for i, (s, t) in enumerate(zip(seqs, first)):
            for k in range(steps):
                t = int(self.step([(s, [t])], [0])[0].argmax())
                out[k, i] = t
        return out

    def close_model(self):
        pass


def counting(prompt, n):
    t = list(prompt)
    for _ in range(n):
        t.append(sum(t) % CountingModel.vocab)
    return t[len(prompt):]


@pytest.mark.parametrize("options", [dict(), dict(max_sequences=1), dict(max_sequences=2, step_tokens=5, burst=3), dict(max_sequences=3, step_tokens=4, burst=1)])
def test_scheduler(options):
    from gpt_b200 import serving
    rng = np.random.default_rng(4)
    prompts = [list(map(int, rng.integers(0, 31, n))) for n in (7, 1, 19, 3, 12, 2)]
    m = CountingModel()
    assert serving.generate(m, prompts, 9, **options) == [counting(p, 9) for p in prompts]
    assert not m.live and m.most <= options.get("max_sequences", 8)
    assert max(sum(s) for s in m.steps) <= options.get("step_tokens", 2048)


def test_scheduler_with_requests_of_different_length():
    from gpt_b200 import serving
    m = CountingModel()
    s = serving.Scheduler(m, max_sequences=2, step_tokens=6, burst=4)
    lens = [3, 0, 8, 1]
    rs = [s.submit(serving.Request([i + 1, 2], n)) for i, n in enumerate(lens)]
    s.run()
    assert [r.output for r in rs] == [counting([i + 1, 2], n) for i, n in enumerate(lens)]
    with pytest.raises(ValueError):
        s.submit(serving.Request([], 1))


def test_sampling_on_the_host():
    from gpt_b200 import serving
    rng = np.random.default_rng(5)
    lg = np.log(np.array([0.6, 0.3, 0.1])) * 2.0
    assert serving.sample(lg, 0.0, rng) == 0
    got = np.bincount([serving.sample(lg, 2.0, rng) for _ in range(4000)], minlength=3) / 4000
    assert np.abs(got - [0.6, 0.3, 0.1]).max() < 0.04


def _trace_run():
    path = os.path.join(ROOT, "bin", "trace_run")
    assert os.access(path, os.X_OK)
    loader = importlib.machinery.SourceFileLoader("trace_run", path)
    module = importlib.util.module_from_spec(importlib.util.spec_from_loader("trace_run", loader))
    loader.exec_module(module)
    return module


def test_trace_runner(tmp_path, monkeypatch, capsys):
    run = _trace_run()
    m = CountingModel()
    monkeypatch.setattr(run.serving, "load_model", lambda folder, dtype: m)
    steps = [dict(step=0, entries=[dict(id="a", tokens=[1, 2, 3], want=[0, 2])], end=[]),
             dict(step=1, entries=[dict(id="a", tokens=[4], want=[])], end=[]),
             dict(step=2, entries=[dict(id="a", tokens=[5, 6], want=[1])], end=["a"]),
             dict(step=3, entries=[dict(id="b", tokens=[9], want=[0])], end=["b"])]
    monkeypatch.setattr("sys.stdin", io.StringIO("".join(json.dumps(s) + "\n" for s in steps)))
    monkeypatch.setattr("sys.argv", ["trace_run", "--model", "m", "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "6"])
    assert run.main() == 0
    assert capsys.readouterr().out.split("\n")[:4] == ["done 0", "done 1", "done 2", "done 3"]
    assert not m.live
    assert sorted(os.listdir(tmp_path)) == ["0.f32", "2.f32", "3.f32"]
    rows = np.fromfile(tmp_path / "0.f32", "<f4").reshape(2, 31)
    assert list(rows.argmax(-1)) == [1, 6]
    assert np.fromfile(tmp_path / "2.f32", "<f4").argmax() == 21


def test_generation_command_line(tmp_path, monkeypatch, capsys):
    from gpt_b200 import generate
    monkeypatch.setattr(generate.serving, "load_model", lambda folder, dtype: CountingModel())
    assert generate.main(["--model", "m", "--prompt", "1,2", "--prompt", "7", "--max-new-tokens", "5"]) == 0
    assert [list(map(int, line.split())) for line in capsys.readouterr().out.splitlines()] == [counting([1, 2], 5), counting([7], 5)]
