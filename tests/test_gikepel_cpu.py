"""The Gikepel decoder without a GPU: the configuration reader and weight admission, the plain restatement's own
consistency, and the sensitivity of the GPU tests' inputs to planted mistakes (planted here, in the restatement)."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest

import gikepel_cases as cases
from layered_cases import logit_error, tokens
from test_layered_cpu import write_checkpoint

ROOT = Path(__file__).resolve().parents[1]
sys.path.insert(0, str(ROOT / "oracle"))
import gikepel  # noqa: E402


# ---- configuration and admission ----
@pytest.mark.parametrize("name", sorted(cases.CASES))
def test_every_size_and_constant_comes_from_the_config(package, name):
    c = cases.CASES[name]
    shape = package.checkpoint.shape_from_config(c, "gikepel_bf16")
    assert (shape.vocab_size, shape.hidden_size, shape.n_layers) == (c["vocab"], c["width"], len(c["layers"]))
    assert shape.norm_eps == c["norm"]["eps"] and shape.logit_softcap == c["logit_softcap"] and not shape.true32
    assert shape.tied_embeddings and shape.block == package.runtime.BLOCK_PARALLEL and shape.loop is None
    pairs = c["embedding"]["bigram"]
    assert (shape.pairs.buckets, shape.pairs.mul_prev, shape.pairs.mul_cur) == (pairs["buckets"], pairs["mul_prev"], pairs["mul_cur"])
    assert package.checkpoint.shape_from_config(c, "gikepel_f32").true32
    for entry, layer in zip(c["layers"], shape.layers):
        m = entry["mixer"]
        if entry["type"] == "latent_attention":
            a, rot = layer.latent, m["rot"]
            assert all(getattr(a, key) == m[key] for key in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "scale"))
            assert (a.rot_dims, a.rot_base) == (rot["dims"], rot["base"])
            assert (a.yarn is None) == (rot["scaling"] is None)
            if a.yarn is not None:
                assert all(getattr(a.yarn, key) == rot["scaling"][key] for key in ("factor", "original", "fast", "slow"))
        elif entry["type"] == "mamba2":
            s = layer.state_space
            assert all(getattr(s, key) == m[key] for key in ("heads", "groups", "state", "vdim", "norm_groups"))
            assert s.taps == m["conv"]
        else:
            d = layer.delta
            assert all(getattr(d, key) == m[key] for key in ("heads", "kv_heads", "dim", "vdim")) and d.taps == m["conv"]
        assert layer.ff == (None if entry["mlp"] is None else entry["mlp"]["ff"])
        assert layer.mlp == package.runtime.MLP_RELU_SQUARED


def test_model_type_follows_the_config(package):
    pick = package.checkpoint.model_type_of
    assert pick({"architecture": "Gikepel"}) == "gikepel_bf16"
    assert pick({"architecture": "Gikepel"}, "float32") == "gikepel_f32"


def test_admission_checks_names_and_shapes_and_finds_the_ranks(package, tmp_path):
    c = cases.CASES["mixed"]
    weights = cases.random_weights(package, c, ranks=(11, 17))
    write_checkpoint(tmp_path, c, weights)
    loaded_config, loaded = package.checkpoint.load_directory(tmp_path)
    shape, tensors = package.checkpoint.admit(loaded_config, loaded, package.checkpoint.model_type_of(loaded_config))
    assert set(tensors) == set(weights)
    assert [(layer.delta.decay_rank, layer.delta.gate_rank) for layer in shape.layers if layer.delta] == [(11, 17)] * 2
    for name, [(kind, data)] in tensors.items():
        assert kind == 0 and np.array_equal(package.synthetic.bf16_to_float(np.asarray(data)).reshape(weights[name].shape), weights[name])
    # Norm and scale of a feed-forward that a layer does not have are passed over.
    _, spare = package.checkpoint.admit(c, {**weights, "l2.norm2": weights["l1.norm2"], "l2.ls2": weights["l1.ls2"]}, "gikepel_bf16")
    assert set(spare) == set(weights)
    for change in (lambda w: w.pop("l0.mix.a1"), lambda w: w.pop("l3.mix.conv.b"), lambda w: w.pop("bigram"),
                   lambda w: w.update({"head": w["embed"]}), lambda w: w.update({"bigram": w["bigram"][:-1]}),
                   lambda w: w.update({"l1.mix.uk": w["l1.mix.uv"]}), lambda w: w.update({"l0.mix.g2": w["l0.mix.a2"]})):
        broken = dict(weights)
        change(broken)
        with pytest.raises(ValueError):
            package.checkpoint.admit(c, broken, "gikepel_bf16")


@pytest.mark.parametrize("edit", [
    lambda c: c["layers"][1]["mixer"].pop("scale"),
    lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("slow"),
    lambda c: c["layers"][0].update(type="other"),
    lambda c: c["layers"][0]["mlp"].update(kind="experts"),
    lambda c: c["layers"][3]["mixer"].update(groups=0),
    lambda c: c["embedding"]["bigram"].update(buckets="many"),
    lambda c: c.update(logit_softcap="high"),
    lambda c: c.update(layers=[]),
])
def test_malformed_configs_are_refused(package, edit):
    c = json.loads(json.dumps(cases.CASES["mixed"]))
    edit(c)
    with pytest.raises(ValueError):
        package.checkpoint.shape_from_config(c, "gikepel_bf16")


# ---- the restatement itself ----
def test_restatement_in_portions_equals_the_whole(package):
    c = cases.CASES["mixed"]
    weights, ids = cases.random_weights(package, c), tokens(c, 41)
    whole = gikepel.GikepelOracle(c, weights).forward(ids)
    pieces, other, at = [], gikepel.GikepelOracle(c, weights), 0
    for size in (2, 7, 1, 16, 1, 14):
        pieces.append(other.forward(ids[at:at + size]))
        at += size
    assert np.abs(np.concatenate(pieces) - whole).max() < 1e-9


def test_restatement_mechanisms_against_closed_forms():
    rng = np.random.default_rng(0)
    # Convolution: the last column meets the current token, zeros before the start, history carried over.
    x, kernel = rng.standard_normal((6, 2)), rng.standard_normal((2, 3))
    out, history = gikepel.short_conv(x, kernel, np.zeros((2, 2)), np.array([1.0, -1.0]))
    assert np.allclose(out[0], x[0] * kernel[:, 2] + [1.0, -1.0])
    assert np.allclose(out[5], x[5] * kernel[:, 2] + x[4] * kernel[:, 1] + x[3] * kernel[:, 0] + [1.0, -1.0])
    assert np.allclose(history, x[4:])
    # State space: the recurrence against its attention form.
    T, H, G, N, dv = 7, 4, 2, 3, 2
    x, b, c = rng.standard_normal((T, H, dv)), rng.standard_normal((T, G, N)), rng.standard_normal((T, G, N))
    dt, a_log, skip = rng.uniform(0.1, 1.0, (T, H)), rng.uniform(-1, 1, H), rng.standard_normal(H)
    out, _ = gikepel.state_space(x, b, c, dt, a_log, skip, np.zeros((H, N, dv)))
    for h in range(H):
        cumulative = np.cumsum(-np.exp(a_log[h]) * dt[:, h])
        weight = np.tril(np.exp(cumulative[:, None] - cumulative[None]) * (c[:, h // 2] @ b[:, h // 2].T) * dt[:, h][None])
        assert np.allclose(out[:, h], weight @ x[:, h] + skip[h] * x[:, h])
    # Delta rule: with full strength and no decay a key's value is replaced by the new one.
    k = gikepel.unit(rng.standard_normal((1, 1, 4)))
    v = rng.standard_normal((2, 1, 3))
    keys = np.concatenate([k, k])
    out, state = gikepel.channel_delta(keys, keys, v, np.zeros((2, 1, 4)), np.ones((2, 1)), np.zeros((1, 4, 3)))
    assert np.allclose(out[:, 0], v[:, 0], atol=1e-5) and np.allclose(state[0].T @ k[0, 0], v[1, 0], atol=1e-5)
    # Rotation: scores depend on the distance, lengths grow by the factor, neighbours form the pairs.
    frequencies, length = gikepel.yarn(8, 100.0, {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0})
    x, y = rng.standard_normal((1, 1, 8)), rng.standard_normal((1, 1, 8))
    score = [float((gikepel.rotate_pairs(x, [p + 5], frequencies, length) * gikepel.rotate_pairs(y, [p], frequencies, length)).sum())
             for p in (0, 11, 400)]
    assert np.allclose(score, score[0])
    assert np.isclose(np.linalg.norm(gikepel.rotate_pairs(x, [9], frequencies, length)), length * np.linalg.norm(x))
    turned = gikepel.rotate_pairs(np.array([[[1.0, 0.0, 0.0, 0.0]]]), [1], np.array([0.5, 0.1]), 1.0)[0, 0]
    assert np.allclose(turned, [np.cos(0.5), np.sin(0.5), 0, 0])
    # Frequencies: the fastest stay, the slowest are divided by the factor; without scaling all stay.
    plain = 100.0 ** (-2.0 * np.arange(4) / 8)
    assert np.isclose(frequencies[0], plain[0]) and np.isclose(frequencies[-1], plain[-1] / 4.0)
    assert np.allclose(gikepel.yarn(8, 100.0, None)[0], plain) and gikepel.yarn(8, 100.0, None)[1] == 1.0
    # Latent attention is attention over the expanded keys and values.
    latent, up_key, up_value = rng.standard_normal((5, 3)), rng.standard_normal((2, 4, 3)), rng.standard_normal((2, 2, 3))
    q = rng.standard_normal((1, 2, 4))
    out = gikepel.latent_attention(q, np.zeros((1, 2, 2)), latent, np.ones((5, 2)), up_key, up_value, 0.3, 4)
    for h in range(2):
        weight = np.exp(0.3 * (latent @ up_key[h].T) @ q[0, h])
        assert np.allclose(out[0, h], (weight / weight.sum()) @ (latent @ up_value[h].T))
    assert gikepel.bigram_rows(None, [3, 4], 10, 7, 2).tolist() == [10, (3 * 7 + 4 * 2) % 10]
    assert gikepel.bigram_rows(5, [3], 10, 7, 2).tolist() == [(5 * 7 + 3 * 2) % 10]


def wrap(name, change):
    return lambda m: m.setattr(gikepel, name, change(getattr(gikepel, name)))


MISTAKES = {
    "sees the next key": wrap("latent_attention", lambda f: lambda q, r, c, k, uk, uv, s, first: f(q, r, c, k, uk, uv, s, first + 1)),
    "keys one token late": wrap("latent_attention", lambda f: lambda q, r, c, k, uk, uv, s, first: f(q, r, np.roll(c, 1, 0), np.roll(k, 1, 0), uk, uv, s, first)),
    "lost first latent": wrap("latent_attention", lambda f: lambda q, r, c, k, uk, uv, s, first: f(q, r, np.concatenate([c[:1] * 0, c[1:]]), k, uk, uv, s, first)),
    "scale times the square of the length factor": wrap("latent_attention", lambda f: lambda q, r, c, k, uk, uv, s, first: f(q, r, c, k, uk, uv, s * 1.87, first)),
    "no rotated part": wrap("latent_attention", lambda f: lambda q, r, c, k, uk, uv, s, first: f(q, r * 0, c, k, uk, uv, s, first)),
    "halves instead of neighbours": wrap("rotate_pairs", lambda f: lambda x, p, w, l: f(x.reshape(x.shape[:-1] + (2, -1)).swapaxes(-1, -2).reshape(x.shape), p, w, l)),
    "no rotation": wrap("rotate_pairs", lambda f: lambda x, p, w, l: l * x),
    "query one position on": wrap("rotate_pairs", lambda f: lambda x, p, w, l: f(x, p + (x.shape[1] > 1) * 3, w, l)),
    "no length factor": wrap("rotate_pairs", lambda f: lambda x, p, w, l: f(x, p, w, 1.0)),
    "plain frequencies": wrap("yarn", lambda f: lambda d, b, s: (f(d, b, None)[0], f(d, b, s)[1])),
    "convolution reversed": wrap("short_conv", lambda f: lambda x, k, h, b=None: f(x, k[:, ::-1], h, b)),
    "lost convolution history": wrap("short_conv", lambda f: lambda x, k, h, b=None: f(x, k, h * 0, b)),
    "no convolution bias": wrap("short_conv", lambda f: lambda x, k, h, b=None: f(x, k, h)),
    "lost state-space state": wrap("state_space", lambda f: lambda x, b, c, dt, a, d, s: f(x, b, c, dt, a, d, s * 0)),
    "no skip": wrap("state_space", lambda f: lambda x, b, c, dt, a, d, s: f(x, b, c, dt, a, d * 0, s)),
    "interleaved groups": wrap("state_space", lambda f: lambda x, b, c, dt, a, d, s: f(x, b[:, ::-1], c[:, ::-1], dt, a, d, s)),
    "B and C exchanged": wrap("state_space", lambda f: lambda x, b, c, dt, a, d, s: f(x, c, b, dt, a, d, s)),
    "lost delta state": wrap("channel_delta", lambda f: lambda q, k, v, g, b, s: f(q, k, v, g, b, s * 0)),
    "no delta": wrap("channel_delta", lambda f: lambda q, k, v, g, b, s: f(q, k, v, g, b * 0 + 1.0, s)),
    "one decay per head": wrap("channel_delta", lambda f: lambda q, k, v, g, b, s: f(q, k, v, np.broadcast_to(g.mean(-1, keepdims=True), g.shape), b, s)),
    "no unit length": wrap("unit", lambda f: lambda x: x),
    "centred nowhere": wrap("layer_norm", lambda f: lambda x, w, e: gikepel.rms(x, e) * w),
    "plain relu": wrap("relu_squared", lambda f: lambda x: np.maximum(x, 0.0)),
    "no cap": wrap("soft_cap", lambda f: lambda x, c: x),
    "pair of a first token everywhere": wrap("bigram_rows", lambda f: lambda p, t, n, a, b: np.full(len(t), n)),
    "portion starts like a sequence": wrap("bigram_rows", lambda f: lambda p, t, n, a, b: f(None, t, n, a, b)),
    "multipliers exchanged": wrap("bigram_rows", lambda f: lambda p, t, n, a, b: f(p, t, n, b, a)),
}


@pytest.mark.parametrize("mistake", sorted(MISTAKES))
def test_inputs_show_a_planted_mistake(package, monkeypatch, mistake):
    """The GPU tests accept 0.06 in BF16 and 5e-5 in 32-bit; each of these mistakes is far beyond both."""
    c = cases.CASES["mixed"]
    weights, ids = cases.random_weights(package, c, seed=2), tokens(c, 60)
    right = gikepel.GikepelOracle(c, weights)
    want = np.concatenate([right.forward(ids[:40]), right.forward(ids[40:])])
    MISTAKES[mistake](monkeypatch)
    wrong = gikepel.GikepelOracle(c, weights)
    got = np.concatenate([wrong.forward(ids[:40]), wrong.forward(ids[40:])])
    assert logit_error(got, want).max() > 0.12


def test_trace_run_reads_the_design(package, tmp_path):
    """Without a GPU the replay gets as far as the model; a broken configuration is refused before that."""
    c = cases.CASES["delta_odd"]
    write_checkpoint(tmp_path, {**c, "layers": [{"type": "other", "mixer": {}}]}, cases.random_weights(package, c))
    run = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(tmp_path), "--dtype", "bfloat16", "--out", str(tmp_path),
                          "--max-tokens", "8"], capture_output=True, text=True, input="")
    assert run.returncode not in (0, 3) and "mixer type" in run.stderr
