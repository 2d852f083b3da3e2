"""Layered decoders without a GPU: the configuration reader and weight admission, the plain restatement's own
consistency, the sensitivity of the GPU tests' inputs to planted mistakes (planted here, in the restatement), and the
trace replay's bookkeeping."""
import json
import struct
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest

import layered_cases as cases

ROOT = Path(__file__).resolve().parents[1]
sys.path.insert(0, str(ROOT / "oracle"))
import hybrid  # noqa: E402


def write_checkpoint(folder, c, weights):
    header, blobs, at = {}, [], 0
    for name, value in weights.items():
        data = (np.asarray(value, dtype=np.float32).view(np.uint32) >> 16).astype("<u2").tobytes()
        header[name] = {"dtype": "BF16", "shape": list(np.shape(value)), "data_offsets": [at, at + len(data)]}
        blobs.append(data)
        at += len(data)
    text = json.dumps(header).encode()
    (folder / "model.safetensors").write_bytes(struct.pack("<Q", len(text)) + text + b"".join(blobs))
    (folder / "config.json").write_text(json.dumps(c))


# ---- configuration and admission ----
@pytest.mark.parametrize("name", sorted(cases.CASES))
def test_every_size_and_constant_comes_from_the_config(package, name):
    c = cases.CASES[name]
    shape = package.checkpoint.shape_from_config(c, "zofesun_bf16")
    assert (shape.vocab_size, shape.hidden_size, shape.n_layers) == (c["vocab"], c["width"], len(c["layers"]))
    assert shape.norm_eps == c["norm"]["eps"] and not shape.true32
    assert package.checkpoint.shape_from_config(c, "zofesun_f32").true32
    for entry, layer in zip(c["layers"], shape.layers):
        if entry["type"] == "mingru":
            assert layer.rnn_width == entry["mixer"]["width"] and layer.attention is None
        else:
            left, right = entry["mixer"]["left"], entry["mixer"]["right"]
            a, l = layer.attention, layer.linear
            assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale) == tuple(left[k] for k in ("heads", "kv_heads", "dim", "vdim", "scale"))
            assert (a.rot_dims, a.rot_base) == (left["rot"]["dims"], left["rot"]["base"])
            assert (l.heads, l.dim, l.vdim, list(l.decay)) == (right["heads"], right["dim"], right["vdim"], right["decay"])
            assert (layer.left_scale, layer.right_scale) == (entry["mixer"]["left_scale"], entry["mixer"]["right_scale"])
        if entry["mlp"] is None:
            assert layer.ff is None
        else:
            assert (layer.ff, layer.limit) == (entry["mlp"]["ff"], entry["mlp"]["limit"])
    oracle = hybrid.HybridOracle(c, cases.random_weights(package, c))
    assert shape.layer_runs() == [layer for layer, _ in oracle.runs]


def test_model_type_follows_the_config(package):
    pick = package.checkpoint.model_type_of
    assert pick({"architecture": "Zofesun"}) == "zofesun_bf16"
    assert pick({"architecture": "Zofesun"}, "float32") == "zofesun_f32"
    assert pick({"model_type": "qwen3"}) == "qwen3_bf16"
    assert pick({"model_type": "qwen2", "quantization_config": {}}) == "qwen_awq"
    with pytest.raises(NotImplementedError):
        pick({"model_type": "qwen3"}, "float32")
    with pytest.raises(ValueError):
        pick({"architecture": "SomethingElse"})


def test_admission_checks_names_and_shapes(package, tmp_path):
    c = cases.CASES["mixed"]
    weights = cases.random_weights(package, c)
    write_checkpoint(tmp_path, c, weights)
    loaded_config, loaded = package.checkpoint.load_directory(tmp_path)
    shape, tensors = package.checkpoint.admit(loaded_config, loaded, package.checkpoint.model_type_of(loaded_config))
    assert set(tensors) == set(weights) and shape.loop == (1, 3, 2)
    for name, [(kind, data)] in tensors.items():
        assert kind == 0 and np.array_equal(package.synthetic.bf16_to_float(np.asarray(data)).reshape(weights[name].shape), weights[name])
    # Norms of a feed-forward that a layer does not have are passed over.
    _, spare = package.checkpoint.admit(c, {**weights, "l2.norm2.alpha": weights["l1.norm2.alpha"]}, "zofesun_bf16")
    assert set(spare) == set(weights)
    for change in (lambda w: w.pop("l1.mix.left.sink"), lambda w: w.update({"l0.mix.left.q": w["l1.mix.left.q"]}),
                   lambda w: w.update({"head": w["head"][:-1]})):
        broken = dict(weights)
        change(broken)
        with pytest.raises(ValueError):
            package.checkpoint.admit(c, broken, "zofesun_bf16")


@pytest.mark.parametrize("edit", [
    lambda c: c["layers"][1]["mixer"]["right"]["decay"].pop(),
    lambda c: c["layers"][1]["mixer"].pop("left_scale"),
    lambda c: c["layers"][0].update(type="other"),
    lambda c: c["layers"][0]["mlp"].update(kind="experts"),
    lambda c: c["loop"].update(stop=9),
    lambda c: c.update(width="wide"),
])
def test_malformed_configs_are_refused(package, edit):
    c = json.loads(json.dumps(cases.CASES["mixed"]))
    edit(c)
    with pytest.raises(ValueError):
        package.checkpoint.shape_from_config(c, "zofesun_bf16")


def test_model_creation_rejects_bad_arguments_without_a_gpu(package):
    import ctypes
    lib = package.abi.load_library()
    with pytest.raises(ValueError):
        package.abi.check(lib.ei_model_create_layered(None, None, None, 0, ctypes.byref(ctypes.c_void_p())))


# ---- the restatement itself ----
def test_restatement_in_portions_equals_the_whole(package):
    c = cases.CASES["mixed"]
    weights, ids = cases.random_weights(package, c), cases.tokens(c, 41)
    whole = hybrid.HybridOracle(c, weights).forward(ids)
    pieces, other, at = [], hybrid.HybridOracle(c, weights), 0
    for size in (2, 7, 1, 16, 1, 14):
        pieces.append(other.forward(ids[at:at + size]))
        at += size
    assert np.abs(np.concatenate(pieces) - whole).max() < 1e-9


def test_restatement_mechanisms_against_closed_forms():
    rng = np.random.default_rng(0)
    # Linear attention: the recurrence against its attention form.
    q, k, v = rng.standard_normal((9, 2, 3)), rng.standard_normal((9, 2, 3)), rng.standard_normal((9, 2, 4))
    decay = np.array([0.5, 0.9])
    out, state = hybrid.lightning(q, k, v, decay, np.zeros((2, 3, 4)))
    for h in range(2):
        weight = np.tril((q[:, h] @ k[:, h].T) * decay[h] ** np.maximum(np.arange(9)[:, None] - np.arange(9)[None], 0))
        assert np.allclose(out[:, h], weight @ v[:, h])
    # Gated recurrence: a closed gate keeps the state, an open one takes the candidate.
    s, _ = hybrid.min_gru(np.array([[-60.0, 60.0, 60.0]]), np.array([[3.0, 3.0, -2.0]]), np.array([7.0, 7.0, 7.0]))
    assert np.allclose(s[0], [7.0, 3.5, 1.0 / (1.0 + np.exp(2.0))])
    # Rotation keeps lengths and turns scores into functions of the distance.
    x, y = rng.standard_normal((1, 1, 8)), rng.standard_normal((1, 1, 8))
    score = [float((hybrid.rotate(x, np.array([p + 5]), 6, 100.0) * hybrid.rotate(y, np.array([p]), 6, 100.0)).sum())
             for p in (0, 11, 400)]
    assert np.allclose(score, score[0])
    # A sink takes its share and has no value.
    one = hybrid.sink_attention(np.zeros((1, 1, 2)), np.zeros((1, 1, 2)), np.ones((1, 1, 3)), 1.0, np.array([0.0]), 0)
    assert np.allclose(one, 0.5)
    # Clamps: gate from above only, up on both sides.
    assert np.allclose(hybrid.clamped_glu(np.array([9.0]), np.array([-9.0]), 1.5),
                       1.5 / (1 + np.exp(-1.702 * 1.5)) * (1 - 1.5))


MISTAKES = {
    "no sink": lambda m: m.setattr(hybrid, "sink_attention", lambda q, k, v, s, sink, first, f=hybrid.sink_attention: f(q, k, v, s, np.full_like(sink, -60.0), first)),
    "scaled sink": lambda m: m.setattr(hybrid, "sink_attention", lambda q, k, v, s, sink, first, f=hybrid.sink_attention: f(q, k, v, s, sink * s, first)),
    "sees the next key": lambda m: m.setattr(hybrid, "sink_attention", lambda q, k, v, s, sink, first, f=hybrid.sink_attention: f(q, k, v, s, sink, first + 1)),
    "misses its own key": lambda m: m.setattr(hybrid, "sink_attention", lambda q, k, v, s, sink, first, f=hybrid.sink_attention: f(q, k, v, s, sink, first - 1)),
    "interleaved groups": lambda m: m.setattr(hybrid, "sink_attention", lambda q, k, v, s, sink, first, f=hybrid.sink_attention: f(q, k[:, ::-1], v[:, ::-1], s, sink, first)),
    "no value norm": lambda m: m.setattr(hybrid, "rms", lambda x, eps, f=hybrid.rms: x if x.ndim == 3 else f(x, eps)),
    "no output norm": lambda m: m.setattr(hybrid, "rms", lambda x, eps, f=hybrid.rms: f(x, eps) if x.ndim == 3 else x),
    "no rotation": lambda m: m.setattr(hybrid, "rotate", lambda x, p, d, b: x),
    "rotation one on": lambda m: m.setattr(hybrid, "rotate", lambda x, p, d, b, f=hybrid.rotate: f(x, p + (x.shape[1] > 3), d, b)),
    "no decay": lambda m: m.setattr(hybrid, "lightning", lambda q, k, v, d, s, f=hybrid.lightning: f(q, k, v, np.ones_like(d), s)),
    "lost linear state": lambda m: m.setattr(hybrid, "lightning", lambda q, k, v, d, s, f=hybrid.lightning: f(q, k, v, d, s * 0)),
    "lost recurrence": lambda m: m.setattr(hybrid, "min_gru", lambda z, u, s, f=hybrid.min_gru: f(z, u, s * 0)),
    "plain gate": lambda m: m.setattr(hybrid, "clamped_glu", lambda g, u, l: np.minimum(g, l) * hybrid.sigmoid(np.minimum(g, l)) * (np.clip(u, -l, l) + 1)),
    "no clamp": lambda m: m.setattr(hybrid, "clamped_glu", lambda g, u, l, f=hybrid.clamped_glu: f(g, u, 1e9)),
}


@pytest.mark.parametrize("mistake", sorted(MISTAKES))
def test_inputs_show_a_planted_mistake(package, monkeypatch, mistake):
    """The GPU tests accept 0.03 in BF16 and 5e-5 in 32-bit; each of these mistakes is far beyond both."""
    c = cases.CASES["mixed"]
    weights, ids = cases.random_weights(package, c), cases.tokens(c, 60)
    right = hybrid.HybridOracle(c, weights)
    want = np.concatenate([right.forward(ids[:40]), right.forward(ids[40:])])
    MISTAKES[mistake](monkeypatch)
    wrong = hybrid.HybridOracle(c, weights)
    got = np.concatenate([wrong.forward(ids[:40]), wrong.forward(ids[40:])])
    assert cases.logit_error(got, want).max() > 0.1


@pytest.mark.parametrize("left_out", ["the added embedding", "a pass's vector"])
def test_inputs_show_a_missing_injection(package, left_out):
    c = cases.CASES["mixed"]
    weights, ids = cases.random_weights(package, c), cases.tokens(c, 30)
    if left_out == "the added embedding":
        weights["loop.step"][1:] = weights["loop.step"][0]
    want = hybrid.HybridOracle(c, weights).forward(ids)
    wrong = hybrid.HybridOracle(c, weights)
    if left_out == "the added embedding":
        wrong.runs = [(layer, 0 if t else t) for layer, t in wrong.runs]  # every pass starts like the first
    else:
        wrong.w["loop.step"][1] = 0
    assert cases.logit_error(wrong.forward(ids), want).max() > 0.1


# ---- trace replay ----
class FakeSession:
    def __init__(self, vocab):
        self.vocab, self.history, self.resets = vocab, [], 0

    def extend(self, tokens, want):
        self.history += tokens
        base = len(self.history) - len(tokens)
        return np.array([[sum(self.history[:base + w + 1])] * self.vocab for w in want], dtype=np.float32).reshape(len(want), self.vocab)

    def reset(self):
        self.history, self.resets = [], self.resets + 1


class FakeModel:
    def __init__(self):
        self.shape = type("Shape", (), {"vocab_size": 3})
        self.made = []

    def new_session(self, capacity, graph):
        self.made.append(FakeSession(3))
        return self.made[-1]


def test_replay_orders_rows_and_reuses_sessions(package):
    model = FakeModel()
    replay = package.trace.Replay(model, 64)
    out = replay.step([{"id": "a", "tokens": [1, 2, 3], "want": [2, 0]}], [])
    assert out[:, 0].tolist() == [6.0, 1.0]
    out = replay.step([{"id": "b", "tokens": [5], "want": []}, {"id": "a", "tokens": [4], "want": [0, 0]}], ["a"])
    assert out[:, 0].tolist() == [10.0, 10.0] and len(model.made) == 2
    out = replay.step([{"id": "c", "tokens": [7], "want": [0]}], ["b", "c"])
    assert out[:, 0].tolist() == [7.0] and len(model.made) == 2 and model.made[0].resets == 2


def test_trace_run_explains_itself_and_refuses_what_cannot_run(package, tmp_path):
    run = str(ROOT / "bin" / "trace_run")
    help_text = subprocess.run([run, "--help"], capture_output=True, text=True)
    assert help_text.returncode == 0 and "--max-tokens" in help_text.stdout
    (tmp_path / "config.json").write_text(json.dumps({"model_type": "qwen3"}))
    write_checkpoint(tmp_path, {"model_type": "qwen3"}, {"x": cases.bf16(np.ones(2))})
    refused = subprocess.run([run, "--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "8"],
                             capture_output=True, text=True, input="")
    assert refused.returncode == 3
