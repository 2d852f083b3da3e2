"""Layered decoders on the GPU against the plain restatement (oracle/hybrid.py, double precision): every mechanism and
size class in true 32-bit and in BF16, prompts against portions against token-by-token decoding, state and caches that
are used again, the verify step's rollback, and generation through the public entry points.

Errors are per position, RMS over the vocabulary in units of the logits' RMS (layered_cases.logit_error). In 32-bit the
limit is 5e-5; in BF16 it is 0.03 for every position (a planted mistake moves the logits by more than 0.1:
test_layered_cpu.py)."""
import sys
from pathlib import Path

import numpy as np
import pytest

import layered_cases as cases

sys.path.insert(0, str(Path(__file__).resolve().parents[1] / "oracle"))
import hybrid  # noqa: E402

pytestmark = pytest.mark.gpu
LIMIT = {"f32": 5e-5, "bf16": 0.03}
KINDS = ("f32", "bf16")


def build(package, c, kind, seed=0, sharp=1.0):
    weights = cases.random_weights(package, c, seed, sharp)
    shape, tensors = package.checkpoint.admit(c, weights, "zofesun_" + kind)
    return package.Model(shape, tensors), hybrid.HybridOracle(c, weights)


def check(got, want, kind, what=""):
    error = cases.logit_error(got, want)
    assert error.max() <= LIMIT[kind], f"{what}: position {int(error.argmax())} is off by {error.max():.3g}"


# ---- mechanisms and sizes ----
@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("name", sorted(cases.CASES))
def test_every_case_whole_stepwise_and_in_portions(cuda, package, name, kind):
    c = cases.CASES[name]
    model, oracle = build(package, c, kind)
    ids = cases.tokens(c, 150)
    want = oracle.forward(ids)
    session = model.new_session(160, graph=True)
    for sizes in ([150], [1], [2, 37, 16, 3, 64, 1]):
        session.reset()
        check(cases.run_portions(session, ids, sizes), want, kind, f"portions {sizes}")


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("name", ["mixed", "loop_first", "loop_last", "gru_wide"])
def test_residual_stream_after_every_layer_run(cuda, package, name, kind):
    c = cases.CASES[name]
    model, oracle = build(package, c, kind)
    ids = cases.tokens(c, 90)
    tap = cuda.zeros((len(oracle.runs), 90, c["width"]), device="cuda")
    for portions in ([(0, 16), (16, 27)], [(0, 90)] if kind == "bf16" else [(0, 11)]):
        oracle.reset()
        session = model.new_session(128)
        session.tap_residual(tap)
        for begin, end in portions:
            oracle.forward(ids[begin:end])
            session.extend(ids[begin:end])
            got = tap[:, :end - begin].cpu().numpy()
            for run, want in enumerate(oracle.taps):
                scale = np.sqrt(np.mean(want * want))
                assert np.abs(got[run] - want).max() <= (2e-5 if kind == "f32" else 0.06) * scale, (run, begin)
    with pytest.raises(ValueError):
        session.tap_residual(tap[:, :4])
        session.extend(ids[:5])


@pytest.mark.parametrize("kind", KINDS)
def test_one_key_that_stands_out(cuda, package, kind):
    """A probe token's query matches one other token's key alone: at every distance, the key's value must come through,
    however the sequence is cut and wherever the key lies (tile, chunk and segment borders, the very first token)."""
    c = cases.config(64, 96, [cases.parallel((4, 2, 32, 32, 8, 1e6), (2, 16, 16), scales=(1.0, 0.05))])
    c["layers"][0]["mixer"]["left"]["scale"] = 0.5
    weights = cases.random_weights(package, c, 3)
    mark, probe = 5, 6
    direction = np.zeros(96, dtype=np.float32)
    direction[7] = 1.0
    weights["embed"][:, 7] = 0
    weights["embed"][[mark, probe], 7] = 3.0
    weights["l0.norm1.b"][7] = 0
    for name, token_size, strength in (("q", 4, 6.0), ("k", 2, 6.0)):
        w = weights["l0.mix.left." + name]
        w[:, 7] = 0
        for head in range(token_size):                       # an unrotated dimension carries the match
            w[head * 32 + 20, :] *= 0.05
            w[head * 32 + 20, 7] = strength
    weights = {k: cases.bf16(v) for k, v in weights.items()}
    shape, tensors = package.checkpoint.admit(c, weights, "zofesun_" + kind)
    model, oracle = package.Model(shape, tensors), hybrid.HybridOracle(c, weights)
    length = 330
    filler = [t for t in cases.tokens(c, 3 * length, 4) if t not in (mark, probe)][:length]
    for place in (0, 1, 15, 16, 63, 64, 65, 127, 128, 200, 255, 256):
        ids = list(filler)
        ids[place] = mark
        for at in (place + 1, place + 3, 257, 320, 321, 329):
            if at > place:
                ids[at] = probe
        oracle.reset()
        want = oracle.forward(ids)
        without = list(ids)
        without[place] = filler[place]
        oracle.reset()
        probes = [i for i, t in enumerate(ids) if t == probe]
        shift = cases.logit_error(oracle.forward(without)[probes], want[probes])
        assert shift.min() > 0.1                             # the key matters at every probe
        for sizes in ([330], [62, 2, 1, 63, 129, 33, 40]) if kind == "bf16" else ([62, 2, 1],):
            session = model.new_session(330, graph=True)
            check(cases.run_portions(session, ids, sizes), want, kind, f"key at {place}, portions {sizes}")


# ---- cuts, long sequences, reuse ----
@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("size", [2, 3, 5, 16, 17, 33, 65, 128, 129])
def test_portions_of_any_size(cuda, package, size, kind):
    c = cases.CASES["mixed"]
    model, oracle = build(package, c, kind, seed=2, sharp=1.5)
    ids = cases.tokens(c, 300, 5)
    session = model.new_session(300, graph=True)
    check(cases.run_portions(session, ids, [size]), oracle.forward(ids), kind, f"portions of {size}")


def test_prompt_beyond_a_segment_then_long_decoding(cuda, package):
    """2048-row segments, attention chunks of more than one tile, and 150 decoded tokens behind them."""
    c = cases.config(150, 96, [cases.parallel((4, 2, 64, 48, 32, 1e5), (2, 32, 48), ff=80), cases.mingru(96, ff=64)],
                     loop=(0, 2, 2))
    model, oracle = build(package, c, "bf16", seed=4)
    ids = cases.tokens(c, 4400, 6)
    want = oracle.forward(ids)
    session = model.new_session(4500, graph=True)
    places = [0, 1, 63, 64, 127, 128, 129, 2046, 2047, 2048, 2049, 2175, 2176, 4095, 4096, 4249]
    got = session.extend(ids[:4250], places)
    check(got, want[places], "bf16", "prompt")
    check(cases.run_portions(session, ids[4250:], [1]), want[4250:], "bf16", "decoding")


def test_long_decoding_in_32_bit(cuda, package):
    c = cases.CASES["mixed"]
    model, oracle = build(package, c, "f32", seed=7)
    ids = cases.tokens(c, 700, 8)
    session = model.new_session(700, graph=True)
    check(cases.run_portions(session, ids, [60, 1]), oracle.forward(ids), "f32")


@pytest.mark.parametrize("kind", KINDS)
def test_reset_and_neighbours_leave_no_trace(cuda, package, kind):
    c = cases.CASES["mixed"]
    model, oracle = build(package, c, kind)
    first, second = cases.tokens(c, 140, 11), cases.tokens(c, 120, 12)
    fresh = model.new_session(160, graph=True)
    alone = cases.run_portions(fresh, second, [70, 1, 9])
    check(alone, oracle.forward(second), kind)
    used = model.new_session(160, graph=True)
    cases.run_portions(used, first, [140])
    used.reset()
    assert np.array_equal(cases.run_portions(used, second, [70, 1, 9]), alone)
    # Two requests taking turns.
    a, b = model.new_session(160, graph=True), model.new_session(160, graph=True)
    rows = []
    for at in range(0, 120, 40):
        rows.append(cases.run_portions(b, second[at:at + 40], [40]))
        cases.run_portions(a, first[at:at + 40], [33, 7])
    other = model.new_session(160)
    assert np.array_equal(np.concatenate(rows), cases.run_portions(other, second, [40]))
    # A prefill replaces what was there.
    used.prefill(first)
    used.prefill(second)
    assert cases.logit_error(used.read_logits_f32(1), alone[-1:]).max() <= LIMIT[kind]


# ---- the verify step: rejected rows never reach the state ----
@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("name", ["mixed", "gru_only", "parallel_only"])
def test_verify_rolls_back_rejected_rows(cuda, package, name, kind):
    c = cases.CASES[name]
    model, oracle = build(package, c, kind)
    rng = np.random.default_rng(3)
    session = model.new_session(400, graph=True)
    prompt = cases.tokens(c, 40, 13)
    session.prefill(prompt)
    oracle.forward(prompt)
    pending, emitted_sizes = session.greedy_next(), set()
    for round_ in range(24):
        rows = int(rng.integers(1, 17))
        # The greedy continuation from here, then one wrong draft somewhere.
        saved, at, drafts = oracle.save(), oracle.position, []
        token = pending
        for _ in range(rows - 1):
            token = int(np.argmax(oracle.forward([token])[0]))
            drafts.append(token)
        oracle.truncate(at, saved)
        if drafts and round_ % 3:
            wrong = int(rng.integers(0, len(drafts)))
            drafts[wrong] = (drafts[wrong] + 1) % c["vocab"]
        saved = oracle.save()
        out = session.verify([pending] + drafts)
        want = oracle.forward([pending] + drafts)
        check(session.read_logits_f32(rows), want, kind, f"round {round_}")
        oracle.truncate(at, saved)
        oracle.forward(([pending] + drafts)[:out.emitted])
        emitted_sizes.add(out.emitted)
        pending = out.tokens[-1]
        if oracle.position > 370:
            break
    assert len(emitted_sizes) > 4
    check(session.extend([pending], [0]), oracle.forward([pending]), kind, "after the rounds")


def test_truncation_reaches_back_over_the_last_step_only(cuda, package):
    c = cases.CASES["mixed"]
    model, oracle = build(package, c, "f32")
    ids = cases.tokens(c, 60, 14)
    session = model.new_session(80, graph=True)
    session.extend(ids[:30])
    session.extend(ids[30:42])                               # a step of 12 rows: 30..42 are pending
    oracle.forward(ids[:35])
    session.truncate(35)
    check(session.extend(ids[40:50], range(10)), oracle.forward(ids[40:50]), "f32")
    with pytest.raises(ValueError):
        session.truncate(34)
    with pytest.raises(ValueError):
        session.truncate(60)
    assert session.context_size() == 45
    session.truncate(0)
    oracle.reset()
    check(session.extend(ids[:9], range(9)), oracle.forward(ids[:9]), "f32")


# ---- generation ----
@pytest.mark.parametrize("name", ["mixed", "loop_last"])
def test_greedy_generation_through_the_model_surface(cuda, package, name):
    c = dict(cases.CASES[name])
    weights = cases.random_weights(package, c)
    bridge = package.model_bridge.Model(c, weights, "zofesun_f32")
    prompt = cases.tokens(c, 50, 15)
    want = cases.greedy(hybrid.HybridOracle(c, weights), prompt, 40)
    session, got = bridge.new_session(128), []
    session.generate(prompt, got.append, max_length=90)
    assert got == want
    again = []
    session.generate(prompt, again.append, max_length=70)
    assert again == want[:20]
    # Stops at the end-of-sequence token of the config.
    stop = package.model_bridge.Model({**c, "eos_token_id": want[7]}, weights, None)
    short = []
    stop.new_session(128).generate(prompt, short.append, max_length=90)
    assert short[-1] == want[7] or want[7] not in short


def test_speculative_rounds_on_a_layered_target(cuda, package):
    """A uniform draft model proposes, the layered target verifies on the device: the output is the target's own."""
    c = cases.CASES["mixed"]
    model, _ = build(package, c, "bf16")
    draft_shape = package.Shape(vocab_size=c["vocab"], n_layers=1, n_heads=2, n_kv_heads=1, hidden_size=128,
                                intermediate_size=128, max_position_embeddings=256)
    draft = package.Model(draft_shape, package.synthetic.make_model(draft_shape, seed=1))
    prompt = cases.tokens(c, 20, 16)
    decoder = package.runtime.SpeculativeDecoder(model.new_session(256, graph=True), draft.new_session(256, graph=True), 3)
    out = decoder.generate(prompt, 24)
    # The target's own rows of the same width: replay the output and compare every greedy choice that is decided.
    plain = model.new_session(256, graph=True)
    plain.extend(prompt)
    rows = plain.extend(out[:-1], range(len(out) - 1))
    top = np.sort(rows, axis=1)
    decided = top[:, -1] - top[:, -2] > 0.1 * np.sqrt(np.mean(rows * rows))
    assert decided.sum() > 5
    assert all(int(np.argmax(row)) == token for row, token, sure in zip(rows, out[1:], decided) if sure)
    with pytest.raises(ValueError):
        package.runtime.SpeculativeDecoder(draft.new_session(64), model.new_session(64), 3)


# ---- the contract around it ----
def test_refusals_leave_the_history(cuda, package):
    c = cases.CASES["mixed"]
    model, oracle = build(package, c, "f32")
    ids = cases.tokens(c, 32, 17)
    session = model.new_session(40, graph=True)
    session.extend(ids[:30])
    oracle.forward(ids[:30])
    with pytest.raises(BufferError):
        session.extend(cases.tokens(c, 11))
    with pytest.raises(ValueError):
        session.extend([c["vocab"]])
    with pytest.raises(ValueError):
        session.extend(ids[:4], [2, 1])
    with pytest.raises(ValueError):
        session.extend(ids[:4], [4])
    with pytest.raises(ValueError):
        session.read_kv(0)
    with pytest.raises(ValueError):
        package.runtime.SessionBatch([session, model.new_session(40)])
    check(session.extend(ids[30:], [0, 1]), oracle.forward(ids[30:]), "f32")


def test_a_wait_that_runs_out_is_reported(cuda, package):
    c = cases.CASES["even_64"]
    model, oracle = build(package, c, "bf16")
    ids = cases.tokens(c, 100, 18)
    session = model.new_session(128)
    session.extend(ids[:40])
    # The attention copies of a step and of a prompt, and the prompt GEMM's (a step's GEMMs of this width have none).
    for hook, rows in ((session.inject_attention_wait_timeout, 3), (session.inject_attention_wait_timeout, 50),
                       (session.inject_wait_timeout, 50)):
        hook(2000)
        with pytest.raises(RuntimeError):
            session.extend(ids[:rows])
        assert session.context_size() == 0                   # drained and forgotten
        session.extend(ids[:10])
    session.reset()
    check(session.extend(ids, range(100)), oracle.forward(ids), "bf16")


def test_the_uniform_decoder_takes_portions_too(cuda, package):
    shape = package.Shape(vocab_size=512, n_layers=2, n_heads=4, n_kv_heads=2, hidden_size=256, intermediate_size=512,
                          max_position_embeddings=256)
    model = package.Model(shape, package.synthetic.make_model(shape, seed=9))
    ids = [int(t) for t in package.synthetic.make_prompt(3, 120, 512)]
    whole = model.new_session(128)
    whole.prefill(ids)
    want = whole.read_logits_f32(1)
    for sizes in ([120], [50, 2, 1, 33, 34], [16]):
        session = model.new_session(128, graph=True)
        got = cases.run_portions(session, ids, sizes)
        assert got.shape == (120, 512)
        assert cases.logit_error(got[-1:], want).max() < 0.02
