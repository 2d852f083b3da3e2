"""The Gikepel decoder on the GPU against the plain restatement (oracle/gikepel.py, double precision): every mechanism
and size class in true 32-bit and in BF16, prompts against portions against token-by-token decoding, state and caches
that are used again, the verify step's rollback, and generation through the public entry points.

Errors are per position, RMS over the vocabulary in units of the logits' RMS (layered_cases.logit_error). In 32-bit the
limit is 5e-5; in BF16 it is 0.06 for every position and 0.02 for their mean (a planted mistake moves some position by
more than 0.12: test_gikepel_cpu.py)."""
import sys
from pathlib import Path

import numpy as np
import pytest

import gikepel_cases as cases
from layered_cases import bf16, greedy, logit_error, run_portions, tokens

sys.path.insert(0, str(Path(__file__).resolve().parents[1] / "oracle"))
import gikepel  # noqa: E402

pytestmark = pytest.mark.gpu
LIMIT = {"f32": 5e-5, "bf16": 0.06}
KINDS = ("f32", "bf16")


def build(package, c, kind, seed=0, sharp=1.0, ranks=(13, 21)):
    weights = cases.random_weights(package, c, seed, sharp, ranks)
    shape, tensors = package.checkpoint.admit(c, weights, "gikepel_" + kind)
    return package.Model(shape, tensors), gikepel.GikepelOracle(c, weights)


def check(got, want, kind, what=""):
    error = logit_error(got, want)
    assert error.max() <= LIMIT[kind], f"{what}: position {int(error.argmax())} is off by {error.max():.3g}"
    if len(error) >= 20:
        assert error.mean() <= LIMIT[kind] / 3, f"{what}: off by {error.mean():.3g} on average"


# ---- mechanisms and sizes ----
@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("name", sorted(cases.CASES))
def test_every_case_whole_stepwise_and_in_portions(cuda, package, name, kind):
    c = cases.CASES[name]
    model, oracle = build(package, c, kind)
    ids = tokens(c, 150)
    want = oracle.forward(ids)
    session = model.new_session(160, graph=True)
    for sizes in ([150], [1], [2, 37, 16, 3, 64, 1]):
        session.reset()
        check(run_portions(session, ids, sizes), want, kind, f"portions {sizes}")


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("ranks", [(1, 1), (64, 100), (130, 7)])
def test_ranks_of_the_decay_and_gate_projections(cuda, package, ranks, kind):
    c = cases.config(97, 72, [cases.delta(3, 1, 24, 40, 3, ff=30)])
    model, oracle = build(package, c, kind, ranks=ranks)
    ids = tokens(c, 100)
    session = model.new_session(100, graph=True)
    check(run_portions(session, ids, [60, 1]), oracle.forward(ids), kind)


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("name", ["mixed", "delta_64", "mamba_cut_heads", "latent_piece_sizes"])
def test_residual_stream_after_every_layer(cuda, package, name, kind):
    c = cases.CASES[name]
    model, oracle = build(package, c, kind)
    ids = tokens(c, 90)
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
                assert np.abs(got[run] - want).max() <= (5e-5 if kind == "f32" else 0.15) * scale, (run, begin)


@pytest.mark.parametrize("kind", KINDS)
def test_one_key_that_stands_out(cuda, package, kind):
    """A probe token's query matches one other token's key alone: at every distance, the key's value must come through,
    however the sequence is cut and wherever the key lies (tile and segment borders, the very first token)."""
    c = cases.config(64, 96, [cases.latent(4, 32, 16, 32, 48, base=1e6, scale=1.0)])
    weights = cases.random_weights(package, c, 3)
    mark, probe, asks, holds, channel = 5, 6, 7, 8, 11
    weights["embed"][:, [asks, holds]] = 0
    weights["embed"][probe, asks] = weights["embed"][mark, holds] = 6.0
    weights["bigram"][:, [asks, holds]] = 0
    weights["l0.norm1"][[asks, holds]] = 1.0
    q, down, up = weights["l0.mix.q"], weights["l0.mix.dkv"], weights["l0.mix.uk"]
    q *= 0.3
    q[:, asks], down[:, holds], up[:, channel] = 0, 0, 0
    down[channel] *= 0.05
    down[channel, holds] = 2.0                               # the mark fills one latent value
    for head in range(4):                                    # an unrotated dimension carries the match
        q[head * 48 + 20] *= 0.05
        q[head * 48 + 20, asks] = 1.5
        up[head * 32 + 20] *= 0.05
        up[head * 32 + 20, channel] = 2.0
    weights = {k: bf16(v) for k, v in weights.items()}
    shape, tensors = package.checkpoint.admit(c, weights, "gikepel_" + kind)
    model, oracle = package.Model(shape, tensors), gikepel.GikepelOracle(c, weights)
    length = 330
    filler = [t for t in tokens(c, 3 * length, 4) if t not in (mark, probe)][:length]
    for place in (0, 1, 15, 16, 63, 64, 65, 127, 128, 200, 255, 256):
        ids = list(filler)
        ids[place] = mark
        for at in (place + 2, place + 4, 257, 320, 321, 329):
            if at > place:
                ids[at] = probe
        oracle.reset()
        want = oracle.forward(ids)
        without = list(ids)
        without[place] = filler[place]
        oracle.reset()
        probes = [i for i, t in enumerate(ids) if t == probe and i > place + 1]
        shift = logit_error(oracle.forward(without)[probes], want[probes])
        assert shift.min() > 0.4                             # the key matters at every probe
        for sizes in ([330], [62, 2, 1, 63, 129, 33, 40]) if kind == "bf16" else ([62, 2, 1],):
            session = model.new_session(330, graph=True)
            check(run_portions(session, ids, sizes), want, kind, f"key at {place}, portions {sizes}")


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("rate", [-9.0, 1.5, 4.0])
@pytest.mark.parametrize("layer", ["delta", "mamba"])
def test_memories_that_never_fade_and_that_fade_at_once(cuda, package, layer, rate, kind):
    """Decays next to one (every token of the sequence still counts at its end) and of many powers of e per token (the
    quotient of two cumulative decays would overflow)."""
    c = cases.config(90, 96, [cases.delta(3, 3, 64, 48, 4, ff=40) if layer == "delta" else cases.mamba(4, 2, 48, 48, 4, 2, ff=40)])
    weights = cases.random_weights(package, c, 5)
    weights["l0.mix.A_log"][:] = rate
    weights["l0.mix.A_log"][0] = -2.0
    shape, tensors = package.checkpoint.admit(c, weights, "gikepel_" + kind)
    model, oracle = package.Model(shape, tensors), gikepel.GikepelOracle(c, weights)
    ids = tokens(c, 400, 9)
    want = oracle.forward(ids)
    session = model.new_session(400, graph=True)
    for sizes in ([400], [33, 100, 1, 1, 66]):
        session.reset()
        check(run_portions(session, ids, sizes), want, kind, f"portions {sizes}")


# ---- cuts, long sequences, reuse ----
@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("size", [2, 3, 5, 16, 17, 33, 63, 64, 65, 128, 129])
def test_portions_of_any_size(cuda, package, size, kind):
    c = cases.CASES["mixed"]
    model, oracle = build(package, c, kind, seed=2)
    ids = tokens(c, 300, 5)
    session = model.new_session(300, graph=True)
    check(run_portions(session, ids, [size]), oracle.forward(ids), kind, f"portions of {size}")


def test_prompt_beyond_a_segment_then_long_decoding(cuda, package):
    """2048-row segments, attention splits of more than one tile, and 150 decoded tokens behind them."""
    c = cases.config(150, 96, [cases.delta(2, 2, 32, 48, 4, ff=64), cases.latent(4, 32, 16, 48, 64, ff=80),
                               cases.mamba(4, 2, 32, 32, 4, 2)])
    model, oracle = build(package, c, "bf16", seed=4)
    ids = tokens(c, 4400, 6)
    want = oracle.forward(ids)
    session = model.new_session(4500, graph=True)
    places = [0, 1, 63, 64, 127, 128, 129, 2046, 2047, 2048, 2049, 2175, 2176, 4095, 4096, 4249]
    got = session.extend(ids[:4250], places)
    check(got, want[places], "bf16", "prompt")
    check(run_portions(session, ids[4250:], [1]), want[4250:], "bf16", "decoding")


def test_long_decoding_in_32_bit(cuda, package):
    c = cases.CASES["mixed"]
    model, oracle = build(package, c, "f32", seed=7)
    ids = tokens(c, 700, 8)
    session = model.new_session(700, graph=True)
    check(run_portions(session, ids, [60, 1]), oracle.forward(ids), "f32")


@pytest.mark.parametrize("kind", KINDS)
def test_the_first_tokens_of_a_sequence(cuda, package, kind):
    """Sequences shorter than the convolutions, and one of one token; the pair table's row of a first token."""
    c = cases.CASES["mamba_many_taps"]
    model, oracle = build(package, c, kind)
    session = model.new_session(64, graph=True)
    for length in (1, 2, 5, 20, 22, 40):
        for sizes in ([length], [1], [1, 3, 2]):
            oracle.reset()
            session.reset()
            ids = tokens(c, length, length)
            check(run_portions(session, ids, sizes), oracle.forward(ids), kind, f"{length} tokens, portions {sizes}")


@pytest.mark.parametrize("kind", KINDS)
def test_the_token_before_a_portion_counts(cuda, package, kind):
    """A large pair table entry: the first token of every portion needs the last one of the portion before it."""
    c = cases.config(50, 64, [cases.delta(2, 2, 16, 16, 2, ff=40)], buckets=1009, muls=(1 << 33, 3))
    weights = cases.random_weights(package, c, 6)
    weights["bigram"] = bf16(weights["bigram"] * 4)
    shape, tensors = package.checkpoint.admit(c, weights, "gikepel_" + kind)
    model, oracle = package.Model(shape, tensors), gikepel.GikepelOracle(c, weights)
    ids = tokens(c, 200, 7)
    want = oracle.forward(ids)
    session = model.new_session(200, graph=True)
    for sizes in ([1], [2], [40, 1, 33, 1, 1, 50], [200]):
        session.reset()
        check(run_portions(session, ids, sizes), want, kind, f"portions {sizes}")


@pytest.mark.parametrize("kind", KINDS)
def test_reset_and_neighbours_leave_no_trace(cuda, package, kind):
    c = cases.CASES["mixed"]
    model, oracle = build(package, c, kind)
    first, second = tokens(c, 140, 11), tokens(c, 120, 12)
    fresh = model.new_session(160, graph=True)
    alone = run_portions(fresh, second, [70, 1, 9])
    check(alone, oracle.forward(second), kind)
    used = model.new_session(160, graph=True)
    run_portions(used, first, [140])
    used.reset()
    assert np.array_equal(run_portions(used, second, [70, 1, 9]), alone)
    # Two requests taking turns.
    a, b = model.new_session(160, graph=True), model.new_session(160, graph=True)
    rows = []
    for at in range(0, 120, 40):
        rows.append(run_portions(b, second[at:at + 40], [40]))
        run_portions(a, first[at:at + 40], [33, 7])
    other = model.new_session(160)
    assert np.array_equal(np.concatenate(rows), run_portions(other, second, [40]))
    # A prefill replaces what was there.
    used.prefill(first)
    used.prefill(second)
    assert logit_error(used.read_logits_f32(1), alone[-1:]).max() <= LIMIT[kind]


def test_sessions_of_unequal_capacity_share_a_model(cuda, package):
    """The room for expanded keys grows with the longest history so far; smaller sessions go on using it."""
    c = cases.CASES["latent_many_heads"]
    model, oracle = build(package, c, "bf16")
    ids = tokens(c, 900, 19)
    want = oracle.forward(ids)
    for capacity, length in ((80, 70), (900, 900), (300, 300), (80, 80)):
        session = model.new_session(capacity)
        check(run_portions(session, ids[:length], [40, 200]), want[:length], "bf16", f"capacity {capacity}")


# ---- the verify step: rejected rows never reach the state ----
@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("name", ["mixed", "delta_odd", "mamba_many_taps", "latent_odd"])
def test_verify_rolls_back_rejected_rows(cuda, package, name, kind):
    c = cases.CASES[name]
    model, oracle = build(package, c, kind)
    rng = np.random.default_rng(3)
    session = model.new_session(400, graph=True)
    prompt = tokens(c, 40, 13)
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
    ids = tokens(c, 60, 14)
    session = model.new_session(80, graph=True)
    session.extend(ids[:30])
    session.extend(ids[30:42])                               # a step of 12 rows: 30..42 are pending
    oracle.forward(ids[:35])
    session.truncate(35)
    check(session.extend(ids[40:50], range(10)), oracle.forward(ids[40:50]), "f32")
    with pytest.raises(ValueError):
        session.truncate(34)
    session.truncate(0)
    oracle.reset()
    check(session.extend(ids[:9], range(9)), oracle.forward(ids[:9]), "f32")


# ---- generation ----
@pytest.mark.parametrize("name", ["mixed", "latent_piece_sizes"])
def test_greedy_generation_through_the_model_surface(cuda, package, name):
    c = dict(cases.CASES[name])
    weights = cases.random_weights(package, c)
    bridge = package.model_bridge.Model(c, weights, "gikepel_f32")
    prompt = tokens(c, 50, 15)
    want = greedy(gikepel.GikepelOracle(c, weights), prompt, 40)
    session, got = bridge.new_session(128), []
    session.generate(prompt, got.append, max_length=90)
    assert got == want
    again = []
    session.generate(prompt, again.append, max_length=70)
    assert again == want[:20]
    # Stops at the end-of-sequence token of the config; the type follows the config.
    stop = package.model_bridge.Model({**c, "eos_token_id": want[7]}, weights, None)
    short = []
    stop.new_session(128).generate(prompt, short.append, max_length=90)
    assert short[-1] == want[7] or want[7] not in short


def test_speculative_rounds_on_the_target(cuda, package):
    """A uniform draft model proposes, the target verifies on the device: the output is the target's own."""
    c = {**cases.CASES["mixed"], "logit_softcap": 300.0}     # top logits apart from one another
    model, _ = build(package, c, "bf16")
    draft_shape = package.Shape(vocab_size=c["vocab"], n_layers=1, n_heads=2, n_kv_heads=1, hidden_size=128,
                                intermediate_size=128, max_position_embeddings=256)
    draft = package.Model(draft_shape, package.synthetic.make_model(draft_shape, seed=1))
    prompt = tokens(c, 20, 16)
    decoder = package.runtime.SpeculativeDecoder(model.new_session(256, graph=True), draft.new_session(256, graph=True), 3)
    out = decoder.generate(prompt, 24)
    plain = model.new_session(256, graph=True)
    plain.extend(prompt)
    rows = plain.extend(out[:-1], range(len(out) - 1))
    top = np.sort(rows, axis=1)
    decided = top[:, -1] - top[:, -2] > 0.1 * np.sqrt(np.mean(rows * rows))
    assert decided.sum() > 5
    assert all(int(np.argmax(row)) == token for row, token, sure in zip(rows, out[1:], decided) if sure)


# ---- refusals and failures ----
def test_refusals_leave_the_history(cuda, package):
    c = cases.CASES["mixed"]
    model, oracle = build(package, c, "f32")
    ids = tokens(c, 32, 17)
    session = model.new_session(40, graph=True)
    session.extend(ids[:30])
    oracle.forward(ids[:30])
    with pytest.raises(BufferError):
        session.extend(tokens(c, 11))
    with pytest.raises(ValueError):
        session.extend([c["vocab"]])
    with pytest.raises(ValueError):
        package.runtime.SessionBatch([session, model.new_session(40)])
    check(session.extend(ids[30:], [0, 1]), oracle.forward(ids[30:]), "f32")


def test_a_wait_that_runs_out_is_reported(cuda, package):
    c = cases.CASES["latent_128"]
    model, oracle = build(package, c, "bf16")
    ids = tokens(c, 100, 18)
    session = model.new_session(128)
    session.extend(ids[:40])
    # The cache copies of a step, the attention copies of a prompt, and the prompt GEMM's.
    for hook, rows in ((session.inject_attention_wait_timeout, 3), (session.inject_attention_wait_timeout, 50),
                       (session.inject_wait_timeout, 50)):
        hook(2000)
        with pytest.raises(RuntimeError):
            session.extend(ids[:rows])
        assert session.context_size() == 0                   # drained and forgotten
        session.extend(ids[:10])
    session.reset()
    check(session.extend(ids, range(100)), oracle.forward(ids), "bf16")
