"""Small configurations and random weights of layered decoders for the tests. Weights are BF16 values held as float32,
scaled so that attention is peaked, sinks matter and norms do not saturate: a wrong key, a lost state or a missing term
then moves the logits by far more than rounding does."""
import copy

import numpy as np


def parallel(left, right, ff=None, limit=1.0, scales=(0.7, 1.1)):
    heads, kv_heads, dim, vdim, rot_dims, base = left
    lin_heads, lin_dim, lin_vdim = right
    return {"type": "parallel",
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": 1.1 / dim ** 0.5,
                               "rot": {"dims": rot_dims, "base": base}},
                      "right": {"heads": lin_heads, "dim": lin_dim, "vdim": lin_vdim,
                                "decay": [1.0 - 0.5 * 0.3 ** (i * 4.0 / lin_heads) for i in range(lin_heads)]},
                      "left_scale": scales[0], "right_scale": scales[1]},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}


def mingru(width, ff=None, limit=1.0):
    return {"type": "mingru", "mixer": {"width": width},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}


def config(vocab, width, layers, loop=None, eps=1e-5):
    c = {"architecture": "Zofesun", "vocab": vocab, "width": width, "layers": copy.deepcopy(layers), "norm": {"eps": eps}}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


# Sizes that are multiples of nothing, head sizes on both sides of every kernel's limits, equal and unequal pairs,
# one head, one group, loops at the start, in the middle and to the end, layers without a feed-forward.
CASES = {
    "gru_only": config(97, 72, [mingru(50)]),
    "gru_wide": config(130, 64, [mingru(64, ff=44, limit=0.8), mingru(200)]),
    "parallel_only": config(97, 72, [parallel((6, 2, 20, 12, 6, 500.0), (3, 24, 40))]),
    "even_64": config(120, 128, [parallel((4, 2, 64, 64, 64, 1e4), (2, 64, 64), ff=96)]),
    "even_128": config(120, 192, [parallel((3, 1, 128, 128, 32, 1e5), (1, 128, 128), ff=70, limit=0.5)]),
    "value_wider": config(101, 96, [parallel((5, 5, 32, 80, 16, 1e4), (4, 16, 112), ff=64, scales=(1.0, 1.0))]),
    "key_wider": config(101, 80, [parallel((8, 1, 112, 16, 112, 3e4), (2, 144, 16))]),
    "largest_tiled": config(90, 64, [parallel((2, 1, 256, 200, 128, 1e6), (1, 256, 72))]),
    "beyond_tiled": config(90, 64, [parallel((2, 2, 272, 40, 64, 1e4), (1, 300, 20), ff=33)]),
    "loop_first": config(113, 88, [mingru(40, ff=30), parallel((4, 4, 24, 24, 8, 1e3), (2, 20, 28), ff=50)],
                         loop=(0, 1, 3)),
    "loop_last": config(113, 88, [parallel((4, 2, 48, 32, 24, 1e3), (2, 32, 16)), mingru(88, ff=40, limit=2.0)],
                        loop=(1, 2, 2)),
    "loop_once": config(77, 66, [mingru(30), mingru(34)], loop=(0, 2, 1)),
    # More inputs than one K slice of a step projection: FP32 slices summed by the joins, and BF16 results by a store.
    "inputs_in_slices": config(60, 72, [mingru(4160, ff=4200, limit=1.2), mingru(1100)]),
    "stream_in_slices": config(60, 4200, [mingru(40, ff=70), parallel((2, 1, 16, 16, 16, 1e3), (1, 16, 16))]),
    "mixed": config(203, 104, [mingru(56, ff=72), parallel((6, 3, 40, 24, 20, 1e4), (5, 24, 32), ff=60, limit=0.7),
                               parallel((6, 3, 40, 24, 20, 1e4), (5, 24, 32)), mingru(120)], loop=(1, 3, 2)),
}


def bf16(values):
    bits = np.ascontiguousarray(values, dtype=np.float32).view(np.uint32).astype(np.uint64)
    rounded = ((bits + 0x7FFF + ((bits >> 16) & 1)) >> 16 << 16).astype(np.uint32)
    return rounded.view(np.float32).reshape(np.shape(values))


def random_weights(package, c, seed=0, sharp=1.0):
    """name -> float32 array (values exact in BF16). `sharp` scales queries and keys: larger is nearer to one-hot."""
    shape = package.checkpoint.zofesun_shape(c)
    rng = np.random.default_rng(seed)
    weights = {}
    for name, dims in package.checkpoint.layered_tensor_shapes(shape).items():
        if name.endswith(".alpha"):
            value = rng.uniform(0.5, 0.9)
        elif name.endswith((".norm1", ".norm2", ".norm1b", ".norm2b", "final.norm", "right.norm")):
            value = 1.0 + 0.3 * rng.standard_normal(dims)
        elif name.endswith("sink"):
            value = rng.uniform(0.5, 2.5, dims)
        elif name.endswith(".b"):
            value = 0.2 * rng.standard_normal(dims)
        elif name in ("embed", "loop.step"):
            value = (1.0 if name == "embed" else 0.4) * rng.standard_normal(dims)
        else:
            value = rng.standard_normal(dims) * 1.6 / dims[-1] ** 0.5
            if name.endswith(("left.q", "left.k")):
                value = value * 1.2 * sharp
            if name.endswith("right.q") or name.endswith("right.k"):
                value = value * 0.7
        weights[name] = bf16(value)
    return weights


def tokens(c, length, seed=1):
    return [int(t) for t in np.random.default_rng(seed).integers(0, c["vocab"], length)]


def logit_error(got, want):
    """Per position: RMS over the vocabulary of the difference with its mean taken off, in units of the logits' RMS."""
    got, want = np.asarray(got, dtype=np.float64), np.asarray(want, dtype=np.float64)
    d = got - want
    d = d - d.mean(axis=-1, keepdims=True)
    scale = np.sqrt(np.mean((want - want.mean(axis=-1, keepdims=True)) ** 2))
    return np.sqrt(np.mean(d * d, axis=-1)) / scale


def run_portions(session, ids, sizes):
    """All positions' logits, the sequence cut into portions (the last size repeats)."""
    out, at, sizes = [], 0, list(sizes)
    while at < len(ids):
        size = min(sizes.pop(0) if len(sizes) > 1 else sizes[0], len(ids) - at)
        out.append(session.extend(ids[at:at + size], range(size)))
        at += size
    return np.concatenate(out)


def greedy(oracle, prompt, count):
    """The restatement's own greedy continuation."""
    logits = oracle.forward(prompt)[-1]
    out = []
    for _ in range(count):
        out.append(int(np.argmax(logits)))
        logits = oracle.forward([out[-1]])[0]
    return out
