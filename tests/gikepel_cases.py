"""Small configurations and random weights of Gikepel decoders for the tests. Weights are BF16 values held as float32,
scaled so that attention is peaked and states matter over long and short ranges: a wrong key, a lost state or a missing
term then moves the logits by far more than rounding does."""
import copy

import numpy as np

from layered_cases import bf16


def delta(heads, kv_heads, dim, vdim, conv, ff=None):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def mamba(heads, groups, state, vdim, conv, norm_groups, ff=None):
    return {"type": "mamba2", "mixer": {"heads": heads, "groups": groups, "state": state, "vdim": vdim, "conv": conv,
                                        "norm_groups": norm_groups},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def latent(heads, dim, rot_dim, vdim, kv_rank, base=1e4, scaling=(8.0, 128, 24.0, 0.5), ff=None, scale=None):
    if scaling is not None:
        scaling = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
                      "scale": scale or 1.1 / (dim + rot_dim) ** 0.5,
                      "rot": {"base": base, "dims": rot_dim, "scaling": scaling}},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(vocab, width, layers, eps=1e-5, buckets=53, muls=(31, 7), cap=18.0):
    return {"architecture": "Gikepel", "vocab": vocab, "width": width, "layers": copy.deepcopy(layers), "norm": {"eps": eps},
            "embedding": {"bigram": {"buckets": buckets, "mul_prev": muls[0], "mul_cur": muls[1]}}, "logit_softcap": cap}


# Sizes that are multiples of nothing, sizes on both sides of every kernel's limits, equal and unequal pairs, one head,
# one group, one tap and more taps than a step has rows, norm parts that cut heads, layers without a feed-forward.
CASES = {
    "delta_odd": config(97, 72, [delta(6, 2, 20, 36, 2)]),
    "delta_64": config(120, 128, [delta(4, 4, 64, 64, 4, ff=96), delta(2, 1, 64, 64, 3)]),
    "delta_128": config(120, 136, [delta(3, 3, 128, 128, 4, ff=72)]),
    "delta_key_wider": config(101, 96, [delta(4, 2, 112, 40, 1, ff=64)]),
    "delta_value_wider": config(101, 80, [delta(5, 1, 24, 168, 5)]),
    "delta_largest_tiled": config(90, 64, [delta(2, 2, 256, 72, 3)]),
    "delta_beyond_tiled": config(90, 64, [delta(2, 1, 280, 24, 20, ff=40)]),
    "mamba_odd": config(97, 72, [mamba(6, 3, 20, 12, 3, 4)]),
    "mamba_cut_heads": config(97, 104, [mamba(5, 1, 40, 24, 4, 3, ff=50), mamba(4, 4, 16, 32, 2, 8)]),
    "mamba_64": config(120, 128, [mamba(4, 2, 64, 64, 4, 2, ff=96)]),
    "mamba_128": config(120, 136, [mamba(6, 2, 128, 64, 4, 1, ff=40), mamba(3, 1, 128, 128, 1, 3, ff=70)]),
    "mamba_wide_norm": config(110, 64, [mamba(18, 2, 16, 128, 4, 1, ff=40)]),
    "mamba_many_taps": config(101, 88, [mamba(3, 3, 24, 200, 21, 1, ff=64)]),
    "mamba_beyond_tiled": config(90, 64, [mamba(2, 1, 272, 24, 4, 1)]),
    "latent_odd": config(97, 72, [latent(3, 20, 6, 12, 40, base=500.0)]),
    "latent_one_head": config(97, 72, [latent(1, 32, 32, 48, 72, scaling=None, ff=30)]),
    "latent_piece_sizes": config(110, 96, [latent(4, 64, 16, 64, 64, ff=64), latent(2, 48, 64, 20, 100)]),
    "latent_128": config(120, 128, [latent(5, 128, 64, 128, 512, base=1e5, scaling=(4.0, 64, 32.0, 1.0))]),
    "latent_many_heads": config(120, 128, [latent(20, 32, 32, 32, 128, scaling=(40.0, 4096, 32.0, 1.0), ff=70)]),
    "latent_wide_rank": config(90, 80, [latent(3, 40, 24, 56, 600, ff=44)]),
    "latent_wide_values": config(90, 80, [latent(2, 24, 8, 200, 72, ff=44)]),
    "latent_beyond_tiled": config(90, 64, [latent(2, 272, 40, 24, 96, ff=50), latent(2, 16, 8, 264, 1000, ff=50)]),
    "inputs_in_slices": config(60, 72, [delta(33, 3, 16, 128, 2, ff=4200), mamba(3, 1, 16, 16, 2, 1, ff=4160)]),
    "stream_in_slices": config(60, 4200, [delta(2, 1, 16, 16, 2, ff=70), mamba(2, 1, 16, 16, 2, 1), latent(2, 16, 8, 16, 24)],
                               cap=90.0),
    "mixed": config(203, 104, [delta(4, 2, 40, 24, 3, ff=72), latent(6, 24, 24, 40, 56, scaling=(40.0, 64, 32.0, 1.0), ff=60, scale=0.1),
                               latent(3, 16, 20, 16, 88, base=300.0),
                               mamba(6, 2, 24, 32, 4, 3, ff=44), delta(3, 3, 32, 48, 4)], buckets=211, muls=(91, 17)),
}


def random_weights(package, c, seed=0, sharp=1.0, ranks=(13, 21)):
    """name -> float32 array (values exact in BF16). `sharp` scales queries: larger is nearer to one-hot."""
    shape = package.checkpoint.gikepel_shape(c)
    for layer in shape.layers:
        if layer.delta is not None:
            layer.delta.decay_rank, layer.delta.gate_rank = ranks
    rng = np.random.default_rng(seed)
    weights = {}
    for name, dims in package.checkpoint.layered_tensor_shapes(shape).items():
        part = name.split(".", 1)[1] if name.startswith("l") else name
        if part in ("norm1", "norm2", "final.norm", "mix.norm", "mix.dkv.norm"):
            value = 1.0 + 0.3 * rng.standard_normal(dims)
        elif part in ("ls1", "ls2"):
            value = 0.8 + 0.3 * rng.standard_normal(dims)
        elif part == "mix.A_log":
            value = rng.uniform(-4.0, 1.0, dims)           # long and short memories
        elif part == "mix.dt_bias":
            value = rng.uniform(-4.0, 0.5, dims)
        elif part == "mix.D":
            value = rng.uniform(0.8, 1.6, dims)
        elif part == "mix.conv.b":
            value = 0.4 * rng.standard_normal(dims)
        elif part.endswith("conv"):
            value = rng.standard_normal(dims) * 1.2 / dims[-1] ** 0.5
        elif name in ("embed", "bigram"):
            value = (1.0 if name == "embed" else 0.7) * rng.standard_normal(dims)
        else:
            value = rng.standard_normal(dims) * 1.5 / dims[-1] ** 0.5
            if part in ("mix.q", "mix.uk"):
                value = value * 1.2 * sharp
        weights[name] = bf16(value)
    return weights
