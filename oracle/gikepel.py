"""Plain restatement of the Gikepel decoder: numpy in double precision, one function per mechanism, token by token where
the mechanism is a recurrence. Test infrastructure only; it shares no code with the library and reads weights as a plain
name -> float array mapping.

Tensor names are those of the checkpoint: `embed`, `bigram`, `final.norm`, and per layer i `l<i>.norm1|norm2|ls1|ls2`,
`l<i>.mix.*`, `l<i>.mlp.up|down`.
"""
from __future__ import annotations

import copy
import math

import numpy as np


def sigmoid(x):
    return 1.0 / (1.0 + np.exp(-x))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return np.logaddexp(0.0, x)


def rms(x, eps):
    """x scaled to unit mean square along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def layer_norm(x, weight, eps):
    centred = x - x.mean(axis=-1, keepdims=True)
    return rms(centred, eps) * weight


def unit(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def relu_squared(x):
    return np.maximum(x, 0.0) ** 2


def soft_cap(x, cap):
    return cap * np.tanh(x / cap)


def bigram_rows(previous, tokens, buckets, mul_prev, mul_cur):
    """Row of the pair table for every token; `previous` is the token ahead of the first one, or None."""
    rows = []
    for token in tokens:
        rows.append(buckets if previous is None else (int(previous) * mul_prev + int(token) * mul_cur) % buckets)
        previous = token
    return np.array(rows)


def yarn(dims, base, scaling):
    """(frequencies, length factor) of a rotation over `dims` entries."""
    i = np.arange(dims // 2, dtype=np.float64)
    plain = base ** (-2.0 * i / dims)
    if scaling is None:
        return plain, 1.0
    factor, original = scaling["factor"], scaling["original"]

    def turns(t):
        return dims * math.log(original / (2.0 * math.pi * t)) / (2.0 * math.log(base))

    low = max(math.floor(turns(scaling["fast"])), 0)
    high = min(math.ceil(turns(scaling["slow"])), dims - 1)
    ramp = np.clip((i - low) / max(high - low, 0.001), 0.0, 1.0)
    return plain / factor * ramp + plain * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


def rotate_pairs(x, positions, frequencies, length):
    """x [T, heads, n]: entries (2 i, 2 i + 1) turned by position * frequencies[i] and scaled by `length`; entries
    beyond the frequencies stay."""
    angle = np.asarray(positions, dtype=np.float64)[:, None] * frequencies
    c, s = length * np.cos(angle)[:, None, :], length * np.sin(angle)[:, None, :]
    dims = 2 * len(frequencies)
    out = np.array(x, dtype=np.float64)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


def latent_attention(q, q_turned, latent, key_turned, up_key, up_value, scale, first):
    """q [T, H, d] and q_turned [T, H, r] at positions first.. over latent [N, R] and key_turned [N, r]; keys and values
    are made from the latent by up_key [H, d, R] and up_value [H, dv, R]. Causal softmax. Returns [T, H, dv]."""
    T, H, _ = q.shape
    N = latent.shape[0]
    causal = np.arange(N)[None, :] <= (first + np.arange(T))[:, None]
    out = np.zeros((T, H, up_value.shape[1]))
    for h in range(H):
        keys, values = latent @ up_key[h].T, latent @ up_value[h].T
        score = (q[:, h] @ keys.T + q_turned[:, h] @ key_turned.T) * scale
        score = np.where(causal, score, -np.inf)
        weight = np.exp(score - score.max(axis=1, keepdims=True))
        out[:, h] = weight @ values / weight.sum(axis=1, keepdims=True)
    return out


def short_conv(x, kernel, history, bias=None):
    """Causal convolution per channel; x [T, C], kernel [C, taps] (last column: the current token), history [taps - 1, C].
    Returns (output, the next history)."""
    taps = kernel.shape[1]
    padded = np.concatenate([history, x])
    out = np.zeros(x.shape)
    for j in range(taps):
        out += padded[j:j + len(x)] * kernel[:, j]
    if bias is not None:
        out = out + bias
    return out, padded[len(padded) - (taps - 1):]


def state_space(x, b, c, dt, a_log, skip, state):
    """x [T, H, dv], b and c [T, G, N], dt [T, H] (after softplus); state [H, N, dv] (returned updated)."""
    T, H, _ = x.shape
    G = b.shape[1]
    out = np.zeros(x.shape)
    state = state.copy()
    for t in range(T):
        for h in range(H):
            g = h // (H // G)
            state[h] = np.exp(-np.exp(a_log[h]) * dt[t, h]) * state[h] + dt[t, h] * np.outer(b[t, g], x[t, h])
            out[t, h] = state[h].T @ c[t, g] + skip[h] * x[t, h]
    return out, state


def channel_delta(q, k, v, log_decay, beta, state):
    """q, k [T, G, d], v [T, H, dv], log_decay [T, H, d], beta [T, H]; state [H, d, dv] (returned updated)."""
    T, H, _ = v.shape
    G = q.shape[1]
    out = np.zeros(v.shape)
    state = state.copy()
    for t in range(T):
        for h in range(H):
            g = h // (H // G)
            s = np.exp(log_decay[t, h])[:, None] * state[h]
            s = s + np.outer(k[t, g], beta[t, h] * (v[t, h] - s.T @ k[t, g]))
            state[h], out[t, h] = s, s.T @ q[t, g]
    return out, state


class GikepelOracle:
    """One sequence: `forward(tokens)` appends tokens and returns their logits; `taps` then holds the stream as each
    layer leaves it."""

    def __init__(self, config, weights):
        self.c = config
        self.w = {name: np.asarray(value, dtype=np.float64) for name, value in weights.items()}
        self.eps = config["norm"]["eps"]
        self.runs = [(i, None) for i in range(len(config["layers"]))]
        self.reset()

    def reset(self):
        self.position = 0
        self.state = [dict() for _ in self.c["layers"]] + [{"token": None}]
        self.taps = []

    def truncate(self, length, snapshot):
        """Back to a snapshot taken with `save` at `length` tokens."""
        self.position, self.state = length, snapshot

    def save(self):
        return copy.deepcopy(self.state)

    # ---- mixers ----
    def convolve(self, s, key, kernel, x, bias=None):
        out, s[key] = short_conv(x, kernel, s.get(key, np.zeros((kernel.shape[1] - 1, x.shape[1]))), bias)
        return silu(out)

    def mix_latent_attention(self, p, m, h, s):
        w, T, H = self.w, h.shape[0], m["heads"]
        d, r, dv, rank = m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        q = (h @ w[p + "q"].T).reshape(T, H, d + r)
        down = h @ w[p + "dkv"].T
        latent = rms(down[:, :rank], self.eps) * w[p + "dkv.norm"]
        frequencies, length = yarn(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
        at = self.position + np.arange(T)
        q_turned = rotate_pairs(q[..., d:], at, frequencies, length)
        key_turned = rotate_pairs(down[:, None, rank:], at, frequencies, length)[:, 0]
        s["latent"] = np.concatenate([s["latent"], latent]) if "latent" in s else latent
        s["turned"] = np.concatenate([s["turned"], key_turned]) if "turned" in s else key_turned
        out = latent_attention(q[..., :d], q_turned, s["latent"], s["turned"], w[p + "uk"].reshape(H, d, rank),
                               w[p + "uv"].reshape(H, dv, rank), m["scale"], self.position)
        return (out.reshape(T, -1) * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T

    def mix_mamba2(self, p, m, h, s):
        w, T, H = self.w, h.shape[0], m["heads"]
        dv, N, G = m["vdim"], m["state"], m["groups"]
        inner = H * dv
        z, mixed, dt = np.split(h @ w[p + "in"].T, [inner, 2 * inner + 2 * G * N], axis=1)
        mixed = self.convolve(s, "conv", w[p + "conv"], mixed, w[p + "conv.b"])
        x, b, c = np.split(mixed, [inner, inner + G * N], axis=1)
        y, s["s"] = state_space(x.reshape(T, H, dv), b.reshape(T, G, N), c.reshape(T, G, N), softplus(dt + w[p + "dt_bias"]),
                                w[p + "A_log"], w[p + "D"], s.get("s", np.zeros((H, N, dv))))
        y = y.reshape(T, inner) * silu(z)
        y = rms(y.reshape(T, m["norm_groups"], -1), self.eps).reshape(T, inner) * w[p + "norm"]
        return y @ w[p + "o"].T

    def mix_channel_delta(self, p, m, h, s):
        w, T, H, G = self.w, h.shape[0], m["heads"], m["kv_heads"]
        d, dv = m["dim"], m["vdim"]
        q, k, v = (self.convolve(s, name, w[p + name + ".conv"], h @ w[p + name].T) for name in "qkv")
        q, k = unit(q.reshape(T, G, d)) * d ** -0.5, unit(k.reshape(T, G, d))
        decay = softplus((h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]).reshape(T, H, d)
        decay = -np.exp(w[p + "A_log"])[None, :, None] * decay
        out, s["s"] = channel_delta(q, k, v.reshape(T, H, dv), decay, sigmoid(h @ w[p + "b"].T),
                                    s.get("s", np.zeros((H, d, dv))))
        gate = sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T)
        return ((rms(out, self.eps) * w[p + "norm"]).reshape(T, -1) * gate) @ w[p + "o"].T

    def forward(self, tokens):
        w, c = self.w, self.c
        tokens = [int(t) for t in tokens]
        x = w["embed"][tokens]
        pairs = c["embedding"]["bigram"]
        x = x + w["bigram"][bigram_rows(self.state[-1]["token"], tokens, pairs["buckets"], pairs["mul_prev"], pairs["mul_cur"])]
        self.state[-1]["token"] = tokens[-1]
        self.taps = []
        for i, layer in enumerate(c["layers"]):
            p = f"l{i}."
            mixer = getattr(self, "mix_" + layer["type"])
            add = mixer(p + "mix.", layer["mixer"], layer_norm(x, w[p + "norm1"], self.eps), self.state[i]) * w[p + "ls1"]
            if layer["mlp"] is not None:
                h = layer_norm(x, w[p + "norm2"], self.eps)
                add = add + relu_squared(h @ w[p + "mlp.up"].T) @ w[p + "mlp.down"].T * w[p + "ls2"]
            x = x + add
            self.taps.append(x.copy())
        self.position += len(tokens)
        return soft_cap(layer_norm(x, w["final.norm"], self.eps) @ w["embed"].T, c["logit_softcap"])
