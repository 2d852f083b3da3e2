"""Plain restatement of the hybrid decoder (architecture Zofesun): numpy in double precision, one function per
mechanism, token by token where the mechanism is a recurrence. Test infrastructure only; it shares no code with
the library and reads weights as a plain name -> float array mapping.

Tensor names are those of the checkpoint: `embed`, `head`, `final.norm`, `loop.step`, and per layer i
`l<i>.norm1|norm1b|norm2|norm2b` (each with `.b` and `.alpha`), `l<i>.mix.*`, `l<i>.mlp.gate|up|down`.
"""
from __future__ import annotations

import copy

import numpy as np


def sigmoid(x):
    return 1.0 / (1.0 + np.exp(-x))


def silu(x):
    return x * sigmoid(x)


def rms(x, eps):
    """x scaled to unit mean square along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def dynamic_tanh(w, name, x):
    return np.tanh(float(w[name + ".alpha"].reshape(-1)[0]) * x) * w[name] + w[name + ".b"]


def rotate(x, positions, dims, base):
    """x [T, heads, dim]: pairs (i, i + dims / 2) of the first `dims` entries turned by position * base^(-2 i / dims)."""
    half = dims // 2
    angle = positions[:, None].astype(np.float64) * base ** (-2.0 * np.arange(half) / dims)
    c, s = np.cos(angle)[:, None, :], np.sin(angle)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., dims:]], axis=-1)


def sink_attention(q, k, v, scale, sink, first):
    """q [T, H, d] at positions first.. over k [N, G, d], v [N, G, dv] (N = first + T): causal softmax per query head
    with exp(sink_h) added to the denominator."""
    T, H, _ = q.shape
    N, G, dv = v.shape
    out = np.zeros((T, H, dv))
    causal = np.arange(N)[None, :] <= (first + np.arange(T))[:, None]
    for h in range(H):
        g = h // (H // G)
        score = np.where(causal, (q[:, h] @ k[:, g].T) * scale, -np.inf)
        top = np.maximum(score.max(axis=1), sink[h])
        weight = np.exp(score - top[:, None])
        out[:, h] = (weight @ v[:, g]) / (weight.sum(axis=1) + np.exp(sink[h] - top))[:, None]
    return out


def lightning(q, k, v, decay, state):
    """Decayed linear attention; q, k [T, H, d], v [T, H, dv], state [H, d, dv] (returned updated)."""
    out = np.zeros(v.shape)
    for t in range(q.shape[0]):
        state = decay[:, None, None] * state + k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hdv,hd->hv", state, q[t])
    return out, state


def min_gru(z, u, state):
    """z (gate) and u pre-activations [T, width]; state [width] (returned updated)."""
    gate = sigmoid(z)
    candidate = np.where(u >= 0, u + 0.5, sigmoid(u))
    out = np.zeros(z.shape)
    for t in range(z.shape[0]):
        state = (1.0 - gate[t]) * state + gate[t] * candidate[t]
        out[t] = state
    return out, state


def clamped_glu(gate, up, limit):
    g, u = np.minimum(gate, limit), np.clip(up, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


class HybridOracle:
    """One sequence: `forward(tokens)` appends tokens and returns their logits; `taps` then holds the stream
    as each layer run leaves it, without what the next pass adds."""

    def __init__(self, config, weights):
        self.c = config
        self.w = {name: np.asarray(value, dtype=np.float64) for name, value in weights.items()}
        layers = list(range(len(config["layers"])))
        loop = config.get("loop")
        self.runs = []                              # (layer, pass or None when nothing is added ahead of it)
        if loop:
            self.runs += [(i, None) for i in layers[:loop["start"]]]
            for t in range(loop["times"]):
                self.runs += [(i, t if i == loop["start"] else None) for i in layers[loop["start"]:loop["stop"]]]
            self.runs += [(i, None) for i in layers[loop["stop"]:]]
        else:
            self.runs = [(i, None) for i in layers]
        self.reset()

    def reset(self):
        self.position = 0
        self.state = [dict() for _ in self.runs]
        self.taps = []

    def truncate(self, length, snapshot):
        """Back to a snapshot taken with `save` at `length` tokens."""
        self.position, self.state = length, snapshot

    def save(self):
        return copy.deepcopy(self.state)

    # ---- mixers ----
    def mix_mingru(self, p, m, h, s):
        w = self.w
        z = h @ w[p + "z"].T + w[p + "z.b"]
        u = h @ w[p + "x"].T + w[p + "x.b"]
        out, s["s"] = min_gru(z, u, s.get("s", np.zeros(m["width"])))
        return (out * silu(h @ w[p + "g"].T)) @ w[p + "o"].T

    def attend(self, p, m, h, s):
        w, T = self.w, h.shape[0]
        q = (h @ w[p + "q"].T).reshape(T, m["heads"], m["dim"])
        k = (h @ w[p + "k"].T).reshape(T, m["kv_heads"], m["dim"])
        v = rms((h @ w[p + "v"].T).reshape(T, m["kv_heads"], m["vdim"]), self.c["norm"]["eps"])
        at = self.position + np.arange(T)
        q, k = (rotate(x, at, m["rot"]["dims"], m["rot"]["base"]) for x in (q, k))
        s["k"] = np.concatenate([s["k"], k]) if "k" in s else k
        s["v"] = np.concatenate([s["v"], v]) if "v" in s else v
        out = sink_attention(q, s["k"], s["v"], m["scale"], w[p + "sink"], self.position)
        return out.reshape(T, -1) @ w[p + "o"].T

    def linear_attend(self, p, m, h, s):
        w, T = self.w, h.shape[0]
        H = m["heads"]
        q = silu(h @ w[p + "q"].T).reshape(T, H, m["dim"])
        k = silu(h @ w[p + "k"].T).reshape(T, H, m["dim"])
        v = silu(h @ w[p + "v"].T).reshape(T, H, m["vdim"])
        out, s["s"] = lightning(q, k, v, np.asarray(m["decay"], dtype=np.float64),
                                s.get("s", np.zeros((H, m["dim"], m["vdim"]))))
        y = rms(out.reshape(T, -1), self.c["norm"]["eps"]) * w[p + "norm"]
        return (y * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T

    def mix(self, i, h, s):
        layer = self.c["layers"][i]
        p, m = f"l{i}.mix.", layer["mixer"]
        if layer["type"] == "mingru":
            return self.mix_mingru(p, m, h, s)
        assert layer["type"] == "parallel"
        left, right = s.setdefault("left", {}), s.setdefault("right", {})
        return (m["left_scale"] * self.attend(p + "left.", m["left"], h, left)
                + m["right_scale"] * self.linear_attend(p + "right.", m["right"], h, right))

    def forward(self, tokens):
        w, c = self.w, self.c
        embedded = w["embed"][np.asarray(tokens, dtype=np.int64)]
        x = embedded.copy()
        self.taps = []
        for run, (i, t) in enumerate(self.runs):
            if t is not None:
                if t:
                    x = x + embedded
                x = x + w["loop.step"][t]
            p = f"l{i}."
            x = x + dynamic_tanh(w, p + "norm1b", self.mix(i, dynamic_tanh(w, p + "norm1", x), self.state[run]))
            mlp = c["layers"][i]["mlp"]
            if mlp is not None:
                h = dynamic_tanh(w, p + "norm2", x)
                y = clamped_glu(h @ w[p + "mlp.gate"].T, h @ w[p + "mlp.up"].T, mlp["limit"]) @ w[p + "mlp.down"].T
                x = x + dynamic_tanh(w, p + "norm2b", y)
            self.taps.append(x.copy())
        self.position += len(tokens)
        return dynamic_tanh(w, "final.norm", x) @ w["head"].T
