"""TEST INFRASTRUCTURE ONLY -- CPU restatement (numpy, f64) of the Tobovik decoder: gated linear
attention with a decay per key channel, grouped-query softmax attention with whole-projection query /
key norms and a position-dependent query temperature, the two side by side in one layer, sinusoidal
positions added to the embedding, norms behind the sublayers and layers that share weights.

Only tests/ may import this module; the product path never does.  One function per mechanism, the
recurrence token by token and every softmax over an explicit list of visible keys.
"""
from __future__ import annotations

import numpy as np


def sigmoid(z):
    z = np.asarray(z, dtype=np.float64)
    return np.where(z < 0, np.exp(np.minimum(z, 0)) / (1.0 + np.exp(np.minimum(z, 0))), 1.0 / (1.0 + np.exp(-np.maximum(z, 0))))


def silu(z):
    return z * sigmoid(z)


def rms_norm(x, w, eps):
    """x / sqrt(mean(x^2) + eps) * w over the last axis."""
    x = np.asarray(x, dtype=np.float64)
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps) * np.asarray(w, dtype=np.float64)


def position_vectors(positions, width, base=10000.0):
    """[T, width]: pairs (sin, cos) of p * base^(-2i / width); an odd width ends with a sine."""
    i = np.arange((width + 1) // 2)
    angle = np.asarray(positions, dtype=np.float64)[:, None] * base ** (-2.0 * i / width)
    return np.stack([np.sin(angle), np.cos(angle)], axis=-1).reshape(len(angle), -1)[:, :width]


def query_temperature(positions, coef, every):
    p = np.asarray(positions, dtype=np.float64)
    return 1.0 + coef * np.log(np.floor((p + 1.0) / every) + 1.0)


def causal_attention(q, k, v, first_pos, scale):
    """q [T, H, D] at positions first_pos.., k [N, G, D], v [N, G, V] at positions 0..N-1; query head h
    reads key / value head h // (H / G)."""
    ratio = q.shape[1] // k.shape[1]
    out = np.zeros((q.shape[0], q.shape[1], v.shape[2]))
    for t in range(q.shape[0]):
        n = first_pos + t + 1
        for h in range(q.shape[1]):
            s = k[:n, h // ratio] @ q[t, h] * scale
            p = np.exp(s - s.max())
            out[t, h] = (p / p.sum()) @ v[:n, h // ratio]
    return out


def channel_decay(low, w2, bias, tau):
    """sigmoid(z)^(1 / tau), z = low . w2^T + bias."""
    z = low @ w2.T + bias
    return np.exp(-np.logaddexp(0.0, -z) / tau)


def gla_scan(q, k, v, alpha, state):
    """q, k, alpha [T, H, D], v [T, H, V], state [H, D, V] (changed in place): the state decays by key
    channel and takes in k v^T, then the query reads it."""
    out = np.zeros_like(v)
    for t in range(q.shape[0]):
        state *= alpha[t][:, :, None]
        state += k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hdv,hd->hv", state, q[t])
    return out


class TobovikOracle:
    """One sequence.  `config` is the parsed config.json, `weights` name -> array (values are used
    in f64).  step(tokens) continues the sequence and returns logits [T, vocab]; `residuals` holds
    the residual stream after every layer of the last step."""

    def __init__(self, config, weights):
        self.cfg = config
        self.w = {n: np.asarray(a, dtype=np.float64) for n, a in weights.items()}
        self.eps = float(config["norm"]["eps"])
        self.reset()

    def reset(self):
        self.pos = 0
        self.state = []
        for layer in self.cfg["layers"]:
            m = layer["mixer"]
            right = m["right"] if layer["type"] == "parallel" else m
            self.state.append({"S": np.zeros((right["heads"], right["dim"], right["vdim"])), "k": [], "v": []})

    def owner(self, i):
        while self.cfg["layers"][i].get("weights_of") is not None:
            i = self.cfg["layers"][i]["weights_of"]
        return i

    def _gla(self, p, m, st, h):
        w, heads, dim, vdim = self.w, m["heads"], m["dim"], m["vdim"]
        q = (h @ w[f"{p}.q"].T).reshape(-1, heads, dim) * dim ** -0.5
        k = (h @ w[f"{p}.k"].T).reshape(-1, heads, dim)
        v = (h @ w[f"{p}.v"].T).reshape(-1, heads, vdim)
        alpha = channel_decay(h @ w[f"{p}.a1"].T, w[f"{p}.a2"], w[f"{p}.a2.b"], float(m["tau"])).reshape(-1, heads, dim)
        o = rms_norm(gla_scan(q, k, v, alpha, st["S"]), w[f"{p}.norm"], self.eps).reshape(len(h), -1)
        return (o * silu(h @ w[f"{p}.g"].T)) @ w[f"{p}.o"].T

    def _attention(self, p, m, st, h):
        w, heads, groups, dim, vdim = self.w, m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        q = rms_norm(h @ w[f"{p}.q"].T + w[f"{p}.q.b"], w[f"{p}.q.norm"], self.eps)
        k = rms_norm(h @ w[f"{p}.k"].T + w[f"{p}.k.b"], w[f"{p}.k.norm"], self.eps)
        v = h @ w[f"{p}.v"].T + w[f"{p}.v.b"]
        q = q * query_temperature(self.pos + np.arange(len(h)), m["q_temp"]["coef"], m["q_temp"]["every"])[:, None]
        st["k"] += list(k.reshape(-1, groups, dim))
        st["v"] += list(v.reshape(-1, groups, vdim))
        o = causal_attention(q.reshape(-1, heads, dim), np.stack(st["k"]), np.stack(st["v"]), self.pos, m["scale"]).reshape(len(h), -1)
        return (o * sigmoid(h @ w[f"{p}.g"].T)) @ w[f"{p}.o"].T

    def step(self, tokens):
        w, cfg = self.w, self.cfg
        x = w["embed"][np.asarray(tokens)] + position_vectors(self.pos + np.arange(len(tokens)), cfg["width"])
        self.residuals = []
        for i, layer in enumerate(cfg["layers"]):
            name, m, st = f"l{self.owner(i)}", layer["mixer"], self.state[i]
            if layer["type"] == "parallel":
                y = m["left_scale"] * self._attention(f"{name}.mix.left", m["left"], st, x) + m["right_scale"] * self._gla(f"{name}.mix.right", m["right"], st, x)
            else:
                y = self._gla(f"{name}.mix", m, st, x)
            x = x + rms_norm(y, w[f"{name}.norm1"], self.eps)
            if layer.get("mlp"):
                f = f"{name}.mlp"
                y = (silu(x @ w[f"{f}.gate"].T) * (x @ w[f"{f}.up"].T)) @ w[f"{f}.down"].T
                x = x + rms_norm(y, w[f"{name}.norm2"], self.eps)
            self.residuals.append(x)
        self.pos += len(tokens)
        return rms_norm(x, w["final.norm"], self.eps) @ w["head"].T
