"""TEST INFRASTRUCTURE ONLY -- CPU restatement (numpy, f64) of the mixers, the feed-forward and the
whole forward pass of the Petotar decoder: RWKV-style time mixing, the mLSTM matrix memory, latent
attention over a sliding window, a clamped GLU, and norms whose weight is stored around zero.

Only tests/ may import this module; the product path never does.  One function per mechanism, every
recurrence token by token and every softmax over an explicit list of visible keys.
"""
from __future__ import annotations

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-np.asarray(z, dtype=np.float64)))


def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    x = np.asarray(x, dtype=np.float64)
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps)


def norm_around_zero(x, w, eps):
    return unit_rms(x, eps) * (1.0 + np.asarray(w, dtype=np.float64))


def rotate_half(x, pos, base):
    """Rotary positions on the whole last axis (dims wide): dimension i turns with i + dims/2."""
    dims = x.shape[-1]
    half = dims // 2
    freq = float(base) ** (-2.0 * np.arange(half) / dims)
    a = float(pos) * freq
    u, v = x[..., :half], x[..., half:]
    return np.concatenate([u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a)], axis=-1)


def token_shift(h, prev, mu):
    """h + (previous token's h - h) * mu for every token; prev is the h before the first one."""
    before = np.concatenate([prev[None, :], h[:-1]], axis=0)
    return h + (before - h) * mu


def wkv_decay(mix_w, w1, w2, w0):
    return np.exp(-np.exp(np.tanh(mix_w @ w1.T) @ w2.T + w0))


def wkv_scan(r, k, v, w, u, state):
    """r, k, v, w [T, H, D], u [H, D], state [H, D, D] (key row, value column; changed in place)."""
    out = np.zeros_like(r)
    for t in range(r.shape[0]):
        for h in range(r.shape[1]):
            kv = np.outer(k[t, h], v[t, h])
            out[t, h] = (state[h] + u[h][:, None] * kv).T @ r[t, h]
            state[h] = w[t, h][:, None] * state[h] + kv
    return out


def mlstm_gates(pre_i, pre_f, cap):
    """Log input gate and log forget gate from the biased pre-activations."""
    f = cap * np.tanh(pre_f / cap)
    return cap * np.tanh(pre_i / cap), -np.logaddexp(0.0, -f)


def mlstm_scan(q, k, v, log_i, log_f, S, n, m):
    """q, k [T, H, D], v [T, H, V], gates [T, H]; S [H, D, V], n [H, D], m [H] change in place."""
    out = np.zeros_like(v)
    for t in range(q.shape[0]):
        for h in range(q.shape[1]):
            m_new = max(log_f[t, h] + m[h], log_i[t, h])
            keep, write = np.exp(log_f[t, h] + m[h] - m_new), np.exp(log_i[t, h] - m_new)
            S[h] = keep * S[h] + write * np.outer(k[t, h], v[t, h])
            n[h] = keep * n[h] + write * k[t, h]
            m[h] = m_new
            out[t, h] = (S[h].T @ q[t, h]) / (max(abs(n[h] @ q[t, h]), np.exp(-m_new)) + 1e-6)
    return out


def window_attention(q, k, v, first_pos, window, scale):
    """q [T, H, D] at positions first_pos.., k [N, H, D], v [N, H, V] at positions 0..N-1."""
    out = np.zeros((q.shape[0], q.shape[1], v.shape[2]))
    for t in range(q.shape[0]):
        i = first_pos + t
        visible = [j for j in range(k.shape[0]) if 0 <= i - j < window]
        for h in range(q.shape[1]):
            s = k[visible, h] @ q[t, h] * scale
            p = np.exp(s - s.max())
            out[t, h] = (p / p.sum()) @ v[visible, h]
    return out


def clamped_glu(gate, up, limit):
    g = np.minimum(gate, limit)
    return g * sigmoid(1.702 * g) * (np.clip(up, -limit, limit) + 1.0)


class PetotarOracle:
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
            if layer["type"] == "wkv":
                self.state.append({"prev": np.zeros(self.cfg["width"]), "S": np.zeros((m["heads"], m["dim"], m["dim"]))})
            elif layer["type"] == "mlstm":
                self.state.append({"S": np.zeros((m["heads"], m["dim"], m["vdim"])), "n": np.zeros((m["heads"], m["dim"])),
                                   "m": np.zeros(m["heads"])})
            else:
                self.state.append({"c": [], "kr": []})

    def _wkv(self, p, m, st, h):
        w, heads, dim = self.w, m["heads"], m["dim"]
        mix = {s: token_shift(h, st["prev"], w[f"{p}.mu.{s}"]) for s in "rkvgw"}
        r, k, v = ((mix[s] @ w[f"{p}.{s}"].T).reshape(-1, heads, dim) for s in "rkv")
        gate = mix["g"] @ w[f"{p}.g"].T
        decay = wkv_decay(mix["w"], w[f"{p}.w1"], w[f"{p}.w2"], w[f"{p}.w0"]).reshape(-1, heads, dim)
        o = wkv_scan(r, k, v, decay, w[f"{p}.u"], st["S"])
        st["prev"] = h[-1].copy()
        o = unit_rms(o, self.eps).reshape(h.shape[0], -1) * w[f"{p}.norm"]
        return (o * gate * sigmoid(gate)) @ w[f"{p}.o"].T

    def _mlstm(self, p, m, st, h):
        w, heads, dim, vdim, cap = self.w, m["heads"], m["dim"], m["vdim"], float(m["gate_cap"])
        q = (h @ w[f"{p}.q"].T).reshape(-1, heads, dim) * dim ** -0.5
        k = (h @ w[f"{p}.k"].T).reshape(-1, heads, dim)
        v = (h @ w[f"{p}.v"].T).reshape(-1, heads, vdim)
        log_i, log_f = mlstm_gates(h @ w[f"{p}.i"].T + w[f"{p}.i.b"], h @ w[f"{p}.f"].T + w[f"{p}.f.b"], cap)
        o = mlstm_scan(q, k, v, log_i, log_f, st["S"], st["n"], st["m"])
        o = unit_rms(o, self.eps).reshape(h.shape[0], -1) * w[f"{p}.norm"]
        return (o * sigmoid(h @ w[f"{p}.g"].T)) @ w[f"{p}.o"].T

    def _latent(self, p, m, st, h, index):
        w, heads, dim, rot, vdim, rank = self.w, m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        q = (h @ w[f"{p}.q"].T).reshape(-1, heads, dim + rot)
        base = m["rot"]["base"]
        q = np.stack([np.concatenate([q[t, :, :dim], rotate_half(q[t, :, dim:], self.pos + t, base)], axis=-1) for t in range(len(q))])
        source = st
        if m.get("kv_from") is not None:
            source = self.state[m["kv_from"]]
        else:
            down = h @ w[f"{p}.dkv"].T
            for t in range(len(down)):
                st["c"].append(unit_rms(down[t, :rank], self.eps) * w[f"{p}.dkv.norm"])
                st["kr"].append(rotate_half(down[t, rank:], self.pos + t, base))
        c, kr = np.stack(source["c"]), np.stack(source["kr"])
        k = (c @ w[f"{p}.uk"].T).reshape(-1, heads, dim)
        k = np.concatenate([k, np.repeat(kr[:, None, :], heads, axis=1)], axis=-1)
        v = (c @ w[f"{p}.uv"].T).reshape(-1, heads, vdim)
        o = window_attention(q, k, v, self.pos, m["mask"]["size"], m["scale"]).reshape(h.shape[0], -1)
        return (o * sigmoid(h @ w[f"{p}.g"].T)) @ w[f"{p}.o"].T

    def step(self, tokens):
        w, cfg = self.w, self.cfg
        x = w["embed"][np.asarray(tokens)] * float(cfg["embedding"]["scale"])
        self.residuals = []
        for i, layer in enumerate(cfg["layers"]):
            h = norm_around_zero(x, w[f"l{i}.norm1"], self.eps)
            p, m, st = f"l{i}.mix", layer["mixer"], self.state[i]
            if layer["type"] == "wkv":
                x = x + self._wkv(p, m, st, h)
            elif layer["type"] == "mlstm":
                x = x + self._mlstm(p, m, st, h)
            else:
                x = x + self._latent(p, m, st, h, i)
            if layer.get("mlp"):
                h, f = norm_around_zero(x, w[f"l{i}.norm2"], self.eps), f"l{i}.mlp"
                y = clamped_glu(h @ w[f"{f}.gate"].T + w[f"{f}.gate.b"], h @ w[f"{f}.up"].T + w[f"{f}.up.b"], float(layer["mlp"]["limit"]))
                x = x + y @ w[f"{f}.down"].T + w[f"{f}.down.b"]
            self.residuals.append(x)
        self.pos += len(tokens)
        return norm_around_zero(x, w["final.norm"], self.eps) @ w["embed"].T
