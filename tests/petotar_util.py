"""Small random Petotar models for the tests: configurations, bf16-representable weights, comparison."""
import numpy as np

from meganeura_b200.weights import to_bf16, write_safetensors


def bf16_round(a):
    return (to_bf16(a).astype(np.uint32) << 16).view(np.float32)


def wkv(heads, dim, ff=0, limit=1.0):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim}, "mlp": {"kind": "dense", "ff": ff, "limit": limit} if ff else None}


def mlstm(heads, dim, vdim, cap, ff=0, limit=1.0):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap},
            "mlp": {"kind": "dense", "ff": ff, "limit": limit} if ff else None}


def latent(heads, dim, rot_dim, vdim, rank, window, base=1e4, scale=None, kv_from=None, ff=0, limit=1.0):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "mask": {"size": window},
         "rot": {"base": base, "dims": rot_dim}, "scale": scale if scale is not None else (dim + rot_dim) ** -0.5}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff, "limit": limit} if ff else None}


def config(vocab, width, layers, eps=1e-5, scale=3.0):
    return {"architecture": "Petotar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers}


# name -> (config, rows of w1 per wkv layer).  "odd" has no size that vector code would like.
CONFIGS = {
    "mixed": (config(320, 128, [latent(4, 32, 8, 24, 48, 21, ff=144, limit=2.0), mlstm(3, 16, 40, 6.0, ff=96, limit=0.7), wkv(2, 64, ff=160),
                                latent(3, 16, 8, 32, 48, 33, kv_from=0, scale=0.3), mlstm(2, 64, 24, 15.0), wkv(5, 16, ff=64, limit=3.0)]), 8),
    "odd": (config(203, 90, [wkv(3, 22, ff=51, limit=0.9), latent(5, 18, 6, 13, 27, 9, base=500.0), mlstm(1, 35, 17, 3.5, ff=33),
                             latent(2, 10, 6, 20, 27, 30, base=500.0, kv_from=1, ff=70)], eps=1e-3, scale=1.0), 5),
    "wide": (config(512, 256, [mlstm(2, 128, 96, 10.0, ff=320), latent(12, 64, 32, 64, 256, 70, base=2e5, ff=256), wkv(2, 128, ff=256)], eps=1e-6,
                    scale=1.5), 32),
}


def weights(cfg, rank, seed=0):
    """name -> f32 array of bf16-representable values."""
    rng = np.random.Generator(np.random.PCG64(seed))
    out = {}

    def mat(name, n, k, gain=1.0):
        out[name] = bf16_round(rng.standard_normal((n, k)).astype(np.float32) * np.float32(gain / np.sqrt(k)))

    def vec(name, n, std=0.3, mean=0.0):
        out[name] = bf16_round((rng.standard_normal(n) * std + mean).astype(np.float32))

    w = cfg["width"]
    out["embed"] = bf16_round(rng.standard_normal((cfg["vocab"], w)).astype(np.float32) * np.float32(w ** -0.5))
    vec("final.norm", w)
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix", layer["mixer"]
        n = m["heads"] * m["dim"]
        vec(f"l{i}.norm1", w)
        if layer["type"] == "wkv":
            for s in "rkvgw":
                out[f"{p}.mu.{s}"] = bf16_round(rng.uniform(0.0, 1.0, w).astype(np.float32))
            for s in "rkvg":
                mat(f"{p}.{s}", n, w)
            mat(f"{p}.w1", rank, w)
            mat(f"{p}.w2", n, rank)
            out[f"{p}.w0"] = bf16_round(rng.uniform(-5.0, 0.5, n).astype(np.float32))
            vec(f"{p}.u", n)
            out[f"{p}.u"] = out[f"{p}.u"].reshape(m["heads"], m["dim"])
            vec(f"{p}.norm", n, mean=1.0)
            mat(f"{p}.o", w, n)
        elif layer["type"] == "mlstm":
            nv = m["heads"] * m["vdim"]
            mat(f"{p}.q", n, w)
            mat(f"{p}.k", n, w)
            mat(f"{p}.v", nv, w)
            mat(f"{p}.g", nv, w)
            mat(f"{p}.i", m["heads"], w, 1.5)
            mat(f"{p}.f", m["heads"], w, 1.5)
            vec(f"{p}.i.b", m["heads"], 2.0)
            vec(f"{p}.f.b", m["heads"], 1.0, 2.5)
            vec(f"{p}.norm", nv, mean=1.0)
            mat(f"{p}.o", w, nv)
        else:
            mat(f"{p}.q", m["heads"] * (m["dim"] + m["rot_dim"]), w, 2.5)
            if m.get("kv_from") is None:
                mat(f"{p}.dkv", m["kv_rank"] + m["rot_dim"], w)
                vec(f"{p}.dkv.norm", m["kv_rank"], mean=1.0)
            mat(f"{p}.uk", n, m["kv_rank"])
            mat(f"{p}.uv", m["heads"] * m["vdim"], m["kv_rank"])
            mat(f"{p}.g", m["heads"] * m["vdim"], w)
            mat(f"{p}.o", w, m["heads"] * m["vdim"])
        if layer["mlp"]:
            f, ff = f"l{i}.mlp", layer["mlp"]["ff"]
            vec(f"l{i}.norm2", w)
            for s in ("gate", "up"):
                mat(f"{f}.{s}", ff, w, 1.5)
                vec(f"{f}.{s}.b", ff)
            mat(f"{f}.down", w, ff)
            vec(f"{f}.down.b", w)
    return out


class Tensors:
    """What Petotar.load reads, from arrays in memory."""

    def __init__(self, arrays):
        self.arrays = arrays

    def shape(self, name):
        return self.arrays[name].shape

    def dtype(self, name):
        return "BF16"

    def raw(self, name):
        return to_bf16(self.arrays[name])

    def f32(self, name):
        return self.arrays[name].astype(np.float32)


def write_folder(folder, cfg, arrays):
    import json
    import os
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(folder, "model.safetensors"), {n: ("BF16", to_bf16(a)) for n, a in arrays.items()})


def row_errors(got, want):
    """RMS error of every row over the RMS spread of the wanted logits (a constant offset does not count)."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    d = got - want
    d -= d.mean(axis=-1, keepdims=True)
    return np.sqrt((d * d).mean(axis=-1)) / want.std()
