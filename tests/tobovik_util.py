"""Small random Tobovik models for the tests: configurations and bf16-representable weights."""
import numpy as np

from petotar_util import bf16_round


def gla(heads, dim, vdim, tau=16.0, ff=0, weights_of=None):
    return _layer("gla", dict(heads=heads, dim=dim, vdim=vdim, tau=tau), ff, weights_of)


def attention(heads, kv_heads, dim, vdim, scale=None, coef=0.2, every=32):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=dim ** -0.5 if scale is None else scale, q_temp=dict(coef=coef, every=every))


def parallel(left, right, left_scale=1.0, right_scale=1.0, ff=0, weights_of=None):
    return _layer("parallel", dict(left=left, right=right, left_scale=left_scale, right_scale=right_scale), ff, weights_of)


def side(heads, dim, vdim, tau=16.0):
    return dict(heads=heads, dim=dim, vdim=vdim, tau=tau)


def _layer(kind, mixer, ff, weights_of):
    out = {"type": kind, "mixer": mixer, "mlp": {"kind": "dense", "ff": ff} if ff else None}
    if weights_of is not None:
        out["weights_of"] = weights_of
    return out


def config(vocab, width, layers, eps=1e-5):
    return {"architecture": "Tobovik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


def _shared():
    a, g = parallel(attention(6, 2, 24, 40, 0.3, 0.25, 16), side(3, 40, 24, 8.0), 0.7, 1.1, 96), gla(2, 72, 56, 4.0, 64)
    return [g, a, dict(a, weights_of=1), dict(g, weights_of=0), dict(g, weights_of=3)]


# name -> (config, rows of a1).  "odd" has no size that vector code would like, "wide" key sizes for which the kernels
# have other instances, "shared" layers that use other layers' weights (one through another), "plain" one head of everything.
CONFIGS = {
    "shared": (config(320, 128, _shared()), 8),
    "odd": (config(203, 90, [parallel(attention(5, 5, 18, 13, 0.4, 0.5, 7), side(3, 22, 9, 2.0), 1.3, 0.6), gla(1, 35, 17, 5.0, 51),
                             parallel(attention(3, 1, 7, 30, coef=0.0), side(2, 10, 21), 0.5, -0.8, 33)], eps=1e-3), 5),
    "wide": (config(512, 256, [gla(1, 136, 200, ff=256), parallel(attention(8, 1, 144, 72, 0.1), side(2, 64, 128), ff=320),
                               parallel(attention(2, 2, 64, 264), side(1, 256, 40, 32.0), 0.9, 0.4)], eps=1e-6), 16),
    "plain": (config(150, 48, [parallel(attention(1, 1, 32, 32, 1.0, 1.0, 1), side(1, 32, 32, 1.0))], eps=1e-6), 1),
}


def weights(cfg, rank, seed=0):
    """name -> f32 array of bf16-representable values."""
    rng = np.random.Generator(np.random.PCG64(seed))
    out, w = {}, cfg["width"]

    def mat(name, n, k, gain=1.0):
        out[name] = bf16_round(rng.standard_normal((n, k)).astype(np.float32) * np.float32(gain / np.sqrt(k)))

    def vec(name, n, std=0.3, mean=0.0):
        out[name] = bf16_round((rng.standard_normal(n) * std + mean).astype(np.float32))

    def gla_weights(p, m):
        n, nv = m["heads"] * m["dim"], m["heads"] * m["vdim"]
        for s, k in (("q", n), ("k", n), ("v", nv), ("g", nv), ("a1", rank)):
            mat(f"{p}.{s}", k, w)
        mat(f"{p}.a2", n, rank, 2.0)
        vec(f"{p}.a2.b", n, 2.0, 1.0)
        vec(f"{p}.norm", m["vdim"], mean=1.0)
        mat(f"{p}.o", w, nv)

    mat("embed", cfg["vocab"], w, np.sqrt(w))
    mat("head", cfg["vocab"], w)
    vec("final.norm", w, mean=1.0)
    for i, layer in enumerate(cfg["layers"]):
        if layer.get("weights_of") is not None:
            continue
        m = layer["mixer"]
        vec(f"l{i}.norm1", w, mean=1.0)
        if layer["type"] == "parallel":
            a, p = m["left"], f"l{i}.mix.left"
            sizes = dict(q=a["heads"] * a["dim"], k=a["kv_heads"] * a["dim"], v=a["kv_heads"] * a["vdim"])
            for s, n in sizes.items():
                mat(f"{p}.{s}", n, w)
                vec(f"{p}.{s}.b", n)
            vec(f"{p}.q.norm", sizes["q"], mean=1.5)
            vec(f"{p}.k.norm", sizes["k"], mean=1.5)
            mat(f"{p}.g", a["heads"] * a["vdim"], w)
            mat(f"{p}.o", w, a["heads"] * a["vdim"])
            gla_weights(f"l{i}.mix.right", m["right"])
        else:
            gla_weights(f"l{i}.mix", m)
        if layer["mlp"]:
            f, ff = f"l{i}.mlp", layer["mlp"]["ff"]
            vec(f"l{i}.norm2", w, mean=1.0)
            mat(f"{f}.gate", ff, w, 1.5)
            mat(f"{f}.up", ff, w, 1.5)
            mat(f"{f}.down", w, ff)
    return out
