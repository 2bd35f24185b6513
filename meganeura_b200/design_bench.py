"""Prefill and decode throughput of a row-dynamic design at sizes of real models' layers (seeded random
weights), the kernels' distance from their rooflines, and the closest decoder of this package at equal
width, layer count and vocabulary (bench.py --design petotar|tobovik)."""
from __future__ import annotations

import time

import numpy as np

from . import decode_model as M
from ._lib import ROWS_PICKED, ROWS_TOKENS
from .engine import Engine
from .graph import ShaderEntry as S
from .petotar import Petotar, PetotarConfig
from .tobovik import Tobovik, TobovikConfig, gla_prefixes
from .weights import to_bf16


def _layers(kind, ff, wkv, mlstm, latent):
    out = []
    for k in kind:
        m = {"w": dict(type="wkv", mixer=dict(wkv)), "m": dict(type="mlstm", mixer=dict(mlstm)), "a": dict(type="latent_attention", mixer=dict(latent)),
             "s": dict(type="latent_attention", mixer=dict(latent, kv_from=kind.index("a")))}[k]
        out.append(dict(m, mlp={"kind": "dense", "ff": ff, "limit": 7.0}))
    return out


def _tobovik_layers(kind, ff, left, right, gla):
    out = []
    for k in kind:
        m = dict(type="gla", mixer=dict(gla)) if k == "g" else dict(type="parallel", mixer=dict(left=left, right=right, left_scale=0.7, right_scale=1.0))
        out.append(dict(m, mlp={"kind": "dense", "ff": ff}))
    return out


# design -> name -> (config, rank of the decay projection, what it stands beside: a design, or a decoder of the package)
def sizes(design):
    def cfg(architecture, vocab, width, layers, **more):
        return dict({"architecture": architecture, "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "layers": layers}, **more)
    if design == "petotar":
        latent2 = dict(heads=16, dim=128, rot_dim=64, vdim=128, kv_rank=512, mask={"size": 2048}, rot={"base": 1e6, "dims": 64}, scale=192 ** -0.5)
        latent4 = dict(latent2, heads=32)
        one = {"embedding": {"scale": 1.0}}
        a = cfg("Petotar", 32768, 2048, _layers("wamwsm", 6144, dict(heads=32, dim=64), dict(heads=8, dim=128, vdim=256, gate_cap=15.0), latent2), **one)
        b = cfg("Petotar", 151936, 4096, _layers("wamwsm", 12288, dict(heads=64, dim=64), dict(heads=16, dim=128, vdim=256, gate_cap=15.0), latent4), **one)
        like_a = M.DecoderConfig("decoder-2048", 32768, 2048, 6, 16, 4, 128, 6144, 1e-6, 1e6, M.FMT_Q4, M.FMT_Q4, M.FMT_Q4)
        like_b = M.replace(M.QWEN3_8B, name="decoder-4096", num_hidden_layers=6)
        return {"2048": (a, 64, like_a), "4096": (b, 64, like_b)}
    def mixers(heads):
        left = dict(heads=heads, kv_heads=heads // 4, dim=128, vdim=128, scale=128 ** -0.5, q_temp={"coef": 0.1, "every": 8192})
        return left, dict(heads=heads // 2, dim=128, vdim=256, tau=16.0), dict(heads=heads // 4, dim=256, vdim=512, tau=16.0)
    return {"2048": (cfg("Tobovik", 32768, 2048, _tobovik_layers("pgppgp", 6144, *mixers(16))), 16, "petotar"),
            "4096": (cfg("Tobovik", 151936, 4096, _tobovik_layers("pgppgp", 12288, *mixers(32))), 16, "petotar")}


def random_model(config, rank, **kw):
    if config["architecture"] == "Tobovik":
        cfg = TobovikConfig.from_dict(config)
        model = Tobovik(cfg, lora_rank={p: rank for p in gla_prefixes(cfg)}, **kw)
    else:
        cfg = PetotarConfig.from_dict(config)
        model = Petotar(cfg, lora_rank={i: rank for i, layer in enumerate(cfg.layers) if layer.type == "wkv"}, **kw)
    rng = np.random.Generator(np.random.PCG64(5))
    noise = rng.standard_normal(1 << 22, dtype=np.float32)
    around_one = isinstance(model, Tobovik)                  # norm weights: stored plain, or around zero
    for idx, (name, shape, bf16) in enumerate(model.parameters()):
        n = int(np.prod(shape))
        start = (idx * 7919) % 65536
        a = np.resize(noise[start:], n) if n > noise.size - start else noise[start:start + n]
        if bf16:
            model.session.upload_param(name, to_bf16(a * np.float32(shape[1] ** -0.5)))
        elif ".mu." in name:
            model.session.set_parameter(name, 1.0 / (1.0 + np.exp(-a)))
        elif name.endswith(".a2.b"):
            model.session.set_parameter(name, a * 1.5 + 2.0)
        elif "norm" in name.rsplit(".", 1)[-1] and (around_one or ".mix." in name):
            model.session.set_parameter(name, a * 0.1 + 1.0)
        elif name.endswith(".w0") and ".mix." in name:
            model.session.set_parameter(name, a * 0.1 - 3.0)
        else:
            model.session.set_parameter(name, a * 0.1 + (3.0 if name.endswith(".f.b") else 0.0))
    return model


def work(model, d, rows: int, pos: int):
    """(algorithmic bytes, flops) of one dispatch for `rows` tokens that start at position `pos`."""
    p, shader = d.params, d.shader
    act = 2 if model.dtype == "bfloat16" else 4
    if shader in (S.Linear, S.LinearGLU):
        r = 1 if p[2] == model.cfg.vocab else rows
        weights = 2 * p[1] * p[2] if shader == S.LinearGLU else p[3]
        out = act if shader == S.LinearGLU else 8 if d.label.endswith("+Add") else 4
        return 2 * weights + r * (act * p[1] + out * p[2]), 2 * r * weights
    if shader == S.Gla:
        h, vdim, dim = p[1:4]                # what one pass needs: q, k, v, the gate, the state in and out (the decay comes from its low-rank input)
        return 8 * h * dim * vdim + rows * h * (8 * dim + vdim * (8 + act)), rows * h * dim * vdim * 5
    if shader == S.Attention:
        h, vdim, dim = p[1:4]
        kv = next(x.attention.kv_heads for x in model.cfg.layers if x.attention and (x.attention.heads, x.attention.dim, x.attention.vdim) == (h, dim, vdim))
        keys = rows * pos + rows * (rows + 1) // 2
        return act * (pos + rows) * kv * (dim + vdim) + rows * h * (4 * dim + vdim * (4 + act)), 2 * h * keys * (dim + vdim)
    if shader == S.AttentionInputs:
        a = next(x.attention for x in model.cfg.layers if x.attention)
        return rows * (a.heads * a.dim * 8 + a.kv_heads * (a.dim + a.vdim) * (4 + act)), 0
    if shader == S.ResidualNorm:
        two = any(x.attention for x in model.cfg.layers)
        return rows * model.cfg.width * (12 + act + (2 if two else 0)), rows * model.cfg.width * 6
    if shader == S.Wkv:
        h, dim = p[1], p[2]
        return 8 * h * dim * dim + rows * h * dim * (4 * 5 + act), rows * h * dim * dim * 7
    if shader == S.Mlstm:
        h, vdim = p[1], p[2]
        dim = next(x.dim for x in model.cfg.layers if x.type == "mlstm" and (x.heads, x.vdim) == (h, vdim))
        return 8 * h * dim * vdim + rows * h * (8 * dim + vdim * (8 + act)), rows * h * dim * vdim * 5
    if shader == S.LatentAttention:
        layer = next(x for x in model.cfg.layers if x.type == "latent_attention" and (x.heads, x.vdim) == (p[1], p[2]))
        keys = sum(min(pos + i + 1, layer.window) for i in range(rows))
        span = min(pos + rows, layer.window - 1 + rows)
        row = layer.kv_rank + layer.rot_dim
        h = layer.heads
        nbytes = act * span * row + 2 * h * layer.kv_rank * (layer.dim + layer.vdim) + rows * h * (4 * (layer.dim + layer.rot_dim) + layer.vdim * (4 + act))
        if rows >= 64:                       # expanded keys and values
            return nbytes, 2 * h * keys * (layer.dim + layer.rot_dim + layer.vdim) + 2 * h * span * layer.kv_rank * (layer.dim + layer.vdim)
        return nbytes, 2 * h * keys * (2 * layer.kv_rank + layer.rot_dim) + 2 * h * rows * layer.kv_rank * (layer.dim + layer.vdim)
    width = model.cfg.width
    if shader == S.TokenShift:
        return rows * width * (4 + 5 * act), rows * width * 20
    if shader == S.Norm:
        return rows * width * (4 + act), rows * width * 4
    if shader == S.LatentCacheWrite:
        return rows * (p[1] + p[2]) * (4 + act), 0
    return rows * width * 6, 0


def kernel_table(model, step, rows: int, pos: int, peaks, repeats: int = 5):
    """Median microseconds of every dispatch (events around each) merged by label, with its roofline share."""
    s = model.session
    s.set_profiling(True)
    runs = []
    for _ in range(repeats):
        step()
        runs.append(s.gpu_timings())
    s.set_profiling(False)
    us = np.median(np.stack(runs), axis=0)
    table = {}
    for d, t in zip(s.plan().dispatches, us):
        nbytes, flops = work(model, d, rows, pos)
        e = table.setdefault(d.label, {"launches": 0, "us": 0.0, "bytes": 0, "flops": 0})
        e["launches"] += 1
        e["us"] += float(t)
        e["bytes"] += nbytes
        e["flops"] += flops
    hbm, tensor = peaks
    out = []
    for label, e in sorted(table.items(), key=lambda kv: -kv[1]["us"]):
        floor = max(e["bytes"] / hbm / 1e3, e["flops"] / tensor / 1e6)
        out.append({"kernel": label, "dispatches": e["launches"], "us_each": round(e["us"] / e["launches"], 2), "roofline": round(floor / e["us"], 4),
                    "bound": "hbm" if e["bytes"] / hbm / 1e3 >= e["flops"] / tensor / 1e6 else "bf16"})
    return out


def row_model_numbers(label, config, rank, peaks, prefill, context, steps, tables) -> dict:
    limit = context + prefill + 2 * steps + 32
    model = random_model(config, rank, dtype="bfloat16", max_rows=prefill, max_picked=1, max_tokens=limit)
    e, s = Engine(model, greedy=True), model.session
    tokens = np.random.default_rng(0).integers(0, model.cfg.vocab, prefill).astype(np.uint32)

    def prompt():
        e.end()
        e._step(tokens, [prefill - 1])
        s.wait()
    for _ in range(3):
        prompt()
    t0 = time.perf_counter()
    for _ in range(5):
        prompt()
    prefill_s = (time.perf_counter() - t0) / 5
    finite = bool(np.isfinite(s.read_output(model.cfg.vocab)).all())
    out = {"model": label, "width": model.cfg.width, "layers": len(model.cfg.layers), "vocab": model.cfg.vocab, "dtype": "bfloat16",
           "prefill_tokens": prefill, "prefill_tokens_per_s": round(prefill / prefill_s), "prefill_ms": round(prefill_s * 1e3, 3), "logits_finite": finite}
    if tables:
        out["prefill_kernels"] = kernel_table(model, prompt, prefill, 0, peaks)
    e.end()
    first = e.generate(tokens[:context], 6)                 # prompt, then single steps until the graph is captured
    s.wait()
    t0 = time.perf_counter()
    for _ in range(steps):
        s.step()
    s.wait()
    dt = (time.perf_counter() - t0) / steps
    weights = sum(int(np.prod(shape)) * 2 for _, shape, bf16 in model.parameters() if bf16)
    out.update(decode_context=context, decode_tokens_per_s=round(1 / dt, 1), decode_ms=round(dt * 1e3, 4), decode_launches=len(s.plan().dispatches) + 1,
               weight_gb=round(weights / 1e9, 3), decode_weight_gbs=round(weights / dt / 1e9, 1), first_tokens=[int(t) for t in first])
    if tables:
        out["decode_kernels"] = kernel_table(model, lambda: (s.step(), s.wait()), 1, context + 5 + steps, peaks)
    return out


def measure(design: str, name: str, peaks, prefill: int = 2048, context: int = 2048, steps: int = 64, tables: bool = True) -> dict:
    config, rank, like = sizes(design)[name]
    out = row_model_numbers(f"{design}-{name}", config, rank, peaks, prefill, context, steps, tables)
    if isinstance(like, str):
        out["closest"] = row_model_numbers(f"{like}-{name}", *sizes(like)[name][:2], peaks, prefill, context, steps, tables)
    else:
        out["closest"] = decoder_numbers(like, peaks, context, steps, tables)
    return out


def decoder_numbers(like, peaks, context, steps, tables) -> dict:
    dec = M.DecodeSession(like, context + steps + 16, seed=3, greedy_history=context + steps + 16)
    dec.fill_caches(context)
    ds = dec.session
    dec.set_position(1, context)
    ds.step()
    ds.wait()
    ds.capture()
    dec.set_position(1, context)
    for _ in range(3):
        ds.step()
    ds.wait()
    t0 = time.perf_counter()
    for _ in range(steps):
        ds.step()
    ds.wait()
    dt = (time.perf_counter() - t0) / steps
    wb = M.packed_weight_bytes(like)
    out = {"model": like.name, "weights": "Q4", "decode_context": context, "decode_tokens_per_s": round(1 / dt, 1), "decode_ms": round(dt * 1e3, 4),
           "decode_launches": len(ds.plan().dispatches) + 1, "weight_gb": round(wb / 1e9, 3), "decode_weight_gbs": round(wb / dt / 1e9, 1),
           "prefill": "token by token (the model has no multi-row step): the decode rate"}
    if tables:
        ds.set_profiling(True)
        runs = []
        for _ in range(5):
            dec.set_position(1, context)
            ds.step()
            runs.append(ds.gpu_timings())
        ds.set_profiling(False)
        us = np.median(np.stack(runs), axis=0)
        agg = {}
        for d, t in zip(ds.plan().dispatches, us):
            a = agg.setdefault(d.label, [0, 0.0, d])
            a[0] += 1
            a[1] += float(t)
        rows = []
        for label, (n, t, d) in sorted(agg.items(), key=lambda kv: -kv[1][1]):
            nb = None
            if d.weight_format.name == "Q4":
                nb = d.params[1] * d.params[2] // 32 * 20
            elif d.shader == S.CachedAttention:
                nb = 2 * (context + 1) * like.kv_dim * 4
            rows.append({"kernel": label, "dispatches": n, "us_each": round(t / n, 2), "roofline": round(nb * n / peaks[0] / 1e3 / t, 4) if nb else None})
        out["decode_kernels"] = rows
    return out
