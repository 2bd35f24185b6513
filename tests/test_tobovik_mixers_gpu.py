"""Each mechanism of the Tobovik decoder alone, through a small graph, against the plain restatement; every
case with and without the session's merges."""
import numpy as np
import pytest

from graph_util import close, rng_of, run, session
from oracle import tobovik_oracle as T
from petotar_util import bf16_round
from test_mixers_gpu import fuse  # noqa: F401

pytestmark = pytest.mark.gpu


def f16_round(a):
    return np.asarray(a, np.float32).astype(np.float16).astype(np.float64)


# ---------------------------------------------------------------- embedding, norms behind sublayers, linear layers
@pytest.mark.parametrize("width", [256, 90, 7])
@pytest.mark.parametrize("first", [0, 31, 4000, 120001])
def test_embedding_positions_and_operand_copy(fuse, width, first):  # noqa: F811
    import meganeura_b200 as mg
    from meganeura_b200._lib import FMT_BF16
    r = rng_of(width)
    table = bf16_round(r.standard_normal((30, width)).astype(np.float32))
    eye = np.eye(width, dtype=np.float32)
    for bf16_table in (True, False):
        g = mg.Graph()
        ids, pos = g.input_u32("ids", [5]), g.input_u32("pos", [1])
        x = g.embedding_positions(ids, (g.parameter_bf16 if bf16_table else g.parameter)("t", [30, width]), pos, 0.5, 300.0)
        y = g.matmul_bt(g.cast(x, FMT_BF16), g.parameter_bf16("eye", [width, width]))
        s = session(g, [x, y], {"t": table, "eye": eye}, None, {"ids": [29, 0, 7, 7, 3], "pos": [first]})
        got, copy = run(s, (5, width), (5, width))
        want = table[[29, 0, 7, 7, 3]] * 0.5 + T.position_vectors(first + np.arange(5), width, 300.0)
        close(got, want, 4e-7)
        assert (copy == bf16_round(got)).all()
        assert len(s.plan().dispatches) == (2 if fuse else 3)


@pytest.mark.parametrize("cols", [7, 90, 256, 1500, 2048, 5000, 9000])
def test_norm_behind_a_sublayer(fuse, cols):  # noqa: F811
    """x + norm(sa * a + sb * b), x + norm(a) and the copy for the next layer."""
    import meganeura_b200 as mg
    from meganeura_b200._lib import FMT_BF16
    r = rng_of(cols)
    a, b, x = (r.standard_normal((3, cols)).astype(np.float32) for _ in range(3))
    b *= 5
    w = r.standard_normal(cols).astype(np.float32)
    g = mg.Graph()
    ai, bi, xi = (g.input(n, [3, cols]) for n in "abx")
    y = g.add(xi, g.norm(g.scaled_sum(ai, bi, 0.75, -0.3), g.parameter("w", [cols]), 0.1))
    z = g.add(g.norm(ai, g.parameter("w2", [cols]), 0.02), xi)
    outs = [y, z]
    if cols < 2000:
        outs.append(g.matmul_bt(g.cast(y, FMT_BF16), g.parameter_bf16("eye", [cols, cols])))
    s = session(g, outs, {"w": w, "w2": w, **({"eye": np.eye(cols, dtype=np.float32)} if cols < 2000 else {})}, {"a": a, "b": b, "x": x})
    got = run(s, *[(3, cols)] * len(outs))
    close(got[0], x + T.rms_norm(0.75 * a.astype(np.float64) - 0.3 * b, w, 0.1), 2e-6)
    close(got[1], x + T.rms_norm(a, w, 0.02), 2e-6)
    if cols < 2000:
        assert (got[2] == bf16_round(got[0])).all()
    if fuse:
        assert sorted(d.shader.name for d in s.plan().dispatches if d.shader.name != "Linear") == ["ResidualNorm"] * 2


@pytest.mark.parametrize("operand", ["f32", "bf16"])
@pytest.mark.parametrize("rows", [1, 3, 8, 40, 200])
def test_linear_layers_of_different_depth_and_silu_glu(fuse, operand, rows):  # noqa: F811
    """Two independent layers of different K next to each other, and silu(gate) * up without biases."""
    import meganeura_b200 as mg
    from meganeura_b200._lib import FMT_BF16, FMT_F32
    r, op = rng_of(rows), FMT_BF16 if operand == "bf16" else FMT_F32
    ks, ns = (72, 200), (40, 96)
    x = [r.standard_normal((rows, k)).astype(np.float32) for k in ks]
    w = [bf16_round(r.standard_normal((n, k)).astype(np.float32) * k ** -0.5) for n, k in zip(ns, ks)]
    wg, wu = (bf16_round(r.standard_normal((56, ks[0])).astype(np.float32) * 0.3) for _ in range(2))
    g = mg.Graph()
    h = [g.norm(g.input(f"x{i}", [rows, k]), g.parameter(f"one{i}", [k]), 1e-6, 0.0, op) for i, k in enumerate(ks)]
    y = [g.matmul_bt(h[i], g.parameter_bf16(f"w{i}", [ns[i], ks[i]])) for i in range(2)]
    glu = g.silu_glu(g.matmul_bt(h[0], g.parameter_bf16("wg", [56, ks[0]])), g.matmul_bt(h[0], g.parameter_bf16("wu", [56, ks[0]])), op)
    z = g.matmul_bt(glu, g.parameter_bf16("eye", [56, 56]))
    s = session(g, y + [z], {"one0": np.ones(72, np.float32), "one1": np.ones(200, np.float32), "w0": w[0], "w1": w[1], "wg": wg, "wu": wu,
                             "eye": np.eye(56, dtype=np.float32)}, {"x0": x[0], "x1": x[1]})
    got = run(s, (rows, 40), (rows, 96), (rows, 56))
    hv = [T.rms_norm(v, 1.0, 1e-6).astype(np.float32) for v in x]
    hv = [(bf16_round(v) if operand == "bf16" else v).astype(np.float64) for v in hv]
    for i in range(2):
        close(got[i], hv[i] @ w[i].T, 2e-3 if operand == "bf16" else 1e-5)
    close(got[2], T.silu(hv[0] @ wg.T) * (hv[0] @ wu.T), 6e-3 if operand == "bf16" else 1e-5)
    from meganeura_b200 import ops
    ops.device_status()


# ---------------------------------------------------------------- gated linear attention
def gla_case(heads, dim, vdim, rank, rows, tau=16.0, product="f32", seed=0, bias=(1.0, 2.5), tabs=None):
    import meganeura_b200 as mg
    from meganeura_b200._lib import FMT_BF16, FMT_F32, GATE_SILU, ROWS_TOKENS, lib
    r = rng_of(heads, dim, vdim, seed)
    n, nv, vocab = heads * dim, heads * vdim, 90
    t = {"q": r.standard_normal((vocab, n)), "k": r.standard_normal((vocab, n)), "v": r.standard_normal((vocab, nv)), "g": r.standard_normal((vocab, nv)),
         "low": r.standard_normal((vocab, rank))}
    t = {c: a.astype(np.float32) for c, a in {**t, **(tabs or {})}.items()}
    w2 = bf16_round(r.standard_normal((n, rank)).astype(np.float32) * rank ** -0.5)
    b = (bias[0] + bias[1] * r.standard_normal(n)).astype(np.float32)
    hw = r.standard_normal(vdim).astype(np.float32)
    g = mg.Graph()
    ids = g.input_u32_rows("ids", rows, ROWS_TOKENS)
    e = {c: g.embedding_scaled(ids, g.parameter(c, list(a.shape)), 1.0) for c, a in t.items()}
    decay = g.lora_sigmoid_decay(e["low"], g.parameter_bf16("w2", [n, rank]), g.parameter("b", [n]), tau)
    state = g.parameter("state", [lib.mgq_gla_state_elements(heads, dim, vdim)])
    o = g.gla(e["q"], e["k"], e["v"], decay, state, heads, FMT_BF16 if product == "split" else FMT_F32)
    y = g.head_gate(o, e["g"], heads, g.parameter("hw", [vdim]), 1e-5, GATE_SILU)
    s = session(g, [y], {**t, "w2": w2, "b": b, "hw": hw})

    def feed(tokens):
        s.set_rows(ROWS_TOKENS, len(tokens))
        s.set_input_u32("ids", tokens)
        return run(s, (len(tokens), nv))

    def oracle(tokens, S):
        a = T.channel_decay(t["low"][tokens].astype(np.float64), w2, b, tau).reshape(-1, heads, dim)
        q, k, v = (t[c][tokens].astype(np.float64).reshape(len(tokens), heads, -1) for c in "qkv")
        return T.rms_norm(T.gla_scan(q * dim ** -0.5, k, v, a, S), hw, 1e-5).reshape(-1, nv) * T.silu(t["g"][tokens].astype(np.float64))
    return feed, oracle, s


@pytest.mark.parametrize("product", ["f32", "split"])
@pytest.mark.parametrize("heads,dim,vdim,rank", [(2, 32, 48, 4), (3, 22, 9, 5), (1, 64, 130, 16), (2, 128, 64, 8), (1, 200, 33, 3), (1, 256, 80, 20), (5, 6, 16, 1)])
def test_gla_portions_carry_the_state(fuse, product, heads, dim, vdim, rank):  # noqa: F811
    """Portions of all sizes of one sequence (cut into chunks and segments or token by token), then a second one
    from cleared state."""
    feed, oracle, s = gla_case(heads, dim, vdim, rank, 700, tau=3.0, product=product)
    for seq in range(2):
        S, at = np.zeros((heads, dim, vdim)), 0
        s.reset_state()
        for cnt in (1, 700, 2, 1, 64, 33, 79, 16, 17, 15, 257, 65) if seq == 0 else (5, 1, 66):
            toks = (np.arange(at, at + cnt) * 7 + seq * 13) % 90
            at += cnt
            close(feed(toks), oracle(toks, S), 1e-4)


@pytest.mark.parametrize("product", ["f32", "split"])
@pytest.mark.parametrize("bias", [(-60.0, 30.0), (8.0, 0.5), (-3.0, 3.0)], ids=["vanishing", "lasting", "strong"])
def test_gla_extreme_decays(fuse, product, bias):  # noqa: F811
    """Decays that underflow, that hardly act over a long portion, and strong ones of every size: no quotient of
    cumulated decays may appear anywhere."""
    feed, oracle, s = gla_case(2, 64, 32, 8, 900, tau=1.0, product=product, bias=bias)
    S, at = np.zeros((2, 64, 32)), 0
    for cnt in (900, 1, 100, 2):
        toks = (np.arange(at, at + cnt) * 11) % 90
        at += cnt
        close(feed(toks), oracle(toks, S), 1e-4)


@pytest.mark.parametrize("product", ["f32", "split"])
def test_gla_remembers_a_far_token(fuse, product):  # noqa: F811
    """One token writes a large value under a key that no other token has; hardly any decay.  Queries hundreds of
    tokens later, at chunk and segment borders and one by one, read it back."""
    heads, dim, vdim = 1, 32, 16
    q, k, v = np.zeros((90, dim)), np.zeros((90, dim)), rng_of(4).standard_normal((90, vdim))
    k[:, 1:] = rng_of(5).standard_normal((90, dim - 1)) * 0.05
    q[:, 0] = 1.0
    k[7] = 0
    k[7, 0] = 30.0
    feed, oracle, s = gla_case(heads, dim, vdim, 2, 800, product=product, bias=(9.0, 0.0), tabs={"q": q, "k": k, "v": v, "low": np.zeros((90, 2))})
    tokens = np.arange(840) % 80 + 10
    tokens[20] = 7
    S = np.zeros((heads, dim, vdim))
    want = oracle(tokens, S)
    assert np.abs(want[:20]).max() < 1e-3 and np.abs(want[800:]).max() > 0.5            # nothing before the token, most of it after 800
    at = 0
    for cnt in (800, 1, 1, 17, 1, 20):
        close(feed(tokens[at:at + cnt]), want[at:at + cnt], 1e-4)
        at += cnt


# ---------------------------------------------------------------- softmax attention over grouped heads
def attention_case(heads, kv_heads, dim, vdim, cap, slots, half, scale=None, coef=0.3, every=16, gain=1.0, seed=0, eps=1e-5):
    import meganeura_b200 as mg
    from meganeura_b200._lib import ROWS_TOKENS
    r = rng_of(heads, kv_heads, dim, vdim, seed)
    vocab = 64
    t = {"q": r.standard_normal((vocab, heads * dim)), "k": r.standard_normal((vocab, kv_heads * dim)), "v": r.standard_normal((vocab, kv_heads * vdim)),
         "gate": r.standard_normal((vocab, heads * vdim))}
    t = {c: a.astype(np.float32) for c, a in t.items()}
    qw, kw = ((gain + 0.2 * r.standard_normal(n)).astype(np.float32) for n in (heads * dim, kv_heads * dim))
    scale = dim ** -0.5 if scale is None else scale
    g = mg.Graph()
    ids, pos = g.input_u32_rows("ids", cap, ROWS_TOKENS), g.input_u32("pos", [1])
    e = {c: g.embedding_scaled(ids, g.parameter(c, list(a.shape)), 1.0) for c, a in t.items()}
    cache = g.parameter_f16 if half else g.parameter
    kc, vc = cache("kc", [slots, kv_heads * dim]), cache("vc", [slots, kv_heads * vdim])
    q = g.norm(e["q"], g.parameter("qw", [heads * dim]), eps)
    k = g.norm(e["k"], g.parameter("kw", [kv_heads * dim]), eps)
    q = g.query_temperature(q, pos, coef, every)
    kc, vc = g.cache_append(k, kc, pos), g.cache_append(e["v"], vc, pos)
    o = g.attention(q, kc, vc, pos, heads, kv_heads, dim, vdim, scale)
    s = session(g, [g.head_gate(o, e["gate"], heads)], {**t, "qw": qw, "kw": kw})

    def oracle(tokens):
        qq = T.rms_norm(t["q"][tokens], qw, eps) * T.query_temperature(np.arange(len(tokens)), coef, every)[:, None]
        kk, vv = T.rms_norm(t["k"][tokens], kw, eps), t["v"][tokens].astype(np.float64)
        if half:
            kk, vv = f16_round(kk), f16_round(vv)
        n = len(tokens)
        o = T.causal_attention(qq.reshape(n, heads, dim), kk.reshape(n, kv_heads, dim), vv.reshape(n, kv_heads, vdim), 0, scale)
        return o.reshape(n, -1) * T.sigmoid(t["gate"][tokens])

    def feed(tokens, first):
        s.set_rows(ROWS_TOKENS, len(tokens))
        s.set_input_u32("ids", tokens)
        s.set_input_u32("pos", [first])
        return run(s, (len(tokens), heads * vdim))
    return feed, oracle, s, t


SHAPES = [(4, 4, 16, 24), (6, 2, 24, 40), (8, 1, 72, 64), (3, 1, 18, 13), (16, 2, 64, 128), (5, 5, 7, 30), (2, 1, 256, 136), (4, 2, 128, 264), (12, 1, 104, 8),
          (2, 2, 136, 72)]


@pytest.mark.parametrize("half", [False, True], ids=["f32", "f16"])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim", SHAPES)
def test_attention_portions(fuse, half, heads, kv_heads, dim, vdim):  # noqa: F811
    """One sequence in portions of all sizes, single tokens among them, then another one in the same cache."""
    feed, oracle, s, _ = attention_case(heads, kv_heads, dim, vdim, 150, 420, half, gain=1.6)
    for seed, sizes in ((1, [1, 1, 150, 2, 1, 17, 64, 3, 1, 63, 65]), (2, [70, 1, 2, 1, 9])):
        tokens = rng_of(seed).integers(0, 64, sum(sizes))
        want, at = oracle(tokens), 0
        for n in sizes:
            close(feed(tokens[at:at + n], at), want[at:at + n], 3e-3 if half else 3e-5)
            at += n
    if fuse:
        names = [d.shader.name for d in s.plan().dispatches]
        assert names.count("AttentionInputs") == 1 and "CacheAppend" not in names and "HeadGate" not in names


@pytest.mark.parametrize("half", [False, True], ids=["f32", "f16"])
@pytest.mark.parametrize("special", [0, 1, 15, 16, 31, 32, 63, 64, 65, 127, 128, 200, 319])
def test_one_key_stands_out_however_far(half, special):
    """A key whose score is far above all others takes the whole softmax from its own position on, and nothing of it
    shows before: in prompts, in portions and token by token."""
    heads, kv_heads, dim, vdim = 4, 2, 32, 32
    total = 330
    for sizes in ([total], [200, 1, 1, 64, 1, 2, 61], [64] * 5 + [10], [1] * total if special in (64, 319) else [2, 62, 1, 100, 3, 162]):
        feed, oracle, s, t = attention_case(heads, kv_heads, dim, vdim, total, total, half, scale=1.0, coef=0.1, every=40)
        q, k = t["q"] * 0.05, t["k"] * 0.5
        q.reshape(64, heads, dim)[:, :, 3] = 2.0
        k.reshape(64, kv_heads, dim)[:, :, 3] = 0.0
        k.reshape(64, kv_heads, dim)[5, :, :] = 0.0
        k.reshape(64, kv_heads, dim)[5, :, 3] = 4.0
        t["q"], t["k"] = q, k
        s.set_parameter("q", q)
        s.set_parameter("k", k)
        tokens = np.arange(total) % 40 + 10
        tokens[special] = 5
        want = oracle(tokens)
        if 0 < special < total - 1:
            v = t["v"][5].reshape(kv_heads, vdim).repeat(heads // kv_heads, 0).reshape(-1)
            gate = T.sigmoid(t["gate"][tokens])
            assert np.abs(want[special] - v * gate[special]).max() < 0.02 and np.abs(want[special - 1] - v * gate[special - 1]).max() > 0.3
            assert np.abs(want[-1] - v * gate[-1]).max() < 0.02                            # still there at the end
        at = 0
        for n in sizes:
            close(feed(tokens[at:at + n], at), want[at:at + n], 3e-3 if half else 5e-5)
            at += n


@pytest.mark.parametrize("every,coef", [(1, 1.0), (7, 0.5), (16, -0.2), (2.5, 0.4)])
def test_query_temperature_steps(every, coef):
    import meganeura_b200 as mg
    r = rng_of(3)
    x = r.standard_normal((40, 12)).astype(np.float32)
    g = mg.Graph()
    y = g.query_temperature(g.input("x", [40, 12]), g.input_u32("pos", [1]), coef, every)
    for first in (0, 5, 100000):
        s = session(g, [y], {}, {"x": x}, {"pos": [first]})
        close(run(s, (40, 12)), x * T.query_temperature(first + np.arange(40), coef, every)[:, None], 1e-6)


def test_rows_beyond_the_cache_are_dropped():
    """A step that runs over the end of the cache writes nothing behind it and stays finite."""
    feed, oracle, s, _ = attention_case(4, 2, 16, 16, 30, 40, True)
    tokens = rng_of(1).integers(0, 64, 50)
    want = oracle(tokens[:40])
    got = np.concatenate([feed(tokens[:25], 0), feed(tokens[25:], 25)])
    close(got[:40], want, 3e-3)
    assert np.isfinite(got).all()


def test_builders_refuse_bad_shapes():
    import meganeura_b200 as mg
    from meganeura_b200._lib import FMT_BF16, FMT_F32
    g = mg.Graph()
    x, y, pos = g.input("x", [4, 32]), g.input("y", [4, 16]), g.input_u32("pos", [1])
    k, v = g.parameter_f16("k", [10, 16]), g.parameter_f16("v", [10, 16])
    for bad in (lambda: g.attention(x, k, v, pos, 3, 2, 8, 8, 1.0),                       # heads do not divide
                lambda: g.attention(x, k, v, pos, 4, 2, 16, 8, 1.0),                      # q too narrow
                lambda: g.attention(x, k, g.parameter("v32", [10, 16]), pos, 4, 2, 8, 8, 1.0),
                lambda: g.attention(x, g.parameter("few", [3, 16]), g.parameter("few2", [3, 16]), pos, 4, 2, 8, 8, 1.0),
                lambda: g.attention(x, k, v, x, 4, 2, 8, 8, 1.0),
                lambda: g.cache_append(x, k, pos), lambda: g.cache_append(y, g.parameter_bf16("b", [10, 16]), pos),
                lambda: g.query_temperature(x, pos, 1.0, 0.0), lambda: g.scaled_sum(x, y, 1.0, 1.0),
                lambda: g.cast(x, FMT_F32), lambda: g.silu_glu(x, y), lambda: g.silu_glu(x, x, 9),
                lambda: g.gla(x, x, y, y, g.parameter("s", [8]), 2), lambda: g.gla(x, x, y, x, g.parameter("s2", [7]), 2),
                lambda: g.lora_sigmoid_decay(y, g.parameter_bf16("w2", [32, 16]), g.parameter("w0", [32]), 0.0),
                lambda: g.head_gate(x, x, 2, g.parameter("w8", [8])),
                lambda: g.embedding_positions(g.input_u32("ids", [4]), g.parameter_bf16("t", [9, 8]), x)):
        with pytest.raises(mg.MgqError):
            bad()
    assert g.cast(x, FMT_BF16) > 0
