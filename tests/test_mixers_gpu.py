"""Each mechanism of the recurrent / latent-attention decoders alone, through a small graph, against the
plain restatement; every case with and without the session's merges."""
import numpy as np
import pytest

from graph_util import close, rng_of, run, session
from oracle import petotar_oracle as P
from petotar_util import bf16_round

pytestmark = pytest.mark.gpu


@pytest.fixture(params=[1, 0], ids=["fused", "unfused"])
def fuse(request):
    from meganeura_b200 import ops
    ops.set_option("session.fuse_mixer", request.param)
    yield request.param
    ops.set_option("session.fuse_mixer", 1)


# ---------------------------------------------------------------- linear layers
@pytest.mark.parametrize("operand", ["f32", "bf16"])
@pytest.mark.parametrize("rows,k,n", [(1, 64, 48), (1, 1000, 7), (2, 72, 130), (3, 33, 65), (8, 256, 96), (9, 256, 96), (17, 40, 33), (130, 72, 200),
                                      (129, 51, 70), (300, 512, 640), (64, 2048, 320)])
def test_linear_bias_addend(fuse, operand, rows, k, n):
    import meganeura_b200 as mg
    from meganeura_b200._lib import FMT_BF16, FMT_F32
    r = rng_of(rows, k, n)
    x, w = r.standard_normal((rows, k)).astype(np.float32), bf16_round(r.standard_normal((n, k)).astype(np.float32))
    b, add = r.standard_normal(n).astype(np.float32), r.standard_normal((rows, n)).astype(np.float32)
    g = mg.Graph()
    xi, ai = g.input("x", [rows, k]), g.input("add", [rows, n])
    h = g.norm(xi, g.parameter("one", [k]), 1e-6, 0.0, FMT_BF16 if operand == "bf16" else FMT_F32)
    y = g.add(g.bias_add(g.matmul_bt(h, g.parameter_bf16("w", [n, k])), g.parameter("b", [n])), ai)
    z = g.matmul_bt(h, g.parameter_bf16("w2", [n + 3, k]))
    s = session(g, [y, z], {"one": np.ones(k, np.float32), "w": w, "b": b, "w2": np.concatenate([w[:3] * 2, w])}, {"x": x, "add": add})
    got, got2 = run(s, (rows, n), (rows, n + 3))
    h = P.unit_rms(x, 1e-6).astype(np.float32)
    h = bf16_round(h) if operand == "bf16" else h
    tol = 2e-3 if operand == "bf16" else 1e-5           # an operand on the edge of two bf16 values may round the other way
    base = h.astype(np.float64) @ w.T.astype(np.float64)
    close(got, base + b + add, tol)
    close(got2, np.concatenate([base[:, :3] * 2, base], axis=1), tol)
    from meganeura_b200 import ops
    ops.device_status()


@pytest.mark.parametrize("operand", ["f32", "bf16"])
@pytest.mark.parametrize("rows,k,n", [(1, 64, 48), (1, 96, 5003), (5, 37, 19), (40, 64, 33), (200, 128, 320), (140, 136, 72)])
def test_clamped_glu(fuse, operand, rows, k, n):
    import meganeura_b200 as mg
    from meganeura_b200._lib import FMT_BF16, FMT_F32
    r = rng_of(rows, k, n, 2)
    op = FMT_BF16 if operand == "bf16" else FMT_F32
    x = r.standard_normal((rows, k)).astype(np.float32) * 3
    wg, wu = (bf16_round(r.standard_normal((n, k)).astype(np.float32) * k ** -0.5 * 2) for _ in range(2))
    bg, bu = r.standard_normal(n).astype(np.float32), r.standard_normal(n).astype(np.float32)
    g = mg.Graph()
    xi = g.input("x", [rows, k])
    h = g.norm(xi, g.parameter("one", [k]), 1e-6, 0.0, op)
    gate = g.bias_add(g.matmul_bt(h, g.parameter_bf16("wg", [n, k])), g.parameter("bg", [n]))
    up = g.bias_add(g.matmul_bt(h, g.parameter_bf16("wu", [n, k])), g.parameter("bu", [n]))
    y = g.clamped_glu(gate, up, 1.3, 1.702, op)
    eye = g.matmul_bt(y, g.parameter_bf16("eye", [n, n])) if n < 512 else None
    if eye is None:
        y = g.clamped_glu(gate, up, 1.3, 1.702, FMT_F32)
    params = {"one": np.ones(k, np.float32), "wg": wg, "wu": wu, "bg": bg, "bu": bu}
    if eye is not None:
        params["eye"] = np.eye(n, dtype=np.float32)
    s = session(g, [y if eye is None else eye], params, {"x": x})
    got = run(s, (rows, n))
    h = P.unit_rms(x, 1e-6).astype(np.float32)
    h = (bf16_round(h) if operand == "bf16" else h).astype(np.float64)
    want = P.clamped_glu(h @ wg.T + bg, h @ wu.T + bu, 1.3)
    assert (np.abs(h @ wu.T + bu) > 1.3).any() and (h @ wg.T + bg > 1.3).any()          # both clamps act
    close(got, want, 6e-3 if operand == "bf16" else 1e-5)


# ---------------------------------------------------------------- norm, rows, embedding
def test_norm_with_offset_and_picked_rows(fuse):
    import meganeura_b200 as mg
    r = rng_of(5)
    for cols in (7, 256, 5000):
        x, w = r.standard_normal((6, cols)).astype(np.float32), r.standard_normal(cols).astype(np.float32)
        g = mg.Graph()
        xi, idx = g.input("x", [6, cols]), g.input_u32("idx", [3])
        y = g.norm(g.pick_rows(xi, idx), g.parameter("w", [cols]), 0.5, 1.0)
        z = g.norm(xi, g.parameter("w2", [cols]), 0.5, 0.0)
        s = session(g, [y, z], {"w": w, "w2": w}, {"x": x}, {"idx": [5, 0, 2]})
        got, plain = run(s, (3, cols), (6, cols))
        close(got, P.norm_around_zero(x[[5, 0, 2]], w, 0.5), 2e-6)
        close(plain, P.unit_rms(x, 0.5) * w, 2e-6)


def test_embedding_scaled():
    import meganeura_b200 as mg
    r = rng_of(6)
    table = bf16_round(r.standard_normal((50, 24)).astype(np.float32))
    g = mg.Graph()
    y = g.embedding_scaled(g.input_u32("ids", [4]), g.parameter_bf16("t", [50, 24]), 2.75)
    s = session(g, [y], {"t": table}, None, {"ids": [49, 0, 7, 7]})
    assert (run(s, (4, 24)) == table[[49, 0, 7, 7]] * np.float32(2.75)).all()


# ---------------------------------------------------------------- token shift and RWKV-style mixing
@pytest.mark.parametrize("heads,dim,rank,width", [(2, 32, 8, 64), (3, 22, 5, 50), (1, 64, 16, 300), (2, 128, 4, 40), (1, 200, 3, 33), (7, 6, 9, 20)])
def test_wkv_portions_carry_state_and_previous_token(fuse, heads, dim, rank, width):
    """Portions of 1, 600 (cut into segments), 2, 1, 33 and 300 tokens of one sequence, then a second sequence from
    cleared state."""
    import meganeura_b200 as mg
    from meganeura_b200._lib import GATE_SILU, ROWS_TOKENS, lib
    r = rng_of(heads, dim, rank)
    n, cap = heads * dim, 600
    table = r.standard_normal((90, width)).astype(np.float32)
    nw = r.standard_normal(width).astype(np.float32) * 0.2
    mus = r.uniform(0, 1, (5, width)).astype(np.float32)
    mats = {s: bf16_round(r.standard_normal((n, width)).astype(np.float32) * width ** -0.5) for s in "rkvg"}
    w1 = bf16_round(r.standard_normal((rank, width)).astype(np.float32) * width ** -0.5 * 2)
    w2 = bf16_round(r.standard_normal((n, rank)).astype(np.float32))
    w0, u, hw = r.uniform(-5, 0, n).astype(np.float32), r.standard_normal(n).astype(np.float32), r.standard_normal(n).astype(np.float32)
    g = mg.Graph()
    ids = g.input_u32_rows("ids", cap, ROWS_TOKENS)
    x = g.embedding_scaled(ids, g.parameter("table", [90, width]), 1.0)
    shift = g.parameter("shift", [2, width])
    mix = g.token_shift(g.norm(x, g.parameter("nw", [width]), 1e-4, 1.0), [g.parameter(f"mu{i}", [width]) for i in range(5)], shift)
    rr, kk, vv, gg = (g.matmul_bt(g.slot(mix, i), g.parameter_bf16(s, [n, width])) for i, s in enumerate("rkvg"))
    low = g.matmul_bt(g.slot(mix, 4), g.parameter_bf16("w1", [rank, width]))
    decay = g.lora_decay(low, g.parameter_bf16("w2", [n, rank]), g.parameter("w0", [n]))
    state = g.parameter("state", [lib.mgq_wkv_state_elements(heads, dim)])
    o = g.wkv(rr, kk, vv, decay, g.parameter("u", [n]), state, heads, shift)
    y = g.head_gate(o, gg, heads, g.parameter("hw", [n]), 1e-4, GATE_SILU)
    params = {"table": table, "nw": nw, "w1": w1, "w2": w2, "w0": w0, "u": u, "hw": hw, **mats, **{f"mu{i}": mus[i] for i in range(5)}}
    s = session(g, [y], params)
    for seq in range(2):
        prev, S = np.zeros(width), np.zeros((heads, dim, dim))
        s.reset_state()
        at = 0
        for cnt in (1, 600, 2, 1, 33, 300) if seq == 0 else (3, 1):
            toks = (np.arange(at, at + cnt) * 7 + seq * 13) % 90
            at += cnt
            s.set_rows(ROWS_TOKENS, cnt)
            s.set_input_u32("ids", toks)
            got = run(s, (cnt, n))
            h = P.norm_around_zero(table[toks], nw, 1e-4)
            m = [P.token_shift(h, prev, mus[i]) for i in range(5)]
            prev = h[-1]
            ro, ko, vo = ((m[i] @ mats[c].T).reshape(cnt, heads, dim) for i, c in enumerate("rkv"))
            go = m[3] @ mats["g"].T
            oo = P.wkv_scan(ro, ko, vo, P.wkv_decay(m[4], w1, w2, w0).reshape(cnt, heads, dim), u.reshape(heads, dim), S)
            close(got, P.unit_rms(oo, 1e-4).reshape(cnt, n) * hw * go * P.sigmoid(go), 1e-4)


# ---------------------------------------------------------------- mLSTM
@pytest.mark.parametrize("heads,dim,vdim,cap", [(2, 32, 48, 12.0), (3, 21, 5, 2.0), (1, 128, 64, 15.0), (2, 64, 100, 4.0), (1, 256, 17, 8.0)])
def test_mlstm_portions(fuse, heads, dim, vdim, cap):
    import meganeura_b200 as mg
    from meganeura_b200._lib import GATE_SIGMOID, ROWS_TOKENS, lib
    r = rng_of(heads, dim, vdim)
    n, nv, rows = heads * dim, heads * vdim, 700
    tabs = {"q": r.standard_normal((90, n)), "k": r.standard_normal((90, n)), "v": r.standard_normal((90, nv)), "g": r.standard_normal((90, nv)),
            "i": r.standard_normal((90, heads)) * 6 - 2, "f": r.standard_normal((90, heads)) * 6 + 3}
    tabs = {c: a.astype(np.float32) for c, a in tabs.items()}
    hw = r.standard_normal(nv).astype(np.float32)
    g = mg.Graph()
    ids = g.input_u32_rows("ids", rows, ROWS_TOKENS)
    e = {c: g.embedding_scaled(ids, g.parameter(c, list(a.shape)), 1.0) for c, a in tabs.items()}
    state = g.parameter("state", [lib.mgq_mlstm_state_elements(heads, dim, vdim)])
    o = g.mlstm(e["q"], e["k"], e["v"], e["i"], e["f"], state, heads, cap)
    y = g.head_gate(o, e["g"], heads, g.parameter("hw", [nv]), 1e-5, GATE_SIGMOID)
    s = session(g, [y], {**tabs, "hw": hw})
    for seq in range(2):
        S, nn, m = np.zeros((heads, dim, vdim)), np.zeros((heads, dim)), np.zeros(heads)
        s.reset_state()
        at = 0
        for cnt in (2, 700, 1, 1, 33, 5, 257) if seq == 0 else (1, 4):
            toks = (np.arange(at, at + cnt) * 11 + seq * 5) % 90
            at += cnt
            s.set_rows(ROWS_TOKENS, cnt)
            s.set_input_u32("ids", toks)
            got = run(s, (cnt, nv))
            li, lf = P.mlstm_gates(tabs["i"][toks].astype(np.float64), tabs["f"][toks].astype(np.float64), cap)
            oo = P.mlstm_scan(tabs["q"][toks].reshape(cnt, heads, dim) * dim ** -0.5, tabs["k"][toks].reshape(cnt, heads, dim).astype(np.float64),
                              tabs["v"][toks].reshape(cnt, heads, vdim).astype(np.float64), li, lf, S, nn, m)
            close(got, P.unit_rms(oo, 1e-5).reshape(cnt, nv) * hw * P.sigmoid(tabs["g"][toks]), 3e-4)


def test_mlstm_running_maximum_starts_at_zero():
    """Strongly closed input gates: with m starting at minus infinity the first output would not be damped by exp(-m)."""
    import meganeura_b200 as mg
    from meganeura_b200._lib import lib
    g = mg.Graph()
    q, k, v, gi, gf = (g.input(c, [2, w]) for c, w in (("q", 4), ("k", 4), ("v", 4), ("i", 1), ("f", 1)))
    y = g.mlstm(q, k, v, gi, gf, g.parameter("state", [lib.mgq_mlstm_state_elements(1, 4, 4)]), 1, 20.0)
    r = rng_of(9)
    a = {c: r.standard_normal((2, 4)).astype(np.float32) for c in "qkv"}
    gi_v, gf_v = np.full((2, 1), -4.0, np.float32), np.full((2, 1), 1.0, np.float32)
    s = session(g, [y], {}, {**a, "i": gi_v, "f": gf_v})
    got = run(s, (2, 4))
    li, lf = P.mlstm_gates(gi_v.astype(float), gf_v.astype(float), 20.0)
    want = P.mlstm_scan(a["q"].reshape(2, 1, 4) * 0.5, a["k"].reshape(2, 1, 4), a["v"].reshape(2, 1, 4).astype(float), li, lf, np.zeros((1, 4, 4)),
                        np.zeros((1, 4)), np.zeros(1))
    close(got, want.reshape(2, 4), 1e-5)
    assert np.abs(want).max() < 0.2                            # the floor exp(-m) is what divides


# ---------------------------------------------------------------- latent attention
def latent_case(heads, dim, rot, vdim, rank, window, cap, base=300.0, cache_bf16=False, seed=0, q_gain=1.0, window2=None):
    import meganeura_b200 as mg
    from meganeura_b200._lib import ROWS_TOKENS
    r = rng_of(heads, dim, rot, vdim, rank, window, seed)
    vocab = 64
    t = {"down": r.standard_normal((vocab, rank + rot)), "q": r.standard_normal((vocab, heads * (dim + rot))) * q_gain,
         "gate": r.standard_normal((vocab, heads * vdim))}
    t = {c: a.astype(np.float32) for c, a in t.items()}
    nw = (1 + 0.3 * r.standard_normal(rank)).astype(np.float32)
    uk = bf16_round(r.standard_normal((heads * dim, rank)).astype(np.float32) * rank ** -0.5)
    uv = bf16_round(r.standard_normal((heads * vdim, rank)).astype(np.float32) * rank ** -0.5)
    scale = (dim + rot) ** -0.5
    slots = max(window, window2 or 0) - 1 + cap
    g = mg.Graph()
    ids, pos = g.input_u32_rows("ids", cap, ROWS_TOKENS), g.input_u32("pos", [1])
    e = {c: g.embedding_scaled(ids, g.parameter(c, list(a.shape)), 1.0) for c, a in t.items()}
    cache = (g.parameter_bf16 if cache_bf16 else g.parameter)("cache", [slots, rank + rot])
    cache = g.latent_cache_write(e["down"], g.parameter("nw", [rank]), cache, pos, rot, base, 1e-5)
    outs = []
    for w in [window] + ([window2] if window2 else []):
        uk_p, uv_p = g.parameter_bf16(f"uk{w}", [heads * dim, rank]), g.parameter_bf16(f"uv{w}", [heads * vdim, rank])
        o = g.latent_attention(e["q"], cache, uk_p, uv_p, pos, heads, dim, rot, vdim, w, scale, base)
        outs.append(g.head_gate(o, e["gate"], heads))
    params = {**t, "nw": nw, **{f"uk{w}": uk for w in (window, window2) if w}, **{f"uv{w}": uv for w in (window, window2) if w}}
    s = session(g, outs, params)

    def oracle(tokens, w):
        down = t["down"][tokens].astype(np.float64)
        c = P.unit_rms(down[:, :rank], 1e-5) * nw
        kr = np.stack([P.rotate_half(down[p, rank:], p, base) for p in range(len(tokens))])
        if cache_bf16:
            c, kr = bf16_round(c.astype(np.float32)).astype(np.float64), bf16_round(kr.astype(np.float32)).astype(np.float64)
        k = (c @ uk.T.astype(np.float64)).reshape(-1, heads, dim)
        k = np.concatenate([k, np.repeat(kr[:, None], heads, 1)], -1)
        v = (c @ uv.T.astype(np.float64)).reshape(-1, heads, vdim)
        q = t["q"][tokens].astype(np.float64).reshape(-1, heads, dim + rot)
        q = np.stack([np.concatenate([q[p, :, :dim], P.rotate_half(q[p, :, dim:], p, base)], -1) for p in range(len(tokens))])
        return P.window_attention(q, k, v, 0, w, scale).reshape(len(tokens), -1) * P.sigmoid(t["gate"][tokens])

    def feed(tokens, first):
        s.set_rows(ROWS_TOKENS, len(tokens))
        s.set_input_u32("ids", tokens)
        s.set_input_u32("pos", [first])
        got = run(s, *[(len(tokens), heads * vdim)] * len(outs))
        return got if len(outs) > 1 else [got]
    return feed, oracle, s, t


@pytest.mark.parametrize("heads,dim,rot,vdim,rank,window", [(2, 16, 8, 24, 32, 10), (9, 32, 16, 33, 128, 70), (3, 10, 6, 7, 27, 1), (1, 64, 32, 64, 256, 100),
                                                            (4, 24, 4, 16, 520, 40)])
@pytest.mark.parametrize("cache_bf16", [False, True])
def test_latent_attention_portions_and_ring(fuse, heads, dim, rot, vdim, rank, window, cache_bf16):
    """A sequence several times as long as the ring, in portions of all sizes (several rows, then single rows)."""
    feed, oracle, _, _ = latent_case(heads, dim, rot, vdim, rank, window, 48, cache_bf16=cache_bf16, q_gain=2.0)
    tokens = rng_of(1, window).integers(0, 64, 48 + 2 * window + 60)
    want = oracle(tokens, window)
    at = 0
    sizes = [48, 2, 17, 1, 1, 3, 40]
    while at < len(tokens):
        n = min(sizes.pop(0) if sizes else 1 + at % 5, len(tokens) - at)
        close(feed(tokens[at:at + n], at)[0], want[at:at + n], 2e-2 if cache_bf16 and n > 16 else 1e-3 if cache_bf16 else 3e-5)
        at += n


@pytest.mark.parametrize("rows", [1, 2, 40, 64, 150])
@pytest.mark.parametrize("cache_bf16", [False, True])
@pytest.mark.parametrize("window", [7, 32, 64, 65, 130])
def test_window_edge_is_exact(rows, cache_bf16, window):
    """One key stands out by a score of about 50: while it is visible it takes the whole softmax."""
    heads, dim, rot, vdim, rank = 2, 16, 8, 16, 32
    feed, oracle, s, tables = latent_case(heads, dim, rot, vdim, rank, window, 150, cache_bf16=cache_bf16, q_gain=0.05, base=1e9)
    r = rng_of(77)
    down = (r.standard_normal((64, rank + rot)) * 0.5).astype(np.float32)
    q = (r.standard_normal((64, heads, dim + rot)) * 0.05).astype(np.float32)
    # the first rotated pair turns by the position itself, so use the last pair (frequency about 0)
    q[:, :, dim + rot // 2 - 1] = 16.0
    down[5, rank + rot // 2 - 1] = 16.0
    s.set_parameter("down", down)
    s.set_parameter("q", q.reshape(64, -1))
    tokens = np.full(3 * window + 50, 1)
    tokens[:] = np.arange(len(tokens)) % 4 + 8
    special = 9
    tokens[special] = 5
    tables["down"], tables["q"] = down, q.reshape(64, -1)
    want = oracle(tokens, window)
    spread = np.abs(want[special + window - 1] - want[special + window]).max()
    assert spread > 0.1 * np.abs(want).max()                   # just inside and just outside differ visibly
    at = 0
    while at < len(tokens):
        n = min(rows, len(tokens) - at)
        close(feed(tokens[at:at + n], at)[0], want[at:at + n], 2e-2 if cache_bf16 else 1e-4)
        at += n


@pytest.mark.parametrize("heads,dim,rot,vdim,rank,window", [(2, 16, 8, 24, 32, 10), (3, 32, 16, 40, 64, 300), (9, 64, 32, 64, 136, 100), (2, 72, 24, 128, 256, 77),
                                                            (1, 128, 64, 128, 512, 128), (4, 184, 8, 8, 40, 64)])
def test_latent_attention_many_rows(heads, dim, rot, vdim, rank, window):
    """Portions of 64 and more rows (expanded keys and values), with fewer rows in between, several rings long."""
    feed, oracle, _, _ = latent_case(heads, dim, rot, vdim, rank, window, 200, cache_bf16=True, q_gain=2.0)
    sizes = [200, 64, 1, 100, 63, 65, 2, 199, 128]
    tokens = rng_of(5, window).integers(0, 64, sum(sizes))
    want, at = oracle(tokens, window), 0
    for n in sizes:
        close(feed(tokens[at:at + n], at)[0], want[at:at + n], 3e-2)
        at += n


def test_two_windows_share_one_cache():
    feed, oracle, _, _ = latent_case(2, 16, 8, 24, 32, 10, 32, window2=37, q_gain=2.0)
    tokens = rng_of(3).integers(0, 64, 150)
    want = [oracle(tokens, 10), oracle(tokens, 37)]
    at = 0
    for n in [32, 1, 2, 30, 5, 1, 32, 32, 15]:
        for got, w in zip(feed(tokens[at:at + n], at), want):
            close(got, w[at:at + n], 3e-5)
        at += n


def test_builders_refuse_bad_shapes():
    import meganeura_b200 as mg
    from meganeura_b200._lib import FMT_Q4, ROWS_TOKENS
    g = mg.Graph()
    x = g.input("x", [4, 32])
    pos = g.input_u32("pos", [1])
    with pytest.raises(mg.MgqError):
        g.norm(x, g.parameter("w", [31]), 1e-5)
    with pytest.raises(mg.MgqError):
        g.norm(x, g.parameter("w32", [32]), 1e-5, 0.0, FMT_Q4)
    with pytest.raises(mg.MgqError):
        g.token_shift(x, [g.parameter("mu", [32])], g.parameter("st", [32]))             # the state has two rows
    with pytest.raises(mg.MgqError):
        g.wkv(x, x, x, x, g.parameter("u", [32]), g.parameter("s", [7]), 2)
    with pytest.raises(mg.MgqError):
        g.latent_attention(x, g.parameter("c", [10, 24]), g.parameter_bf16("uk", [16, 16]), g.parameter_bf16("uv", [16, 16]), pos, 2, 8, 8, 8, 8, 1.0, 1e4)
    with pytest.raises(mg.MgqError):
        g.input_u32_rows("ids", 4, 9)
    ids = g.input_u32_rows("ids", 4, ROWS_TOKENS)
    y = g.embedding_scaled(ids, g.parameter("t", [8, 32]), 1.0)
    with pytest.raises(mg.MgqError):
        g.add(x, y)                                           # fixed rows and rows set per step
    g.set_outputs([y])
    s = mg.build_inference_session(g)
    with pytest.raises(mg.MgqError):
        s.set_rows(ROWS_TOKENS, 5)
    with pytest.raises(mg.MgqError):
        s.set_rows(ROWS_TOKENS, 0)
    with pytest.raises(mg.MgqError):
        s.set_rows(2, 1)                                      # no picked rows in this graph
