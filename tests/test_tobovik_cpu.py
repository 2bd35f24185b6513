"""CPU checks: the configuration reader and the oracle's own consistency."""
import numpy as np
import pytest

from meganeura_b200.registry import ARCHITECTURES, model_class
from meganeura_b200.tobovik import TobovikConfig, gla_prefixes
from oracle import tobovik_oracle as T
from tobovik_util import CONFIGS, attention, config, gla, parallel, side, weights


def test_config_reads_every_size_and_constant():
    cfg = TobovikConfig.from_dict(config(77, 40, [parallel(attention(6, 3, 10, 7, 0.25, 0.125, 9), side(2, 5, 11, 3.0), 0.5, -2.0, 20), gla(4, 6, 8, 7.0),
                                                  gla(4, 6, 8, 7.0, weights_of=1)], eps=0.01))
    assert (cfg.vocab, cfg.width, cfg.eps) == (77, 40, 0.01)
    a, b, c = cfg.layers
    assert (a.left_scale, a.right_scale, a.ff, a.weights) == (0.5, -2.0, 20, 0)
    m = a.attention
    assert (m.heads, m.kv_heads, m.dim, m.vdim, m.scale, m.temp_coef, m.temp_every) == (6, 3, 10, 7, 0.25, 0.125, 9.0)
    assert (a.gla.heads, a.gla.dim, a.gla.vdim, a.gla.tau) == (2, 5, 11, 3.0)
    assert b.attention is None and (b.gla.heads, b.gla.tau, b.ff, b.weights) == (4, 7.0, 0, 1)
    assert c.weights == 1 and c.gla == b.gla
    assert gla_prefixes(cfg) == ["l0.mix.right", "l1.mix"]
    assert model_class(config(4, 4, [])) is ARCHITECTURES["Tobovik"]


def test_weights_of_follows_to_the_owner():
    cfg = TobovikConfig.from_dict(config(8, 8, [gla(1, 4, 4, weights_of=2), gla(1, 4, 4, weights_of=0), gla(1, 4, 4)]))
    assert [layer.weights for layer in cfg.layers] == [2, 2, 2]


def test_config_refuses_what_it_cannot_build():
    def bad(layers):
        with pytest.raises(ValueError):
            TobovikConfig.from_dict(config(10, 8, layers))
    bad([{"type": "other", "mixer": {"heads": 1, "dim": 2, "vdim": 2, "tau": 1}, "mlp": None}])
    bad([dict(gla(1, 4, 4), mlp={"kind": "sparse", "ff": 4})])
    bad([gla(1, 4, 4, weights_of=0)])                                        # itself
    bad([gla(1, 4, 4, weights_of=1), gla(1, 4, 4, weights_of=0)])            # a ring
    bad([gla(1, 4, 4, weights_of=5)])
    bad([gla(1, 4, 4), gla(1, 8, 4, weights_of=0)])                          # other sizes
    bad([parallel(attention(3, 2, 4, 4), side(1, 4, 4))])                    # heads that do not divide


@pytest.mark.parametrize("name", ["shared", "odd"])
def test_oracle_does_not_depend_on_the_cut(name):
    cfg, rank = CONFIGS[name]
    w = weights(cfg, rank)
    tokens = np.random.default_rng(1).integers(0, cfg["vocab"], 40)
    whole = T.TobovikOracle(cfg, w).step(tokens)
    o = T.TobovikOracle(cfg, w)
    parts = [o.step(tokens[a:b]) for a, b in ((0, 1), (1, 3), (3, 20), (20, 21), (21, 40))]
    assert np.abs(np.concatenate(parts) - whole).max() < 1e-9 * np.abs(whole).max()


def test_oracle_mechanisms_by_hand():
    # one head, one dimension: the recurrence written out (decay first, then the token itself, then the reading)
    q, k, v, a = (np.array([[[x]], [[y]]], float) for x, y in ((2, 3), (5, 7), (11, 13), (0.5, 0.25)))
    state = np.full((1, 1, 1), 8.0)
    o = T.gla_scan(q, k, v, a, state)
    assert np.allclose(o.reshape(-1), [2 * (4 + 55), 3 * (0.25 * 59 + 91)]) and np.isclose(state[0, 0, 0], 0.25 * 59 + 91)
    assert np.isclose(T.channel_decay(np.array([[2.0]]), np.array([[0.5]]), np.array([-1.0]), 4.0)[0, 0], 0.5 ** 0.25)
    assert np.allclose(T.query_temperature([0, 2, 3, 7], 0.5, 4), [1, 1, 1 + 0.5 * np.log(2), 1 + 0.5 * np.log(3)])
    # two query heads share a key head; token 1 sees tokens 0 and 1
    out = T.causal_attention(np.zeros((2, 2, 1)), np.zeros((2, 1, 1)), np.array([[[1.0]], [[4.0]]]), 0, 1.0)
    assert np.allclose(out.reshape(-1), [1, 1, 2.5, 2.5])
    p = T.position_vectors([3], 3)[0]
    assert np.allclose(p, [np.sin(3), np.cos(3), np.sin(3 * 10000 ** (-2 / 3))])
    assert np.isclose(T.silu(2.0), 2 / (1 + np.exp(-2))) and np.isclose(T.rms_norm([3.0, 4.0], [1.0, 2.0], 0.5)[1], 8 / np.sqrt(13))
