"""CPU checks: the configuration reader, the weight container, the oracle's own consistency."""
import numpy as np
import pytest

from meganeura_b200.petotar import PetotarConfig
from meganeura_b200.registry import ARCHITECTURES, model_class
from meganeura_b200.weights import SafeTensors, to_bf16, write_safetensors
from oracle import petotar_oracle as P
from petotar_util import CONFIGS, config, latent, mlstm, weights, wkv


def test_config_reads_every_size_and_constant():
    cfg = PetotarConfig.from_dict(config(77, 40, [wkv(2, 6), latent(3, 10, 4, 7, 12, 5, base=321.0, scale=0.25, ff=20, limit=1.25),
                                                  mlstm(1, 9, 11, 4.5), latent(1, 8, 4, 3, 12, 6, base=321.0, kv_from=1)], eps=0.01, scale=2.5))
    assert (cfg.vocab, cfg.width, cfg.eps, cfg.embedding_scale) == (77, 40, 0.01, 2.5)
    a, b, c, d = cfg.layers
    assert (a.type, a.heads, a.dim, a.vdim, a.ff) == ("wkv", 2, 6, 6, 0)
    assert (b.heads, b.dim, b.rot_dim, b.vdim, b.kv_rank, b.window, b.rot_base, b.scale, b.ff, b.limit) == (3, 10, 4, 7, 12, 5, 321.0, 0.25, 20, 1.25)
    assert (c.dim, c.vdim, c.gate_cap) == (9, 11, 4.5)
    assert d.kv_from == 1 and b.kv_from is None


def test_config_refuses_what_it_cannot_build():
    def bad(layers):
        with pytest.raises(ValueError):
            PetotarConfig.from_dict(config(10, 8, layers))
    bad([{"type": "other", "mixer": {"heads": 1, "dim": 2}, "mlp": None}])
    bad([latent(1, 4, 2, 4, 8, 3, kv_from=0)])                                           # its own cache
    bad([wkv(1, 4), latent(1, 4, 2, 4, 8, 3, kv_from=0)])                                # no cache there
    bad([latent(1, 4, 2, 4, 8, 3), latent(1, 4, 2, 4, 9, 3, kv_from=0)])                 # another rank
    bad([latent(1, 4, 2, 4, 8, 3), latent(1, 4, 2, 4, 8, 3, base=5.0, kv_from=0)])       # another rotation
    with pytest.raises(ValueError):
        model_class({"architecture": "Unknown"})
    assert "Petotar" in ARCHITECTURES


def test_safetensors_round_trip_and_damage(tmp_path):
    a = np.arange(12, dtype=np.float32).reshape(3, 4) / 7
    path = tmp_path / "m.safetensors"
    write_safetensors(str(path), {"x": ("BF16", to_bf16(a)), "y": ("F32", a)})
    t = SafeTensors(str(path))
    assert t.shape("x") == (3, 4) and t.dtype("x") == "BF16" and (t.raw("x") == to_bf16(a)).all() and (t.f32("y") == a).all()
    assert np.abs(t.f32("x") - a).max() <= 2 ** -8 * np.abs(a).max()
    with pytest.raises(KeyError):
        t.shape("z")
    path.write_bytes(path.read_bytes()[:-8])
    with pytest.raises(ValueError):
        SafeTensors(str(path))
    path.write_bytes(b"\x01")
    with pytest.raises(ValueError):
        SafeTensors(str(path))


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_oracle_does_not_depend_on_the_cut(name):
    cfg, rank = CONFIGS[name]
    w = weights(cfg, rank)
    tokens = np.random.default_rng(1).integers(0, cfg["vocab"], 40)
    whole = P.PetotarOracle(cfg, w).step(tokens)
    o = P.PetotarOracle(cfg, w)
    parts = [o.step(tokens[a:b]) for a, b in ((0, 1), (1, 3), (3, 20), (20, 21), (21, 40))]
    assert np.abs(np.concatenate(parts) - whole).max() < 1e-9 * np.abs(whole).max()


def test_oracle_mechanisms_by_hand():
    # one head, one dimension: the recurrences written out
    r, k, v, w = (np.array([[[x]], [[y]]], float) for x, y in ((2, 3), (5, 7), (11, 13), (0.5, 0.25)))
    state = np.zeros((1, 1, 1))
    o = P.wkv_scan(r, k, v, w, np.array([[0.1]]), state)
    assert np.allclose(o.reshape(-1), [2 * 0.1 * 55, 3 * (55 + 0.1 * 91)]) and np.isclose(state[0, 0, 0], 0.25 * 55 + 91)
    S, n, m = np.zeros((1, 1, 1)), np.zeros((1, 1)), np.zeros(1)
    o = P.mlstm_scan(r, k, v, np.array([[1.0], [-2.0]]), np.array([[-0.5], [-0.25]]), S, n, m)
    assert np.isclose(m[0], 0.75)                                   # max(0 - .5, 1) = 1, then max(1 - .25, -2)
    assert np.isclose(o[0, 0, 0], 2 * 55 / (max(10, np.exp(-1)) + 1e-6))
    keep, write = np.exp(-0.25 + 1 - 0.75), np.exp(-2 - 0.75)
    assert np.isclose(S[0, 0, 0], keep * 55 + write * 91)
    i, f = P.mlstm_gates(np.array([100.0]), np.array([-100.0]), 3.0)
    assert np.isclose(i[0], 3.0) and np.isclose(f[0], -np.log1p(np.exp(3.0)))
    assert np.isclose(P.clamped_glu(9.0, -9.0, 2.0), 2 * P.sigmoid(3.404) * -1)
    x = P.rotate_half(np.array([1.0, 0.0, 0.0, 0.0]), 3, 100.0)
    assert np.allclose(x, [np.cos(3), 0, np.sin(3), 0])
    # a window of 2: token 2 sees tokens 1 and 2 only
    q = np.ones((3, 1, 1))
    out = P.window_attention(q, np.zeros((3, 1, 1)), np.arange(3.0).reshape(3, 1, 1), 0, 2, 1.0)
    assert np.allclose(out.reshape(-1), [0, 0.5, 1.5])
