"""Kugalorn without a GPU: configuration checks, the registry entry, weight names, and closed-form self-checks of the plain oracle
(slopes and windows, the turning of pairs, the gate per head, the choice of experts, the clamped unit, mixed copies, looped spans)."""
import json
import math

import numpy as np
import pytest

from tests import oracle_kugalorn as O


def _att(**kw):
    m = {"heads": 2, "kv_heads": 1, "dim": 4, "vdim": 6, "scale": 0.5, "mask": {"size": 3}}
    m.update(kw)
    return {"type": "attention", "mixer": m, "mlp": None}


def _latent(mlp=None, **kw):
    m = {"heads": 2, "dim": 4, "rot_dim": 2, "vdim": 6, "kv_rank": 5, "scale": 0.5, "rot": {"base": 100.0, "dims": 2}}
    m.update(kw)
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def _moe(shared=True):
    m = {"kind": "moe", "router": {"experts": 3, "top": 2}, "expert": {"ff": 7, "limit": 0.5}}
    return dict(m, shared={"ff": 9, "limit": 2.0}) if shared else m


def _cfg(layers, **kw):
    return dict({"architecture": "Kugalorn", "vocab": 11, "width": 8, "norm": {"eps": 1e-5}, "streams": 3, "layers": layers}, **kw)


def test_config_checks():
    from krasis_b200.kugalorn import KugalornConfig
    cfg = KugalornConfig.from_dict(_cfg([_att(), _latent(_moe())], loop={"start": 0, "stop": 1, "times": 3}))
    assert cfg.vocab == 11 and cfg.width == 8 and cfg.eps == 1e-5 and cfg.streams == 3 and cfg.runs() == [0, 0, 0, 1]
    assert KugalornConfig.from_dict(_cfg([_att(), _latent()])).runs() == [0, 1]
    for bad in (_cfg([dict(_att(), type="delta")]), _cfg([_att(heads=3, kv_heads=2)]), _cfg([_latent({"kind": "dense", "ff": 4})]), _cfg([], streams=0),
                _cfg([_latent(rot={"base": 10.0, "dims": 4})]), _cfg([_att()], loop={"start": 0, "stop": 2, "times": 2}),
                _cfg([_att()], loop={"start": 0, "stop": 1, "times": 0})):
        with pytest.raises(ValueError):
            KugalornConfig.from_dict(bad)


def test_layer_runs():
    from krasis_b200.mixers import layer_runs
    assert layer_runs(3) == [(0, False), (1, False), (2, False)]
    assert layer_runs(4, 1, 3, 2) == [(0, False), (1, True), (2, False), (1, True), (2, False), (3, False)]
    for n, loop in ((4, (0, 4, 3)), (5, (4, 5, 2)), (5, (2, 2, 9)), (3, (0, 1, 1))):
        assert [i for i, _ in layer_runs(n, *loop)] == O.layer_order(n, dict(zip(("start", "stop", "times"), loop)))


def test_registry_knows_the_design(tmp_path):
    from krasis_b200.registry import architecture_of
    (tmp_path / "config.json").write_text(json.dumps(_cfg([])))
    assert architecture_of(str(tmp_path)) == "Kugalorn"


def test_random_weights_have_the_designs_names():
    from krasis_b200.kugalorn import KugalornConfig, random_weights
    w = random_weights(KugalornConfig.from_dict(_cfg([_att(), _latent(_moe()), _att(kv_heads=2)])), 0)
    assert w["embed"].shape == (11, 8) and w["head"].shape == (11, 8) and w["final.norm"].shape == (8,)
    assert w["l0.mix.q"].shape == (8, 8) and w["l0.mix.k"].shape == (4, 8) and w["l0.mix.v"].shape == (6, 8) and w["l0.mix.o"].shape == (8, 12)
    assert w["l0.hc1.in"].shape == (3,) and w["l0.hc1.out"].shape == (3,) and w["l0.hc1.mix"].shape == (3, 3)
    assert "l0.norm2" not in w and "l0.hc2.in" not in w and "l1.norm2" in w and "l1.hc2.mix" in w
    assert w["l1.mix.q"].shape == (12, 8) and w["l1.mix.dkv"].shape == (7, 8) and w["l1.mix.dkv.norm"].shape == (5,)
    assert w["l1.mix.uk"].shape == (8, 5) and w["l1.mix.uv"].shape == (12, 5) and w["l1.mix.g"].shape == (2, 8)
    assert w["l1.mlp.router"].shape == (3, 8) and w["l1.mlp.router.b"].shape == (3,) and w["l1.mlp.e2.up"].shape == (7, 8)
    assert w["l1.mlp.shared.down"].shape == (8, 9) and "l1.mlp.e3.up" not in w and w["l2.mix.k"].shape == (8, 8)


def test_slopes_and_windows():
    from krasis_b200.mixers import distance_slopes
    assert O.head_slopes(4) == [2.0 ** -2, 2.0 ** -4, 2.0 ** -6, 2.0 ** -8]
    for H in (1, 3, 4, 12):
        assert np.allclose(distance_slopes(H).numpy(), O.head_slopes(H), rtol=1e-14, atol=0)
    assert O.window_keys(10, 4) == [7, 8, 9, 10] and O.window_keys(2, 4) == [0, 1, 2] and O.window_keys(5, 1) == [5]


def test_oracle_attention_weights_fall_with_the_distance():
    """Equal keys: the weights of a head are exp(-slope (i - j)), normalised, and unit-RMS queries make the scale of h irrelevant."""
    m = {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 3, "scale": 0.7, "mask": {"size": 2}}
    w = {"q": np.eye(2, 5), "k": np.eye(2, 5), "v": np.eye(3, 5, 2), "o": np.eye(3)}
    h = np.array([[1.0, 1.0, 1.0, 0, 0], [2.0, 2.0, 0, 1.0, 0], [5.0, 5.0, 0, 0, 1.0]])
    e = math.exp(-2.0 ** -8)
    assert np.allclose(O.windowed_attention(h, w, m, 0.0)[2], [0.0, e / (1 + e), 1 / (1 + e)])


def test_oracle_turns_neighbouring_pairs():
    x = np.zeros((3, 4))
    x[:, 2] = 1.0
    r = O.turn_pairs(x, [0, 1, 7], 16.0)                       # pair 1 of two turns by p * 16^(-1/2)
    assert np.allclose(r[:, 2], np.cos(np.array([0, 1, 7]) / 4)) and np.allclose(r[:, 3], np.sin(np.array([0, 1, 7]) / 4)) and np.all(r[:, :2] == 0)


def test_oracle_latent_gate_is_one_number_per_head():
    rng = np.random.default_rng(0)
    m = _latent()["mixer"]
    w = {"q": rng.normal(size=(12, 8)), "dkv": rng.normal(size=(7, 8)), "dkv.norm": np.ones(5), "uk": rng.normal(size=(8, 5)), "uv": rng.normal(size=(12, 5)),
         "g": np.zeros((2, 8)), "o": np.eye(12)}
    h = rng.normal(size=(6, 8))
    half = O.latent_attention(h, w, m, 1e-5)
    w["g"] = np.stack([np.zeros(8), 1e6 * np.ones(8)])
    moved = O.latent_attention(np.abs(h), w, m, 1e-5)
    w["g"] = np.zeros((2, 8))
    plain = O.latent_attention(np.abs(h), w, m, 1e-5)
    assert np.allclose(moved[:, :6], plain[:, :6]) and np.allclose(moved[:, 6:], 2 * plain[:, 6:]) and half.shape == (6, 12)


def test_oracle_choice_and_clamped_unit():
    z = np.array([0.0, 3.0, 1.0, 2.0])
    e = math.exp(-1.0)
    assert [i for i, _ in O.choose(z, 2)] == [1, 3] and np.allclose([p for _, p in O.choose(z, 2)], [1 / (1 + e), e / (1 + e)])
    w = {"gate": np.eye(1), "up": np.eye(1), "down": np.eye(1)}
    s = lambda v: v * O.sigmoid(1.702 * v)
    assert np.allclose(O.clamped_unit(np.array([[5.0]]), w, 2.0), s(2.0) * 3.0)       # gate cut from above, up on both sides
    assert np.allclose(O.clamped_unit(np.array([[-5.0]]), w, 2.0), s(-5.0) * -1.0)
    assert np.allclose(O.clamped_unit(np.array([[0.5]]), w, 2.0), s(0.5) * 1.5)


def test_oracle_copies_are_mixed_from_the_old_ones():
    xs = [np.array([[1.0]]), np.array([[10.0]])]
    mix = np.array([[1.0, 2.0], [3.0, 4.0]])                   # [from, to]
    new = O.write_streams(xs, mix, np.array([0.5, -1.0]), np.array([[100.0]]))
    assert new[0].item() == 1 + 30 + 50 and new[1].item() == 2 + 40 - 100
    assert O.read_streams(xs, np.array([2.0, 0.5])).item() == 7.0
    assert O.layer_order(4, {"start": 1, "stop": 3, "times": 2}) == [0, 1, 2, 1, 2, 3] and O.layer_order(2, None) == [0, 1]
