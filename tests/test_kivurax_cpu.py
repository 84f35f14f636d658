"""Kivurax without a GPU: configuration checks, the registry entry, weight names, the frequency table, and closed-form self-checks of the plain
oracle (the matrix memory's gates and divisor, the delta rule, the added one, keys as values, the recurrent block, weights on the experts'
inputs, the norm on the output)."""
import json
import math

import numpy as np
import pytest

from tests import oracle_kivurax as O


def _mem(mlp=None, **kw):
    return {"type": "mlstm", "mixer": dict({"heads": 2, "dim": 3, "vdim": 5, "gate_cap": 4.0}, **kw), "mlp": mlp}


def _delta(mlp=None, **kw):
    return {"type": "delta", "mixer": dict({"heads": 4, "kv_heads": 2, "dim": 3, "vdim": 5, "conv": 2}, **kw), "mlp": mlp}


def _par(mlp=None, left=None, right=None):
    a = {"heads": 2, "kv_heads": 1, "dim": 6, "vdim": 6, "scale": 0.5, "mask": {"size": 3},
         "rot": {"base": 100.0, "dims": 4, "scaling": {"factor": 2.0, "original": 32, "fast": 4.0, "slow": 1.0}}}
    b = {"width": 12, "blocks": 3, "conv": 3}
    return {"type": "parallel", "mixer": {"left": dict(a, **(left or {})), "right": dict(b, **(right or {})), "left_scale": 0.5, "right_scale": 2.0}, "mlp": mlp}


DENSE, MOE = {"kind": "dense", "ff": 7}, {"kind": "moe", "router": {"experts": 3, "top": 2}, "expert": {"ff": 7}}


def _cfg(layers, **kw):
    return dict({"architecture": "Kivurax", "vocab": 11, "width": 8, "norm": {"eps": 1e-5}, "residual_mult": 0.4, "layers": layers}, **kw)


def test_config_checks():
    from krasis_b200.kivurax import KivuraxConfig
    cfg = KivuraxConfig.from_dict(_cfg([_mem(), _delta(MOE), _par(DENSE)]))
    assert cfg.vocab == 11 and cfg.width == 8 and cfg.eps == 1e-5 and cfg.residual_mult == 0.4 and len(cfg.layers) == 3
    for bad in ([dict(_mem(), type="attention")], [_delta(kv_heads=3)], [_par(left={"kv_heads": 3})], [_par(left={"vdim": 4})], [_par(right={"blocks": 5})],
                [_mem({"kind": "sparse"})]):
        with pytest.raises(ValueError):
            KivuraxConfig.from_dict(_cfg(bad))


def test_registry_knows_the_design(tmp_path):
    from krasis_b200.registry import architecture_of
    (tmp_path / "config.json").write_text(json.dumps(_cfg([])))
    assert architecture_of(str(tmp_path)) == "Kivurax"


def test_random_weights_have_the_designs_names():
    from krasis_b200.kivurax import KivuraxConfig, random_weights
    w = random_weights(KivuraxConfig.from_dict(_cfg([_mem(), _delta(MOE), _par(DENSE)])), 0)
    shapes = {k: tuple(v.shape) for k, v in w.items()}
    assert shapes["embed"] == (11, 8) and "head" not in w and shapes["final.norm"] == (8,) and "l0.norm2" not in w and shapes["l1.norm2"] == (8,)
    assert shapes["l0.mix.q"] == (6, 8) and shapes["l0.mix.v"] == (10, 8) and shapes["l0.mix.i"] == (2, 8) and shapes["l0.mix.f.b"] == (2,) and shapes["l0.mix.norm"] == (10,)
    assert shapes["l1.mix.k"] == (6, 8) and shapes["l1.mix.v.conv"] == (20, 2) and shapes["l1.mix.norm"] == (5,) and shapes["l1.mix.A_log"] == (4,)
    assert shapes["l1.mlp.router"] == (3, 8) and shapes["l1.mlp.e2.down"] == (8, 7) and "l1.mlp.e3.up" not in w
    assert "l2.mix.left.v" not in w and shapes["l2.mix.left.k.norm"] == (6,) and shapes["l2.mix.left.o"] == (8, 12)
    assert shapes["l2.mix.right.ra"] == (3, 4, 4) and shapes["l2.mix.right.conv"] == (12, 3) and shapes["l2.mix.right.lam"] == (12,)
    assert shapes["l2.mlp.gate.b"] == (7,) and shapes["l2.mlp.down.b"] == (8,)


def test_frequency_table_matches_the_plain_one():
    from krasis_b200.mixers import yarn_table
    for rot in ({"base": 100.0, "dims": 4, "scaling": {"factor": 2.0, "original": 32, "fast": 4.0, "slow": 1.0}}, {"base": 1e4, "dims": 48, "scaling": None},
                {"base": 5e5, "dims": 32, "scaling": {"factor": 16.0, "original": 8192, "fast": 32.0, "slow": 1.0}}):
        f, amp = O.pair_frequencies(rot)
        got, got_amp = yarn_table(rot["dims"], rot["base"], rot["scaling"])
        assert np.allclose(got.numpy(), f, rtol=1e-13, atol=0) and abs(got_amp - amp) < 1e-15


def test_mixer_options_that_exclude_each_other():
    import torch
    from krasis_b200.mixers import GatedRecurrentUnit, MultiMapAttention, RoutedExperts, SideBySide
    w = {k: torch.zeros(4, 8) for k in ("q", "k")}
    w["o"] = torch.zeros(8, 4)
    cpu = torch.device("cpu")
    MultiMapAttention(w, 1, 1, 1, 4, 4, 1.0, 1e-5, torch.float32, cpu, window=3, keys_as_values=True, off_by_one=True)
    for kw in (dict(weights=dict(w, v=torch.zeros(4, 8))), dict(weights=dict(w, sink=torch.zeros(1)))):
        with pytest.raises(ValueError):
            MultiMapAttention(kw["weights"], 1, 1, 1, 4, 4, 1.0, 1e-5, torch.float32, cpu, window=3, keys_as_values=True, off_by_one=True)
    with pytest.raises(ValueError):
        RoutedExperts({"router": torch.zeros(3, 8)}, 2, 1, 1, torch.float32, cpu, weight_input=True)
    with pytest.raises(ValueError):
        SideBySide(None, None)
    with pytest.raises(ValueError):
        GatedRecurrentUnit({}, 10, 3, 2, torch.float32, cpu)
    assert SideBySide(None, None, scales=(0.5, 2)).scales == (0.5, 2.0)


def test_oracle_matrix_memory_of_two_tokens():
    """One head, one key channel, gates without input: both tokens by hand, with the floor of the divisor at work in the first."""
    c = {"heads": 1, "dim": 1, "vdim": 2, "gate_cap": 2.0}
    w = {"q": np.array([[1.0, 0, 0]]), "k": np.array([[0, 1.0, 0]]), "v": np.array([[0, 0, 1.0], [0, 0, 3.0]]), "i": np.zeros((1, 3)), "f": np.zeros((1, 3)),
         "i.b": np.array([-1.0]), "f.b": np.array([0.5]), "g": np.zeros((2, 3)), "norm": np.ones(2), "o": np.eye(2)}
    i, f = 2 * math.tanh(-0.5), -math.log1p(math.exp(-2 * math.tanh(0.25)))
    h = np.array([[1.0, 0.2, 1.0], [1.0, 3.0, -1.0]])
    m1 = max(f, i)
    S1, n1 = math.exp(i - m1) * 0.2 * np.array([1.0, 3.0]), math.exp(i - m1) * 0.2
    o1 = S1 / (max(n1, math.exp(-m1)) + 1e-6)
    m2 = max(f + m1, i)
    S2 = math.exp(f + m1 - m2) * S1 + math.exp(i - m2) * 3.0 * np.array([-1.0, -3.0])
    n2 = math.exp(f + m1 - m2) * n1 + math.exp(i - m2) * 3.0
    o2 = S2 / (max(n2, math.exp(-m2)) + 1e-6)
    assert n1 < math.exp(-m1)
    want = np.stack([o / np.sqrt((o * o).mean() + 0.1) * 0.5 for o in (o1, o2)])
    assert np.allclose(O.matrix_memory(h, w, c, 0.1), want)


def test_oracle_delta_rule_replaces_what_a_key_holds():
    """No decay, full write strength: the second write to the same unit key replaces the first."""
    c = {"heads": 1, "kv_heads": 1, "dim": 1, "vdim": 1, "conv": 1}
    one = np.array([[1.0, 0, 0]])
    w = {"q": one, "k": one, "v": np.array([[0, 1.0, 0]]), "q.conv": np.ones((1, 1)), "k.conv": np.ones((1, 1)), "v.conv": np.ones((1, 1)), "b": np.array([[50.0, 0, 0]]),
         "a": np.zeros((1, 3)), "A_log": np.array([-50.0]), "dt_bias": np.zeros(1), "norm": np.ones(1), "g": np.array([[0, 0, 1.0]]), "o": np.eye(1)}
    h = np.array([[1.0, 2.0, 4.0], [1.0, 5.0, 4.0]])
    k = O.silu(1.0) / math.sqrt(O.silu(1.0) ** 2 + 1e-6)
    s1 = k * O.silu(2.0)
    s2 = s1 + k * (O.silu(5.0) - s1 * k)
    got = O.delta_rule(h, w, c, 0.5)[:, 0]
    assert np.allclose(got, [s * k / math.sqrt((s * k) ** 2 + 0.5) * O.silu(4.0) for s in (s1, s2)], rtol=1e-9)


def test_oracle_added_one_and_keys_as_values():
    assert np.allclose(O.softmax_plus_one(np.array([0.0, math.log(2.0)])), [0.25, 0.5])
    assert np.allclose(O.softmax_plus_one(np.array([-800.0])), [0.0]) and np.allclose(O.softmax_plus_one(np.array([800.0])), [1.0])
    m = {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 2, "scale": 0.0, "mask": {"size": 2}, "rot": {"base": 10.0, "dims": 2, "scaling": None}}
    w = {"q": np.eye(2), "k": np.eye(2), "q.norm": np.ones(2), "k.norm": np.full(2, 7.0), "o": np.eye(2)}
    h = np.array([[1.0, 2.0], [30.0, 4.0], [5.0, 60.0]])
    assert np.allclose(O.key_value_attention(h, w, m, 1e-5), [h[0] / 2, (h[0] + h[1]) / 3, (h[1] + h[2]) / 3])     # equal scores, values unnormed and unturned


def test_oracle_turns_neighbouring_pairs_with_an_amplitude():
    rot = {"base": 16.0, "dims": 4, "scaling": {"factor": math.e, "original": 1e-9, "fast": 2.0, "slow": 1.0}}       # original tiny: all pairs but the first slowed
    f, amp = O.pair_frequencies(rot)
    assert np.allclose(f, [1.0, 0.25 / math.e]) and abs(amp - 1.1) < 1e-12
    x = np.zeros((3, 1, 5))
    x[:, 0, 2], x[:, 0, 4] = 1.0, 2.0
    r = O.turn_pairs(x, rot)[:, 0]
    p = np.arange(3) * 0.25 / math.e
    assert np.allclose(r[:, 2], 1.1 * np.cos(p)) and np.allclose(r[:, 3], 1.1 * np.sin(p)) and np.all(r[:, 4] == 2.0) and np.all(r[:, :2] == 0)
    assert O.window_keys(10, 4) == [7, 8, 9, 10] and O.window_keys(2, 4) == [0, 1, 2] and O.window_keys(5, 1) == [5]


def test_oracle_recurrent_block_of_two_tokens():
    """Gates at one half, a convolution of two taps whose inputs carry their bias only where there is a token."""
    c = {"width": 1, "blocks": 1, "conv": 2}
    w = {"x": np.array([[1.0, 0]]), "x.b": np.array([0.5]), "y": np.array([[0, 1.0]]), "y.b": np.array([0.25]), "conv": np.array([[2.0, 3.0]]), "conv.b": np.array([-1.0]),
         "ra": np.zeros((1, 1, 1)), "ra.b": np.zeros((1, 1)), "ri": np.zeros((1, 1, 1)), "ri.b": np.zeros((1, 1)), "lam": np.array([-2.0]), "o": np.eye(1)}
    h = np.array([[1.0, 0.75], [2.0, -0.25]])
    u = [3 * 1.5 - 1, 2 * 1.5 + 3 * 2.5 - 1]
    a = math.exp(-4.0 * math.log1p(math.exp(-2.0)))
    b = math.sqrt(1 - a * a) * 0.5
    s = [b * u[0], a * b * u[0] + b * u[1]]
    assert np.allclose(O.recurrent_block(h, w, c)[:, 0], [s[0] * O.gelu_tanh(1.0), 0.0])
    assert np.allclose(O.block_product(np.arange(4.0)[None], np.stack([np.eye(2), 2 * np.ones((2, 2))])), [[0, 1, 10, 10]])


def test_oracle_weights_on_the_experts_inputs_and_biases():
    z = np.array([0.0, 3.0, 1.0, 2.0])
    assert [e for e, _ in O.choose(z, 2)] == [1, 3] and np.allclose([p for _, p in O.choose(z, 2)], [1 / (1 + math.exp(-3)), 1 / (1 + math.exp(-2))])
    w = {"router": np.array([[0.0]]), "e0.gate": np.eye(1), "e0.up": np.eye(1), "e0.down": np.eye(1)}
    got = O.routed_experts(np.array([[4.0]]), w, {"router": {"experts": 1, "top": 1}, "expert": {"ff": 1}})
    assert np.allclose(got, O.silu(2.0) * 2.0)                            # half of 4 goes in
    d = {"gate": np.eye(1), "up": np.eye(1), "down": 3 * np.eye(1), "gate.b": np.array([1.0]), "up.b": np.array([-0.5]), "down.b": np.array([7.0])}
    assert np.allclose(O.dense(np.array([[2.0]]), d), 3 * O.silu(3.0) * 1.5 + 7)


def test_oracle_norms_the_output_only():
    """A layer whose mixer and feed-forward are replaced: the stream is read as it is, and the added terms are unit rows times m w."""
    keep = O.mixer, O.feed_forward
    seen = []
    try:
        O.mixer = lambda kind, h, w, c, eps: seen.append(h) or 5.0 * np.ones_like(h)
        O.feed_forward = lambda h, w, c: seen.append(h) or -2.0 * np.ones_like(h)
        w = {"embed": np.array([[10.0, 20.0], [1.0, 3.0]]), "l0.norm1": np.array([1.0, 2.0]), "l0.norm2": np.array([4.0, 1.0]), "final.norm": np.ones(2)}
        tr = []
        O.forward({"norm": {"eps": 0.0}, "residual_mult": 0.5, "layers": [{"type": "mlstm", "mixer": {}, "mlp": {"kind": "dense"}}]}, w, [1, 0], tr)
    finally:
        O.mixer, O.feed_forward = keep
    assert np.allclose(seen[0], [[1, 3], [10, 20]]) and np.allclose(seen[1], [[1.5, 4], [10.5, 21]]) and np.allclose(tr[0], [[-0.5, 3.5], [8.5, 20.5]])
