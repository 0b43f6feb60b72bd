"""CPU tests of the plain statement of the Zufilorn decoder (zufilorn_ref.py): its mechanisms against identities that do not
go through the same code, and the size of what single mistakes do to it (so that the GPU tests' tolerances are known to be
tight enough)."""
import copy
import math

import numpy as np
import pytest

import zufilorn_ref as R

RNG = np.random.default_rng(7)
CFG = {"architecture": "Zufilorn", "width": 60, "vocab": 83, "streams": 3, "max_positions": 64, "norm": {"eps": 1e-5}, "layers": [
    {"type": "channel_delta", "mixer": {"heads": 4, "kv_heads": 2, "dim": 12, "vdim": 20, "conv": 4}, "mlp": {"kind": "dense", "ff": 44}},
    {"type": "attention", "mlp": None, "mixer": {"heads": 4, "kv_heads": 2, "dim": 16, "vdim": 24, "scale": 0.25, "softcap": 10.0, "diff": 0.4,
                                                 "q_temp": {"coef": 0.5, "every": 6}}},
    {"type": "mlstm", "mixer": {"heads": 3, "dim": 12, "vdim": 16, "gate_cap": 6.0}, "mlp": {"kind": "dense", "ff": 44}}]}


def test_one_stream_of_ones_is_the_plain_residual():
    x, y = RNG.standard_normal((1, 5, 7)), RNG.standard_normal((5, 7))
    w = {"in": np.ones(1), "out": np.ones(1), "mix": np.ones((1, 1))}
    assert np.allclose(R.stream_input(x, w), x[0]) and np.allclose(R.stream_update(x, y, w), x + y)


def test_streams_mix_from_rows_to_columns():
    x = RNG.standard_normal((2, 1, 1))
    w = {"in": np.array([2.0, 3.0]), "out": np.array([0.0, 5.0]), "mix": np.array([[1.0, 10.0], [0.0, 1.0]])}
    assert np.allclose(R.stream_input(x, w), 2 * x[0] + 3 * x[1])
    new = R.stream_update(x, np.ones((1, 1)), w)
    assert np.allclose(new[0], x[0]) and np.allclose(new[1], 10 * x[0] + x[1] + 5)


def test_equal_channel_decays_are_the_scalar_rule():
    import vivezen_ref as V
    q, k, v = R.unit_norm(RNG.standard_normal((9, 5))), R.unit_norm(RNG.standard_normal((9, 5))), RNG.standard_normal((9, 4))
    beta, g = RNG.uniform(0, 1, 9), RNG.uniform(0.5, 1, 9)
    a, b = V.gated_delta_scan(q, k, v, beta, g), R.channel_delta_scan(q, k, v, beta, np.repeat(g[:, None], 5, 1))
    assert np.allclose(a[0], b[0]) and np.allclose(a[1], b[1])
    # decays act on rows of the state, which belong to key channels
    _, S = R.channel_delta_scan(q[:1], k[:1], v[:1], beta[:1], np.ones((1, 5)))
    g2 = RNG.uniform(0, 1, (1, 5))
    _, S2 = R.channel_delta_scan(q[:1], k[:1], v[:1], np.zeros(1), g2, S)
    assert np.allclose(S2, g2[0][:, None] * S)


def test_mlstm_is_carried_by_its_state_and_matches_its_closed_form():
    T = 12
    q, k, v = (RNG.standard_normal((T, n)) for n in (6, 6, 4))
    i, f = 3 * RNG.standard_normal(T), R.log_sigmoid(3 * RNG.standard_normal(T))
    o, st = R.mlstm_scan(q, k, v, i, f)
    o1, s1 = R.mlstm_scan(q[:5], k[:5], v[:5], i[:5], f[:5])
    o2, s2 = R.mlstm_scan(q[5:], k[5:], v[5:], i[5:], f[5:], s1)
    assert np.allclose(np.concatenate([o1, o2]), o) and all(np.allclose(a, b) for a, b in zip(st, s2))
    # without the running maximum: weights e^(i_s + sum of later f), read-out floor 1 (the maximum starts at 0)
    for t in range(T):
        wt = np.array([math.exp(i[s] + f[s + 1:t + 1].sum()) for s in range(t + 1)])
        m = max([f[:t + 1].sum()] + [i[s] + f[s + 1:t + 1].sum() for s in range(t + 1)])
        num, den = (wt * (k[:t + 1] @ q[t])) @ v[:t + 1], (wt * (k[:t + 1] @ q[t])).sum()
        assert np.allclose(o[t], num / (max(abs(den), 1.0) + 1e-6 * math.exp(m)))


def test_temperature_and_cap():
    t = R.query_temperature([0, 4, 5, 10, 11], {"coef": 2.0, "every": 6})
    assert np.allclose(t, 1 + 2 * np.log([1, 1, 2, 2, 3]))
    assert abs(R.soft_cap(1e9, 5.0) - 5.0) < 1e-9 and abs(R.soft_cap(0.01, 5.0) - 0.01) < 1e-6


def test_maps_cancel_when_equal_and_the_result_is_normalised():
    a = RNG.standard_normal((3, 8))
    assert np.allclose(R.combine_maps(a, a, 1.0, 0.2, 1e-5), 0.0)
    o = R.combine_maps(a, 0 * a, 0.7, 0.2, 0.0)
    assert np.allclose(np.sqrt((o ** 2).mean(-1)), 0.8)


def test_later_tokens_do_not_matter():
    w = R.random_weights(CFG, 1)
    t = RNG.integers(0, 83, 30).tolist()
    assert np.allclose(R.forward(CFG, w, t[:17]), R.forward(CFG, w, t)[:17])


CONFIG_MISTAKES = {
    "temperature step": lambda c: c["layers"][1]["mixer"]["q_temp"].update(every=7),
    "cap": lambda c: c["layers"][1]["mixer"].update(softcap=11.0),
    "share of the second map": lambda c: c["layers"][1]["mixer"].update(diff=0.41),
    "gate cap": lambda c: c["layers"][2]["mixer"].update(gate_cap=6.5),
    "epsilon": lambda c: c["norm"].update(eps=1e-2),
}
WEIGHT_MISTAKES = {
    "mix matrix transposed": ("l1.hc1.mix", lambda a: a.T),
    "streams swapped": ("l2.hc1.in", lambda a: a[::-1]),
    "taps reversed": ("l0.mix.k.conv", lambda a: a[:, ::-1]),
    "decay channels shifted": ("l0.mix.dt_bias", lambda a: np.roll(a, 1)),
    "maps swapped": ("l1.mix.k", lambda a: a.reshape(2, 2, 16, 60)[:, ::-1].reshape(64, 60)),
    "positions one off": ("pos", lambda a: np.roll(a, 1, 0)),
    "forget bias lost": ("l2.mix.f.b", lambda a: 0 * a),
    "norm weight around one": ("final.norm", lambda a: a - 1),
}


def _distance(cfg_a, w_a, cfg_b, w_b):
    t = np.random.default_rng(3).integers(0, 83, 40).tolist()
    a, b = R.forward(cfg_a, w_a, t), R.forward(cfg_b, w_b, t)
    return np.sqrt(((a - b) ** 2).mean(-1) / (a ** 2).mean()).max()


@pytest.mark.parametrize("name", sorted(CONFIG_MISTAKES))
def test_single_mistakes_in_constants_are_far_above_the_f32_tolerance(name):
    w, bad = R.random_weights(CFG, 1), copy.deepcopy(CFG)
    CONFIG_MISTAKES[name](bad)
    assert _distance(CFG, w, bad, w) > 10 * 1e-4


@pytest.mark.parametrize("name", sorted(WEIGHT_MISTAKES))
def test_single_mistakes_in_weights_are_far_above_the_f32_tolerance(name):
    w = R.random_weights(CFG, 1)
    key, f = WEIGHT_MISTAKES[name]
    assert _distance(CFG, w, CFG, dict(w, **{key: f(w[key])})) > 30 * 1e-4


def test_lost_states_show():
    """What a request would give if its second portion started from empty states."""
    w = R.random_weights(CFG, 1)
    w["pos"] = 0 * w["pos"]
    t = np.random.default_rng(4).integers(0, 83, 40).tolist()
    whole, cut = R.forward(CFG, w, t), R.forward(CFG, w, t[20:])
    assert (np.sqrt(((whole[20:] - cut) ** 2).mean(-1) / (whole ** 2).mean()))[:5].min() > 0.01
