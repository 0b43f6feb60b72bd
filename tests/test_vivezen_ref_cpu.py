"""CPU tests of the plain statement of the hybrid decoder (vivezen_ref.py): its mechanisms against identities that
do not go through the same code, and the size of what single mistakes do to it (so that the GPU tests' tolerances
are known to be tight enough)."""
import copy
import math
import os
import subprocess
import sys

import numpy as np
import pytest

import vivezen_ref as R

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
RNG = np.random.default_rng(3)

CFG = {"architecture": "Vivezen", "width": 60, "vocab": 83, "norm": {"eps": 1e-5}, "layers": [
    {"type": "delta", "mixer": {"heads": 4, "kv_heads": 2, "dim": 12, "vdim": 20, "conv": 4}, "mlp": {"kind": "dense", "ff": 44}},
    {"type": "latent_attention", "mlp": None,
     "mixer": {"heads": 3, "dim": 20, "rot_dim": 8, "vdim": 16, "q_rank": 24, "kv_rank": 28, "mask": {"size": 11}, "scale": 28 ** -0.5,
               "rot": {"base": 500.0, "dims": 8, "scaling": {"factor": 4.0, "fast": 8.0, "slow": 0.5, "original": 64}}}},
    {"type": "delta", "mixer": {"heads": 4, "kv_heads": 2, "dim": 12, "vdim": 20, "conv": 4}, "mlp": {"kind": "dense", "ff": 44}, "weights_of": 0}]}


def test_rotation_keeps_lengths_and_depends_on_distance_only():
    rot = {"base": 200.0, "dims": 6}
    q, k = RNG.standard_normal((1, 9)), RNG.standard_normal((1, 9))
    a = R.rotate(q, [5], rot)
    assert abs(np.linalg.norm(a) - np.linalg.norm(q)) < 1e-12 and (a[:, 6:] == q[:, 6:]).all()
    d = [float(R.rotate(q, [p + 7], rot)[0] @ R.rotate(k, [p], rot)[0]) for p in (0, 3, 400)]
    assert max(d) - min(d) < 1e-10
    # one pair by hand: entries 1 and 4 at position 2
    t = 2 * 200.0 ** (-2 / 6)
    x = np.arange(9.0)[None]
    assert np.allclose(R.rotate(x, [2], rot)[0, [1, 4]], [1 * math.cos(t) - 4 * math.sin(t), 4 * math.cos(t) + 1 * math.sin(t)])


def test_frequency_scaling_ends():
    rot = {"base": 10000.0, "dims": 64, "scaling": {"factor": 8.0, "fast": 32.0, "slow": 1.0, "original": 4096}}
    f, m = R.rotary_frequencies(rot)
    plain, one = R.rotary_frequencies({"base": 10000.0, "dims": 64})
    assert one == 1.0 and abs(m - (0.1 * math.log(8.0) + 1.0)) < 1e-12
    assert np.allclose(f[:3], plain[:3]) and np.allclose(f[-3:], plain[-3:] / 8.0)
    assert (f <= plain + 1e-15).all() and (np.diff(f) < 0).all()


def test_window_and_convolution_by_hand():
    m = R.visible(6, 3)
    assert [[j for j in range(6) if m[i, j]] for i in (0, 1, 2, 5)] == [[0], [0, 1], [0, 1, 2], [3, 4, 5]]
    assert R.visible(4, None).sum() == 10
    x, w = RNG.standard_normal((5, 2)), RNG.standard_normal((2, 3))
    y = R.causal_conv(x, w)
    assert np.allclose(y[0], x[0] * w[:, 2]) and np.allclose(y[4], x[2] * w[:, 0] + x[3] * w[:, 1] + x[4] * w[:, 2])
    assert np.allclose(R.causal_conv(x[3:], w, x[1:3]), y[3:])


def test_delta_scan_is_carried_by_its_state_and_solves_for_the_value():
    q, k = R.unit_norm(RNG.standard_normal((9, 5))), R.unit_norm(RNG.standard_normal((9, 5)))
    v, beta, g = RNG.standard_normal((9, 4)), RNG.uniform(0, 1, 9), RNG.uniform(0.5, 1, 9)
    o, S = R.gated_delta_scan(q, k, v, beta, g)
    o1, S1 = R.gated_delta_scan(q[:4], k[:4], v[:4], beta[:4], g[:4])
    o2, S2 = R.gated_delta_scan(q[4:], k[4:], v[4:], beta[4:], g[4:], S1)
    assert np.allclose(np.concatenate([o1, o2]), o) and np.allclose(S, S2)
    # with a full step the state answers the written key with the written value
    o, S = R.gated_delta_scan(k, k, v, np.ones(9), g)
    assert np.allclose(o, v, atol=1e-4)


def test_unused_positions_do_not_matter():
    w = R.random_weights(CFG, 1)
    t = RNG.integers(0, 83, 30).tolist()
    full = R.forward(CFG, w, t)
    assert np.allclose(R.forward(CFG, w, t[:17]), full[:17])


MISTAKES = {
    "window one wider": lambda c: c["layers"][1]["mixer"]["mask"].update(size=12),
    "window one narrower": lambda c: c["layers"][1]["mixer"]["mask"].update(size=10),
    "plain frequencies": lambda c: c["layers"][1]["mixer"]["rot"].pop("scaling"),
    "shared weights not shared": lambda c: c["layers"].pop(),
    "epsilon": lambda c: c["norm"].update(eps=1e-3),
}


@pytest.mark.parametrize("name", sorted(MISTAKES))
def test_single_mistakes_are_far_above_the_f32_tolerance(name):
    w = R.random_weights(CFG, 1)
    t = RNG.integers(0, 83, 40).tolist()
    bad = copy.deepcopy(CFG)
    MISTAKES[name](bad)
    a, b = R.forward(CFG, w, t), R.forward(bad, w, t)
    assert (np.sqrt(((a - b) ** 2).mean(-1) / (a ** 2).mean())).max() > 20 * 5e-5


def test_lost_state_and_lost_convolution_inputs_show():
    """What a request would give if its second portion started from an empty state."""
    w = R.random_weights(CFG, 1)
    t = RNG.integers(0, 83, 40).tolist()
    whole, cut = R.forward(CFG, w, t), R.forward(CFG, w, t[20:])
    assert (np.sqrt(((whole[20:] - cut) ** 2).mean(-1) / (whole ** 2).mean()))[:5].min() > 0.01


def test_trace_runner_describes_itself():
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--help"], capture_output=True, text=True, timeout=60)
    assert r.returncode == 0 and "--max-tokens" in r.stdout and os.access(os.path.join(ROOT, "bin", "trace_run"), os.X_OK)
