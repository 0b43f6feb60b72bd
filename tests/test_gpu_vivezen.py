"""GPU parity tests of the hybrid decoder (Vivezen) against the plain float64 statement in vivezen_ref.py: each
mechanism alone, whole models, portions, batches, reused slots, decoding and generation.

Tolerances, as relative RMS per row: f32 models 5e-5 (rounding is around 2e-6; a single missed key, tap or
decay is above 1e-3), bfloat16 models 0.08 for any row and 0.025 on average over rows (measured: 0.01 to 0.02 on
average; these models are narrow, so single rows scatter).
The bfloat16 attention kernels are also tested alone with one key standing out, where a key that is missed or
wrongly seen changes the output by more than half."""
import json
import os
import struct
import subprocess
import sys

import numpy as np
import pytest

import b200nn
import vivezen_ref as R
from b200nn import ops

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {"float32": 5e-5, "bfloat16": 0.08}
YARN = {"factor": 4.0, "fast": 8.0, "slow": 0.5, "original": 64}


def latent(heads, dim, rot, vdim, q_rank, kv_rank, window, base=3000.0, scaling=YARN, scale=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
         "rot": {"base": base, "dims": rot, **({"scaling": scaling} if scaling else {})}, "scale": scale or (dim + rot) ** -0.5}
    if window:
        m["mask"] = {"size": window}
    return {"type": "latent_attention", "mixer": m}


def delta(heads, kv_heads, dim, vdim, conv):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def layer(mixer, ff=None, weights_of=None):
    out = dict(mixer, mlp={"kind": "dense", "ff": ff} if ff else None)
    if weights_of is not None:
        out["weights_of"] = weights_of
    return out


def config(width, vocab, layers, eps=1e-5):
    return {"architecture": "Vivezen", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers}


_L1 = latent(3, 24, 8, 40, 36, 20, 37)
_D1 = delta(6, 2, 24, 20, 4)
_L2 = latent(5, 96, 32, 112, 72, 136, 150, base=700.0, scaling=None)
_D2 = delta(4, 1, 80, 144, 2)
CONFIGS = {
    # grouped query/key heads, feed-forward on either kind of mixer or on none, shared weights
    "small": config(90, 203, [layer(_D1, 70), layer(_L1), layer(_D1), layer(_L1, 54), layer(_D1, 70, 0), layer(_L1, None, 1),
                              layer(_L1, 54, 3)]),
    # sizes of the tensor-core attention with two value boxes, no frequency scaling, another window
    "wide": config(160, 331, [layer(_L2, 200), layer(_D2), layer(_L2), layer(_L1, 40)], eps=1e-3),
    # one mixer each, no feed-forward
    "delta": config(64, 101, [layer(delta(4, 4, 64, 48, 3))]),
    "delta_taps1": config(40, 67, [layer(delta(3, 1, 16, 36, 1), 33)]),
    "latent": config(72, 130, [layer(latent(2, 64, 16, 64, 48, 80, 21))]),
    "latent_window1": config(48, 61, [layer(latent(4, 20, 12, 28, 18, 30, 1), 21)]),
    "latent_full": config(48, 61, [layer(latent(2, 40, 64, 72, 24, 48, None))]),
    "big_heads": config(96, 77, [layer(latent(2, 144, 80, 160, 40, 70, 29)), layer(delta(2, 1, 136, 168, 5))]),
}
_models: dict = {}


def weights(name):
    if ("w", name) not in _models:
        _models["w", name] = R.random_weights(CONFIGS[name], sum(map(ord, name)))
    return _models["w", name]


def model(reg, name, dtype):
    if (name, dtype) not in _models:
        _models[name, dtype] = b200nn.LanguageModel.from_weights(CONFIGS[name], weights(name), reg, dtype)
    return _models[name, dtype]


def tokens(name, n, seed=0):
    return np.random.default_rng(seed + 11 * n).integers(0, CONFIGS[name]["vocab"], n).tolist()


def reference(name, toks):
    key = ("r", name, tuple(toks))
    if key not in _models:
        _models[key] = R.forward(CONFIGS[name], weights(name), toks)
    return _models[key]


def check(got, want, tol, what=""):
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    err = np.sqrt(((got - want) ** 2).mean(-1) / (want ** 2).mean())
    assert got.shape == want.shape and np.isfinite(got).all() and err.max() < tol, f"{what}: row {int(err.argmax())}, error {err.max():.2e}"
    assert tol != TOL["bfloat16"] or err.size < 8 or err.mean() < 0.025, f"{what}: mean error {err.mean():.2e}"


def run(rb, name, toks, portions):
    """Feeds toks in the given portions (the last repeats); all logits."""
    out, at, i = [], 0, 0
    while at < len(toks):
        n = portions[min(i, len(portions) - 1)]
        part = toks[at:at + n]
        out.append(rb.step([(name, part, range(len(part)))]))
        at, i = at + n, i + 1
    return np.concatenate(out)


# ---- whole models --------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompt(reg, name, dtype):
    for n in (1, 2, 47, 290):
        t = tokens(name, n)
        rb = b200nn.RequestBatch(model(reg, name, dtype), 1, 300)
        check(run(rb, "a", t, [n]), reference(name, t), TOL[dtype], f"{name} {n} tokens")
    assert reg.device_error() == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["small", "wide", "delta_taps1", "latent_full", "big_heads"])
@pytest.mark.parametrize("portions", [[1], [2], [5, 2, 3, 1, 7], [36, 2, 37, 38, 1], [150, 1, 1, 2, 99]])
def test_portions(reg, name, dtype, portions):
    """The logits do not depend on the cut; portions of one token take the decoding kernels."""
    t = tokens(name, 290)
    rb = b200nn.RequestBatch(model(reg, name, dtype), 1, 290)
    check(run(rb, "a", t, portions), reference(name, t), TOL[dtype], f"{name} {portions}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_unequal_requests_in_one_step(reg, dtype):
    """Requests of different lengths, joining and leaving at different steps, prompts and single tokens mixed:
    each as if alone."""
    name = "small"
    rng = np.random.default_rng(5)
    reqs = {k: tokens(name, n, k) for k, n in enumerate((130, 1, 64, 290, 17, 99, 2))}
    rb = b200nn.RequestBatch(model(reg, name, dtype), 4, 290)
    got = {k: [] for k in reqs}
    at, live, waiting = dict.fromkeys(reqs, 0), [], list(reqs)
    while live or waiting:
        while waiting and len(live) < 4:
            live.append(waiting.pop(0))
        part = [k for k in live if rng.random() < 0.8] or live[:1]
        rng.shuffle(part)
        entries = []
        for k in part:
            n = int(rng.choice([1, 1, 2, 9, 40]))
            seg = reqs[k][at[k]:at[k] + n]
            entries.append((k, seg, range(len(seg))))
        lg = rb.step(entries)
        for k, seg, _ in entries:
            got[k].append(lg[:len(seg)])
            lg = lg[len(seg):]
            at[k] += len(seg)
            if at[k] == len(reqs[k]):
                rb.end(k)
                live.remove(k)
    for k, t in reqs.items():
        check(np.concatenate(got[k]), reference(name, t), TOL[dtype], f"request {k}")
    assert len(rb) == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_decode_only_steps_of_several_requests(reg, dtype):
    name = "wide"
    reqs = {k: tokens(name, 60 + 5 * k, k) for k in range(5)}
    rb = b200nn.RequestBatch(model(reg, name, dtype), 6, 120)
    rb.step([(k, t[:20 + 7 * k], []) for k, t in reqs.items()])
    got = {k: [] for k in reqs}
    for i in range(20):
        order = list(reqs)[i % 5:] + list(reqs)[:i % 5]
        lg = rb.step([(k, [reqs[k][20 + 7 * k + i]], [0]) for k in order])
        for k, row in zip(order, lg):
            got[k].append(row)
    for k, t in reqs.items():
        a = 20 + 7 * k
        check(np.stack(got[k]), reference(name, t[:a + 20])[a:], TOL[dtype], f"request {k}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_slots_are_used_again(reg, dtype):
    """A slot that held another sequence shows nothing of it: not its keys, state or convolution inputs."""
    for name in ("small", "wide"):
        rb = b200nn.RequestBatch(model(reg, name, dtype), 2, 290)
        run(rb, "old", tokens(name, 290, 3), [100])
        run(rb, "other", tokens(name, 50, 4), [50])
        for i, portions in enumerate(([1], [2, 1], [64])):
            old = rb.slot("old")
            rb.end("old")
            t = tokens(name, 41 + i, 50 + i)
            got = run(rb, "old", t, portions)
            assert rb.slot("old") == old
            check(got, reference(name, t), TOL[dtype], f"{name} reuse {i}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_ring_wraps_under_long_sequences(reg, dtype):
    """A windowed layer keeps its window plus one portion: with short portions the ring (128 or 256 rows here)
    is overwritten several times."""
    reg.set_tuning("lm_portion", 24)
    try:
        for name in ("small", "latent", "wide"):
            t = tokens(name, 700)
            rb = b200nn.RequestBatch(model(reg, name, dtype), 2, 720)
            rb.step([("pad", t[:3], [])])  # the sequence under test is not in slot 0
            got = run(rb, "a", t, [101, 24, 25, 1, 1, 1, 60, 2, 23])
            check(got, reference(name, t), TOL[dtype], name)
            for tok, row in zip(tokens(name, 18, 9), range(18)):
                check(rb.step([("a", [tok], [0])])[0], R_tail(name, t, tokens(name, 18, 9)[:row + 1]), TOL[dtype], f"{name} decoded {row}")
                if row == 3:
                    break
    finally:
        reg.set_tuning("lm_portion", 0)


def R_tail(name, t, more):
    return R.forward(CONFIGS[name], weights(name), t + more)[-1]


def test_long_decoding(reg):
    """Hundreds of single-token steps: the state neither drifts nor leaks."""
    name = "small"
    t = tokens(name, 420, 2)
    rb = b200nn.RequestBatch(model(reg, name, "float32"), 1, 420)
    check(run(rb, "a", t, [3, 1]), reference(name, t), 2e-4)


# ---- generation ----------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name,plen,new", [("small", 5, 60), ("small", 60, 20), ("wide", 1, 30), ("delta", 9, 12), ("latent", 33, 12)])
def test_greedy_generation(reg, name, plen, new, dtype):
    """generate_batch (prefill, captured decode steps, greedy pick on the device) against the recomputing
    reference; tokens may differ only where the reference's best two logits are as close as the rounding."""
    m = model(reg, name, dtype)
    prompts = np.array([tokens(name, plen, 100 + b) for b in range(3)], dtype=np.uint32)
    out, lens = m.generate_batch(prompts, new)
    assert (lens == plen + new).all() and (out[:, :plen] == prompts).all()
    for b in range(3):
        lg = R.forward(CONFIGS[name], weights(name), out[b, :-1])[plen - 1:]
        scale = np.sqrt((lg ** 2).mean())
        for i, row in enumerate(lg):
            best, tok = row.max(), out[b, plen + i]
            assert best - row[tok] <= (4 * TOL[dtype]) * scale, f"sequence {b} token {i}: {tok} is not the best"
    if dtype == "float32":
        ref, _ = R.greedy(CONFIGS[name], weights(name), prompts[0].tolist(), min(new, 12))
        assert out[0, :len(ref)].tolist() == ref


def test_generation_with_a_split_prompt_and_many_sequences(reg):
    """Prompts longer than a pass takes go through in portions; the result is that of one pass."""
    m = model(reg, "small", "float32")
    prompts = np.array([tokens("small", 100, b) for b in range(5)], dtype=np.uint32)
    whole, _ = m.generate_batch(prompts, 10)
    reg.set_tuning("lm_portion", 30)
    try:
        parts, _ = m.generate_batch(prompts, 10)
    finally:
        reg.set_tuning("lm_portion", 0)
    assert (whole == parts).all()
    for b in (0, 4):
        alone, _ = m.generate_batch(prompts[b:b + 1], 10)
        assert (alone[0] == whole[b]).all()


def test_sessions_and_sampling(reg):
    m = model(reg, "wide", "float32")
    p = tokens("wide", 25)
    greedy = m.generate(p, 8)
    assert m.generate_sampling(p, 8, 1, 1.0, b200nn.SimpleRng(3)).tolist() == greedy.tolist()
    s = b200nn.DecodeSession(m, 2, 40)
    s.prefill(np.array([p, p], dtype=np.uint32))
    s.step(7)
    assert (s.tokens() == greedy[25:]).all()
    check(s.logits()[0], reference("wide", greedy[:-1].tolist())[-1], TOL["float32"])
    fam, _ = s.profile_step()
    assert fam["recurrence"] > 0 and fam["attention"] > 0
    # seeded sampling stays inside the top k of the reference's logits
    out = m.generate_sampling(p, 8, 5, 1.0, b200nn.SimpleRng(8)).tolist()
    lg = reference("wide", out[:-1])
    for i in range(8):
        assert out[25 + i] in np.argsort(-lg[24 + i])[:6]


# ---- mechanisms alone ------------------------------------------------------------------------------
def _bf(a):
    import torch
    return torch.tensor(np.asarray(a, np.float32), device="cuda").to(torch.bfloat16)


def _dev(a, dt=None):
    import torch
    return torch.tensor(np.ascontiguousarray(a), device="cuda", dtype=dt or torch.float32)


def _ints(*rows):
    import torch
    return torch.tensor(np.concatenate([np.asarray(r) for r in rows]), device="cuda", dtype=torch.int32)


@pytest.mark.parametrize("shape", [(2, 64, 32, 48, 112, 75), (3, 128, 64, 128, 192, 300), (2, 48, 32, 80, 64, 128), (1, 112, 16, 48, 48, 1),
                                   (2, 64, 64, 64, 64, 0), (1, 160, 80, 144, 64, 90)])
@pytest.mark.parametrize("spike", ["inside", "outside", "none"])
def test_latent_prefill_attention(reg, shape, spike):
    """Ragged sequences with cached keys before them.  With a spike, query i of a sequence matches one key far
    above all others: the oldest one it sees, or the one just before that, which must not show."""
    import torch
    H, dim, rot, vdim, rank, window = shape
    rng = np.random.default_rng(sum(shape))
    seqs = [(0, 1), (0, 200), (37, 2), (500, 129), (130, 300)]  # (past, new rows)
    w = window or 100000
    first = [max(0, p - (w - 1)) for p, _ in seqs]
    klen = [p + n - f for (p, n), f in zip(seqs, first)]
    krow0 = np.concatenate([[0], np.cumsum(klen)[:-1]])
    row0 = np.concatenate([[0], np.cumsum([n for _, n in seqs])[:-1]])
    rows, krows = sum(n for _, n in seqs), sum(klen)
    q = R.bf16_round(rng.standard_normal((rows, H, dim + rot)) * 0.5)
    kn = R.bf16_round(rng.standard_normal((krows, H, dim)) * 0.5)
    v = R.bf16_round(rng.standard_normal((krows, H, vdim)))
    lat = R.bf16_round(rng.standard_normal((krows, rank + rot)) * 0.5)
    gate = rng.uniform(0.2, 1.0, (rows, H)).astype(np.float32)
    scale = (dim + rot) ** -0.5
    if spike != "none":
        for s, (p, n) in enumerate(seqs):
            for i in range(0, n, 3):
                a = p + i - (w - 1) - (1 if spike == "outside" else 0) - first[s]  # gathered row of the edge key
                if 0 <= a < klen[s]:
                    q[row0[s] + i, :, :dim] = R.bf16_round(kn[krow0[s] + a] * 12)
    tq, tkv, tlat, tg = _bf(q.reshape(rows, -1)), _bf(np.concatenate([kn.reshape(krows, -1), v.reshape(krows, -1)], 1)), _bf(lat), _dev(gate)
    out = torch.full((rows, H, vdim), 7.0, device="cuda", dtype=torch.bfloat16)
    meta = _ints(row0, [n for _, n in seqs], [p for p, _ in seqs], krow0, first)
    torch.cuda.synchronize()
    ops.latent_prefill_attention((H, dim, rot, vdim, rank, window, scale), tq.data_ptr(), tkv.data_ptr(), tlat.data_ptr(), tg.data_ptr(), rows,
                                 krows, len(seqs), max(n for _, n in seqs), meta.data_ptr(), out.data_ptr(), reg)
    reg.synchronize()
    got = out.float().cpu().numpy()
    for s, (p, n) in enumerate(seqs):
        kk = slice(krow0[s], krow0[s] + klen[s])
        qpos, kpos = p + np.arange(n), first[s] + np.arange(klen[s])
        mask = (qpos[:, None] >= kpos[None]) & (qpos[:, None] - kpos[None] < w)
        for h in range(H):
            k = np.concatenate([kn[kk, h], lat[kk, rank:]], 1).astype(np.float64)
            r = row0[s] + np.arange(n)
            want = R.softmax_attention(q[r, h].astype(np.float64), k, v[kk, h].astype(np.float64), scale, mask) * gate[r, h:h + 1]
            assert np.abs(got[r, h] - want).max() < 0.03, f"sequence {s} head {h}: row {np.abs(got[r, h] - want).max(1).argmax()}"
    assert reg.device_error() == 0


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("shape", [(8, 64, 32, 48, 112, 75), (16, 128, 64, 128, 512, 1000), (3, 48, 32, 80, 64, 128), (40, 64, 16, 32, 256, 1),
                                   (20, 64, 64, 64, 144, 0), (128, 128, 64, 128, 512, 300), (2, 64, 80, 64, 1008, 200)])
@pytest.mark.parametrize("spike", ["inside", "outside", "none"])
def test_latent_decode_attention(reg, shape, spike, dtype):
    """One query per row against a ring of cached latents at many positions, slots permuted."""
    import torch
    H, dim, rot, vdim, rank, window = shape
    rng = np.random.default_rng(sum(shape))
    cap = 1500
    ring = -(-(window + 24 if window else cap) // 128) * 128
    poss = np.array([0, 1, 15, window - 1 if window else 7, window or 900, 127, 128, 129, ring - 1, min(cap - 1, ring + 3), 1023, 1499])
    poss = np.minimum(np.maximum(poss, 0), cap - 1)
    B = len(poss)
    slots = rng.permutation(B + 2)[:B]
    rnd = R.bf16_round if dtype == "bfloat16" else (lambda a: np.asarray(a, np.float32))
    cache = rnd(rng.standard_normal((B + 2, ring, rank + rot)) * 0.6)
    ql = rnd(rng.standard_normal((B, H, rank)) * 0.4)
    q = rnd(rng.standard_normal((B, H, dim + rot)) * 0.4)
    w = window or 100000
    scale = (dim + rot) ** -0.5
    for b, p in enumerate(poss):
        edge = p - (w - 1) - (1 if spike == "outside" else 0)
        if spike != "none" and edge >= 0:
            ql[b] = rnd(cache[slots[b], edge % ring, :rank] * (60.0 / rank ** 0.5))
    mk = _bf if dtype == "bfloat16" else _dev
    tc, tql, tq = mk(cache), mk(ql), mk(q)
    out = torch.full((B, H, rank), 7.0, device="cuda", dtype=tc.dtype)
    tp, ts = _ints(poss), _ints(slots)
    torch.cuda.synchronize()
    ops.latent_decode_attention((H, dim, rot, vdim, rank, window, scale), tq.data_ptr(), tql.data_ptr(), tc.data_ptr(), ring, tp.data_ptr(),
                                ts.data_ptr(), B + 2, B, cap, out.data_ptr(), reg, flags=0 if dtype == "bfloat16" else b200nn.LM_F32)
    reg.synchronize()
    got = out.float().cpu().numpy()
    for b, p in enumerate(poss):
        kp = np.arange(max(0, p - w + 1), p + 1)
        rows = cache[slots[b], kp % ring].astype(np.float64)
        qq = np.concatenate([ql[b], q[b, :, dim:]], 1).astype(np.float64)
        s = qq @ rows.T * scale
        e = np.exp(s - s.max(1, keepdims=True))
        want = (e / e.sum(1, keepdims=True)) @ rows[:, :rank]
        tol = 0.02 if dtype == "bfloat16" else 2e-5
        assert np.abs(got[b] - want).max() < tol, f"row {b} at position {p}: {np.abs(got[b] - want).max()}"
    assert reg.device_error() == 0


@pytest.mark.parametrize("shape", [(4, 2, 32, 48, 4), (2, 2, 128, 128, 3), (3, 1, 64, 16, 1), (1, 1, 96, 208, 2), (2, 1, 176, 32, 6),
                                   (64, 16, 64, 128, 2)])
@pytest.mark.parametrize("cols", [0, 1, 2])
def test_delta_rule(reg, shape, cols):
    reg.set_tuning("delta_cols", cols)
    try:
        delta_rule_case(reg, shape)
    finally:
        reg.set_tuning("delta_cols", 0)


def delta_rule_case(reg, shape):
    """Prompt portions, then single tokens, on ragged sequences; outputs and the states they leave.  Decays from
    instant forgetting to none, so that a state that is lost, doubled or shifted shows."""
    import torch
    H, KH, dim, vdim, taps = shape
    rng = np.random.default_rng(sum(shape))
    eps = 1e-5
    pw = 2 * KH * dim + 2 * H * vdim + 2 * H
    pad = -pw % 4
    cw = 2 * KH * dim + H * vdim
    lens = [1, 2, 5, 33, 100, 257]
    E = len(lens)
    proj = [rng.standard_normal((n + 3, pw)).astype(np.float32) for n in lens]
    conv = rng.standard_normal((cw, taps)).astype(np.float32)
    a_log = np.linspace(-6.0, 3.0, H)
    dt = rng.uniform(-3, 1, H).astype(np.float32)
    norm = rng.uniform(0.5, 1.5, vdim).astype(np.float32)

    def want(p):
        T = len(p)
        p = p.astype(np.float64)
        y = R.silu(R.causal_conv(p[:, :cw], conv.astype(np.float64)))
        q = R.unit_norm(y[:, :KH * dim].reshape(T, KH, dim)) * dim ** -0.5
        k = R.unit_norm(y[:, KH * dim:2 * KH * dim].reshape(T, KH, dim))
        v = y[:, 2 * KH * dim:].reshape(T, H, vdim)
        gate = p[:, cw:cw + H * vdim].reshape(T, H, vdim)
        beta = R.sigmoid(p[:, -2 * H:-H])
        g = np.exp(-np.exp(a_log) * R.softplus(p[:, -H:] + dt))
        o, S = np.zeros((T, H, vdim)), []
        for h in range(H):
            o[:, h], s = R.gated_delta_scan(q[:, h // (H // KH)], k[:, h // (H // KH)], v[:, h], beta[:, h], g[:, h])
            S.append(s)
        return R.rms_norm(o, norm.astype(np.float64), eps) * R.silu(gate), np.stack(S)

    slots = rng.permutation(E + 1)[:E]
    cs = torch.full((E + 1, taps, cw), float("nan"), device="cuda")
    st = torch.full((E + 1, H, dim, vdim), float("nan"), device="cuda")
    wt = [_dev(conv.T), _dev(np.exp(a_log)), _dev(dt), _dev(norm)]
    ptrs = tuple(t.data_ptr() for t in wt)
    got = [[] for _ in lens]
    at = [0] * E
    for cut in (0.4, 1.0):  # two portions
        part = [(i, at[i], max(at[i], int(np.ceil(n * cut)))) for i, n in enumerate(lens)]
        part = [(i, a, b) for i, a, b in part if b > a]
        rows = np.pad(np.concatenate([proj[i][a:b] for i, a, b in part]), ((0, 0), (0, pad)))
        pos = np.concatenate([np.arange(a, b) for _, a, b in part])
        sl = np.concatenate([np.full(b - a, slots[i]) for i, a, b in part])
        n = [b - a for _, a, b in part]
        row0 = np.concatenate([[0], np.cumsum(n)[:-1]])
        meta = _ints([slots[i] for i, _, _ in part], row0, n, [a for _, a, _ in part], np.repeat(np.arange(len(part)), n))
        tp, tpos, tsl = _dev(rows), _ints(pos), _ints(sl)
        out = torch.zeros((len(rows), H, vdim), device="cuda")
        scratch = torch.empty(len(rows) * (cw + 2 * H + KH + 4 + H * vdim), device="cuda")
        torch.cuda.synchronize()
        ops.delta_rule((H, KH, dim, vdim, taps, eps), ptrs, tp.data_ptr(), cs.data_ptr(), st.data_ptr(), tpos.data_ptr(), tsl.data_ptr(), len(rows),
                       out.data_ptr(), reg, len(part), max(n), meta.data_ptr(), scratch.data_ptr(), flags=b200nn.LM_F32)
        reg.synchronize()
        o = out.cpu().numpy()
        for (i, a, b), r in zip(part, row0):
            got[i].append(o[r:r + b - a])
            at[i] = b
    for step in range(3):
        tp, tpos, tsl = _dev(np.pad(np.stack([proj[i][lens[i] + step] for i in range(E)]), ((0, 0), (0, pad)))), _ints([n + step for n in lens]), _ints(slots)
        out = torch.zeros((E, H, vdim), device="cuda")
        torch.cuda.synchronize()
        ops.delta_rule((H, KH, dim, vdim, taps, eps), ptrs, tp.data_ptr(), cs.data_ptr(), st.data_ptr(), tpos.data_ptr(), tsl.data_ptr(), E,
                       out.data_ptr(), reg, flags=b200nn.LM_F32)
        reg.synchronize()
        for i, row in enumerate(out.cpu().numpy()):
            got[i].append(row[None])
    state = st.cpu().numpy()
    for i in range(E):
        o, S = want(proj[i])
        check(np.concatenate(got[i]).reshape(len(o), -1), o.reshape(len(o), -1), 3e-5, f"sequence {i}")
        check(state[slots[i]].reshape(H, -1), S.reshape(H, -1), 3e-5, f"state {i}")


# ---- checkpoints, configuration, command line -----------------------------------------------------------
def write_checkpoint(path, cfg, w):
    """config.json and a BF16 model.safetensors."""
    os.makedirs(path, exist_ok=True)
    json.dump(cfg, open(os.path.join(path, "config.json"), "w"))
    head, blobs, at = {}, [], 0
    for n, a in w.items():
        raw = (np.ascontiguousarray(a, np.float32).view(np.uint32) >> 16).astype(np.uint16).tobytes()
        head[n] = {"dtype": "BF16", "shape": list(a.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    h = json.dumps(head).encode()
    open(os.path.join(path, "model.safetensors"), "wb").write(struct.pack("<Q", len(h)) + h + b"".join(blobs))


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_runner(reg, tmp_path, dtype):
    name = "small"
    write_checkpoint(str(tmp_path / "m"), CONFIGS[name], weights(name))
    a, b = tokens(name, 40), tokens(name, 9, 7)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:30], "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": a[30:33], "want": []}, {"id": "y", "tokens": b[:4], "want": [3]}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": a[33:], "want": [6]}], "end": ["x"]},
             {"step": 3, "entries": [{"id": "y", "tokens": b[4:], "want": [4, 0]}], "end": ["y"]}]
    out = tmp_path / "out"
    out.mkdir()
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(out),
                        "--max-tokens", "60"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.split("\n") if x.startswith("done")] == [f"done {i}" for i in range(4)]
    ra, rb_ = reference(name, a), reference(name, b)
    for i, want in ((0, ra[[0, 29]]), (1, rb_[[3]]), (2, ra[[39]]), (3, rb_[[8, 4]])):
        check(np.fromfile(out / f"{i}.f32", "<f4").reshape(-1, CONFIGS[name]["vocab"]), want, TOL[dtype], f"step {i}")


def test_bad_configurations_are_refused(reg):
    w = weights("small")
    L = b200nn.LanguageModel

    def refuse(mutate, code, drop=None):
        cfg = json.loads(json.dumps(CONFIGS["small"]))
        mutate(cfg)
        ww = {k: v for k, v in w.items() if k != drop}
        with pytest.raises(b200nn.NnError) as e:
            L.from_weights(cfg, ww, reg)
        assert e.value.code == code

    refuse(lambda c: c.update(architecture="Nothing"), b200nn.ERR_UNSUPPORTED)
    refuse(lambda c: c["layers"][0].update(type="other"), b200nn.ERR_UNSUPPORTED)
    refuse(lambda c: c["layers"][0]["mixer"].pop("conv"), b200nn.ERR_UNSUPPORTED)
    refuse(lambda c: c["layers"][4].update(weights_of=6), b200nn.ERR_UNSUPPORTED)
    refuse(lambda c: c["layers"][4].update(weights_of=1), b200nn.ERR_SHAPE)
    refuse(lambda c: c.update(vocab=204), b200nn.ERR_SHAPE)
    refuse(lambda c: None, b200nn.ERR_MISSING, drop="l1.mix.uk")
    refuse(lambda c: None, b200nn.ERR_MISSING, drop="l0.mix.q.conv")


def test_serving_step_refuses_bad_calls(reg):
    rb = b200nn.RequestBatch(model(reg, "delta", "float32"), 1, 8)
    with pytest.raises(b200nn.NnError):
        rb.step([("a", [101], [])])  # not a token
    with pytest.raises(b200nn.NnError):
        rb.step([("a", [1] * 9, [])])  # more than the cache holds
    with pytest.raises(b200nn.NnError):
        rb.step([("b", [1], [])])  # no slot left
    t = tokens("delta", 8)
    check(run(rb, "a", t, [8]), reference("delta", t), TOL["float32"])


def test_gpt2_through_the_same_serving_step(reg):
    """The registry's other family: unequal GPT-2 requests in one cache, each as its own forward pass."""
    from b200nn import Gpt2Config, Gpt2Model, synth
    cfg = Gpt2Config(n_layer=2, n_embd=128, n_head=2, vocab_size=97, n_positions=64)
    m = Gpt2Model.from_weights(synth.gpt2_weights(cfg, base_seed=4, std=0.08, random_ln=True), cfg, reg)
    reqs = {k: np.random.default_rng(n).integers(0, 97, n).tolist() for k, n in (("a", 30), ("b", 12), ("c", 51))}
    rb = b200nn.RequestBatch(m, 3, 64)
    got = {k: [] for k in reqs}
    at = dict.fromkeys(reqs, 0)
    for n in (5, 1, 1, 9, 40):
        entries = [(k, t[at[k]:at[k] + n], range(len(t[at[k]:at[k] + n]))) for k, t in reqs.items() if at[k] < len(t)]
        lg = rb.step(entries)
        for k, seg, _ in entries:
            got[k].append(lg[:len(seg)])
            lg = lg[len(seg):]
            at[k] += len(seg)
    for k, t in reqs.items():
        check(np.concatenate(got[k]), m.forward(t).to_host()[:sum(map(len, got[k]))], 3e-3, k)
