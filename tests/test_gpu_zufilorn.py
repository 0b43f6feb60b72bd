"""GPU parity tests of the Zufilorn decoder against the plain float64 statement in zufilorn_ref.py: each mechanism alone,
whole models, portions, batches, reused slots, decoding and generation.

Tolerances, as relative RMS per row: f32 models 1e-4 (rounding is a few 1e-6; a single missed key, tap, decay or stream
is above 1e-3), bfloat16 models 0.1 for any row and 0.03 on average over rows (these models are narrow, so single rows
scatter).  The attention kernels are also tested alone with one key standing out, where a key that is missed or wrongly
seen changes the output by more than half."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import b200nn
import zufilorn_ref as R
from b200nn import ops
from test_gpu_vivezen import _bf, _dev, _ints, write_checkpoint

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {"float32": 1e-4, "bfloat16": 0.1}
MEAN_TOL = {"float32": 2e-5, "bfloat16": 0.03}


def attention(heads, kv_heads, dim, vdim, every=7, coef=0.4, cap=6.0, diff=0.3, scale=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5,
                                           "softcap": cap, "q_temp": {"coef": coef, "every": every}, "diff": diff}}


def delta(heads, kv_heads, dim, vdim, conv):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def mlstm(heads, dim, vdim, cap=5.0):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}


def layer(mixer, ff=None):
    return dict(mixer, mlp={"kind": "dense", "ff": ff} if ff else None)


def config(width, vocab, streams, layers, eps=1e-5, positions=800):
    return {"architecture": "Zufilorn", "width": width, "vocab": vocab, "streams": streams, "max_positions": positions, "norm": {"eps": eps},
            "layers": layers}


CONFIGS = {
    # grouped heads, every mixer with and without feed-forward
    "small": config(90, 203, 2, [layer(delta(6, 2, 24, 20, 4), 70), layer(attention(6, 2, 24, 40)), layer(mlstm(3, 24, 20), 54),
                                 layer(attention(2, 2, 20, 24, every=50, coef=1.0, cap=30.0, diff=0.8), 33), layer(mlstm(2, 40, 24)),
                                 layer(delta(2, 2, 16, 52, 3))]),
    # head sizes of two 64-column boxes, three streams, another epsilon
    "wide": config(160, 331, 3, [layer(attention(4, 1, 96, 112, cap=15.0), 200), layer(mlstm(4, 80, 144, cap=12.0)), layer(delta(4, 1, 80, 144, 2)),
                                 layer(attention(2, 1, 64, 128, every=100), 40)], eps=1e-3),
    # one mixer each
    "delta": config(64, 101, 2, [layer(delta(4, 4, 64, 48, 3))]),
    "delta_taps1": config(40, 67, 1, [layer(delta(3, 1, 16, 36, 1), 33)]),
    "mlstm": config(72, 130, 4, [layer(mlstm(2, 64, 16, cap=20.0), 50)]),
    "attention": config(48, 61, 2, [layer(attention(3, 3, 48, 64, every=1))]),
    "attention_one_head": config(48, 61, 5, [layer(attention(1, 1, 36, 28, coef=0.0, diff=0.1), 21)]),
    # many query heads on one key / value head; sizes beyond the tensor-core kernels
    "group": config(96, 77, 2, [layer(attention(12, 1, 16, 32)), layer(attention(20, 1, 16, 16), 31)]),
    "big_heads": config(96, 77, 2, [layer(attention(2, 1, 144, 160)), layer(delta(2, 1, 136, 168, 5)), layer(mlstm(1, 200, 264))]),
}
RANKS = {"small": (20, 12), "wide": (9, 33), "delta_taps1": (1, 5)}
_models: dict = {}


def weights(name):
    if ("w", name) not in _models:
        _models["w", name] = R.random_weights(CONFIGS[name], sum(map(ord, name)), RANKS.get(name, (24, 24)))
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


def errors(got, want):
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    assert got.shape == want.shape and np.isfinite(got).all()
    return np.sqrt(((got - want) ** 2).mean(-1) / (want ** 2).mean())


def check(got, want, dtype, what="", factor=1.0):
    err = errors(got, want)
    assert err.max() < factor * TOL[dtype], f"{what}: row {int(err.argmax())}, error {err.max():.2e}"
    assert err.size < 8 or err.mean() < factor * MEAN_TOL[dtype], f"{what}: mean error {err.mean():.2e}"


def run(rb, name, toks, portions):
    """Feeds toks in the given portions (the last repeats); all logits."""
    out, at, i = [], 0, 0
    while at < len(toks):
        part = toks[at:at + portions[min(i, len(portions) - 1)]]
        out.append(rb.step([(name, part, range(len(part)))]))
        at, i = at + len(part), i + 1
    return np.concatenate(out)


# ---- whole models --------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompt(reg, name, dtype):
    for n in (1, 2, 47, 290):
        t = tokens(name, n)
        rb = b200nn.RequestBatch(model(reg, name, dtype), 1, 300)
        check(run(rb, "a", t, [n]), reference(name, t), dtype, f"{name} {n} tokens")
    assert reg.device_error() == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["small", "wide", "mlstm", "group", "big_heads"])
@pytest.mark.parametrize("portions", [[1], [2], [5, 2, 3, 1, 7], [127, 2, 128, 1, 32], [150, 1, 1, 2, 99]])
def test_portions(reg, name, dtype, portions):
    """The logits do not depend on the cut; portions of one token take the decoding kernels."""
    t = tokens(name, 290)
    rb = b200nn.RequestBatch(model(reg, name, dtype), 1, 290)
    check(run(rb, "a", t, portions), reference(name, t), dtype, f"{name} {portions}")
    assert reg.device_error() == 0


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
        check(np.concatenate(got[k]), reference(name, t), dtype, f"request {k}")
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
        check(np.stack(got[k]), reference(name, t[:a + 20])[a:], dtype, f"request {k}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_slots_are_used_again(reg, dtype):
    """A slot that held another sequence shows nothing of it: not its keys, states or convolution inputs."""
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
            check(got, reference(name, t), dtype, f"{name} reuse {i}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_passes_of_a_long_portion(reg, dtype):
    """A portion longer than a pass takes goes through in several."""
    reg.set_tuning("lm_portion", 24)
    try:
        for name in ("small", "wide"):
            t = tokens(name, 400)
            rb = b200nn.RequestBatch(model(reg, name, dtype), 2, 420)
            rb.step([("pad", t[:3], [])])  # the sequence under test is not in slot 0
            check(run(rb, "a", t, [101, 24, 25, 1, 1, 1, 60, 2, 185]), reference(name, t), dtype, name)
    finally:
        reg.set_tuning("lm_portion", 0)


def test_long_decoding(reg):
    """Hundreds of single-token steps: the states neither drift nor leak."""
    name = "small"
    t = tokens(name, 520, 2)
    rb = b200nn.RequestBatch(model(reg, name, "float32"), 1, 520)
    check(run(rb, "a", t, [3, 1]), reference(name, t), "float32", factor=4.0)


def test_positions_end_where_the_table_does(reg):
    m = model(reg, "mlstm", "float32")
    assert m.max_positions == 800
    with pytest.raises(b200nn.NnError):
        b200nn.RequestBatch(m, 1, 801)
    rb = b200nn.RequestBatch(m, 1, 800)
    t = tokens("mlstm", 800)
    check(run(rb, "a", t, [797, 2, 1])[-3:], reference("mlstm", t)[-3:], "float32", factor=4.0)
    with pytest.raises(b200nn.NnError):
        rb.step([("a", [1], [0])])


# ---- generation ----------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name,plen,new", [("small", 5, 60), ("small", 60, 20), ("wide", 1, 30), ("delta", 9, 12), ("attention", 126, 12),
                                           ("mlstm", 33, 12)])
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
        ref = R.greedy(CONFIGS[name], weights(name), prompts[0].tolist(), min(new, 12))
        assert out[0, :len(ref)].tolist() == ref


def test_generation_with_a_split_prompt_and_many_sequences(reg):
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
    check(s.logits()[:1], reference("wide", greedy[:-1].tolist())[-1:], "float32")
    fam, _ = s.profile_step()
    assert fam["recurrence"] > 0 and fam["attention"] > 0
    out = m.generate_sampling(p, 8, 5, 1.0, b200nn.SimpleRng(8)).tolist()
    lg = reference("wide", out[:-1])
    for i in range(8):
        assert out[25 + i] in np.argsort(-lg[24 + i])[:6]


# ---- mechanisms alone ------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rows", [7, 200])  # a decode step's and a prompt's block shapes
@pytest.mark.parametrize("n,width", [(1, 24), (2, 90), (3, 1500), (4, 2052), (5, 64), (8, 4100), (2, 8192)])
def test_stream_step(reg, n, width, rows, dtype):
    import torch
    rng = np.random.default_rng(n + width)
    eps, flags = 1e-4, 0 if dtype == "bfloat16" else b200nn.LM_F32
    x0, y, norm = (rng.standard_normal(s).astype(np.float32) for s in ((rows, width), (rows, width), (width,)))
    c = [{"in": rng.standard_normal(n), "out": rng.standard_normal(n), "mix": rng.standard_normal((n, n))} for _ in range(2)]
    dc = [_dev(np.concatenate([v["in"], v["out"], v["mix"].reshape(-1)])) for v in c]
    xs = torch.full((rows, n, width), float("nan"), device="cuda")
    out = torch.zeros(rows, width, device="cuda", dtype=torch.bfloat16 if dtype == "bfloat16" else torch.float32)
    total = torch.zeros(rows, width, device="cuda")
    tx, ty, tn = _dev(x0), _dev(y), _dev(norm)
    torch.cuda.synchronize()
    p = lambda t: t.data_ptr()
    tol = 1e-2 if dtype == "bfloat16" else 2e-6

    def step(y_, prev, nxt, sum_out):
        ops.stream_step(rows, n, width, p(xs), p(tx), y_, prev, nxt, p(tn), eps, p(out), sum_out, reg, flags=flags)
        reg.synchronize()

    want = np.stack([x0.astype(np.float64)] * n)
    step(None, None, p(dc[0]), None)
    assert errors(out.float().cpu().numpy(), R.rms_norm(R.stream_input(want, c[0]), norm, eps)).max() < tol
    want = R.stream_update(want, y, c[0])
    step(p(ty), p(dc[0]), p(dc[1]), None)
    assert errors(out.float().cpu().numpy(), R.rms_norm(R.stream_input(want, c[1]), norm, eps)).max() < tol
    assert errors(xs.cpu().numpy().transpose(1, 0, 2), want).max() < 2e-6
    step(p(ty), p(dc[1]), None, p(total))
    assert errors(total.cpu().numpy(), R.stream_update(want, y, c[1]).sum(0)).max() < 2e-6


def recurrence_case(reg, lens, proj, call, want, state_of):
    """Prompt portions in two cuts, then three single tokens, on ragged sequences in permuted slots.  proj: per sequence
    [tokens, columns]; call(rows, n_rows, pos, slot, out, n_seq, max_n, seq); want(sequence rows) -> (out [T, .], states)."""
    import torch
    E = len(lens)
    rng = np.random.default_rng(E)
    slots = rng.permutation(E + 1)[:E]
    got, at = [[] for _ in lens], [0] * E
    for cut in (0.4, 1.0):
        part = [(i, at[i], max(at[i], int(np.ceil(n * cut)))) for i, n in enumerate(lens)]
        part = [(i, a, b) for i, a, b in part if b > a]
        rows = [np.concatenate([x[i][a:b] for i, a, b in part]) for x in proj]
        n = [b - a for _, a, b in part]
        row0 = np.concatenate([[0], np.cumsum(n)[:-1]])
        pos, sl = np.concatenate([np.arange(a, b) for _, a, b in part]), np.concatenate([np.full(b - a, slots[i]) for i, a, b in part])
        meta = _ints([slots[i] for i, _, _ in part], row0, n, [a for _, a, _ in part], np.repeat(np.arange(len(part)), n))
        o = call([_dev(r) for r in rows], sum(n), _ints(pos), _ints(sl), len(part), max(n), meta)
        for (i, a, b), r in zip(part, row0):
            got[i].append(o[r:r + b - a])
            at[i] = b
    for step in range(3):
        o = call([_dev(np.stack([x[i][lens[i] + step] for i in range(E)])) for x in proj], E, _ints([n + step for n in lens]), _ints(slots), 0, 0, None)
        for i, row in enumerate(o):
            got[i].append(row[None])
    torch.cuda.synchronize()
    for i in range(E):
        o, states = want([x[i] for x in proj])
        assert errors(np.concatenate(got[i]).reshape(len(o), -1), o.reshape(len(o), -1)).max() < 1e-4, f"sequence {i}"
        for s, t in zip(states, state_of(slots[i])):
            assert errors(t.reshape(1, -1), s.reshape(1, -1)).max() < 3e-5, f"state {i}"


LENS = [1, 2, 5, 33, 100, 257]


@pytest.mark.parametrize("shape", [(4, 2, 32, 48, 4), (2, 2, 128, 128, 3), (3, 1, 64, 16, 1), (1, 1, 96, 208, 2), (2, 1, 176, 32, 6), (32, 16, 64, 128, 2)])
@pytest.mark.parametrize("cols", [0, 1, 2])
def test_channel_delta_rule(reg, shape, cols):
    """Decays from instant forgetting to none, different along the channels."""
    import torch
    H, KH, dim, vdim, taps = shape
    rng = np.random.default_rng(sum(shape))
    eps, cw, E, ext = 1e-5, 2 * KH * dim + H * vdim, len(LENS), H * max(dim, vdim)
    pw = -(-(cw + H) // 16) * 16
    proj = [rng.standard_normal((n + 3, pw)).astype(np.float32) for n in LENS]
    exts = [rng.standard_normal((n + 3, 2 * ext)).astype(np.float32) for n in LENS]
    conv = rng.standard_normal((cw, taps)).astype(np.float32)
    a_log = np.linspace(-6.0, 3.0, H)
    dt = rng.uniform(-4, 1, H * dim).astype(np.float32)
    norm = rng.uniform(0.5, 1.5, vdim).astype(np.float32)
    cs = torch.full((E + 1, taps, cw), float("nan"), device="cuda")
    st = torch.full((E + 1, H, dim, vdim), float("nan"), device="cuda")
    wt = [_dev(conv.T), _dev(np.exp(a_log)), _dev(dt), _dev(norm)]

    def call(rows, n, pos, slot, n_seq, max_n, seq):
        out = torch.zeros((n, H, vdim), device="cuda")
        scratch = torch.empty(n * (cw + H * vdim + H * dim + H + KH + 4), device="cuda")
        torch.cuda.synchronize()
        ops.channel_delta_rule((H, KH, dim, vdim, taps, eps), tuple(t.data_ptr() for t in wt), rows[0].data_ptr(), rows[1].data_ptr(), cs.data_ptr(),
                               st.data_ptr(), pos.data_ptr(), slot.data_ptr(), n, out.data_ptr(), reg, n_seq, max_n,
                               seq.data_ptr() if seq is not None else None, scratch.data_ptr(), flags=b200nn.LM_F32)
        reg.synchronize()
        return out.cpu().numpy()

    def want(x):
        p, e = x[0].astype(np.float64), x[1].astype(np.float64)
        T = len(p)
        y = R.silu(R.causal_conv(p[:, :cw], conv.astype(np.float64)))
        q = R.unit_norm(y[:, :KH * dim].reshape(T, KH, dim)) * dim ** -0.5
        k = R.unit_norm(y[:, KH * dim:2 * KH * dim].reshape(T, KH, dim))
        v = y[:, 2 * KH * dim:].reshape(T, H, vdim)
        beta = R.sigmoid(p[:, cw:cw + H])
        g = np.exp(-np.exp(a_log)[:, None] * R.softplus(e[:, :H * dim] + dt).reshape(T, H, dim))
        gate = R.sigmoid(e[:, ext:ext + H * vdim]).reshape(T, H, vdim)
        res = [R.channel_delta_scan(q[:, h // (H // KH)], k[:, h // (H // KH)], v[:, h], beta[:, h], g[:, h]) for h in range(H)]
        return R.rms_norm(np.stack([o for o, _ in res], 1), norm.astype(np.float64), eps) * gate, [np.stack([s for _, s in res])]

    reg.set_tuning("delta_cols", cols)
    try:
        recurrence_case(reg, LENS, [proj, exts], call, want, lambda s: [st.cpu().numpy()[s]])
    finally:
        reg.set_tuning("delta_cols", 0)


@pytest.mark.parametrize("shape", [(4, 32, 48, 5.0), (2, 128, 128, 12.0), (3, 64, 16, 1.0), (1, 96, 208, 30.0), (2, 176, 32, 8.0), (2, 256, 272, 8.0),
                                   (32, 64, 128, 15.0)])
@pytest.mark.parametrize("cols", [0, 1, 2])
def test_mlstm(reg, shape, cols):
    """Gates from closed to open on both sides of the cap, so that the running maximum both follows the forget gates down
    and jumps with the input gates, and the read-out's floor is reached."""
    import torch
    H, dim, vdim, cap = shape
    rng = np.random.default_rng(int(sum(shape)))
    eps, E = 1e-5, len(LENS)
    pw = -(-(2 * H * dim + 2 * H * vdim + 2 * H) // 4) * 4
    gi = 2 * H * (dim + vdim)
    proj = [rng.standard_normal((n + 3, pw)).astype(np.float32) for n in LENS]
    for p in proj:
        p[:, gi:gi + 2 * H] *= 2.0
        p[rng.random(len(p)) < 0.05, gi:gi + H] += 8.0
    ib, fb = np.linspace(-3.0, 2.0, H).astype(np.float32), np.linspace(-1.0, 7.0, H).astype(np.float32)
    norm = rng.uniform(0.5, 1.5, (H, vdim)).astype(np.float32)
    mem = torch.full((E + 1, H, dim, vdim), float("nan"), device="cuda")
    nrm, mx = torch.full((E + 1, H, dim), float("nan"), device="cuda"), torch.full((E + 1, H), float("nan"), device="cuda")
    wt = [_dev(ib), _dev(fb), _dev(norm)]

    def call(rows, n, pos, slot, n_seq, max_n, seq):
        out = torch.zeros((n, H, vdim), device="cuda")
        scratch = torch.empty(n * H * (vdim + 4), device="cuda")
        torch.cuda.synchronize()
        ops.mlstm((H, dim, vdim, cap, eps), tuple(t.data_ptr() for t in wt), rows[0].data_ptr(), mem.data_ptr(), nrm.data_ptr(), mx.data_ptr(),
                  pos.data_ptr(), slot.data_ptr(), n, out.data_ptr(), reg, n_seq, seq.data_ptr() if seq is not None else None, scratch.data_ptr(),
                  flags=b200nn.LM_F32)
        reg.synchronize()
        return out.cpu().numpy()

    def want(x):
        p = x[0].astype(np.float64)
        T, at = len(p), np.cumsum([0, H * dim, H * dim, H * vdim, H * vdim, H, H])
        q, k, v, g, i, f = (p[:, a:b] for a, b in zip(at[:-1], at[1:]))
        i, f = R.soft_cap(i + ib, cap), R.log_sigmoid(R.soft_cap(f + fb, cap))
        q, k, v = q.reshape(T, H, dim) * dim ** -0.5, k.reshape(T, H, dim), v.reshape(T, H, vdim)
        res = [R.mlstm_scan(q[:, h], k[:, h], v[:, h], i[:, h], f[:, h]) for h in range(H)]
        o = R.rms_norm(np.stack([o for o, _ in res], 1), norm.astype(np.float64), eps) * R.sigmoid(g).reshape(T, H, vdim)
        return o, [np.stack([s[j] for _, s in res]) for j in range(3)]

    reg.set_tuning("delta_cols", cols)
    try:
        recurrence_case(reg, LENS, [proj], call, want, lambda s: [t.cpu().numpy()[s] for t in (mem, nrm, mx)])
    finally:
        reg.set_tuning("delta_cols", 0)


DIFF_SHAPES = [(6, 2, 32, 48, 0.35, 45.0), (2, 1, 64, 128, 0.5, 9.0), (3, 3, 128, 48, 0.0, 20.0), (2, 2, 96, 128, 0.7, 0.0), (12, 1, 48, 112, 0.3, 30.0),
               (20, 1, 16, 32, 0.2, 5.0), (2, 2, 160, 96, 0.4, 25.0), (4, 2, 64, 160, 0.6, 40.0)]


def diff_expected(shape, q, rows, pos, gate, lam, every, scale):
    """One query [H, 2, dim] at position pos over the cache rows [G, pos + 1, 2 dim + vdim]."""
    H, G, dim, vdim, coef, cap = shape[:6]
    t = float(R.query_temperature([pos], {"coef": coef, "every": every})[0])
    out = np.zeros((H, vdim))
    for h in range(H):
        r = rows[h // (H // G)].astype(np.float64)
        a = [R.capped_attention(q[h, m][None].astype(np.float64) * t, r[:, m * dim:(m + 1) * dim], r[:, 2 * dim:], scale, cap or 1e9, True)
             for m in (0, 1)]
        out[h] = R.combine_maps(a[0], a[1], lam, 0.25, 1e-5)[0] * gate[h]
    return out


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("shape", DIFF_SHAPES)
@pytest.mark.parametrize("spike", ["edges", "next", "none"])
def test_diff_attention_prompt(reg, shape, spike, dtype):
    """Ragged sequences with cached keys before them.  With spikes, rows match one key far above all others in one map or
    the other: the first positions, their own, those at borders of 128, or (next) the one after their own, which must not
    show."""
    import torch
    H, G, dim, vdim, coef, cap = shape
    rng = np.random.default_rng(int(sum(shape)))
    rnd = R.bf16_round if dtype == "bfloat16" else (lambda a: np.asarray(a, np.float32))
    seqs, capacity, every, lam, scale = [(0, 1), (0, 200), (37, 2), (500, 129), (130, 300), (255, 1)], 640, 90, 0.45, dim ** -0.5
    E = len(seqs)
    slots = rng.permutation(E + 1)[:E]
    row0 = np.concatenate([[0], np.cumsum([n for _, n in seqs])[:-1]])
    rows, kw = sum(n for _, n in seqs), 2 * dim + vdim
    q = rnd(rng.standard_normal((rows, H, 2, dim)))
    cache = rnd(rng.standard_normal((E + 1, G, capacity, kw)))
    gate = rng.standard_normal((rows, H)).astype(np.float32)
    if spike != "none":
        for s, (p, n) in enumerate(seqs):
            for i in range(0, n, 3):
                pos, h, m = p + i, int(rng.integers(H)), int(rng.integers(2))
                a = pos + 1 if spike == "next" else int(rng.choice([0, 1, pos, max(pos - 1, 0), pos // 128 * 128, max(pos // 128 * 128 - 1, 0)]))
                q[row0[s] + i, h, m] = rnd(cache[slots[s], h // (H // G), a, m * dim:(m + 1) * dim] * 6)
    mk = _bf if dtype == "bfloat16" else _dev
    tq, tc, tg = mk(q.reshape(rows, -1)), mk(cache), _dev(gate)
    out = torch.full((rows, H, vdim), 7.0, device="cuda", dtype=tq.dtype)
    n = [n for _, n in seqs]
    pos, sl = _ints(np.concatenate([np.arange(p, p + n) for p, n in seqs])), _ints(np.repeat(slots, n))
    meta = _ints(slots, row0, n, [p for p, _ in seqs])
    torch.cuda.synchronize()
    ops.diff_attention((H, G, dim, vdim, every, scale, cap, coef, lam, 0.25, 1e-5), tq.data_ptr(), tc.data_ptr(), capacity, E + 1, pos.data_ptr(),
                       sl.data_ptr(), tg.data_ptr(), rows, out.data_ptr(), reg, E, max(n), meta.data_ptr(),
                       flags=0 if dtype == "bfloat16" else b200nn.LM_F32)
    reg.synchronize()
    got = out.float().cpu().numpy()
    tol = 0.05 if dtype == "bfloat16" else 5e-5
    for s, (p, cnt) in enumerate(seqs):
        for i in sorted({0, 1, 2, 3, 6, 63, 66, 126, 127, 128, 129, 150, 198, 199, 252, 255, 297, 299} & set(range(cnt))):
            r = row0[s] + i
            want = diff_expected(shape, q[r], cache[slots[s]][:, :p + i + 1], p + i, R.sigmoid(gate[r].astype(np.float64)), lam, every, scale)
            err = errors(got[r], want).max()
            assert err < tol, f"sequence {s} row {i}: {err:.2e}"
    assert reg.device_error() == 0


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
@pytest.mark.parametrize("shape", DIFF_SHAPES + [(6, 2, 256, 512, 0.3, 30.0)])
@pytest.mark.parametrize("spike", ["edges", "next", "none"])
def test_diff_attention_decode(reg, shape, spike, dtype):
    """One query per row at many positions, slots permuted; the cache past a row's position holds other values."""
    import torch
    H, G, dim, vdim, coef, cap = shape
    rng = np.random.default_rng(int(sum(shape)))
    rnd = R.bf16_round if dtype == "bfloat16" else (lambda a: np.asarray(a, np.float32))
    poss, capacity, every, lam, scale = np.array([0, 1, 15, 89, 90, 126, 127, 128, 129, 255, 256, 383, 700, 1022, 1023]), 1030, 90, 0.45, dim ** -0.5
    B, kw = len(poss), 2 * dim + vdim
    slots = rng.permutation(B + 2)[:B]
    q = rnd(rng.standard_normal((B, H, 2, dim)))
    cache = rnd(rng.standard_normal((B + 2, G, capacity, kw)))
    gate = rng.standard_normal((B, H)).astype(np.float32)
    if spike != "none":
        for b, pos in enumerate(poss):
            for h in range(H):
                m = int(rng.integers(2))
                a = pos + 1 if spike == "next" else int(rng.choice([0, 1, pos, max(pos - 1, 0), pos // 128 * 128, max(pos // 128 * 128 - 1, 0), pos // 2]))
                q[b, h, m] = rnd(cache[slots[b], h // (H // G), a, m * dim:(m + 1) * dim] * 6)
    mk = _bf if dtype == "bfloat16" else _dev
    tq, tc, tg = mk(q.reshape(B, -1)), mk(cache), _dev(gate)
    out = torch.full((B, H, vdim), 7.0, device="cuda", dtype=tq.dtype)
    tp, ts = _ints(poss), _ints(slots)
    torch.cuda.synchronize()
    ops.diff_attention((H, G, dim, vdim, every, scale, cap, coef, lam, 0.25, 1e-5), tq.data_ptr(), tc.data_ptr(), capacity, B + 2, tp.data_ptr(),
                       ts.data_ptr(), tg.data_ptr(), B, out.data_ptr(), reg, flags=0 if dtype == "bfloat16" else b200nn.LM_F32)
    reg.synchronize()
    got = out.float().cpu().numpy()
    tol = 0.05 if dtype == "bfloat16" else 5e-5
    for b, p in enumerate(poss):
        want = diff_expected(shape, q[b], cache[slots[b]][:, :p + 1], int(p), R.sigmoid(gate[b].astype(np.float64)), lam, every, scale)
        err = errors(got[b], want).max()
        assert err < tol, f"row {b} at position {p}: {err:.2e}"
    assert reg.device_error() == 0


# ---- checkpoints, configuration, command line -----------------------------------------------------------
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
        check(np.fromfile(out / f"{i}.f32", "<f4").reshape(-1, CONFIGS[name]["vocab"]), want, dtype, f"step {i}")


def test_bad_configurations_are_refused(reg):
    w = weights("small")

    def refuse(mutate, code, drop=None):
        cfg = json.loads(json.dumps(CONFIGS["small"]))
        mutate(cfg)
        with pytest.raises(b200nn.NnError) as e:
            b200nn.LanguageModel.from_weights(cfg, {k: v for k, v in w.items() if k != drop}, reg)
        assert e.value.code == code

    mixer = lambda c, i: c["layers"][i]["mixer"]
    refuse(lambda c: c["layers"][0].update(type="other"), b200nn.ERR_UNSUPPORTED)
    refuse(lambda c: c.pop("streams"), b200nn.ERR_UNSUPPORTED)
    refuse(lambda c: c.update(streams=9), b200nn.ERR_UNSUPPORTED)
    refuse(lambda c: c.pop("max_positions"), b200nn.ERR_UNSUPPORTED)
    refuse(lambda c: mixer(c, 1).pop("diff"), b200nn.ERR_UNSUPPORTED)
    refuse(lambda c: mixer(c, 1)["q_temp"].pop("every"), b200nn.ERR_UNSUPPORTED)
    refuse(lambda c: mixer(c, 1).update(kv_heads=4), b200nn.ERR_UNSUPPORTED)
    refuse(lambda c: mixer(c, 2).update(gate_cap=0), b200nn.ERR_UNSUPPORTED)
    refuse(lambda c: mixer(c, 2).update(dim=25), b200nn.ERR_SHAPE)
    refuse(lambda c: c.update(streams=3), b200nn.ERR_SHAPE)
    refuse(lambda c: c.update(max_positions=801), b200nn.ERR_SHAPE)
    for name in ("pos", "head", "l0.hc2.mix", "l0.mix.a1", "l0.mix.g2", "l1.mix.lk2", "l2.mix.f.b"):
        refuse(lambda c: None, b200nn.ERR_MISSING, drop=name)
