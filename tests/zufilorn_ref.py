"""Plain float64 numpy statement of the Zufilorn decoder, one function per mechanism: what the GPU tests compare
with.  Recurrences run token by token, attention is dense; nothing of the library is used.  Element-wise pieces,
convolution and synthetic rounding come from vivezen_ref.py.

A configuration is the dict of config.json; weights are a dict name -> array, Linear weights [out, in].
"""
import math

import numpy as np

from vivezen_ref import bf16_round, causal_conv, rms_norm, sigmoid, silu, softplus, sub, unit_norm, visible  # noqa: F401


def log_sigmoid(z):
    return -np.logaddexp(0.0, -z)


def soft_cap(z, cap):
    return cap * np.tanh(z / cap)


# ---- residual streams ----------------------------------------------------------------------------
def stream_input(xs, w):
    """What a sublayer reads: the weighted sum of the streams xs [streams, T, width]."""
    return np.einsum("s,std->td", w["in"], xs)


def stream_update(xs, y, w):
    """The streams after a sublayer's output y: mixed among themselves (mix is [from, to]), plus y per stream."""
    return np.einsum("st,snd->tnd", w["mix"], xs) + w["out"][:, None, None] * y


# ---- gated delta rule with a decay per key channel -------------------------------------------------
def channel_delta_scan(q, k, v, beta, g, state=None):
    """One head: q, k, g [T, dim], v [T, vdim], beta [T]; returns (o [T, vdim], final state [dim, vdim])."""
    S = np.zeros((q.shape[1], v.shape[1])) if state is None else state.copy()
    o = np.zeros((len(q), v.shape[1]))
    for t in range(len(q)):
        S = g[t][:, None] * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + np.outer(k[t], u)
        o[t] = S.T @ q[t]
    return o, S


def channel_decay(h, w, heads):
    """Decays [T, heads, dim] of a whole sequence."""
    z = softplus((h @ w["a1"].T) @ w["a2"].T + w["dt_bias"]).reshape(len(h), heads, -1)
    return np.exp(-np.exp(w["A_log"])[:, None] * z)


def channel_delta_mixer(h, mx, w, eps):
    T, H, KH, dim, vdim = len(h), mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    q, k, v = (silu(causal_conv(h @ w[n].T, w[n + ".conv"])) for n in ("q", "k", "v"))
    q = unit_norm(q.reshape(T, KH, dim)) * dim ** -0.5
    k = unit_norm(k.reshape(T, KH, dim))
    v = v.reshape(T, H, vdim)
    beta = sigmoid(h @ w["b"].T)
    g = channel_decay(h, w, H)
    o = np.stack([channel_delta_scan(q[:, n // (H // KH)], k[:, n // (H // KH)], v[:, n], beta[:, n], g[:, n])[0] for n in range(H)], 1)
    gate = sigmoid((h @ w["g1"].T) @ w["g2"].T).reshape(T, H, vdim)
    return (rms_norm(o, w["norm"], eps) * gate).reshape(T, -1) @ w["o"].T


# ---- matrix memory with exponential gates ----------------------------------------------------------
def mlstm_scan(q, k, v, i, f, state=None):
    """One head: q, k [T, dim], v [T, vdim], log input gate i and log forget gate f [T]; state (S, n, m).
    Returns (o [T, vdim], state)."""
    S, n, m = (np.zeros((q.shape[1], v.shape[1])), np.zeros(q.shape[1]), 0.0) if state is None else state
    o = np.zeros((len(q), v.shape[1]))
    for t in range(len(q)):
        m_new = max(f[t] + m, i[t])
        keep, write = math.exp(f[t] + m - m_new), math.exp(i[t] - m_new)
        S = keep * S + write * np.outer(k[t], v[t])
        n = keep * n + write * k[t]
        m = m_new
        o[t] = S.T @ q[t] / (max(abs(n @ q[t]), math.exp(-m)) + 1e-6)
    return o, (S, n, m)


def mlstm_gates(h, w, cap):
    """Log input and log forget gates [T, heads]."""
    return soft_cap(h @ w["i"].T + w["i.b"], cap), log_sigmoid(soft_cap(h @ w["f"].T + w["f.b"], cap))


def mlstm_mixer(h, mx, w, eps):
    T, H, dim, vdim = len(h), mx["heads"], mx["dim"], mx["vdim"]
    q = (h @ w["q"].T).reshape(T, H, dim) * dim ** -0.5
    k, v = (h @ w["k"].T).reshape(T, H, dim), (h @ w["v"].T).reshape(T, H, vdim)
    i, f = mlstm_gates(h, w, mx["gate_cap"])
    o = np.stack([mlstm_scan(q[:, n], k[:, n], v[:, n], i[:, n], f[:, n])[0] for n in range(H)], 1)
    return (rms_norm(o, 1.0, eps).reshape(T, -1) * w["norm"] * sigmoid(h @ w["g"].T)) @ w["o"].T


# ---- differential attention ------------------------------------------------------------------------
def query_temperature(positions, spec):
    p = np.asarray(positions, dtype=np.float64)
    return 1.0 + spec["coef"] * np.log(np.floor((p + 1.0) / spec["every"]) + 1.0)


def capped_attention(q, k, v, scale, cap, mask):
    """One map of one head: q, k [T, dim], v [T, vdim]."""
    s = np.where(mask, soft_cap((q @ k.T) * scale, cap), -np.inf)
    p = np.exp(s - s.max(-1, keepdims=True))
    return (p / p.sum(-1, keepdims=True)) @ v


def diff_lambda(w, diff):
    return math.exp(float(w["lq1"] @ w["lk1"])) - math.exp(float(w["lq2"] @ w["lk2"])) + diff


def combine_maps(a1, a2, lam, diff, eps):
    return rms_norm(a1 - lam * a2, 1.0, eps) * (1.0 - diff)


def attention_mixer(h, mx, w, eps):
    T, H, G, dim, vdim = len(h), mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    q = (h @ w["q"].T).reshape(T, H, 2, dim) * query_temperature(np.arange(T), mx["q_temp"])[:, None, None, None]
    k, v = (h @ w["k"].T).reshape(T, G, 2, dim), (h @ w["v"].T).reshape(T, G, vdim)
    lam, mask, gate = diff_lambda(w, mx["diff"]), visible(T, None), sigmoid(h @ w["g"].T)
    o = np.zeros((T, H, vdim))
    for n in range(H):
        g = n // (H // G)
        a1, a2 = (capped_attention(q[:, n, m], k[:, g, m], v[:, g], mx["scale"], mx["softcap"], mask) for m in (0, 1))
        o[:, n] = combine_maps(a1, a2, lam, mx["diff"], eps) * gate[:, n:n + 1]
    return o.reshape(T, -1) @ w["o"].T


def gated_mlp(h, w):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


MIXERS = {"channel_delta": channel_delta_mixer, "mlstm": mlstm_mixer, "attention": attention_mixer}


# ---- the model -----------------------------------------------------------------------------------
def forward(cfg, weights, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence; layers_out (a list) receives the sum of the streams after every layer."""
    w = {n: np.asarray(a, np.float64) for n, a in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens, dtype=np.int64)] + w["pos"][:len(tokens)]
    xs = np.stack([x] * cfg["streams"])
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        sublayers = [("hc1.", "norm1", lambda u: MIXERS[layer["type"]](u, layer["mixer"], sub(w, p + "mix."), eps))]
        if layer.get("mlp"):
            sublayers.append(("hc2.", "norm2", lambda u: gated_mlp(u, sub(w, p + "mlp."))))
        for hc, norm, f in sublayers:
            hw = sub(w, p + hc)
            y = f(rms_norm(stream_input(xs, hw), 1.0 + w[p + norm], eps))
            xs = stream_update(xs, y, hw)
        if layers_out is not None:
            layers_out.append(xs.sum(0))
    return rms_norm(xs.sum(0), 1.0 + w["final.norm"], eps) @ w["head"].T


def greedy(cfg, weights, prompt, max_new):
    """Greedy continuation, the whole sequence recomputed for every token."""
    ids = list(prompt)
    for _ in range(max_new):
        ids.append(int(np.argmax(forward(cfg, weights, ids)[-1])))
    return ids


# ---- synthetic models ----------------------------------------------------------------------------
def tensor_shapes(cfg, ranks=(20, 12)):
    """name -> shape of every tensor; ranks: inner sizes of the two-step decay and gate projections."""
    d, s = cfg["width"], cfg["streams"]
    out = {"embed": (cfg["vocab"], d), "pos": (cfg["max_positions"], d), "final.norm": (d,), "head": (cfg["vocab"], d)}
    for i, layer in enumerate(cfg["layers"]):
        p, mx = f"l{i}.", layer["mixer"]
        m, H, dim, vdim = p + "mix.", mx["heads"], mx["dim"], mx["vdim"]
        out[p + "norm1"] = (d,)
        if layer["type"] == "channel_delta":
            KH, taps = mx["kv_heads"], mx["conv"]
            for n, c in (("q", KH * dim), ("k", KH * dim), ("v", H * vdim)):
                out[m + n], out[m + n + ".conv"] = (c, d), (c, taps)
            out.update({m + "b": (H, d), m + "A_log": (H,), m + "norm": (vdim,), m + "a1": (ranks[0], d), m + "a2": (H * dim, ranks[0]),
                        m + "dt_bias": (H * dim,), m + "g1": (ranks[1], d), m + "g2": (H * vdim, ranks[1])})
        elif layer["type"] == "mlstm":
            out.update({m + "q": (H * dim, d), m + "k": (H * dim, d), m + "v": (H * vdim, d), m + "g": (H * vdim, d), m + "norm": (H * vdim,),
                        m + "i": (H, d), m + "i.b": (H,), m + "f": (H, d), m + "f.b": (H,)})
        else:
            G = mx["kv_heads"]
            out.update({m + "q": (H * 2 * dim, d), m + "k": (G * 2 * dim, d), m + "v": (G * vdim, d), m + "g": (H, d)})
            out.update({m + n: (dim,) for n in ("lq1", "lk1", "lq2", "lk2")})
        out[m + "o"] = (d, H * vdim)
        out.update({p + "hc1.in": (s,), p + "hc1.out": (s,), p + "hc1.mix": (s, s)})
        if layer.get("mlp"):
            ff = layer["mlp"]["ff"]
            out.update({p + "norm2": (d,), p + "mlp.gate": (ff, d), p + "mlp.up": (ff, d), p + "mlp.down": (d, ff),
                        p + "hc2.in": (s,), p + "hc2.out": (s,), p + "hc2.mix": (s, s)})
    return out


def random_weights(cfg, seed, ranks=(20, 12)):
    """bfloat16-valued random weights (as float32): matrices with about unit row gain, decays and gates from
    forgetting within a few tokens to remembering hundreds, streams that differ from one another."""
    rng = np.random.default_rng(seed)
    out = {}
    for n, s in tensor_shapes(cfg, ranks).items():
        leaf = n.split(".", 1)[-1]
        if n.endswith("norm1") or n.endswith("norm2") or n == "final.norm":
            a = 0.2 * rng.standard_normal(s)
        elif n.endswith("norm"):
            a = 1.0 + 0.2 * rng.standard_normal(s)
        elif n.endswith("A_log"):
            a = rng.uniform(-4.0, 0.5, s)
        elif n.endswith("dt_bias"):
            a = rng.uniform(-2.0, 1.0, s)
        elif n.endswith("f.b"):
            a = rng.uniform(1.0, 6.0, s)
        elif n.endswith("i.b"):
            a = rng.uniform(-2.0, 2.0, s)
        elif n.endswith(".conv"):
            a = rng.standard_normal(s) * s[1] ** -0.5
        elif n.rsplit(".", 1)[-1] in ("lq1", "lk1", "lq2", "lk2"):
            a = 0.6 * rng.standard_normal(s) * s[0] ** -0.25
        elif leaf.endswith("hc1.in") or leaf.endswith("hc2.in"):
            a = (1.0 + 0.4 * rng.standard_normal(s)) / s[0] ** 0.5
        elif leaf.endswith(".out"):
            a = 0.7 + 0.4 * rng.standard_normal(s)
        elif leaf.endswith(".mix") and "hc" in leaf:
            a = 0.8 * np.eye(s[0]) + 0.2 * rng.standard_normal(s)
        elif n in ("embed", "pos"):
            a = rng.standard_normal(s) * (1.0 if n == "embed" else 0.5)
        else:
            a = rng.standard_normal(s) * 1.2 * s[1] ** -0.5
        out[n] = bf16_round(a)
    return out
