"""Plain float64 numpy statement of the Vivezen decoder, one function per mechanism: what the GPU tests
compare with.  Token by token where the mechanism is a recurrence, dense where it is not; nothing of the
library is used.

A configuration is the dict of config.json; weights are a dict name -> array, Linear weights [out, in].
"""
import math

import numpy as np


# ---- element-wise and per-row mechanisms ---------------------------------------------------------
def silu(z):
    return z / (1.0 + np.exp(-z))


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def softplus(z):
    return np.logaddexp(0.0, z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rms_norm(x, w, eps):
    """Rows of x over their root mean square (eps inside the root), times w."""
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * w


def unit_norm(x):
    """Rows of x over their Euclidean length (1e-6 inside the root)."""
    return x / np.sqrt((x * x).sum(-1, keepdims=True) + 1e-6)


def causal_conv(x, w, taps_before=None):
    """Per-channel causal convolution over time.  x [T, C], w [C, taps], the last column weighting the
    current token; taps_before [taps-1, C]: the inputs before x (zeros at the start of a sequence)."""
    T, C = x.shape
    taps = w.shape[1]
    before = np.zeros((taps - 1, C)) if taps_before is None else taps_before
    xx = np.concatenate([before, x], 0)
    return sum(xx[j:j + T] * w[:, j] for j in range(taps))


# ---- rotary positions ----------------------------------------------------------------------------
def rotary_frequencies(rot):
    """(frequencies [dims/2], factor of cos and sin) of a 'rot' entry, with its frequency scaling if any."""
    n = rot["dims"]
    base = float(rot["base"])
    f = np.array([base ** (-2.0 * i / n) for i in range(n // 2)])
    s = rot.get("scaling")
    if not s:
        return f, 1.0

    def index_of(turns):  # the (fractional) index whose wave turns this often over the original length
        return n * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(index_of(s["fast"])), 0)
    hi = min(math.ceil(index_of(s["slow"])), n - 1)
    ramp = np.array([min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(n // 2)])
    return f / s["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(s["factor"]) + 1.0


def rotate(x, positions, rot):
    """Rotates the first rot.dims entries of the last axis of x [T, ..., n]: entry i with entry i + dims/2."""
    f, m = rotary_frequencies(rot)
    h = len(f)
    a = np.asarray(positions, dtype=np.float64)[:, None] * f[None, :]
    shape = (len(positions),) + (1,) * (x.ndim - 2) + (h,)
    c, s = (np.cos(a) * m).reshape(shape), (np.sin(a) * m).reshape(shape)
    u, v = x[..., :h], x[..., h:2 * h]
    out = x.copy()
    out[..., :h] = u * c - v * s
    out[..., h:2 * h] = v * c + u * s
    return out


# ---- the two mixers ------------------------------------------------------------------------------
def gated_delta_scan(q, k, v, beta, g, state=None):
    """The recurrence of one head: decay, write by the delta rule, read.  q, k [T, dim], v [T, vdim],
    beta, g [T]; returns (o [T, vdim], final state [dim, vdim])."""
    S = np.zeros((q.shape[1], v.shape[1])) if state is None else state.copy()
    o = np.zeros((len(q), v.shape[1]))
    for t in range(len(q)):
        S *= g[t]
        u = beta[t] * (v[t] - S.T @ k[t])
        S += np.outer(k[t], u)
        o[t] = S.T @ q[t]
    return o, S


def delta_mixer(h, mx, w, eps):
    """h [T, width] of a whole sequence; w: this mixer's tensors without their prefix."""
    T = len(h)
    H, KH, dim, vdim = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    q, k, v = (silu(causal_conv(h @ w[n].T, w[n + ".conv"])) for n in ("q", "k", "v"))
    q = unit_norm(q.reshape(T, KH, dim)) * dim ** -0.5
    k = unit_norm(k.reshape(T, KH, dim))
    v = v.reshape(T, H, vdim)
    beta = sigmoid(h @ w["b"].T)
    g = np.exp(-np.exp(w["A_log"]) * softplus(h @ w["a"].T + w["dt_bias"]))
    o = np.zeros((T, H, vdim))
    for n in range(H):
        kh = n // (H // KH)
        o[:, n], _ = gated_delta_scan(q[:, kh], k[:, kh], v[:, n], beta[:, n], g[:, n])
    o = rms_norm(o, w["norm"], eps) * silu(h @ w["g"].T).reshape(T, H, vdim)
    return o.reshape(T, -1) @ w["o"].T


def visible(T, window):
    """[query, key] mask: the query's own position and the window - 1 before it (None: all before it)."""
    d = np.arange(T)[:, None] - np.arange(T)[None, :]
    return (d >= 0) & (d < (window if window else T))


def softmax_attention(q, k, v, scale, mask):
    """q, k [T, n], v [T, m] of one head."""
    s = np.where(mask, (q @ k.T) * scale, -np.inf)
    p = np.exp(s - s.max(-1, keepdims=True))
    return (p / p.sum(-1, keepdims=True)) @ v


def latent_mixer(h, mx, w, eps):
    """h [T, width] of a whole sequence; w: this mixer's tensors without their prefix."""
    T = len(h)
    H, dim, rd, vdim, R = mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"], mx["kv_rank"]
    rot = dict(mx["rot"], dims=rd)
    pos = np.arange(T)
    q = (rms_norm(h @ w["dq"].T, w["dq.norm"], eps) @ w["uq"].T).reshape(T, H, dim + rd)
    q_rot = rotate(q[..., dim:], pos, rot)
    ckr = h @ w["dkv"].T
    c = rms_norm(ckr[:, :R], w["dkv.norm"], eps)
    k_rot = rotate(ckr[:, R:], pos, rot)
    k = (c @ w["uk"].T).reshape(T, H, dim)
    v = (c @ w["uv"].T).reshape(T, H, vdim)
    gate = sigmoid(h @ w["g"].T)
    mask = visible(T, (mx.get("mask") or {}).get("size"))
    o = np.stack([softmax_attention(np.concatenate([q[:, n, :dim], q_rot[:, n]], -1),
                                    np.concatenate([k[:, n], k_rot], -1), v[:, n], mx["scale"], mask) * gate[:, n:n + 1]
                  for n in range(H)], 1)
    return o.reshape(T, -1) @ w["o"].T


def gated_mlp(h, w):
    return (gelu_tanh(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


MIXERS = {"delta": delta_mixer, "latent_attention": latent_mixer}


# ---- the model -----------------------------------------------------------------------------------
def sub(w, prefix):
    return {n[len(prefix):]: np.asarray(a, np.float64) for n, a in w.items() if n.startswith(prefix)}


def forward(cfg, weights, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence; layers_out (a list) receives the residual stream after every layer."""
    w = {n: np.asarray(a, np.float64) for n, a in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens, dtype=np.int64)]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{layer.get('weights_of', i)}."
        x = x + MIXERS[layer["type"]](rms_norm(x, w[p + "norm1"], eps), layer["mixer"], sub(w, p + "mix."), eps)
        if layer.get("mlp"):
            x = x + gated_mlp(rms_norm(x, w[p + "norm2"], eps), sub(w, p + "mlp."))
        if layers_out is not None:
            layers_out.append(x.copy())
    return rms_norm(x, w["final.norm"], eps) @ w["embed"].T


def greedy(cfg, weights, prompt, max_new):
    """Greedy continuation, the whole sequence recomputed for every token; also the logits each pick was made from."""
    ids, rows = list(prompt), []
    for _ in range(max_new):
        rows.append(forward(cfg, weights, ids)[-1])
        ids.append(int(np.argmax(rows[-1])))
    return ids, rows


# ---- synthetic models ----------------------------------------------------------------------------
def tensor_shapes(cfg):
    """name -> shape of every tensor the configuration calls for."""
    d, out = cfg["width"], {"embed": (cfg["vocab"], cfg["width"]), "final.norm": (cfg["width"],)}
    for i, layer in enumerate(cfg["layers"]):
        if "weights_of" in layer:
            continue
        p, mx = f"l{i}.", layer["mixer"]
        out[p + "norm1"] = (d,)
        m = p + "mix."
        if layer["type"] == "delta":
            H, KH, dim, vdim, taps = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"], mx["conv"]
            for n, c in (("q", KH * dim), ("k", KH * dim), ("v", H * vdim)):
                out[m + n], out[m + n + ".conv"] = (c, d), (c, taps)
            out.update({m + "b": (H, d), m + "a": (H, d), m + "A_log": (H,), m + "dt_bias": (H,), m + "norm": (vdim,),
                        m + "g": (H * vdim, d), m + "o": (d, H * vdim)})
        else:
            H, dim, rd, vdim, R, Q = (mx[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank"))
            out.update({m + "dq": (Q, d), m + "dq.norm": (Q,), m + "uq": (H * (dim + rd), Q), m + "dkv": (R + rd, d),
                        m + "dkv.norm": (R,), m + "uk": (H * dim, R), m + "uv": (H * vdim, R), m + "g": (H, d),
                        m + "o": (d, H * vdim)})
        if layer.get("mlp"):
            ff = layer["mlp"]["ff"]
            out.update({p + "norm2": (d,), p + "mlp.gate": (ff, d), p + "mlp.up": (ff, d), p + "mlp.down": (d, ff)})
    return out


def bf16_round(a):
    """float32 array rounded to the nearest bfloat16 (ties to even), as float32."""
    b = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32).astype(np.uint64)
    return ((b + 0x7FFF + ((b >> 16) & 1)) & 0xFFFF0000).astype(np.uint32).view(np.float32)


def random_weights(cfg, seed):
    """bfloat16-valued random weights (as float32): matrices with unit row gain, norms around 1, decays spread
    from forgetting within a few tokens to remembering hundreds."""
    rng = np.random.default_rng(seed)
    out = {}
    for n, s in tensor_shapes(cfg).items():
        if n.endswith("norm") or ".norm" in n.split("mix")[-1][-6:]:
            a = 1.0 + 0.2 * rng.standard_normal(s)
        elif n.endswith("A_log"):
            a = rng.uniform(-4.0, 0.5, s)
        elif n.endswith("dt_bias"):
            a = rng.uniform(-2.0, 1.0, s)
        elif n.endswith(".conv"):
            a = rng.standard_normal(s) * s[1] ** -0.5
        elif n == "embed":
            a = rng.standard_normal(s)
        else:
            a = rng.standard_normal(s) * 1.2 * s[1] ** -0.5
        out[n] = bf16_round(a)
    return out
