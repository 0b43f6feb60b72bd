"""Seeded synthetic GPT-2 weights and token ids (no checkpoint files are needed).

Every tensor is drawn from its own stream so that any two processes that agree on (config, base seed)
hold bit-identical weights: N(0, std) for embeddings, dense weights and biases, gamma = 1 and beta = 0
for LayerNorm unless ``random_ln``.  Dense weights use the checkpoint's Conv1D layout [in, out].

Two sources.  ``"pcg64"`` (the default): ``numpy.random.Generator(PCG64(seed))``.  ``"simple_rng"``:
the reference's own ``SimpleRng`` xorshift64 (gpt2.rs:1000-1023) seeded per tensor, normals by
Box-Muller on pairs of its uniforms (``b200nn_simple_rng_fill_normal``), so that a Rust caller that has
nothing but ``SimpleRng`` regenerates the same tensors.  The per-tensor seed is the same in both:
``base + 1`` wte, ``+ 2`` wpe, ``+ 3 / + 4`` ln_f, and for layer i with ``s = base + 1000 (i + 1)``:
``s+1 / s+2`` ln_1, ``s+3 / s+4`` c_attn weight / bias, ``s+5 / s+6`` attn c_proj, ``s+7 / s+8`` ln_2,
``s+9 / s+10`` mlp c_fc, ``s+11 / s+12`` mlp c_proj.
"""
from __future__ import annotations

import numpy as np

BASE_SEED = 20260101


def _normal(seed, shape, std, source="pcg64"):
    if source == "simple_rng":
        import ctypes as C

        from . import load_library
        lib = load_library()
        out = np.empty(int(np.prod(shape)), dtype=np.float32)
        state = C.c_uint64(lib.b200nn_simple_rng_new(seed))
        rc = lib.b200nn_simple_rng_fill_normal(C.byref(state), out.size, std, out.ctypes.data_as(C.POINTER(C.c_float)))
        assert rc == 0
        return out.reshape(shape)
    return (np.random.Generator(np.random.PCG64(seed)).standard_normal(shape, dtype=np.float32) * np.float32(std))


def gpt2_weights(cfg, base_seed: int = BASE_SEED, std: float = 0.02, random_ln: bool = False, source: str = "pcg64") -> dict:
    if source not in ("pcg64", "simple_rng"):
        raise ValueError("source must be 'pcg64' or 'simple_rng'")
    draw = _normal
    _normal_of = lambda seed, shape, s: draw(seed, shape, s, source)
    return _build(cfg, base_seed, std, random_ln, _normal_of)


def _build(cfg, base_seed, std, random_ln, _normal) -> dict:
    d, V, P = cfg.n_embd, cfg.vocab_size, cfg.n_positions
    w = {"wte": _normal(base_seed + 1, (V, d), std), "wpe": _normal(base_seed + 2, (P, d), std)}

    def ln(seed):
        if random_ln:
            return (1.0 + _normal(seed, (d,), 0.1)).astype(np.float32), _normal(seed + 1, (d,), 0.1)
        return np.ones(d, dtype=np.float32), np.zeros(d, dtype=np.float32)

    w["ln_f.weight"], w["ln_f.bias"] = ln(base_seed + 3)
    for i in range(cfg.n_layer):
        s = base_seed + 1000 * (i + 1)
        p = f"h.{i}."
        w[p + "ln_1.weight"], w[p + "ln_1.bias"] = ln(s + 1)
        w[p + "attn.c_attn.weight"] = _normal(s + 3, (d, 3 * d), std)
        w[p + "attn.c_attn.bias"] = _normal(s + 4, (3 * d,), std)
        w[p + "attn.c_proj.weight"] = _normal(s + 5, (d, d), std)
        w[p + "attn.c_proj.bias"] = _normal(s + 6, (d,), std)
        w[p + "ln_2.weight"], w[p + "ln_2.bias"] = ln(s + 7)
        w[p + "mlp.c_fc.weight"] = _normal(s + 9, (d, 4 * d), std)
        w[p + "mlp.c_fc.bias"] = _normal(s + 10, (4 * d,), std)
        w[p + "mlp.c_proj.weight"] = _normal(s + 11, (4 * d, d), std)
        w[p + "mlp.c_proj.bias"] = _normal(s + 12, (d,), std)
    return w


def token_ids(seed: int, shape, vocab: int) -> np.ndarray:
    """Uniform ids in [0, vocab)."""
    return np.random.Generator(np.random.PCG64(seed)).integers(0, vocab, size=shape, dtype=np.int64).astype(np.uint32)


def int4_linear_case(seed: int, m: int, k: int, n: int, group: int = 128):
    """Isolated int4 Linear inputs: signed nibbles uniform in [-8,7] packed in the reference layout
    [K/8,N] (stored +8), fp16-representable scales uniform in [0.005,0.02], activations N(0,1)."""
    g = np.random.Generator(np.random.PCG64(seed))
    q = g.integers(-8, 8, size=(k, n), dtype=np.int64)
    u = (q + 8).astype(np.uint32).reshape(k // 8, 8, n)
    packed = np.zeros((k // 8, n), dtype=np.uint32)
    for i in range(8):
        packed |= u[:, i, :] << np.uint32(4 * i)
    n_groups = (k + group - 1) // group
    scales = g.uniform(0.005, 0.02, size=(n_groups, n)).astype(np.float16).astype(np.float32)
    x = g.standard_normal((m, k), dtype=np.float32)
    return packed, scales, x, q


def hybrid_config(width, layers, vocab, heads, kv_heads, dim, rot_dim, kv_rank, q_rank, window, ff, conv=4):
    """config.json of a Vivezen decoder whose every fourth layer is latent attention and the others gated delta
    rule, all with a feed-forward (head sizes equal for both mixers)."""
    lat = {"type": "latent_attention", "mlp": {"kind": "dense", "ff": ff},
           "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": dim, "kv_rank": kv_rank, "q_rank": q_rank, "mask": {"size": window},
                     "rot": {"base": 10000.0, "dims": rot_dim}, "scale": (dim + rot_dim) ** -0.5}}
    dlt = {"type": "delta", "mlp": {"kind": "dense", "ff": ff},
           "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "conv": conv}}
    return {"architecture": "Vivezen", "width": width, "vocab": vocab, "norm": {"eps": 1e-5},
            "layers": [lat if i % 4 == 3 else dlt for i in range(layers)]}


def hybrid_weights(cfg, base_seed=BASE_SEED):
    """Random f32 weights of a hybrid decoder by tensor name: matrices with unit row gain, norms of one, decays spread
    from a few tokens to hundreds."""
    d, out = cfg["width"], {}

    def mat(name, *shape):
        out[name] = np.random.default_rng(base_seed + len(out)).standard_normal(shape, dtype=np.float32) * np.float32(shape[-1] ** -0.5)

    def ones(name, n):
        out[name] = np.ones(n, dtype=np.float32)

    mat("embed", cfg["vocab"], d)
    ones("final.norm", d)
    for i, layer in enumerate(cfg["layers"]):
        p, x = f"l{i}.", layer["mixer"]
        m = p + "mix."
        ones(p + "norm1", d)
        if layer["type"] == "delta":
            H, KH, dim, vd = x["heads"], x["kv_heads"], x["dim"], x["vdim"]
            for n, c in (("q", KH * dim), ("k", KH * dim), ("v", H * vd)):
                mat(m + n, c, d)
                mat(m + n + ".conv", c, x["conv"])
            for n, c in (("b", H), ("a", H), ("g", H * vd)):
                mat(m + n, c, d)
            out[m + "A_log"] = np.linspace(-4.0, 0.5, H, dtype=np.float32)
            out[m + "dt_bias"] = np.full(H, -1.0, dtype=np.float32)
            ones(m + "norm", vd)
            mat(m + "o", d, H * vd)
        else:
            H, dim, rd, vd, R, Q = (x[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank"))
            mat(m + "dq", Q, d)
            ones(m + "dq.norm", Q)
            mat(m + "uq", H * (dim + rd), Q)
            mat(m + "dkv", R + rd, d)
            ones(m + "dkv.norm", R)
            mat(m + "uk", H * dim, R)
            mat(m + "uv", H * vd, R)
            mat(m + "g", H, d)
            mat(m + "o", d, H * vd)
        if layer.get("mlp"):
            ff = layer["mlp"]["ff"]
            ones(p + "norm2", d)
            mat(p + "mlp.gate", ff, d)
            mat(p + "mlp.up", ff, d)
            mat(p + "mlp.down", d, ff)
    return out


def zufilorn_config(width, layers, vocab, heads, kv_heads, dim, vdim, ff, positions, streams=2, conv=4):
    """config.json of a Zufilorn decoder whose layers repeat channel delta rule, mLSTM, mLSTM, differential attention, all
    with a feed-forward (mixer heads of vdim x vdim states; attention maps of dim columns over vdim values)."""
    mlp = {"kind": "dense", "ff": ff}
    dlt = {"type": "channel_delta", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": vdim, "vdim": vdim, "conv": conv}}
    mem = {"type": "mlstm", "mlp": mlp, "mixer": {"heads": heads, "dim": vdim, "vdim": vdim, "gate_cap": 15.0}}
    att = {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5,
                                                      "softcap": 30.0, "q_temp": {"coef": 0.1, "every": 1024}, "diff": 0.5}}
    return {"architecture": "Zufilorn", "width": width, "vocab": vocab, "streams": streams, "max_positions": positions, "norm": {"eps": 1e-5},
            "layers": [(dlt, mem, mem, att)[i % 4] for i in range(layers)]}


def zufilorn_weights(cfg, rank, base_seed=BASE_SEED):
    """Random f32 weights of a Zufilorn decoder by tensor name: matrices with unit row gain, norms of one, decays and gates
    spread from a few tokens to hundreds; rank: inner size of the two-step projections."""
    d, n, out = cfg["width"], cfg["streams"], {}

    def mat(name, *shape):
        out[name] = np.random.default_rng(base_seed + len(out)).standard_normal(shape, dtype=np.float32) * np.float32(shape[-1] ** -0.5)

    def full(name, value, *shape):
        out[name] = np.full(shape, value, dtype=np.float32)

    mat("embed", cfg["vocab"], d)
    mat("head", cfg["vocab"], d)
    mat("pos", cfg["max_positions"], d)
    full("final.norm", 0.0, d)
    for i, layer in enumerate(cfg["layers"]):
        p, x = f"l{i}.", layer["mixer"]
        m, H, dim, vd = p + "mix.", x["heads"], x["dim"], x["vdim"]
        full(p + "norm1", 0.0, d)
        if layer["type"] == "channel_delta":
            KH = x["kv_heads"]
            for t, c in (("q", KH * dim), ("k", KH * dim), ("v", H * vd)):
                mat(m + t, c, d)
                mat(m + t + ".conv", c, x["conv"])
            for t, r, c in (("b", H, d), ("a1", rank, d), ("a2", H * dim, rank), ("g1", rank, d), ("g2", H * vd, rank)):
                mat(m + t, r, c)
            out[m + "A_log"] = np.linspace(-4.0, 0.5, H, dtype=np.float32)
            full(m + "dt_bias", -1.0, H * dim)
            full(m + "norm", 1.0, vd)
        elif layer["type"] == "mlstm":
            for t, c in (("q", H * dim), ("k", H * dim), ("v", H * vd), ("g", H * vd), ("i", H), ("f", H)):
                mat(m + t, c, d)
            full(m + "i.b", 0.0, H)
            out[m + "f.b"] = np.linspace(2.0, 6.0, H, dtype=np.float32)
            full(m + "norm", 1.0, H * vd)
        else:
            G = x["kv_heads"]
            for t, c in (("q", H * 2 * dim), ("k", G * 2 * dim), ("v", G * vd), ("g", H)):
                mat(m + t, c, d)
            for t in ("lq1", "lk1", "lq2", "lk2"):
                mat(m + t, dim)
        mat(m + "o", d, H * vd)
        sub = 1
        if layer.get("mlp"):
            ff, sub = layer["mlp"]["ff"], 2
            full(p + "norm2", 0.0, d)
            mat(p + "mlp.gate", ff, d)
            mat(p + "mlp.up", ff, d)
            mat(p + "mlp.down", d, ff)
        for q in range(1, sub + 1):
            full(f"{p}hc{q}.in", 1.0 / n, n)
            full(f"{p}hc{q}.out", 1.0, n)
            out[f"{p}hc{q}.mix"] = np.eye(n, dtype=np.float32)
    return out
