"""Language models by architecture: ``load_model`` reads a checkpoint folder with the family its config.json
names; ``LanguageModel`` generates, ``KvCache`` / ``DecodeSession`` take it like a GPT-2 model, and
``RequestBatch`` feeds requests of unequal length, each in a cache slot of its own."""
from __future__ import annotations

import ctypes as C
import json
import os

import numpy as np

from . import NnError, ERR_UNSUPPORTED, KernelRegistry, _f32, _f32p, _LmInfo, _u32, _u32p, LM_F32
from .gpt2 import KvCache

DTYPES = {"bfloat16": 0, "float32": LM_F32}


class LanguageModel:
    """A decoder-only model of any family of the registry (``dtype``: "bfloat16" or "float32")."""

    def __init__(self, reg: KernelRegistry, handle):
        self.reg, self.h, self.flags = reg, handle, 0
        info = _LmInfo()
        reg.check(reg.lib.b200nn_lm_get_info(handle, C.byref(info)))
        self.n_layer, self.width, self.vocab_size = info.n_layer, info.width, info.vocab_size
        self.max_positions = info.n_positions or None
        self.eos_token = info.eos_token if info.eos_token >= 0 else None
        self.family = reg.lib.b200nn_lm_family(handle).decode()

    @classmethod
    def load(cls, path, reg: KernelRegistry, dtype: str = "bfloat16", flags: int = 0):
        """A folder with config.json and model.safetensors."""
        h = C.c_void_p()
        reg.check(reg.lib.b200nn_lm_load(reg.h, os.fsencode(path), DTYPES[dtype] | flags, C.byref(h)))
        return cls(reg, h)

    @classmethod
    def from_weights(cls, config: dict, weights: dict, reg: KernelRegistry, dtype: str = "bfloat16", flags: int = 0):
        """``config`` as config.json holds it, ``weights`` name -> array (Linear weights [out, in])."""
        arrs = {n: _f32(a) for n, a in weights.items()}
        n = len(arrs)
        names = (C.c_char_p * n)(*[k.encode() for k in arrs])
        data = (_f32p * n)(*[p for _, p in arrs.values()])
        numels = (C.c_size_t * n)(*[a.size for a, _ in arrs.values()])
        h = C.c_void_p()
        reg.check(reg.lib.b200nn_lm_create(reg.h, json.dumps(config).encode(), n, names, data, numels, DTYPES[dtype] | flags, C.byref(h)))
        return cls(reg, h)

    def lm_handle(self):
        return self.h

    def generate_batch(self, prompts, max_new_tokens, flags: int = 0):
        """Greedy: prompts [batch, prompt_len] -> (tokens [batch, prompt_len + max_new], lengths [batch])."""
        p = np.ascontiguousarray(prompts, dtype=np.uint32)
        batch, plen = p.shape
        out = np.zeros((batch, plen + max_new_tokens), dtype=np.uint32)
        lens = (C.c_size_t * batch)()
        self.reg.check(self.reg.lib.b200nn_lm_generate_batch(self.h, p.ctypes.data_as(_u32p), batch, plen, max_new_tokens, flags,
                                                             out.ctypes.data_as(_u32p), lens))
        return out, np.array(list(lens), dtype=np.int64)

    def generate(self, prompt, max_new_tokens, flags: int = 0):
        out, lens = self.generate_batch(np.asarray(prompt)[None, :], max_new_tokens, flags)
        return out[0, : lens[0]]

    def generate_sampling(self, prompt, max_new_tokens, top_k, temperature, rng):
        """Top-k sampling; ``rng`` (SimpleRng) advances one draw per token."""
        p, pp = _u32(prompt)
        out = np.zeros(p.size + max_new_tokens, dtype=np.uint32)
        n = C.c_size_t()
        self.reg.check(self.reg.lib.b200nn_lm_generate_sampling(self.h, pp, p.size, max_new_tokens, top_k, temperature, C.byref(rng.state),
                                                                out.ctypes.data_as(_u32p), C.byref(n)))
        return out[: n.value]

    def __del__(self):
        try:
            if self.h and self.reg.h:
                self.reg.lib.b200nn_lm_destroy(self.h)
                self.h = None
        except Exception:
            pass


def load_model(path, reg: KernelRegistry, dtype: str = "bfloat16", flags: int = 0) -> LanguageModel:
    if dtype not in DTYPES:
        raise NnError(ERR_UNSUPPORTED, f"dtype {dtype}: expected one of {sorted(DTYPES)}")
    return LanguageModel.load(path, reg, dtype, flags)


class RequestBatch:
    """Live requests of a model by name, each holding one slot of a shared cache."""

    def __init__(self, model, slots: int, capacity: int):
        self.model, self.reg = model, model.reg
        self.cache = KvCache(model, slots, capacity)
        self._slots: dict = {}

    def __len__(self):
        return len(self._slots)

    def length(self, name) -> int:
        """Tokens the request has brought so far."""
        return int(self.reg.lib.b200nn_kvcache_slot_len(self.cache.h, self._slots[name]))

    def slot(self, name) -> int:
        return self._slots[name]

    def step(self, entries):
        """``entries``: (name, tokens, want) of every request that takes part; ``want`` are places among its
        tokens.  A new name takes a free slot.  Returns the logits [number wanted, vocab] in that order."""
        slots, counts, toks, want, row = [], [], [], [], 0
        for name, tokens, places in entries:
            if name not in self._slots:
                s = C.c_int32()
                self.reg.check(self.reg.lib.b200nn_kvcache_acquire(self.cache.h, C.byref(s)))
                self._slots[name] = s.value
            slots.append(self._slots[name])
            counts.append(len(tokens))
            toks.extend(tokens)
            want.extend(row + int(p) for p in places)
            row += len(tokens)
        t, tp = _u32(toks)
        out = np.empty((len(want), self.model.vocab_size), dtype=np.float32)
        n = len(slots)
        self.reg.check(self.reg.lib.b200nn_lm_step(self.cache.h, n, (C.c_int32 * n)(*slots), (C.c_size_t * n)(*counts), tp, len(want),
                                                   (C.c_size_t * max(1, len(want)))(*want), out.ctypes.data_as(_f32p)))
        return out

    def end(self, name):
        """Gives the request's slot back."""
        self.reg.check(self.reg.lib.b200nn_kvcache_release(self.cache.h, self._slots.pop(name)))
