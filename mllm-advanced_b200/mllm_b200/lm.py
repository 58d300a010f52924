"""ctypes driver of the bf16 language-model engine (include/mllmb200_lm.h): a model described layer by layer, its
slots of per-sequence state, the ragged step and the graph-replayed decode.  The engine's library is separate from the
quantized one (libmllm_b200_lm.so); without it nothing here works, there is no CPU fallback."""
import ctypes as C
import os
import subprocess

import numpy as np

_HERE = os.path.dirname(os.path.abspath(__file__))
BF16, F32 = 0, 1
ATTENTION, RETENTION, LATENT = 0, 1, 2
CLAMPED, GELU, SILU = 0, 1, 2  # gated feed-forwards
NORM_SANDWICH, NORM_POST = 0, 1
TENSORS = {n: i for i, n in enumerate(("q", "k", "v", "g", "o", "gate", "up", "down", "norm1", "norm1b", "norm2", "norm2b",
                                       "conv", "rel", "decay", "dkv", "dkv_norm", "uk", "uv", "router", "router_b"))}
MODEL_TENSORS = {"embed": 100, "head": 101, "final_norm": 102}
_LINEARS = {"q", "k", "v", "g", "o", "gate", "up", "down", "embed", "head", "dkv", "uk", "uv", "router"}


class Config(C.Structure):
    _fields_ = [(n, C.c_int) for n in ("vocab", "width", "layers", "dtype", "conv_taps", "max_seqs", "max_ctx", "max_rows")] + \
               [("eps", C.c_float), ("logit_scale", C.c_float), ("norm_place", C.c_int), ("residual_scale", C.c_float)]


class Layer(C.Structure):
    _fields_ = [(n, C.c_int) for n in ("mixer", "heads", "kv_heads", "dim", "vdim")] + [("score_scale", C.c_float)] + \
               [(n, C.c_int) for n in ("sink", "bias_rows", "bias_max", "rot_dims")] + [("rot_base", C.c_double), ("ff", C.c_int),
                                                                                      ("ff_limit", C.c_float), ("weights_of", C.c_int)] + \
               [(n, C.c_int) for n in ("kv_rank", "kv_from", "act", "experts", "top")]


class EngineError(RuntimeError):
    def __init__(self, status, where, text):
        self.status = status
        super().__init__(f"{where}: {text or 'failed'} (status {status})")


_lib = None


def lib_path():
    return os.path.join(os.path.dirname(_HERE), "lib", "libmllm_b200_lm.so")


def ensure_built():
    """Compiles the engine's library if it is not that of the sources beside it (messages go to stderr)."""
    subprocess.run(["bash", os.path.join(os.path.dirname(_HERE), "build.sh"), "lm"], check=True, stdin=subprocess.DEVNULL, stdout=2)


def lib():
    global _lib
    if _lib is not None:
        return _lib
    if not os.path.exists(lib_path()):
        raise ImportError(f"{lib_path()} is missing: build it with mllm-advanced_b200/build.sh lm; there is no CPU fallback")
    L = C.CDLL(lib_path())
    vp, ci = C.c_void_p, C.c_int
    sig = {"create": [C.POINTER(Config), C.POINTER(Layer), C.POINTER(vp)], "set_tensor": [vp, ci, ci, vp, ci, ci],
           "set_expert": [vp, ci, ci, ci, vp, ci, ci],
           "step": [vp, ci, vp, vp, vp, ci, vp, vp, ci], "decode": [vp, ci, vp, ci], "free_slot": [vp, ci],
           "read": [vp, ci, ci, ci, vp, vp], "keep_residual": [vp, ci], "read_residual": [vp, ci, ci, vp],
           "stats": [vp, C.POINTER(C.c_size_t), C.POINTER(C.c_longlong)], "synchronize": [vp], "check_device_status": [vp],
           "distance_buckets": [ci, ci, ci, vp]}
    for name, args in sig.items():
        fn = getattr(L, "mllmb200_lm_" + name)
        fn.argtypes, fn.restype = args, ci
    L.mllmb200_lm_destroy.argtypes, L.mllmb200_lm_destroy.restype = [vp], None
    L.mllmb200_lm_stream.argtypes, L.mllmb200_lm_stream.restype = [vp], vp
    L.mllmb200_lm_last_error.argtypes, L.mllmb200_lm_last_error.restype = [vp], C.c_char_p
    _lib = L
    return L


def distance_buckets(bias_rows, bias_max, count):
    """Rows of a distance-bias table for distances 0 .. count - 1 (host only)."""
    out = np.zeros(count, np.int32)
    st = lib().mllmb200_lm_distance_buckets(bias_rows, bias_max, count, out.ctypes.data)
    if st:
        raise EngineError(st, "distance_buckets", "invalid table")
    return out


def _ints(a):
    return np.ascontiguousarray(a, np.int32)


class LanguageModel:
    """config: fields of Config without `layers` and `dtype`; layers: one dict of Layer fields per layer."""

    def __init__(self, config, layers, dtype=BF16):
        self.config = dict({"norm_place": NORM_SANDWICH, "residual_scale": 1.0}, **config, layers=len(layers), dtype=dtype)
        self.layers = [dict({"sink": 0, "bias_rows": 0, "bias_max": 0, "rot_dims": 0, "rot_base": 1.0, "ff": 0, "ff_limit": 0.0,
                             "score_scale": 1.0, "weights_of": -1, "kv_rank": 0, "kv_from": -1, "act": CLAMPED, "experts": 0, "top": 0}, **d) for d in layers]
        self.vocab, self.max_seqs = self.config["vocab"], self.config["max_seqs"]
        self.max_ctx, self.max_rows = self.config["max_ctx"], self.config["max_rows"]
        self._L, self._h = lib(), C.c_void_p()
        descs = (Layer * len(layers))(*[Layer(**d) for d in self.layers])
        st = self._L.mllmb200_lm_create(C.byref(Config(**self.config)), descs, C.byref(self._h))
        if st:
            raise EngineError(st, "create", self._L.mllmb200_lm_last_error(None).decode())
        self.length = [0] * self.max_seqs
        self._free = list(range(self.max_seqs - 1, -1, -1))

    def close(self):
        if self._h:
            self._L.mllmb200_lm_destroy(self._h)
            self._h = C.c_void_p()

    def __del__(self):
        try:
            self.close()
        except Exception:
            pass

    def _check(self, st, where):
        if st:
            raise EngineError(st, where, self._L.mllmb200_lm_last_error(self._h).decode())

    # ---- weights
    @staticmethod
    def _tensor(name, data):
        """(what keeps the memory, address, rows, columns)"""
        if isinstance(data, (np.ndarray, np.generic)):
            data = np.ascontiguousarray(data, np.uint16 if name in _LINEARS else np.float64 if name == "decay" else np.float32)
            ptr, shape = data.ctypes.data, data.shape
        else:
            data = data.contiguous()
            ptr, shape = data.data_ptr(), tuple(data.shape)
        rows, cols = shape if len(shape) == 2 else (1, int(np.prod(shape)))
        return data, ptr, rows, cols

    def set_tensor(self, layer, name, data):
        """layer -1: a tensor of the model.  numpy (bf16 as uint16 bits for the linear maps), or a torch tensor on the
        device (bf16 for the linear maps)."""
        which = (MODEL_TENSORS if layer < 0 else TENSORS)[name]
        data, ptr, rows, cols = self._tensor(name, data)
        self._check(self._L.mllmb200_lm_set_tensor(self._h, layer, which, ptr, rows, cols), f"tensor {name} of layer {layer}")

    def set_expert(self, layer, expert, name, data):
        """gate, up or down of one expert of a mixture."""
        data, ptr, rows, cols = self._tensor(name, data)
        self._check(self._L.mllmb200_lm_set_expert(self._h, layer, expert, TENSORS[name], ptr, rows, cols),
                    f"tensor {name} of expert {expert} of layer {layer}")

    # ---- slots
    def acquire(self):
        """A free slot, or None."""
        return self._free.pop() if self._free else None

    def release(self, slot):
        self._check(self._L.mllmb200_lm_free_slot(self._h, slot), "free_slot")
        self.length[slot] = 0
        self._free.append(slot)

    # ---- steps
    def step(self, entries, want=(), sample=False):
        """entries: [(slot, tokens)], at most max_rows tokens in all; want: places among all these tokens.  Returns the
        logits of the wanted places, fp32 [len(want), vocab]."""
        slots, counts = _ints([s for s, _ in entries]), _ints([len(t) for _, t in entries])
        tokens = _ints(np.concatenate([np.asarray(t, np.int32) for _, t in entries]))
        want = _ints(want)
        logits = np.empty((len(want), self.vocab), np.float32)
        self._check(self._L.mllmb200_lm_step(self._h, len(slots), slots.ctypes.data, counts.ctypes.data, tokens.ctypes.data, len(want),
                                             want.ctypes.data, logits.ctypes.data, int(sample)), "step")
        for s, n in zip(slots, counts):
            self.length[s] += int(n)
        return logits

    def decode(self, slots, steps):
        """Greedy steps for these slots together; the tokens are read with `read`."""
        s = _ints(slots)
        self._check(self._L.mllmb200_lm_decode(self._h, len(s), s.ctypes.data, steps), "decode")
        for i in s:
            self.length[i] += steps

    def read(self, slot, first, count):
        """Tokens sampled after positions first .. first + count - 1 of a slot."""
        out = np.zeros(max(count, 1), np.int32)
        self._check(self._L.mllmb200_lm_read(self._h, slot, first, count, out.ctypes.data, None), "read")
        return out[:count]

    # ---- inspection
    def keep_residual(self, on):
        self._check(self._L.mllmb200_lm_keep_residual(self._h, int(on)), "keep_residual")

    def residual(self, layer, rows):
        out = np.zeros((rows, self.config["width"]), np.float32)
        self._check(self._L.mllmb200_lm_read_residual(self._h, layer, rows, out.ctypes.data), "read_residual")
        return out

    def stats(self):
        b, n = C.c_size_t(), C.c_longlong()
        self._check(self._L.mllmb200_lm_stats(self._h, C.byref(b), C.byref(n)), "stats")
        return {"state_bytes": b.value, "launches": n.value}

    def synchronize(self):
        self._check(self._L.mllmb200_lm_synchronize(self._h), "synchronize")

    def check_device_status(self):
        self._check(self._L.mllmb200_lm_check_device_status(self._h), "device status")

    def stream(self):
        import torch
        return torch.cuda.ExternalStream(self._L.mllmb200_lm_stream(self._h))
