"""Importable ``mk_hybrid`` module: a ctypes shim over ``libmkb200_hybrid.so``.

Marshals pointers and sizes into the structs of ``include/mkb200_hybrid.h``; all work happens in
the CUDA library, and a missing library is an ImportError, never a fallback.
"""

from __future__ import annotations

import ctypes
from pathlib import Path

import torch

from megakernels_b200.hybrid import RopeSpec

_HERE = Path(__file__).resolve().parent
LIB_PATH = _HERE / "libmkb200_hybrid.so"

MKBH_ABI_VERSION = 2
STATUS_WORDS = 16
FLAG_RECORD_TIMINGS = 1
ERROR_NAMES = {
    0: "MKBH_OK", 1: "MKBH_ERR_INVALID_ARGUMENT", 2: "MKBH_ERR_CUDA", 3: "MKBH_ERR_DEVICE_TIMEOUT",
    4: "MKBH_ERR_BAD_OPCODE", 5: "MKBH_ERR_UNSUPPORTED",
}
MIXERS = {"delta_rule": 0, "diff_attention": 1, "attention": 2, "latent_attention": 3}
NORMS = {"layer_norm": 0, "rms_norm": 1}
FEED_FORWARDS = {"poly_norm": 0, "clamped_glu": 1}

_i32, _f32, _ptr, _i64, _u32 = ctypes.c_int32, ctypes.c_float, ctypes.c_void_p, ctypes.c_int64, ctypes.c_uint32


class MkbhLayer(ctypes.Structure):
    _fields_ = [
        *[(n, _i32) for n in ("mixer", "heads", "kv_heads", "dim", "vdim", "rank", "window", "keep_first", "owns_kv",
                              "cache_keep", "cache_ring", "ff", "in_rows", "chunk", "ff_kind", "parallel", "x_buf", "canon_taps",
                              "conv_taps", "rot_dim", "rope_dims")],
        *[(n, _f32) for n in ("scale", "diff", "diff_lambda", "decay_scale", "unit_eps")],
        ("act", _f32 * 4),
        ("glu_limit", _f32), ("glu_alpha", _f32),
        *[(n, _ptr) for n in ("in_w", "out_w", "up_w", "down_w", "in_bias", "norm1", "norm2", "ls1", "ls2", "decay_w2",
                              "decay_w0", "out_norm", "k_cache", "v_cache", "state", "enter_w", "canon_w", "canon_gain", "canon_hist",
                              "canon_part", "conv_w", "conv_hist", "conv_part", "q_norm", "k_norm", "temp", "sink", "rope",
                              "value_rope", "absorb_w", "expand_w")],
    ]


class MkbhGlobals(ctypes.Structure):
    _fields_ = [
        ("abi_version", _u32), ("struct_bytes", _u32),
        *[(n, _i32) for n in ("dtype", "num_layers", "width", "vocab", "max_positions", "slots")],
        ("norm_kind", _i32), ("reserved", _i32),
        ("eps", _f32), ("embed_scale", _f32),
        *[(n, _ptr) for n in ("embed", "pos", "head", "final_norm", "layers_host", "layers_device", "tokens")],
        ("num_tokens", _i32), ("slot", _i32), ("pos0", _i32),
        ("pos_device", _ptr), ("want_rows", _ptr), ("num_want", _i32),
        ("logits", _ptr), ("argmax_out", _ptr), ("layers_out", _ptr),
        ("counters", _ptr), ("num_counters", _i32), ("max_kv_heads", _i32),
        ("instructions", _ptr), ("timings", _ptr), ("num_sms", _i32), ("queue_len", _i32),
        ("arrivals", _ptr), ("attn_part", _ptr), ("max_splits", _i32), ("part_vdim", _i32),
        *[(n, _ptr) for n in ("x", "proj", "mixed", "decay", "act")],
        *[(n, _i64) for n in ("x_elems", "proj_elems", "mixed_elems", "act_elems", "decay_elems")],
        *[(n, _ptr) for n in ("query", "act2", "ffn", "keys", "tail", "side")],
        *[(n, _i64) for n in ("query_elems", "act2_elems", "ffn_elems", "keys_elems", "tail_elems", "side_elems")],
        ("side_ff", _i32), ("side_rank", _i32),
        ("portion_capacity", _i32), ("reserved2", _i32),
        ("flags", _u32), ("wait_timeout_ms", _u32), ("status", _ptr),
    ]


class HybridKernelError(RuntimeError):
    def __init__(self, code: int, message: str, status=None):
        super().__init__(f"{ERROR_NAMES.get(code, code)}: {message}")
        self.code = code
        self.status = status


_lib = None


def load_library() -> ctypes.CDLL:
    global _lib
    if _lib is not None:
        return _lib
    if not LIB_PATH.exists():
        raise ImportError(f"{LIB_PATH} is missing: build it with `python -m megakernels_b200.build hybrid`. "
                          "There is no CPU fallback.")
    lib = ctypes.CDLL(str(LIB_PATH))
    G = ctypes.POINTER(MkbhGlobals)
    for name, args in (("decode", [G, _ptr]), ("prefill", [G, _ptr]), ("validate", [G, _ptr]),
                       ("sync_status", [G, _ptr, ctypes.POINTER(_i32 * STATUS_WORDS)])):
        fn = getattr(lib, f"mkb_hybrid_{name}")
        fn.argtypes, fn.restype = args, ctypes.c_int
    lib.mkb_hybrid_last_error.restype = ctypes.c_char_p
    lib.mkb_hybrid_layer_bytes.restype = lib.mkb_hybrid_globals_bytes.restype = ctypes.c_size_t
    if lib.mkb_hybrid_abi_version() != MKBH_ABI_VERSION:
        raise ImportError(f"libmkb200_hybrid.so has ABI {lib.mkb_hybrid_abi_version()}, expected {MKBH_ABI_VERSION}")
    sizes = (lib.mkb_hybrid_layer_bytes(), lib.mkb_hybrid_globals_bytes())
    if sizes != (ctypes.sizeof(MkbhLayer), ctypes.sizeof(MkbhGlobals)):
        raise ImportError(f"struct layouts of libmkb200_hybrid.so {sizes} differ from this shim")
    _lib = lib
    return lib


def _raise(code: int) -> None:
    if code:
        raise HybridKernelError(code, load_library().mkb_hybrid_last_error().decode())


def _p(t) -> int | None:
    if t is None:
        return None
    assert t.is_contiguous()
    return t.data_ptr()


def layer_structs(model):
    """Host array of layer descriptors, one per run."""
    runs, state, buf = model.config.runs, model.state, 0
    out = (MkbhLayer * len(runs))()
    for i, (layer, enters) in enumerate(runs):
        spec, w, s = model.config.layers[layer], model.layers[layer], out[i]
        m = spec.mixer
        s.mixer, s.heads, s.dim, s.in_rows = MIXERS[m.kind], m.heads, m.dim, m.in_rows
        if enters:  # (reads one residual buffer and writes the other)
            buf ^= 1
            s.enter_w = _p(model.enter)
        s.x_buf, s.parallel, s.canon_taps = buf, int(spec.parallel), spec.canon_taps
        if m.kind == "delta_rule":
            s.rank, s.decay_scale, s.unit_eps = m.rank, m.decay_scale, m.unit_eps
            s.decay_w2, s.decay_w0, s.out_norm = _p(w.decay_w2), _p(w.decay_w0), _p(w.out_norm)
            s.state = _p(state.matrices[i])
        else:
            src = i if m.kv_from is None else m.kv_from
            s.kv_heads, s.vdim, s.scale = m.key_groups, m.vdim, m.scale
            s.window, s.keep_first, s.owns_kv = m.window, min(m.keep_first, model.max_len()), int(m.kv_from is None)
            s.cache_keep, s.cache_ring = state.rows[src].keep, state.rows[src].ring
            s.k_cache, s.v_cache = _p(state.keys[src]), _p(state.values.get(src))
        if m.kind == "diff_attention":
            s.diff, s.diff_lambda = m.diff, w.diff_lambda
        elif m.kind == "attention":
            s.chunk, s.conv_taps = m.chunk, m.conv_taps
            if m.turn_values:
                s.value_rope = _p(model.rope_table(RopeSpec(m.vdim, m.rope.base)))
            if m.conv_taps:
                s.conv_hist, s.conv_part = _p(state.projected[i]), _p(state.projected_terms[i])
        elif m.kind == "latent_attention":
            s.rank, s.rot_dim = m.rank, m.rot_dim
        if m.kind in ("attention", "latent_attention"):
            s.rope, s.rope_dims = _p(model.rope_table(m.rope)), m.rope.dims
        if spec.canon_taps:
            s.canon_hist, s.canon_part = _p(state.inputs[i]), _p(state.input_terms[i])
        for name in ("in_w", "out_w", "up_w", "down_w", "in_bias", "norm1", "norm2", "ls1", "ls2", "canon_w", "canon_gain", "conv_w",
                     "q_norm", "k_norm", "temp", "sink", "absorb_w", "expand_w"):
            setattr(s, name, _p(getattr(w, name)))
        if spec.mlp is not None:
            s.ff, s.ff_kind, s.act = spec.mlp.ff, FEED_FORWARDS[spec.mlp.kind], (_f32 * 4)(*w.act)
            if spec.mlp.kind == "clamped_glu":
                s.glu_limit, s.glu_alpha = spec.mlp.limit, spec.mlp.alpha
    return out


class Call:
    """The launch struct of one ``HybridGlobals``; holds references to everything it points at."""

    def __init__(self, globs):
        lib = load_library()
        model = globs.model
        if model.device.type != "cuda":
            raise ValueError("the hybrid kernels run on a CUDA device only")
        self.globs, self.lib = globs, lib
        self.layers = layer_structs(model)
        raw = torch.frombuffer(bytearray(bytes(self.layers)), dtype=torch.uint8)
        self.layers_device = raw.to(model.device)
        g = self.g = MkbhGlobals()
        g.abi_version, g.struct_bytes = MKBH_ABI_VERSION, ctypes.sizeof(MkbhGlobals)
        cfg = model.config
        g.dtype = 1 if model.dtype == torch.float32 else 0
        g.num_layers, g.width, g.vocab = len(cfg.runs), cfg.width, cfg.vocab_size
        g.norm_kind = NORMS[cfg.norm]
        g.max_positions, g.slots = model.max_len(), model.state.pool.count
        g.eps, g.embed_scale = cfg.eps, cfg.embed_scale
        g.embed, g.pos, g.head, g.final_norm = _p(model.embed), _p(model.positions), _p(model.head), _p(model.final_norm)
        g.layers_host = ctypes.cast(self.layers, _ptr).value
        g.layers_device = _p(self.layers_device)
        g.max_kv_heads, g.max_splits, g.part_vdim = globs.max_kv_heads, globs.max_splits, globs.part_vdim
        for name in ("tokens", "want_rows", "argmax_out", "counters", "arrivals", "attn_part", "x", "proj", "mixed",
                     "decay", "act", "query", "act2", "ffn", "keys", "tail", "side", "status"):
            setattr(g, name, _p(getattr(globs, name)))
        g.num_counters = globs.counters.numel()
        for name in ("x", "proj", "mixed", "act", "decay", "query", "act2", "ffn", "keys", "tail", "side"):
            setattr(g, f"{name}_elems", getattr(globs, name).numel())
        g.side_ff, g.side_rank = globs.side_ff, globs.side_rank
        g.portion_capacity = globs.portion
        self._validated = None

    def _schedule(self):
        globs, g = self.globs, self.g
        ins = globs.instructions
        if ins is None:
            raise ValueError("no instructions: tensorize a schedule first")
        g.instructions, g.num_sms, g.queue_len = _p(ins), ins.shape[0], ins.shape[1]
        g.timings = _p(globs.timings)
        if self._validated is not ins:  # once per schedule
            host = ins.cpu()
            _raise(self.lib.mkb_hybrid_validate(ctypes.byref(g), _p(host)))
            self._validated = ins

    def decode(self, stream, record_timings=False):
        globs, g = self.globs, self.g
        self._schedule()
        g.num_tokens, g.num_want, g.slot, g.pos0 = 1, 1, globs.slot, globs.pos_id
        g.pos_device, g.logits, g.layers_out = _p(globs.pos_id_device), _p(globs.logits), None
        g.flags = FLAG_RECORD_TIMINGS if record_timings else 0
        _raise(self.lib.mkb_hybrid_decode(ctypes.byref(g), stream.cuda_stream))

    def prefill(self, num_tokens, num_want, logits, layers_out, stream):
        globs, g = self.globs, self.g
        g.num_tokens, g.num_want, g.slot, g.pos0 = num_tokens, num_want, globs.slot, globs.pos_id
        g.logits, g.layers_out = _p(logits), _p(layers_out)
        _raise(self.lib.mkb_hybrid_prefill(ctypes.byref(g), stream.cuda_stream))


def sync_status(call: Call, stream=None):
    """Synchronise; raise if a device-side wait gave up."""
    out = (_i32 * STATUS_WORDS)()
    stream = stream or torch.cuda.current_stream(call.globs.device)
    code = call.lib.mkb_hybrid_sync_status(ctypes.byref(call.g), stream.cuda_stream, ctypes.byref(out))
    if code == 2:
        _raise(code)
    if code:
        raise HybridKernelError(code, f"device status {list(out)[:8]}", list(out))
    return list(out)
