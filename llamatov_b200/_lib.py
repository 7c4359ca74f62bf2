"""ctypes binding of libllamatov_b200.so (the C ABI declared in include/llamatov_b200.h) and of
libllamatov_b200_dense.so (include/llamatov_b200_dense.h).  Each is loaded when one of its entry
points is first called; both share errors, status word and launch counter through
libllamatov_b200_common.so.

There is no CPU fallback: if the shared library is missing or a call fails, a RuntimeError
is raised with the library's own error text.
"""
import ctypes
import os

_HERE = os.path.dirname(os.path.abspath(__file__))
LIB_PATH = os.path.join(_HERE, "libllamatov_b200.so")
COMMON_PATH = os.path.join(_HERE, "libllamatov_b200_common.so")
DENSE_PATH = os.path.join(_HERE, "libllamatov_b200_dense.so")
_lib = None
_common = None
_dense = None

LT_OK = 0
STATUS_BITS = {1: "kv_overflow", 2: "bad_length", 4: "bad_token", 8: "wait_timeout"}

_vp = ctypes.c_void_p
_i = ctypes.c_int
_f = ctypes.c_float
_l = ctypes.c_long

# name -> argtypes (all return int unless listed in _RESTYPES)
SIGNATURES = {
    "lt_device_status": [ctypes.POINTER(ctypes.c_uint), _vp],
    "lt_quant_q8": [_vp, _vp, _vp, _i, _i, _vp],
    "lt_silu_mul_quant": [_vp, _vp, _vp, _vp, _i, _i, _vp],
    "lt_silu_mul": [_vp, _vp, _vp, _i, _vp],
    "lt_add": [_vp, _vp, _vp, _i, _vp],
    "lt_q8_gemv": [_vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _vp],
    "lt_q8_gemm_tc": [_vp, _vp, _vp, _vp, _vp, _i, _vp, _i, _i, _i, _i, _vp],
    "lt_quant_q8_ggml": [_vp, _vp, _vp, _i, _i, _vp],
    "lt_q8_gemm_ggml": [_vp, _vp, _vp, _vp, _vp, _i, _i, _i, _vp],
    "lt_rmsnorm": [_vp, _vp, _vp, _i, _i, _f, _vp],
    "lt_rmsnorm_quant": [_vp, _vp, _vp, _vp, _vp, _i, _i, _f, _vp],
    "lt_q8_gemv_allreduce": [_vp, _vp, _vp, _vp, _vp, _vp, _vp, _i, _i, _vp],
    "lt_rmsnorm_q8_gemv": [_vp, _vp, _vp, _vp, _f, _vp, _vp, _i, _i, _vp],
    "lt_rope": [_vp, _vp, _i, _i, _i, _f, _vp],
    "lt_append_kv": [_vp, _vp, _vp, _vp, _vp, _i, _i, _i, _vp],
    "lt_incr_len": [_vp, _vp],
    "lt_attn_decode_masked": [_vp, _vp, _vp, _vp, _vp, _i, _i, _i, _f, _i, _vp],
    "lt_argmax": [_vp, _i, _vp, _vp, _vp],
    "lt_argmax_scratch_bytes": [],
    "lt_argmax_rows_scratch_bytes": [_i],
    "lt_embed_q8": [_vp, _vp, _vp, _vp, _i, _i, _vp],
    "lt_token_record": [_vp, _vp, _vp, _i, _vp],
    "lt_graph_replay_token": [_vp, _vp, _vp, _vp, _vp, _vp],
    "lt_embed_q8_rows": [_vp, _vp, _vp, _vp, _i, _i, _i, _vp],
    "lt_rope_rows": [_vp, _i, _vp, _i, _i, _i, _f, _vp],
    "lt_append_kv_rows": [_vp, _vp, _vp, _vp, _i, _vp, _i, _i, _i, _i, _vp],
    "lt_silu_mul_quant_rows": [_vp, _vp, _i, _vp, _vp, _i, _i, _vp],
    "lt_attn_prefill": [_vp, _i, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _f, _i, _i, _vp],
    "lt_rope_batch": [_vp, _i, _vp, _i, _i, _i, _f, _vp],
    "lt_append_kv_batch": [_vp, _vp, _vp, _vp, _i, _vp, _i, _i, _i, _i, _vp],
    "lt_attn_decode_batch": [_vp, _i, _vp, _vp, _vp, _vp, _i, _vp, _i, _i, _i, _f, _i, _i, _vp, _vp, _vp],
    "lt_attn_decode_split": [_vp, _i, _vp, _vp, _vp, _vp, _i, _vp, _i, _i, _i, _f, _i, _i, _i, _vp, _vp, _vp],
    "lt_rope_attn_decode_split": [_vp, _i, _vp, _vp, _vp, _vp, _i, _vp, _i, _i, _i, _f, _f, _i, _i, _i, _vp, _vp, _vp, _vp],
    "lt_rope_append_batch": [_vp, _i, _i, _i, _i, _f, _vp, _vp, _vp, _i, _i, _vp, _vp],
    "lt_comm_alloc": [_i, _i, _vp, _vp],
    "lt_comm_connect": [_vp, _i, _vp],
    "lt_comm_free": [_vp],
    "lt_allreduce_add": [_vp, _vp, _vp, _vp, _i, _vp],
    "lt_allreduce_add_tree": [_vp, _vp, _vp, _vp, _i, _vp],
    "lt_argmax_rows": [_vp, _vp, _l, _i, _i, _i, _vp, _vp, _vp],
    "lt_q8_gemv_lanes": [_vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _vp],
    "lt_q8_linear_static": [_vp, _vp, _vp, _vp, _vp, _i, _i, _vp],
    "lt_q8_linear_static_max_k": [],
    "lt_decode_step": [_vp, _vp],
    "lt_decode_step_supported": [_vp],
    "lt_decode_num_ctas": [],
    "lt_decode_ws_replicas": [],
    "lt_decode_step_pdl": [_vp, _vp],
    "lt_decode_pdl_num_parts": [],
}
_RESTYPES = {"lt_last_error": ctypes.c_char_p, "lt_version": ctypes.c_char_p,
             "lt_launch_count": ctypes.c_ulonglong}
# name -> (argtypes, restype) for the entries that return something other than a status code
_QUERIES = {"lt_attn_decode_batch_scratch_floats": ([_i, _i, _i], ctypes.c_long),
            "lt_attn_decode_split_scratch_floats": ([_i, _i, _i, _i], ctypes.c_long),
            "lt_set_chained_launch": ([_i], ctypes.c_int)}


# ---- include/llamatov_b200_dense.h
DN_MAX_SEG = 6
DN_STORE, DN_RESID, DN_GLU, DN_STORE_GLU = 0, 1, 2, 3
DN_GLU_GELU, DN_GLU_CLAMPED = 0, 1
DN_ACT = {None: 0, "silu": 1, "sigmoid": 2, "logsigmoid": 3}
DN_IN_TYPED, DN_IN_CAST, DN_IN_NORM = 0, 1, 2


class DnEpilogue(ctypes.Structure):
    _fields_ = [("kind", _i), ("out_f32", _i), ("nseg", _i), ("seg_end", _i * DN_MAX_SEG), ("seg_act", _i * DN_MAX_SEG),
                ("seg_scale", _f * DN_MAX_SEG), ("bias", _vp), ("ls", _vp), ("glu_act", _i), ("glu_alpha", _f), ("glu_limit", _f),
                ("tail_from", _i), ("ldtail", _i), ("tail", _vp), ("glu_from", _i), ("y2", _vp)]


class DnPrologue(ctypes.Structure):
    _fields_ = [("kind", _i), ("n1", _i), ("group", _i), ("count", _i), ("eps", _f), ("x", _vp), ("x2", _vp), ("w", _vp),
                ("w_period", _i), ("gate", _vp), ("gate_first", _i), ("seg", _i), ("segp", _i)]


class DnDecay(ctypes.Structure):
    _fields_ = [("decay", _vp), ("la", _vp), ("ldla", _i), ("a1", _vp), ("a2", _vp), ("lda2", _i), ("rank", _i),
                ("bias", _vp), ("inv_tau", _f), ("hla", _vp), ("hdt", _vp), ("D", _vp), ("ldh", _i), ("per", _i)]


class DnLatent(ctypes.Structure):
    _fields_ = [(n, _i) for n in ("H", "dp", "rtp", "dvp", "rot", "rp", "rank", "window", "cap")] + \
               [("scale", _f), ("eps", _f), ("freq", _vp), ("cnorm", _vp)]


class DnSsd(ctypes.Structure):
    _fields_ = [(n, _i) for n in ("H", "G", "dp", "dvp", "taps")] + [(n, _vp) for n in ("conv", "conv_b", "dt_bias", "A", "D")]


class DnGqa(ctypes.Structure):
    _fields_ = [(n, _i) for n in ("H", "G", "dp", "dvp", "rot", "qcount", "kcount", "cap")] + \
               [(n, _f) for n in ("scale", "softcap", "eps", "vmix")] + [(n, _vp) for n in ("freq", "qnorm", "knorm")]


DENSE_SIGNATURES = {
    "lt_dn_embed": [_vp, _i, _i, _vp, _f, _vp, _f, _vp, _vp, _i, _i, _i, _i, _vp],
    "lt_dn_norm_rows": [_vp, _i, _vp, _vp, _i, _vp, _i, _vp, _i, _i, _i, _i, _i, _i, _f, _i, _i, _i, _vp],
    "lt_dn_concat_rows": [_vp, _i, _i, _vp, _i, _i, _vp, _i, _i, _i, _vp],
    "lt_dn_linear": [_vp, _i, _vp, _i, _vp, _i, _i, _i, _i, _i, ctypes.POINTER(DnEpilogue), _i, _vp],
    "lt_dn_gemv": [_vp, _i, _vp, _i, _i, _i, ctypes.POINTER(DnPrologue), ctypes.POINTER(DnEpilogue), _vp],
    "lt_dn_recurrence": [_vp, _vp, _vp, _i, _vp, _vp, _i, _i, _i, _i, _i, _i, ctypes.POINTER(DnDecay), _vp],
    "lt_dn_recurrence_chunked": [_vp, _vp, _vp, _i, _vp, _vp, _i, _i, _i, _i, _i, ctypes.POINTER(DnDecay), _vp, _vp],
    "lt_dn_latent_rows": [_vp, _i, _vp, _vp, _i, _i, _i, _i, ctypes.POINTER(DnLatent), _vp],
    "lt_dn_window_attn": [_vp, _i, _vp, _i, _vp, _i, _vp, _i, _vp, _i, _i, _i, _i, ctypes.POINTER(DnLatent), _vp],
    "lt_dn_latent_step": [_vp, _vp, _vp, _vp, _vp, _vp, _i, ctypes.POINTER(DnLatent), _i, _vp, _vp],
    "lt_dn_ssd_rows": [_vp, _i, _vp, _i, _vp, _vp, _i, _vp, _vp, _i, _i, _i, ctypes.POINTER(DnSsd), _vp],
    "lt_dn_ssd_step": [_vp, _vp, _vp, _vp, _vp, _i, _vp, _vp, ctypes.POINTER(DnSsd), _vp],
    "lt_dn_gqa_rows": [_vp, _i, _vp, _vp, _vp, _i, _i, _i, _i, ctypes.POINTER(DnGqa), _vp],
    "lt_dn_gqa_attn": [_vp, _i, _vp, _vp, _vp, _i, _vp, _i, _i, _i, _i, ctypes.POINTER(DnGqa), _vp],
    "lt_dn_gqa_step": [_vp, _vp, _vp, _vp, _i, _vp, _vp, _i, _vp, ctypes.POINTER(DnGqa), _i, _vp, _vp, _vp],
}
_DENSE_QUERIES = {"lt_dn_gqa_step_ws": ([_i, _i, _i], ctypes.c_long),
                  "lt_dn_gqa_step_tickets": ([_i, _i], _i),
                  "lt_dn_latent_step_ws": ([_i, _i, _i, _i], ctypes.c_long),
                  "lt_dn_recurrence_chunked_ws": ([_i, _i, _i, _i], ctypes.c_long)}
# what the common library exports (the Q8_0 library passes these through to its users as well)
_COMMON_NAMES = ("lt_last_error", "lt_version", "lt_launch_count", "lt_set_chained_launch", "lt_device_status",
                 "lt_graph_replay_token", "lt_token_record", "lt_quant_q8", "lt_silu_mul_quant", "lt_silu_mul", "lt_add",
                 "lt_rmsnorm", "lt_rmsnorm_quant", "lt_rope", "lt_append_kv", "lt_incr_len", "lt_argmax_scratch_bytes",
                 "lt_argmax", "lt_embed_q8")


def _bind(L, names):
    for name in names:
        fn = getattr(L, name)
        if name in SIGNATURES:
            fn.argtypes, fn.restype = SIGNATURES[name], ctypes.c_int
        elif name in _RESTYPES:
            fn.argtypes, fn.restype = [], _RESTYPES[name]
        else:
            fn.argtypes, fn.restype = _QUERIES[name]


def _load(path):
    if not os.path.exists(path):
        raise RuntimeError(
            "%s is not built (%s). Run `python -m llamatov_b200.build`; "
            "this package has no CPU or PyTorch fallback." % (os.path.basename(path), path))
    return ctypes.CDLL(path)


def lib():
    """The loaded Q8_0 library (loads on first use)."""
    global _lib
    if _lib is None:
        L = _load(LIB_PATH)
        _bind(L, list(SIGNATURES) + list(_RESTYPES) + list(_QUERIES))
        _lib = L
    return _lib


def common():
    """The library that the other two share (loads on first use)."""
    global _common
    if _common is None:
        L = _load(COMMON_PATH)
        _bind(L, _COMMON_NAMES)
        _common = L
    return _common


def dense():
    """The library of the bf16 / fp32 models (loads on first use)."""
    global _dense
    if _dense is None:
        L = _load(DENSE_PATH)
        for name, args in DENSE_SIGNATURES.items():
            fn = getattr(L, name)
            fn.argtypes, fn.restype = args, ctypes.c_int
        for name, (args, rt) in _DENSE_QUERIES.items():
            fn = getattr(L, name)
            fn.argtypes, fn.restype = args, rt
        _dense = L
    return _dense


def last_error():
    return common().lt_last_error().decode("utf-8", "replace")


def check(rc, what=""):
    """Raise RuntimeError if a launcher returned a non-zero code."""
    if rc != LT_OK:
        raise RuntimeError("llamatov_b200 %s failed (code %d): %s" % (what, rc, last_error()))


def call(name, *args):
    if name in DENSE_SIGNATURES:
        L = dense()
    else:
        L = common() if name in _COMMON_NAMES else lib()
    check(getattr(L, name)(*args), name)


def launch_count():
    return int(common().lt_launch_count())


def device_status(stream=None):
    """Read and clear the device status word; returns the set of flag names."""
    v = ctypes.c_uint(0)
    check(common().lt_device_status(ctypes.byref(v), stream), "lt_device_status")
    return {n for bit, n in STATUS_BITS.items() if v.value & bit}
