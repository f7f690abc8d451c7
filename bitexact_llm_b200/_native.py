"""ctypes bindings of libbitexact_b200.so (`lib()`, C ABI in include/bitexact_b200.h: integer engines, sampler) and
libbitexact_float.so (`float_lib()`, include/bitexact_float.h: float models).

The libraries are built in-tree by `bitexact_llm_b200.build` (nvcc, sm_100a).  Loading fails loudly when one is
missing: there is deliberately no fallback path.
"""

import ctypes
import os

_HERE = os.path.dirname(os.path.abspath(__file__))
LIB_PATH = os.path.join(_HERE, "_lib", "libbitexact_b200.so")
FLOAT_LIB_PATH = os.path.join(_HERE, "_lib", "libbitexact_float.so")

BX_OK, BX_EARG, BX_ELAUNCH, BX_EDEVICE, BX_ELIMIT = 0, -1, -2, -3, -4
_ERR = {BX_EARG: "argument contract violated (shape / alignment / null pointer)",
        BX_ELAUNCH: "CUDA launch or driver call failed", BX_EDEVICE: "a device-side wait timed out",
        BX_ELIMIT: "request exceeds the fixed capacity of this entry point"}

_libs = {}

P, I, L, Z, R = ctypes.c_void_p, ctypes.c_int, ctypes.c_int64, ctypes.c_size_t, ctypes.c_float

_SIGNATURES = {
    "bx_version": (I, []),
    "bx_launch_count": (ctypes.c_longlong, []),
    "bx_device_status": (I, []),
    "bx_clear_device_status": (I, []),
    "bx_set_device_status": (I, [I]),
    "bx_i8_tensor_peak": (I, [I, I, P, P]),
    "bx_exact_linear_scratch_bytes": (Z, [I, I]),
    "bx_exact_linear": (I, [P, L, P, P, P, P, P, P, P, I, P, P, P, I, I, I, I, I, P]),
    "bx_exact_linear_planes": (I, [P, P, L, P, P, P, P, P, P, P, I, P, P, I, I, I, I, I, P]),
    "bx_exact_linear_static_max_bytes": (Z, []),
    "bx_exact_linear_static": (I, [P, L, P, P, P, P, P, P, P, I, P, P, I, I, I, I, I, P]),
    "bx_split_limbs": (I, [P, L, P, I, I, P]),
    "bx_int8_mm": (I, [P, P, P, I, I, I, I, P]),
    "bx_int8_linear_post": (I, [P, P, P, L, P, P, P, P, I, I, I, I, I, P]),
    "bx_exact_norm": (I, [I, P, P, P, P, P, P, P, P, P, P, I, I, I, P]),
    "bx_exact_qkv": (I, [P, P, P, P, P, P, L, L, L, I, P, P, P, I, I, I, I, P]),
    "bx_kv_store": (I, [P, L, L, L, I, P, P, L, L, P, L, L, I, I, I, P]),
    "bx_exact_attn_out": (I, [P, P, P, P, P, I, I, I, P]),
    "bx_exact_silu_quant": (I, [P, P, P, P, P, P, I, I, P]),
    "bx_attention_scratch_bytes": (Z, [I, I]),
    "bx_exact_attention_ws": (I, [P, P, P, P, L, L, L, L, I, P, I, L, I, P, P, L, P, P, I, I, I, I, I, I, P, Z, P]),
    "bx_int8_attention_ws": (I, [P, P, P, L, L, L, L, I, P, I, L, I, P, P, P, P, I, I, I, I, I, I, P, Z, P]),
    "bx_exact_attention": (I, [P, P, P, P, L, L, L, L, I, P, I, L, I, P, P, L, P, P, I, I, I, I, I, I, P]),
    "bx_int8_attention": (I, [P, P, P, L, L, L, L, I, P, I, L, I, P, P, P, P, I, I, I, I, I, I, P]),
    "bx_prefill_attention": (I, [P, P, P, P, I, P, L, L, L, L, I, P, I, L, I, P, L, P, P, P, I, I, I, I, P]),
    "bx_int8_norm": (I, [I, P, P, P, P, P, P, P, P, P, I, I, I, P]),
    "bx_int8_qkv": (I, [P, P, P, P, P, P, L, L, L, I, P, P, P, I, I, I, I, P]),
    "bx_int8_attn_out": (I, [P, P, P, P, P, I, I, I, P]),
    "bx_int8_silu_quant": (I, [P, P, P, P, P, P, I, I, P]),
    "bx_int8_flag_end": (I, [P, P, I, P]),
    "bx_int8_silu_prod": (I, [P, P, P, P, P, I, I, P]),
    "bx_int8_quant_rows": (I, [P, P, P, P, P, I, I, P]),
    "bx_int8_post": (I, [P, P, L, P, P, P, P, I, I, I, P]),
    "bx_pcg_raw": (I, [P, P, I, I, P]),
    "bx_pcg_seed_state": (I, [P, P, I, P]),
    "bx_pcg_raw_from_state": (I, [P, P, I, I, P]),
    "bx_exact_rms": (I, [P, P, P, P, I, I, P]),
    "bx_exact_ndiv": (I, [P, P, P, P, P, P, I, I, P]),
    "bx_rowmax_abs": (I, [P, P, I, I, P]),
    "bx_exact_rope": (I, [P, P, P, P, P, P, P, I, I, I, I, P]),
    "bx_softmax_w": (I, [P, P, P, P, P, L, P, P, P, I, I, P]),
    "bx_exact_attn_div": (I, [P, P, P, I, I, P]),
    "bx_int8_post_acc": (I, [P, P, L, P, P, P, P, I, I, I, P]),
    "bx_exact_silu_prod": (I, [P, P, P, P, P, I, I, P]),
    "bx_exact_quant_rows": (I, [P, P, I, P, L, P, P, L, I, I, P]),
    "bx_bmm": (I, [P, I, P, I, P, I, I, I, I, L, L, L, L, L, L, P]),
    "bx_bmm_limb_scratch_bytes": (Z, [I, I, I, I]),
    "bx_bmm_limb": (I, [P, I, P, I, P, I, I, I, I, L, L, L, L, L, L, P, I, P]),
    "bx_exact_epilogue": (I, [P, P, P, L, P, P, P, I, P, P, P, P, P, I, I, I, P]),
    "bx_sample_scratch_bytes": (Z, [I, I]),
    "bx_sample": (I, [P, L, P, P, P, P, I, I, I, P]),
    "bx_sample_shard": (I, [P, L, P, P, P, P, P, I, I, L, I, P]),
    "bx_decompose_rows": (I, [P, L, P, P, P, P, P, I, I, P]),
    "bx_decompose_residual": (I, [P, L, P, P, P, P, P, P, I, I, P]),
    "bx_logp_scratch_bytes": (Z, [I, I]),
    "bx_logp_pair_table": (I, [P, I, P, P]),
    "bx_int_logp": (I, [P, L, P, P, P, I, P, P, I, I, I, P]),
    "bx_logp_rowmax": (I, [P, L, P, P, I, I, P]),
    "bx_logp_rowsum": (I, [P, L, P, P, I, P, P, I, I, I, P]),
    "bx_logp_finish": (I, [P, P, P, P, I, I, P]),
}



class Epilogue(ctypes.Structure):
    """bxf_epilogue."""
    _fields_ = [("kind", I), ("out_type", I), ("act", I), ("n_main", I), ("act_p", R), ("act_q", R), ("out", P), ("ldo", L),
                ("gso", L), ("side", P), ("lds", L), ("bias", P), ("gate", P), ("ldg", L), ("cs", P), ("rot_out", P),
                ("ldr", L), ("hsr", L), ("rot_dim", I), ("pad_", I), ("main_bias", P)]


class Gru(ctypes.Structure):
    """bxf_gru."""
    _fields_ = [("bias_z", P), ("bias_x", P), ("state", P), ("flags", P), ("seq", P), ("out", P), ("ldo", L)]


class StreamsStep(ctypes.Structure):
    """bxf_streams_step."""
    _fields_ = [("x", P), ("ids", P), ("embed", P), ("vocab", L), ("y", P), ("out", P), ("mix", P), ("in_", P), ("w", P),
                ("h", P), ("ldh", L), ("sum", P), ("eps", R), ("streams", I), ("D", I), ("pad_", I)]


class GqaRows(ctypes.Structure):
    """bxf_gqa_rows."""
    _fields_ = [("y", P), ("ldy", L), ("heads", I), ("kv_heads", I), ("dim", I), ("vdim", I), ("rot_dims", I), ("page", I),
                ("q_norm", P), ("k_norm", P), ("cs", P), ("slot", P), ("q", P), ("ldq", L), ("cache", P), ("ldc", L),
                ("voff", L), ("eps", R), ("pad_", I)]


class Conv(ctypes.Structure):
    """bxf_conv."""
    _fields_ = [("u", P), ("ldu", L), ("w", P), ("b", P), ("state", P), ("flags", P), ("seq", P), ("pos", P),
                ("channels", I), ("taps", I)]


class RecurrenceRows(ctypes.Structure):
    """bxf_recurrence_rows."""
    _fields_ = [("kind", I), ("heads", I), ("groups", I), ("K", I), ("V", I), ("rank", I), ("q0", I), ("k0", I), ("v0", I),
                ("batch", I), ("y", P), ("ldy", L), ("side", P), ("lds", L), ("a2", P), ("a2_b", P), ("inv_tau", R),
                ("q_scale", R), ("decays", P), ("A_log", P), ("skip", P), ("state", P), ("flags", P), ("seq", P), ("out", P), ("ldo", L)]


class ChunkTable(ctypes.Structure):
    """bxf_chunk_table."""
    _fields_ = [("runs", P), ("chunks", P), ("segments", P), ("spans", P), ("nruns", I), ("nchunks", I), ("nsegments", I),
                ("pad_", I)]


class GateRows(ctypes.Structure):
    """bxf_gate_rows."""
    _fields_ = [("o", P), ("z", P), ("ldo", L), ("ldz", L), ("w", P), ("out", P), ("ldout", L), ("n", I), ("parts", I),
                ("wn", I), ("gate_first", I), ("eps", R), ("pad_", I), ("conv", Conv)]


_FLOAT_SIGNATURES = {
    "bxf_version": (I, []),
    "bxf_launch_count": (ctypes.c_longlong, []),
    "bxf_device_status": (I, []),
    "bxf_clear_device_status": (I, []),
    "bxf_set_device_status": (I, [I]),
    "bxf_linear": (I, [I, P, L, L, P, L, L, I, I, I, I, P, ctypes.POINTER(Epilogue), I, P]),
    "bxf_gru_rows": (I, [I]),
    "bxf_gru_chunks": (I, [I]),
    "bxf_gru_linear": (I, [I, P, L, P, L, I, I, I, ctypes.POINTER(Gru), P]),
    "bxf_gru_scan": (I, [I, P, P, I, I, ctypes.POINTER(Gru), P]),
    "bxf_row_flags": (I, [P, P, P, P, I, P]),
    "bxf_norm": (I, [I, P, P, P, L, P, P, P, I, P, P, R, P, L, P, I, I, I, P]),
    "bxf_route": (I, [P, L, I, I, P, P, P, P, I, P]),
    "bxf_gather": (I, [I, P, L, I, P, P, P, I, I, P, P, I, P]),
    "bxf_latent_prepare": (I, [I, P, L, I, I, I, I, P, P, R, P, P, P, P, L, P, L, P, P, I, P]),
    "bxf_latent_attention_scratch": (Z, [I, I, I]),
    "bxf_latent_attention_tile": (I, [I]),
    "bxf_latent_attention": (I, [I, P, L, I, I, I, I, P, L, I, I, P, I, L, I, P, P, P, I, I, P, R, P, L, P, Z, I, P]),
    "bxf_angles": (I, [P, I, P, P, I, P]),
    "bxf_gqa_prepare": (I, [I, ctypes.POINTER(GqaRows), I, P]),
    "bxf_gqa_attention_scratch": (Z, [I, I, I, I]),
    "bxf_gqa_attention": (I, [I, P, L, I, I, I, I, I, P, L, L, I, I, P, I, L, I, P, P, P, I, I, P, R, P, L, P, Z, I, P]),
    "bxf_streams": (I, [I, ctypes.POINTER(StreamsStep), I, P]),
    "bxf_causal_conv": (I, [I, ctypes.POINTER(Conv), P, L, I, P]),
    "bxf_recurrence": (I, [I, ctypes.POINTER(RecurrenceRows), I, P]),
    "bxf_recurrence_chunk_rows": (I, [I, I, I]),
    "bxf_recurrence_chunk_scratch": (Z, [I, I, I, I, I, I, I]),
    "bxf_recurrence_chunks": (I, [I, ctypes.POINTER(RecurrenceRows), ctypes.POINTER(ChunkTable), P, Z, I, P]),
    "bxf_gated_norm": (I, [I, ctypes.POINTER(GateRows), I, P]),
}


def _load(path, signatures):
    if path not in _libs:
        if not os.path.exists(path):
            raise RuntimeError(f"{path} is missing: build it with `python -m bitexact_llm_b200.build` "
                               "(nvcc, sm_100a). There is no fallback path.")
        h = ctypes.CDLL(path)
        for name, (res, args) in signatures.items():
            fn = getattr(h, name)                       # AttributeError if the library is stale
            fn.restype, fn.argtypes = res, args
        _libs[path] = h
    return _libs[path]


def lib():
    return _load(LIB_PATH, _SIGNATURES)


def float_lib():
    return _load(FLOAT_LIB_PATH, _FLOAT_SIGNATURES)


def exported_symbols(float_models=False):
    return sorted(_FLOAT_SIGNATURES if float_models else _SIGNATURES)


def check(rc, what):
    if rc != BX_OK:
        raise RuntimeError(f"{what}: {_ERR.get(rc, rc)}")


def ptr(t):
    """Device pointer of a tensor (None -> NULL)."""
    return None if t is None else t.data_ptr()


def stream():
    import torch
    return torch.cuda.current_stream().cuda_stream


def device_status():
    """Number of device-side waits that gave up since the last clear (synchronises the device)."""
    return lib().bx_device_status()


def float_device_status():
    """`device_status` of the float-model library."""
    return float_lib().bxf_device_status()


def clear_device_status():
    check(lib().bx_clear_device_status(), "bx_clear_device_status")


def i8_tensor_peak(iters=1 << 17, repeats=5):
    """(best, mean) int8 TOPS of a shared-memory-resident tcgen05 kind::i8 loop on the current device."""
    import torch
    out = (ctypes.c_double * 2)()
    check(lib().bx_i8_tensor_peak(iters, repeats, ctypes.cast(out, ctypes.c_void_p), stream()), "bx_i8_tensor_peak")
    torch.cuda.synchronize()
    return out[0], out[1]


class DeviceWaitError(RuntimeError):
    """A bounded device-side wait gave up: kernels launched since then may have left their outputs unwritten."""


def check_device_status(status=device_status):
    """Raises DeviceWaitError when the device status word is non-zero (the state stays set until
    `clear_device_status`)."""
    n = status()
    if n != 0:
        raise DeviceWaitError(f"{n} device-side wait(s) timed out: results since then are not valid; "
                              "call clear_device_status() and rerun the step")
