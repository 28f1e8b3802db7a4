"""ctypes mirrors of the structures that kernel launchers take (include/logismos_kernels.h)."""
import ctypes as C

from ._lib import f32, i32, vp


def _ints(*names):
    return [(n, i32) for n in names]


def _pointers(*names):
    return [(n, vp) for n in names]


class Groups(C.Structure):
    _fields_ = [("n_groups", i32), ("end", i32 * 8), ("n_main", i32), ("tail", vp), ("ld_tail", i32), ("tail_cap", f32), ("tail_parts", vp), ("bias", vp),
                ("silu_begin", i32), ("silu_end", i32)]


class TimeMix(C.Structure):
    _fields_ = _pointers("proj") + _ints("ld", "off_r", "off_k", "off_v", "off_g") + [("z", vp), ("ld_z", i32), ("low", vp), ("ld_low", i32), ("w2", vp),
               ("ld_w2", i32), ("rank", i32)] + _pointers("w0", "u", "gain", "state", "state_slots", "fresh", "cu", "out") + _ints("ld_out", "heads", "d", "dp") + [
               ("scale", f32), ("eps", f32), ("mode", i32), ("vp", i32), ("tau", f32), ("q_scale", f32)]


class Ssd(C.Structure):
    _fields_ = [("proj", vp), ("ld", i32), ("dt", vp), ("ld_dt", i32)] + _pointers("conv_w", "conv_b", "conv_state") + _ints("taps") + _pointers(
               "dt_bias", "log_a", "skip", "state", "state_slots", "fresh", "phase", "cu", "y") + _ints("ld_y", "heads", "groups", "np", "vp") + [("xbc", vp), ("ld_xbc", i32), ("decay", vp)]


class ScoreBias(C.Structure):
    _fields_ = [("scale", f32), ("cap", f32), ("bias", vp), ("far", i32), ("max_abs_bias", f32), ("max_abs_qk", f32), ("gate", vp), ("ld_gate", i32), ("gate_scale", f32)]


class Window(C.Structure):
    _fields_ = [("scale", f32)] + _ints("size", "keep_first", "sink") + [("gate", vp), ("ld_gate", i32)] + _ints("chunked", "pool") + _pointers("k_mean", "v_mean") + [("out_f32", i32)]


class LatentRotary(C.Structure):
    _fields_ = _pointers("table", "positions") + _ints("at", "dims") + [("gate", vp)] + _ints("n_gate", "ld_gate")


class TanhNorm(C.Structure):
    _fields_ = [("alpha", f32)] + _pointers("w", "b")


class MixtureOut(C.Structure):
    _fields_ = _pointers("rows", "pair_row", "weights", "identity") + _ints("n_pairs", "top") + [("counts", vp), ("n_counts", i32)]


class MoeRoute(C.Structure):
    _fields_ = [("logits", vp)] + _ints("ld", "zero_logits") + [("correction", vp)] + _ints("n_experts", "n_identity", "top", "n_always") + _pointers(
               "weights", "pair_row", "identity", "offsets", "row_token", "counts", "pair_expert", "tiles", "n_tiles", "h", "w") + [("width", i32), ("arrived", vp)] + _ints("scoring", "groups", "keep_groups")


class HeadNorm(C.Structure):
    _fields_ = [("qkv", vp)] + _ints("ld", "rows", "heads", "n_kv", "maps", "hd", "dim") + _pointers("gain_q", "gain_k") + [("eps", f32), ("table", vp), ("rot_dims", i32),
               ("q_out", vp), ("ld_q", i32)] + _pointers("k_pool", "v_pool", "slots", "positions") + [("n_pool_slots", C.c_int64)] + _ints("pool", "pool_rows") + _pointers(
               "k_mean", "v_mean", "tables", "seq_ids") + _ints("max_blocks", "n_pool_blocks")


class GatedResidual(C.Structure):
    _fields_ = [("x", vp), ("branch", vp * 2), ("zero_branches", i32), ("branch_gain", vp * 2), ("mixture", C.POINTER(MixtureOut)), ("gate", vp), ("ld_gate", i32)] + _pointers(
               "kept", "embed", "ids", "step") + [("vocab", i32), ("h", vp), ("gain", f32), ("eps", f32), ("row_idx", vp)] + _ints("n_src_rows", "rows", "n", "ld", "is_f32")
