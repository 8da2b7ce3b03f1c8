"""ctypes bindings of libfloatops.so, the kernels of the floating-point decoder designs (include/zkds_float.h).

Tensors go in as torch CUDA tensors; every call is launched on torch's current stream and its status is checked.
There is no CPU or PyTorch fallback: a missing library raises at import, a failed launch raises `FloatOpsError`.
"""
import ctypes
import os

import torch

_HERE = os.path.dirname(os.path.abspath(__file__))
F32, BF16 = 0, 1
STORE, ROTATE, GATE, GLU = 0, 1, 2, 3


def _find_library():
    path = os.environ.get("ZKDS_FLOAT_LIB") or os.path.join(_HERE, "libfloatops.so")
    if not os.path.exists(path):
        raise OSError("libfloatops.so not found (looked at %s); build it with `python zk-deepseek_b200/build.py "
                      "libfloatops.so`" % path)
    return path


lib = ctypes.CDLL(_find_library())
_vp, _ll, _i, _f, _d = ctypes.c_void_p, ctypes.c_longlong, ctypes.c_int, ctypes.c_float, ctypes.c_double


class LinearArgs(ctypes.Structure):
    _fields_ = [("A", _vp), ("W", _vp), ("out", _vp), ("aux", _vp), ("table", _vp), ("start", _vp),
                ("lda", _ll), ("ldw", _ll), ("ldo", _ll), ("ldaux", _ll), ("M", _ll), ("N", _ll), ("K", _ll),
                ("seq", _ll), ("positions", _ll), ("dtype", _i), ("out_dtype", _i), ("epilogue", _i), ("pairs", _i), ("period", _i),
                ("offset", _i), ("rot_begin", _i), ("rot_end", _i), ("bias", _vp), ("out2", _vp), ("ldo2", _ll), ("split", _ll)]


class LatentArgs(ctypes.Structure):
    _fields_ = [("y", _vp), ("wq", _vp), ("wc", _vp), ("cq", _vp), ("cache", _vp), ("table", _vp), ("start", _vp),
                ("slots", _vp), ("ldy", _ll), ("ldq", _ll), ("rows", _ll), ("seq", _ll), ("slot_stride", _ll),
                ("pitch", _ll), ("capacity", _ll), ("q_rank", _i), ("q_pad", _i), ("c", _i), ("c_pad", _i),
                ("pairs", _i), ("own_kv", _i), ("dtype", _i), ("eps", _d)]


class PerHeadArgs(ctypes.Structure):
    _fields_ = [("x", _vp), ("W", _vp), ("out", _vp), ("x_tok", _ll), ("x_head", _ll), ("o_tok", _ll),
                ("o_head", _ll), ("w_head", _ll), ("ldw", _ll), ("tokens", _ll), ("heads", _ll), ("n_out", _i),
                ("n_in", _i), ("transposed", _i), ("dtype", _i), ("copy_from", _i), ("copy_to", _i), ("copy_n", _i)]


class AttentionArgs(ctypes.Structure):
    _fields_ = [("q", _vp), ("k1", _vp), ("k2", _vp), ("v", _vp), ("out", _vp), ("start", _vp), ("slots", _vp),
                ("scratch", _vp), ("q_head", _ll), ("o_head", _ll), ("k1_tok", _ll), ("k1_head", _ll),
                ("k2_tok", _ll), ("v_tok", _ll), ("v_head", _ll), ("slot_stride", _ll), ("base", _ll),
                ("keys", _ll), ("batch", _ll), ("seq", _ll), ("heads", _ll), ("d1", _i), ("d2", _i), ("dv", _i),
                ("window", _i), ("shared", _i), ("dtype", _i), ("scale", _f), ("max_keys", _i), ("heads_per_kv", _i),
                ("gate", _vp), ("gate_tok", _ll), ("gate_head", _ll), ("o_tok", _ll), ("out_scale", _f)]


class HeadsArgs(ctypes.Structure):
    _fields_ = [("y", _vp), ("wq", _vp), ("wk", _vp), ("q", _vp), ("cache", _vp), ("table", _vp), ("start", _vp),
                ("slots", _vp), ("ldy", _ll), ("q_col", _ll), ("k_col", _ll), ("rows", _ll), ("seq", _ll),
                ("slot_stride", _ll), ("pitch", _ll), ("capacity", _ll), ("heads", _i), ("kv_heads", _i), ("d", _i),
                ("dim", _i), ("pairs", _i), ("dtype", _i), ("eps", _d)]


class GroupedArgs(ctypes.Structure):
    _fields_ = [("q", _vp), ("cache", _vp), ("out", _vp), ("gate", _vp), ("start", _vp), ("slots", _vp), ("scratch", _vp),
                ("slot_stride", _ll), ("pitch", _ll), ("capacity", _ll), ("v_off", _ll), ("o_tok", _ll), ("gate_tok", _ll),
                ("batch", _ll), ("seq", _ll), ("heads", _i), ("kv_heads", _i), ("d", _i), ("window", _i), ("max_keys", _i),
                ("dtype", _i), ("scale", _f), ("out_scale", _f)]


class ConvArgs(ctypes.Structure):
    _fields_ = [("x", _vp), ("w", _vp), ("b", _vp), ("out", _vp), ("state", _vp), ("start", _vp), ("slots", _vp),
                ("ldx", _ll), ("ldo", _ll), ("batch", _ll), ("seq", _ll), ("n_slots", _ll), ("channels", _i), ("taps", _i),
                ("dtype", _i)]


class ScanArgs(ctypes.Structure):
    _fields_ = [("q", _vp), ("k", _vp), ("v", _vp), ("out", _vp), ("decay", _vp), ("step", _vp), ("step_bias", _vp),
                ("skip", _vp), ("state", _vp), ("scratch", _vp), ("start", _vp), ("slots", _vp), ("q_tok", _ll),
                ("k_tok", _ll), ("v_tok", _ll), ("o_tok", _ll), ("qk_head", _ll), ("v_head", _ll), ("o_head", _ll),
                ("step_tok", _ll), ("batch", _ll), ("seq", _ll), ("heads", _ll), ("n_slots", _ll), ("heads_per_qk", _i),
                ("n", _i), ("p", _i), ("dtype", _i), ("k_scale", _f)]


class GatedNormArgs(ctypes.Structure):
    _fields_ = [("x", _vp), ("g", _vp), ("weight", _vp), ("out", _vp), ("ldx", _ll), ("ldg", _ll), ("ldo", _ll), ("rows", _ll),
                ("heads", _i), ("vdim", _i), ("p", _i), ("part", _i), ("dtype", _i), ("scale", _f), ("eps", _d)]


def _sig(name, argtypes, restype=_i):
    fn = getattr(lib, name)
    fn.argtypes, fn.restype = argtypes, restype
    return fn


_linear = _sig("zkfp_linear", [ctypes.POINTER(LinearArgs), _vp])
_latent = _sig("zkfp_latent_post", [ctypes.POINTER(LatentArgs), _vp])
_perhead = _sig("zkfp_perhead", [ctypes.POINTER(PerHeadArgs), _vp])
_attention = _sig("zkfp_attention", [ctypes.POINTER(AttentionArgs), _vp])
_scratch = _sig("zkfp_attention_scratch", [ctypes.POINTER(AttentionArgs)], _ll)
linear_path = _sig("zkfp_linear_path", [ctypes.POINTER(LinearArgs)])
attention_path = _sig("zkfp_attention_path", [ctypes.POINTER(AttentionArgs)])
_heads_post = _sig("zkfp_heads_post", [ctypes.POINTER(HeadsArgs), _vp])
_grouped = _sig("zkfp_grouped_attention", [ctypes.POINTER(GroupedArgs), _vp])
_grouped_scratch = _sig("zkfp_grouped_scratch", [ctypes.POINTER(GroupedArgs)], _ll)
_conv = _sig("zkfp_short_conv", [ctypes.POINTER(ConvArgs), _vp])
_scan = _sig("zkfp_scan", [ctypes.POINTER(ScanArgs), _vp])
_scan_scratch = _sig("zkfp_scan_scratch", [ctypes.POINTER(ScanArgs)], _ll)
scan_path = _sig("zkfp_scan_path", [ctypes.POINTER(ScanArgs)])
_gated_norm = _sig("zkfp_gated_norm", [ctypes.POINTER(GatedNormArgs), _vp])
_embed = _sig("zkfp_embed", [_vp, _vp, _ll, _ll, _vp, _vp, _ll, _ll, _f, _i, _vp])
_add_norm = _sig("zkfp_add_norm", [_vp, _vp, _vp, _vp, _vp, _ll, _ll, _ll, _ll, _d, _i, _vp])
_norm_rows = _sig("zkfp_norm_rows", [_vp, _ll, _vp, _vp, _vp, _ll, _ll, _ll, _d, _i, _vp])
_sig("zkfp_device_status", [])
launches = _sig("zkfp_launches", [], _ll)
_sig("zkfp_cuda_error", [])


class FloatOpsError(RuntimeError):
    def __init__(self, message, status=0):
        super().__init__(message)
        self.status = status


def _check(status, what):
    if status:
        text = {1: "bad argument", 3: "CUDA error %d" % lib.zkfp_cuda_error(), 5: "a bounded wait ran out",
                6: "unsupported shape"}.get(status, "status %d" % status)
        raise FloatOpsError("%s: %s" % (what, text), status)


def _stream():
    return torch.cuda.current_stream().cuda_stream


def device_status(sync=False):
    """raises if a finished kernel gave up a bounded wait"""
    if sync:
        torch.cuda.current_stream().synchronize()
    _check(lib.zkfp_device_status(), "device status")


class Recording:
    """Calls made while recording, with their argument structures and the tensors they point to, to be issued again
    without rebuilding anything: the host side of a one-token step is a loop over prepared calls."""

    active = None

    def __init__(self):
        self.calls, self.held = [], []

    def __enter__(self):
        Recording.active = self
        return self

    def __exit__(self, *exc):
        Recording.active = None
        return False

    def replay(self):
        st = _stream()
        for fn, args, what in self.calls:
            rc = fn(*args, st)
            if rc:
                _check(rc, what)


def _call(fn, args, what, *tensors):
    _check(fn(*args, _stream()), what)
    if Recording.active is not None:
        Recording.active.calls.append((fn, args, what))
        Recording.active.held.extend(tensors)


def code(dtype):
    return BF16 if dtype == torch.bfloat16 else F32


def pad8(n):
    return (n + 7) // 8 * 8


def ptr(t):
    return None if t is None else t.data_ptr()


def embed(tokens, table, vocab, x, xb, scale=1.0):
    """x [rows, pitch] = scale * table[tokens] in 32-bit, xb the same in bfloat16 (None: not wanted)"""
    _call(_embed, (tokens.data_ptr(), table.data_ptr(), table.stride(0), vocab, x.data_ptr(), ptr(xb), x.stride(0),
                   x.shape[0], scale, code(table.dtype)), "embed", tokens, table, x, xb)


def add_norm(x, y, w, h, width, eps, w2=None):
    """x += w * y / rms(y); h (None: not wanted) = x or, with w2, w2 * x / rms(x)"""
    _call(_add_norm, (x.data_ptr(), y.data_ptr(), w.data_ptr(), ptr(w2), ptr(h), x.stride(0), y.stride(0), x.shape[0],
                      width, eps, code(h.dtype) if h is not None else F32), "add_norm", x, y, w, w2, h)


def norm_rows(x, index, w, out, width, eps):
    """out[i] = w * x[index[i]] / rms(x[index[i]]); index None takes every row"""
    _call(_norm_rows, (x.data_ptr(), x.stride(0), ptr(index), w.data_ptr(), out.data_ptr(), out.stride(0), out.shape[0],
                       width, eps, code(out.dtype)), "norm_rows", x, index, w, out)


def linear(A, W, out, epilogue=STORE, aux=None, table=None, start=None, seq=1, pairs=0, period=0, offset=0,
           rotated=(0, 0), bias=None, out2=None):
    """out = epilogue(A W^T + bias); A [M, K], W [N, K], out [M, N] (N / 2 columns with GLU).  out2: the last
    out2.shape[1] columns go there in 32-bit; rotated: the columns that turn, (0, 0) for all."""
    a = LinearArgs(A.data_ptr(), W.data_ptr(), out.data_ptr(), ptr(aux), ptr(table), ptr(start), A.stride(0),
                   W.stride(0), out.stride(0), aux.stride(0) if aux is not None else 0, A.shape[0], W.shape[0],
                   W.shape[1], seq, table.shape[0] if table is not None else 0, code(A.dtype), code(out.dtype),
                   epilogue, pairs, period, offset, rotated[0], rotated[1], ptr(bias), ptr(out2),
                   out2.stride(0) if out2 is not None else 0, W.shape[0] - out2.shape[1] if out2 is not None else 0)
    _call(_linear, (ctypes.byref(a),), "linear", A, W, out, aux, table, start, bias, out2)
    return out


def latent_post(args, *tensors):
    _call(_latent, (ctypes.byref(args),), "latent_post", *tensors)


def perhead(x, W, out, transposed, copy=(0, 0, 0)):
    """per-head products: x [tokens, heads, n_in], W [heads, rows, cols], out [tokens, heads, n_out] (strided views,
    last dimension contiguous).  transposed: out = x W (rows = n_in); otherwise out = x W^T (cols = n_in)."""
    n_out, n_in = (W.shape[2], W.shape[1]) if transposed else (W.shape[1], W.shape[2])
    a = PerHeadArgs(x.data_ptr(), W.data_ptr(), out.data_ptr(), x.stride(0), x.stride(1), out.stride(0),
                    out.stride(1), W.stride(0), W.stride(1), x.shape[0], x.shape[1], n_out, n_in, int(transposed),
                    code(x.dtype), *copy)
    _call(_perhead, (ctypes.byref(a),), "perhead", x, W, out)


def attention(args, *tensors):
    _call(_attention, (ctypes.byref(args),), "attention", *tensors)


def attention_scratch(args):
    return int(_scratch(ctypes.byref(args)))


def heads_post(args, *tensors):
    _call(_heads_post, (ctypes.byref(args),), "heads_post", *tensors)


def _with_scratch(fn, size, args, what, device, tensors):
    n = int(size(ctypes.byref(args)))
    scratch = torch.empty(n, dtype=torch.float32, device=device) if n else None
    args.scratch = ptr(scratch)
    _call(fn, (ctypes.byref(args),), what, scratch, *tensors)


def grouped_attention(args, device, *tensors):
    _with_scratch(_grouped, _grouped_scratch, args, "grouped_attention", device, tensors)


def short_conv(args, *tensors):
    _call(_conv, (ctypes.byref(args),), "short_conv", *tensors)


def scan(args, device, *tensors):
    _with_scratch(_scan, _scan_scratch, args, "scan", device, tensors)


def gated_norm(args, *tensors):
    _call(_gated_norm, (ctypes.byref(args),), "gated_norm", *tensors)
