"""CUDA implementations of the sequence-model ops (`xl/ops/sequence.py`): bf16 models run hand-written kernels throughout;
32-bit models use plain fp32 matrix products (never a reduced-precision matrix mode) and the same kernels for the rest."""
import torch

from ..xl.opdef import native
from ..xl.ops.sequence import SUMSQ_BLOCK
from .native import (_CODE, _c_f, _c_int, _c_ll, _c_p, _check, _count, _ok, _sig, _sms, _stream, gemm,
                     gemm_error_flag)

_stream_dyt = _sig("xl_stream_dyt", _c_p, _c_p, _c_f, _c_p, _c_p, _c_int, _c_p, _c_p, _c_p, _c_p, _c_ll, _c_int, _c_int, _c_p)
_select_dyt = _sig("xl_select_dyt", _c_p, _c_p, _c_int, _c_int, _c_ll, _c_p, _c_p, _c_p, _c_p, _c_int, _c_int, _c_int, _c_p)
_swiglu_packed = _sig("xl_swiglu_packed", _c_p, _c_p, _c_ll, _c_int, _c_int, _c_p)
_advance_by = _sig("xl_advance_by", _c_p, _c_p, _c_int, _c_p)
_min_gru = _sig("xl_min_gru", _c_p, _c_p, _c_p, _c_p, _c_p, _c_p, _c_p, _c_p, _c_int, _c_int, _c_int, _c_int, _c_p)
_min_gru_scratch = _sig("xl_min_gru_scratch", _c_int, _c_int, _c_int, restype=_c_ll)
_rope_append = _sig("xl_diff_rope_append", _c_p, _c_ll, _c_p, _c_p, _c_p, _c_p, _c_p, _c_p, _c_int, _c_int, _c_int, _c_int,
                    _c_int, _c_int, _c_int, _c_int, _c_int, _c_p)
_diff_general = _sig("xl_diff_attn_general", _c_p, _c_ll, _c_p, _c_p, _c_p, _c_ll, _c_p, _c_p, _c_p, _c_int, _c_int, _c_int,
                     _c_int, _c_int, _c_int, _c_int, _c_int, _c_f, _c_f, _c_f, _c_int, _c_p)
_diff_decode = _sig("xl_diff_attn_decode", _c_p, _c_ll, _c_p, _c_p, _c_p, _c_p, _c_p, _c_ll, _c_p, _c_p, _c_p, _c_int, _c_int,
                    _c_int, _c_int, _c_int, _c_int, _c_int, _c_int, _c_f, _c_f, _c_f, _c_int, _c_p, _c_p, _c_p)
_diff_tcgen05 = _sig("xl_diff_attn_tcgen05", _c_p, _c_ll, _c_p, _c_p, _c_p, _c_ll, _c_p, _c_p, _c_p, _c_int, _c_int, _c_int, _c_int,
                     _c_int, _c_int, _c_int, _c_int, _c_f, _c_f, _c_f, _c_p, _c_p)
_stream_rms = _sig("xl_stream_rms", _c_p, _c_p, _c_f, _c_p, _c_p, _c_int, _c_p, _c_f, _c_p, _c_ll, _c_int, _c_int, _c_p)
_select_rms = _sig("xl_select_rms", _c_p, _c_p, _c_int, _c_int, _c_ll, _c_p, _c_f, _c_p, _c_int, _c_int, _c_int, _c_p)
_clamped_glu = _sig("xl_clamped_glu", _c_p, _c_ll, _c_p, _c_ll, _c_ll, _c_int, _c_f, _c_f, _c_f, _c_int, _c_p)
_qk_norm_append = _sig("xl_qk_norm_append", _c_p, _c_ll, _c_p, _c_p, _c_p, _c_p, _c_p, _c_p, _c_p, _c_int, _c_int, _c_int, _c_int,
                       _c_int, _c_int, _c_int, _c_f, _c_int, _c_p)
_WINDOW_ARGS = (_c_p, _c_p, _c_p, _c_p, _c_ll, _c_p, _c_ll, _c_p, _c_p, _c_int, _c_int, _c_int, _c_int, _c_int, _c_int, _c_int,
                _c_int, _c_int, _c_f, _c_f)
_window_general = _sig("xl_window_attn_general", *_WINDOW_ARGS, _c_int, _c_p)
_window_tcgen05 = _sig("xl_window_attn_tcgen05", *_WINDOW_ARGS, _c_p, _c_p)
_window_decode = _sig("xl_window_attn_decode", _c_p, _c_ll, _c_p, _c_p, _c_p, _c_p, _c_p, _c_ll, _c_p, _c_p, _c_int, _c_int, _c_int,
                      _c_int, _c_int, _c_int, _c_int, _c_int, _c_int, _c_f, _c_f, _c_f, _c_int, _c_p, _c_p, _c_p)
_small_m_slots = _sig("xl_linear_small_m_slots", _c_int)
_SMALL_TAIL = (_c_int, _c_int, _c_int, _c_p, _c_p, _c_int, _c_int, _c_p)
_SUMSQ = (_c_p, _c_int, _c_f)  # sums of squares of a deferred norm, parts per row, eps
_small_store = _sig("xl_linear_small_m", _c_p, _c_ll, _c_p, _c_p, _c_ll, _c_int, *_SUMSQ, *_SMALL_TAIL)
_small_split_glu = _sig("xl_linear_small_m_split_glu", _c_p, _c_ll, _c_p, _c_p, _c_ll, _c_int, _c_p, _c_ll, _c_f, _c_f, _c_f, *_SUMSQ,
                        *_SMALL_TAIL)
_small_residual_rms = _sig("xl_linear_small_m_residual_rms", _c_p, _c_ll, _c_p, _c_p, _c_f, _c_p, _c_p, _c_p, *_SMALL_TAIL)
_small_residual = _sig("xl_linear_small_m_residual", _c_p, _c_ll, _c_p, _c_p, _c_f, _c_p, _c_p, _c_int, _c_p, _c_p, _c_p, _c_p,
                       *_SMALL_TAIL)
_small_swiglu = _sig("xl_linear_small_m_swiglu", _c_p, _c_ll, _c_p, _c_p, *_SMALL_TAIL)
_small_min_gru = _sig("xl_linear_small_m_min_gru", _c_p, _c_ll, _c_p, _c_p, _c_p, _c_p, _c_p, _c_p, _c_p, *_SMALL_TAIL)

_MAX_TILES = 1 << 14  # column tiles the split-K counters of the small-M kernel cover
_SCRATCH = {}


def _scratch(device):
    """Per-device scratch of the decoding kernels: partial sums, and counters that every launch leaves at zero. Allocated
    once at its final size, since captured graphs keep the addresses."""
    idx = device.index or 0
    if idx not in _SCRATCH:
        _SCRATCH[idx] = (torch.empty(_small_m_slots(_sms(device)), dtype=torch.float32, device=device),
                         torch.zeros(_MAX_TILES, dtype=torch.int32, device=device),
                         torch.zeros(1 << 16, dtype=torch.int32, device=device))
    return _SCRATCH[idx]


def _small(a, weight) -> bool:
    """Whether the small-M kernels take this product."""
    return (a.dtype == torch.bfloat16 and weight.dtype == torch.bfloat16 and a.shape[0] <= 16 and a.is_cuda
            and a.stride(1) == 1 and weight.is_contiguous() and a.shape[1] % 8 == 0)


def _small_tail(a, rows, weight):
    slots, counters, _ = _scratch(a.device)
    return (a.shape[0], rows, weight.shape[1], slots.data_ptr(), counters.data_ptr(), _MAX_TILES, _sms(a.device), _stream())


def _small_ok(rc, name) -> bool:
    if rc == -1:
        return False
    _check(rc, name)
    _count(name)
    return True


def _ptr(t):
    return t.data_ptr() if t is not None else None


def _f32(*ts) -> bool:
    return all(t is None or t.dtype == torch.float32 for t in ts)


def _i32(*ts) -> bool:
    return all(t is None or (t.is_cuda and t.is_contiguous() and t.dtype == torch.int32) for t in ts)


def _sumsq_args(sumsq, eps):
    return (_ptr(sumsq), sumsq.shape[1] if sumsq is not None else 0, float(eps))


def product(a, weight, out_dtype=None, sumsq=None, eps=0.0):
    """`a (n, K) @ weight (N, K)^T` with 32-bit accumulation: the tcgen05 GEMM for 16-bit operands, the vendor product for
    sizes it does not take and for 32-bit models. `sumsq`: `a` is half of a deferred norm (few rows only, else
    NotImplemented)."""
    out_dtype = out_dtype or a.dtype
    if a.dtype != torch.float32:
        if _small(a, weight) and out_dtype in (torch.bfloat16, torch.float32):
            y = torch.empty((a.shape[0], weight.shape[0]), dtype=out_dtype, device=a.device)
            if _small_ok(_small_store(a.data_ptr(), a.stride(0), weight.data_ptr(), y.data_ptr(), y.stride(0),
                                      int(out_dtype == torch.float32), *_sumsq_args(sumsq, eps),
                                      *_small_tail(a, weight.shape[0], weight)), "linear_small_m"):
                return y
        if sumsq is not None:
            return NotImplemented
        y = gemm(a, weight.t(), out_dtype=out_dtype)
        if y is not NotImplemented:
            return y
        y = torch.mm(a, weight.t())
        return y if y.dtype == out_dtype else y.to(out_dtype)
    if sumsq is not None:
        return NotImplemented
    if torch.backends.cuda.matmul.allow_tf32:
        raise RuntimeError("32-bit models need true fp32 matrix products: set torch.backends.cuda.matmul.allow_tf32 = False")
    return torch.mm(a, weight.t()).to(out_dtype)


def stream_dyt(x, y, mult, tokens, table, norm, out_dtype):
    """One pass over the residual stream: `x += mult * y (+ table[tokens])`, or `x = table[tokens]` without `y`; returns the
    Dynamic Tanh of it when `norm` is given."""
    rows = y.shape[0] if y is not None else tokens.numel()
    cols = x.shape[1]
    if not _ok(x, y, table) or not _f32(x, *(norm or ())) or not _i32(tokens) or rows > x.shape[0]:
        return NotImplemented
    alpha, w, b = norm if norm is not None else (None, None, None)
    if norm is not None and not _ok(w, b):
        return NotImplemented
    h = torch.empty((rows, cols), dtype=out_dtype, device=x.device) if norm is not None else None
    rc = _stream_dyt(x.data_ptr(), _ptr(y), float(mult), _ptr(tokens), _ptr(table), table.shape[0] if table is not None else 0,
                     _ptr(alpha), _ptr(w), _ptr(b), _ptr(h), rows, cols, _CODE[out_dtype], _stream())
    if rc == -1:
        return NotImplemented
    _check(rc, "stream_dyt")
    _count("stream_dyt")
    return h if norm is not None else ()


@native("embed_dyt_")
def embed_dyt_cuda(x, tokens, table, alpha, w, b):
    return stream_dyt(x, None, 0.0, tokens.reshape(-1), table, (alpha, w, b), table.dtype)


@native("linear_residual_dyt_")
def linear_residual_dyt_cuda(x, a, weight, *rest, mult, has_norm, has_inject):
    norm = rest[:3] if has_norm else None
    tokens, table = rest[-2:] if has_inject else (None, None)
    if (_small(a, weight) and x.dtype == torch.float32 and x.is_contiguous() and a.shape[0] <= x.shape[0]
            and (tokens is None or (_i32(tokens) and table.dtype == a.dtype and table.is_contiguous())) and _f32(*(norm or ()))):
        h = torch.empty((a.shape[0], x.shape[1]), dtype=a.dtype, device=a.device) if has_norm else None
        alpha, nw, nb = norm or (None, None, None)
        rc = _small_residual(a.data_ptr(), a.stride(0), weight.data_ptr(), x.data_ptr(), float(mult), _ptr(tokens), _ptr(table),
                             table.shape[0] if has_inject else 0, _ptr(alpha), _ptr(nw), _ptr(nb), _ptr(h),
                             *_small_tail(a, weight.shape[0], weight))
        if _small_ok(rc, "linear_small_m_residual"):
            return h if has_norm else ()
    y = product(a, weight)
    return stream_dyt(x, y, mult, tokens.reshape(-1) if tokens is not None else None, table, norm, a.dtype)


@native("select_dyt")
def select_dyt_cuda(x, idx, alpha, w, b, stride, offset, out_dtype):
    if not _ok(x) or not _f32(x, alpha, w, b) or not _i32(idx):
        return NotImplemented
    h = torch.empty((idx.shape[0], x.shape[1]), dtype=out_dtype, device=x.device)
    rc = _select_dyt(x.data_ptr(), idx.data_ptr(), stride, offset, x.shape[0], alpha.data_ptr(), w.data_ptr(), b.data_ptr(),
                     h.data_ptr(), idx.shape[0], x.shape[1], _CODE[out_dtype], _stream())
    if rc == -1:
        return NotImplemented
    _check(rc, "select_dyt")
    _count("select_dyt")
    return h


@native("linear_rows")
def linear_rows_cuda(a, weight, *sumsq, out_dtype, eps=0.0):
    return product(a, weight, out_dtype, sumsq[0] if sumsq else None, eps)


@native("linear_swiglu")
def linear_swiglu_cuda(h, weight):
    f = weight.shape[0] // 2
    if _small(h, weight):
        y = torch.empty((h.shape[0], f), dtype=h.dtype, device=h.device)
        if _small_ok(_small_swiglu(h.data_ptr(), h.stride(0), weight.data_ptr(), y.data_ptr(), *_small_tail(h, f, weight)),
                     "linear_small_m_swiglu"):
            return y
    gu = product(h, weight)
    y = torch.empty((h.shape[0], f), dtype=h.dtype, device=h.device)
    rc = _swiglu_packed(gu.data_ptr(), y.data_ptr(), h.shape[0], f, _CODE[h.dtype], _stream())
    _check(rc, "swiglu_packed")
    _count("swiglu_packed")
    return y


@native("min_gru_")
def min_gru_cuda(h, weight, bz, bx, state, pos, count, T):
    B, width = state.shape
    if not _f32(bz, bx, state) or not _i32(pos, count) or not state.is_contiguous() or h.shape[0] != B * T:
        return NotImplemented
    y = torch.empty((B * T, width), dtype=h.dtype, device=h.device)
    if T == 1 and _small(h, weight):
        rc = _small_min_gru(h.data_ptr(), h.stride(0), weight.data_ptr(), bz.data_ptr(), bx.data_ptr(), state.data_ptr(),
                            pos.data_ptr(), count.data_ptr(), y.data_ptr(), *_small_tail(h, width, weight))
        if _small_ok(rc, "linear_small_m_min_gru"):
            return y
    zxg = product(h, weight)
    pairs = torch.empty(_min_gru_scratch(B, T, width), dtype=torch.float32, device=h.device)
    rc = _min_gru(zxg.data_ptr(), bz.data_ptr(), bx.data_ptr(), state.data_ptr(), y.data_ptr(), pairs.data_ptr(), pos.data_ptr(),
                  count.data_ptr(), B, T, width, _CODE[h.dtype], _stream())
    if rc == -1:
        return NotImplemented
    _check(rc, "min_gru")
    _count("min_gru")
    return y


@native("diff_attention_")
def diff_attention_cuda(qkv, cos, sin, kc, vc, pos, count, lam, T, heads, rotary_dim, chunk, scale, eps, out_scale):
    B, G, _, smax, dim = kc.shape
    vdim = vc.shape[-1]
    if not _ok(qkv, kc, vc) or not (qkv.dtype == kc.dtype == vc.dtype) or not _f32(cos, sin, lam) or not _i32(pos, count):
        return NotImplemented
    if qkv.shape != (B * T, (heads + G) * 2 * dim + G * vdim) or (rotary_dim and cos.shape[0] < smax):
        return NotImplemented
    code, s = _CODE[qkv.dtype], _stream()
    out = torch.empty((B * T, heads * vdim), dtype=qkv.dtype, device=qkv.device)
    if T == 1 and qkv.dtype == torch.bfloat16 and dim % 8 == 0 and vdim % 8 == 0 and dim <= 128 and vdim <= 256:
        units = B * G * ((heads // G + 7) // 8)
        longest = min(smax, chunk) if chunk else smax
        splits = max(1, min(2 * _sms(qkv.device) // units, (longest + 63) // 64, 64))  # one wave, two CTAs per SM
        counters = _scratch(qkv.device)[2]
        part = torch.empty(units * splits * 16 * (vdim + 2), dtype=torch.float32, device=qkv.device) if splits > 1 else None
        if units <= counters.numel():
            rc = _diff_decode(qkv.data_ptr(), qkv.stride(0), _ptr(cos), _ptr(sin), kc.data_ptr(), vc.data_ptr(), out.data_ptr(),
                              out.stride(0), pos.data_ptr(), count.data_ptr(), lam.data_ptr(), B, heads, G, dim, vdim,
                              rotary_dim, smax, chunk, float(scale), float(eps), float(out_scale), splits, _ptr(part),
                              counters.data_ptr(), s)
            if _small_ok(rc, "diff_attn_decode"):
                return out
    rc = _rope_append(qkv.data_ptr(), qkv.stride(0), _ptr(cos), _ptr(sin), kc.data_ptr(), vc.data_ptr(), pos.data_ptr(),
                      count.data_ptr(), B, T, heads, G, dim, vdim, rotary_dim, smax, code, s)
    if rc == -1:
        return NotImplemented
    _check(rc, "diff_rope_append")
    _count("diff_rope_append")
    if qkv.dtype == torch.bfloat16:
        rc = _diff_tcgen05(qkv.data_ptr(), qkv.stride(0), kc.data_ptr(), vc.data_ptr(), out.data_ptr(), out.stride(0),
                           pos.data_ptr(), count.data_ptr(), lam.data_ptr(), B, T, heads, G, dim, vdim, smax, chunk, float(scale),
                           float(eps), float(out_scale), gemm_error_flag(qkv.device).data_ptr(), s)
        if rc >= 0:
            _check(rc, "diff_attn_tcgen05")
            _count("diff_attn_tcgen05")
            return out
    rc = _diff_general(qkv.data_ptr(), qkv.stride(0), kc.data_ptr(), vc.data_ptr(), out.data_ptr(), out.stride(0),
                       pos.data_ptr(), count.data_ptr(), lam.data_ptr(), B, T, heads, G, dim, vdim, smax, chunk, float(scale),
                       float(eps), float(out_scale), code, s)
    _check(rc, "diff_attn_general")
    _count("diff_attn_general")
    return out


def stream_rms(x, y, mult, tokens, table, w, eps, out_dtype):
    """One pass over the residual stream: `x += mult * y`, or `x = mult * table[tokens]` without `y`; returns the RMS norm of
    it when its factors `w` are given."""
    rows, cols = y.shape[0] if y is not None else tokens.numel(), x.shape[1]
    if not _ok(x, y, table, w) or not _f32(x, w) or not _i32(tokens) or rows > x.shape[0]:
        return NotImplemented
    h = torch.empty((rows, cols), dtype=out_dtype, device=x.device) if w is not None else None
    rc = _stream_rms(x.data_ptr(), _ptr(y), float(mult), _ptr(tokens), _ptr(table), table.shape[0] if table is not None else 0,
                     _ptr(w), float(eps), _ptr(h), rows, cols, _CODE[out_dtype], _stream())
    if rc == -1:
        return NotImplemented
    _check(rc, "stream_rms")
    _count("stream_rms")
    return h if w is not None else ()


@native("embed_rms_")
def embed_rms_cuda(x, tokens, table, w, scale, eps):
    return stream_rms(x, None, scale, tokens.reshape(-1), table, w, eps, table.dtype)


@native("linear_residual_rms_")
def linear_residual_rms_cuda(x, a, weight, *norm, mult, eps, deferred):
    w = norm[0] if norm else None
    if (_small(a, weight) and (deferred or w is None) and _f32(x, w) and x.is_contiguous() and a.shape[0] <= x.shape[0]):
        n, cols = a.shape[0], x.shape[1]
        h = torch.empty((n, cols), dtype=a.dtype, device=a.device) if deferred else None
        sumsq = torch.empty((n, -(-cols // SUMSQ_BLOCK)), dtype=torch.float32, device=a.device) if deferred else None
        rc = _small_residual_rms(a.data_ptr(), a.stride(0), weight.data_ptr(), x.data_ptr(), float(mult), _ptr(w), _ptr(h),
                                 _ptr(sumsq), *_small_tail(a, weight.shape[0], weight))
        if _small_ok(rc, "linear_small_m_residual"):
            return (h, sumsq) if deferred else ()
    if deferred:
        return NotImplemented
    return stream_rms(x, product(a, weight), mult, None, None, w, eps, a.dtype)


@native("select_rms")
def select_rms_cuda(x, idx, w, stride, offset, eps, out_dtype):
    if not _ok(x) or not _f32(x, w) or not _i32(idx):
        return NotImplemented
    h = torch.empty((idx.shape[0], x.shape[1]), dtype=out_dtype, device=x.device)
    rc = _select_rms(x.data_ptr(), idx.data_ptr(), stride, offset, x.shape[0], w.data_ptr(), float(eps), h.data_ptr(),
                     idx.shape[0], x.shape[1], _CODE[out_dtype], _stream())
    if rc == -1:
        return NotImplemented
    _check(rc, "select_rms")
    _count("select_rms")
    return h


@native("linear_split_glu")
def linear_split_glu_cuda(h, weight, *sumsq, cols, lead, limit, slope, shift, eps=0.0):
    n, N = h.shape[0], weight.shape[0]
    f, sq = (N - cols) // 2, sumsq[0] if sumsq else None
    joint = torch.empty((n, lead + f), dtype=h.dtype, device=h.device)
    unit = joint.data_ptr() + lead * joint.element_size()
    if _small(h, weight):
        proj = torch.empty((n, cols), dtype=h.dtype, device=h.device)
        rc = _small_split_glu(h.data_ptr(), h.stride(0), weight.data_ptr(), proj.data_ptr(), cols, cols, unit, lead + f, limit,
                              slope, shift, *_sumsq_args(sq, eps), *_small_tail(h, N, weight))
        if _small_ok(rc, "linear_small_m_split_glu"):
            return proj, joint
    y = product(h, weight, None, sq, eps)
    if y is NotImplemented:
        return NotImplemented
    if f:
        rc = _clamped_glu(y.data_ptr() + cols * y.element_size(), N, unit, lead + f, n, f, limit, slope, shift, _CODE[h.dtype],
                          _stream())
        _check(rc, "clamped_glu")
        _count("clamped_glu")
    return y[:, :cols], joint


@native("window_attention_")
def window_attention_cuda(proj, q_norm, k_norm, kc, vc, pos, count, joint, T, heads, window, keep_first, scale, sink, eps):
    B, G, smax, dim = kc.shape
    vdim = vc.shape[-1]
    plain = (heads + G) * dim + G * vdim
    gated = proj.shape[1] > plain
    if not _ok(kc, vc, joint) or not (proj.dtype == kc.dtype == vc.dtype == joint.dtype) or not _f32(q_norm, k_norm):
        return NotImplemented
    if not _i32(pos, count) or proj.stride(1) != 1 or proj.shape != (B * T, plain + (heads * vdim if gated else 0)):
        return NotImplemented
    code, s, ld, ldo = _CODE[proj.dtype], _stream(), proj.stride(0), joint.stride(0)
    sink = float("-inf") if sink is None else sink
    if T == 1 and proj.dtype == torch.bfloat16:
        units = B * G * ((heads // G + 15) // 16)
        longest = min(smax, window + keep_first) if window else smax
        # one wave, two CTAs per SM; a slice of fewer keys costs more in the merge than it saves
        splits = max(1, min(2 * _sms(proj.device) // units, (longest + 383) // 384, 64))
        counters = _scratch(proj.device)[2]
        part = torch.empty(units * splits * 16 * (vdim + 2), dtype=torch.float32, device=proj.device) if splits > 1 else None
        if units <= counters.numel():
            rc = _window_decode(proj.data_ptr(), ld, q_norm.data_ptr(), k_norm.data_ptr(), kc.data_ptr(), vc.data_ptr(),
                                joint.data_ptr(), ldo, pos.data_ptr(), count.data_ptr(), B, heads, G, dim, vdim, smax, window,
                                keep_first, int(gated), scale, sink, eps, splits, _ptr(part), counters.data_ptr(), s)
            if _small_ok(rc, "window_attn_decode"):
                return joint
    qn = torch.empty((B, G, T, heads // G, dim), dtype=proj.dtype, device=proj.device)
    rc = _qk_norm_append(proj.data_ptr(), ld, q_norm.data_ptr(), k_norm.data_ptr(), qn.data_ptr(), kc.data_ptr(), vc.data_ptr(),
                         pos.data_ptr(), count.data_ptr(), B, T, heads, G, dim, vdim, smax, eps, code, s)
    if rc == -1:
        return NotImplemented
    _check(rc, "qk_norm_append")
    _count("qk_norm_append")
    args = (qn.data_ptr(), kc.data_ptr(), vc.data_ptr(), proj.data_ptr() + plain * proj.element_size() if gated else None, ld,
            joint.data_ptr(), ldo, pos.data_ptr(), count.data_ptr(), B, T, heads, G, dim, vdim, smax, window, keep_first, scale,
            sink)
    if proj.dtype == torch.bfloat16:
        rc = _window_tcgen05(*args, gemm_error_flag(proj.device).data_ptr(), s)
        if rc >= 0:
            _check(rc, "window_attn_tcgen05")
            _count("window_attn_tcgen05")
            return joint
    _check(_window_general(*args, code, s), "window_attn_general")
    _count("window_attn_general")
    return joint


@native("advance_by_")
def advance_by_cuda(pos, count):
    if not _i32(pos, count):
        return NotImplemented
    _check(_advance_by(pos.data_ptr(), count.data_ptr(), pos.numel(), _stream()), "advance_by")
    _count("advance_by")
    return pos

