"""Ops of sequence models served with per-sequence state: a 32-bit residual stream, Dynamic Tanh and RMS norms, gated linear
recurrences, differential attention and sliding-window attention against a cache.

A *portion* holds the next tokens of every sequence of a batch: `(batch * T)` rows, sequence-major, of which the first
`count[b]` rows of sequence `b` are real and the rest is padding. `pos[b]` is the position of its first row. Both live on the
device, so a portion of a given `T` is a fixed program (and `T = 1` is the decoding step). State is updated in place, only by
the real rows; a sequence at position 0 starts from the empty state whatever its slot held before.

An RMS norm needs a whole row before its first output. Where the rows are few the ops can leave it half done (*deferred*):
the stream update returns `x * w` together with sums of squares over blocks of `SUMSQ_BLOCK` columns, and the product that
reads it multiplies its results by `1 / sqrt(mean(x^2) + eps)`.

No counterpart in the reference (it ships no recurrent layers, cache or generation loop).
"""
from typing import Optional, Sequence, Tuple

import torch

from ..core import Tensor
from ..dtypes import dtype as _dtype
from ..opdef import OpDef, emit, emit1

SUMSQ_BLOCK = 64  # columns per partial sum of squares of a deferred norm

# ---- references ------------------------------------------------------------------------------------------------------


def _dyt(x, alpha, w, b):
    return torch.tanh(alpha * x.float()) * w + b


def _mm(a, w):
    """`a @ w^T` with 32-bit accumulation and result."""
    return a.float() @ w.float().t()


def _embed_dyt_ref(x, tokens, table, alpha, w, b):
    n = tokens.numel()
    if x.device.type == "meta":
        return torch.empty((n, x.shape[1]), dtype=table.dtype, device="meta")
    x[:n].copy_(table[tokens.reshape(-1).long().clamp(0, table.shape[0] - 1)].float())
    return _dyt(x[:n], alpha, w, b).to(table.dtype)


def _split_residual(rest, has_norm, has_inject):
    rest = list(rest)
    norm = [rest.pop(0) for _ in range(3)] if has_norm else None
    inject = [rest.pop(0) for _ in range(2)] if has_inject else None
    return norm, inject


def _linear_residual_dyt_ref(x, a, weight, *rest, mult, has_norm, has_inject):
    norm, inject = _split_residual(rest, has_norm, has_inject)
    n = a.shape[0]
    if x.device.type == "meta":
        return torch.empty((n, x.shape[1]), dtype=a.dtype, device="meta") if has_norm else ()
    x[:n] += mult * _mm(a, weight).to(a.dtype).float()
    if inject is not None:
        tokens, table = inject
        x[:n] += table[tokens.reshape(-1).long().clamp(0, table.shape[0] - 1)].float()
    return _dyt(x[:n], *norm).to(a.dtype) if norm is not None else ()


def _select_dyt_ref(x, idx, alpha, w, b, stride, offset, out_dtype):
    if x.device.type == "meta":
        return torch.empty((idx.shape[0], x.shape[1]), dtype=out_dtype, device="meta")
    rows = torch.arange(idx.shape[0], device=x.device) * stride + idx.long() - offset
    return _dyt(x[rows.clamp(0, x.shape[0] - 1)], alpha, w, b).to(out_dtype)


def _rms_factor(sumsq, cols, eps):
    """Row factors of a deferred norm, `(rows, 1)`."""
    return 1.0 / torch.sqrt(sumsq.sum(-1, keepdim=True) / cols + eps)


def _deferred_mm(a, weight, sumsq, eps):
    y = _mm(a, weight)
    return y * _rms_factor(sumsq[0], a.shape[1], eps) if sumsq else y


def _linear_rows_ref(a, weight, *sumsq, out_dtype, eps=0.0):
    if a.device.type == "meta":
        return torch.empty((a.shape[0], weight.shape[0]), dtype=out_dtype, device="meta")
    return _deferred_mm(a, weight, sumsq, eps).to(out_dtype)


def _rms(x, w, eps):
    x = x.float()
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def _embed_rms_ref(x, tokens, table, w, scale, eps):
    n = tokens.numel()
    if x.device.type == "meta":
        return torch.empty((n, x.shape[1]), dtype=table.dtype, device="meta")
    x[:n].copy_(table[tokens.reshape(-1).long().clamp(0, table.shape[0] - 1)].float() * scale)
    return _rms(x[:n], w, eps).to(table.dtype)


def _linear_residual_rms_ref(x, a, weight, *norm, mult, eps, deferred):
    n, cols = a.shape[0], x.shape[1]
    blocks = -(-cols // SUMSQ_BLOCK)
    if x.device.type == "meta":
        out = [torch.empty((n, cols), dtype=a.dtype, device="meta")] if norm else []
        return out + ([torch.empty((n, blocks), dtype=torch.float32, device="meta")] if deferred else [])
    y = _mm(a, weight)
    x[:n] += mult * (y if deferred else y.to(a.dtype).float())
    if not norm:
        return ()
    if not deferred:
        return _rms(x[:n], norm[0], eps).to(a.dtype)
    sq = torch.nn.functional.pad(x[:n] * x[:n], (0, blocks * SUMSQ_BLOCK - cols))
    return (x[:n] * norm[0]).to(a.dtype), sq.reshape(n, blocks, SUMSQ_BLOCK).sum(-1)


def _select_rms_ref(x, idx, w, stride, offset, eps, out_dtype):
    if x.device.type == "meta":
        return torch.empty((idx.shape[0], x.shape[1]), dtype=out_dtype, device="meta")
    rows = torch.arange(idx.shape[0], device=x.device) * stride + idx.long() - offset
    return _rms(x[rows.clamp(0, x.shape[0] - 1)], w, eps).to(out_dtype)


def _linear_split_glu_ref(h, weight, *sumsq, cols, lead, limit, slope, shift, eps=0.0):
    n, f = h.shape[0], (weight.shape[0] - cols) // 2
    if h.device.type == "meta":
        return [torch.empty((n, c), dtype=h.dtype, device="meta") for c in (cols, lead + f)]
    y = _deferred_mm(h, weight, sumsq, eps).to(h.dtype)
    g, u = y[:, cols:cols + f].float().clamp(max=limit), y[:, cols + f:].float().clamp(-limit, limit)
    joint = torch.zeros((n, lead + f), dtype=h.dtype, device=h.device)
    joint[:, lead:] = (g * torch.sigmoid(slope * g) * (u + shift)).to(h.dtype)
    return y[:, :cols], joint


def _linear_swiglu_ref(h, weight):
    f = weight.shape[0] // 2
    if h.device.type == "meta":
        return torch.empty((h.shape[0], f), dtype=h.dtype, device="meta")
    gu = _mm(h, weight).to(h.dtype).float()
    return (torch.nn.functional.silu(gu[:, :f]) * gu[:, f:]).to(h.dtype)


def _min_gru_ref(h, weight, bz, bx, state, pos, count, T):
    width = state.shape[1]
    if h.device.type == "meta":
        return torch.empty((h.shape[0], width), dtype=h.dtype, device="meta")
    z, u, g = _mm(h, weight).to(h.dtype).float().reshape(-1, T, 3, width).unbind(2)
    z, u = torch.sigmoid(z + bz), u + bx
    cand = torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
    y = torch.zeros_like(z)
    for b in range(z.shape[0]):
        s = state[b].clone() if int(pos[b]) > 0 else torch.zeros_like(state[b])
        for t in range(min(int(count[b]), T)):
            s = (1.0 - z[b, t]) * s + z[b, t] * cand[b, t]
            y[b, t] = s * torch.nn.functional.silu(g[b, t])
        state[b].copy_(s)
    return y.reshape(-1, width).to(h.dtype)


def _rotate_interleaved(x, cos, sin):
    """`x (t, heads, dim)`, tables `(t, r)`: rotate the pairs of the first `2r` features."""
    r = cos.shape[1]
    xr = x[..., :2 * r].float()
    u, v = xr[..., 0::2], xr[..., 1::2]
    c, s = cos[:, None], sin[:, None]
    rot = torch.stack((u * c - v * s, v * c + u * s), dim=-1).flatten(-2)
    return torch.cat((rot.to(x.dtype), x[..., 2 * r:]), dim=-1)


def _diff_attention_ref(qkv, cos, sin, kc, vc, pos, count, lam, T, heads, rotary_dim, chunk, scale, eps, out_scale):
    B, G, _, smax, dim = kc.shape
    vdim = vc.shape[-1]
    if qkv.device.type == "meta":
        return torch.empty((qkv.shape[0], heads * vdim), dtype=qkv.dtype, device="meta")
    out = torch.zeros((B, T, heads * vdim), dtype=qkv.dtype, device=qkv.device)
    rows = qkv.reshape(B, T, -1)
    for b in range(B):
        p, n = int(pos[b]), min(int(count[b]), T)
        if n <= 0:
            continue
        cur = rows[b, :n]
        q = cur[:, :heads * 2 * dim].reshape(n, heads * 2, dim)
        k = cur[:, heads * 2 * dim:(heads + G) * 2 * dim].reshape(n, G * 2, dim)
        v = cur[:, (heads + G) * 2 * dim:].reshape(n, G, vdim)
        if rotary_dim:
            q = _rotate_interleaved(q, cos[p:p + n], sin[p:p + n])
            k = _rotate_interleaved(k, cos[p:p + n], sin[p:p + n])
        kc[b, :, :, p:p + n].copy_(k.reshape(n, G, 2, dim).permute(1, 2, 0, 3))
        vc[b, :, p:p + n].copy_(v.permute(1, 0, 2))
        qp = torch.arange(p, p + n, device=qkv.device)
        kp = torch.arange(0, p + n, device=qkv.device)
        mask = kp[None] <= qp[:, None]
        if chunk:
            mask &= (kp[None] // chunk) == (qp[:, None] // chunk)
        qf = q.float().reshape(n, G, heads // G, 2, dim)
        s = torch.einsum("ngrmd,gmkd->grmnk", qf, kc[b, :, :, :p + n].float()) * scale
        a = torch.softmax(s.masked_fill(~mask, float("-inf")), dim=-1)
        a = torch.einsum("grmnk,gkv->grmnv", a, vc[b, :, :p + n].float())
        o = a[:, :, 0] - lam * a[:, :, 1]
        o = o * (out_scale / torch.sqrt((o * o).mean(-1, keepdim=True) + eps))
        out[b, :n] = o.permute(2, 0, 1, 3).reshape(n, heads * vdim).to(qkv.dtype)
    return out.reshape(B * T, heads * vdim)


def _window_attention_ref(proj, q_norm, k_norm, kc, vc, pos, count, joint, T, heads, window, keep_first, scale, sink, eps):
    if proj.device.type == "meta":
        return torch.empty(joint.shape, dtype=joint.dtype, device="meta")
    B, G, smax, dim = kc.shape
    vdim, dt = vc.shape[-1], proj.dtype
    qk = (heads + G) * dim
    for b in range(B):
        p, n = int(pos[b]), min(int(count[b]), T)
        if n <= 0:
            continue
        cur = proj.reshape(B, T, -1)[b, :n]
        q = _rms(cur[:, :heads * dim].reshape(n, heads, dim), q_norm, eps).to(dt)
        k = _rms(cur[:, heads * dim:qk].reshape(n, G, dim), k_norm, eps).to(dt)
        kc[b, :, p:p + n].copy_(k.permute(1, 0, 2))
        vc[b, :, p:p + n].copy_(cur[:, qk:qk + G * vdim].reshape(n, G, vdim).permute(1, 0, 2))
        qp, kp = torch.arange(p, p + n, device=proj.device)[:, None], torch.arange(0, p + n, device=proj.device)[None]
        mask = kp <= qp
        if window:
            mask &= (qp - kp < window) | (kp < keep_first)
        s = torch.einsum("ngrd,gkd->grnk", q.float().reshape(n, G, heads // G, dim), kc[b, :, :p + n].float()) * scale
        s = s.masked_fill(~mask, float("-inf"))
        if sink is not None:
            s = torch.cat((s, torch.full_like(s[..., :1], sink)), dim=-1)
        a = torch.softmax(s, dim=-1)[..., :p + n]
        o = torch.einsum("grnk,gkv->ngrv", a, vc[b, :, :p + n].float()).reshape(n, heads * vdim)
        if cur.shape[1] > qk + G * vdim:
            o = o * torch.sigmoid(cur[:, qk + G * vdim:].float())
        joint.reshape(B, T, -1)[b, :n, :heads * vdim] = o.to(joint.dtype)
    return joint


def _advance_by_ref(pos, count):
    if pos.device.type != "meta":
        pos.add_(count)
    return pos


OpDef("embed_dyt_", impl=_embed_dyt_ref)
OpDef("linear_residual_dyt_", impl=_linear_residual_dyt_ref)
OpDef("select_dyt", impl=_select_dyt_ref)
OpDef("linear_rows", impl=_linear_rows_ref)
OpDef("linear_swiglu", impl=_linear_swiglu_ref)
OpDef("min_gru_", impl=_min_gru_ref)
OpDef("diff_attention_", impl=_diff_attention_ref)
OpDef("embed_rms_", impl=_embed_rms_ref)
OpDef("linear_residual_rms_", impl=_linear_residual_rms_ref)
OpDef("select_rms", impl=_select_rms_ref)
OpDef("linear_split_glu", impl=_linear_split_glu_ref)
OpDef("window_attention_", impl=_window_attention_ref, inplace=True)
OpDef("advance_by_", impl=_advance_by_ref, inplace=True)

# ---- graph functions -------------------------------------------------------------------------------------------------

Norm = Tuple[Tensor, Tensor, Tensor]  # Dynamic Tanh: (alpha (1,), weight, bias), all fp32


def embed_dyt_(x: Tensor, tokens: Tensor, table: Tensor, norm: Norm) -> Tensor:
    """Start the residual stream: rows `[0, tokens)` of `x (rows, width)` fp32 become the table rows; returns the first
    norm of them in the table's dtype."""
    return emit1("embed_dyt_", [x, tokens, table, *norm])


def linear_residual_dyt_(x: Tensor, a: Tensor, weight: Tensor, mult: float = 1.0, norm: Optional[Norm] = None,
                         inject: Optional[Sequence[Tensor]] = None) -> Optional[Tensor]:
    """`x += mult * (a @ weight^T)` on the fp32 residual stream (rows `[0, len(a))`), `weight (width, K)`. `inject =
    (tokens, table)` adds the table rows afterwards; with `norm`, returns the Dynamic Tanh of the updated stream in the
    dtype of `a`."""
    ins = [x, a, weight, *(norm or ()), *(inject or ())]
    out = emit("linear_residual_dyt_", ins,
               dict(mult=float(mult), has_norm=norm is not None, has_inject=inject is not None))
    return out[0] if norm is not None else None


def select_dyt(x: Tensor, idx: Tensor, norm: Norm, stride: int = 0, offset: int = 0, dtype: _dtype = None) -> Tensor:
    """Dynamic Tanh of the stream's rows `r * stride + idx[r] - offset`."""
    return emit1("select_dyt", [x, idx, *norm], dict(stride=int(stride), offset=int(offset), out_dtype=dtype.as_torch()))


def linear_rows(a: Tensor, weight: Tensor, dtype: Optional[_dtype] = None, sumsq: Optional[Tensor] = None,
                eps: float = 0.0) -> Tensor:
    """`a (n, K) @ weight (N, K)^T`, 32-bit accumulation, result in `dtype` (default: that of `a`). `sumsq` finishes a
    deferred norm of `a`."""
    ins = [a, weight] + ([sumsq] if sumsq is not None else [])
    return emit1("linear_rows", ins, dict(out_dtype=(dtype or a.dtype).as_torch(), eps=float(eps)))


def embed_rms_(x: Tensor, tokens: Tensor, table: Tensor, norm: Tensor, scale: float = 1.0, eps: float = 1e-6) -> Tensor:
    """Start the residual stream: rows `[0, tokens)` of `x (rows, width)` fp32 become the table rows times `scale`; returns
    their RMS norm (`norm (width,)` fp32 factors) in the table's dtype."""
    return emit1("embed_rms_", [x, tokens, table, norm], dict(scale=float(scale), eps=float(eps)))


def linear_residual_rms_(x: Tensor, a: Tensor, weight: Tensor, norm: Optional[Tensor] = None, eps: float = 1e-6,
                         mult: float = 1.0, deferred: bool = False) -> Tuple[Optional[Tensor], Optional[Tensor]]:
    """`x += mult * (a @ weight^T)` on the fp32 residual stream (rows `[0, len(a))`). With `norm`, returns the RMS norm of the
    updated stream in the dtype of `a` and None; `deferred` (few rows): the stream times `norm`, and its sums of squares."""
    out = emit("linear_residual_rms_", [x, a, weight] + ([norm] if norm is not None else []),
               dict(mult=float(mult), eps=float(eps), deferred=bool(deferred and norm is not None)))
    return (*out, None, None)[:2]


def select_rms(x: Tensor, idx: Tensor, norm: Tensor, stride: int = 0, offset: int = 0, eps: float = 1e-6,
               dtype: _dtype = None) -> Tensor:
    """RMS norm of the stream's rows `r * stride + idx[r] - offset`."""
    return emit1("select_rms", [x, idx, norm], dict(stride=int(stride), offset=int(offset), eps=float(eps),
                                                    out_dtype=dtype.as_torch()))


def linear_split_glu(h: Tensor, weight: Tensor, cols: int, lead: int, limit: float, slope: float = 1.0, shift: float = 0.0,
                     sumsq: Optional[Tensor] = None, eps: float = 0.0) -> Tuple[Tensor, Tensor]:
    """One product for several readers of `h`: `weight` = rows `[cols plain ones | gate | up]`. Returns the plain results
    `(n, cols)` and a joint buffer `(n, lead + F)` that ends in the clamped gated unit `g * sigmoid(slope * g) * (u + shift)`,
    `g = min(gate, limit)`, `u = clamp(up, -limit, limit)`; its first `lead` columns are for another op to fill. `sumsq`
    finishes a deferred norm of `h`."""
    return tuple(emit("linear_split_glu", [h, weight] + ([sumsq] if sumsq is not None else []),
                      dict(cols=int(cols), lead=int(lead), limit=float(limit), slope=float(slope), shift=float(shift),
                           eps=float(eps))))


def linear_swiglu(h: Tensor, weight: Tensor) -> Tensor:
    """`silu(h @ gate^T) * (h @ up^T)` with `weight` = rows `[gate | up]`."""
    return emit1("linear_swiglu", [h, weight])


def min_gru_(h: Tensor, weight: Tensor, z_bias: Tensor, x_bias: Tensor, state: Tensor, pos: Tensor, count: Tensor,
             T: int) -> Tensor:
    """minGRU mixer up to its output gate: with `[z | u | g] = h @ weight^T`, `z = sigmoid(z + z_bias)` and the candidate
    `c = u' + 1/2` for `u' = u + x_bias >= 0`, `sigmoid(u')` otherwise, the state `(batch, width)` fp32 follows
    `S = (1 - z) S + z c`; returns `S * silu(g)`."""
    return emit1("min_gru_", [h, weight, z_bias, x_bias, state, pos, count], dict(T=int(T)))


def diff_attention_(qkv: Tensor, cos: Tensor, sin: Tensor, k_cache: Tensor, v_cache: Tensor, pos: Tensor, count: Tensor,
                    lam: Tensor, T: int, heads: int, rotary_dim: int, scale: float, chunk: int = 0, eps: float = 1e-6,
                    out_scale: float = 1.0) -> Tensor:
    """Differential attention of a portion against the cache. `qkv` rows are `[q: heads x 2 x dim | k: G x 2 x dim |
    v: G x vdim]`; q and k are rotated (interleaved pairs of the first `rotary_dim` features of each map; tables
    `(max_seq, rotary_dim/2)` fp32) and keys and values are appended to `k_cache (batch, G, 2, max_seq, dim)` and
    `v_cache (batch, G, max_seq, vdim)`. Each head's `a_1 - lam * a_2` is divided by its root mean square and multiplied by
    `out_scale`. `chunk > 0` limits a position to the keys of its own chunk of that many positions."""
    return emit1("diff_attention_", [qkv, cos, sin, k_cache, v_cache, pos, count, lam],
                 dict(T=int(T), heads=int(heads), rotary_dim=int(rotary_dim), chunk=int(chunk), scale=float(scale),
                      eps=float(eps), out_scale=float(out_scale)))


def window_attention_(proj: Tensor, q_norm: Tensor, k_norm: Tensor, k_cache: Tensor, v_cache: Tensor, pos: Tensor,
                      count: Tensor, joint: Tensor, T: int, heads: int, scale: float, window: int = 0, keep_first: int = 0,
                      sink: Optional[float] = None, eps: float = 1e-6) -> Tensor:
    """Attention of a portion against the cache, written into the first `heads * vdim` columns of `joint`. `proj` rows are
    `[q: heads x dim | k: G x dim | v: G x vdim | gate: heads x vdim]`, the gate may be absent. Every query and key head gets
    an RMS norm with the fp32 factors `q_norm` / `k_norm (dim,)`; keys and values are appended to `k_cache (batch, G, max_seq,
    dim)` and `v_cache (batch, G, max_seq, vdim)`. With `window > 0` position i sees `j <= i` if `i - j < window` or `j <
    keep_first`. `sink`: a score without a value that takes part in the softmax. The output is multiplied by
    `sigmoid(gate)`."""
    return emit1("window_attention_", [proj, q_norm, k_norm, k_cache, v_cache, pos, count, joint],
                 dict(T=int(T), heads=int(heads), window=int(window), keep_first=int(keep_first), scale=float(scale),
                      sink=None if sink is None else float(sink), eps=float(eps)))


def advance_by_(pos: Tensor, count: Tensor) -> Tensor:
    """`pos += count` (both `(batch,)` int32)."""
    return emit1("advance_by_", [pos, count])
