"""Ops of sequence models served with per-sequence state: a 32-bit residual stream, Dynamic Tanh norms, gated linear
recurrences and differential attention against a cache.

A *portion* holds the next tokens of every sequence of a batch: `(batch * T)` rows, sequence-major, of which the first
`count[b]` rows of sequence `b` are real and the rest is padding. `pos[b]` is the position of its first row. Both live on the
device, so a portion of a given `T` is a fixed program (and `T = 1` is the decoding step). State is updated in place, only by
the real rows; a sequence at position 0 starts from the empty state whatever its slot held before.

No counterpart in the reference (it ships no recurrent layers, cache or generation loop).
"""
from typing import Optional, Sequence, Tuple

import torch

from ..core import Tensor
from ..dtypes import dtype as _dtype
from ..opdef import OpDef, emit, emit1

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


def _linear_rows_ref(a, weight, out_dtype):
    if a.device.type == "meta":
        return torch.empty((a.shape[0], weight.shape[0]), dtype=out_dtype, device="meta")
    return _mm(a, weight).to(out_dtype)


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


def linear_rows(a: Tensor, weight: Tensor, dtype: Optional[_dtype] = None) -> Tensor:
    """`a (n, K) @ weight (N, K)^T`, 32-bit accumulation, result in `dtype` (default: that of `a`)."""
    return emit1("linear_rows", [a, weight], dict(out_dtype=(dtype or a.dtype).as_torch()))


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


def advance_by_(pos: Tensor, count: Tensor) -> Tensor:
    """`pos += count` (both `(batch,)` int32)."""
    return emit1("advance_by_", [pos, count])
