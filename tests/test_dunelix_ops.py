"""The sequence-model ops one by one against the plain oracle, with inputs in which a wrong key, a chunk edge that is one
position off, a lost state or a wrong row stands out. CPU backend, and marked `gpu` the kernels (32-bit and bf16)."""
import numpy as np
import pytest
import torch

import plain_dunelix as plain
from popxl_addons_b200.xl.opdef import OPS
import popxl_addons_b200.xl.ops  # noqa: F401  (registers the ops)

BACKENDS = [("cpu", torch.float32), pytest.param(("cuda", torch.float32), marks=pytest.mark.gpu),
            pytest.param(("cuda", torch.bfloat16), marks=pytest.mark.gpu)]


@pytest.fixture(params=BACKENDS, ids=lambda b: f"{b[0]}-{str(b[1])[6:]}")
def backend(request):
    return request.param


def op(name, backend, *args, **kw):
    if backend[0] == "cpu":
        return OPS[name].impl(*args, **kw)
    from popxl_addons_b200.ops import native  # noqa: F401

    res = OPS[name].native["cuda"](*args, **kw)
    assert res is not NotImplemented
    torch.cuda.synchronize()
    native.check_gemm_errors()
    return res


def rnd(backend, *shape, std=1.0, seed=0):
    """Random values that are exact in the backend's dtype: `(device tensor, float64 copy)`."""
    t = (torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * std).to(backend[1])
    return t.to(backend[0]), t.double()


def close(got, want, backend, tol32=2e-5, tol16=1.2e-2):
    got, want = got.detach().double().cpu(), want.double()
    err = (got - want).abs().max().item() / max(1e-30, want.abs().max().item())
    assert err < (tol32 if backend[1] == torch.float32 else tol16), err


def i32(backend, *v):
    return torch.tensor(v, dtype=torch.int32, device=backend[0])


def norm_params(backend, n, seed=0):
    f32 = (backend[0], torch.float32)
    return [rnd(f32, 1, std=0.7, seed=seed), rnd(f32, n, seed=seed + 1), rnd(f32, n, seed=seed + 2)]


@pytest.mark.parametrize("rows,width", [(1, 8), (5, 33), (70, 256), (16, 1030)])
def test_residual_stream_ops(backend, rows, width):
    dev = backend[0]
    norm = norm_params(backend, width)
    table, table64 = rnd(backend, 19, width, seed=5)
    tokens = torch.randint(0, 19, (rows,), generator=torch.Generator().manual_seed(1)).int().to(dev)
    tok = tokens.long().cpu()
    x = torch.full((rows + 3, width), 7.0, device=dev)
    n64 = [n[1] for n in norm]
    h = op("embed_dyt_", backend, x, tokens, table, *[n[0] for n in norm])
    close(x[:rows], table64[tok], backend, 1e-7, 1e-7)
    close(h, plain.dynamic_tanh(table64[tok], *n64), backend)
    # product, multiplier, injected rows and norm in every combination; rows past the portion stay as they are
    for K in (8, 24, 200):
        a, a64 = rnd(backend, rows, K, seed=7)
        w, w64 = rnd(backend, width, K, std=K ** -0.5, seed=8)
        for has_norm in (True, False):
            for has_inject in (True, False):
                x = torch.randn(rows + 3, width, generator=torch.Generator().manual_seed(3)).to(dev)
                want = x.double().cpu()
                want[:rows] += 0.7 * (a64 @ w64.T) + (table64[tok] if has_inject else 0.0)
                rest = ([n[0] for n in norm] if has_norm else []) + ([tokens, table] if has_inject else [])
                h = op("linear_residual_dyt_", backend, x, a, w, *rest, mult=0.7, has_norm=has_norm, has_inject=has_inject)
                close(x, want, backend, 2e-6, 4e-3)
                if has_norm:
                    close(h, plain.dynamic_tanh(want[:rows], *n64), backend)
    sel = op("select_dyt", backend, x, i32(backend, 0, rows - 1, 0), *[n[0] for n in norm], stride=0, offset=0,
             out_dtype=backend[1])
    close(sel, plain.dynamic_tanh(x.double().cpu()[[0, rows - 1, 0]], *n64), backend)


@pytest.mark.parametrize("rows,N,K", [(1, 7, 8), (3, 130, 72), (16, 640, 264), (16, 96, 4096), (40, 96, 64), (5, 12, 10)])
def test_linear_rows(backend, rows, N, K):
    a, a64 = rnd(backend, rows, K, seed=1)
    w, w64 = rnd(backend, N, K, std=K ** -0.5, seed=2)
    for out in (backend[1], torch.float32):
        for _ in range(2):  # the second launch finds the counters as the first one left them
            y = op("linear_rows", backend, a, w, out_dtype=out)
        assert y.dtype == out
        close(y, a64 @ w64.T, backend)


@pytest.mark.parametrize("rows,F,K", [(1, 8, 8), (2, 45, 48), (16, 352, 200), (33, 64, 64), (4, 9, 10)])
def test_linear_swiglu(backend, rows, F, K):
    h, h64 = rnd(backend, rows, K, seed=1)
    w, w64 = rnd(backend, 2 * F, K, std=K ** -0.5, seed=2)
    y = op("linear_swiglu", backend, h, w)
    close(y, plain.silu(h64 @ w64[:F].T) * (h64 @ w64[F:].T), backend, 2e-5, 2e-2)


def gru_oracle(h64, w64, bz, bx, s0):
    W = w64.shape[0] // 3
    z, u, g = (h64 @ w64.T).split(W, dim=-1)
    s = plain.min_gru_scan(torch.sigmoid(z + bz), plain.min_gru_candidate(u + bx), s0)
    return s * plain.silu(g), s


@pytest.mark.parametrize("W,T", [(8, 1), (70, 1), (33, 5), (64, 16), (20, 130), (130, 700)])
def test_min_gru(backend, W, T):
    """Three sequences: one fresh (its slot holds rubbish), one continued, one idle; long memories (small z) so that a state
    that was lost or taken twice shows at every later token."""
    B, K = 3, 24
    f32 = (backend[0], torch.float32)
    h, h64 = rnd(backend, B * T, K, seed=1)
    w, w64 = rnd(backend, 3 * W, K, std=K ** -0.5, seed=2)
    (bz, bz64), (bx, bx64) = rnd(f32, W, seed=3), rnd(f32, W, seed=4)
    bz, bz64 = bz - 4.0, bz64 - 4.0
    state, state64 = rnd(f32, B, W, std=5.0, seed=5)
    keep = state.clone()
    n = [T, max(1, T - 3), 0]
    y = op("min_gru_", backend, h, w, bz, bx, state, i32(backend, 0, 9, 4), i32(backend, *n), T=T)
    y = y.reshape(B, T, W)
    for b, s0 in ((0, None), (1, state64[1])):
        rows = h64.reshape(B, T, K)[b, :n[b]]
        wy, ws = gru_oracle(rows, w64, bz64, bx64, s0)
        close(y[b, :n[b]], wy, backend, 3e-5, 2e-2)
        close(state[b], ws[-1], backend, 3e-5, 2e-2)
    assert torch.equal(state[2], keep[2])


def diff_oracle(qkv64, H, G, dim, vdim, rot, scale, chunk, eps, out_scale, lam, freqs):
    """All positions of one sequence from position 0."""
    n = qkv64.shape[0]
    q = qkv64[:, :H * 2 * dim].reshape(n, H, 2, dim)
    k = qkv64[:, H * 2 * dim:(H + G) * 2 * dim].reshape(n, G, 2, dim)
    v = qkv64[:, (H + G) * 2 * dim:].reshape(n, G, vdim)
    pos = torch.arange(n)
    if rot:
        q, k = plain.rotate(q, pos, freqs), plain.rotate(k, pos, freqs)
    mask = plain.chunk_mask(n, chunk or None)
    out = []
    for h in range(H):
        g = h // (H // G)
        a = [plain.masked_attention(q[:, h, m], k[:, g, m], v[:, g], mask, scale) for m in (0, 1)]
        out.append(plain.differential_combine(a[0], a[1], lam, 1.0 - out_scale, eps))
    return torch.cat(out, dim=-1)


SHAPES = [  # H, G, dim, vdim, rot, chunk, positions
    (2, 1, 8, 8, 4, 5, 23),
    (4, 2, 16, 24, 16, 13, 60),
    (3, 3, 10, 7, 2, 0, 40),        # sizes no vector access divides
    (9, 1, 32, 16, 0, 17, 70),      # more than eight query heads on one key head, no rotation
    (4, 2, 64, 128, 32, 100, 330),
    (8, 2, 64, 128, 64, 0, 300),
    (2, 2, 128, 256, 128, 129, 400),
    (2, 1, 40, 72, 12, 64, 200),
    (4, 1, 128, 128, 64, 256, 520),
    (2, 1, 64, 64, 20, 128, 260),
    (1, 1, 288, 320, 36, 20, 70),   # beyond what the tensor-core kernels take
    (2, 1, 16, 16, 2, 1, 40),       # chunks of one position
]


@pytest.mark.parametrize("shape", SHAPES, ids=lambda s: "x".join(map(str, s)))
@pytest.mark.parametrize("plant", ["none", "edges"])
def test_diff_attention(backend, shape, plant):
    """One sequence in portions of several sizes and then token by token, next to an idle slot and a second sequence that runs
    the same tokens in one portion. With `edges`, some queries match single keys strongly: the first key of their chunk (just
    inside), the key before it (just outside), themselves and the first token, in prompts and in decoding."""
    H, G, dim, vdim, rot, chunk, n = shape
    eps, out_scale, lam, scale = 1e-5, 0.4, 0.83, dim ** -0.5
    from popxl_addons_b200.ops.rotary_pos_embed import frequency_tables, rotary_frequencies

    sc = {"factor": 4.0, "low": 1.0, "high": 3.0, "original": 64}
    gen = torch.Generator().manual_seed(n)
    width = (H + G) * 2 * dim + G * vdim
    raw = torch.randn(n, width, generator=gen)
    freqs = plain.rotary_frequencies(300.0, rot, sc) if rot else []
    if plant == "edges":
        size = chunk or n
        k = raw[:, H * 2 * dim:(H + G) * 2 * dim].reshape(n, G, 2, dim)
        q = raw[:, :H * 2 * dim].reshape(n, H, 2, dim)
        kr = plain.rotate(k.double(), torch.arange(n), freqs)
        back = [-f for f in freqs]  # inverse rotation: the query that, rotated at its own position, equals the wanted key
        for i in range(1, n, 3):
            start = i // size * size
            target = [start, max(0, start - 1), i, 0][(i // 3) % 4]
            for h in range(H):
                want = kr[target, h // (H // G)]
                un = plain.rotate(want[None], torch.tensor([i]), back)[0]
                q[i, h, 0] = (un[0] * (12.0 / (scale * (want[0] ** 2).sum()))).float()  # score 12 on that key, map 1
    raw = raw.to(backend[1])
    want = diff_oracle(raw.double(), H, G, dim, vdim, rot, scale, chunk, eps, out_scale, lam, freqs)
    dev, B, smax = backend[0], 3, n + 2
    sin, cos = (torch.tensor(t, device=dev) for t in frequency_tables(smax, rotary_frequencies(rot, 300.0, sc))) if rot else (
        torch.zeros(1, device=dev), torch.zeros(1, device=dev))
    kc = torch.full((B, G, 2, smax, dim), 3.0, dtype=backend[1], device=dev)
    vc = torch.full((B, G, smax, vdim), 50.0, dtype=backend[1], device=dev)
    kw = dict(heads=H, rotary_dim=rot, chunk=chunk, scale=scale, eps=eps, out_scale=out_scale)
    lam_t = torch.tensor([lam], device=dev)
    got = torch.zeros(n, H * vdim, dtype=torch.float64)

    def portion(T, rows):  # rows: slot -> (first position, count)
        block = torch.zeros(B, T, width, dtype=backend[1])
        pos, count = [5, 5, 5], [0, 0, 0]
        for b, (p, c) in rows.items():
            block[b, :c], pos[b], count[b] = raw[p:p + c], p, c
        out = op("diff_attention_", backend, block.reshape(B * T, width).to(dev), cos, sin, kc, vc, i32(backend, *pos),
                 i32(backend, *count), lam_t, T=T, **kw)
        return out.reshape(B, T, -1).double().cpu()

    tol = (3e-5, 4e-2)
    whole = portion(n + 3, {1: (0, n)})[1, :n]
    close(whole, want, backend, *tol)
    at, sizes = 0, [1, 2, 9, 30, n // 3]
    tail = min(24, n // 2)
    while at < n:
        c = min(sizes.pop(0) if sizes else n, n - tail - at) if at < n - tail else 1
        if c <= 0:
            c = 1
        out = portion(c if c == 1 else c + 1, {2: (at, c), **({0: (at, c)} if at < 12 else {})})
        got[at:at + c] = out[2, :c]
        at += c
    close(got, want, backend, *tol)
    assert torch.equal(kc[1, :, :, n:].cpu(), torch.full_like(kc[1, :, :, n:].cpu(), 3.0))  # padding rows are not appended
    if backend[1] == torch.float32:
        torch.testing.assert_close(kc[1, :, :, :n], kc[2, :, :, :n], rtol=0, atol=0)


def test_rotary_frequencies_match_the_oracle():
    from popxl_addons_b200.ops.rotary_pos_embed import frequency_tables, rotary_frequencies

    for base, dims, sc in ((10000.0, 64, None), (500.0, 24, {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 100}),
                           (20000.0, 2, {"factor": 3.0, "low": 2.0, "high": 5.0, "original": 5000})):
        f = rotary_frequencies(dims, base, sc)
        np.testing.assert_allclose(f, plain.rotary_frequencies(base, dims, sc), rtol=1e-12)
    sin, cos = frequency_tables(50, f)
    assert sin.dtype == np.float32 and sin.shape == (50, 1)
    np.testing.assert_allclose(cos[7], np.cos(7 * f), rtol=1e-6)


def test_advance_and_position_rows(backend):
    pos, count = i32(backend, 4, 0, 9), i32(backend, 3, 0, 1)
    op("advance_by_", backend, pos, count)
    assert pos.tolist() == [7, 0, 10]
    x = torch.arange(24.0, device=backend[0]).reshape(12, 2) * 0.01
    one = torch.ones(1, device=backend[0])
    w, b = torch.ones(2, device=backend[0]), torch.zeros(2, device=backend[0])
    # last real row of every sequence in a portion of four rows each
    h = op("select_dyt", backend, x, i32(backend, 3, 1, 4), one, w, b, stride=4, offset=1, out_dtype=backend[1])
    close(h, torch.tanh(x.double().cpu()[[2, 4, 11]]), backend)
