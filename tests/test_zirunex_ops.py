"""The ops of RMS-normalised parallel layers and of sliding-window attention one by one against the plain oracle, with inputs
in which a wrong key, a window that is one position off, a missing kept token or a missing sink stands out. CPU backend, and
marked `gpu` the kernels (32-bit and bf16)."""
import pytest
import torch

import plain_zirunex as plain
from test_dunelix_ops import backend, close, i32, op, rnd  # noqa: F401  (fixture and helpers)


def f32(backend):  # noqa: F811
    return backend[0], torch.float32


@pytest.mark.parametrize("rows,width", [(1, 8), (5, 33), (70, 256), (16, 1032), (3, 4100), (2, 9000)])
def test_residual_stream_ops(backend, rows, width):  # noqa: F811
    dev, eps = backend[0], 1e-3
    w, w64 = rnd(f32(backend), width, seed=2)
    table, table64 = rnd(backend, 19, width, std=0.1, seed=5)
    tokens = torch.randint(0, 19, (rows,), generator=torch.Generator().manual_seed(1)).int().to(dev)
    x = torch.full((rows + 3, width), 7.0, device=dev)
    h = op("embed_rms_", backend, x, tokens, table, w, scale=3.5, eps=eps)
    start = 3.5 * table64[tokens.long().cpu()]
    close(x[:rows], start, backend, 1e-6, 1e-6)
    close(h, plain.rms_unit(start, eps) * w64, backend)
    # updates with and without a norm; rows past the portion stay as they are
    for K in (8, 24, 200):
        a, a64 = rnd(backend, rows, K, seed=7)
        m, m64 = rnd(backend, width, K, std=K ** -0.5, seed=8)
        for mode in ("norm", "deferred", "none"):
            if mode == "deferred" and (rows > 16 or dev == "cuda" and backend[1] == torch.float32):
                continue
            x = torch.randn(rows + 3, width, generator=torch.Generator().manual_seed(3)).to(dev)
            want = x.double().cpu()
            want[:rows] += 0.7 * (a64 @ m64.T)
            out = op("linear_residual_rms_", backend, x, a, m, *([] if mode == "none" else [w]), mult=0.7, eps=eps,
                     deferred=mode == "deferred")
            close(x, want, backend, 2e-6, 4e-3)
            if mode == "norm":
                close(out, plain.rms_unit(want[:rows], eps) * w64, backend)
            elif mode == "deferred":
                close(out[0], want[:rows] * w64, backend)
                assert out[1].shape == (rows, -(-width // 64))
                close(out[1].sum(-1), (want[:rows] ** 2).sum(-1), backend, 1e-5, 1e-2)
    sel = op("select_rms", backend, x, i32(backend, 0, rows - 1, 0), w, stride=0, offset=0, eps=eps, out_dtype=backend[1])
    close(sel, plain.rms_unit(x.double().cpu()[[0, rows - 1, 0]], eps) * w64, backend)


@pytest.mark.parametrize("rows,N,K", [(1, 7, 8), (3, 130, 72), (16, 640, 264), (9, 96, 4096)])
def test_products_that_finish_a_deferred_norm(backend, rows, N, K):  # noqa: F811
    """A row that is a hundred times larger than the others: its norm must not leak into them."""
    if backend == ("cuda", torch.float32):
        pytest.skip("32-bit models do not defer norms")
    eps = 1e-3
    x = torch.randn(rows, K, generator=torch.Generator().manual_seed(1)).double()
    x[rows // 2] *= 100.0
    w, w64 = rnd(f32(backend), K, seed=2)
    m, m64 = rnd(backend, N, K, std=K ** -0.5, seed=3)
    h = (x * w64).to(backend[1]).to(backend[0])
    sq = torch.nn.functional.pad(x * x, (0, -K % 64)).reshape(rows, -1, 64).sum(-1).float().to(backend[0])
    want = (plain.rms_unit(x, eps) * w64) @ m64.T
    for _ in range(2):  # the second launch finds the counters as the first one left them
        close(op("linear_rows", backend, h, m, sq, out_dtype=torch.float32, eps=eps), want, backend)
    if N % 2 == 0:
        cols = N // 2 - N // 2 % 2
        proj, joint = op("linear_split_glu", backend, h, m, sq, cols=cols, lead=5, limit=0.9, slope=1.3, shift=0.5, eps=eps)
        f = (N - cols) // 2
        close(proj, want[:, :cols], backend)
        g, u = want[:, cols:cols + f].clamp(max=0.9), want[:, cols + f:].clamp(-0.9, 0.9)
        close(joint[:, 5:], g * torch.sigmoid(1.3 * g) * (u + 0.5), backend)


@pytest.mark.parametrize("rows,cols,F,K", [(1, 8, 8, 8), (2, 70, 45, 48), (16, 200, 352, 200), (33, 64, 64, 64), (4, 9, 10, 10),
                                           (5, 72, 0, 16), (40, 24, 0, 16), (300, 136, 96, 128)])
def test_linear_split_glu(backend, rows, cols, F, K):  # noqa: F811
    """Gates and ups on both sides of their limits; the plain columns are not clamped."""
    h, h64 = rnd(backend, rows, K, seed=1)
    w, w64 = rnd(backend, cols + 2 * F, K, std=2.0 * K ** -0.5, seed=2)
    for limit in (0.7, 3.0):
        proj, joint = op("linear_split_glu", backend, h, w, cols=cols, lead=16, limit=limit, slope=1.702, shift=1.0)
        y = h64 @ w64.T
        assert proj.shape == (rows, cols) and joint.shape == (rows, 16 + F)
        close(proj, y[:, :cols], backend)
        if F:
            close(joint[:, 16:], plain.clamped_glu(y[:, cols:cols + F], y[:, cols + F:], limit), backend, 2e-5, 2e-2)


def attention_oracle(proj64, wq, wk, H, G, dim, vdim, scale, window, keep, sink, eps, gated):
    """All positions of one sequence from position 0."""
    n, qk = proj64.shape[0], (H + G) * dim
    q = plain.head_norm(proj64[:, :H * dim].reshape(n, H, dim), wq, eps)
    k = plain.head_norm(proj64[:, H * dim:qk].reshape(n, G, dim), wk, eps)
    v = proj64[:, qk:qk + G * vdim].reshape(n, G, vdim)
    mask = plain.window_mask(n, window or None, keep)
    out = []
    for h in range(H):
        g = h // (H // G)
        if sink is None:
            s = ((q[:, h] @ k[:, g].T) * scale).masked_fill(~mask, float("-inf"))
            out.append(torch.softmax(s, dim=-1) @ v[:, g])
        else:  # a shifted sink is a shift of all scores
            s = ((q[:, h] @ k[:, g].T) * scale - sink).masked_fill(~mask, float("-inf"))
            out.append(plain.sink_weights(s) @ v[:, g])
    o = torch.cat(out, dim=-1)
    return plain.gated(o, proj64[:, qk + G * vdim:]) if gated else o


SHAPES = [  # H, G, dim, vdim, window, keep, positions
    (2, 1, 8, 8, 5, 2, 23),
    (4, 2, 16, 24, 13, 6, 60),
    (3, 3, 10, 7, 0, 0, 40),         # sizes no vector access divides, no window
    (18, 1, 32, 16, 17, 3, 70),      # more query heads on one key head than a decoding tile holds
    (4, 2, 64, 128, 100, 5, 330),
    (8, 2, 64, 64, 0, 0, 300),
    (2, 2, 128, 128, 129, 131, 400),  # kept tokens past a block's edge, window past a block's edge
    (6, 2, 40, 72, 64, 1, 200),      # three query heads per key head: rows of a token straddle tiles
    (4, 1, 128, 64, 256, 16, 520),
    (5, 1, 64, 64, 128, 128, 390),
    (1, 1, 144, 160, 20, 4, 70),     # beyond what the tensor-core kernels take
    (2, 1, 64, 200, 30, 4, 90),      # values that only the decoding kernel takes
    (2, 1, 16, 16, 1, 0, 40),        # windows of one position
    (2, 1, 16, 16, 1, 3, 40),
    (16, 2, 48, 96, 7, 40, 90),      # more kept tokens than window
]


@pytest.mark.parametrize("shape", SHAPES, ids=lambda s: "x".join(map(str, s)))
@pytest.mark.parametrize("plant", ["none", "edges"])
def test_window_attention(backend, shape, plant):  # noqa: F811
    """One sequence in portions of several sizes and then token by token, next to an idle slot and a second sequence that runs
    the same tokens in one portion. With `edges`, queries match single keys strongly: the window's first key (just inside),
    the key before it (just outside), the last kept and the first not kept token, themselves and the first token, in
    prompts and in decoding."""
    H, G, dim, vdim, window, keep, n = shape
    eps, R = 1e-5, H // G
    gated, sink = (n // 10) % 3 != 0, (0.0, -1.5, None)[n % 3]
    gen = torch.Generator().manual_seed(n + dim)
    qk = (H + G) * dim
    width = qk + G * vdim + (H * vdim if gated else 0)
    raw = torch.randn(n, width, generator=gen)
    wq, wk = 1.0 + 0.2 * torch.randn(dim, generator=gen), 1.0 + 0.2 * torch.randn(dim, generator=gen)
    scale = 1.4 * dim ** -0.5
    if plant == "edges":
        scale = 12.0 / dim  # a query in the direction of a key scores about 12
        k = plain.head_norm(raw[:, H * dim:qk].reshape(n, G, dim), wk, eps)
        q = raw[:, :H * dim].reshape(n, H, dim)
        size = window or n
        for i in range(n):
            target = [i - size + 1, i - size, keep - 1, keep, i, 0][i % 6]
            target = min(max(0, target), i)
            for h in range(H):
                q[i, h] = k[target, h // R] / wq
    raw = raw.to(backend[1])
    want = attention_oracle(raw.double(), wq.double(), wk.double(), H, G, dim, vdim, scale, window, keep, sink, eps, gated)
    dev, B, smax, lead, extra = backend[0], 3, n + 2, H * vdim, 8
    kc = torch.full((B, G, smax, dim), 3.0, dtype=backend[1], device=dev)
    vc = torch.full((B, G, smax, vdim), 50.0, dtype=backend[1], device=dev)
    kw = dict(heads=H, window=window, keep_first=keep, scale=scale, sink=sink, eps=eps)
    got = torch.zeros(n, lead, dtype=torch.float64)

    def portion(T, rows):  # rows: slot -> (first position, count)
        block = torch.zeros(B, T, width, dtype=backend[1])
        pos, count = [5, 5, 5], [0, 0, 0]
        for b, (p, c) in rows.items():
            block[b, :c], pos[b], count[b] = raw[p:p + c], p, c
        joint = torch.full((B * T, lead + extra), 9.0, dtype=backend[1], device=dev)
        out = op("window_attention_", backend, block.reshape(B * T, width).to(dev), wq.to(dev), wk.to(dev), kc, vc,
                 i32(backend, *pos), i32(backend, *count), joint, T=T, **kw)
        assert (out[:, lead:] == 9.0).all()
        return out[:, :lead].reshape(B, T, -1).double().cpu()

    tol = (3e-5, 4e-2)
    whole = portion(n + 3, {1: (0, n)})[1, :n]
    close(whole, want, backend, *tol)
    at, sizes, tail = 0, [1, 2, 9, 30, n // 3], min(24, n // 2)
    while at < n:
        c = max(1, min(sizes.pop(0) if sizes else n, n - tail - at)) if at < n - tail else 1
        out = portion(c if c == 1 else c + 1, {2: (at, c), **({0: (at, c)} if at < 12 else {})})
        got[at:at + c] = out[2, :c]
        at += c
    close(got, want, backend, *tol)
    assert torch.equal(kc[1, :, n:].cpu(), torch.full_like(kc[1, :, n:].cpu(), 3.0))  # padding rows are not appended
    if backend[1] == torch.float32:
        torch.testing.assert_close(kc[1, :, :n], kc[2, :, :n], rtol=0, atol=0)


def test_planted_edges_stand_out():
    """The oracle's output moves visibly when the window or the number of kept tokens is wrong by one: what the comparison
    above relies on."""
    H, G, dim, vdim, n = 2, 1, 32, 16, 40
    raw = torch.randn(n, (H + G) * dim + G * vdim, generator=torch.Generator().manual_seed(0)).double()
    one = torch.ones(dim).double()
    k = plain.head_norm(raw[:, H * dim:(H + G) * dim].reshape(n, G, dim), one, 1e-5)
    for i in range(n):
        raw[i, :dim] = raw[i, dim:2 * dim] = k[max(0, [i - 8, i - 9, min(i, 3), min(i, 4)][i % 4]), 0]

    def out(window=9, keep=4, sink=0.0):
        return attention_oracle(raw, one, one, H, G, dim, vdim, 12.0 / dim, window, keep, sink, 1e-5, False)

    for other in (dict(window=8), dict(window=10), dict(keep=3), dict(keep=5)):
        assert (out() - out(**other)).abs().max() > 0.5, other


@pytest.mark.parametrize("fill", [-6.0, 0.0, 6.0])
def test_sink_against_equal_scores(backend, fill):  # noqa: F811
    """All scores equal: the weights sum to n e^s / (1 + n e^s), far from 1 where the scores are low."""
    n, dim, vdim = 20, 16, 8
    unit = torch.zeros(dim)
    unit[0] = dim ** 0.5  # its own RMS norm
    proj = torch.cat((unit.repeat(n, 2), torch.ones(n, vdim)), dim=1).to(backend[1]).to(backend[0])
    one = torch.ones(dim, device=backend[0])
    signed = one.clone()
    signed[0] = fill / dim  # the score of every pair is `fill`
    kc, vc = (torch.zeros(1, 1, n, c, dtype=backend[1], device=backend[0]) for c in (dim, vdim))
    e = torch.exp(torch.tensor(fill)).double()
    for T, start in ((n - 1, 0), (1, n - 1)):
        joint = torch.zeros(T, vdim, dtype=backend[1], device=backend[0])
        op("window_attention_", backend, proj[start:start + T], signed, one, kc, vc, i32(backend, start), i32(backend, T), joint,
           T=T, heads=1, window=6, keep_first=2, scale=1.0, sink=0.0, eps=0.0)
        seen = plain.window_mask(n, 6, 2).sum(-1)[start:start + T].double()
        close(joint[:, 0], seen * e / (1 + seen * e), backend)
