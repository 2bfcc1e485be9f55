"""Plain, slow oracle of the Dunelix decoder: one function per mechanism, no cache, whole sequences, written with
elementary torch expressions only. Works in the precision of the tensors it is given (float64 in the tests). Nothing here
is imported from the package under test."""
import math

import torch


def dynamic_tanh(x, alpha, w, b):
    return torch.tanh(alpha * x) * w + b


def rotary_frequencies(base, dims, scaling=None):
    """Angle per position of every rotated pair, optionally stretched for long wavelengths."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling is not None:
            lo, hi, orig, factor = scaling["low"], scaling["high"], scaling["original"], scaling["factor"]
            wavelength = 2.0 * math.pi / f
            if wavelength > orig / lo:
                f = f / factor
            elif wavelength >= orig / hi:
                s = (orig / wavelength - lo) / (hi - lo)
                f = (1.0 - s) * f / factor + s * f
        out.append(f)
    return out


def rotate(x, positions, freqs):
    """`x (tokens, ..., dim)`: rotate the pairs (2i, 2i+1) of the leading `2 * len(freqs)` features."""
    y = x.clone()
    for i, f in enumerate(freqs):
        a = positions.to(x.dtype) * f
        shape = (-1,) + (1,) * (x.dim() - 2)
        c, s = torch.cos(a).reshape(shape), torch.sin(a).reshape(shape)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        y[..., 2 * i] = u * c - v * s
        y[..., 2 * i + 1] = v * c + u * s
    return y


def chunk_mask(n, size=None):
    """`(n, n)` bool: may query i look at key j."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    m = j <= i
    if size is not None:
        m = m & (i // size == j // size)
    return m


def masked_attention(q, k, v, mask, scale):
    """One head, one map: `q (n, d)`, `k (n, d)`, `v (n, dv)`."""
    s = (q @ k.T) * scale
    s = s.masked_fill(~mask, float("-inf"))
    e = torch.exp(s - s.max(dim=-1, keepdim=True).values)
    return (e / e.sum(dim=-1, keepdim=True)) @ v


def differential_lambda(lq1, lk1, lq2, lk2, diff):
    return torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum()) + diff


def differential_combine(a1, a2, lam, diff, eps):
    o = a1 - lam * a2
    return o / torch.sqrt((o * o).mean(dim=-1, keepdim=True) + eps) * (1.0 - diff)


def differential_attention(h, w, mix, eps):
    """The whole attention mixer on `h (n, width)`; `w` maps tensor names (q, k, v, o, lq1, ...) to weights."""
    n = h.shape[0]
    H, G, d, dv = mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    pos = torch.arange(n)
    q = (h @ w["q"].T).reshape(n, H, 2, d)
    k = (h @ w["k"].T).reshape(n, G, 2, d)
    v = (h @ w["v"].T).reshape(n, G, dv)
    rot = mix.get("rot")
    if rot:
        f = rotary_frequencies(rot["base"], rot["dims"], rot.get("scaling"))
        q, k = rotate(q, pos, f), rotate(k, pos, f)
    mask = chunk_mask(n, (mix.get("mask") or {}).get("size"))
    lam = differential_lambda(w["lq1"], w["lk1"], w["lq2"], w["lk2"], mix["diff"])
    heads = []
    for hh in range(H):
        g = hh // (H // G)
        a = [masked_attention(q[:, hh, m], k[:, g, m], v[:, g], mask, mix["scale"]) for m in (0, 1)]
        heads.append(differential_combine(a[0], a[1], lam, mix["diff"], eps))
    return torch.cat(heads, dim=-1) @ w["o"].T


def min_gru_scan(z, cand, s0=None):
    """`S_t = (1 - z_t) S_{t-1} + z_t c_t`, token by token; returns all states."""
    s = torch.zeros_like(z[0]) if s0 is None else s0
    out = []
    for t in range(z.shape[0]):
        s = (1.0 - z[t]) * s + z[t] * cand[t]
        out.append(s)
    return torch.stack(out)


def min_gru_candidate(u):
    return torch.where(u >= 0, u + 0.5, torch.sigmoid(u))


def silu(x):
    return x * torch.sigmoid(x)


def min_gru(h, w):
    z = torch.sigmoid(h @ w["z"].T + w["z.b"])
    cand = min_gru_candidate(h @ w["x"].T + w["x.b"])
    s = min_gru_scan(z, cand)
    return (s * silu(h @ w["g"].T)) @ w["o"].T


def swiglu_mlp(h, w):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def layer_schedule(n_layers, loop):
    """`[(layer index, whether the embedding output is added first)]` in execution order."""
    if not loop:
        return [(i, False) for i in range(n_layers)]
    out = [(i, False) for i in range(loop["start"])]
    for r in range(loop["times"]):
        out += [(i, r > 0 and i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return out + [(i, False) for i in range(loop["stop"], n_layers)]


def forward(cfg, weights, tokens, trace=None):
    """Logits `(n, vocab)` of one sequence. `trace`: list that receives the residual stream after every layer run."""
    W = weights
    x = x0 = W["embed"][torch.as_tensor(tokens)]
    m, eps = cfg.get("residual_mult", 1.0), cfg["norm"]["eps"]

    def norm(name, x):
        return dynamic_tanh(x, W[name + ".alpha"], W[name], W[name + ".b"])

    for i, inject in layer_schedule(len(cfg["layers"]), cfg.get("loop")):
        L = cfg["layers"][i]
        if inject:
            x = x + x0
        mw = {k[len(f"l{i}.mix."):]: v for k, v in W.items() if k.startswith(f"l{i}.mix.")}
        h = norm(f"l{i}.norm1", x)
        y = min_gru(h, mw) if L["type"] == "mingru" else differential_attention(h, mw, L["mixer"], eps)
        x = x + m * y
        if L.get("mlp"):
            fw = {k[len(f"l{i}.mlp."):]: v for k, v in W.items() if k.startswith(f"l{i}.mlp.")}
            x = x + m * swiglu_mlp(norm(f"l{i}.norm2", x), fw)
        if trace is not None:
            trace.append(x)
    return norm("final.norm", x) @ W["head"].T
