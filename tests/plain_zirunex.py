"""Plain, slow oracle of the Zirunex decoder: one function per mechanism, no cache, whole sequences, written with elementary
torch expressions only. Works in the precision of the tensors it is given (float64 in the tests). Nothing here is imported
from the package under test."""
import torch


def rms_unit(x, eps):
    """Rows divided by their root mean square."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def norm_around_one(x, w, eps):
    """RMS norm whose stored weight is the difference from one."""
    return rms_unit(x, eps) * (1.0 + w)


def head_norm(x, w, eps):
    """`x (tokens, heads, dim)`: every head's RMS norm, one plain weight for all heads."""
    return rms_unit(x, eps) * w


def window_mask(n, size=None, keep_first=0):
    """`(n, n)` bool: may query i look at key j."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    near = torch.ones(n, n, dtype=torch.bool) if size is None else i - j < size
    return (j <= i) & (near | (j < keep_first))


def sink_weights(s):
    """Softmax over the last axis with one more score of 0 that takes part in the sum only."""
    top = s.max(dim=-1, keepdim=True).values.clamp(min=0.0)
    e = torch.exp(s - top)
    return e / (torch.exp(-top) + e.sum(dim=-1, keepdim=True))


def sink_attention(q, k, v, mask, scale):
    """One head: `q (n, d)`, `k (n, d)`, `v (n, dv)`."""
    s = (q @ k.T) * scale
    return sink_weights(s.masked_fill(~mask, float("-inf"))) @ v


def gated(o, g):
    return o * torch.sigmoid(g)


def window_attention(h, w, mix, eps):
    """The whole attention mixer on `h (n, width)`; `w` maps tensor names (q, k, v, g, o, q.norm, k.norm) to weights."""
    n = h.shape[0]
    H, G, d, dv = mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    q = head_norm((h @ w["q"].T).reshape(n, H, d), w["q.norm"], eps)
    k = head_norm((h @ w["k"].T).reshape(n, G, d), w["k.norm"], eps)
    v = (h @ w["v"].T).reshape(n, G, dv)
    m = mix.get("mask") or {}
    mask = window_mask(n, m.get("size"), m.get("keep_first") or 0)
    heads = []
    for i in range(H):
        g = i // (H // G)
        heads.append(sink_attention(q[:, i], k[:, g], v[:, g], mask, mix["scale"]))
    return gated(torch.cat(heads, dim=-1), h @ w["g"].T) @ w["o"].T


def clamped_glu(gate, up, limit):
    g = torch.minimum(gate, torch.full_like(gate, limit))
    u = up.clamp(-limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1.0)


def feed_forward(h, w, limit):
    return clamped_glu(h @ w["gate"].T, h @ w["up"].T, limit) @ w["down"].T


def weights_index(layers, i):
    """The layer whose tensors layer `i` uses."""
    while layers[i].get("weights_of") is not None:
        i = layers[i]["weights_of"]
    return i


def forward(cfg, weights, tokens, trace=None):
    """Logits `(n, vocab)` of one sequence. `trace`: list that receives the residual stream after every layer."""
    W, eps = weights, cfg["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    for i, L in enumerate(cfg["layers"]):
        j = weights_index(cfg["layers"], i)

        def sub(part):
            p = f"l{j}.{part}."
            return {k[len(p):]: v for k, v in W.items() if k.startswith(p)}

        h = norm_around_one(x, W[f"l{j}.norm1"], eps)
        y = window_attention(h, sub("mix"), L["mixer"], eps)
        if L.get("mlp"):
            y = y + feed_forward(h, sub("mlp"), L["mlp"]["limit"])
        x = x + y
        if trace is not None:
            trace.append(x)
    return norm_around_one(x, W["final.norm"], eps) @ W["head"].T
