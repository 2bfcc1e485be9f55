"""Small configurations, random weights and helpers shared by the Zirunex tests."""
import torch

import plain_zirunex as plain
from dunelix_cases import TOLERANCE, error, prompt, write_model  # noqa: F401  (not specific to a design)


def attention(heads=4, kv_heads=2, dim=16, vdim=24, size=11, keep=3, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale}
    if size:
        m["mask"] = {"size": size, "keep_first": keep}
    return m


def layer(mixer, ff=40, limit=1.5, weights_of=None):
    d = {"type": "attention", "mixer": mixer, "mlp": {"ff": ff, "kind": "dense", "limit": limit} if ff else None}
    if weights_of is not None:
        d["weights_of"] = weights_of
    return d


def config(layers, width=48, vocab=91, scale=5.0, eps=1e-5):
    return {"architecture": "Zirunex", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps},
            "embedding": {"scale": scale}}


_WIDE = attention(heads=6, kv_heads=1, dim=24, vdim=16, size=7, keep=9, scale=0.3)

CASES = {
    # every layer has sizes of its own; shared weights in an order that is not the first layers'; a window shorter than the
    # kept tokens; a layer without feed-forward
    "mixed": config([layer(attention(), 40), layer(_WIDE, 56, 0.8), layer(attention(heads=3, kv_heads=3, dim=8, vdim=40, size=16,
                                                                                  keep=1), 0),
                     layer(_WIDE, 56, 0.8, weights_of=1), layer(attention(), 40, weights_of=0),
                     layer(_WIDE, 56, 0.8, weights_of=1)]),
    # no window; no kept tokens; the owner of the weights comes later; an embedding scale of 1
    "later_owner": config([layer(attention(heads=2, kv_heads=1, dim=32, vdim=8, size=0), 24, 2.0, weights_of=2),
                           layer(attention(heads=8, kv_heads=2, dim=8, vdim=16, size=5, keep=0), 32, 0.5),
                           layer(attention(heads=2, kv_heads=1, dim=32, vdim=8, size=0), 24, 2.0)],
                          width=40, vocab=70, scale=1.0, eps=1e-3),
    # one layer, windows of one position, one query head
    "single": config([layer(attention(heads=1, kv_heads=1, dim=16, vdim=16, size=1, keep=2), 16, 3.0)], width=32, vocab=40),
    # sizes that vector accesses do not divide
    "odd": config([layer(attention(heads=2, kv_heads=1, dim=10, vdim=7, size=9, keep=4), 13),
                   layer(attention(heads=3, kv_heads=1, dim=5, vdim=3, size=4, keep=2), 0)], width=23, vocab=37, scale=0.7),
}


def checkpoint(cfg, seed=0, dtype=torch.bfloat16):
    """Random tensors under the names of a checkpoint, rounded to `dtype`. Queries and keys are large enough for single keys to
    stand out, gates and clamped inputs reach both sides of their limits."""
    g = torch.Generator().manual_seed(seed)

    def n(*shape, std=1.0, mean=0.0):
        return (torch.randn(*shape, generator=g) * std + mean).to(dtype)

    w, v = cfg["width"], cfg["vocab"]
    out = {"embed": n(v, w), "head": n(v, w, std=w ** -0.5), "final.norm": n(w, std=0.3)}
    for i, L in enumerate(cfg["layers"]):
        if L.get("weights_of") is not None:
            continue
        m, p = L["mixer"], f"l{i}.mix."
        H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        out[f"l{i}.norm1"] = n(w, std=0.3)
        out[p + "q"], out[p + "k"] = n(H * d, w, std=w ** -0.5), n(G * d, w, std=w ** -0.5)
        out[p + "v"], out[p + "g"] = n(G * dv, w, std=w ** -0.5), n(H * dv, w, std=2.0 * w ** -0.5)
        out[p + "o"] = n(w, H * dv, std=3.0 * (H * dv) ** -0.5)
        out[p + "q.norm"], out[p + "k.norm"] = n(d, std=0.3, mean=1.6), n(d, std=0.3, mean=1.2)
        if L["mlp"]:
            f = L["mlp"]["ff"]
            out[f"l{i}.mlp.gate"], out[f"l{i}.mlp.up"] = n(f, w, std=1.5 * w ** -0.5), n(f, w, std=1.5 * w ** -0.5)
            out[f"l{i}.mlp.down"] = n(w, f, std=f ** -0.5)
    return out


def oracle_logits(cfg, ckpt, tokens):
    return plain.forward(cfg, {k: v.double() for k, v in ckpt.items()}, tokens).numpy()


def generator(cfg, ckpt, device="cpu", dtype="float32", **kw):
    from popxl_addons_b200.models.sequence_generator import SequenceGenerator
    from popxl_addons_b200.models.zirunex import Zirunex, ZirunexConfig

    kw.setdefault("max_seq", 96)
    return SequenceGenerator(Zirunex(ZirunexConfig.from_dict(cfg), dtype), device=device, **kw).load_checkpoint(ckpt)
