"""Small configurations, random weights and helpers shared by the Dunelix tests."""
import json
import struct

import numpy as np
import torch

import plain_dunelix as plain

RNG = np.random.RandomState


def attention(heads=4, kv_heads=2, dim=16, vdim=24, diff=0.55, size=13, dims=8, base=500.0, scaling=True, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "diff": diff,
         "scale": dim ** -0.5 if scale is None else scale}
    if size:
        m["mask"] = {"size": size}
    if dims:
        m["rot"] = {"base": base, "dims": dims}
        if scaling:
            m["rot"]["scaling"] = {"factor": 4.0, "low": 1.0, "high": 3.0, "original": 64}
    return m


def layer(mixer, ff=40):
    kind = "attention" if "heads" in mixer else "mingru"
    return {"type": kind, "mixer": mixer, "mlp": {"ff": ff, "kind": "dense"} if ff else None}


def config(layers, width=48, vocab=91, loop=None, mult=0.8, eps=1e-5):
    d = {"architecture": "Dunelix", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps},
         "residual_mult": mult}
    if loop:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


CASES = {
    # every layer has sizes of its own; the loop holds both mixers; lengths that are no multiples of anything
    "mixed": config([layer({"width": 40}, 56), layer(attention(), 40), layer({"width": 34}, 0),
                     layer(attention(heads=3, kv_heads=1, dim=24, vdim=16, size=7, dims=24, scaling=False), 24)],
                    loop=(1, 3, 3)),
    # attention first, the loop starts at layer 0, one query head per key head, no rotation, no chunks
    "attention_first": config([layer(attention(heads=2, kv_heads=2, dim=8, vdim=40, dims=0, size=0), 0),
                               layer({"width": 24}, 32)], width=40, vocab=70, loop=(0, 2, 2), mult=1.0),
    # no loop; many query heads on one key head; values narrower than keys; a scale that is not dim^-1/2
    "grouped": config([layer(attention(heads=10, kv_heads=1, dim=32, vdim=8, size=5, dims=6, scale=0.31), 48),
                       layer({"width": 50}, 30), layer({"width": 16}, 16)], width=56, vocab=64, mult=0.6, eps=1e-3),
    # sizes that vector accesses do not divide
    "odd": config([layer({"width": 19}, 21), layer(attention(heads=2, kv_heads=1, dim=10, vdim=7, size=9, dims=4), 13)],
                  width=23, vocab=37, loop=(0, 1, 2), mult=0.9),
}


def checkpoint(cfg, seed=0, dtype=torch.bfloat16):
    """Random tensors under the names of a checkpoint, rounded to `dtype`."""
    g = torch.Generator().manual_seed(seed)

    def n(*shape, std=1.0):
        return (torch.randn(*shape, generator=g) * std).to(dtype)

    w, v = cfg["width"], cfg["vocab"]
    out = {"embed": n(v, w), "head": n(v, w, std=w ** -0.5)}

    def norm(name):
        out[name] = (1.0 + 0.3 * torch.randn(w, generator=g)).to(dtype)
        out[name + ".b"] = n(w, std=0.2)
        out[name + ".alpha"] = torch.tensor(0.4 + 0.4 * float(torch.rand((), generator=g))).to(dtype)

    for i, L in enumerate(cfg["layers"]):
        m, p = L["mixer"], f"l{i}.mix."
        norm(f"l{i}.norm1")
        if L["type"] == "mingru":
            k = m["width"]
            for name in ("z", "x", "g"):
                out[p + name] = n(k, w, std=w ** -0.5)
            out[p + "z.b"], out[p + "x.b"] = (torch.randn(k, generator=g) - 2.0).to(dtype), n(k, std=0.5)
            out[p + "o"] = n(w, k, std=k ** -0.5)
        else:
            H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            out[p + "q"], out[p + "k"] = n(H * 2 * d, w, std=2.0 * w ** -0.5), n(G * 2 * d, w, std=2.0 * w ** -0.5)
            out[p + "v"], out[p + "o"] = n(G * dv, w, std=w ** -0.5), n(w, H * dv, std=(H * dv) ** -0.5)
            for name in ("lq1", "lk1", "lq2", "lk2"):
                out[p + name] = n(d, std=0.15)
        if L["mlp"]:
            f = L["mlp"]["ff"]
            norm(f"l{i}.norm2")
            out[f"l{i}.mlp.gate"], out[f"l{i}.mlp.up"] = n(f, w, std=w ** -0.5), n(f, w, std=w ** -0.5)
            out[f"l{i}.mlp.down"] = n(w, f, std=f ** -0.5)
    norm("final.norm")
    return out


def oracle_logits(cfg, ckpt, tokens):
    return plain.forward(cfg, {k: v.double() for k, v in ckpt.items()}, tokens).numpy()


def generator(cfg, ckpt, device="cpu", dtype="float32", **kw):
    from popxl_addons_b200.models.dunelix import Dunelix, DunelixConfig
    from popxl_addons_b200.models.sequence_generator import SequenceGenerator

    kw.setdefault("max_seq", 96)
    return SequenceGenerator(Dunelix(DunelixConfig.from_dict(cfg), dtype), device=device, **kw).load_checkpoint(ckpt)


def prompt(cfg, n, seed=1):
    return RNG(seed).randint(0, cfg["vocab"], n).tolist()


def error(got, want):
    """Largest root-mean-square difference of a row, relative to the spread of all wanted logits."""
    d = np.asarray(got, np.float64) - want
    return float(np.sqrt((d * d).mean(-1)).max() / want.std())


TOLERANCE = {"float32": 3e-5, "bfloat16": 6e-2}


def write_model(folder, cfg, ckpt):
    names = {torch.bfloat16: "BF16", torch.float32: "F32"}
    header, blob = {}, b""
    for k, v in ckpt.items():
        raw = v.contiguous().reshape(-1).view(torch.uint8).numpy().tobytes()
        header[k] = {"dtype": names[v.dtype], "shape": list(v.shape), "data_offsets": [len(blob), len(blob) + len(raw)]}
        blob += raw
    head = json.dumps(header).encode()
    with open(folder / "model.safetensors", "wb") as f:
        f.write(struct.pack("<Q", len(head)) + head + blob)
    (folder / "config.json").write_text(json.dumps(cfg))
    return str(folder)
