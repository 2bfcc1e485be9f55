"""Zirunex: a decoder-only language model of parallel layers with sliding-window attention.

    x = scale * embed[token];   every layer: h = norm(x), x += attention(h) + feed_forward(h);   logits = head(norm(x))

Norms are RMS norms with weights around one. The attention has grouped heads with normalised queries and keys, no positions,
a window beside the first tokens, which stay visible, a sink in the softmax, and a gate on its output; the feed-forward is a
gated unit with clamped inputs. A layer may share another layer's weights; its cache is its own. The configuration gives each
layer its own sizes.

Both sublayers read the same h and end in the same sum, so a layer is two products: `[q | k | v | g | gate | up]` on h and
`[o | down]` on the attention's and the feed-forward's results side by side.

`Zirunex` describes the model to `SequenceGenerator`: which tensors it needs, how they are made from a checkpoint, what state
a sequence has, and the ops of one portion of tokens.
"""
from dataclasses import dataclass
from typing import Any, Callable, Dict, List, Mapping, Optional, Tuple

import torch

from .. import xl
from ..xl import ops
from .checkpoint import check_tensors, take

__all__ = ["ZirunexConfig", "LayerConfig", "WindowAttentionConfig", "ClampedGluConfig", "Zirunex"]

SINK_SCORE = 0.0  # score of the sink of every attention head
GLU_SLOPE, GLU_SHIFT = 1.702, 1.0  # g * sigmoid(slope * g) * (u + shift)

Rows = Tuple[xl.Tensor, Optional[xl.Tensor]]  # normalised rows, or rows of a deferred norm and their sums of squares


@dataclass(frozen=True)
class WindowAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int = 0  # 0: all earlier positions are visible
    keep_first: int = 0

    @classmethod
    def from_dict(cls, d):
        d = take(d, "attention", ("heads", "kv_heads", "dim", "vdim", "scale"), ("mask",))
        mask = take(d["mask"], "mask", ("size",), ("keep_first",)) if d["mask"] else {"size": 0, "keep_first": 0}
        c = cls(int(d["heads"]), int(d["kv_heads"]), int(d["dim"]), int(d["vdim"]), float(d["scale"]), int(mask["size"]),
                int(mask["keep_first"] or 0))
        if max(c.dim, c.vdim) > 512:
            raise ValueError(f"the attention kernels take dim and vdim up to 512, not {c.dim} and {c.vdim}")
        if c.heads % c.kv_heads:
            raise ValueError(f"heads ({c.heads}) must be a multiple of kv_heads ({c.kv_heads})")
        if c.scale <= 0 or (d["mask"] and (c.window < 1 or c.keep_first < 0)):
            raise ValueError(f"scale ({c.scale}) and mask.size ({c.window}) must be positive, mask.keep_first "
                             f"({c.keep_first}) not negative")
        return c

    @property
    def proj_cols(self) -> int:
        """Columns of `[q | k | v | g]`."""
        return (self.heads + self.kv_heads) * self.dim + (self.kv_heads + self.heads) * self.vdim

    @property
    def out_cols(self) -> int:
        return self.heads * self.vdim


@dataclass(frozen=True)
class ClampedGluConfig:
    ff: int
    limit: float

    @classmethod
    def from_dict(cls, d):
        d = take(d, "mlp", ("ff", "limit"), ("kind",))
        if d["kind"] not in (None, "dense"):
            raise ValueError(f"unknown feed-forward kind {d['kind']!r}")
        return cls(int(d["ff"]), float(d["limit"]))


@dataclass(frozen=True)
class LayerConfig:
    mixer: WindowAttentionConfig
    mlp: Optional[ClampedGluConfig] = None
    weights_of: Optional[int] = None  # the layer whose tensors this one uses

    @classmethod
    def from_dict(cls, d):
        d = take(d, "layer", ("type", "mixer"), ("mlp", "weights_of"))
        if d["type"] != "attention":
            raise ValueError(f"unknown layer type {d['type']!r}")
        return cls(WindowAttentionConfig.from_dict(d["mixer"]), ClampedGluConfig.from_dict(d["mlp"]) if d["mlp"] else None,
                   None if d["weights_of"] is None else int(d["weights_of"]))

    @property
    def ff(self) -> int:
        return self.mlp.ff if self.mlp else 0

    @property
    def joint_cols(self) -> int:
        """Columns of the attention's and the feed-forward's results side by side."""
        return self.mixer.out_cols + self.ff


@dataclass(frozen=True)
class ZirunexConfig:
    vocab: int
    width: int
    layers: Tuple[LayerConfig, ...]
    eps: float = 1e-6
    embed_scale: float = 1.0

    ARCHITECTURE = "Zirunex"

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "ZirunexConfig":
        d = take(d, "configuration", ("vocab", "width", "layers", "norm"), ("architecture", "embedding"))
        emb = take(d["embedding"], "embedding", ("scale",)) if d["embedding"] else {"scale": 1.0}
        layers = tuple(LayerConfig.from_dict(e) for e in d["layers"])
        for i, L in enumerate(layers):
            j = L.weights_of
            if j is not None and not (0 <= j < len(layers) and j != i):
                raise ValueError(f"layer {i} cannot share the weights of layer {j}")
        c = cls(int(d["vocab"]), int(d["width"]), layers, float(take(d["norm"], "norm", ("eps",))["eps"]), float(emb["scale"]))
        for i, L in enumerate(layers):
            owner = layers[c.weights_index(i)]
            if (L.mixer, L.mlp) != (owner.mixer, owner.mlp):
                raise ValueError(f"layer {i} differs from layer {c.weights_index(i)}, whose weights it shares")
        return c

    def weights_index(self, i: int) -> int:
        """The layer that owns the tensors of layer `i`."""
        for _ in self.layers:
            if self.layers[i].weights_of is None:
                return i
            i = self.layers[i].weights_of
        raise ValueError(f"layer {i} shares its weights in a circle")

    def owners(self) -> List[int]:
        """Layers with tensors of their own."""
        return [i for i, L in enumerate(self.layers) if L.weights_of is None]

    def param_count(self) -> int:
        return 2 * self.vocab * self.width + sum(self.width * (L.mixer.proj_cols + 2 * L.ff + L.joint_cols)
                                                 for L in (self.layers[i] for i in self.owners()))


class Zirunex:
    """Weights, state and step of the model for `SequenceGenerator`."""

    config_class = ZirunexConfig

    def __init__(self, cfg: ZirunexConfig, dtype: str = "bfloat16"):
        self.cfg = cfg
        self.dtype = xl.dtype.as_dtype(dtype)
        self.vocab, self.width = cfg.vocab, cfg.width

    # -- weights ---------------------------------------------------------------------------------------------------
    def checkpoint_tensors(self) -> Dict[str, Tuple[int, ...]]:
        """Names and shapes of the tensors of a checkpoint."""
        c = self.cfg
        out: Dict[str, Tuple[int, ...]] = {"embed": (c.vocab, c.width), "head": (c.vocab, c.width), "final.norm": (c.width,)}
        for i in c.owners():
            L, m, p = c.layers[i], c.layers[i].mixer, f"l{i}.mix."
            out.update({f"l{i}.norm1": (c.width,), p + "q": (m.heads * m.dim, c.width), p + "k": (m.kv_heads * m.dim, c.width),
                        p + "v": (m.kv_heads * m.vdim, c.width), p + "g": (m.out_cols, c.width), p + "o": (c.width, m.out_cols),
                        p + "q.norm": (m.dim,), p + "k.norm": (m.dim,)})
            if L.ff:
                out.update({f"l{i}.mlp.gate": (L.ff, c.width), f"l{i}.mlp.up": (L.ff, c.width),
                            f"l{i}.mlp.down": (c.width, L.ff)})
        return out

    def weights(self) -> Dict[str, Tuple[Tuple[int, ...], xl.dtype]]:
        """The tensors the program runs on: linears that read the same input or end in the same sum share one matrix, norms
        are fp32 factors."""
        c, dt, f32 = self.cfg, self.dtype, xl.float32
        out: Dict[str, Tuple[Tuple[int, ...], xl.dtype]] = {
            "embed": ((c.vocab, c.width), dt), "head": ((c.vocab, c.width), dt), "final.norm": ((c.width,), f32)}
        for i in c.owners():
            L, m = c.layers[i], c.layers[i].mixer
            out.update({f"l{i}.norm": ((c.width,), f32), f"l{i}.q_norm": ((m.dim,), f32), f"l{i}.k_norm": ((m.dim,), f32),
                        f"l{i}.in": ((m.proj_cols + 2 * L.ff, c.width), dt), f"l{i}.out": ((c.width, L.joint_cols), dt)})
        return out

    def convert(self, ckpt: Mapping[str, torch.Tensor], device) -> Dict[str, torch.Tensor]:
        """Checkpoint tensors -> program tensors (in the checkpoint's precision; the caller casts on copy)."""
        check_tensors(ckpt, self.checkpoint_tensors())

        def get(k):
            return ckpt[k].to(device)

        out = {"embed": get("embed"), "head": get("head"), "final.norm": 1.0 + get("final.norm").float()}
        for i in self.cfg.owners():
            p, mlp = f"l{i}.mix.", f"l{i}.mlp."
            has_ff = self.cfg.layers[i].ff > 0
            out[f"l{i}.norm"] = 1.0 + get(f"l{i}.norm1").float()
            out[f"l{i}.q_norm"], out[f"l{i}.k_norm"] = get(p + "q.norm"), get(p + "k.norm")
            out[f"l{i}.in"] = torch.cat([get(p + k) for k in ("q", "k", "v", "g")]
                                        + ([get(mlp + "gate"), get(mlp + "up")] if has_ff else []))
            out[f"l{i}.out"] = torch.cat([get(p + "o")] + ([get(mlp + "down")] if has_ff else []), dim=1)
        return out

    def random_weights(self, seed: int, device) -> Dict[str, torch.Tensor]:
        """Random program tensors that keep the stream in a sensible range (benchmarks)."""
        gen = torch.Generator(device=device).manual_seed(seed)

        def normal(shape, std):
            return torch.empty(shape, dtype=torch.float32, device=device).normal_(0.0, std, generator=gen)

        return {name: 1.0 + normal(shape, 0.1) if len(shape) == 1 else normal(shape, shape[-1] ** -0.5)
                for name, (shape, _) in self.weights().items()}

    # -- state and constants -----------------------------------------------------------------------------------------
    def state(self, batch: int, max_seq: int) -> Dict[str, Tuple[Tuple[int, ...], xl.dtype]]:
        """Per-sequence caches of every layer (also of those that share weights)."""
        out = {}
        for i, L in enumerate(self.cfg.layers):
            m = L.mixer
            out[f"l{i}.k"] = ((batch, m.kv_heads, max_seq, m.dim), self.dtype)
            out[f"l{i}.v"] = ((batch, m.kv_heads, max_seq, m.vdim), self.dtype)
        return out

    def tables(self, max_seq: int) -> Dict[str, Any]:
        return {}

    # -- one portion ---------------------------------------------------------------------------------------------------
    def _deferred(self, rows: int) -> bool:
        """Whether the norms inside the layers are finished by the products that read them: few rows, sizes that the small-M
        kernels take."""
        c = self.cfg
        return (rows <= 16 and self.dtype == xl.bfloat16 and c.width % 8 == 0
                and all(L.joint_cols % 8 == 0 for L in c.layers))

    def portion(self, T: int, t: Callable[[str], xl.Tensor], tokens: xl.Tensor, pos: xl.Tensor, count: xl.Tensor,
                final_norm: bool) -> Optional[Rows]:
        """Run `T` tokens per sequence through all layers. `t(name)` gives weights, state and the stream buffer
        (`"stream"`); `tokens (batch * T,)`. With `final_norm` the last residual update also returns the final norm of
        every row (decoding), else the stream is left for `select`."""
        c = self.cfg
        x, deferred = t("stream"), self._deferred(tokens.shape[0])
        norms = [f"l{c.weights_index(i)}.norm" for i in range(len(c.layers))] + (["final.norm"] if final_norm else [])
        h = ops.embed_rms_(x, tokens, t("embed"), t(norms[0]), c.embed_scale, c.eps)
        rows: Rows = (h, None)
        for i, L in enumerate(c.layers):
            m, w = L.mixer, f"l{c.weights_index(i)}."
            h, sumsq = rows
            proj, joint = ops.linear_split_glu(h, t(w + "in"), m.proj_cols, m.out_cols, L.mlp.limit if L.mlp else 0.0,
                                               GLU_SLOPE, GLU_SHIFT, sumsq, c.eps)
            joint = ops.window_attention_(proj, t(w + "q_norm"), t(w + "k_norm"), t(f"l{i}.k"), t(f"l{i}.v"), pos, count, joint,
                                          T, m.heads, m.scale, m.window, m.keep_first, SINK_SCORE, c.eps)
            after = t(norms[i + 1]) if i + 1 < len(norms) else None
            rows = ops.linear_residual_rms_(x, joint, t(w + "out"), after, c.eps, deferred=deferred)
        return rows if final_norm else None

    def logits(self, t: Callable[[str], xl.Tensor], rows: Rows) -> xl.Tensor:
        h, sumsq = rows
        return ops.linear_rows(h, t("head"), xl.float32, sumsq, self.cfg.eps)

    def select(self, t: Callable[[str], xl.Tensor], idx: xl.Tensor, stride: int = 0, offset: int = 0) -> Rows:
        """Final norm of selected rows of the stream."""
        return ops.select_rms(t("stream"), idx, t("final.norm"), stride, offset, self.cfg.eps, self.dtype), None
