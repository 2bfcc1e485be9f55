"""Dunelix: a decoder-only language model of minGRU and differential-attention layers with Dynamic Tanh norms, an optional
loop over a range of layers, and a scaled residual.

    x = embed[token];   every layer: x += m * mixer(norm1(x)), x += m * feed_forward(norm2(x));   logits = head(norm(x))

The looped layers run several times with the same weights; before every pass but the first the embedding output is added to
the stream. Every pass keeps its own cache and state. The configuration gives each layer its own sizes.

`Dunelix` describes the model to `SequenceGenerator`: which tensors it needs, how they are made from a checkpoint, what state
a sequence has, and the ops of one portion of tokens.
"""
from dataclasses import dataclass
from typing import Any, Callable, Dict, List, Mapping, Optional, Tuple, Union

import torch

from .. import xl
from ..ops.rotary_pos_embed import frequency_tables, rotary_frequencies
from ..xl import ops
from .checkpoint import check_tensors, take

__all__ = ["DunelixConfig", "LayerConfig", "MinGRUConfig", "DiffAttentionConfig", "RotaryConfig", "Dunelix"]


@dataclass(frozen=True)
class RotaryConfig:
    dims: int
    base: float
    scaling: Optional[Tuple[Tuple[str, float], ...]] = None  # (name, value) pairs: factor, low, high, original

    @classmethod
    def from_dict(cls, d):
        d = take(d, "rot", ("base", "dims"), ("scaling",))
        sc = d["scaling"]
        if sc:
            sc = tuple(sorted(take(sc, "rot.scaling", ("factor", "low", "high", "original")).items()))
        return cls(int(d["dims"]), float(d["base"]), sc or None)


@dataclass(frozen=True)
class MinGRUConfig:
    width: int


@dataclass(frozen=True)
class DiffAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    diff: float
    scale: float
    chunk: int = 0
    rot: Optional[RotaryConfig] = None


@dataclass(frozen=True)
class LayerConfig:
    mixer: Union[MinGRUConfig, DiffAttentionConfig]
    ff: int = 0  # 0: the layer has no feed-forward

    @classmethod
    def from_dict(cls, d):
        d = take(d, "layer", ("type", "mixer"), ("mlp",))
        kind, m = d["type"], d["mixer"]
        if kind == "mingru":
            mixer = MinGRUConfig(int(take(m, "mingru", ("width",))["width"]))
        elif kind == "attention":
            m = take(m, "attention", ("heads", "kv_heads", "dim", "vdim", "diff", "scale"), ("mask", "rot"))
            mask = take(m["mask"], "mask", ("size",)) if m["mask"] else {"size": 0}
            mixer = DiffAttentionConfig(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["diff"]),
                                        float(m["scale"]), int(mask["size"]),
                                        RotaryConfig.from_dict(m["rot"]) if m["rot"] else None)
            if max(mixer.dim, mixer.vdim) > 512:
                raise ValueError(f"the attention kernels take dim and vdim up to 512, not {mixer.dim} and {mixer.vdim}")
            if mixer.heads % mixer.kv_heads:
                raise ValueError(f"heads ({mixer.heads}) must be a multiple of kv_heads ({mixer.kv_heads})")
            if mixer.rot and (mixer.rot.dims % 2 or mixer.rot.dims > mixer.dim):
                raise ValueError(f"rot.dims ({mixer.rot.dims}) must be even and at most dim ({mixer.dim})")
        else:
            raise ValueError(f"unknown layer type {kind!r}")
        ff = 0
        if d["mlp"]:
            mlp = take(d["mlp"], "mlp", ("ff",), ("kind",))
            if mlp["kind"] not in (None, "dense"):
                raise ValueError(f"unknown feed-forward kind {mlp['kind']!r}")
            ff = int(mlp["ff"])
        return cls(mixer, ff)


@dataclass(frozen=True)
class DunelixConfig:
    vocab: int
    width: int
    layers: Tuple[LayerConfig, ...]
    loop: Optional[Tuple[int, int, int]] = None  # start, stop, times
    eps: float = 1e-6
    residual_mult: float = 1.0

    ARCHITECTURE = "Dunelix"

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "DunelixConfig":
        d = take(d, "configuration", ("vocab", "width", "layers", "norm"), ("architecture", "loop", "residual_mult"))
        loop = None
        if d["loop"]:
            lp = take(d["loop"], "loop", ("start", "stop", "times"))
            loop = (int(lp["start"]), int(lp["stop"]), int(lp["times"]))
            if not 0 <= loop[0] < loop[1] <= len(d["layers"]) or loop[2] < 1:
                raise ValueError(f"loop {loop} does not fit {len(d['layers'])} layers")
        mult = d["residual_mult"]
        return cls(int(d["vocab"]), int(d["width"]), tuple(LayerConfig.from_dict(e) for e in d["layers"]), loop,
                   float(take(d["norm"], "norm", ("eps",))["eps"]), 1.0 if mult is None else float(mult))

    def schedule(self) -> List[Tuple[int, bool]]:
        """Layer runs in order: `(layer, whether the embedding output is added to the stream before it)`."""
        start, stop, times = self.loop or (0, 0, 0)
        if not times:
            return [(i, False) for i in range(len(self.layers))]
        runs = [(i, False) for i in range(start)]
        for t in range(times):
            runs += [(i, t > 0 and i == start) for i in range(start, stop)]
        return runs + [(i, False) for i in range(stop, len(self.layers))]

    def param_count(self) -> int:
        n = 2 * self.vocab * self.width
        for L in self.layers:
            m = L.mixer
            if isinstance(m, MinGRUConfig):
                n += 4 * m.width * self.width
            else:
                n += self.width * (2 * (m.heads + m.kv_heads) * m.dim + (m.kv_heads + m.heads) * m.vdim)
            n += 3 * L.ff * self.width
        return n


class Dunelix:
    """Weights, state and step of the model for `SequenceGenerator`."""

    config_class = DunelixConfig

    def __init__(self, cfg: DunelixConfig, dtype: str = "bfloat16"):
        self.cfg = cfg
        self.dtype = xl.dtype.as_dtype(dtype)
        self.vocab, self.width = cfg.vocab, cfg.width

    # -- weights ---------------------------------------------------------------------------------------------------
    def _norm_names(self) -> List[str]:
        names = []
        for i, L in enumerate(self.cfg.layers):
            names += [f"l{i}.norm1"] + ([f"l{i}.norm2"] if L.ff else [])
        return names + ["final.norm"]

    def checkpoint_tensors(self) -> Dict[str, Tuple[int, ...]]:
        """Names and shapes of the tensors of a checkpoint."""
        c = self.cfg
        out: Dict[str, Tuple[int, ...]] = {"embed": (c.vocab, c.width), "head": (c.vocab, c.width)}
        for n in self._norm_names():
            out.update({n: (c.width,), f"{n}.b": (c.width,), f"{n}.alpha": ()})
        for i, L in enumerate(c.layers):
            m, p = L.mixer, f"l{i}.mix."
            if isinstance(m, MinGRUConfig):
                out.update({p + k: (m.width, c.width) for k in ("z", "x", "g")})
                out.update({p + "z.b": (m.width,), p + "x.b": (m.width,), p + "o": (c.width, m.width)})
            else:
                out.update({p + "q": (m.heads * 2 * m.dim, c.width), p + "k": (m.kv_heads * 2 * m.dim, c.width),
                            p + "v": (m.kv_heads * m.vdim, c.width), p + "o": (c.width, m.heads * m.vdim)})
                out.update({p + k: (m.dim,) for k in ("lq1", "lk1", "lq2", "lk2")})
            if L.ff:
                out.update({f"l{i}.mlp.gate": (L.ff, c.width), f"l{i}.mlp.up": (L.ff, c.width),
                            f"l{i}.mlp.down": (c.width, L.ff)})
        return out

    def weights(self) -> Dict[str, Tuple[Tuple[int, ...], xl.dtype]]:
        """The tensors the program runs on: linears that read the same input share one matrix, norms and biases are fp32."""
        c, dt, f32 = self.cfg, self.dtype, xl.float32
        out: Dict[str, Tuple[Tuple[int, ...], xl.dtype]] = {"embed": ((c.vocab, c.width), dt), "head": ((c.vocab, c.width), dt)}
        for n in self._norm_names():
            out.update({f"{n}.alpha": ((1,), f32), f"{n}.w": ((c.width,), f32), f"{n}.b": ((c.width,), f32)})
        for i, L in enumerate(c.layers):
            m = L.mixer
            if isinstance(m, MinGRUConfig):
                out.update({f"l{i}.zxg": ((3 * m.width, c.width), dt), f"l{i}.z_bias": ((m.width,), f32),
                            f"l{i}.x_bias": ((m.width,), f32), f"l{i}.o": ((c.width, m.width), dt)})
            else:
                rows = 2 * (m.heads + m.kv_heads) * m.dim + m.kv_heads * m.vdim
                out.update({f"l{i}.qkv": ((rows, c.width), dt), f"l{i}.o": ((c.width, m.heads * m.vdim), dt),
                            f"l{i}.lambda": ((1,), f32)})
            if L.ff:
                out.update({f"l{i}.gate_up": ((2 * L.ff, c.width), dt), f"l{i}.down": ((c.width, L.ff), dt)})
        return out

    def convert(self, ckpt: Mapping[str, torch.Tensor], device) -> Dict[str, torch.Tensor]:
        """Checkpoint tensors -> program tensors (in the checkpoint's precision; the caller casts on copy)."""
        check_tensors(ckpt, self.checkpoint_tensors())

        def get(k):
            return ckpt[k].to(device)

        out = {"embed": get("embed"), "head": get("head")}
        for n in self._norm_names():
            out.update({f"{n}.alpha": get(f"{n}.alpha").reshape(1), f"{n}.w": get(n), f"{n}.b": get(f"{n}.b")})
        for i, L in enumerate(self.cfg.layers):
            m, p = L.mixer, f"l{i}.mix."
            out[f"l{i}.o"] = get(p + "o")
            if isinstance(m, MinGRUConfig):
                out[f"l{i}.zxg"] = torch.cat([get(p + k) for k in ("z", "x", "g")])
                out[f"l{i}.z_bias"], out[f"l{i}.x_bias"] = get(p + "z.b"), get(p + "x.b")
            else:
                out[f"l{i}.qkv"] = torch.cat([get(p + k) for k in ("q", "k", "v")])
                lq1, lk1, lq2, lk2 = (get(p + k).float() for k in ("lq1", "lk1", "lq2", "lk2"))
                out[f"l{i}.lambda"] = (torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum()) + m.diff).reshape(1)
            if L.ff:
                out[f"l{i}.gate_up"] = torch.cat([get(f"l{i}.mlp.gate"), get(f"l{i}.mlp.up")])
                out[f"l{i}.down"] = get(f"l{i}.mlp.down")
        return out

    def random_weights(self, seed: int, device) -> Dict[str, torch.Tensor]:
        """Random program tensors that keep the stream and the recurrences in a sensible range (benchmarks)."""
        gen = torch.Generator(device=device).manual_seed(seed)

        def normal(shape, std):
            return torch.empty(shape, dtype=torch.float32, device=device).normal_(0.0, std, generator=gen)

        out = {}
        for name, (shape, _) in self.weights().items():
            leaf = name.rsplit(".", 1)[-1]
            if leaf == "alpha":
                out[name] = torch.full(shape, 0.5, device=device)
            elif leaf == "w":
                out[name] = 1.0 + normal(shape, 0.1)
            elif leaf == "z_bias":
                out[name] = normal(shape, 1.0) - 3.0
            elif leaf == "lambda":
                out[name] = torch.full(shape, 0.6, device=device)
            elif len(shape) == 1:
                out[name] = normal(shape, 0.1)
            else:
                out[name] = normal(shape, 1.0 if leaf == "embed" else shape[-1] ** -0.5)
        return out

    # -- state and constants -----------------------------------------------------------------------------------------
    def state(self, batch: int, max_seq: int) -> Dict[str, Tuple[Tuple[int, ...], xl.dtype]]:
        """Per-sequence state of every layer run (each pass of the loop has its own)."""
        out = {}
        for r, (i, _) in enumerate(self.cfg.schedule()):
            m = self.cfg.layers[i].mixer
            if isinstance(m, MinGRUConfig):
                out[f"run{r}.state"] = ((batch, m.width), xl.float32)
            else:
                out[f"run{r}.k"] = ((batch, m.kv_heads, 2, max_seq, m.dim), self.dtype)
                out[f"run{r}.v"] = ((batch, m.kv_heads, max_seq, m.vdim), self.dtype)
        return out

    def tables(self, max_seq: int) -> Dict[str, Any]:
        """Constant fp32 tables: cosine and sine of every rotary setting in use."""
        out = {}
        for L in self.cfg.layers:
            rot = getattr(L.mixer, "rot", None)
            if rot and rot.dims and f"{self._table_name(rot)}.cos" not in out:
                sin, cos = frequency_tables(max_seq, rotary_frequencies(rot.dims, rot.base, dict(rot.scaling or ())))
                out[f"{self._table_name(rot)}.cos"], out[f"{self._table_name(rot)}.sin"] = cos, sin
        return out

    @staticmethod
    def _table_name(rot: RotaryConfig) -> str:
        return "rot_" + "_".join(str(v) for v in (rot.dims, rot.base, *(v for _, v in rot.scaling or ())))

    # -- one portion ---------------------------------------------------------------------------------------------------
    def portion(self, T: int, t: Callable[[str], xl.Tensor], tokens: xl.Tensor, pos: xl.Tensor, count: xl.Tensor,
                final_norm: bool) -> Optional[xl.Tensor]:
        """Run `T` tokens per sequence through all layers. `t(name)` gives weights, state, tables and the stream buffer
        (`"stream"`); `tokens (batch * T,)`. With `final_norm` the last residual update also returns the final norm of
        every row (decoding), else the stream is left for `select_dyt`."""
        c = self.cfg
        x = t("stream")

        def norm(name):
            return t(f"{name}.alpha"), t(f"{name}.w"), t(f"{name}.b")

        runs = c.schedule()
        h = ops.embed_dyt_(x, tokens, t("embed"), norm(f"l{runs[0][0]}.norm1"))
        for r, (i, _) in enumerate(runs):
            L = c.layers[i]
            if r + 1 < len(runs):
                after, inject = norm(f"l{runs[r + 1][0]}.norm1"), (tokens, t("embed")) if runs[r + 1][1] else None
            else:
                after, inject = norm("final.norm") if final_norm else None, None
            if isinstance(L.mixer, MinGRUConfig):
                y = ops.min_gru_(h, t(f"l{i}.zxg"), t(f"l{i}.z_bias"), t(f"l{i}.x_bias"), t(f"run{r}.state"), pos, count, T)
            else:
                y = self._attention(T, t, h, i, r, pos, count)
            if L.ff:
                h = ops.linear_residual_dyt_(x, y, t(f"l{i}.o"), c.residual_mult, norm(f"l{i}.norm2"))
                y = ops.linear_swiglu(h, t(f"l{i}.gate_up"))
                h = ops.linear_residual_dyt_(x, y, t(f"l{i}.down"), c.residual_mult, after, inject)
            else:
                h = ops.linear_residual_dyt_(x, y, t(f"l{i}.o"), c.residual_mult, after, inject)
        return h

    def _attention(self, T, t, h, i, r, pos, count):
        m = self.cfg.layers[i].mixer
        rot = m.rot.dims if m.rot else 0
        lam = t(f"l{i}.lambda")
        # without rotation the tables are never read: any fp32 tensor stands in
        cos, sin = (t(f"{self._table_name(m.rot)}.{k}") for k in ("cos", "sin")) if rot else (lam, lam)
        qkv = ops.linear_rows(h, t(f"l{i}.qkv"))
        return ops.diff_attention_(qkv, cos, sin, t(f"run{r}.k"), t(f"run{r}.v"), pos, count, lam, T, m.heads, rot, m.scale,
                                   m.chunk, self.cfg.eps, 1.0 - m.diff)

    def logits(self, t: Callable[[str], xl.Tensor], h: xl.Tensor) -> xl.Tensor:
        return ops.linear_rows(h, t("head"), xl.float32)

    def select(self, t: Callable[[str], xl.Tensor], idx: xl.Tensor, stride: int = 0, offset: int = 0) -> xl.Tensor:
        """Final norm of selected rows of the stream."""
        return ops.select_dyt(t("stream"), idx, (t("final.norm.alpha"), t("final.norm.w"), t("final.norm.b")), stride, offset,
                              self.dtype)
