"""The Dezelorn decoder: configuration record and parameter layout.

A decoder whose layers are listed one by one in the configuration, each with its own sizes:

* every norm is a Dynamic Tanh, ``tanh(alpha * x) * w + b`` (elementwise, no statistics), before AND after each sublayer;
* attention over a sliding window with grouped key heads. The values are the keys, q and k pass through a short causal
  convolution over time, the query carries a position-dependent temperature, a per-head logarithmic distance bias is
  subtracted from the scores, the softmax weights are mixed across heads by a matrix, and the result is gated;
* an optional SwiGLU feed-forward.

The kernels want head sizes that are multiples of 64 and row pitches that are multiples of 8 elements. The layout
therefore pads heads, width and feed-forward with zeros, which changes nothing: a padded channel has zero weights on both
sides, its norm weight and bias are zero, and the gate multiplies a zero. The checkpoint boundary (``hf_items``) hands
out views without the padding.
"""
from __future__ import annotations

import math
from dataclasses import asdict, dataclass, replace
from typing import Any, Dict, Iterator, List, Optional, Tuple

import torch

from .layout import ParamLayout


def _up(x: int, m: int) -> int:
    return (x + m - 1) // m * m


@dataclass(frozen=True)
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    conv: int            # taps of the short convolution on q and k
    window: int          # a position sees itself and the window - 1 tokens before it
    temp_coef: float
    temp_every: float
    scale: float

    @property
    def group(self) -> int:
        return self.heads // self.kv_heads

    @property
    def dim_p(self) -> int:
        return _up(self.dim, 64)

    @property
    def q_dim(self) -> int:
        return self.heads * self.dim_p

    @property
    def k_dim(self) -> int:
        return self.kv_heads * self.dim_p

    @property
    def qk_dim(self) -> int:
        return self.q_dim + self.k_dim

    @property
    def u_dim(self) -> int:
        """Columns of the fused projection: q, k, gate."""
        return self.qk_dim + self.q_dim


@dataclass(frozen=True)
class LayerSpec:
    mixer: AttentionSpec
    ff: Optional[int]    # None = no feed-forward

    @property
    def ff_p(self) -> int:
        return _up(self.ff or 0, 8)


@dataclass(frozen=True)
class DezelornConfig:
    vocab_size: int
    width: int
    layers: Tuple[LayerSpec, ...]
    embedding_scale: float
    norm_eps: float = 1e-6      # part of the configuration format; Dynamic Tanh has no use for it
    max_position_embeddings: int = 131072
    eos_token_id: int = -1
    bos_token_id: Optional[int] = None
    initializer_range: float = 0.02
    model_type: str = "dezelorn"
    architecture: str = "Dezelorn"

    @property
    def hidden_size(self) -> int:
        return _up(self.width, 8)

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @property
    def max_window(self) -> int:
        return max(l.mixer.window for l in self.layers)

    def first_layers(self, n: int) -> "DezelornConfig":
        """The same model with its first ``n`` layers (benchmarks)."""
        return replace(self, layers=self.layers[:n])

    def num_parameters(self) -> int:
        n = 2 * self.vocab_size * self.width + 2 * self.width + 1
        for l in self.layers:
            m = l.mixer
            q, k = m.heads * m.dim, m.kv_heads * m.dim
            n += (3 * q + k) * self.width + (q + k) * m.conv + 2 * m.heads + m.heads ** 2 + 2 * (2 * self.width + 1)
            if l.ff is not None:
                n += 3 * l.ff * self.width + 2 * (2 * self.width + 1)
        return n

    # ---- config.json ----
    @staticmethod
    def from_dict(d: Dict[str, Any]) -> "DezelornConfig":
        layers = []
        for i, e in enumerate(d["layers"]):
            if e.get("type") != "attention":
                raise ValueError(f"layer {i}: unknown mixer type {e.get('type')!r}")
            m = e["mixer"]
            heads, kv = int(m["heads"]), int(m["kv_heads"])
            if heads % kv:
                raise ValueError(f"layer {i}: {kv} key heads do not divide {heads} query heads")
            if int(m.get("vdim", m["dim"])) != int(m["dim"]):
                raise ValueError(f"layer {i}: the values are the keys, so vdim must equal dim")
            spec = AttentionSpec(heads=heads, kv_heads=kv, dim=int(m["dim"]), conv=int(m["conv"]), window=int(m["mask"]["size"]),
                                 temp_coef=float(m["q_temp"]["coef"]), temp_every=float(m["q_temp"]["every"]), scale=float(m["scale"]))
            if spec.conv < 1 or spec.window < 1:
                raise ValueError(f"layer {i}: the convolution needs at least one tap and the window at least one token")
            mlp = e.get("mlp")
            if mlp is not None and mlp.get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
            layers.append(LayerSpec(spec, None if mlp is None else int(mlp["ff"])))
        eos = d.get("eos_token_id", -1)
        return DezelornConfig(vocab_size=int(d["vocab"]), width=int(d["width"]), layers=tuple(layers),
                              embedding_scale=float(d["embedding"]["scale"]), norm_eps=float(d.get("norm", {}).get("eps", 1e-6)),
                              max_position_embeddings=int(d.get("max_position_embeddings", 131072)),
                              eos_token_id=int(-1 if eos is None else eos), bos_token_id=d.get("bos_token_id"),
                              initializer_range=float(d.get("initializer_range", 0.02)))

    def to_hf_dict(self) -> Dict[str, Any]:
        layers = []
        for l in self.layers:
            m = l.mixer
            every = int(m.temp_every) if float(m.temp_every).is_integer() else m.temp_every
            layers.append({"type": "attention",
                           "mixer": {"conv": m.conv, "dim": m.dim, "heads": m.heads, "kv_heads": m.kv_heads, "mask": {"size": m.window},
                                     "q_temp": {"coef": m.temp_coef, "every": every}, "scale": m.scale, "vdim": m.dim},
                           "mlp": None if l.ff is None else {"kind": "dense", "ff": l.ff}})
        return {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.width,
                "embedding": {"scale": self.embedding_scale}, "norm": {"eps": self.norm_eps}, "layers": layers,
                "max_position_embeddings": self.max_position_embeddings, "eos_token_id": self.eos_token_id,
                "bos_token_id": self.bos_token_id, "initializer_range": self.initializer_range}

    def to_dict(self) -> Dict[str, Any]:
        return asdict(self)

    @staticmethod
    def uniform(vocab: int, width: int, n_layers: int, heads: int, kv_heads: int, dim: int, ff: Optional[int], window: int,
                conv: int = 4, temp_coef: float = 0.1, temp_every: int = 4096, **kw: Any) -> "DezelornConfig":
        """All layers alike (presets, benchmarks)."""
        spec = AttentionSpec(heads, kv_heads, dim, conv, window, temp_coef, float(temp_every), 1.0 / math.sqrt(dim))
        return DezelornConfig(vocab_size=vocab, width=width, layers=(LayerSpec(spec, ff),) * n_layers, embedding_scale=math.sqrt(width), **kw)


PRESETS: Dict[str, DezelornConfig] = {
    # the sizes of the framework's dense presets, with this design's layers
    "dezelorn-1.5b": DezelornConfig.uniform(151936, 1536, 28, 12, 2, 128, 8960, window=4096, max_position_embeddings=32768, eos_token_id=151643),
    "dezelorn-7b": DezelornConfig.uniform(152064, 3584, 28, 28, 4, 128, 18944, window=4096, max_position_embeddings=32768, eos_token_id=151643),
    "dezelorn-tiny": DezelornConfig.uniform(2048, 320, 3, 6, 2, 40, 640, window=48, conv=3, temp_coef=0.3, temp_every=16,
                                            max_position_embeddings=4096, eos_token_id=1),
}

_NORM_PARTS = ("w", "b", "alpha")


class DezelornLayout(ParamLayout):
    """Flat layout of a Dezelorn model: unit 0 = embedding group, unit 1 + i = layer i with q, k and gate projections fused
    into ``wqkg`` and the feed-forward's gate / up into ``wgu``."""

    def _declare(self) -> List[List[Tuple[str, Tuple[int, ...]]]]:
        cfg = self.cfg
        w, v = cfg.hidden_size, cfg.vocab_size

        def norm(name: str) -> List[Tuple[str, Tuple[int, ...]]]:
            return [(name + ".w", (w,)), (name + ".b", (w,)), (name + ".alpha", (1,))]

        units = [[("embed", (v, w)), *norm("final_norm"), ("lm_head", (v, w))]]
        for i, l in enumerate(cfg.layers):
            p, m = f"layers.{i}.", l.mixer
            unit = [*norm(p + "norm1"), (p + "wqkg", (m.u_dim, w)), (p + "conv", (m.qk_dim, m.conv)), (p + "r1", (m.heads,)),
                    (p + "r2", (m.heads,)), (p + "talk", (m.heads, m.heads)), (p + "wo", (w, m.q_dim)), *norm(p + "norm1b")]
            if l.ff is not None:
                unit += [*norm(p + "norm2"), (p + "wgu", (2 * l.ff_p, w)), (p + "wd", (w, l.ff_p)), *norm(p + "norm2b")]
            units.append(unit)
        return units

    def lm_head_name(self) -> str:
        return "lm_head"

    # ---- random init ----
    def init_value(self, name: str) -> Optional[float]:
        leaf = name.split(".")[-1]
        return {"w": 1.0, "b": 0.0, "alpha": 0.5, "r1": 0.5, "r2": 0.1}.get(leaf)

    def init_finish_(self, flat: torch.Tensor) -> None:
        """Head mixing starts near the identity and a convolution near "take the current token"; the padding is cleared."""
        for i, l in enumerate(self.cfg.layers):
            p, m = f"layers.{i}.", l.mixer
            self.view(flat, p + "talk").diagonal().add_(1.0)
            self.view(flat, p + "conv")[:, -1].add_(1.0)
        keep = flat.clone()
        flat.zero_()
        for (_, dst), (_, src) in zip(self.hf_items(flat), self.hf_items(keep)):
            dst.copy_(src)

    # ---- checkpoint boundary ----
    def hf_items(self, flat: torch.Tensor) -> Iterator[Tuple[str, torch.Tensor]]:
        cfg = self.cfg
        w = cfg.width

        def norm(ck: str, name: str) -> Iterator[Tuple[str, torch.Tensor]]:
            yield ck, self.view(flat, name + ".w")[:w]
            yield ck + ".b", self.view(flat, name + ".b")[:w]
            yield ck + ".alpha", self.view(flat, name + ".alpha")

        yield "embed", self.view(flat, "embed")[:, :w]
        for i, l in enumerate(cfg.layers):
            p, c, m = f"layers.{i}.", f"l{i}.", l.mixer
            yield from norm(c + "norm1", p + "norm1")
            yield from norm(c + "norm1b", p + "norm1b")
            rows = self.view(flat, p + "wqkg").view(2 * m.heads + m.kv_heads, m.dim_p, -1)[:, :m.dim, :w]
            yield c + "mix.q", rows[:m.heads]
            yield c + "mix.k", rows[m.heads:m.heads + m.kv_heads]
            yield c + "mix.g", rows[m.heads + m.kv_heads:]
            taps = self.view(flat, p + "conv").view(m.heads + m.kv_heads, m.dim_p, m.conv)[:, :m.dim]
            yield c + "mix.q.conv", taps[:m.heads]
            yield c + "mix.k.conv", taps[m.heads:]
            for leaf in ("r1", "r2", "talk"):
                yield c + "mix." + leaf, self.view(flat, p + leaf)
            yield c + "mix.o", self.view(flat, p + "wo").view(-1, m.heads, m.dim_p)[:w, :, :m.dim]
            if l.ff is not None:
                yield from norm(c + "norm2", p + "norm2")
                yield from norm(c + "norm2b", p + "norm2b")
                gu = self.view(flat, p + "wgu")
                yield c + "mlp.gate", gu[:l.ff, :w]
                yield c + "mlp.up", gu[l.ff_p:l.ff_p + l.ff, :w]
                yield c + "mlp.down", self.view(flat, p + "wd")[:w, :l.ff]
        yield from norm("final.norm", "final_norm")
        yield "head", self.view(flat, "lm_head")[:, :w]

    def hf_shape(self, name: str, view: torch.Tensor) -> Tuple[int, ...]:
        leaf = name.split(".")[-1]
        s = tuple(view.shape)
        if leaf == "alpha":
            return ()
        if name.endswith(("mix.q", "mix.k", "mix.g", "mix.q.conv", "mix.k.conv")):
            return (s[0] * s[1], s[2])
        if name.endswith("mix.o"):
            return (s[0], s[1] * s[2])
        return s
