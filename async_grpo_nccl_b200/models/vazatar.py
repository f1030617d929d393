"""The Vazatar decoder: configuration record and parameter layout.

A decoder whose layers are listed one by one in the configuration, some of them attention, some a selective scan:

* a layer is parallel: mixer and feed-forward read the same residual through a norm of their own, and both are added to it;
* attention inside fixed chunks of positions with grouped key heads, an RMS norm over the whole query and key projections,
  partial rotation with wavelength-dependent frequency scaling, and soft-capped scores;
* the selective scan (Mamba) carries a short convolution's last inputs and a matrix of states per channel;
* the feed-forward is one matrix, squared ReLU, one matrix;
* a range of layers runs several times with the same weights (each pass has its own cache and state), and every pass begins
  with a projection of the residual beside the embedding output.

The kernels want head sizes that are multiples of 64 and row pitches that are multiples of 8 elements. The layout therefore
pads with zeros, which changes nothing: a padded channel has zero weights on both sides and norms divide by the true sizes.
Everything that reads the same input is one matrix (``win``: mixer projections, then the feed-forward's), everything that is
added to the residual is one matrix (``wout``). The checkpoint boundary (``hf_items``) hands out views without the padding.
"""
from __future__ import annotations

import math
from dataclasses import asdict, dataclass, replace
from typing import Any, Dict, Iterator, List, Optional, Tuple, Union

import torch

from .layout import ParamLayout


def _up(x: int, m: int) -> int:
    return (x + m - 1) // m * m


@dataclass(frozen=True)
class RotationSpec:
    """Rotary positions on the first ``dims`` dimensions of a head. Scaling: wavelengths above ``original / low`` are slowed by
    ``factor``, those below ``original / high`` are kept, the ones between are interpolated."""
    dims: int
    base: float
    factor: float = 1.0
    low: float = 1.0
    high: float = 4.0
    original: float = 8192.0

    def frequencies(self) -> List[float]:
        out = []
        for i in range(self.dims // 2):
            f = self.base ** (-2.0 * i / self.dims)
            wavelength = 2.0 * math.pi / f
            if wavelength < self.original / self.high:
                keep = 1.0
            elif wavelength > self.original / self.low:
                keep = 0.0
            else:
                keep = (self.original / wavelength - self.low) / (self.high - self.low)
            out.append(keep * f + (1.0 - keep) * f / self.factor)
        return out


@dataclass(frozen=True)
class ChunkAttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    chunk: int           # a position sees the tokens of its own chunk up to itself
    scale: float
    softcap: float       # 0 = none
    rot: RotationSpec

    @property
    def dim_p(self) -> int:
        return _up(self.dim, 64)

    @property
    def vdim_p(self) -> int:
        return _up(self.vdim, 64)

    @property
    def q_dim(self) -> int:
        return self.heads * self.dim_p

    @property
    def k_dim(self) -> int:
        return self.kv_heads * self.dim_p

    @property
    def v_dim(self) -> int:
        return self.kv_heads * self.vdim_p

    @property
    def u_dim(self) -> int:
        """Columns of the fused projection: q, k, v."""
        return self.q_dim + self.k_dim + self.v_dim

    @property
    def out_dim(self) -> int:
        return self.heads * self.vdim_p


@dataclass(frozen=True)
class ScanSpec:
    inner: int
    state: int
    dt_rank: int
    conv: int

    @property
    def inner_p(self) -> int:
        return _up(self.inner, 64)

    @property
    def rank_p(self) -> int:
        return _up(self.dt_rank, 16)

    @property
    def x_dim(self) -> int:
        """Rows of the projection of the convolved input: step size, B, C (columns of a padded ``wdt`` reach into B: times zero)."""
        return max(_up(self.dt_rank + 2 * self.state, 8), self.rank_p)

    @property
    def u_dim(self) -> int:
        return 2 * self.inner_p

    @property
    def out_dim(self) -> int:
        return self.inner_p


@dataclass(frozen=True)
class LayerSpec:
    mixer: Union[ChunkAttentionSpec, ScanSpec]
    ff: Optional[int]    # None = no feed-forward

    @property
    def ff_p(self) -> int:
        return _up(self.ff or 0, 8)

    @property
    def attends(self) -> bool:
        return isinstance(self.mixer, ChunkAttentionSpec)


@dataclass(frozen=True)
class LoopSpec:
    """Layers ``start`` to ``stop - 1`` run ``times`` times in a row."""
    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class VazatarConfig:
    vocab_size: int
    width: int
    layers: Tuple[LayerSpec, ...]
    embedding_scale: float
    loop: Optional[LoopSpec] = None
    norm_eps: float = 1e-5
    logit_softcap: float = 0.0      # 0 = none
    max_position_embeddings: int = 131072
    eos_token_id: int = -1
    bos_token_id: Optional[int] = None
    initializer_range: float = 0.02
    model_type: str = "vazatar"
    architecture: str = "Vazatar"

    @property
    def hidden_size(self) -> int:
        return _up(self.width, 8)

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def runs(self) -> List[Tuple[int, bool]]:
        """(layer, first of a pass of the loop) in the order of execution."""
        n, loop = len(self.layers), self.loop
        if loop is None:
            return [(i, False) for i in range(n)]
        body = [(i, i == loop.start) for i in range(loop.start, loop.stop)]
        return [(i, False) for i in range(loop.start)] + body * loop.times + [(i, False) for i in range(loop.stop, n)]

    def first_layers(self, n: int) -> "VazatarConfig":
        """The same model with its first ``n`` layers (benchmarks)."""
        loop = self.loop
        if loop is not None:
            loop = replace(loop, start=min(loop.start, n - 1), stop=min(loop.stop, n))
        return replace(self, layers=self.layers[:n], loop=loop)

    def num_parameters(self) -> int:
        w = self.width
        n = 2 * self.vocab_size * w + w + (2 * w * w if self.loop is not None else 0)
        for l in self.layers:
            m = l.mixer
            n += w
            if isinstance(m, ChunkAttentionSpec):
                q, k = m.heads * m.dim, m.kv_heads * m.dim
                n += (q + k + m.kv_heads * m.vdim + m.heads * m.vdim) * w + q + k
            else:
                n += 3 * m.inner * w + m.inner * (m.conv + 1) + m.inner * (m.dt_rank + 2 * m.state) + m.inner * (m.dt_rank + 1)
                n += m.inner * m.state + m.inner
            if l.ff is not None:
                n += w + 2 * l.ff * w
        return n

    # ---- config.json ----
    @staticmethod
    def from_dict(d: Dict[str, Any]) -> "VazatarConfig":
        layers = []
        for i, e in enumerate(d["layers"]):
            m, kind = e["mixer"], e.get("type")
            if kind == "attention":
                heads, kv = int(m["heads"]), int(m["kv_heads"])
                if heads % kv:
                    raise ValueError(f"layer {i}: {kv} key heads do not divide {heads} query heads")
                rot = m.get("rot") or {"dims": 0, "base": 1.0}
                s = rot.get("scaling") or {}
                rotation = RotationSpec(int(rot["dims"]), float(rot["base"]), float(s.get("factor", 1.0)), float(s.get("low", 1.0)),
                                        float(s.get("high", 4.0)), float(s.get("original", 8192)))
                spec: Any = ChunkAttentionSpec(heads, kv, int(m["dim"]), int(m.get("vdim", m["dim"])), int(m["mask"]["size"]),
                                               float(m["scale"]), float(m.get("softcap") or 0.0), rotation)
                if spec.chunk < 1 or spec.rot.dims % 2 or not 0 <= spec.rot.dims <= spec.dim:
                    raise ValueError(f"layer {i}: a chunk has at least one token, and an even number of a head's dimensions is rotated")
            elif kind == "mamba1":
                spec = ScanSpec(int(m["inner"]), int(m["state"]), int(m["dt_rank"]), int(m["conv"]))
                if min(spec.inner, spec.state, spec.dt_rank, spec.conv) < 1:
                    raise ValueError(f"layer {i}: sizes of the scan must be positive")
            else:
                raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
            mlp = e.get("mlp")
            if mlp is not None and mlp.get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
            layers.append(LayerSpec(spec, None if mlp is None else int(mlp["ff"])))
        loop = None
        if d.get("loop"):
            loop = LoopSpec(*(int(d["loop"][k]) for k in ("start", "stop", "times")))
            if not (0 <= loop.start < loop.stop <= len(layers) and loop.times >= 1):
                raise ValueError(f"loop {loop} does not fit {len(layers)} layers")
        eos = d.get("eos_token_id", -1)
        return VazatarConfig(vocab_size=int(d["vocab"]), width=int(d["width"]), layers=tuple(layers),
                             embedding_scale=float(d["embedding"]["scale"]), loop=loop, norm_eps=float(d["norm"]["eps"]),
                             logit_softcap=float(d.get("logit_softcap") or 0.0),
                             max_position_embeddings=int(d.get("max_position_embeddings", 131072)),
                             eos_token_id=int(-1 if eos is None else eos), bos_token_id=d.get("bos_token_id"),
                             initializer_range=float(d.get("initializer_range", 0.02)))

    def to_hf_dict(self) -> Dict[str, Any]:
        layers = []
        for l in self.layers:
            m = l.mixer
            if isinstance(m, ChunkAttentionSpec):
                r = m.rot
                mixer: Dict[str, Any] = {"dim": m.dim, "heads": m.heads, "kv_heads": m.kv_heads, "mask": {"size": m.chunk}, "scale": m.scale,
                                         "softcap": m.softcap, "vdim": m.vdim,
                                         "rot": {"base": r.base, "dims": r.dims, "scaling": {"factor": r.factor, "high": r.high, "low": r.low,
                                                                                             "original": r.original}}}
            else:
                mixer = {"conv": m.conv, "dt_rank": m.dt_rank, "inner": m.inner, "state": m.state}
            layers.append({"type": "attention" if l.attends else "mamba1", "mixer": mixer,
                           "mlp": None if l.ff is None else {"kind": "dense", "ff": l.ff}})
        d = {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.width,
             "embedding": {"scale": self.embedding_scale}, "norm": {"eps": self.norm_eps}, "layers": layers,
             "logit_softcap": self.logit_softcap, "max_position_embeddings": self.max_position_embeddings,
             "eos_token_id": self.eos_token_id, "bos_token_id": self.bos_token_id, "initializer_range": self.initializer_range}
        if self.loop is not None:
            d["loop"] = asdict(self.loop)
        return d

    def to_dict(self) -> Dict[str, Any]:
        return asdict(self)

    @staticmethod
    def alternating(vocab: int, width: int, n_layers: int, heads: int, kv_heads: int, dim: int, ff: Optional[int], chunk: int, state: int = 16,
                    conv: int = 4, times: int = 1, **kw: Any) -> "VazatarConfig":
        """Attention and scan in turn (presets, benchmarks); the scan is twice as wide as the model."""
        rot = RotationSpec(dim, 500000.0, 8.0, 1.0, 4.0, 8192.0)
        a = LayerSpec(ChunkAttentionSpec(heads, kv_heads, dim, dim, chunk, 1.0 / math.sqrt(dim), 50.0, rot), ff)
        s = LayerSpec(ScanSpec(2 * width, state, max(1, width // 16), conv), ff)
        return VazatarConfig(vocab_size=vocab, width=width, layers=tuple(s if i % 2 else a for i in range(n_layers)),
                             embedding_scale=math.sqrt(width), loop=LoopSpec(n_layers // 4, n_layers - n_layers // 4, times), logit_softcap=30.0, **kw)


PRESETS: Dict[str, VazatarConfig] = {
    # the sizes of the framework's dense presets, with this design's layers
    "vazatar-1.5b": VazatarConfig.alternating(151936, 1536, 28, 12, 2, 128, 11904, chunk=8192, max_position_embeddings=32768, eos_token_id=151643),
    "vazatar-7b": VazatarConfig.alternating(152064, 3584, 28, 28, 4, 128, 25088, chunk=8192, max_position_embeddings=32768, eos_token_id=151643),
    "vazatar-tiny": VazatarConfig.alternating(2048, 320, 5, 6, 2, 40, 640, chunk=48, state=8, conv=3, times=2, max_position_embeddings=4096,
                                              eos_token_id=1),
}


class VazatarLayout(ParamLayout):
    """Flat layout of a Vazatar model: unit 0 = embedding group, unit 1 + i = layer i."""

    def _declare(self) -> List[List[Tuple[str, Tuple[int, ...]]]]:
        cfg = self.cfg
        w, v = cfg.hidden_size, cfg.vocab_size
        top = [("embed", (v, w)), ("final_norm", (w,)), ("lm_head", (v, w))]
        if cfg.loop is not None:
            top.append(("loop_in", (w, 2 * w)))
        units = [top]
        for i, l in enumerate(cfg.layers):
            p, m = f"layers.{i}.", l.mixer
            unit = [(p + "norm1", (w,)), (p + "norm2", (w,)), (p + "win", (m.u_dim + l.ff_p, w)), (p + "wout", (w, m.out_dim + l.ff_p))]
            if isinstance(m, ChunkAttentionSpec):
                unit += [(p + "q_norm", (m.q_dim,)), (p + "k_norm", (m.k_dim,))]
            else:
                unit += [(p + "conv", (m.inner_p, m.conv)), (p + "conv_b", (m.inner_p,)), (p + "wx", (m.x_dim, m.inner_p)),
                         (p + "wdt", (m.inner_p, m.rank_p)), (p + "dt_b", (m.inner_p,)), (p + "A_log", (m.inner_p, m.state)), (p + "D", (m.inner_p,))]
            units.append(unit)
        return units

    def lm_head_name(self) -> str:
        return "lm_head"

    # ---- random init ----
    def init_value(self, name: str) -> Optional[float]:
        leaf = name.split(".")[-1]
        return {"norm1": 0.0, "norm2": 0.0, "final_norm": 0.0, "q_norm": 1.0, "k_norm": 1.0, "conv_b": 0.0, "dt_b": -4.0, "D": 1.0}.get(leaf)

    def init_finish_(self, flat: torch.Tensor) -> None:
        """Decays of a channel's states start at rates 1 .. N, a convolution near "take the current token"; padding is cleared."""
        for i, l in enumerate(self.cfg.layers):
            if not l.attends:
                p, m = f"layers.{i}.", l.mixer
                self.view(flat, p + "A_log").copy_(torch.log(torch.arange(1, m.state + 1, dtype=torch.float32)).expand(m.inner_p, m.state))
                self.view(flat, p + "conv")[:, -1].add_(1.0)
        keep = flat.clone()
        flat.zero_()
        for (_, dst), (_, src) in zip(self.hf_items(flat), self.hf_items(keep)):
            dst.copy_(src)

    # ---- checkpoint boundary ----
    def hf_items(self, flat: torch.Tensor) -> Iterator[Tuple[str, torch.Tensor]]:
        cfg = self.cfg
        w, wp = cfg.width, cfg.hidden_size
        yield "embed", self.view(flat, "embed")[:, :w]
        if cfg.loop is not None:
            yield "loop.in", self.view(flat, "loop_in").view(wp, 2, wp)[:w, :, :w]
        for i, l in enumerate(cfg.layers):
            p, c, m = f"layers.{i}.", f"l{i}.", l.mixer
            yield c + "norm1", self.view(flat, p + "norm1")[:w]
            win, wout = self.view(flat, p + "win")[:, :w], self.view(flat, p + "wout")[:w]
            if isinstance(m, ChunkAttentionSpec):
                yield c + "mix.q", win[:m.q_dim].view(m.heads, m.dim_p, w)[:, :m.dim]
                yield c + "mix.k", win[m.q_dim:m.q_dim + m.k_dim].view(m.kv_heads, m.dim_p, w)[:, :m.dim]
                yield c + "mix.v", win[m.q_dim + m.k_dim:m.u_dim].view(m.kv_heads, m.vdim_p, w)[:, :m.vdim]
                yield c + "mix.q.norm", self.view(flat, p + "q_norm").view(m.heads, m.dim_p)[:, :m.dim]
                yield c + "mix.k.norm", self.view(flat, p + "k_norm").view(m.kv_heads, m.dim_p)[:, :m.dim]
                yield c + "mix.o", wout[:, :m.out_dim].unflatten(1, (m.heads, m.vdim_p))[:, :, :m.vdim]
            else:
                n = m.inner
                yield c + "mix.in", win[:m.u_dim].view(2, m.inner_p, w)[:, :n]
                yield c + "mix.conv", self.view(flat, p + "conv")[:n]
                yield c + "mix.conv.b", self.view(flat, p + "conv_b")[:n]
                yield c + "mix.x", self.view(flat, p + "wx")[:m.dt_rank + 2 * m.state, :n]
                yield c + "mix.dt", self.view(flat, p + "wdt")[:n, :m.dt_rank]
                yield c + "mix.dt.b", self.view(flat, p + "dt_b")[:n]
                yield c + "mix.A_log", self.view(flat, p + "A_log")[:n]
                yield c + "mix.D", self.view(flat, p + "D")[:n]
                yield c + "mix.o", wout[:, :n]
            if l.ff is not None:
                yield c + "norm2", self.view(flat, p + "norm2")[:w]
                yield c + "mlp.up", win[m.u_dim:m.u_dim + l.ff]
                yield c + "mlp.down", wout[:, m.out_dim:m.out_dim + l.ff]
        yield "final.norm", self.view(flat, "final_norm")[:w]
        yield "head", self.view(flat, "lm_head")[:, :w]

    def hf_shape(self, name: str, view: torch.Tensor) -> Tuple[int, ...]:
        s = tuple(view.shape)
        if name.endswith(("mix.q", "mix.k", "mix.v", "mix.in")):
            return (s[0] * s[1], s[2])
        if name == "loop.in" or (name.endswith("mix.o") and len(s) == 3):
            return (s[0], s[1] * s[2])
        if name.endswith((".q.norm", ".k.norm")):
            return (s[0] * s[1],)
        return s

    def hf_unused(self, name: str) -> bool:
        """A layer without a feed-forward has no use for the norm ahead of one."""
        return any(l.ff is None and name == f"l{i}.norm2" for i, l in enumerate(self.cfg.layers))
