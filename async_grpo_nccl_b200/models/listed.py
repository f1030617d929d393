"""Native executor of decoders whose layers are listed one by one: the kernels of one layer, in order.

The executor owns no cache and no loop over steps: the engine hands it the residual stream, the paged keys and the
convolution rings, and a ``StepBatch`` that says where every token row lives. The same layer code serves whole prompts,
portions of prompts, mixed batches and decode steps; decode differs only in the kernels that are picked.

A layer is four or five launches around two sublayers:
  fused q | k | gate projection -> short convolution (+ key write) -> attention with mixed heads and gate ->
  output projection whose epilogue is [norm of the output, residual add, norm ahead of the feed-forward] ->
  gate/up projection with SwiGLU -> down projection with the same kind of epilogue.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Sequence, Tuple

import numpy as np
import torch

from .dezelorn import DezelornConfig
from .layout import ParamLayout

LOG2E = 1.4426950408889634
TILE = 128  # query rows per attention tile
PAGE = 16   # tokens per cache block


@dataclass
class StepBatch:
    """Where the token rows of a step live. Decode steps (``rows`` None): row = slot, position = seq_lens - 1."""
    T: int
    block_tables: torch.Tensor
    rows: Optional[torch.Tensor] = None      # [T, 4] int32: slot, position, first row of the segment, 0
    ring_rows: Optional[Dict[int, torch.Tensor]] = None  # taps -> the last `taps` rows of each segment
    tiles: Optional[torch.Tensor] = None     # [n, 4]: first row, rows, position of the first row, row of position 0 in the gathered keys
    pages: Optional[torch.Tensor] = None     # [n, 2]: slot, page: the key pages that the step can see, in the order they are gathered
    seq_lens: Optional[torch.Tensor] = None
    splits: int = 1
    scratch: Optional[Tuple[torch.Tensor, torch.Tensor, torch.Tensor]] = None  # decode: partial products, (max, sum), tickets


def host_batch(segments: Sequence[Tuple[int, int, np.ndarray]], taps: Sequence[int], window: int) -> Tuple[np.ndarray, Dict[str, Tuple[int, int]]]:
    """(slot, tokens already there, new tokens) per segment -> one int32 array with the step's tables and where each of them
    is in it: token ids, rows, attention tiles, the key pages within ``window`` and, for every length in ``taps``, the rows
    that the convolution rings keep."""
    ids, rows, tiles, pages = [], [], [], []
    n_pages = 0
    keep: Dict[int, List[np.ndarray]] = {k: [] for k in sorted(set(taps))}
    t0 = 0
    for slot, past, toks in segments:
        n = len(toks)
        ids.append(np.asarray(toks, dtype=np.int32))
        r = np.zeros((n, 4), np.int32)
        r[:, 0], r[:, 1], r[:, 2] = slot, past + np.arange(n), t0
        rows.append(r)
        first = max(0, past - window + 1) // PAGE
        count = (past + n - 1) // PAGE + 1 - first
        pages.append(np.stack([np.full(count, slot, np.int32), np.arange(first, first + count, dtype=np.int32)], axis=1))
        tiles += [(t0 + a, min(TILE, n - a), past + a, (n_pages - first) * PAGE) for a in range(0, n, TILE)]
        n_pages += count
        for k, v in keep.items():
            v.append(np.arange(t0 + max(0, n - k), t0 + n, dtype=np.int32))
        t0 += n
    tiles.sort(key=lambda t: -t[2])
    parts = {"rows": np.concatenate(rows).ravel(), "tiles": np.asarray(tiles, np.int32).ravel(),
             "pages": np.concatenate(pages).ravel(), "ids": np.concatenate(ids),
             **{f"ring{k}": np.concatenate(v) for k, v in keep.items()}}   # tables of int4 and int2 come first: aligned
    where, o = {}, 0
    for k, v in parts.items():
        where[k] = (o, len(v))
        o += len(v)
    return np.concatenate(list(parts.values())), where


def split_batch(flat: torch.Tensor, where: Dict[str, Tuple[int, int]], block_tables: torch.Tensor) -> Tuple[torch.Tensor, StepBatch]:
    part = {k: flat[o:o + n] for k, (o, n) in where.items()}
    T = where["ids"][1]
    return part["ids"], StepBatch(T, block_tables, rows=part["rows"].view(T, 4), tiles=part["tiles"].view(-1, 4),
                                  pages=part["pages"].view(-1, 2),
                                  ring_rows={int(k[4:]): v for k, v in part.items() if k.startswith("ring")})


class ListedDecoder:
    def __init__(self, cfg: DezelornConfig, layout: ParamLayout, params: torch.Tensor, max_len: int):
        from ..ops import native

        self.C = native()
        self.cfg, self.layout, self.params = cfg, layout, params
        self.dev, self.dtype = params.device, params.dtype
        self.fp32 = params.dtype == torch.float32
        self.max_len = int(max_len)
        self.status = torch.zeros(1, dtype=torch.int32, device=self.dev)
        self.launches = 0
        self._w: Dict[str, torch.Tensor] = {n: layout.view(params, n) for n in layout.segments}
        self._norms: Dict[str, List[torch.Tensor]] = {}
        self.refresh_tables()

    def w(self, name: str) -> torch.Tensor:
        return self._w[name]

    def norm(self, name: str) -> List[torch.Tensor]:
        n = self._norms.get(name)
        if n is None:
            n = self._norms[name] = [self._w[f"{name}.{p}"] for p in ("w", "b", "alpha")]
        return n

    def refresh_tables(self) -> None:
        """Tables that follow from the configuration and the weights: the distance bias of every head (entry d =
        r1 ln(1 + r2 d)) and the score factor of a query at each position (scale x temperature), both computed in 64-bit
        and in log2 units, and the convolution weights with the channels contiguous. They keep their storage when the weights change, so captured graphs stay valid."""
        if not hasattr(self, "bias"):
            self.bias: List[torch.Tensor] = []
            self.qscale: List[torch.Tensor] = []
            self.conv: List[torch.Tensor] = [torch.empty(l.mixer.conv, l.mixer.qk_dim, dtype=self.dtype, device=self.dev)
                                             for l in self.cfg.layers]
            shared: Dict[Tuple[float, float, float], torch.Tensor] = {}
            for l in self.cfg.layers:
                m = l.mixer
                self.bias.append(torch.empty(m.heads, min(m.window, self.max_len), dtype=torch.float32, device=self.dev))
                key = (m.temp_coef, m.temp_every, m.scale)
                if key not in shared:
                    p = torch.arange(self.max_len, dtype=torch.float64)
                    temp = 1.0 + m.temp_coef * torch.log(torch.floor((p + 1.0) / m.temp_every) + 1.0)
                    shared[key] = (temp * (m.scale * LOG2E)).float().to(self.dev)
                self.qscale.append(shared[key])
        for i, t in enumerate(self.bias):
            self.conv[i].copy_(self.w(f"layers.{i}.conv").t())
            d = torch.arange(t.shape[1], dtype=torch.float64, device=self.dev)
            r1, r2 = self.w(f"layers.{i}.r1").double(), self.w(f"layers.{i}.r2").double()
            t.copy_(r1[:, None] * torch.log1p(r2[:, None] * d[None]) * LOG2E)

    def check_status(self) -> None:
        code = int(self.status.item())
        if code != 0:
            self.status.zero_()
            raise RuntimeError(f"device kernel reported status {code} (bounded wait ran out or bad index)")

    def decode_ctas_per_sm(self, i: int) -> int:
        """CTAs of the fused decode mixer that fit an SM; 0 = the layer decodes with the plain kernels."""
        m = self.cfg.layers[i].mixer
        return 0 if self.fp32 else int(self.C.talk_decode_ctas_per_sm(m.heads, m.kv_heads, m.dim_p))

    def next_norm(self, i: int) -> str:
        return f"layers.{i + 1}.norm1" if i + 1 < len(self.cfg.layers) else "final_norm"

    # ---- pieces ----
    def embed(self, ids: torch.Tensor, x: torch.Tensor, h: torch.Tensor) -> None:
        self.C.embed_dyt(ids, self.w("embed"), self.cfg.embedding_scale, x, h, self.norm("layers.0.norm1"))
        self.launches += 1

    def _project(self, h: torch.Tensor, w: torch.Tensor, out: torch.Tensor) -> None:
        if self.fp32:
            self.C.gemm_f32(h, w, out)
        else:
            self.C.gemm_bf16(h, w, out, False, False, None, 1.0, False, self.status, None)
        self.launches += 1

    def _swiglu(self, h: torch.Tensor, w: torch.Tensor, out: torch.Tensor) -> None:
        if self.fp32:
            self.C.gemm_swiglu_f32(h, w, out)
        else:
            self.C.gemm_swiglu(h, w, out, None, 0.0, self.status)
        self.launches += 1

    def _close_sublayer(self, a: torch.Tensor, w: torch.Tensor, x: torch.Tensor, h: torch.Tensor, out_norm: str, next_norm: str) -> None:
        """x += out_norm(a w^T); h = next_norm(x)."""
        self.C.gemm_dyt(a, w, x, self.norm(out_norm), self.norm(next_norm), h, self.status)
        self.launches += 1

    def _attention(self, i: int, u: torch.Tensor, sb: StepBatch, k_cache: torch.Tensor, ring: torch.Tensor, q: torch.Tensor,
                   out: torch.Tensor) -> None:
        m, C, p = self.cfg.layers[i].mixer, self.C, f"layers.{i}."
        gate = u[:, m.qk_dim:]
        if sb.rows is None and sb.scratch is not None and self.decode_ctas_per_sm(i):
            C.talk_attn_decode(u, self.conv[i], ring, k_cache, sb.seq_lens, sb.block_tables, self.bias[i], self.qscale[i],
                               self.w(p + "talk"), gate, m.window, out, sb.splits, *sb.scratch, self.status)
            self.launches += 1
            return
        C.short_conv(u, self.conv[i], ring, sb.rows, sb.ring_rows[m.conv] if sb.rows is not None else None, sb.seq_lens, sb.block_tables, q, k_cache, self.status)
        if sb.rows is not None and not self.fp32:
            acc = torch.empty(sb.T * m.heads * m.k_dim, dtype=self.dtype, device=self.dev)
            keys = torch.empty(sb.pages.shape[0] * PAGE * m.k_dim, dtype=self.dtype, device=self.dev)
            if C.talk_attn_prefill(q, k_cache, sb.tiles, sb.pages, keys, sb.block_tables, self.bias[i], self.qscale[i], self.w(p + "talk"), gate, m.window,
                                   acc, out, self.status):
                self.launches += 5
                return
        C.window_attn(q, k_cache, sb.rows, sb.seq_lens, sb.block_tables, self.bias[i], self.qscale[i], self.w(p + "talk"), gate,
                      m.window, out, self.status)
        self.launches += 3

    def layer(self, i: int, x: torch.Tensor, h: torch.Tensor, sb: StepBatch, k_cache: torch.Tensor, ring: torch.Tensor,
              buf: Dict[str, torch.Tensor]) -> None:
        """``x`` fp32 residual stream and ``h`` = norm1(x), both updated in place (``h`` to the next layer's norm)."""
        l, p, T = self.cfg.layers[i], f"layers.{i}.", sb.T
        m = l.mixer
        u = buf["u"][:T * m.u_dim].view(T, m.u_dim)
        q = buf["q"][:T * m.q_dim].view(T, m.q_dim)
        a = buf["a"][:T * m.q_dim].view(T, m.q_dim)
        self._project(h, self.w(p + "wqkg"), u)
        self._attention(i, u, sb, k_cache, ring, q, a)
        self._close_sublayer(a, self.w(p + "wo"), x, h, p + "norm1b", p + "norm2" if l.ff is not None else self.next_norm(i))
        if l.ff is not None:
            act = buf["act"][:T * l.ff_p].view(T, l.ff_p)
            self._swiglu(h, self.w(p + "wgu"), act)
            self._close_sublayer(act, self.w(p + "wd"), x, h, p + "norm2b", self.next_norm(i))

    def buffers(self, T: int) -> Dict[str, torch.Tensor]:
        ls = self.cfg.layers
        dims = {"u": max(l.mixer.u_dim for l in ls), "q": max(l.mixer.q_dim for l in ls), "a": max(l.mixer.q_dim for l in ls),
                "act": max(l.ff_p for l in ls)}
        return {k: torch.empty(T * d, dtype=self.dtype, device=self.dev) for k, d in dims.items()}

    def logits(self, h: torch.Tensor) -> torch.Tensor:
        wl = self.w("lm_head")
        out = torch.empty(h.shape[0], wl.shape[0], dtype=torch.float32, device=self.dev)
        if self.fp32:
            self.C.gemm_f32(h, wl, out)
        else:
            self.C.gemm_bf16(h, wl, out, False, False, None, 1.0, False, self.status, None)
        self.launches += 1
        return out
