"""Native executor of the Dezelorn decoder: the kernels of one layer, in order.

A layer is four or five launches around two sublayers:
  fused q | k | gate projection -> short convolution (+ key write) -> attention with mixed heads and gate ->
  output projection whose epilogue is [norm of the output, residual add, norm ahead of the feed-forward] ->
  gate/up projection with SwiGLU -> down projection with the same kind of epilogue.
"""
from __future__ import annotations

from typing import Any, Dict, List, Sequence, Tuple

import numpy as np
import torch

from .layout import ParamLayout
from .listed import LOG2E, PAGE, ListedDecoder, StepBatch, host_batch


class DezelornDecoder(ListedDecoder):
    def __init__(self, cfg: Any, layout: ParamLayout, params: torch.Tensor, max_len: int):
        self._norms: Dict[str, List[torch.Tensor]] = {}
        super().__init__(cfg, layout, params, max_len)
        self.ctas_per_sm = max(1, min(self.decode_ctas_per_sm(i) for i in range(len(cfg.layers))))

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

    # ---- cache and state ----
    def paged(self) -> List[Tuple[int, int]]:
        return [(l.mixer.kv_heads, l.mixer.dim_p) for l in self.cfg.layers]

    def slot_state(self) -> List[Tuple[Tuple[int, ...], torch.dtype]]:
        """Rings of the short convolutions, one row per slot for all layers: position p of a sequence at p % taps."""
        return [((sum(l.mixer.conv * l.mixer.qk_dim for l in self.cfg.layers),), self.dtype)]

    def bind(self, paged: List[torch.Tensor], slots: List[torch.Tensor]) -> None:
        self.cache, ring = paged, slots[0]
        sizes = [l.mixer.conv * l.mixer.qk_dim for l in self.cfg.layers]
        offs = np.concatenate([[0], np.cumsum(sizes)])
        self.rings = [ring[:, int(o):int(o) + n].view(ring.shape[0], l.mixer.conv, l.mixer.qk_dim) for o, n, l in zip(offs, sizes, self.cfg.layers)]

    def reach(self) -> int:
        return self.cfg.max_window

    def tables_of(self, segments: Sequence[Tuple[int, int, np.ndarray]]) -> Tuple[np.ndarray, Dict[str, Tuple[int, int]]]:
        return host_batch(segments, [l.mixer.conv for l in self.cfg.layers], self.cfg.max_window)

    def decode_scratch(self, S: int, max_splits: int) -> Tuple[torch.Tensor, ...]:
        ms = [l.mixer for l in self.cfg.layers]
        f32 = dict(dtype=torch.float32, device=self.dev)
        return (torch.empty(S * max_splits * max(m.heads * m.k_dim for m in ms), **f32), torch.empty(S * max_splits * max(m.heads for m in ms) * 2, **f32),
                torch.zeros(S, dtype=torch.int32, device=self.dev))

    def decode_launches(self) -> int:
        return 1 + sum((3 if self.decode_ctas_per_sm(i) else 5) + (0 if l.ff is None else 2) for i, l in enumerate(self.cfg.layers))

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
                "act": max(l.ff_p for l in ls), "h": self.cfg.hidden_size}
        buf = {k: torch.empty(T * d, dtype=self.dtype, device=self.dev) for k, d in dims.items()}
        buf["h"] = buf["h"].view(T, -1)
        buf["x"] = torch.empty(T, self.cfg.hidden_size, dtype=torch.float32, device=self.dev)
        return buf

    def forward(self, ids: torch.Tensor, sb: StepBatch, buf: Dict[str, torch.Tensor]) -> None:
        x, h = buf["x"][:sb.T], buf["h"][:sb.T]
        self.embed(ids, x, h)
        for i in range(len(self.cfg.layers)):
            self.layer(i, x, h, sb, self.cache[i], self.rings[i], buf)

    def hidden(self, buf: Dict[str, torch.Tensor], rows: Any) -> torch.Tensor:
        return buf["h"][rows]
