"""Native executor of the Vazatar decoder: the kernels of one layer run, in order.

A layer run is three launches around its mixer:
  one GEMM for the mixer's projections and the feed-forward's first matrix (two norms of the same residual, side by side as its
  input) -> mixer -> one GEMM over [mixer output | feed-forward activation] that adds to the fp32 residual and writes the inputs
  of the next run.
The mixer is norm + rotation + cache write + attention (one launch in decode), or convolution -> narrow projection -> selective
scan. In bf16 no norm runs by itself: x * (1 + w) and the squares of the rows come out of the GEMM that makes x, the row scale
goes into the GEMM that reads it. In fp32 the same steps run one by one.
"""
from __future__ import annotations

from typing import Any, Dict, List, Optional, Sequence, Tuple

import numpy as np
import torch

from .layout import ParamLayout
from .listed import LOG2E, PAGE, ListedDecoder, StepBatch, host_batch
from .vazatar import ChunkAttentionSpec, RotationSpec

Target = Tuple[Optional[torch.Tensor], Optional[torch.Tensor], Optional[torch.Tensor], Optional[torch.Tensor], Optional[torch.Tensor]]


class VazatarDecoder(ListedDecoder):
    ctas_per_sm = 3

    def __init__(self, cfg: Any, layout: ParamLayout, params: torch.Tensor, max_len: int):
        self.runs = cfg.runs()
        super().__init__(cfg, layout, params, max_len)
        self.softcap = cfg.logit_softcap
        ms = [self.cfg.layers[i].mixer for i, _ in self.runs if self.cfg.layers[i].attends]
        self.chunks = sorted({m.chunk for m in ms})
        self.taps = sorted({l.mixer.conv for l in cfg.layers if not l.attends})
        if ms:  # CTAs are per key head
            self.ctas_per_sm = 3 / max(m.kv_heads for m in ms)

    # ---- tables ----
    def refresh_tables(self) -> None:
        """Rotation tables (angles in 64-bit), and of the scan layers: convolution weights with the channels contiguous, fp32 copies
        of step-size bias, skip and A = -exp(A_log). The packed scan kernel wants the states in quarters of equal, even size."""
        if not hasattr(self, "scan"):
            self.rot: Dict[RotationSpec, Tuple[torch.Tensor, torch.Tensor]] = {}
            self.scan: Dict[int, Dict[str, torch.Tensor]] = {}
            p = torch.arange(self.max_len, dtype=torch.float64)
            f32 = dict(dtype=torch.float32, device=self.dev)
            for i, l in enumerate(self.cfg.layers):
                m = l.mixer
                if isinstance(m, ChunkAttentionSpec):
                    if m.rot not in self.rot:
                        a = p[:, None] * torch.tensor(m.rot.frequencies(), dtype=torch.float64)[None]
                        self.rot[m.rot] = (torch.cos(a).float().to(self.dev), torch.sin(a).float().to(self.dev))
                    continue
                packed = not self.fp32 and self.C.selective_scan_serves(m.state, m.dt_rank)
                n = 4 * self.C.scan_states_per_lane(m.state) if packed else m.state
                rows = m.rank_p + 2 * n if packed else m.x_dim
                self.scan[i] = {"conv": torch.empty(m.conv, m.inner_p, dtype=self.dtype, device=self.dev), "dt_b": torch.empty(m.inner_p, **f32),
                                "D": torch.empty(m.inner_p, **f32), "A": torch.zeros(m.inner_p, n, **f32),
                                "wx": torch.zeros(rows, m.inner_p, dtype=self.dtype, device=self.dev) if packed else self.w(f"layers.{i}.wx")}
        for i, t in self.scan.items():
            p, m = f"layers.{i}.", self.cfg.layers[i].mixer
            t["conv"].copy_(self.w(p + "conv").t())
            t["dt_b"].copy_(self.w(p + "dt_b"))
            t["D"].copy_(self.w(p + "D"))
            a = -torch.exp(self.w(p + "A_log").double())
            if not self.packed(i):
                t["A"].copy_(a)
                continue
            t["A"][:, :m.state].copy_(a * LOG2E)
            wx, n, q = self.w(p + "wx"), m.state, t["A"].shape[1] // 4
            t["wx"][:m.dt_rank].copy_(wx[:m.dt_rank])
            for k in range(n):   # state k: place k % q of quarter k // q, B before C
                row = m.rank_p + (k // q) * 2 * q + k % q
                t["wx"][row].copy_(wx[m.dt_rank + k])
                t["wx"][row + q].copy_(wx[m.dt_rank + n + k])

    def packed(self, i: int) -> bool:
        return not self.fp32 and bool(self.C.selective_scan_serves(self.cfg.layers[i].mixer.state, self.cfg.layers[i].mixer.dt_rank))

    # ---- cache and state ----
    def paged(self) -> List[Tuple[int, int]]:
        out: List[Tuple[int, int]] = []
        for i, _ in self.runs:
            m = self.cfg.layers[i].mixer
            if isinstance(m, ChunkAttentionSpec):
                out += [(m.kv_heads, m.dim_p), (m.kv_heads, m.vdim_p)]
        return out

    def _scan_runs(self) -> List[int]:
        return [j for j, (i, _) in enumerate(self.runs) if not self.cfg.layers[i].attends]

    def slot_state(self) -> List[Tuple[Tuple[int, ...], torch.dtype]]:
        """One row per slot for all scan runs: rings of the convolutions' inputs (position p at p % taps), and the states."""
        ms = [self.cfg.layers[self.runs[j][0]].mixer for j in self._scan_runs()]
        if not ms:
            return []
        ns = [self.scan[self.runs[j][0]]["A"].shape[1] for j in self._scan_runs()]
        return [((sum(m.conv * m.inner_p for m in ms),), self.dtype), ((sum(m.inner_p * n for m, n in zip(ms, ns)),), torch.float32)]

    def bind(self, paged: List[torch.Tensor], slots: List[torch.Tensor]) -> None:
        self.kv: Dict[int, Tuple[torch.Tensor, torch.Tensor]] = {}
        self.state: Dict[int, Tuple[torch.Tensor, torch.Tensor]] = {}
        k = ring_at = state_at = 0
        for j, (i, _) in enumerate(self.runs):
            m = self.cfg.layers[i].mixer
            if isinstance(m, ChunkAttentionSpec):
                self.kv[j] = (paged[k], paged[k + 1])
                k += 2
                continue
            n = self.scan[i]["A"].shape[1]
            ring = slots[0][:, ring_at:ring_at + m.conv * m.inner_p].view(-1, m.conv, m.inner_p)
            state = slots[1][:, state_at:state_at + m.inner_p * n].view(-1, m.inner_p, n)
            self.state[j] = (ring, state)
            ring_at += m.conv * m.inner_p
            state_at += m.inner_p * n

    def reach(self) -> int:
        return max(self.chunks, default=1)

    def tables_of(self, segments: Sequence[Tuple[int, int, np.ndarray]]) -> Tuple[np.ndarray, Dict[str, Tuple[int, int]]]:
        return host_batch(segments, self.taps, 1, self.chunks)

    def buffers(self, T: int) -> Dict[str, torch.Tensor]:
        ls, W = self.cfg.layers, self.cfg.hidden_size
        kw = dict(dtype=self.dtype, device=self.dev)
        scans = [l.mixer for l in ls if not l.attends]
        flat = {"u": max(l.mixer.u_dim for l in ls), "cat": max(l.mixer.out_dim + l.ff_p for l in ls), "xc": max([m.inner_p for m in scans], default=0)}
        buf = {k: torch.empty(T * d, **kw) for k, d in flat.items()}
        buf["code"] = torch.empty(T * max([self.C.scan_code_pitch(m.dt_rank) for m in scans], default=0), **kw)
        buf["x"] = torch.empty(T, W, dtype=torch.float32, device=self.dev)
        buf["h"] = torch.empty(T, 2 * W, **kw)
        buf["loop"] = torch.empty(T if self.cfg.loop is not None else 0, 2 * W, **kw)
        buf["r"] = torch.empty(T * max([t["wx"].shape[0] for t in self.scan.values()], default=0), dtype=torch.float32, device=self.dev)
        # sums of squares per run: residual, queries, keys
        buf["ss"] = torch.empty(0 if self.fp32 else 3 * len(self.runs), T, dtype=torch.int64, device=self.dev)
        return buf

    def decode_scratch(self, S: int, max_splits: int) -> Tuple[torch.Tensor, ...]:
        ms = [l.mixer for l in self.cfg.layers if l.attends]
        f32 = dict(dtype=torch.float32, device=self.dev)
        return (torch.empty(S * max_splits * max([m.out_dim for m in ms], default=1), **f32),
                torch.empty(S * max_splits * max([m.heads for m in ms], default=1) * 2, **f32),
                torch.zeros(S * max([m.heads for m in ms], default=1), dtype=torch.int32, device=self.dev))

    def decode_launches(self) -> int:
        n = 2  # embedding, final norm
        for i, first in self.runs:
            l = self.cfg.layers[i]
            n += int(first) + (3 if l.attends and self._decode_fused(l.mixer) else 4 if l.attends else 5)
        return n

    def _decode_fused(self, m: ChunkAttentionSpec) -> bool:
        return not self.fp32 and bool(self.C.chunk_decode_serves(m.heads, m.kv_heads, m.dim_p, m.vdim_p))

    # ---- pieces ----
    def _target(self, j: int, T: int, buf: Dict[str, torch.Tensor], entered: bool = False) -> Target:
        """Where the residual ahead of run j goes: (h1, w1, h2, w2, sums of squares). A pass of the loop begins with a projection,
        which takes the residual as it is; ``entered`` says that it has been done."""
        if j == len(self.runs):
            return None, None, None, None, None
        i, first = self.runs[j]
        W, p = self.cfg.hidden_size, f"layers.{i}."
        if first and not entered:
            return buf["loop"][:T, :W], None, None, None, None
        h2 = buf["h"][:T, W:] if self.cfg.layers[i].ff is not None else None
        return buf["h"][:T, :W], self.w(p + "norm1"), h2, self.w(p + "norm2"), None if self.fp32 else buf["ss"][3 * j, :T]

    def _spread(self, x: torch.Tensor, to: Target) -> None:
        """fp32: the residual's consumers, as a step of its own."""
        h1, w1, h2, w2, _ = to
        if h1 is None:
            return
        if w1 is None:
            h1.copy_(x)
        else:
            self.C.rms_rows(x, self.cfg.norm_eps, self.cfg.width, h1, w1, h2, w2 if h2 is not None else None)
        self.launches += 1

    def _residual(self, a: torch.Tensor, w: torch.Tensor, x: torch.Tensor, accumulate: bool, to: Target) -> None:
        """x (+)= a w^T, then what the next run reads."""
        if self.fp32:
            self.C.gemm_f32(a, w, x, accumulate=accumulate)
            self._spread(x, to)
        else:
            h1, w1, h2, w2, ss = to
            self.C.gemm_residual(a, w, x, accumulate, h1, w1, h2, w2, ss, self.status)
        self.launches += 1

    def _project(self, j: int, h: torch.Tensor, u: torch.Tensor, act: Optional[torch.Tensor], ss: torch.Tensor) -> None:
        """Mixer projections and squared-ReLU activation of the feed-forward."""
        i = self.runs[j][0]
        m, w, W = self.cfg.layers[i].mixer, self.w(f"layers.{i}.win"), self.cfg.hidden_size
        if self.fp32:
            self.C.gemm_f32(h[:, :W], w[:m.u_dim], u)
            if act is not None:
                self.C.gemm_f32(h[:, W:], w[m.u_dim:], act, relu2=True)
                self.launches += 1
        else:
            stats = (ss[3 * j + 1], ss[3 * j + 2], m.q_dim, m.q_dim + m.k_dim) if isinstance(m, ChunkAttentionSpec) else (None, None, 0, 0)
            self.C.gemm_parallel_proj(h, w, u, act, ss[3 * j], self.cfg.width, self.cfg.norm_eps, *stats, self.status)
        self.launches += 1

    def _attention(self, j: int, u: torch.Tensor, out: torch.Tensor, sb: StepBatch, ss: torch.Tensor) -> None:
        i = self.runs[j][0]
        m, C, p = self.cfg.layers[i].mixer, self.C, f"layers.{i}."
        (cos, sin), (kc, vc) = self.rot[m.rot], self.kv[j]
        qn, kn, eps = self.w(p + "q_norm"), self.w(p + "k_norm"), self.cfg.norm_eps
        sq, sk = (None, None) if self.fp32 else (ss[3 * j + 1], ss[3 * j + 2])
        if sb.rows is None and sb.scratch is not None and self._decode_fused(m):
            C.chunk_attn_decode(u, qn, kn, eps, m.dim, cos, sin, sq, sk, sb.seq_lens, sb.block_tables, kc, vc, m.scale, m.softcap, m.chunk, out,
                                sb.splits, *sb.scratch, self.status)
            self.launches += 1
            return
        C.qk_norm_rope(u, qn, kn, eps, m.dim, cos, sin, sq, sk, sb.rows, sb.seq_lens, sb.block_tables, kc, vc, self.status)
        self.launches += 1
        if sb.rows is not None and not self.fp32:
            n = sb.pages.shape[0] * PAGE
            keys = torch.empty(n * m.k_dim, dtype=self.dtype, device=self.dev)
            values = torch.empty(n * m.v_dim, dtype=self.dtype, device=self.dev)
            if C.chunk_attn_prefill(u, kc, vc, sb.tiles, sb.pages, keys, values, sb.block_tables, m.scale, m.softcap, m.chunk, out, self.status):
                self.launches += 3
                return
        C.chunk_attn(u, kc, vc, sb.rows, sb.seq_lens, sb.block_tables, m.scale, m.softcap, m.chunk, out, self.status)
        self.launches += 1

    def _scan(self, j: int, u: torch.Tensor, out: torch.Tensor, sb: StepBatch, buf: Dict[str, torch.Tensor]) -> None:
        i = self.runs[j][0]
        m, C, T, t = self.cfg.layers[i].mixer, self.C, sb.T, self.scan[i]
        ring, state = self.state[j]
        xc = buf["xc"][:T * m.inner_p].view(T, m.inner_p)
        C.conv_silu(u, t["conv"], self.w(f"layers.{i}.conv_b"), ring, sb.rows, sb.ring_rows[m.conv] if sb.rows is not None else None, sb.seq_lens, xc,
                    self.status)
        n, rest = t["wx"].shape[0], (self.w(f"layers.{i}.wdt"), m.dt_rank, t["dt_b"], t["A"], t["D"], state, sb.segs if sb.rows is not None else None,
                                     sb.seq_lens, out)
        if self.packed(i):
            pitch = C.scan_code_pitch(m.dt_rank)
            code, bc = buf["code"][:T * pitch].view(T, pitch)[:, :m.rank_p], buf["r"][:T * (n - m.rank_p)].view(T, n - m.rank_p)
            C.gemm_split_store(xc, t["wx"], code, bc, self.status)
            C.selective_scan(xc, code, bc, u[:, m.inner_p:], *rest)
        else:
            r = buf["r"][:T * n].view(T, n)
            if self.fp32:
                C.gemm_f32(xc, t["wx"], r)
            else:
                C.gemm_bf16(xc, t["wx"], r, False, False, None, 1.0, False, self.status, None)
            C.selective_scan_plain(xc, r, u[:, m.inner_p:], *rest)
        self.launches += 3 if sb.rows is None else 4

    # ---- a step ----
    def forward(self, ids: torch.Tensor, sb: StepBatch, buf: Dict[str, torch.Tensor]) -> None:
        T, W, ss = sb.T, self.cfg.hidden_size, buf["ss"]
        x, h = buf["x"][:T], buf["h"][:T]
        x0 = buf["loop"][:T, W:] if self.cfg.loop is not None else None
        to = self._target(0, T, buf)
        if self.fp32:
            self.C.embed_norm(ids, self.w("embed"), self.cfg.embedding_scale, x, x0, None, None, None, None, None)
            self._spread(x, to)
        else:
            self.C.embed_norm(ids, self.w("embed"), self.cfg.embedding_scale, x, x0, *to[:4], ss)
        self.launches += 1
        for j, (i, first) in enumerate(self.runs):
            l = self.cfg.layers[i]
            m = l.mixer
            if first:
                self._residual(buf["loop"][:T], self.w("loop_in"), x, False, self._target(j, T, buf, entered=True))
            u = buf["u"][:T * m.u_dim].view(T, m.u_dim)
            cat = buf["cat"][:T * (m.out_dim + l.ff_p)].view(T, m.out_dim + l.ff_p)
            mixed, act = cat[:, :m.out_dim], cat[:, m.out_dim:] if l.ff is not None else None
            self._project(j, h, u, act, ss)
            if l.attends:
                self._attention(j, u, mixed, sb, ss)
            else:
                self._scan(j, u, mixed, sb, buf)
            self._residual(cat, self.w(f"layers.{i}.wout"), x, True, self._target(j + 1, T, buf))

    def hidden(self, buf: Dict[str, torch.Tensor], rows: Any) -> torch.Tensor:
        x = buf["x"][rows]
        h = torch.empty(x.shape, dtype=self.dtype, device=self.dev)
        self.C.rms_rows(x, self.cfg.norm_eps, self.cfg.width, h, self.w("final_norm"))
        self.launches += 1
        return h
