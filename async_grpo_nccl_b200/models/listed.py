"""Native executors of decoders whose layers are listed one by one: what all such designs share.

An executor owns no cache and no loop over steps. It says which paged tensors and which per-slot state each of its layer runs
needs; the engine allocates them, hands them back through ``bind`` and drives ``forward`` with a ``StepBatch`` that says where
every token row lives. The same layer code serves whole prompts, portions of prompts, mixed batches and decode steps; decode
differs only in the kernels that are picked. ``models/dezelorn_decoder.py`` and ``models/vazatar_decoder.py`` fill in the layers.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Sequence, Tuple

import numpy as np
import torch

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
    segs: Optional[torch.Tensor] = None      # [n, 4]: first row, rows, slot, position of the first row
    ring_rows: Optional[Dict[int, torch.Tensor]] = None  # taps -> the last `taps` rows of each segment
    tiles: Optional[torch.Tensor] = None     # [n, 4]: first row, rows, position of the first row, row of position 0 in the gathered keys
    pages: Optional[torch.Tensor] = None     # [n, 2]: slot, page: the key pages that the step can see, in the order they are gathered
    seq_lens: Optional[torch.Tensor] = None
    splits: int = 1
    scratch: Optional[Tuple[torch.Tensor, ...]] = None  # decode: partial products, (max, sum), tickets


def host_batch(segments: Sequence[Tuple[int, int, np.ndarray]], taps: Sequence[int], window: int,
               chunks: Sequence[int] = ()) -> Tuple[np.ndarray, Dict[str, Tuple[int, int]]]:
    """(slot, tokens already there, new tokens) per segment -> one int32 array with the step's tables and where each of them
    is in it: token ids, rows, segments, attention tiles, the key pages that can be seen (those within ``window``; with
    ``chunks``, those of the chunks that the segment's first token lies in) and, for every length in ``taps``, the rows that
    the convolution rings keep."""
    ids, rows, segs, tiles, pages = [], [], [], [], []
    n_pages = 0
    keep: Dict[int, List[np.ndarray]] = {k: [] for k in sorted(set(taps))}
    t0 = 0
    for slot, past, toks in segments:
        n = len(toks)
        ids.append(np.asarray(toks, dtype=np.int32))
        r = np.zeros((n, 4), np.int32)
        r[:, 0], r[:, 1], r[:, 2] = slot, past + np.arange(n), t0
        rows.append(r)
        segs.append((t0, n, slot, past))
        first = min(past // c * c for c in chunks) // PAGE if chunks else max(0, past - window + 1) // PAGE
        count = (past + n - 1) // PAGE + 1 - first
        pages.append(np.stack([np.full(count, slot, np.int32), np.arange(first, first + count, dtype=np.int32)], axis=1))
        tiles += [(t0 + a, min(TILE, n - a), past + a, (n_pages - first) * PAGE) for a in range(0, n, TILE)]
        n_pages += count
        for k, v in keep.items():
            v.append(np.arange(t0 + max(0, n - k), t0 + n, dtype=np.int32))
        t0 += n
    tiles.sort(key=lambda t: -t[2])
    parts = {"rows": np.concatenate(rows).ravel(), "tiles": np.asarray(tiles, np.int32).ravel(), "segs": np.asarray(segs, np.int32).ravel(),
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
                                  segs=part["segs"].view(-1, 4), pages=part["pages"].view(-1, 2),
                                  ring_rows={int(k[4:]): v for k, v in part.items() if k.startswith("ring")})


class ListedDecoder:
    """What the engine relies on. ``slot_state`` tensors travel with a sequence when slots move and are copied when samples share a
    prompt; a sequence that starts finds whatever the slot's last one left, so a mechanism must not read state before position 0."""

    launches: int
    ctas_per_sm = 1            # decode attention CTAs that fit an SM
    softcap = 0.0              # of the logits, 0 = none

    def __init__(self, cfg: Any, layout: ParamLayout, params: torch.Tensor, max_len: int):
        from ..ops import native

        self.C = native()
        self.cfg, self.layout, self.params = cfg, layout, params
        self.dev, self.dtype = params.device, params.dtype
        self.fp32 = params.dtype == torch.float32
        self.max_len = int(max_len)
        self.status = torch.zeros(1, dtype=torch.int32, device=self.dev)
        self.launches = 0
        self._w: Dict[str, torch.Tensor] = {n: layout.view(params, n) for n in layout.segments}
        self.refresh_tables()

    def w(self, name: str) -> torch.Tensor:
        return self._w[name]

    def check_status(self) -> None:
        code = int(self.status.item())
        if code != 0:
            self.status.zero_()
            raise RuntimeError(f"device kernel reported status {code} (bounded wait ran out or bad index)")

    # ---- what a design supplies ----
    def refresh_tables(self) -> None:
        """Tables that follow from configuration and weights. They keep their storage when the weights change, so captured
        graphs stay valid."""
        raise NotImplementedError

    def paged(self) -> List[Tuple[int, int]]:
        """(heads, size) of every paged tensor; each holds [blocks, heads, 16, size] values of the activation type."""
        raise NotImplementedError

    def slot_state(self) -> List[Tuple[Tuple[int, ...], torch.dtype]]:
        """Shape (without the slot) and type of every per-slot tensor."""
        raise NotImplementedError

    def bind(self, paged: List[torch.Tensor], slots: List[torch.Tensor]) -> None:
        raise NotImplementedError

    def reach(self) -> int:
        """No layer looks further back than this many tokens (the current one included)."""
        raise NotImplementedError

    def tables_of(self, segments: Sequence[Tuple[int, int, np.ndarray]]) -> Tuple[np.ndarray, Dict[str, Tuple[int, int]]]:
        raise NotImplementedError

    def buffers(self, T: int) -> Dict[str, torch.Tensor]:
        raise NotImplementedError

    def decode_scratch(self, S: int, max_splits: int) -> Tuple[torch.Tensor, ...]:
        raise NotImplementedError

    def forward(self, ids: torch.Tensor, sb: StepBatch, buf: Dict[str, torch.Tensor]) -> None:
        raise NotImplementedError

    def hidden(self, buf: Dict[str, torch.Tensor], rows: Any) -> torch.Tensor:
        """Final normed hidden states of rows of the last ``forward`` (a slice or an index tensor)."""
        raise NotImplementedError

    def decode_launches(self) -> int:
        """Kernels of a decode step without sampling."""
        raise NotImplementedError

    # ---- shared ----
    def logits(self, h: torch.Tensor) -> torch.Tensor:
        wl = self.w("lm_head")
        out = torch.empty(h.shape[0], wl.shape[0], dtype=torch.float32, device=self.dev)
        if self.fp32:
            self.C.gemm_f32(h, wl, out, softcap=self.softcap)
        else:
            self.C.gemm_bf16(h, wl, out, False, False, None, 1.0, False, self.status, None)
            if self.softcap > 0:
                self.C.softcap_rows(out, self.softcap)
                self.launches += 1
        self.launches += 1
        return out
