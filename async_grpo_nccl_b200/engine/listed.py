"""Rollout engine for decoders whose layers are listed one by one (``models/listed.py``).

Scheduling, slots, sampling, token history, EOS handling, slot compaction, preemption, captured decode graphs and the step
loop are ``RolloutEngine``'s. This class supplies what differs:

* the cache: the paged tensors and the per-slot state that the design's executor asks for (keys, values, convolution rings,
  scan states; layers may differ, a layer that runs twice has two); blocks that no layer can see any more go back to the pool
  while their sequence still runs;
* prompts go through in portions of at most ``max_prefill_tokens`` tokens, each from the state that the portion before left,
  so activation memory is bounded whatever the prompt's length;
* step-wise driving (``open_sequence`` / ``extend`` / ``close_sequence``): the caller supplies the tokens, in portions of any
  size, and gets logits.
"""
from __future__ import annotations

from typing import Any, Dict, List, Sequence, Tuple

import numpy as np
import torch

from ..models.listed import StepBatch, split_batch
from ..models.registry import architecture_of
from .engine import RolloutEngine, _Request


class ListedEngine(RolloutEngine):
    # ------------------------------------------------------------------ model-specific parts of the engine
    def _check_model(self, cfg: Any, params: torch.Tensor, block_size: int) -> None:
        if params.dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("parameters must be bf16 or fp32")
        if block_size != 16:
            raise ValueError("the engine supports block_size 16")

    def _init_sharing(self, tp: Any, prefix_caching: bool) -> None:
        if tp is not None and tp.size > 1:
            raise ValueError("tensor-parallel replicas are not built for this design")
        self.tp, self.tp_size, self.tp_rank = None, 1, 0
        # a cached prefix would also need the per-slot state at its end, which blocks do not carry
        self.prefix_caching = False

    def _init_decoder(self) -> None:
        self.dec = architecture_of(self.cfg).decoder()(self.cfg, self.layout, self.params, self.max_model_len)
        self.dtype = self.params.dtype

    def _bytes_per_block(self) -> int:
        n = sum(heads * size for heads, size in self.dec.paged()) * self.block_size * self.params.element_size()
        return n or 1 << 20  # a design without paged tensors still counts tokens in blocks, which then cost nothing

    def _alloc_cache(self) -> None:
        self.cache = [torch.zeros(self.num_blocks, heads, self.block_size, size, dtype=self.dtype, device=self.dev)
                      for heads, size in self.dec.paged()]
        self.slot_state = [torch.zeros(self.max_seqs, *shape, dtype=dt, device=self.dev) for shape, dt in self.dec.slot_state()]
        self.dec.bind(self.cache, self.slot_state)

    def _window_tokens(self) -> int:
        return self.dec.reach()

    def _slot_tensors(self) -> List[torch.Tensor]:
        return self.slot_state

    def _init_decode_path(self) -> None:
        S = self.max_seqs
        self.b_buf = {k: t.zero_() for k, t in self.dec.buffers(S).items()}  # idle rows hold numbers, not garbage
        self.max_splits = 8
        self.b_scratch = self.dec.decode_scratch(S, self.max_splits)
        self.b_logits = torch.empty(S, self.cfg.vocab_size, dtype=torch.float32, device=self.dev) if self.dec.fp32 else None

    def _weights_changed(self) -> None:
        self.dec.refresh_tables()

    def _copy_blocks(self, src: torch.Tensor, dst: torch.Tensor) -> None:
        for c in self.cache:
            c[dst] = c[src]

    def _share_prompt_state(self, plan: Dict[str, Any], reqs: List[_Request]) -> None:
        super()._share_prompt_state(plan, reqs)
        slots, k, src, dst = plan["seq_slots"], 0, [], []
        for r in reqs:
            src += [slots[k]] * (r.n - 1)
            dst += slots[k + 1:k + r.n]
            k += r.n
        if dst:
            idx = torch.tensor([src, dst], dtype=torch.int64).pin_memory().to(self.dev, non_blocking=True)
            self.h2d_bytes += idx.numel() * 8
            for t in self.slot_state:
                t.index_copy_(0, idx[1], t.index_select(0, idx[0]))

    def _sample(self, hidden, rows, seeds, tokens, temperature, logprobs=None) -> None:
        wl = self.dec.w("lm_head")
        if self.dec.fp32:
            z = self.b_logits[:rows]
            self.C.gemm_f32(hidden[:rows], wl, z, softcap=self.dec.softcap)
            self.C.sample_logits(z, temperature, seeds, tokens, logprobs)
        else:
            self.C.lm_sample(hidden[:rows], wl, temperature, seeds, self.b_sample_f, self.b_sample_i, tokens, logprobs, self.status,
                             softcap=self.dec.softcap)
        self.launches += 2

    # ------------------------------------------------------------------ forward passes
    def _forward(self, segments: Sequence[Tuple[int, int, np.ndarray]]) -> Dict[str, torch.Tensor]:
        """One step over segments (slot, tokens already cached, new tokens): cache and state are updated, the buffers with the
        step's rows come back (``dec.hidden`` reads them)."""
        flat, where = self.dec.tables_of(segments)
        dev_flat = torch.from_numpy(flat).pin_memory().to(self.dev, non_blocking=True)
        self.h2d_bytes += flat.nbytes
        ids, sb = split_batch(dev_flat, where, self.block_tables)
        buf = self.dec.buffers(sb.T)
        self.dec.forward(ids, sb, buf)
        return buf

    def _portions(self, segments: Sequence[Tuple[int, int, np.ndarray]]) -> List[List[Tuple[int, int, np.ndarray]]]:
        """Cuts segments into steps of at most ``max_prefill_tokens`` tokens, in order."""
        steps, cur, room = [], [], self.max_prefill_tokens
        for slot, past, toks in segments:
            a = 0
            while a < len(toks):
                n = min(room, len(toks) - a)
                cur.append((slot, past + a, toks[a:a + n]))
                a += n
                room -= n
                if room == 0:
                    steps.append(cur)
                    cur, room = [], self.max_prefill_tokens
        return steps + ([cur] if cur else [])

    def _prompt_hidden(self, plan: Dict[str, Any], reqs: List[_Request]) -> torch.Tensor:
        self._apply_table_updates(plan)
        segs, k = [], 0
        for r in reqs:
            segs.append((plan["seq_slots"][k], 0, r.prompt))
            k += r.n
        last: List[torch.Tensor] = []
        lens = {s: len(t) for s, _, t in segs}
        for step in self._portions(segs):
            buf = self._forward(step)
            t, ends = 0, []
            for slot, past, toks in step:
                t += len(toks)
                if past + len(toks) == lens[slot]:
                    ends.append(t - 1)
            if ends:
                last.append(self.dec.hidden(buf, torch.tensor(ends, device=self.dev)))
        return torch.cat(last, dim=0)

    def _decode_forward(self, B: int, temperature: float, splits: int) -> None:
        self._decode_layers(B, splits)
        self._sample(self.dec.hidden(self.b_buf, slice(0, B)), B, self.step_seeds, self.b_tokens, temperature, self.b_lp)
        self._feed_back(B)

    def _decode_layers(self, B: int, splits: int) -> None:
        sb = StepBatch(B, self.block_tables, seq_lens=self.seq_lens, splits=splits, scratch=self.b_scratch)
        self.C.set_pdl(self.use_pdl)  # this thread only: prologues overlap the tail of the kernel before
        try:
            self.dec.forward(self.last_tokens[:B], sb, self.b_buf)
        finally:
            self.C.set_pdl(False)

    def _choose_splits(self, B: int, n_active: int, max_len: int) -> int:
        """One wave of CTAs where there are few sequences, each with at least two tiles of 64 keys."""
        want = int(self.sm_count * self.dec.ctas_per_sm) // max(1, n_active)
        return int(max(1, min(self.max_splits, want, min(max_len, self.dec.reach()) // 128)))

    def _launch_count_decode(self, splits: int, B: int = 0) -> int:
        return self.dec.decode_launches() + 2

    # ------------------------------------------------------------------ step-wise driving
    def open_sequence(self) -> int:
        seq_id, slot = self.sched.open_seq()
        self.h_lens[slot] = 0
        return int(seq_id)

    def close_sequence(self, seq_id: int) -> None:
        slot = self.sched.seq_info(seq_id)["slot"]
        self.sched.finish(seq_id)
        self.h_lens[slot] = 0

    @torch.no_grad()
    def extend(self, entries: Sequence[Tuple[int, Sequence[int], Sequence[int]]]) -> torch.Tensor:
        """Each entry brings the next tokens of one open sequence and the places among them whose logits are wanted.
        Single tokens of sequences that have begun go through the decode step, everything else through the prompt step.
        Returns fp32 logits [wanted, vocab] in the order of the entries and of their places."""
        segs, dec, updates = [], [], []
        for n_entry, (seq_id, tokens, want) in enumerate(entries):
            toks = np.ascontiguousarray(np.asarray(tokens, dtype=np.int32))
            info = self.sched.seq_info(seq_id)
            past, slot = int(info["len"]), int(info["slot"])
            if past + len(toks) > self.max_model_len:
                raise ValueError("sequence would exceed max_model_len")
            updates += self.sched.extend_seq(seq_id, len(toks))
            (dec if len(toks) == 1 and past > 0 else segs).append((n_entry, slot, past, toks, list(want)))
        out: Dict[int, torch.Tensor] = {}
        if updates:
            u = np.asarray(updates, dtype=np.int64)
            self._apply_table_updates({"upd_slot": u[:, 0].tolist(), "upd_index": u[:, 1].tolist(), "upd_block": u[:, 2].tolist()})
        for step in self._portions([(s, p, t) for _, s, p, t, _ in segs]):
            buf = self._forward(step)
            t0 = 0
            for slot, past, toks in step:
                n_entry, _, past0, _, want = next(e for e in segs if e[1] == slot)
                rows = [t0 + past0 + w - past for w in want if past <= past0 + w < past + len(toks)]
                if rows:
                    z = self.dec.logits(self.dec.hidden(buf, torch.tensor(rows, device=self.dev)))
                    out[n_entry] = torch.cat([out[n_entry], z]) if n_entry in out else z
                self.h_lens[slot] = past + len(toks)
                t0 += len(toks)
        if dec:
            active = np.asarray([d[1] for d in dec], dtype=np.int64)
            feed = torch.tensor([[d[1] for d in dec], [int(d[3][0]) for d in dec]], dtype=torch.int64).pin_memory().to(self.dev, non_blocking=True)
            self.last_tokens.index_copy_(0, feed[0], feed[1].to(torch.int32))
            self.h_lens[active] = [d[2] for d in dec]
            none = np.zeros(0, np.int64)
            self._stage_decode(active, none, none, none)
            B = min(self.max_seqs, (int(active.max()) + 32) // 32 * 32)
            self._decode_layers(B, self._choose_splits(B, len(dec), int(self.h_lens[active].max())))
            for n_entry, slot, _, _, want in dec:
                if want:
                    out[n_entry] = self.dec.logits(self.dec.hidden(self.b_buf, slice(slot, slot + 1))).expand(len(want), -1)
        self.launches += self.dec.launches
        self.dec.launches = 0
        if not out:
            return torch.empty(0, self.cfg.vocab_size)
        return torch.cat([out[k] for k in sorted(out)], dim=0)
