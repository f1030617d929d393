"""Rollout engine for decoders whose layers are listed one by one (``models/listed.py``).

Scheduling, slots, sampling, token history, EOS handling, slot compaction, preemption, captured decode graphs and the step
loop are ``RolloutEngine``'s. This class supplies what differs:

* the cache: one paged key tensor per layer (layers may differ in heads and head size; the values are the keys) and one
  ring per slot and layer with the last projected values of the short convolutions; blocks that have left every layer's
  window go back to the pool while their sequence still runs;
* prompts go through in portions of at most ``max_prefill_tokens`` tokens, each from the state that the portion before left,
  so activation memory is bounded whatever the prompt's length;
* step-wise driving (``open_sequence`` / ``extend`` / ``close_sequence``): the caller supplies the tokens, in portions of any
  size, and gets logits.
"""
from __future__ import annotations

from typing import Any, Dict, List, Sequence, Tuple

import numpy as np
import torch

from ..models.listed import ListedDecoder, StepBatch, host_batch, split_batch
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
        # a cached prefix would also need the convolution state at its end, which blocks do not carry
        self.prefix_caching = False

    def _init_decoder(self) -> None:
        self.dec = ListedDecoder(self.cfg, self.layout, self.params, self.max_model_len)
        self.dtype = self.params.dtype

    def _bytes_per_block(self) -> int:
        return sum(l.mixer.k_dim for l in self.cfg.layers) * self.block_size * self.params.element_size()

    def _alloc_cache(self) -> None:
        kw = dict(dtype=self.dtype, device=self.dev)
        ms = [l.mixer for l in self.cfg.layers]
        self.cache = [torch.zeros(self.num_blocks, m.kv_heads, self.block_size, m.dim_p, **kw) for m in ms]
        # convolution rings: position p of a sequence at p % taps; one row per slot for all layers
        sizes = [m.conv * m.qk_dim for m in ms]
        self.ring = torch.zeros(self.max_seqs, sum(sizes), **kw)
        offs = np.concatenate([[0], np.cumsum(sizes)])
        self.rings = [self.ring[:, int(o):int(o) + n].view(self.max_seqs, m.conv, m.qk_dim) for o, n, m in zip(offs, sizes, ms)]

    def _window_tokens(self) -> int:
        return self.cfg.max_window

    def _slot_tensors(self) -> List[torch.Tensor]:
        return [self.ring]

    def _init_decode_path(self) -> None:
        S, W = self.max_seqs, self.cfg.hidden_size
        self.b_x = torch.zeros(S, W, dtype=torch.float32, device=self.dev)
        self.b_h = torch.zeros(S, W, dtype=self.dtype, device=self.dev)
        self.b_buf = {k: t.zero_() for k, t in self.dec.buffers(S).items()}  # idle rows hold numbers, not garbage
        self.max_splits = 8
        self.ctas_per_sm = max(1, min(self.dec.decode_ctas_per_sm(i) for i in range(len(self.cfg.layers))))
        ms = [l.mixer for l in self.cfg.layers]
        f32 = dict(dtype=torch.float32, device=self.dev)
        self.b_scratch = (torch.empty(S * self.max_splits * max(m.heads * m.k_dim for m in ms), **f32),
                          torch.empty(S * self.max_splits * max(m.heads for m in ms) * 2, **f32),
                          torch.zeros(S, dtype=torch.int32, device=self.dev))
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
            self.ring.index_copy_(0, idx[1], self.ring.index_select(0, idx[0]))

    def _sample(self, hidden, rows, seeds, tokens, temperature, logprobs=None) -> None:
        if not self.dec.fp32:
            return super()._sample(hidden, rows, seeds, tokens, temperature, logprobs)
        z = self.b_logits[:rows]
        self.C.gemm_f32(hidden[:rows], self.dec.w("lm_head"), z)
        self.C.sample_logits(z, temperature, seeds, tokens, logprobs)
        self.launches += 2

    # ------------------------------------------------------------------ forward passes
    def _forward(self, segments: Sequence[Tuple[int, int, np.ndarray]]) -> torch.Tensor:
        """One step over segments (slot, tokens already cached, new tokens): keys and rings are updated, the final normed
        hidden states of all rows come back."""
        flat, where = host_batch(segments, [l.mixer.conv for l in self.cfg.layers], self.cfg.max_window)
        dev_flat = torch.from_numpy(flat).pin_memory().to(self.dev, non_blocking=True)
        self.h2d_bytes += flat.nbytes
        ids, sb = split_batch(dev_flat, where, self.block_tables)
        T = sb.T
        x = torch.empty(T, self.cfg.hidden_size, dtype=torch.float32, device=self.dev)
        h = torch.empty(T, self.cfg.hidden_size, dtype=self.dtype, device=self.dev)
        self._layers(ids, x, h, sb, self.dec.buffers(T))
        return h

    def _layers(self, ids: torch.Tensor, x: torch.Tensor, h: torch.Tensor, sb: StepBatch, buf: Dict[str, torch.Tensor]) -> None:
        self.dec.embed(ids, x, h)
        for i in range(len(self.cfg.layers)):
            self.dec.layer(i, x, h, sb, self.cache[i], self.rings[i], buf)

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
            h = self._forward(step)
            t = 0
            for slot, past, toks in step:
                t += len(toks)
                if past + len(toks) == lens[slot]:
                    last.append(h[t - 1:t])
        return torch.cat(last, dim=0)

    def _decode_forward(self, B: int, temperature: float, splits: int) -> None:
        self._decode_layers(B, splits)
        self._sample(self.b_h[:B], B, self.step_seeds, self.b_tokens, temperature, self.b_lp)
        self._feed_back(B)

    def _decode_layers(self, B: int, splits: int) -> None:
        sb = StepBatch(B, self.block_tables, seq_lens=self.seq_lens, splits=splits, scratch=self.b_scratch)
        self.C.set_pdl(self.use_pdl)  # this thread only: prologues overlap the tail of the kernel before
        try:
            self._layers(self.last_tokens[:B], self.b_x[:B], self.b_h[:B], sb, self.b_buf)
        finally:
            self.C.set_pdl(False)

    def _choose_splits(self, B: int, n_active: int, max_len: int) -> int:
        """One wave of CTAs where there are few sequences, each with at least two tiles of 64 keys."""
        want = (self.sm_count * self.ctas_per_sm) // max(1, n_active)
        return int(max(1, min(self.max_splits, want, min(max_len, self.cfg.max_window) // 128)))

    def _launch_count_decode(self, splits: int, B: int = 0) -> int:
        n = 1 + 2
        for i, l in enumerate(self.cfg.layers):
            n += (3 if self.dec.decode_ctas_per_sm(i) else 5) + (0 if l.ff is None else 2)
        return n

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
            h = self._forward(step)
            t0 = 0
            for slot, past, toks in step:
                n_entry, _, past0, _, want = next(e for e in segs if e[1] == slot)
                rows = [t0 + past0 + w - past for w in want if past <= past0 + w < past + len(toks)]
                if rows:
                    z = self.dec.logits(h.index_select(0, torch.tensor(rows, device=self.dev)))
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
                    out[n_entry] = self.dec.logits(self.b_h[slot:slot + 1]).expand(len(want), -1)
        self.launches += self.dec.launches
        self.dec.launches = 0
        if not out:
            return torch.empty(0, self.cfg.vocab_size)
        return torch.cat([out[k] for k in sorted(out)], dim=0)
