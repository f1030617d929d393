"""Serving throughput of a listed-layer design beside the dense model of equal size, and the kernels behind it.

    python bench.py --serving vazatar-1.5b:qwen2.5-1.5b,dezelorn-7b:qwen2.5-7b

Random weights, synthetic prompts; every preset with its first layers only. Prefill: prompts of ``--serving-prompt`` tokens through the engine's own prompt step;
decode: the engine's captured decode step. Times are CUDA events on the launching stream after warm-up; kernel times are
medians with the L2 flushed (a buffer larger than L2 is written) between iterations. One JSON line per record.
"""
from __future__ import annotations

import json
import os
from typing import Any, Callable, Dict, List, Tuple

import numpy as np
import torch

from .microbench import flush_l2, timeit


def peaks() -> Dict[str, Any]:
    root = os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
    for p in (os.environ.get("AGRPO_PEAKS_FILE"), os.path.join(root, "MEASURED_PEAKS.json")):
        if p and os.path.exists(p):
            with open(p) as f:
                d = json.load(f)
            return {"hbm_gbs": float(d["hbm_gbs"]), "bf16_tflops": float(d["bf16_tflops"]), "source": "measured"}
    return {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "source": "fallback"}


def out(rec: Dict[str, Any]) -> None:
    print(json.dumps(rec), flush=True)


def make_engine(model: str, max_seqs: int, max_len: int, n_layers: int, blocks: int, **kw: Any) -> Any:
    """Engine on the first ``n_layers`` layers of a preset (a stack of equal layers: time per layer does not depend on how many)."""
    from dataclasses import replace

    from ..models.registry import architecture_of, build_engine, make_layout, resolve_model_config

    cfg = resolve_model_config(model)
    if architecture_of(cfg).name == "dense":
        cfg = replace(cfg, num_hidden_layers=n_layers)
    else:
        cfg = cfg.first_layers(n_layers)
    layout = make_layout(cfg)
    params = torch.empty(layout.total, dtype=torch.bfloat16, device="cuda")
    layout.init_random_device_(params, 0)
    return cfg, build_engine(cfg, layout, params, max_seqs=max_seqs, max_model_len=max_len, num_blocks=blocks, use_cuda_graph=True,
                             max_prefill_tokens=1 << 20, **kw)


def bench_prefill(model: str, prompt: int, n_prompts: int, n_layers: int, iters: int = 5) -> Dict[str, Any]:
    max_len = prompt + 32
    cfg, eng = make_engine(model, 32, max_len, n_layers, n_prompts * (prompt // 16 + 4) + 64)
    rng = np.random.default_rng(0)
    times = []
    for it in range(iters + 3):
        for i in range(n_prompts):
            eng.add_request((it, i), rng.integers(0, cfg.vocab_size, prompt).astype(np.int32), n=1, max_new_tokens=1, temperature=0.0,
                            ignore_eos=True)
        eng._admit_pending()
        plan = eng.sched.plan_prefill()
        assert len(plan["group_ids"]) == n_prompts
        reqs = [eng.requests[g] for g in plan["group_ids"]]
        torch.cuda.synchronize()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        eng._prompt_hidden(plan, reqs)
        e1.record()
        torch.cuda.synchronize()
        if it >= 3:
            times.append(e0.elapsed_time(e1))
        for s in plan["seq_ids"]:
            eng.sched.finish(s)
    eng.check_status()
    ms = sorted(times)[len(times) // 2]
    return {"bench": "prefill", "model": model, "layers": n_layers, "prompts": n_prompts, "prompt_len": prompt, "ms": round(ms, 3),
            "tokens_per_s": round(prompt * n_prompts / ms * 1e3), "us_per_layer": round(ms * 1e3 / n_layers, 1)}


def bench_decode(model: str, batch: int, context: int, n_layers: int, steps: int = 40) -> Dict[str, Any]:
    max_len = context + steps + 64
    cfg, eng = make_engine(model, max(32, batch), max_len, n_layers, batch * (max_len // 16 + 2) + 256)
    rng = np.random.default_rng(0)
    for i in range(batch):
        eng.add_request(i, rng.integers(0, cfg.vocab_size, context).astype(np.int32), n=1, max_new_tokens=steps + 16, temperature=1.0, seed=i,
                        forced_new_tokens=[steps + 16])
    while eng.sched.num_waiting > 0 or eng.pending:
        eng.step()
    for _ in range(4):
        eng.step()
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    for _ in range(steps):
        eng.step()
    e1.record()
    torch.cuda.synchronize()
    eng.check_status()
    ms = e0.elapsed_time(e1) / steps
    return {"bench": "decode", "model": model, "layers": n_layers, "batch": batch, "context": context, "ms_per_step": round(ms, 4),
            "tokens_per_s": round(batch / ms * 1e3)}


Case = Tuple[str, str, Callable[[], Any], float, float]


def dezelorn_cases(new: Any, old: Any, T: int, prompt: int, B: int, ctx: int) -> List[Case]:
    """(phase / role, side, launch, FLOPs, bytes) of like kernels of one layer: ``new`` a listed-layer configuration, ``old`` the
    dense one. FLOPs count what the operation needs, not what a kernel spends (scores and one product per pair)."""
    from ..ops import native
    from .microbench import _tiles
    from ..models.listed import host_batch, split_batch

    C = native()
    bf, dev = torch.bfloat16, "cuda"
    st = torch.zeros(1, dtype=torch.int32, device=dev)
    m = new.layers[0].mixer
    W, F, H, G, D = new.hidden_size, new.layers[0].ff_p, m.heads, m.kv_heads, m.dim_p
    R = lambda *s: torch.randn(*s, device=dev).to(bf)
    Wr = lambda *s: (torch.randn(*s, device=dev) * 0.02).to(bf)
    cases: List[Case] = []

    def add(role: str, side: str, fn: Callable[[], Any], flops: float, nbytes: float) -> None:
        cases.append((role, side, fn, flops, nbytes))

    n_seq = T // prompt
    wqkg, wqkv, wo, wgu, wd = Wr(m.u_dim, W), Wr(old.qkv_dim, W), Wr(W, H * D), Wr(2 * F, W), Wr(W, F)
    nrm = [torch.ones(W, device=dev, dtype=bf), torch.zeros(W, device=dev, dtype=bf), torch.full((1,), 0.5, device=dev, dtype=bf)]
    ln = torch.ones(W, device=dev, dtype=bf)
    maxlen = max(prompt, ctx) + 64
    bias = torch.rand(H, min(m.window, maxlen), device=dev)
    qscale = torch.full((maxlen,), 0.1, device=dev)
    talk = (torch.eye(H, device=dev) + 0.02 * torch.randn(H, H, device=dev)).to(bf)
    conv = R(m.conv, m.qk_dim)

    # ---------------- prompts ----------------
    h, x, ho = R(T, W), torch.randn(T, W, device=dev), torch.empty(T, W, device=dev, dtype=bf)
    xb, xb2 = R(T, W), torch.empty(T, W, device=dev, dtype=bf)
    u, qkv = R(T, m.u_dim), R(T, old.qkv_dim)
    a, act, gu = R(T, H * D), torch.empty(T, F, device=dev, dtype=bf), torch.empty(T, 2 * F, device=dev, dtype=bf)
    q = R(T, H * D)
    nb = (prompt + 15) // 16
    cache = R(n_seq * nb, G, 16, D)
    tables = torch.randperm(n_seq * nb, device=dev).int().view(n_seq, nb).contiguous()
    ring = torch.zeros(max(n_seq, B), m.conv, m.qk_dim, device=dev, dtype=bf)
    flat, where = host_batch([(i, 0, np.zeros(prompt, np.int32)) for i in range(n_seq)], [m.conv], m.window)
    _, sb = split_batch(torch.from_numpy(flat).to(dev), where, tables)
    acc = torch.empty(T * H * G * D, device=dev, dtype=bf)
    keys = torch.empty(sb.pages.shape[0] * 16 * G * D, device=dev, dtype=bf)
    lse = torch.empty(H, T, device=dev)
    tiles = _tiles([prompt] * n_seq)
    pairs = n_seq * sum(min(i + 1, m.window) for i in range(prompt))
    pairs_old = n_seq * prompt * (prompt + 1) / 2
    gm = lambda M, N, K: (2.0 * M * N * K, 2.0 * (M * K + N * K + M * N))
    add("prompt projection", "new", lambda: C.gemm_bf16(h, wqkg, u, False, False, None, 1.0, False, st, None), *gm(T, m.u_dim, W))
    add("prompt projection", "old", lambda: C.gemm_bf16(h, wqkv, qkv, False, False, None, 1.0, False, st, None), *gm(T, old.qkv_dim, W))
    add("prompt position op", "new", lambda: C.short_conv(u, conv, ring, sb.rows, sb.ring_rows[m.conv], None, tables, q, cache, st), 0.0, 4.0 * T * m.qk_dim)
    pos = torch.arange(T, device=dev, dtype=torch.int32) % prompt
    cos = torch.rand(maxlen, D // 2, device=dev)
    slots = torch.arange(T, device=dev, dtype=torch.int32)
    kc, vc = torch.zeros(n_seq * nb, G, 16, D, device=dev, dtype=bf), torch.zeros(n_seq * nb, G, 16, D, device=dev, dtype=bf)

    def rope():
        C.rope_inplace(qkv, pos, cos, cos, H + G, D, False)
        C.kv_cache_write(qkv, slots, kc, vc, H, G, D, st, 0)
    add("prompt position op", "old", rope, 0.0, 4.0 * T * (H + G) * D + 8.0 * T * G * D)
    add("prompt attention", "new", lambda: C.talk_attn_prefill(q, cache, sb.tiles, sb.pages, keys, tables, bias, qscale, talk, u[:, m.qk_dim:], m.window, acc, a, st),
        4.0 * pairs * H * D, 0.0)
    add("prompt attention", "old", lambda: C.attn_varlen_fwd(qkv, a, lse, tiles, H, G, D, 0.1, st), 4.0 * pairs_old * H * D, 0.0)
    add("prompt out projection + tail", "new", lambda: C.gemm_dyt(a, wo, x, nrm, nrm, ho, st), *gm(T, W, H * D))

    def wo_old():
        C.gemm_bf16(a, wo, xb2, False, False, None, 1.0, False, st, xb)
        C.rmsnorm_fwd(xb2, ln, ho, None, 1e-6)
    add("prompt out projection + tail", "old", wo_old, *gm(T, W, H * D))
    add("prompt gate/up", "new", lambda: C.gemm_swiglu(ho, wgu, act, None, 0.0, st), *gm(T, 2 * F, W))

    def gu_old():
        C.gemm_bf16(ho, wgu, gu, False, False, None, 1.0, False, st, None)
        C.swiglu_fwd(gu, act)
    add("prompt gate/up", "old", gu_old, *gm(T, 2 * F, W))
    add("prompt down + tail", "new", lambda: C.gemm_dyt(act, wd, x, nrm, nrm, ho, st), *gm(T, W, F))

    def wd_old():
        C.gemm_bf16(act, wd, xb2, False, False, None, 1.0, False, st, xb)
        C.rmsnorm_fwd(xb2, ln, ho, None, 1e-6)
    add("prompt down + tail", "old", wd_old, *gm(T, W, F))

    # ---------------- decode ----------------
    nbd = (ctx + 15) // 16 + 1
    dcache, dk, dv = R(B * nbd, G, 16, D), R(B * nbd, G, 16, D), R(B * nbd, G, 16, D)
    dtab = torch.randperm(B * nbd, device=dev).int().view(B, nbd).contiguous()
    lens = torch.full((B,), ctx, device=dev, dtype=torch.int32)
    hb, ub, qb = R(B, W), R(B, m.u_dim), R(B, old.qkv_dim)
    ab, actb, xbd, hob = R(B, H * D), R(B, F), torch.randn(B, W, device=dev), torch.empty(B, W, device=dev, dtype=bf)
    part_o, part_ml = torch.empty(B * 8 * H * G * D, device=dev), torch.empty(B * 8 * H * G * 16, device=dev)
    tick = torch.zeros(B * G, device=dev, dtype=torch.int32)
    n_sm = torch.cuda.get_device_properties(0).multi_processor_count
    seen = min(ctx, m.window)
    sp_new = max(1, min(8, C.talk_decode_ctas_per_sm(H, G, D) * n_sm // B, seen // 128))
    sp_old = max(1, min(8, 3 * n_sm // (B * G), ctx // 256))
    wb = lambda N, K, extra=0: 2.0 * N * K + 2.0 * B * (N + K) + extra
    ss = torch.full((B,), W << 30, device=dev, dtype=torch.int64)
    add("decode projection", "new", lambda: C.gemm_bf16(hb, wqkg, ub, False, False, None, 1.0, False, st, None), 0.0, wb(m.u_dim, W))
    add("decode projection", "old", lambda: C.gemm_decode(hb, wqkv, qb, None, None, ss, None, 1e-6, st), 0.0, wb(old.qkv_dim, W))
    add("decode attention", "new", lambda: C.talk_attn_decode(ub, conv, ring[:B], dcache, lens, dtab, bias, qscale, talk, ub[:, m.qk_dim:],
                                                              m.window, ab, sp_new, part_o, part_ml, tick, st), 0.0, 2.0 * B * seen * G * D)
    add("decode attention", "old", lambda: C.paged_decode_attn(qb, dk, dv, dtab, lens, ab, H, G, D, 0.1, sp_old, part_o, part_ml, st, tick),
        0.0, 4.0 * B * ctx * G * D)
    add("decode out projection + tail", "new", lambda: C.gemm_dyt(ab, wo, xbd, nrm, nrm, hob, st), 0.0, wb(W, H * D, 12 * B * W))
    so = torch.zeros(B, device=dev, dtype=torch.int64)
    xs = R(B, W)
    add("decode out projection + tail", "old", lambda: C.gemm_decode(ab, wo, hob, None, xs, None, so, 1e-6, st), 0.0, wb(W, H * D, 4 * B * W))
    add("decode gate/up", "new", lambda: C.gemm_swiglu(hb, wgu, actb, None, 0.0, st), 0.0, wb(2 * F, W))
    add("decode gate/up", "old", lambda: C.gemm_swiglu(hb, wgu, actb, ss, 1e-6, st), 0.0, wb(2 * F, W))
    add("decode down + tail", "new", lambda: C.gemm_dyt(actb, wd, xbd, nrm, nrm, hob, st), 0.0, wb(W, F, 12 * B * W))
    add("decode down + tail", "old", lambda: C.gemm_decode(actb, wd, hob, None, xs, None, so, 1e-6, st), 0.0, wb(W, F, 4 * B * W))
    return cases


def vazatar_cases(new: Any, old: Any, T: int, prompt: int, B: int, ctx: int) -> List[Case]:
    """Like kernels of one attention layer and one scan layer against those of a dense layer. The input GEMM of a parallel block
    stands against the dense layer's two norms, two projections and SwiGLU, its output GEMM against two projections with residual.
    Convolution, narrow projection and scan have no counterpart."""
    from ..models.listed import LOG2E, host_batch, split_batch
    from ..ops import native
    from .microbench import _tiles

    C, bf, dev = native(), torch.bfloat16, "cuda"
    st = torch.zeros(1, dtype=torch.int32, device=dev)
    la, ls = next(l for l in new.layers if l.attends), next(l for l in new.layers if not l.attends)
    m, sc = la.mixer, ls.mixer
    W, F, Fo, H, G, D, E = new.hidden_size, la.ff_p, old.intermediate_size, m.heads, m.kv_heads, m.dim_p, m.vdim_p
    R = lambda *s: torch.randn(*s, device=dev).to(bf)
    Wr = lambda *s: (torch.randn(*s, device=dev) * 0.02).to(bf)
    Z = lambda *s: torch.empty(*s, device=dev, dtype=bf)
    cases: List[Case] = []
    add = lambda role, side, fn, flops, nbytes: cases.append((role, side, fn, flops, nbytes))
    win, wout = Wr(m.u_dim + F, W), Wr(W, m.out_dim + F)
    swin, swout = Wr(sc.u_dim + F, W), Wr(W, sc.out_dim + F)
    wqkv, wo, wgu, wd = Wr(old.qkv_dim, W), Wr(W, H * D), Wr(2 * Fo, W), Wr(W, Fo)
    ln, qn, kn = Wr(W), 1 + Wr(m.q_dim), 1 + Wr(m.k_dim)
    maxlen = max(prompt, ctx) + 64
    ang = torch.rand(maxlen, m.rot.dims // 2, device=dev)
    cos, sin = torch.cos(ang), torch.sin(ang)
    n_st = 4 * C.scan_states_per_lane(sc.state)
    wx, wdt, conv, conv_b = Wr(sc.rank_p + 2 * n_st, sc.inner_p), Wr(sc.inner_p, sc.rank_p), R(sc.conv, sc.inner_p), Wr(sc.inner_p)
    dt_b, skip = torch.full((sc.inner_p,), -4.0, device=dev), torch.ones(sc.inner_p, device=dev)
    A = -torch.arange(1, n_st + 1, device=dev, dtype=torch.float32).expand(sc.inner_p, n_st).contiguous() * LOG2E
    gm = lambda M, N, K: (2.0 * M * N * K, 2.0 * (M * K + N * K + M * N))

    def gemms(*shapes: Tuple[int, int, int], extra: float = 0.0) -> Tuple[float, float]:
        f, b = zip(*(gm(*s) for s in shapes))
        return sum(f), sum(b) + extra

    def pair(phase: str, M: int) -> Tuple[torch.Tensor, ...]:
        """Input and output GEMMs of a layer; returns what the mixer cases of the phase work on."""
        h, x, u, cat, ss = R(M, 2 * W), torch.randn(M, W, device=dev), R(M, m.u_dim), R(M, m.out_dim + F), torch.zeros(6, M, dtype=torch.int64, device=dev)
        su, scat = R(M, sc.u_dim), R(M, sc.out_dim + F)
        ss[0] = W << 30
        ss[4], ss[5] = (H * m.dim) << 30, (G * m.dim) << 30
        add(f"{phase} input projections", "new", lambda: C.gemm_parallel_proj(h, win, u, cat[:, m.out_dim:], ss[0], W, 1e-5, ss[1], ss[2], m.q_dim,
                                                                              m.q_dim + m.k_dim, st), *gemms((M, m.u_dim + F, W), extra=2.0 * M * W))
        add(f"{phase} scan input projections", "new", lambda: C.gemm_parallel_proj(h, swin, su, scat[:, sc.out_dim:], ss[0], W, 1e-5, None, None, 0, 0, st),
            *gemms((M, sc.u_dim + F, W), extra=2.0 * M * W))
        add(f"{phase} output projections", "new", lambda: C.gemm_residual(cat, wout, x, True, h[:, :W], ln, h[:, W:], ln, ss[3], st),
            *gemms((M, W, m.out_dim + F), extra=10.0 * M * W))
        add(f"{phase} scan output projections", "new", lambda: C.gemm_residual(scat, swout, x, True, h[:, :W], ln, h[:, W:], ln, ss[3], st),
            *gemms((M, W, sc.out_dim + F), extra=10.0 * M * W))
        return u, cat, ss, su, scat

    # ---------------- prompts ----------------
    n_seq, nb = T // prompt, (prompt + 15) // 16
    u, cat, ss, su, scat = pair("prompt", T)
    hb, xb, xb2, qkv, a, gu, act = R(T, W), R(T, W), Z(T, W), R(T, old.qkv_dim), R(T, H * D), Z(T, 2 * Fo), R(T, Fo)

    def in_old():
        C.rmsnorm_fwd(xb, ln, hb, None, 1e-6)
        C.gemm_bf16(hb, wqkv, qkv, False, False, None, 1.0, False, st, None)
        C.rmsnorm_fwd(xb, ln, hb, None, 1e-6)
        C.gemm_bf16(hb, wgu, gu, False, False, None, 1.0, False, st, None)
        C.swiglu_fwd(gu, act)

    def out_old():
        C.gemm_bf16(a, wo, xb2, False, False, None, 1.0, False, st, xb)
        C.gemm_bf16(act, wd, xb2, False, False, None, 1.0, False, st, xb)
    in_shapes, out_shapes = [(T, old.qkv_dim, W), (T, 2 * Fo, W)], [(T, W, H * D), (T, W, Fo)]
    for role in ("prompt input projections", "prompt scan input projections"):
        add(role, "old", in_old, *gemms(*in_shapes))
    for role in ("prompt output projections", "prompt scan output projections"):
        add(role, "old", out_old, *gemms(*out_shapes))
    kc, vc = R(n_seq * nb, G, 16, D), R(n_seq * nb, G, 16, E)
    tables = torch.randperm(n_seq * nb, device=dev).int().view(n_seq, nb).contiguous()
    flat, where = host_batch([(i, 0, np.zeros(prompt, np.int32)) for i in range(n_seq)], [sc.conv], 1, [m.chunk])
    _, sb = split_batch(torch.from_numpy(flat).to(dev), where, tables)
    rows = sb.pages.shape[0] * 16
    keys, values = Z(rows * G * D), Z(rows * G * E)
    uq, kc2, vc2 = R(T, m.u_dim), torch.zeros_like(kc), torch.zeros_like(vc)   # the op works in place: attention gets inputs of its own
    C.qk_norm_rope(uq, qn, kn, 1e-5, m.dim, cos, sin, None, None, sb.rows, None, tables, kc2, vc2, st)
    add("prompt position op", "new", lambda: C.qk_norm_rope(u, qn, kn, 1e-5, m.dim, cos, sin, ss[4], ss[5], sb.rows, None, tables, kc, vc, st), 0.0,
        4.0 * T * (H + G) * D + 4.0 * T * G * E)
    pos, slots, cs = torch.arange(T, device=dev, dtype=torch.int32) % prompt, torch.arange(T, device=dev, dtype=torch.int32), torch.rand(maxlen, D // 2, device=dev)

    def rope():
        C.rope_inplace(qkv, pos, cs, cs, H + G, D, False)
        C.kv_cache_write(qkv, slots, kc, vc, H, G, D, st, 0)
    add("prompt position op", "old", rope, 0.0, 4.0 * T * (H + G) * D + 8.0 * T * G * D)
    pairs_n = n_seq * sum(i % m.chunk + 1 for i in range(prompt))
    pairs_o = n_seq * prompt * (prompt + 1) / 2
    add("prompt attention", "new", lambda: C.chunk_attn_prefill(uq, kc2, vc2, sb.tiles, sb.pages, keys, values, tables, m.scale, m.softcap, m.chunk, cat[:, :m.out_dim], st),
        2.0 * pairs_n * H * (D + E), 0.0)
    lse, tiles = torch.empty(H, T, device=dev), _tiles([prompt] * n_seq)
    add("prompt attention", "old", lambda: C.attn_varlen_fwd(qkv, a, lse, tiles, H, G, D, 0.1, st), 4.0 * pairs_o * H * D, 0.0)
    n_slots = max(n_seq, B)
    ring, state = torch.zeros(n_slots, sc.conv, sc.inner_p, device=dev, dtype=bf), torch.zeros(n_slots, sc.inner_p, n_st, device=dev)
    xc, code, r = R(T, sc.inner_p), R(T, C.scan_code_pitch(sc.dt_rank))[:, :sc.rank_p], torch.randn(T, 2 * n_st, device=dev)
    add("prompt convolution", "new", lambda: C.conv_silu(su, conv, conv_b, ring, sb.rows, sb.ring_rows[sc.conv], None, xc, st), 0.0, 4.0 * T * sc.inner_p)
    add("prompt narrow projection", "new", lambda: C.gemm_split_store(xc, wx, code, r, st), *gemms((T, wx.shape[0], sc.inner_p)))
    add("prompt scan", "new", lambda: C.selective_scan(xc, code, r, su[:, sc.inner_p:], wdt, sc.dt_rank, dt_b, A, skip, state, sb.segs, None, scat[:, :sc.inner_p]), 0.0,
        6.0 * T * sc.inner_p + T * (2.0 * sc.rank_p + 8.0 * n_st))

    # ---------------- decode ----------------
    nbd = (ctx + 15) // 16 + 1
    dk, dv = R(B * nbd, G, 16, D), R(B * nbd, G, 16, E)
    dtab = torch.randperm(B * nbd, device=dev).int().view(B, nbd).contiguous()
    lens = torch.full((B,), ctx, device=dev, dtype=torch.int32)
    du, dcat, dss, dsu, dscat = pair("decode", B)
    xr, qb, ab, actb, hob, xs = R(B, W), R(B, old.qkv_dim), R(B, H * D), R(B, Fo), Z(B, W), R(B, W)
    ssq, so = torch.full((B,), W << 30, device=dev, dtype=torch.int64), torch.zeros(B, device=dev, dtype=torch.int64)

    def din_old():
        C.gemm_decode(xr, wqkv, qb, None, None, ssq, None, 1e-6, st)
        C.gemm_swiglu(xr, wgu, actb, ssq, 1e-6, st)

    def dout_old():
        C.gemm_decode(ab, wo, hob, None, xs, None, so, 1e-6, st)
        C.gemm_decode(actb, wd, hob, None, xs, None, so, 1e-6, st)
    for role in ("decode input projections", "decode scan input projections"):
        add(role, "old", din_old, *gemms((B, old.qkv_dim, W), (B, 2 * Fo, W)))
    for role in ("decode output projections", "decode scan output projections"):
        add(role, "old", dout_old, *gemms((B, W, H * D), (B, W, Fo), extra=8.0 * B * W))
    n_sm = torch.cuda.get_device_properties(0).multi_processor_count
    part = (torch.empty(B * 8 * H * max(D, E) * 2, device=dev), torch.empty(B * 8 * H * 16, device=dev), torch.zeros(B * H, device=dev, dtype=torch.int32))
    seen = (ctx - 1) % m.chunk + 1
    sp_new = max(1, min(8, 3 * n_sm // (B * G), seen // 128))
    sp_old = max(1, min(8, 3 * n_sm // (B * G), ctx // 256))
    add("decode attention", "new", lambda: C.chunk_attn_decode(du, qn, kn, 1e-5, m.dim, cos, sin, dss[4], dss[5], lens, dtab, dk, dv, m.scale, m.softcap, m.chunk,
                                                               dcat[:, :m.out_dim], sp_new, *part, st), 0.0, 2.0 * B * seen * G * (D + E))
    add("decode attention", "old", lambda: C.paged_decode_attn(qb, dk, dv, dtab, lens, ab, H, G, D, 0.1, sp_old, part[0], part[1], st, part[2]), 0.0,
        4.0 * B * ctx * G * D)
    dxc, dcode, dr = R(B, sc.inner_p), R(B, C.scan_code_pitch(sc.dt_rank))[:, :sc.rank_p], torch.randn(B, 2 * n_st, device=dev)
    add("decode convolution", "new", lambda: C.conv_silu(dsu, conv, conv_b, ring[:B], None, None, lens, dxc, st), 0.0, 2.0 * B * sc.inner_p * (sc.conv + 2))
    add("decode narrow projection", "new", lambda: C.gemm_split_store(dxc, wx, dcode, dr, st), *gemms((B, wx.shape[0], sc.inner_p)))
    add("decode scan", "new", lambda: C.selective_scan(dxc, dcode, dr, dsu[:, sc.inner_p:], wdt, sc.dt_rank, dt_b, A, skip, state[:B], None, lens, dscat[:, :sc.inner_p]), 0.0,
        8.0 * B * sc.inner_p * n_st + 2.0 * sc.inner_p * sc.rank_p + 4.0 * sc.inner_p * n_st + 6.0 * B * sc.inner_p)
    return cases


KERNEL_CASES = {"Dezelorn": dezelorn_cases, "Vazatar": vazatar_cases}


def bench_kernels(new_name: str, old_name: str, T: int, prompt: int, B: int, ctx: int) -> None:
    from ..models.registry import PRESETS

    pk = peaks()
    res: Dict[str, Dict[str, Dict[str, float]]] = {}
    cases = KERNEL_CASES[PRESETS[new_name].architecture](PRESETS[new_name], PRESETS[old_name], T, prompt, B, ctx)
    for role, side, fn, flops, nbytes in cases:
        ms = timeit(fn, iters=10, flush=True)
        bound = max(flops / (pk["bf16_tflops"] * 1e9), nbytes / (pk["hbm_gbs"] * 1e6))  # ms
        res.setdefault(role, {})[side] = {"us": round(ms * 1e3, 1), "of_roofline": round(bound / ms, 3)}
    for role, r in res.items():
        rec = {"bench": "kernel", "pair": f"{new_name}:{old_name}", "shape": f"T={T} prompt={prompt}" if role.startswith("prompt") else f"B={B} ctx={ctx}",
               "role": role, **r}
        if "old" in r:
            rec["distance_ratio"] = round(r["old"]["of_roofline"] / max(1e-9, r["new"]["of_roofline"]), 2)
        out({**rec, "peaks": pk["source"]})


def run(pairs: str, prompt: int = 4096, n_layers: int = 8, kernels: bool = True) -> None:
    for pair in pairs.split(","):
        new, _, old = pair.partition(":")
        for model in (new, old):
            out(bench_prefill(model, prompt, max(1, 16384 // prompt), n_layers))
            torch.cuda.empty_cache()
        for batch, ctx in ((16, 2048), (64, 2048), (256, 1024)):
            for model in (new, old):
                out(bench_decode(model, batch, ctx, n_layers))
                torch.cuda.empty_cache()
        if kernels:
            for B, ctx in ((16, 4096), (128, 2048)):
                bench_kernels(new, old, 16384, prompt, B, ctx)
                torch.cuda.empty_cache()
