"""The Vazatar decoder on the GPU against the plain oracle: each mechanism, whole prompts, portions, decoding, mixed batches, reused
pages, slots and states, chunk and page edges, and generation through the scheduler and the command line."""
import functools
import json
import math
import subprocess
import sys

import numpy as np
import pytest
import torch

import vazatar_oracle as O
import vazatar_util as U

pytestmark = pytest.mark.gpu

DTYPES = ["float32", "bfloat16"]
TORCH = {"float32": torch.float32, "bfloat16": torch.bfloat16}
TOL = {"float32": 1e-4, "bfloat16": 0.08}       # row-wise rms difference over the rms of all logits


def native():
    from async_grpo_nccl_b200.ops import native as _n

    return _n()


def build(name, dtype, **kw):
    from async_grpo_nccl_b200.models.registry import build_engine, config_from_dict, make_layout

    cfg = config_from_dict(U.CONFIGS[name])
    layout = make_layout(cfg)
    flat = torch.zeros(layout.total)
    w = U.weights(name)
    for k, dst in layout.hf_items(flat):
        dst.copy_(w[k].float().reshape(dst.shape))
    args = dict(max_seqs=8, max_model_len=640, num_blocks=160)
    args.update(kw)
    return build_engine(cfg, layout, flat.to(TORCH[dtype]).cuda(), **args)


@functools.lru_cache(maxsize=None)
def engine(name, dtype):
    return build(name, dtype)


def run_pieces(eng, toks, pieces):
    """Feeds one sequence in pieces; logits of every token."""
    sid = eng.open_sequence()
    out, a = [], 0
    for n in pieces:
        out.append(eng.extend([(sid, toks[a:a + n], list(range(n)))]).cpu())
        a += n
    assert a == len(toks)
    eng.close_sequence(sid)
    eng.check_status()
    return torch.cat(out)


# ---------------------------------------------------------------- whole prompts, portions, decoding
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(U.CONFIGS))
def test_whole_prompt(name, dtype):
    n = 1 if name == "tiny" else 330 if name in ("wide", "chunks") else 211
    got = run_pieces(engine(name, dtype), U.tokens(name, n), [n])
    assert U.worst_row(got, U.oracle_logits(name, n)) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(U.CONFIGS))
def test_prompt_then_token_by_token(name, dtype):
    n, head = 150, 95
    got = run_pieces(engine(name, dtype), U.tokens(name, n), [head] + [1] * (n - head))
    assert U.worst_row(got, U.oracle_logits(name, n)) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["odd", "scans", "chunks", "wide", "plain"])
def test_token_by_token_from_the_start(name, dtype):
    n = 60
    got = run_pieces(engine(name, dtype), U.tokens(name, n), [1] * n)
    assert U.worst_row(got, U.oracle_logits(name, n)) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("pieces", [[2] * 100, [3, 2, 16, 17, 15, 1, 1, 2, 48, 49, 46], [1, 2, 129, 1, 67], [150, 2, 2, 46]])
@pytest.mark.parametrize("name", ["odd", "scans", "chunks", "wide", "big"])
def test_portions(name, dtype, pieces):
    got = run_pieces(engine(name, dtype), U.tokens(name, 200), pieces)
    assert U.worst_row(got, U.oracle_logits(name, 200)) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["odd", "group"])
def test_long_decoding(name, dtype):
    """Decoding passes over several chunks and many pages."""
    n = 300
    got = run_pieces(engine(name, dtype), U.tokens(name, n), [10] + [1] * (n - 10))
    assert U.worst_row(got, U.oracle_logits(name, n)) < TOL[dtype]


@pytest.mark.parametrize("name,n", [("tiny", 3), ("odd", 1), ("odd", 2), ("scans", 1), ("chunks", 4), ("scans", 7)])
def test_first_tokens(name, n):
    for pieces in ([n], [1] * n):
        for dtype in DTYPES:
            got = run_pieces(engine(name, dtype), U.tokens(name, n), pieces)
            assert U.worst_row(got, U.oracle_logits(name, n)) < TOL[dtype]


@pytest.mark.parametrize("name", ["odd", "wide"])
def test_portions_do_not_change_rounding(name):
    eng, toks = engine(name, "bfloat16"), U.tokens(name, 200)
    whole = run_pieces(eng, toks, [200])
    for pieces in ([77, 123], [16] * 12 + [8], [199, 1]):
        assert U.worst_row(run_pieces(eng, toks, pieces), whole.double()) < 0.04


def test_prefill_budget_cuts_long_prompts():
    eng = build("odd", "float32", max_prefill_tokens=37)
    got = run_pieces(eng, U.tokens("odd", 200), [150, 50])
    assert U.worst_row(got, U.oracle_logits("odd", 200)) < TOL["float32"]


# ---------------------------------------------------------------- batches, slots, pages, states
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["odd", "scans", "group", "wide"])
def test_unequal_requests_in_one_step(name, dtype):
    eng = engine(name, dtype)
    lens = [1, 40, 97, 3]
    seqs = [(eng.open_sequence(), U.tokens(name, n + 12, seed=10 + i), n) for i, n in enumerate(lens)]
    outs = [[] for _ in lens]
    at = [0] * len(lens)

    def step(counts):
        entries = [(seqs[i][0], seqs[i][1][at[i]:at[i] + c], list(range(c))) for i, c in counts]
        z = eng.extend(entries).cpu()
        o = 0
        for i, c in counts:
            outs[i].append(z[o:o + c])
            at[i] += c
            o += c

    step([(0, 1), (2, 50)])
    step([(2, 47), (1, 40), (0, 1)])            # a decode row and two prompts, out of order
    step([(3, 3), (0, 1), (1, 1), (2, 1)])
    for _ in range(5):
        step([(2, 1), (0, 1)])                   # slots 1 and 3 idle: their states must stay as they are
    step([(i, len(seqs[i][1]) - at[i]) for i in range(4)])
    for i, (sid, toks, _) in enumerate(seqs):
        assert U.worst_row(torch.cat(outs[i]), U.oracle_logits(name, len(toks), 10 + i)) < TOL[dtype]
        eng.close_sequence(sid)
    eng.check_status()


@pytest.mark.parametrize("dtype", DTYPES)
def test_pages_slots_and_states_are_reused(dtype):
    """A cache with room for little more than one sequence: pages come back in another order, rings and states hold old values."""
    eng = build("odd", dtype, num_blocks=16, max_seqs=2)
    free = eng.sched.num_free_blocks
    for r in range(4):
        n = [130, 200, 61, 180][r]
        other = eng.open_sequence()
        eng.extend([(other, U.tokens("odd", 20, seed=50 + r), [])])
        got = run_pieces(eng, U.tokens("odd", n, seed=r), [40] * (n // 40) + [1] * (n % 40))
        assert U.worst_row(got, U.oracle_logits("odd", n, r)) < TOL[dtype]
        eng.close_sequence(other)
    assert eng.sched.num_free_blocks == free


def test_passed_chunks_release_pages_while_running():
    eng = build("odd", "bfloat16", num_blocks=12, max_seqs=2)  # 192 tokens of cache, chunks of 48
    n = 400
    got = run_pieces(eng, U.tokens("odd", n), [60] * 5 + [1] * 100)
    assert U.worst_row(got, U.oracle_logits("odd", n)) < TOL["bfloat16"]


def test_cache_overflow_is_an_error_and_leaves_the_sequence_usable():
    eng = build("odd", "float32", num_blocks=8, max_seqs=2)
    sid = eng.open_sequence()
    toks = U.tokens("odd", 200)
    eng.extend([(sid, toks[:50], [])])
    with pytest.raises(RuntimeError):
        eng.extend([(sid, toks[50:200], [])])
    z = eng.extend([(sid, toks[50:60], list(range(10)))])
    assert U.worst_row(z, U.oracle_logits("odd", 200)[50:60]) < TOL["float32"]


# ---------------------------------------------------------------- mechanisms alone
def rnd(g, *shape, std=1.0):
    return (torch.randn(*shape, generator=g) * std).to(torch.bfloat16).double()


def dev(t, dt=torch.bfloat16):
    return t.to(dt).cuda().contiguous()


def from_fixed(ss):
    return ss.double().cpu() / 2 ** 30


def close(got, ref, tol):
    """Largest element error relative to the largest reference value of its row."""
    err = (got.double().cpu() - ref).abs().max(-1).values / ref.abs().max(-1).values.clamp(min=1e-6)
    assert float(err.max()) < tol, (float(err.max()), int(err.argmax()))


@pytest.mark.parametrize("dtype", DTYPES)
def test_embedding_and_norms(dtype):
    C, dt, g = native(), TORCH[dtype], torch.Generator().manual_seed(3)
    V, W, T, width = 50, 136, 37, 131
    table, w1, w2 = rnd(g, V, W), rnd(g, W), rnd(g, W)
    table[:, width:] = 0
    table[0] *= 2 ** -10                                 # eps decides
    ids = torch.randint(0, V, (T,), generator=g)
    ids[0] = 0
    x = torch.empty(T, W, device="cuda")
    copy, h1, h2 = (torch.empty(T, 2 * W, device="cuda", dtype=dt)[:, W:] for _ in range(3))
    ss = torch.full((4, 64), 7, dtype=torch.int64, device="cuda")
    C.embed_norm(ids.int().cuda(), dev(table, dt), 7.5, x, copy, h1, dev(w1, dt), h2, dev(w2, dt), ss)
    e = table[ids] * 7.5
    assert torch.allclose(x.double().cpu(), e, rtol=1e-6)
    tol = 1e-6 if dtype == "float32" else 5e-3
    close(copy, e, tol)
    close(h1, e * (1 + w1), tol)
    close(h2, e * (1 + w2), tol)
    assert torch.allclose(from_fixed(ss[0, :T]), (e * e).sum(-1), rtol=1e-5, atol=1e-8)
    assert int(ss[1:, :T].abs().sum()) == 0 and int((ss[:, T:] != 7).sum()) == 0
    y1, y2 = torch.empty(T, W, device="cuda", dtype=dt), torch.empty(T, W, device="cuda", dtype=dt)
    C.rms_rows(x, 1e-3, width, y1, dev(w1, dt), y2, dev(w2, dt))
    for y, w in ((y1, w1), (y2, w2)):
        close(y[:, :width], O.norm_zero_centred(e[:, :width], w[:width], 1e-3), tol)


# M, n1, n2, K: split-K and persistent kernels, a second product that starts off the tile grid, widths off the 64 grid
PROJ = [(1, 64, 64, 512), (7, 192, 40, 520), (100, 576, 1032, 640), (200, 320, 72, 1024), (5, 128, 96, 72), (300, 192, 200, 136), (1000, 2048, 264, 256),
        (140, 256, 0, 192), (33, 1536, 0, 768)]


@pytest.mark.parametrize("M,n1,n2,K", PROJ)
def test_parallel_projection(M, n1, n2, K):
    C, g = native(), torch.Generator().manual_seed(M)
    width, eps = K - 3, 1e-4
    h, w = rnd(g, M, 2 * K), rnd(g, n1 + n2, K, std=K ** -0.5)
    x2 = torch.rand(M, generator=g, dtype=torch.float64) * K
    ss = (x2 * 2 ** 30).round().long().cuda()
    u = torch.full((M, n1), 9.0, device="cuda", dtype=torch.bfloat16)
    big = torch.full((M, 64 + n2 + 8), 9.0, device="cuda", dtype=torch.bfloat16)
    act = big[:, 64:64 + n2] if n2 else None
    sq, sk, st = (torch.zeros(M, dtype=torch.int64, device="cuda") for _ in range(2)), None, torch.zeros(1, dtype=torch.int32, device="cuda")
    sq, sk = sq
    q_end = n1 // 2 // 64 * 64
    k_end = min(n1, q_end + 64)
    C.gemm_parallel_proj(dev(h), dev(w), u, act, ss, width, eps, sq, sk, q_end, k_end, st)
    rs = 1 / torch.sqrt(x2 / width + eps)
    p1, p2 = rs[:, None] * (h[:, :K] @ w[:n1].T), rs[:, None] * (h[:, K:] @ w[n1:].T)
    assert int(st.item()) == 0
    close(u, p1, 5e-3)
    assert torch.allclose(from_fixed(sq), (p1[:, :q_end] ** 2).sum(-1), rtol=1e-4, atol=1e-6)
    assert torch.allclose(from_fixed(sk), (p1[:, q_end:k_end] ** 2).sum(-1), rtol=1e-4, atol=1e-6)
    if n2:
        close(act, torch.relu(p2) ** 2, 5e-3)
        assert float(big[:, :64].min()) == 9.0 and float(big[:, 64 + n2:].min()) == 9.0
    u2 = torch.empty_like(u)
    C.gemm_parallel_proj(dev(h), dev(w), u2, act, None, width, eps, None, None, 0, 0, st)
    close(u2, h[:, :K] @ w[:n1].T, 5e-3)


@pytest.mark.parametrize("M,N,K", [(1, 64, 64), (7, 104, 72), (33, 1536, 1600), (200, 256, 512), (300, 192, 136), (1000, 2048, 264)])
@pytest.mark.parametrize("accumulate", [True, False])
def test_residual_gemm(M, N, K, accumulate):
    C, g = native(), torch.Generator().manual_seed(M)
    a, w, w1, w2 = rnd(g, M, K), rnd(g, N, K, std=K ** -0.5), rnd(g, N), rnd(g, N)
    x = torch.randn(M, N, generator=g)
    st = torch.zeros(1, dtype=torch.int32, device="cuda")
    ref = a @ w.T + (x.double() if accumulate else 0)
    for first_weight in (w1, None):
        xd, h = x.cuda(), torch.empty(M, 2 * N, device="cuda", dtype=torch.bfloat16)
        ss = torch.zeros(M, dtype=torch.int64, device="cuda")
        C.gemm_residual(dev(a), dev(w), xd, accumulate, h[:, :N], None if first_weight is None else dev(w1), h[:, N:], dev(w2), ss, st)
        assert int(st.item()) == 0 and float((xd.double().cpu() - ref).abs().max()) < 2e-5
        close(h[:, :N], ref * (1 + w1) if first_weight is not None else ref, 5e-3)
        close(h[:, N:], ref * (1 + w2), 5e-3)
        assert torch.allclose(from_fixed(ss), (ref ** 2).sum(-1), rtol=1e-5, atol=1e-6)
    xd = x.cuda()
    C.gemm_residual(dev(a), dev(w), xd, accumulate, None, None, None, None, None, st)
    assert float((xd.double().cpu() - ref).abs().max()) < 2e-5


@pytest.mark.parametrize("M,n1,n2,K", [(3, 16, 8, 64), (100, 96, 32, 640), (200, 112, 64, 512), (300, 32, 128, 200)])
def test_gemm_with_two_kinds_of_output(M, n1, n2, K):
    C, g = native(), torch.Generator().manual_seed(M)
    a, w = rnd(g, M, K), rnd(g, n1 + n2, K, std=K ** -0.5)
    d16, d32 = torch.empty(M, n1 + 8, device="cuda", dtype=torch.bfloat16)[:, :n1], torch.empty(M, n2, device="cuda")
    st = torch.zeros(1, dtype=torch.int32, device="cuda")
    C.gemm_split_store(dev(a), dev(w), d16, d32, st)
    y = a @ w.T
    assert int(st.item()) == 0
    close(d16, y[:, :n1], 5e-3)
    close(d32, y[:, n1:], 1e-5)


def test_gemm_32_bit_on_its_way_out():
    C, g = native(), torch.Generator().manual_seed(4)
    a, b, d = torch.randn(70, 130, generator=g), torch.randn(90, 130, generator=g), torch.randn(70, 90, generator=g)
    y = a.double() @ b.double().T
    for kw, ref in (({}, y), ({"relu2": True}, torch.relu(y) ** 2), ({"softcap": 5.0}, O.softcap(y, 5.0)), ({"accumulate": True}, d.double() + y)):
        out = d.cuda()
        C.gemm_f32(a.cuda(), b.cuda(), out, **kw)
        close(out, ref, 2e-6)
    z = (y.float() * 30).cuda()
    C.softcap_rows(z, 25.0)
    close(z, O.softcap(y * 30, 25.0), 1e-6)


class AttnCase:
    """One mixer's attention with its own cache: pages in shuffled order, projections given directly."""

    def __init__(self, H, G, D, E, chunk, n, dtype, rot=None, cap=20.0, dim=None, seed=0, gain=1.0):
        g = torch.Generator().manual_seed(seed)
        self.H, self.G, self.D, self.E, self.chunk, self.n, self.dt, self.cap = H, G, D, E, chunk, n, TORCH[dtype], cap
        self.dim = dim or D                              # true head size, the rest is padding
        self.rot = self.dim // 2 * 2 if rot is None else rot
        self.q, self.k, self.v = rnd(g, n, H, D), rnd(g, n, G, D), rnd(g, n, G, E)
        self.qn, self.kn = 1.2 + 0.3 * rnd(g, H, D), 1.2 + 0.3 * rnd(g, G, D)
        self.qn, self.kn = self.qn.to(torch.bfloat16).double(), self.kn.to(torch.bfloat16).double()
        for t in (self.q, self.k, self.qn, self.kn):
            t[..., self.dim:] = 0
        self.scale, self.eps = gain / math.sqrt(self.dim), 1e-4
        self.freqs = O.frequencies(self.rot, 300.0, U.SCALING)
        nb = (n + 15) // 16
        self.nblk = nb + 3
        self.tables = torch.zeros(3, nb, dtype=torch.int32)
        self.tables[1] = torch.randperm(nb + 3, generator=g)[:nb].int()
        self.slot = 1

    def oracle(self):
        n, dim = self.n, self.dim
        q = (O.rms(self.q[..., :dim].flatten(1), self.eps) * self.qn[:, :dim].flatten()).view(n, self.H, dim)
        k = (O.rms(self.k[..., :dim].flatten(1), self.eps) * self.kn[:, :dim].flatten()).view(n, self.G, dim)
        q, k = O.rotate(q, self.freqs), O.rotate(k, self.freqs)
        if self.dt == torch.bfloat16:                    # as the kernels keep them
            q, k = q.to(torch.bfloat16).double(), k.to(torch.bfloat16).double()
        return O.attend(q, k, self.v, self.scale, self.cap if self.cap > 0 else 1e30, self.chunk).flatten(1)

    def run(self, prompt, plain=False, splits=1):
        """`prompt` tokens in one prompt step, the rest one by one."""
        from async_grpo_nccl_b200.models.listed import host_batch, split_batch

        C, dt, n, H, G, E = native(), self.dt, self.n, self.H, self.G, self.E
        plain = plain or dt == torch.float32
        u = dev(torch.cat([self.q.flatten(1), self.k.flatten(1), self.v.flatten(1)], 1), dt)
        kc, vc = (torch.full((self.nblk, G, 16, s), 3.0, device="cuda", dtype=dt) for s in (self.D, E))  # stale values everywhere
        tables, qn, kn = self.tables.cuda(), dev(self.qn.flatten(), dt), dev(self.kn.flatten(), dt)
        a = torch.arange(n, dtype=torch.float64)[:, None] * torch.tensor(self.freqs, dtype=torch.float64)
        cos, sin = torch.cos(a).float().cuda(), torch.sin(a).float().cuda()
        sums = [(t.flatten(1).pow(2).sum(-1) * 2 ** 30).round().long().cuda() for t in (self.q, self.k)]
        norm = (qn, kn, self.eps, self.dim, cos, sin)
        st = torch.zeros(1, dtype=torch.int32, device="cuda")
        out = torch.zeros(n, H * E + 64, device="cuda", dtype=dt)[:, :H * E]
        part = (torch.empty(3 * 8 * H * E, device="cuda"), torch.empty(3 * 8 * H * 2, device="cuda"), torch.zeros(3 * H, dtype=torch.int32, device="cuda"))
        if prompt:
            flat, where = host_batch([(self.slot, 0, np.arange(prompt))], [], 1, [self.chunk])
            _, sb = split_batch(torch.from_numpy(flat).cuda(), where, tables)
            s = (None, None) if plain else sums           # given, or found by the kernel
            C.qk_norm_rope(u[:prompt], *norm, *s, sb.rows, None, tables, kc, vc, st)
            if plain:
                C.chunk_attn(u[:prompt], kc, vc, sb.rows, None, tables, self.scale, self.cap, self.chunk, out[:prompt], st)
            else:
                rows = sb.pages.shape[0] * 16 * G
                keys, values = (torch.empty(rows * s, device="cuda", dtype=dt) for s in (self.D, E))
                assert C.chunk_attn_prefill(u[:prompt], kc, vc, sb.tiles, sb.pages, keys, values, tables, self.scale, self.cap, self.chunk, out[:prompt], st)
        for t in range(prompt, n):
            lens = torch.tensor([0, t + 1, 0], dtype=torch.int32, device="cuda")
            ub = torch.zeros(3, u.shape[1], device="cuda", dtype=dt)
            ub[1] = u[t]
            ob = torch.zeros(3, H * E, device="cuda", dtype=dt)
            if plain:
                C.qk_norm_rope(ub, *norm, None, None, None, lens, tables, kc, vc, st)
                C.chunk_attn(ub, kc, vc, None, lens, tables, self.scale, self.cap, self.chunk, ob, st)
            else:
                sq, sk = (torch.zeros(3, dtype=torch.int64, device="cuda") for _ in range(2))
                sq[1], sk[1] = sums[0][t], sums[1][t]
                C.chunk_attn_decode(ub, *norm, sq, sk, lens, tables, kc, vc, self.scale, self.cap, self.chunk, ob, splits, *part, st)
            out[t] = ob[1]
        assert int(st.item()) == 0
        return out


SHAPES = [(1, 1, 64, 64, 1000), (4, 2, 64, 128, 100), (6, 2, 128, 64, 37), (12, 2, 128, 128, 300), (8, 8, 64, 64, 70), (3, 3, 128, 128, 129),
          (20, 1, 64, 128, 16), (28, 4, 128, 128, 200), (18, 1, 128, 64, 64), (34, 2, 64, 64, 1)]


@pytest.mark.parametrize("cap", [20.0, 0.0, 150.0])
@pytest.mark.parametrize("H,G,D,E,chunk", SHAPES)
def test_attention_prompt(H, G, D, E, chunk, cap):
    c = AttnCase(H, G, D, E, chunk, 283, "bfloat16", cap=cap, dim=D - 24, rot=16)
    ref = c.oracle()
    close(c.run(283), ref, 0.03)
    if cap == 20.0:
        close(c.run(283, plain=True), ref, 0.03)


@pytest.mark.parametrize("H,G,D,E,chunk", SHAPES)
def test_attention_decode(H, G, D, E, chunk):
    c = AttnCase(H, G, D, E, chunk, 283, "bfloat16", cap=0.0 if H == 4 else 25.0)
    ref = c.oracle()
    for splits, prompt in ((1, 270), (3, 262), (8, 275)):
        close(c.run(prompt, splits=splits)[prompt:], ref[prompt:], 0.03)
    if chunk == 37:
        close(c.run(0, splits=2)[:80], ref[:80], 0.03)


@pytest.mark.parametrize("gain", [1.0, 30.0, 400.0])
def test_caps_that_bite(gain):
    """Scores well inside the cap (series), around it and far beyond it (saturated), in both kernels."""
    c = AttnCase(4, 2, 64, 64, 200, 220, "bfloat16", cap=8.0, gain=gain)
    ref = c.oracle()
    close(c.run(215, splits=2), ref, 0.03)
    f = AttnCase(4, 2, 64, 64, 200, 220, "float32", cap=8.0, gain=gain)
    close(f.run(215), f.oracle(), 3e-5)


@pytest.mark.parametrize("H,G,D,E,chunk", [(4, 2, 72, 40, 50), (2, 1, 256, 264, 33), (5, 5, 40, 48, 90)])
def test_attention_32_bit(H, G, D, E, chunk):
    for rot in (D // 2 * 2, 14, 0):                      # halves of pairs on and off the vector grid, no rotation at all
        c = AttnCase(H, G, D, E, chunk, 120, "float32", rot=rot)
        ref = c.oracle()
        close(c.run(120), ref, 1e-5)
        close(c.run(90), ref, 1e-5)


@pytest.mark.parametrize("chunk", [1, 16, 17, 128, 129, 200])
@pytest.mark.parametrize("dtype", DTYPES)
def test_one_key_stands_out(dtype, chunk):
    """A query that agrees strongly with one key: the key dominates when it is in the query's chunk and must have no trace when it
    is the last of the chunk before; keys far back, at page borders, at the start and at the query itself."""
    H, G, D, n = 4, 2, 64, 300
    places = [(q, k) for q in (299, 256, 255, 200, 130) for start in [q // chunk * chunk]
              for k in {start - 1, start, min(start + 1, q), (start + q) // 2, start + (q - start) // 16 * 16, q} if 0 <= k <= q]
    for qi, kj in places:
        c = AttnCase(H, G, D, 64, chunk, n, dtype, rot=0, cap=50.0)
        mark = 3 * torch.randn(D, generator=torch.Generator().manual_seed(9)).to(torch.bfloat16).double()
        c.k[kj], c.q[qi] = mark, mark
        c.kn[:], c.qn[:] = 2.0, 2.0
        c.v[kj] *= 4
        ref = c.oracle()
        for prompt in (n, qi):
            close(c.run(prompt, splits=2)[qi:qi + 1], ref[qi:qi + 1], 3e-5 if dtype == "float32" else 0.03)
            if dtype == "float32" and prompt == qi:
                break


def test_a_page_outside_the_cache_is_reported():
    c = AttnCase(4, 2, 64, 64, 50, 40, "bfloat16")
    c.tables[1, 1] = 10 ** 6
    with pytest.raises(AssertionError):
        c.run(40)


class ScanCase:
    """Convolution, narrow projection and scan of several sequences, projections given directly."""

    def __init__(self, C, N, R, taps, dtype, seed=0):
        g = torch.Generator().manual_seed(seed)
        self.C, self.N, self.R, self.taps, self.dt = C, N, R, taps, TORCH[dtype]
        self.conv, self.conv_b = rnd(g, C, taps), rnd(g, C, std=0.3)
        self.wdt, self.dt_b = rnd(g, C, R, std=R ** -0.5), rnd(g, C) - 2
        self.A = -torch.exp(torch.randn(C, N, generator=g).double() * 1.5 - 1)
        self.D = rnd(g, C)
        self.g = g

    def inputs(self, n):
        return rnd(self.g, n, self.C), rnd(self.g, n, self.C), rnd(self.g, n, self.R), rnd(self.g, n, self.N), rnd(self.g, n, self.N)

    def oracle(self, x, z, code, B, Cm):
        xc = O.silu(O.causal_conv(x, self.conv, self.conv_b))
        if self.dt == torch.bfloat16:
            xc = xc.to(torch.bfloat16).double()
        dt = O.softplus(code @ self.wdt.T + self.dt_b)
        y, S = O.selective_scan(xc, dt, self.A, B, Cm, self.D)
        return y * O.silu(z), S

    def run(self, data, steps, plain):
        """data: inputs per slot; steps: lists of (slot, rows) that go through together, single rows of all slots as decode."""
        C, k, dt = native(), self, self.dt
        q = C.scan_states_per_lane(k.N)
        n_st = k.N if plain else 4 * q
        R = k.R if plain else (k.R + 15) // 16 * 16
        A = torch.zeros(k.C, n_st, device="cuda")
        A[:, :k.N] = (self.A if plain else self.A / math.log(2)).float().cuda()
        wdt = torch.zeros(k.C, (k.R + 15) // 16 * 16, device="cuda", dtype=dt)
        wdt[:, :k.R] = dev(k.wdt, dt)
        S = len(data)
        state = torch.full((S, k.C, n_st), 5.0, device="cuda")         # stale
        ring = torch.full((S, k.taps, k.C), 5.0, device="cuda", dtype=dt)
        at, outs = [0] * S, [[] for _ in range(S)]
        for step in steps:
            decode = len(step) == S and all(n == 1 for _, n in step) and all(at)
            parts = [[t[at[s]:at[s] + n] for t in data[s]] for s, n in step]
            x, z, code, B, Cm = (torch.cat(t) for t in zip(*parts))
            T = x.shape[0]
            if plain:
                r = torch.zeros(T, (R + 2 * n_st + 7) // 8 * 8)
                r[:, :R + 2 * k.N] = torch.cat([code, B, Cm], 1)
                given = (r.cuda(),)
            else:   # the code by itself, states in quarters: B, then C of each
                c16, r = torch.zeros(T, C.scan_code_pitch(k.R)), torch.zeros(T, 4, 2, q)
                c16[:, :k.R] = code
                for i in range(k.N):
                    r[:, i // q, 0, i % q], r[:, i // q, 1, i % q] = B[:, i], Cm[:, i]
                given = (dev(c16)[:, :R], r.view(T, 2 * n_st).cuda())
            rows, segs, keep, t0 = [], [], [], 0
            for s, n in step:
                rows += [(s, at[s] + i, t0, 0) for i in range(n)]
                segs.append((t0, n, s, at[s]))
                keep += range(t0 + max(0, n - k.taps), t0 + n)
                t0 += n
            i32 = dict(dtype=torch.int32, device="cuda")
            lens = torch.tensor([p + 1 for p in at], **i32)
            where = (None, None, lens) if decode else (torch.tensor(rows, **i32), torch.tensor(keep, **i32), None)
            u = dev(torch.cat([x, z], 1), dt)
            xc, out = torch.empty(T, k.C, device="cuda", dtype=dt), torch.zeros(T, k.C + 8, device="cuda", dtype=dt)[:, :k.C]
            C.conv_silu(u, dev(k.conv.T, dt), dev(k.conv_b, dt), ring, *where, xc, None)
            scan = C.selective_scan_plain if plain else C.selective_scan
            scan(xc, *given, u[:, k.C:], wdt, k.R, dev(k.dt_b, torch.float32), A, dev(k.D, torch.float32), state,
                 None if decode else torch.tensor(segs, **i32), lens if decode else None, out)
            t0 = 0
            for s, n in step:
                outs[s].append(out[t0:t0 + n])
                at[s] += n
                t0 += n
        return [torch.cat(o) for o in outs], self.unpack(state)

    def unpack(self, state):
        return state[:, :, :self.N].double().cpu()


@pytest.mark.parametrize("C,N,R,taps", [(64, 16, 4, 4), (128, 1, 1, 1), (192, 5, 33, 3), (64, 24, 16, 2), (64, 64, 130, 6), (320, 12, 200, 4)])
@pytest.mark.parametrize("kind", ["float32", "bfloat16", "bfloat16 plain"])
def test_selective_scan(C, N, R, taps, kind):
    dtype, plain = kind.split()[0], kind != "bfloat16"
    c = ScanCase(C, N, R, taps, dtype, seed=N)
    data = [c.inputs(n) for n in (90, 41, 70)]
    want = [c.oracle(*d) for d in data]
    steps = [[(0, 40), (2, 1)], [(1, 33), (0, 2)], [(2, 62), (1, 1), (0, 41)]] + [[(0, 1), (1, 1), (2, 1)]] * 7
    outs, state = c.run(data, steps, plain)
    tol = 3e-5 if dtype == "float32" else 0.01
    for o, (y, S), st in zip(outs, want, state):
        close(o, y, tol)
        assert float((st - S).abs().max() / S.abs().max()) < (1e-5 if dtype == "float32" else 5e-3)


def test_step_sizes_over_the_whole_range():
    """softplus from tiny to large arguments, seen through a state that takes one step from zero."""
    C, c = 64, ScanCase(64, 2, 1, 1, "bfloat16")
    c.dt_b = torch.linspace(-30, 30, C).double().to(torch.bfloat16).double()
    c.wdt[:], c.conv[:], c.conv_b[:] = 0, 0, 1.0
    data = [c.inputs(1)]
    _, state = c.run(data, [[(0, 1)]], False)
    x = float(torch.tensor(O.silu(torch.tensor(1.0))).to(torch.bfloat16))
    got, ref = state[0][:, 0] / (data[0][3][0, 0] * x), O.softplus(c.dt_b)
    assert float((got / ref - 1).abs().max()) < 2e-6


@pytest.mark.parametrize("cap", [0.0, 4.0])
def test_sampling_with_capped_logits(cap):
    """Greedy tokens, log-probabilities and the distribution of samples follow the capped logits."""
    C, g = native(), torch.Generator().manual_seed(2)
    rows, W, V = 64, 128, 37
    h, w = rnd(g, 1, W).expand(rows, W).contiguous(), rnd(g, V, W, std=0.5)
    z = h[0] @ w.T
    z = O.softcap(z, cap) if cap else z
    n = max(int(C.lm_sample_num_groups(V, rows)), int(C.lm_sample_num_groups(V, 1)))
    f, i = torch.empty(4 * n * rows, device="cuda"), torch.empty(n * rows, dtype=torch.int32, device="cuda")
    tok, lp = torch.empty(rows, dtype=torch.int32, device="cuda"), torch.empty(rows, device="cuda")
    seeds = torch.arange(rows, dtype=torch.int64, device="cuda") * 7919
    C.lm_sample(dev(h), dev(w), 0.0, seeds, f, i, tok, lp, None, softcap=cap)
    best = int((h[0] @ w.T).argmax())
    assert set(tok.tolist()) == {best} and abs(float(lp[0]) - float(torch.log_softmax(z, -1)[best])) < 1e-3
    T, counts = 1.5, torch.zeros(V)
    for k in range(40):
        C.lm_sample(dev(h), dev(w), T, seeds + k * 1000003, f, i, tok, lp, None, softcap=cap)
        counts += torch.bincount(tok.cpu().long(), minlength=V)
        assert torch.allclose(lp.double().cpu(), torch.log_softmax(z / T, -1)[tok.cpu().long()], atol=1e-3)
    p = torch.softmax(z / T, -1)
    assert float((counts / counts.sum() - p).abs().sum()) < 0.12


# ---------------------------------------------------------------- generation
def generate(name, dtype, prompts, n_new, **kw):
    req = {k: kw.pop(k) for k in ("n", "seed", "temperature", "ignore_eos") if k in kw}
    eng = build(name, dtype, **kw)
    for i, p in enumerate(prompts):
        eng.add_request(i, p, max_new_tokens=n_new, **{"temperature": 0.0, "ignore_eos": True, **req})
    out = eng.run_until_done()
    eng.check_status()
    return eng, sorted(out, key=lambda f: (f.request_id, f.child))


@pytest.mark.parametrize("name,dtype,graph", [("odd", "float32", False), ("odd", "float32", True), ("odd", "bfloat16", True), ("wide", "bfloat16", True)])
def test_greedy_generation_matches_the_oracle(name, dtype, graph):
    lens = [5, 70, 33, 1, 48]
    prompts = [U.tokens(name, n, seed=20 + i) for i, n in enumerate(lens)]
    _, out = generate(name, dtype, prompts, 24, use_cuda_graph=graph, max_seqs=4, max_prefill_tokens=40)
    assert len(out) == 5
    checked = 0
    for f, p in zip(out, prompts):
        ids, margins = U.oracle_greedy(name, p, 24)
        sure = next((i for i, m in enumerate(margins) if m < (2e-3 if dtype == "float32" else 0.5)), 24)  # before the first near-tie
        assert f.output_ids[:sure].tolist() == ids[:sure]
        checked += sure
    assert checked >= (80 if dtype == "float32" else 5)


def test_a_model_without_attention_needs_no_cache():
    p = U.tokens("scans", 30, seed=33)
    eng, out = generate("scans", "float32", [p], 10, num_blocks=None)
    ids, margins = U.oracle_greedy("scans", p, 10)
    sure = next((i for i, m in enumerate(margins) if m < 2e-3), 10)
    assert not eng.cache and out[0].output_ids[:sure].tolist() == ids[:sure]


def test_samples_of_a_prompt_share_it():
    """n samples start from one prefill: pages are shared, the partial page, the rings and the states are copied."""
    p = U.tokens("odd", 37, seed=31)
    _, one = generate("odd", "float32", [p], 20, temperature=1.0, seed=5, n=1)
    _, many = generate("odd", "float32", [p], 20, temperature=1.0, seed=5, n=4)
    assert many[0].output_ids.tolist() == one[0].output_ids.tolist()
    assert len({tuple(f.output_ids.tolist()) for f in many}) > 1
    _, greedy = generate("odd", "float32", [p], 20, n=3)
    want, _ = U.oracle_greedy("odd", p, 20)
    assert all(f.output_ids.tolist() == want for f in greedy)


def test_generation_with_holes_preemption_and_reuse():
    """More requests than slots, different lengths (slots are compacted), a cache that forces preemption."""
    prompts = [U.tokens("odd", 10 + 7 * i, seed=40 + i) for i in range(6)]
    eng = build("odd", "float32", max_seqs=64, num_blocks=26)
    for i, p in enumerate(prompts):
        eng.add_request(i, p, n=6, max_new_tokens=40, temperature=0.0, ignore_eos=True, forced_new_tokens=[1 + (5 * i + 7 * c) % 40 for c in range(6)])
    out = eng.run_until_done()
    eng.check_status()
    assert len(out) == 36
    ref = {i: U.oracle_greedy("odd", p, 40)[0] for i, p in enumerate(prompts)}
    for f in out:
        n = len(f.output_ids)
        assert f.output_ids[:n - 1].tolist() == ref[f.request_id][:n - 1]


def test_compaction_moves_rings_and_states():
    prompts = [U.tokens("scans", 6, seed=60 + i) for i in range(40)]
    eng = build("scans", "bfloat16", max_seqs=64, num_blocks=400)
    for i, p in enumerate(prompts):
        eng.add_request(i, p, max_new_tokens=30, temperature=0.0, ignore_eos=True, forced_new_tokens=[3 if i < 30 else 30])
    out = {f.request_id: f for f in eng.run_until_done()}
    assert eng.n_compactions >= 1
    _, alone = generate("scans", "bfloat16", prompts[30:32], 30, max_seqs=64, num_blocks=400)
    for a, i in zip(alone, (30, 31)):
        assert out[i].output_ids[:-1].tolist() == a.output_ids[:29].tolist()


def test_eos_and_logprobs():
    p = U.tokens("odd", 20, seed=70)
    ids, _ = U.oracle_greedy("odd", p, 30)
    eos = ids[7]
    eng = build("odd", "float32", eos_token_id=eos)
    eng.enable_logprobs()
    eng.add_request(0, p, max_new_tokens=30, temperature=0.0)
    f = eng.run_until_done()[0]
    stop = ids.index(eos)
    assert f.finish_reason == "stop" and f.output_ids.tolist() == ids[:stop + 1]
    lp = torch.log_softmax(O.forward(U.CONFIGS["odd"], U.weights("odd"), p + ids[:stop])[len(p) - 1:], -1)
    assert np.allclose(f.output_logprobs, [float(lp[i, t]) for i, t in enumerate(ids[:stop + 1])], atol=1e-3)


@pytest.mark.parametrize("dtype", DTYPES)
def test_weight_update_refreshes_tables(dtype):
    eng, toks = build("odd", dtype), U.tokens("odd", 60)
    before = run_pieces(eng, toks, [60])
    for leaf in ("A_log", "conv", "wx"):
        eng.dec.w(f"layers.1.{leaf}").mul_(0.5)
    eng.update_weights_done()
    w = {k: v / 2 if k in ("l1.mix.A_log", "l1.mix.conv", "l1.mix.x") else v for k, v in U.weights("odd").items()}
    after = run_pieces(eng, toks, [60])
    assert U.worst_row(after, O.forward(U.CONFIGS["odd"], w, toks)) < TOL[dtype] and U.rel_rms(after, before) > 0.05


def test_command_lines(tmp_path):
    d = U.save_checkpoint(tmp_path / "model", "odd")
    p = U.tokens("odd", 30, seed=80)
    want, _ = U.oracle_greedy("odd", p, 12)
    r = subprocess.run([sys.executable, "-m", "async_grpo_nccl_b200.generate", "--model", d, "--dtype", "float32", "--prompt-ids",
                        ",".join(map(str, p)), "--max-new-tokens", "12", "--kv-gb", "0.1"], capture_output=True, text=True, timeout=120)
    assert r.returncode == 0, r.stderr[-2000:]
    assert json.loads(r.stdout.strip().splitlines()[-1])["output_token_ids"] == want
    out = tmp_path / "out"
    out.mkdir()
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": p[:20], "want": [0, 19]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": p[20:22], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": p[22:23], "want": [0]}], "end": ["a"]}]
    r = subprocess.run(["bin/trace_run", "--model", d, "--dtype", "float32", "--out", str(out), "--max-tokens", "64"],
                       input="\n".join(map(json.dumps, steps)), capture_output=True, text=True, timeout=120)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"] and not (out / "1.f32").exists()
    z = torch.from_numpy(np.concatenate([np.fromfile(out / f, dtype="<f4") for f in ("0.f32", "2.f32")]).reshape(3, -1))
    assert U.worst_row(z, O.forward(U.CONFIGS["odd"], U.weights("odd"), p[:23])[[0, 19, 22]]) < TOL["float32"]
