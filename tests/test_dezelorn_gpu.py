"""The Dezelorn decoder on the GPU against the plain oracle: each mechanism, whole prompts, portions, decoding, mixed batches,
reused pages and slots, window and page edges, and generation through the scheduler and the command line."""
import functools
import json
import math
import subprocess
import sys

import numpy as np
import pytest
import torch

import dezelorn_oracle as O
import dezelorn_util as U

pytestmark = pytest.mark.gpu

DTYPES = ["float32", "bfloat16"]
TORCH = {"float32": torch.float32, "bfloat16": torch.bfloat16}
TOL = {"float32": 3e-5, "bfloat16": 0.05}       # row-wise rms difference over the rms of all logits


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


def run_pieces(eng, toks, pieces, all_logits=True):
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
    n = 1 if name == "tiny" else 330 if name in ("wide", "many") else 211
    got = run_pieces(engine(name, dtype), U.tokens(name, n), [n])
    assert U.worst_row(got, U.oracle_logits(name, n)) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(U.CONFIGS))
def test_prompt_then_token_by_token(name, dtype):
    n, head = 150, 95
    got = run_pieces(engine(name, dtype), U.tokens(name, n), [head] + [1] * (n - head))
    assert U.worst_row(got, U.oracle_logits(name, n)) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["odd", "mixed", "mha", "wide"])
def test_token_by_token_from_the_start(name, dtype):
    n = 60
    got = run_pieces(engine(name, dtype), U.tokens(name, n), [1] * n)
    assert U.worst_row(got, U.oracle_logits(name, n)) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("pieces", [[2] * 100, [3, 2, 16, 17, 15, 1, 1, 2, 48, 49, 46], [1, 2, 129, 1, 67], [150, 2, 2, 46]])
@pytest.mark.parametrize("name", ["odd", "mixed", "wide"])
def test_portions(name, dtype, pieces):
    got = run_pieces(engine(name, dtype), U.tokens(name, 200), pieces)
    assert U.worst_row(got, U.oracle_logits(name, 200)) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["odd", "mixed"])
def test_long_decoding(name, dtype):
    """Decoding passes over several windows and many pages."""
    n = 300
    got = run_pieces(engine(name, dtype), U.tokens(name, n), [10] + [1] * (n - 10))
    assert U.worst_row(got, U.oracle_logits(name, n)) < TOL[dtype]


@pytest.mark.parametrize("name,n", [("tiny", 3), ("odd", 1), ("odd", 2), ("mixed", 1), ("mha", 4)])
def test_first_tokens(name, n):
    for pieces in ([n], [1] * n):
        for dtype in DTYPES:
            got = run_pieces(engine(name, dtype), U.tokens(name, n), pieces)
            assert U.worst_row(got, U.oracle_logits(name, n)) < TOL[dtype]


def test_portions_do_not_change_rounding():
    """Same kernels, same sums: how a prompt is cut shows only in rounding, also in bf16."""
    eng, toks = engine("odd", "bfloat16"), U.tokens("odd", 200)
    whole = run_pieces(eng, toks, [200])
    for pieces in ([77, 123], [16] * 12 + [8], [199, 1]):
        assert U.worst_row(run_pieces(eng, toks, pieces), whole.double()) < 0.02


def test_prefill_budget_cuts_long_prompts():
    eng = build("odd", "float32", max_prefill_tokens=37)
    got = run_pieces(eng, U.tokens("odd", 200), [150, 50])
    assert U.worst_row(got, U.oracle_logits("odd", 200)) < TOL["float32"]


# ---------------------------------------------------------------- batches, slots and pages
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["odd", "mixed", "many"])
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
        step([(2, 1), (0, 1)])                   # slots 1 and 3 idle
    step([(i, len(seqs[i][1]) - at[i]) for i in range(4)])
    for i, (sid, toks, _) in enumerate(seqs):
        got = torch.cat(outs[i])
        assert U.worst_row(got, U.oracle_logits(name, len(toks), 10 + i)) < TOL[dtype]
        eng.close_sequence(sid)
    eng.check_status()


@pytest.mark.parametrize("dtype", DTYPES)
def test_pages_and_slots_are_reused(dtype):
    """A cache with room for little more than one sequence: pages come back in another order, rings hold old state."""
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


def test_window_releases_pages_while_running():
    eng = build("odd", "bfloat16", num_blocks=12, max_seqs=2)  # 192 tokens of cache, 48 of window
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
@pytest.mark.parametrize("dtype", DTYPES)
def test_embedding_and_dynamic_tanh(dtype):
    C, dt = native(), TORCH[dtype]
    g = torch.Generator().manual_seed(3)
    V, W, T, scale = 50, 136, 37, 7.5
    table, w, b = (torch.randn(*s, generator=g).to(torch.bfloat16) for s in ((V, W), (W,), (W,)))
    alpha = torch.tensor([0.37]).to(torch.bfloat16)
    table[0] *= 1e-3                                     # tanh near zero
    table[1] *= 50                                       # and saturated
    ids = torch.randint(0, V, (T,), generator=g)
    ids[:2] = torch.tensor([0, 1])
    x, h = torch.empty(T, W, device="cuda"), torch.empty(T, W, device="cuda", dtype=dt)
    C.embed_dyt(ids.int().cuda(), table.to(dt).cuda(), scale, x, h, [w.to(dt).cuda(), b.to(dt).cuda(), alpha.to(dt).cuda()])
    e = table.double()[ids] * scale
    assert torch.allclose(x.double().cpu(), e, rtol=1e-6)
    ref = O.dyt(e, alpha.double(), w.double(), b.double())
    assert float((h.double().cpu() - ref).abs().max()) < (2e-6 if dtype == "float32" else 0.03)


def test_tanh_accuracy_in_the_fused_norm():
    """The 32-bit tanh of the epilogues over its whole range, seen through unit weights."""
    C = native()
    z = torch.cat([torch.linspace(-0.3, 0.3, 4001), torch.linspace(-20, 20, 4095), torch.logspace(-8, 2, 4096)])[:12192].reshape(12, 1016)
    one, zero = torch.ones(1016, device="cuda"), torch.zeros(1016, device="cuda")
    x, h = torch.empty(12, 1016, device="cuda"), torch.empty(12, 1016, device="cuda")
    C.embed_dyt(torch.arange(12, dtype=torch.int32, device="cuda"), z.cuda(), 1.0, x, h, [one, zero, torch.ones(1, device="cuda")])
    ref = torch.tanh(z.double())
    assert float(((h.double().cpu() - ref).abs() / ref.abs().clamp(min=1e-30)).max()) < 8e-7


@pytest.mark.parametrize("M,N,K", [(1, 64, 64), (7, 104, 72), (33, 1536, 1536), (200, 256, 512), (300, 192, 136), (1000, 2048, 256)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_sublayer_tail_in_the_gemm(dtype, M, N, K):
    C, dt = native(), TORCH[dtype]
    g = torch.Generator().manual_seed(M)
    a, b = (torch.randn(*s, generator=g).to(torch.bfloat16) for s in ((M, K), (N, K)))
    b = (b.float() * K ** -0.5).to(torch.bfloat16)
    n1 = [torch.randn(N, generator=g).to(torch.bfloat16), torch.randn(N, generator=g).to(torch.bfloat16), torch.tensor([0.7]).to(torch.bfloat16)]
    n2 = [torch.randn(N, generator=g).to(torch.bfloat16), torch.randn(N, generator=g).to(torch.bfloat16), torch.tensor([-0.4]).to(torch.bfloat16)]
    x = torch.randn(M, N, generator=g)
    xd, h, st = x.cuda(), torch.empty(M, N, device="cuda", dtype=dt), torch.zeros(1, dtype=torch.int32, device="cuda")
    C.gemm_dyt(a.to(dt).cuda(), b.to(dt).cuda(), xd, [t.to(dt).cuda() for t in n1], [t.to(dt).cuda() for t in n2], h, st)
    y = a.double() @ b.double().T
    xr = x.double() + O.dyt(y, n1[2].double(), n1[0].double(), n1[1].double())
    hr = O.dyt(xr, n2[2].double(), n2[0].double(), n2[1].double())
    assert int(st.item()) == 0
    assert float((xd.double().cpu() - xr).abs().max()) < 2e-5
    assert float((h.double().cpu() - hr).abs().max()) < (2e-5 if dtype == "float32" else 0.04)


class AttnCase:
    """One mixer's attention with its own cache: tables, pages in shuffled order, q and k given directly."""

    def __init__(self, H, G, D, window, n, dtype, coef=0.5, every=7, taps=1, seed=0):
        g = torch.Generator().manual_seed(seed)
        self.H, self.G, self.D, self.window, self.n, self.dt, self.taps = H, G, D, window, n, TORCH[dtype], taps
        bf = lambda *s: torch.randn(*s, generator=g).to(torch.bfloat16).double()
        self.uq, self.uk, self.gate = bf(n, H, D), bf(n, G, D), bf(n, H * D)
        self.conv = torch.cat([bf(H * D, taps), bf(G * D, taps)]) if taps > 1 else torch.ones(H * D + G * D, 1, dtype=torch.float64)
        self.r1, self.r2 = torch.rand(H, generator=g, dtype=torch.float64), torch.rand(H, generator=g, dtype=torch.float64)
        self.talk = (torch.eye(H) + 0.4 * torch.randn(H, H, generator=g)).to(torch.bfloat16).double()
        self.scale = 1.0 / math.sqrt(D)
        self.coef, self.every = coef, every
        nb = (n + 15) // 16
        perm = torch.randperm(nb + 3, generator=g)[:nb].int()
        self.nblk = nb + 3
        self.tables = torch.zeros(3, nb, dtype=torch.int32)
        self.tables[1] = perm
        self.slot = 1

    def device_inputs(self):
        dev = "cuda"
        dist = torch.arange(min(self.window, self.n), dtype=torch.float64)
        self.bias = (self.r1[:, None] * torch.log1p(self.r2[:, None] * dist) / math.log(2)).float().to(dev)
        temp = O.query_temperature(self.n, self.coef, self.every, torch.float64)
        self.qscale = (temp * self.scale / math.log(2)).float().to(dev)
        u = torch.cat([self.uq.flatten(1), self.uk.flatten(1), self.gate], 1).to(self.dt).to(dev)
        cache = torch.full((self.nblk, self.G, 16, self.D), 3.0, device=dev, dtype=self.dt)  # stale values everywhere
        ring = torch.full((3, self.taps, (self.H + self.G) * self.D), -2.0, device=dev, dtype=self.dt)
        return u, cache, ring, self.conv.t().contiguous().to(self.dt).to(dev), self.talk.to(self.dt).to(dev), self.tables.to(dev)

    def oracle(self):
        """Output [n, H * D] (q and k rounded as the kernels store them)."""
        H, G, D = self.H, self.G, self.D
        q, k = O.short_conv(self.uq.flatten(1), self.conv[:H * D]), O.short_conv(self.uk.flatten(1), self.conv[H * D:])
        if self.dt == torch.bfloat16:
            q, k = q.to(torch.bfloat16).double(), k.to(torch.bfloat16).double()
        q, k = q.view(self.n, H, D), k.view(self.n, G, D)
        a = O.attention_weights(q, k, self.scale, O.query_temperature(self.n, self.coef, self.every, torch.float64), self.r1, self.r2, self.window)
        return O.apply_weights(O.mix_heads(a, self.talk), k).flatten(1) * torch.sigmoid(self.gate)

    def run(self, prompt, plain=False, splits=1):
        """`prompt` tokens in one prompt step, the rest one by one."""
        from async_grpo_nccl_b200.models.listed import host_batch, split_batch

        C = native()
        u, cache, ring, conv, talk, tables = self.device_inputs()
        H, G, D, n = self.H, self.G, self.D, self.n
        qk = (H + G) * D
        st = torch.zeros(1, dtype=torch.int32, device="cuda")
        out = torch.zeros(n, H * D, device="cuda", dtype=self.dt)
        part = (torch.empty(3 * 8 * H * G * D, device="cuda"), torch.empty(3 * 8 * H * 2, device="cuda"), torch.zeros(3, dtype=torch.int32, device="cuda"))
        if prompt:
            flat, where = host_batch([(self.slot, 0, np.arange(prompt))], [self.taps], self.window)
            _, sb = split_batch(torch.from_numpy(flat).cuda(), where, tables)
            q = torch.empty(prompt, H * D, device="cuda", dtype=self.dt)
            C.short_conv(u[:prompt], conv, ring, sb.rows, sb.ring_rows[self.taps], None, tables, q, cache, st)
            o = out[:prompt]
            acc = torch.empty(prompt * H * G * D, device="cuda", dtype=self.dt)
            if plain or self.dt == torch.float32:
                C.window_attn(q, cache, sb.rows, None, tables, self.bias, self.qscale, talk, u[:prompt, qk:], self.window, o, st)
            else:
                keys = torch.empty(sb.pages.shape[0] * 16 * G * D, device="cuda", dtype=self.dt)
                assert C.talk_attn_prefill(q, cache, sb.tiles, sb.pages, keys, tables, self.bias, self.qscale, talk, u[:prompt, qk:], self.window, acc, o, st)
        for t in range(prompt, n):
            lens = torch.tensor([0, t + 1, 0], dtype=torch.int32, device="cuda")
            ub = torch.zeros(3, u.shape[1], device="cuda", dtype=self.dt)
            ub[1] = u[t]
            ob = torch.zeros(3, H * D, device="cuda", dtype=self.dt)
            if plain or self.dt == torch.float32:
                q = torch.empty(3, H * D, device="cuda", dtype=self.dt)
                C.short_conv(ub, conv, ring, None, None, lens, tables, q, cache, st)
                C.window_attn(q, cache, None, lens, tables, self.bias, self.qscale, talk, ub[:, qk:], self.window, ob, st)
            else:
                C.talk_attn_decode(ub, conv, ring, cache, lens, tables, self.bias, self.qscale, talk, ub[:, qk:], self.window, ob, splits, *part, st)
            out[t] = ob[1]
        assert int(st.item()) == 0
        return out


def close(got, ref, dtype):
    """Largest element error relative to the largest reference value of the row."""
    err = (got.double().cpu() - ref).abs().max(-1).values / ref.abs().max(-1).values.clamp(min=1e-6)
    assert float(err.max()) < (1e-5 if dtype == "float32" else 0.03), (float(err.max()), int(err.argmax()))


SHAPES = [(1, 1, 64, 1000), (4, 2, 64, 100), (6, 2, 128, 37), (12, 2, 128, 300), (8, 8, 64, 70), (3, 3, 128, 129), (20, 4, 64, 16), (28, 4, 128, 200),
          (16, 1, 128, 64), (40, 8, 64, 1)]


@pytest.mark.parametrize("H,G,D,window", SHAPES)
def test_attention_prompt(H, G, D, window):
    c = AttnCase(H, G, D, window, 283, "bfloat16", taps=4)
    ref = c.oracle()
    close(c.run(283), ref, "bfloat16")
    close(c.run(283, plain=True), ref, "bfloat16")


@pytest.mark.parametrize("H,G,D,window", SHAPES)
def test_attention_decode(H, G, D, window):
    c = AttnCase(H, G, D, window, 283, "bfloat16", taps=3)
    ref = c.oracle()
    for splits, prompt in ((1, 270), (3, 262), (8, 275)):
        close(c.run(prompt, splits=splits)[prompt:], ref[prompt:], "bfloat16")
    close(c.run(0, splits=2)[:40], ref[:40], "bfloat16") if window == 37 else None


@pytest.mark.parametrize("H,G,D,window", [(4, 2, 72, 50), (2, 1, 256, 33), (5, 5, 40, 90)])
def test_attention_32_bit(H, G, D, window):
    c = AttnCase(H, G, D, window, 120, "float32", taps=5)
    ref = c.oracle()
    close(c.run(120), ref, "float32")
    close(c.run(90), ref, "float32")


@pytest.mark.parametrize("window", [1, 16, 17, 128, 129, 200])
@pytest.mark.parametrize("dtype", DTYPES)
def test_one_key_stands_out(dtype, window):
    """A query that agrees strongly with one key: the key dominates when it is visible and must have no trace when it is
    one token outside; keys just inside, just outside, at page borders, at the start and at the query itself."""
    H, G, D, n = 4, 2, 64, 300
    places = [(299, 299 - d) for d in (0, 1, 15, 16, window - 1, window, window + 1) if d <= 299]
    places += [(q, q - window + e) for q in (255, 256, 271) for e in (0, 1) if 0 <= q - window + e <= q]
    for qi, kj in places:
        c = AttnCase(H, G, D, window, n, dtype, coef=0.0)
        c.r1 *= 0.1
        mark = torch.randn(D, generator=torch.Generator().manual_seed(9)).to(torch.bfloat16).double()
        c.uk[kj] = 4 * mark
        c.uq[qi] = 4 * mark
        ref = c.oracle()
        for prompt in (n, qi):
            got = c.run(prompt, splits=2)
            close(got[qi:qi + 1], ref[qi:qi + 1], dtype)
            if dtype == "float32" and prompt == qi:
                break


def test_idle_rows_and_bad_pages():
    """Idle decode rows are skipped; a page index outside the cache is reported, not followed."""
    c = AttnCase(4, 2, 64, 50, 40, "bfloat16")
    c.tables[1, 1] = 10 ** 6
    with pytest.raises(AssertionError):
        c.run(40)


# ---------------------------------------------------------------- generation
def generate(name, dtype, prompts, n_new, **kw):
    req = {k: kw.pop(k) for k in ("n", "seed", "temperature", "ignore_eos") if k in kw}
    eng = build(name, dtype, **kw)
    for i, p in enumerate(prompts):
        eng.add_request(i, p, max_new_tokens=n_new, **{"temperature": 0.0, "ignore_eos": True, **req})
    out = eng.run_until_done()
    eng.check_status()
    return eng, sorted(out, key=lambda f: (f.request_id, f.child))


@pytest.mark.parametrize("dtype,graph", [("float32", False), ("float32", True), ("bfloat16", True)])
def test_greedy_generation_matches_the_oracle(dtype, graph):
    lens = [5, 70, 33, 1, 48]
    prompts = [U.tokens("odd", n, seed=20 + i) for i, n in enumerate(lens)]
    _, out = generate("odd", dtype, prompts, 24, use_cuda_graph=graph, max_seqs=4, max_prefill_tokens=40)
    assert len(out) == 5
    checked = 0
    for f, p in zip(out, prompts):
        ids, margins = U.oracle_greedy("odd", p, 24)
        sure = next((i for i, m in enumerate(margins) if m < (1e-3 if dtype == "float32" else 0.2)), 24)  # before the first near-tie
        assert f.output_ids[:sure].tolist() == ids[:sure]
        checked += sure
    assert checked >= (5 * 24 if dtype == "float32" else 3)


def test_samples_of_a_prompt_share_it():
    """n samples start from one prefill: pages are shared, the partial page and the rings are copied."""
    p = U.tokens("odd", 37, seed=31)
    _, one = generate("odd", "float32", [p], 20, temperature=1.0, seed=5, n=1)
    eng, many = generate("odd", "float32", [p], 20, temperature=1.0, seed=5, n=4)
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
        eng.add_request(i, p, n=6, max_new_tokens=40, temperature=0.0, ignore_eos=True,
                        forced_new_tokens=[1 + (5 * i + 7 * c) % 40 for c in range(6)])
    out = eng.run_until_done()
    eng.check_status()
    assert len(out) == 36
    ref = {i: U.oracle_greedy("odd", p, 40)[0] for i, p in enumerate(prompts)}
    for f in out:
        n = len(f.output_ids)
        assert f.output_ids[:n - 1].tolist() == ref[f.request_id][:n - 1]


def test_compaction_moves_rings():
    prompts = [U.tokens("mixed", 6, seed=60 + i) for i in range(40)]
    eng = build("mixed", "bfloat16", max_seqs=64, num_blocks=400)
    for i, p in enumerate(prompts):
        eng.add_request(i, p, max_new_tokens=30, temperature=0.0, ignore_eos=True, forced_new_tokens=[3 if i < 30 else 30])
    out = {f.request_id: f for f in eng.run_until_done()}
    assert eng.n_compactions >= 1
    _, alone = generate("mixed", "bfloat16", prompts[30:32], 30, max_seqs=64, num_blocks=400)
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
    want = [float(lp[i, t]) for i, t in enumerate(ids[:stop + 1])]
    assert np.allclose(f.output_logprobs, want, atol=1e-3)


def test_weight_update_refreshes_tables():
    eng = build("odd", "float32")
    toks = U.tokens("odd", 60)
    before = run_pieces(eng, toks, [60])
    for i in range(3):
        eng.dec.w(f"layers.{i}.r1").mul_(3.0)
    eng.update_weights_done()
    w = {k: v * 3 if k.endswith("r1") else v for k, v in U.weights("odd").items()}
    after = run_pieces(eng, toks, [60])
    assert U.worst_row(after, O.forward(U.CONFIGS["odd"], w, toks)) < TOL["float32"] and U.rel_rms(after, before) > 0.01


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
    ref = O.forward(U.CONFIGS["odd"], U.weights("odd"), p[:23])[[0, 19, 22]]
    assert U.worst_row(z, ref) < TOL["float32"]
