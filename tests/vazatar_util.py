"""Small Vazatar models with random weights for the tests, and their oracle logits."""
import functools
import json

import torch

import vazatar_oracle as O

SCALING = {"factor": 3.0, "low": 1.0, "high": 5.0, "original": 90}


def attn(heads, kv, dim, chunk, ff, vdim=None, rot=None, cap=20.0, base=500.0, gain=1.0, scaling=None):
    return {"type": "attention",
            "mixer": {"dim": dim, "heads": heads, "kv_heads": kv, "mask": {"size": chunk}, "scale": gain / dim ** 0.5, "softcap": cap,
                      "vdim": dim if vdim is None else vdim,
                      "rot": {"base": base, "dims": dim if rot is None else rot, "scaling": dict(scaling or SCALING)}},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def mamba(inner, state, rank, conv, ff):
    return {"type": "mamba1", "mixer": {"conv": conv, "dt_rank": rank, "inner": inner, "state": state},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(vocab, width, layers, loop=(0, 1, 1), scale=2.0, cap=15.0, eps=1e-5):
    return {"architecture": "Vazatar", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps}, "layers": layers,
            "logit_softcap": cap, "loop": dict(zip(("start", "stop", "times"), loop))}


CONFIGS = {
    # odd sizes everywhere: padded heads, width, channels and states; value heads of another size, a part of a head rotated
    "odd": config(333, 100, [attn(6, 2, 40, 48, 172, vdim=24, rot=32), mamba(72, 5, 3, 3, 60), attn(3, 1, 24, 31, None, vdim=40, rot=6)], (1, 3, 2)),
    # a loop over everything, from the first layer on; layers without feed-forward, one tap, six taps, one state
    "scans": config(200, 64, [mamba(128, 16, 4, 1, None), mamba(32, 1, 1, 6, 96)], (0, 2, 3), scale=1.0, eps=1e-3),
    # attention only: chunks of one token, of a page, around the tile; caps too large for weights without a maximum
    "chunks": config(160, 72, [attn(5, 5, 64, 1, 80), attn(4, 2, 16, 16, None, cap=300.0, rot=2), attn(2, 2, 64, 17, 40), attn(2, 1, 128, 129, 40)], (2, 3, 1)),
    # widths that take the split-K forms, four key heads of 128, long chunks
    "wide": config(300, 512, [attn(8, 4, 128, 150, 520, vdim=128), mamba(576, 24, 32, 4, 512), attn(8, 4, 128, 100000, 512, vdim=64, rot=64)], (1, 2, 2)),
    # more query heads per key head than one row tile holds
    "group": config(256, 128, [attn(20, 1, 128, 70, 128, vdim=64), attn(24, 2, 64, 40, 128, vdim=128)], (1, 2, 1)),
    # heads and states larger than the fast kernels take
    "big": config(128, 96, [attn(3, 1, 136, 50, 64, vdim=200), mamba(64, 70, 40, 2, 64), attn(2, 2, 256, 20, 64, cap=100.0), mamba(96, 40, 17, 4, None)], (1, 3, 2)),
    # one head, one channel block, everything small; a pass count of three
    "tiny": config(64, 8, [attn(1, 1, 2, 5, 8), mamba(8, 2, 1, 2, 8)], (0, 1, 3)),
    # no loop at all, frequencies unscaled
    "plain": {k: v for k, v in config(150, 80, [attn(4, 2, 48, 33, 64, scaling={"factor": 1.0, "low": 1.0, "high": 4.0, "original": 64}),
                                                mamba(80, 12, 5, 4, 64)]).items() if k != "loop"},
}


def make_weights(cfg, seed=0):
    """Checkpoint-named weights, rounded to bf16, in float64: every mechanism has a visible effect, some states fade slowly."""
    g = torch.Generator().manual_seed(seed)

    def rnd(*shape, std=1.0, mean=0.0):
        return (torch.randn(*shape, generator=g) * std + mean).to(torch.bfloat16).double()

    W, V = cfg["width"], cfg["vocab"]
    w = {"embed": rnd(V, W, std=0.5), "head": rnd(V, W, std=4 * W ** -0.5), "final.norm": rnd(W, std=0.2)}
    if "loop" in cfg:
        w["loop.in"] = torch.cat([torch.eye(W, dtype=torch.float64) * 0.7, torch.eye(W, dtype=torch.float64) * 0.4], 1) + rnd(W, 2 * W, std=0.3 * W ** -0.5)
    for i, l in enumerate(cfg["layers"]):
        m, n = l["mixer"], f"l{i}."
        w[n + "norm1"] = rnd(W, std=0.3)
        if l["type"] == "attention":
            H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for leaf, rows in (("q", H * D), ("k", G * D), ("v", G * E)):
                w[n + "mix." + leaf] = rnd(rows, W, std=W ** -0.5)
            w[n + "mix.q.norm"], w[n + "mix.k.norm"] = rnd(H * D, std=0.3, mean=1.3), rnd(G * D, std=0.3, mean=1.3)
            w[n + "mix.o"] = rnd(W, H * E, std=(H * E) ** -0.5)
        else:
            C, N, R = m["inner"], m["state"], m["dt_rank"]
            w[n + "mix.in"] = rnd(2 * C, W, std=W ** -0.5)
            w[n + "mix.conv"], w[n + "mix.conv.b"] = rnd(C, m["conv"], std=0.6), rnd(C, std=0.2)
            w[n + "mix.x"] = rnd(R + 2 * N, C, std=C ** -0.5)
            w[n + "mix.dt"], w[n + "mix.dt.b"] = rnd(C, R, std=R ** -0.5), rnd(C, std=1.0, mean=-1.5)
            w[n + "mix.A_log"], w[n + "mix.D"] = rnd(C, N, std=1.5, mean=-1.0), rnd(C, mean=0.5)
            w[n + "mix.o"] = rnd(W, C, std=C ** -0.5)
        if l["mlp"] is not None:
            F = l["mlp"]["ff"]
            w[n + "norm2"] = rnd(W, std=0.3)
            w[n + "mlp.up"], w[n + "mlp.down"] = rnd(F, W, std=W ** -0.5), rnd(W, F, std=0.7 * F ** -0.5)
    return {k: v.to(torch.bfloat16).double() for k, v in w.items()}


def tokens(name, n, seed=0):
    g = torch.Generator().manual_seed(1000 + seed)
    return torch.randint(0, CONFIGS[name]["vocab"], (n,), generator=g).tolist()


@functools.lru_cache(maxsize=None)
def weights(name):
    return make_weights(CONFIGS[name])


@functools.lru_cache(maxsize=None)
def oracle_logits(name, n, seed=0):
    return O.forward(CONFIGS[name], weights(name), tokens(name, n, seed))


def oracle_greedy(name, prompt, n_new):
    """Greedy continuation and the margin between the two best logits at every step."""
    ids, margins = list(prompt), []
    for _ in range(n_new):
        top = torch.topk(O.forward(CONFIGS[name], weights(name), ids)[-1], 2)
        margins.append(float(top.values[0] - top.values[1]))
        ids.append(int(top.indices[0]))
    return ids[len(prompt):], margins


def save_checkpoint(path, name, **extra):
    from safetensors.torch import save_file

    path.mkdir(parents=True, exist_ok=True)
    save_file({k: v.to(torch.bfloat16).contiguous() for k, v in {**weights(name), **extra}.items()}, str(path / "model.safetensors"))
    (path / "config.json").write_text(json.dumps(CONFIGS[name]))
    return str(path)


def rel_rms(a, b):
    a, b = a.double().cpu(), b.double()
    return float((a - b).pow(2).mean().sqrt() / b.pow(2).mean().sqrt())


def worst_row(a, b):
    """Largest row-wise rms difference relative to the overall rms."""
    a, b = a.double().cpu(), b.double()
    return float((a - b).pow(2).mean(-1).sqrt().max() / b.pow(2).mean().sqrt())
