"""Small Dezelorn models with random weights for the tests, and their oracle logits."""
import functools
import json

import torch

import dezelorn_oracle as O


def layer(heads, kv, dim, ff, window, conv=4, coef=0.4, every=8, gain=1.0):
    return {"type": "attention",
            "mixer": {"conv": conv, "dim": dim, "heads": heads, "kv_heads": kv, "mask": {"size": window},
                      "q_temp": {"coef": coef, "every": every}, "scale": gain / dim ** 0.5, "vdim": dim},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(vocab, width, layers, scale=3.0):
    return {"architecture": "Dezelorn", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": 1e-6},
            "layers": layers}


CONFIGS = {
    # odd sizes everywhere: padded heads, width and feed-forward
    "odd": config(333, 100, [layer(6, 2, 40, 172, 48, conv=3), layer(6, 2, 40, 172, 48, conv=3), layer(6, 2, 40, 172, 48, conv=3)]),
    # one key head, one tap, layers that differ, a layer without feed-forward, a window of one token
    "mixed": config(200, 64, [layer(4, 1, 64, 96, 17, conv=1, every=3), layer(2, 2, 16, None, 1, conv=4), layer(3, 1, 64, 64, 200, conv=2, every=1)],
                    scale=1.0),
    # every query head has its own keys; six taps
    "mha": config(160, 72, [layer(5, 5, 72, 80, 33, conv=6), layer(5, 5, 72, None, 65, conv=5, coef=0.0)]),
    # four key heads of 128: more value heads than one prompt CTA takes
    "wide": config(300, 256, [layer(8, 4, 128, 256, 150, every=50), layer(8, 4, 128, 512, 40, every=50)]),
    # two row tiles of heads in the decode kernel
    "many": config(256, 128, [layer(20, 4, 96, 128, 300), layer(20, 4, 96, 128, 129)]),
    # one head of one token's size; a window longer than any sequence
    "tiny": config(64, 8, [layer(1, 1, 8, 8, 100000, conv=2)]),
    # heads larger than the tensor-core kernels take
    "big-head": config(128, 96, [layer(3, 1, 136, 64, 50), layer(2, 1, 256, 64, 20)]),
}


def make_weights(cfg, seed=0):
    """Checkpoint-named weights, rounded to bf16, in float64: every mechanism has a visible effect."""
    g = torch.Generator().manual_seed(seed)

    def rnd(*shape, std=1.0, mean=0.0):
        return (torch.randn(*shape, generator=g) * std + mean).to(torch.bfloat16).double()

    W, V = cfg["width"], cfg["vocab"]
    w = {"embed": rnd(V, W, std=0.5), "head": rnd(V, W, std=W ** -0.5)}

    def norm(name):
        w[name] = rnd(W, std=0.2, mean=1.0)
        w[name + ".b"] = rnd(W, std=0.1)
        w[name + ".alpha"] = rnd(1, std=0.1, mean=0.6).reshape(())

    for i, l in enumerate(cfg["layers"]):
        m, n = l["mixer"], f"l{i}."
        H, G, D = m["heads"], m["kv_heads"], m["dim"]
        norm(n + "norm1")
        norm(n + "norm1b")
        for leaf, heads in (("q", H), ("k", G), ("g", H)):
            w[n + "mix." + leaf] = rnd(heads * D, W, std=1.5 * W ** -0.5)
        w[n + "mix.q.conv"] = rnd(H * D, m["conv"], std=0.5)
        w[n + "mix.k.conv"] = rnd(G * D, m["conv"], std=0.5)
        w[n + "mix.q.conv"][:, -1] += 1
        w[n + "mix.k.conv"][:, -1] += 1
        w[n + "mix.r1"] = rnd(H, std=0.6, mean=1.0)
        w[n + "mix.r2"] = rnd(H, std=0.1, mean=0.3).abs()
        w[n + "mix.talk"] = rnd(H, H, std=0.4) + torch.eye(H, dtype=torch.float64)
        w[n + "mix.o"] = rnd(W, H * D, std=(H * D) ** -0.5)
        if l["mlp"] is not None:
            F = l["mlp"]["ff"]
            norm(n + "norm2")
            norm(n + "norm2b")
            w[n + "mlp.gate"], w[n + "mlp.up"], w[n + "mlp.down"] = rnd(F, W, std=W ** -0.5), rnd(F, W, std=W ** -0.5), rnd(W, F, std=F ** -0.5)
    norm("final.norm")
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


def oracle_greedy(name, prompt, n_new, stop=None):
    """Greedy continuation and the margin between the two best logits at every step."""
    ids, margins = list(prompt), []
    for _ in range(n_new):
        top = torch.topk(O.forward(CONFIGS[name], weights(name), ids)[-1], 2)
        margins.append(float(top.values[0] - top.values[1]))
        ids.append(int(top.indices[0]))
        if stop is not None and ids[-1] == stop:
            break
    return ids[len(prompt):], margins


def save_checkpoint(path, name):
    from safetensors.torch import save_file

    path.mkdir(parents=True, exist_ok=True)
    save_file({k: v.to(torch.bfloat16).contiguous() for k, v in weights(name).items()}, str(path / "model.safetensors"))
    (path / "config.json").write_text(json.dumps(CONFIGS[name]))
    return str(path)


def rel_rms(a, b):
    a, b = a.double().cpu(), b.double()
    return float((a - b).pow(2).mean().sqrt() / b.pow(2).mean().sqrt())


def worst_row(a, b):
    """Largest row-wise rms difference relative to the overall rms."""
    a, b = a.double().cpu(), b.double()
    return float((a - b).pow(2).mean(-1).sqrt().max() / b.pow(2).mean().sqrt())
