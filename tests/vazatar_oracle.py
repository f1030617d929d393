"""Plain, slow restatement of the Vazatar decoder in PyTorch: one function per mechanism, straight from the equations.

Nothing here is shared with the product code. Everything runs in the dtype of the weights that are passed in (float64 in
the tests), over whole sequences, with explicit score matrices and a Python loop over tokens for the recurrence.

Notation: T tokens of one sequence at positions 0..T-1. Attention: H query heads, G key heads, query head h reads key head
h // (H // G). Selective scan: C channels, N states per channel.
"""
import math

import torch


def rms(x, eps):
    """x over its root mean square along the last axis, eps added under the root."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_zero_centred(x, w, eps):
    """The stored weight is the deviation from one."""
    return rms(x, eps) * (1 + w)


def silu(x):
    return x * torch.sigmoid(x)


# ---- rotation ----
def frequencies(dims, base, scaling):
    """Angle per position of each rotated pair. Pairs whose wavelength is short against `original` keep their frequency, long ones
    are slowed by `factor`, between the two limits the frequency is interpolated."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        length = 2 * math.pi / f
        if length < scaling["original"] / scaling["high"]:
            out.append(f)
        elif length > scaling["original"] / scaling["low"]:
            out.append(f / scaling["factor"])
        else:
            s = (scaling["original"] / length - scaling["low"]) / (scaling["high"] - scaling["low"])
            out.append((1 - s) * f / scaling["factor"] + s * f)
    return out


def rotate(x, freqs):
    """x [T, heads, D]: dimension i turns with dimension i + dims / 2 by the angle position * freqs[i]; the rest stays."""
    half = len(freqs)
    a = torch.arange(x.shape[0], dtype=torch.float64)[:, None] * torch.tensor(freqs, dtype=torch.float64)
    c, s = torch.cos(a).to(x.dtype)[:, None], torch.sin(a).to(x.dtype)[:, None]
    u, v, rest = x[..., :half], x[..., half:2 * half], x[..., 2 * half:]
    return torch.cat([u * c - v * s, v * c + u * s, rest], -1)


# ---- attention ----
def softcap(s, cap):
    return cap * torch.tanh(s / cap)


def chunk_mask(T, size):
    """True where position i may look at position j: not ahead of it and in the same chunk."""
    i = torch.arange(T)
    return (i[:, None] >= i[None]) & (i[:, None] // size == i[None] // size)


def attend(q, k, v, scale, cap, size):
    """q [T, H, D], k [T, G, D], v [T, G, E] -> [T, H, E]."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    mask = chunk_mask(T, size)
    out = []
    for h in range(H):
        s = softcap((q[:, h] @ k[:, h // per].T) * scale, cap)
        out.append(torch.softmax(s.masked_fill(~mask, float("-inf")), -1) @ v[:, h // per])
    return torch.stack(out, 1)


def attention_block(h, w, p, m, eps):
    T = h.shape[0]
    q = rms(h @ w[p + "q"].T, eps) * w[p + "q.norm"]
    k = rms(h @ w[p + "k"].T, eps) * w[p + "k.norm"]
    v = (h @ w[p + "v"].T).view(T, m["kv_heads"], m["vdim"])
    f = frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"]["scaling"])
    q, k = rotate(q.view(T, m["heads"], m["dim"]), f), rotate(k.view(T, m["kv_heads"], m["dim"]), f)
    return attend(q, k, v, m["scale"], m["softcap"], m["mask"]["size"]).reshape(T, -1) @ w[p + "o"].T


# ---- selective scan ----
def causal_conv(x, w, b):
    """x [T, C], w [C, taps] (the last column meets the current token), zeros before the start."""
    taps = w.shape[1]
    y = b.expand_as(x).clone()
    for j in range(taps):
        back = taps - 1 - j
        if back < x.shape[0]:
            y[back:] += w[:, j] * x[:x.shape[0] - back]
    return y


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def selective_scan(x, dt, A, B, C, D, S=None):
    """x, dt [T, C]; A [C, N]; B, C [T, N]; D [C] -> y [T, C] and the state after the last token."""
    S = torch.zeros_like(A) if S is None else S
    y = []
    for t in range(x.shape[0]):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None]
        y.append(S @ C[t] + D * x[t])
    return torch.stack(y), S


def mamba_block(h, w, p, m):
    inner, rank, N = m["inner"], m["dt_rank"], m["state"]
    xz = h @ w[p + "in"].T
    x, z = xz[:, :inner], xz[:, inner:]
    x = silu(causal_conv(x, w[p + "conv"], w[p + "conv.b"]))
    r = x @ w[p + "x"].T
    dt = softplus(r[:, :rank] @ w[p + "dt"].T + w[p + "dt.b"])
    y, _ = selective_scan(x, dt, -torch.exp(w[p + "A_log"]), r[:, rank:rank + N], r[:, rank + N:], w[p + "D"])
    return (y * silu(z)) @ w[p + "o"].T


# ---- the rest ----
def feed_forward(h, w, p):
    return torch.relu(h @ w[p + "up"].T) ** 2 @ w[p + "down"].T


def layer_order(config):
    """(layer, first of a pass of the loop) in the order they run."""
    n, loop = len(config["layers"]), config.get("loop")
    if loop is None:
        return [(i, False) for i in range(n)]
    order = [(i, False) for i in range(loop["start"])]
    for _ in range(loop["times"]):
        order += [(i, i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return order + [(i, False) for i in range(loop["stop"], n)]


def forward(config, w, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence; appends the residual stream after every layer run to `layers_out`."""
    eps = config["norm"]["eps"]
    x0 = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * config["embedding"]["scale"]
    x = x0
    for i, first in layer_order(config):
        l, n = config["layers"][i], f"l{i}."
        if first:
            x = torch.cat([x, x0], -1) @ w["loop.in"].T
        h = norm_zero_centred(x, w[n + "norm1"], eps)
        if l["type"] == "attention":
            y = attention_block(h, w, n + "mix.", l["mixer"], eps)
        else:
            y = mamba_block(h, w, n + "mix.", l["mixer"])
        if l["mlp"] is not None:
            y = y + feed_forward(norm_zero_centred(x, w[n + "norm2"], eps), w, n + "mlp.")
        x = x + y
        if layers_out is not None:
            layers_out.append(x.clone())
    cap = config["logit_softcap"]
    return softcap(norm_zero_centred(x, w["final.norm"], eps) @ w["head"].T, cap)
