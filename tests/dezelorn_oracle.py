"""Plain, slow restatement of the Dezelorn decoder in PyTorch: one function per mechanism, straight from the equations.

Nothing here is shared with the product code. Everything runs in the dtype of the weights that are passed in (float64 in
the tests), over whole sequences, with explicit [T, T] score matrices and Python loops where that is the clearest.

Notation: T tokens of one sequence at positions 0..T-1; H query heads, G key heads, query head h reads key head
h // (H // G); D the head size.
"""
import math

import torch


def dyt(x, alpha, w, b):
    """Dynamic Tanh: an elementwise squashing in place of a mean / variance norm."""
    return torch.tanh(alpha * x) * w + b


def short_conv(u, w):
    """Causal convolution over time, each channel with its own taps; u [T, C], w [C, taps]; zeros before the start."""
    T, C = u.shape
    taps = w.shape[1]
    y = torch.zeros_like(u)
    for t in range(T):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                y[t] += w[:, j] * u[s]
    return y


def query_temperature(T, coef, every, dtype):
    """Factor of the query at each position: grows with the logarithm of the number of finished stretches of `every`."""
    return torch.tensor([1.0 + coef * math.log(math.floor((p + 1) / every) + 1) for p in range(T)], dtype=dtype)


def distance_bias(T, r1, r2):
    """[H, T, T]: r1 * ln(1 + r2 * (i - j)) for j <= i (0 elsewhere; those entries are masked anyway)."""
    i = torch.arange(T)
    d = (i[:, None] - i[None, :]).clamp(min=0).to(r1.dtype)
    return r1[:, None, None] * torch.log(1 + r2[:, None, None] * d[None])


def window_mask(T, size):
    """True where position i may look at position j: itself and the size - 1 tokens before it."""
    i = torch.arange(T)
    d = i[:, None] - i[None, :]
    return (d >= 0) & (d < size)


def attention_weights(q, k, scale, temp, r1, r2, window):
    """Softmax weights [H, T, T] of q [T, H, D] on k [T, G, D]."""
    T, H, _ = q.shape
    G = k.shape[1]
    bias = distance_bias(T, r1, r2)
    mask = window_mask(T, window)
    out = torch.zeros(H, T, T, dtype=q.dtype)
    for h in range(H):
        s = ((q[:, h] * temp[:, None]) @ k[:, h // (H // G)].T) * scale - bias[h]
        out[h] = torch.softmax(s.masked_fill(~mask, float("-inf")), dim=-1)
    return out


def mix_heads(weights, talk):
    """Weights of head h become the talk[h]-weighted sum of all heads' weights."""
    return torch.einsum("hg,gij->hij", talk, weights)


def apply_weights(weights, v):
    """[T, H, D]: every head's weights on the values of its own key head; v [T, G, D]."""
    H, T, _ = weights.shape
    G = v.shape[1]
    return torch.stack([weights[h] @ v[:, h // (H // G)] for h in range(H)], dim=1)


def attention_block(h, w, p, spec):
    """Mixer on h [T, width]. `w` maps tensor names to weights, `p` is the prefix of the layer's mixer."""
    T = h.shape[0]
    H, G, D = spec["heads"], spec["kv_heads"], spec["dim"]
    q = short_conv(h @ w[p + "q"].T, w[p + "q.conv"]).view(T, H, D)
    k = short_conv(h @ w[p + "k"].T, w[p + "k.conv"]).view(T, G, D)
    temp = query_temperature(T, spec["q_temp"]["coef"], spec["q_temp"]["every"], h.dtype)
    a = attention_weights(q, k, spec["scale"], temp, w[p + "r1"], w[p + "r2"], spec["mask"]["size"])
    o = apply_weights(mix_heads(a, w[p + "talk"]), k).reshape(T, H * D)
    o = o * torch.sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


def feed_forward(h, w, p):
    g = h @ w[p + "gate"].T
    return (g * torch.sigmoid(g) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def forward(config, w, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence; appends the residual stream after every layer to `layers_out`."""
    def norm(x, name):
        return dyt(x, w[name + ".alpha"], w[name], w[name + ".b"])

    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * config["embedding"]["scale"]
    for i, layer in enumerate(config["layers"]):
        n = f"l{i}."
        x = x + norm(attention_block(norm(x, n + "norm1"), w, n + "mix.", layer["mixer"]), n + "norm1b")
        if layer["mlp"] is not None:
            x = x + norm(feed_forward(norm(x, n + "norm2"), w, n + "mlp."), n + "norm2b")
        if layers_out is not None:
            layers_out.append(x.clone())
    return norm(x, "final.norm") @ w["head"].T
