"""CPU restatement of the Bidasun decoder (TEST INFRASTRUCTURE ONLY), one function per mechanism.

Plain numpy over whole sequences, in the precision of the arrays it is given (the tests use float64).
No cache, no portions: every position is computed from the full list of tokens, so whatever the
product keeps between steps has nothing to agree with but the definition.

Weights are a dict of arrays by tensor name ([out, in] matrices); the configuration is the parsed
config.json.
"""
from __future__ import annotations

import math

import numpy as np


def rms_norm(x, w, eps):
    """The last axis scaled to unit root mean square, eps under the root, then weighted."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + x.dtype.type(eps)) * w


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def sigmoid(z):
    out = np.empty_like(z)
    pos = z >= 0
    out[pos] = 1.0 / (1.0 + np.exp(-z[pos]))
    e = np.exp(z[~pos])
    out[~pos] = e / (1.0 + e)
    return out


def embed_with_positions(tokens, table, pos_table, start=0):
    return table[tokens] + pos_table[start:start + len(tokens)]


def token_shift(x, mix):
    """h_t = x_t + (x_{t-1} - x_t) * mix, x_{-1} = 0."""
    before = np.concatenate([np.zeros_like(x[:1]), x[:-1]], axis=0)
    return x + (before - x) * mix


def distance_bias(r1, r2, distance):
    """What is taken off a score at the given distance: r1 * ln(1 + r2 * distance)."""
    return r1 * np.log(1.0 + r2 * distance)


def visible(n, size, keep_first):
    """[query, key] mask: causal, and inside the window or among the first keys of the sequence."""
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    return (j <= i) & ((i - j < size) | (j < keep_first))


def sigmoid_attention(q, k, v, scale, r1, r2, pb, mask):
    """q [n, H, dim], k [n, G, dim], v [n, G, vdim] -> [n, H, vdim]; weights sigmoid(score), not normalised."""
    n, heads, _ = q.shape
    group = heads // k.shape[1]
    dist = np.maximum(np.arange(n)[:, None] - np.arange(n)[None, :], 0).astype(q.dtype)
    out = np.zeros((n, heads, v.shape[2]), q.dtype)
    for h in range(heads):
        s = (q[:, h] @ k[:, h // group].T) * q.dtype.type(scale) - distance_bias(r1[h], r2[h], dist) + pb[h]
        out[:, h] = np.where(mask, sigmoid(s), 0.0) @ v[:, h // group]
    return out


def attention_mixer(x, w, pre, m, eps):
    """Token shift, projections, whole-row q/k norm, windowed sigmoid attention, output gate, W_o."""
    h = token_shift(x, w[pre + "shift"])
    q = rms_norm(h @ w[pre + "mix.q"].T, w[pre + "mix.q.norm"], eps)
    k = rms_norm(h @ w[pre + "mix.k"].T, w[pre + "mix.k.norm"], eps)
    v = h @ w[pre + "mix.v"].T
    n = x.shape[0]
    mask = m.get("mask") or {"size": n, "keep_first": 0}
    o = sigmoid_attention(q.reshape(n, m["heads"], m["dim"]), k.reshape(n, m["kv_heads"], m["dim"]),
                          v.reshape(n, m["kv_heads"], m["vdim"]), m["scale"], w[pre + "mix.r1"], w[pre + "mix.r2"],
                          w[pre + "mix.pb"], visible(n, mask["size"], mask["keep_first"]))
    o = o.reshape(n, -1) * sigmoid(h @ w[pre + "mix.g"].T)
    return o @ w[pre + "mix.o"].T


def gated_mlp(x, w, pre):
    return (gelu_tanh(x @ w[pre + "mlp.gate"].T) * (x @ w[pre + "mlp.up"].T)) @ w[pre + "mlp.down"].T


def forward(cfg, w, tokens, collect=None):
    """Logits [n, vocab] of every position.  `collect`, a list, receives the residual stream after each layer."""
    eps = cfg["norm"]["eps"]
    x = embed_with_positions(np.asarray(tokens), w["embed"], w["pos"])
    for i, layer in enumerate(cfg["layers"]):
        pre = f"l{i}."
        x = x + rms_norm(attention_mixer(x, w, pre, layer["mixer"], eps), w[pre + "norm1"], eps)
        if layer["mlp"] is not None:
            x = x + rms_norm(gated_mlp(x, w, pre), w[pre + "norm2"], eps)
        if collect is not None:
            collect.append(x.copy())
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T
