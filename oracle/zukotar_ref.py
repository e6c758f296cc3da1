"""CPU restatement of the Zukotar decoder (TEST INFRASTRUCTURE ONLY), one function per mechanism.

Plain numpy over whole sequences, in the precision of the arrays it is given (the tests use float64).
No cache, no portions, no chunks: attention looks at the full list of tokens, the recurrence walks it
token by token, every expert is applied to one token at a time.

Weights are a dict of arrays by tensor name ([out, in] matrices); the configuration is the parsed
config.json.
"""
from __future__ import annotations

import numpy as np


def rms_norm(x, w, eps):
    """The last axis scaled to unit root mean square, eps under the root, then weighted."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + x.dtype.type(eps)) * w


def sigmoid(z):
    out = np.empty_like(z)
    pos = z >= 0
    out[pos] = 1.0 / (1.0 + np.exp(-z[pos]))
    e = np.exp(z[~pos])
    out[~pos] = e / (1.0 + e)
    return out


def softmax(z):
    e = np.exp(z - z.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def silu(z):
    return z * sigmoid(z)


def squared_relu(z):
    return np.maximum(z, 0.0) ** 2


def rotate(x, positions, base):
    """x [n, ..., r]: elements 2i and 2i + 1 turned by the angle position * base^(-2i/r)."""
    r = x.shape[-1]
    angle = positions[:, None] * float(base) ** (-2.0 * np.arange(r // 2) / r)
    angle = angle.reshape((len(positions),) + (1,) * (x.ndim - 2) + (r // 2,))
    c, s = np.cos(angle).astype(x.dtype), np.sin(angle).astype(x.dtype)
    out = np.empty_like(x)
    out[..., 0::2] = x[..., 0::2] * c - x[..., 1::2] * s
    out[..., 1::2] = x[..., 1::2] * c + x[..., 0::2] * s
    return out


def visible(n, size):
    """[query, key] mask: causal, the last `size` positions (None: all)."""
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    return (j <= i) & ((i - j < size) if size is not None else True)


def softmax_attention(q, k, v, scale, mask):
    """q, k [n, H, d], v [n, H, e] -> [n, H, e]."""
    out = np.zeros((q.shape[0], q.shape[1], v.shape[2]), q.dtype)
    for h in range(q.shape[1]):
        s = np.where(mask, (q[:, h] @ k[:, h].T) * q.dtype.type(scale), -np.inf)
        out[:, h] = softmax(s) @ v[:, h]
    return out


def latent_attention(h, w, pre, m, eps):
    """Keys and values of every head from one normed latent per token, and one rotated key part for all heads."""
    n, heads, d, r, e, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = np.arange(n)
    q = (h @ w[pre + "q"].T).reshape(n, heads, d + r)
    down = h @ w[pre + "dkv"].T
    latent = rms_norm(down[:, :rank], w[pre + "dkv.norm"], eps)
    q_rot, k_rot = rotate(q[:, :, d:], pos, m["rot"]["base"]), rotate(down[:, rank:], pos, m["rot"]["base"])
    k = (latent @ w[pre + "uk"].T).reshape(n, heads, d)
    v = (latent @ w[pre + "uv"].T).reshape(n, heads, e)
    k = np.concatenate([k, np.broadcast_to(k_rot[:, None, :], (n, heads, r))], axis=2)
    q = np.concatenate([q[:, :, :d], q_rot], axis=2)
    o = softmax_attention(q, k, v, m["scale"], visible(n, (m.get("mask") or {}).get("size")))
    o = o * sigmoid(h @ w[pre + "g"].T)[:, :, None]
    return o.reshape(n, heads * e) @ w[pre + "o"].T


def decays(h, w, pre, tau):
    """[n, heads * dim] in (0, 1): sigmoid(z)^(1/tau) of a low-rank projection z."""
    z = (h @ w[pre + "a1"].T) @ w[pre + "a2"].T + w[pre + "a2.b"]
    return np.exp(-np.logaddexp(0.0, -z) / tau)


def recurrence(q, k, v, alpha, state=None):
    """q, k, alpha [n, H, d], v [n, H, e]: S_t = alpha_t (rows) S_{t-1} + k_t v_t^T, o_t = S_t^T q_t."""
    n, heads, d = q.shape
    s = np.zeros((heads, d, v.shape[2]), q.dtype) if state is None else state.copy()
    out = np.zeros_like(v)
    for t in range(n):
        s = alpha[t][:, :, None] * s + k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hde,hd->he", s, q[t])
    return out, s


def gated_linear_attention(h, w, pre, m, eps):
    n, heads, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w[pre + "q"].T).reshape(n, heads, d) * h.dtype.type(d ** -0.5)
    k = (h @ w[pre + "k"].T).reshape(n, heads, d)
    v = (h @ w[pre + "v"].T).reshape(n, heads, e)
    o, _ = recurrence(q, k, v, decays(h, w, pre, m["tau"]).reshape(n, heads, d))
    o = rms_norm(o, w[pre + "norm"], eps).reshape(n, heads * e) * silu(h @ w[pre + "g"].T)
    return o @ w[pre + "o"].T


def route(logits, top, groups):
    """One token's chosen experts and their weights: softmax over all, the best of the best groups."""
    s = softmax(logits)
    count, keep = (groups["count"], groups["keep"]) if groups else (1, 1)
    best = s.reshape(count, -1).max(axis=1)
    allowed = np.repeat(np.isin(np.arange(count), np.argsort(-best, kind="stable")[:keep]), len(s) // count)
    chosen = np.argsort(-np.where(allowed, s, -1.0), kind="stable")[:top]
    return chosen, s[chosen]


def experts(h, w, pre, mlp):
    logits = h @ w[pre + "router"].T
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        chosen, weight = route(logits[t], mlp["router"]["top"], mlp["router"].get("groups"))
        for e, s in zip(chosen, weight):
            out[t] += s * (squared_relu(h[t] @ w[f"{pre}e{e}.up"].T) @ w[f"{pre}e{e}.down"].T)
    return out


MIXERS = {"latent_attention": latent_attention, "gla": gated_linear_attention}


def layer_runs(cfg):
    """(layer, pass) in the order they run; pass is None outside the loop."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    inner = [(i, t) for t in range(loop["times"]) for i in range(loop["start"], loop["stop"])]
    return [(i, None) for i in range(loop["start"])] + inner + [(i, None) for i in range(loop["stop"], n)]


def forward(cfg, w, tokens, collect=None):
    """Logits [n, vocab] of every position.  `collect`, a list, receives the residual stream after each layer run."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)] * w["embed"].dtype.type(cfg["embedding"]["scale"])
    for i, t in layer_runs(cfg):
        layer, pre = cfg["layers"][i], f"l{i}."
        if t is not None and i == cfg["loop"]["start"]:
            x = x + w["loop.step"][t]
        mixed = MIXERS[layer["type"]](rms_norm(x, w[pre + "norm1"], eps), w, pre + "mix.", layer["mixer"], eps)
        x = x + rms_norm(mixed, w[pre + "norm1b"], eps)
        if layer["mlp"] is not None:
            x = x + rms_norm(experts(rms_norm(x, w[pre + "norm2"], eps), w, pre + "mlp.", layer["mlp"]), w[pre + "norm2b"], eps)
        if collect is not None:
            collect.append(x.copy())
    return rms_norm(x, w["final.norm"], eps) @ w["embed"].T
