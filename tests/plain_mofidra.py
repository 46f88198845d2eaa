"""The Mofidra decoder in plain, slow arithmetic: one function per mechanism, float64, no cache.

A whole sequence goes in and all its logits come out.  Nothing here is shared with the engine's parts
or kernels.  ``cfg`` is the dictionary that config.json holds, ``W`` maps tensor names to tensors.

Notation: ``x`` is the residual stream [T, width]; ``h`` is what both sublayers of a layer read; a
linear map stored [out, in] is applied as ``h @ M.T``; ``pos`` are the tokens' places in their sequence.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


# ------------------------------------------------------------------ small functions
def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def offset_norm(x, w, eps):
    """RMS norm whose stored weight is the distance from one."""
    return unit_rms(x, eps) * (1.0 + w)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def relu_squared(z):
    return torch.clamp(z, min=0.0) ** 2


def turn_halves(v, pos, dims, base):
    """Dim i of the last axis turns together with dim i + dims/2 by ``pos * base^(-2i/dims)``, i < dims/2;
    the dims from ``dims`` on stay.  ``v``: [T, heads, maps, n]."""
    out = v.clone()
    half = dims // 2
    for i in range(half):
        ang = pos.to(F64) * float(base) ** (-2.0 * i / dims)
        c, s = torch.cos(ang)[:, None, None], torch.sin(ang)[:, None, None]
        a, b = v[..., i], v[..., i + half]
        out[..., i] = a * c - b * s
        out[..., i + half] = b * c + a * s
    return out


def causal_softmax(scores):
    """Softmax over the keys j <= i of every row i; ``scores`` [T, T]."""
    T = scores.shape[-1]
    seen = torch.tril(torch.ones(T, T, dtype=torch.bool))
    return torch.softmax(scores.masked_fill(~seen, float("-inf")), dim=-1)


# ------------------------------------------------------------------ mixer
def map_mixing(W, p, diff):
    """The number that multiplies the second map of a layer."""
    first = torch.exp((W[p + "lq1"] * W[p + "lk1"]).sum())
    second = torch.exp((W[p + "lq2"] * W[p + "lk2"]).sum())
    return float(first - second + diff)


def differential_attention(h, W, p, m, pos, eps):
    """Every head attends twice to the same values, with queries and keys of its own each time; the second
    result, times one number of the layer, is taken off the first, and what is left is brought to unit
    root mean square over the head and multiplied by ``1 - diff``."""
    T = h.shape[0]
    H, G, D, V, diff = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["diff"]
    q = (h @ W[p + "q"].T).view(T, H, 2, D)
    k = (h @ W[p + "k"].T).view(T, G, 2, D)
    v = (h @ W[p + "v"].T).view(T, G, V)
    rot = m.get("rot")
    if rot:
        q, k = turn_halves(q, pos, rot["dims"], rot["base"]), turn_halves(k, pos, rot["dims"], rot["base"])
    lam = map_mixing(W, p, diff)
    heads = []
    for j in range(H):
        g = j // (H // G)
        a1, a2 = (causal_softmax(q[:, j, i] @ k[:, g, i].T * m["scale"]) @ v[:, g] for i in (0, 1))
        heads.append(unit_rms(a1 - lam * a2, eps) * (1.0 - diff))
    return torch.cat(heads, dim=-1) @ W[p + "o"].T


# ------------------------------------------------------------------ feed-forwards
def dense(h, W, p):
    return gelu_tanh(h @ W[p + "up"].T) @ W[p + "down"].T


def expert(h, W, p):
    return relu_squared(h @ W[p + ".up"].T) @ W[p + ".down"].T


def choose(z, top):
    """The ``top`` largest of every row of logits and the softmax over those alone."""
    vals, ids = torch.topk(z, top, dim=-1)
    return ids, torch.softmax(vals, dim=-1)


def routed(h, W, p, mlp):
    """Experts chosen per token by biased logits, weighted by the softmax over the chosen, beside a shared
    expert that every token passes and a sigmoid of one number per token scales."""
    z = h @ W[p + "router"].T + W[p + "router.b"]
    ids, wts = choose(z, mlp["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(ids[t].tolist(), wts[t]):
            out[t] = out[t] + w * expert(h[t:t + 1], W, f"{p}e{e}")[0]
    if mlp.get("shared"):
        out = out + torch.sigmoid(h @ W[p + "shared.sg"].T) * expert(h, W, p + "shared")
    return out


# ------------------------------------------------------------------ model
def run_order(cfg):
    """Layer numbers in the order they run."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


def forward(cfg, weights, tokens, trail=None):
    """Logits [T, vocab] of a whole sequence; ``trail``: a list that gets the stream after every layer run."""
    W = {n: t.to(F64) for n, t in weights.items()}
    eps = cfg["norm"]["eps"]
    pos = torch.arange(len(tokens))
    x = W["embed"][tokens] * float((cfg.get("embedding") or {}).get("scale", 1.0))
    for i in run_order(cfg):
        l, p = cfg["layers"][i], f"l{i}."
        h = offset_norm(x, W[p + "norm1"], eps)
        y = differential_attention(h, W, p + "mix.", l["mixer"], pos, eps)
        mlp = l["mlp"]
        if mlp is not None:
            y = y + (dense(h, W, p + "mlp.") if mlp["kind"] == "dense" else routed(h, W, p + "mlp.", mlp))
        x = x + y
        if trail is not None:
            trail.append(x)
    return offset_norm(x, W["final.norm"], eps) @ W["head"].T
