"""The Lilupel decoder in plain, slow arithmetic: one function per mechanism, float64, no cache.

A whole sequence goes in and all its logits come out; where a mechanism carries something from one
token to the next it is walked token by token.  Nothing here is shared with the engine's parts or
kernels.  ``cfg`` is the dictionary that config.json holds, ``W`` maps tensor names to tensors.

Notation: ``x`` is the residual stream [T, width], which the sublayers read as it is; a linear map
stored [out, in] is applied as ``x @ M.T``; ``pos`` are the tokens' places in their sequence.
"""
from __future__ import annotations

import torch

F64 = torch.float64


# ------------------------------------------------------------------ small functions
def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def offset_norm(x, w, eps):
    """RMS norm whose stored weight is the distance from one."""
    return unit_rms(x, eps) * (1.0 + w)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + torch.clamp(z, min=0.0)


def turn_halves(v, pos, dims, base):
    """Dim i of the last axis turns together with dim i + dims/2 by ``pos * base^(-2i/dims)``, i < dims/2;
    the dims from ``dims`` on stay.  ``v``: [T, heads, n]."""
    out = v.clone()
    half = dims // 2
    for i in range(half):
        ang = pos.to(F64) * float(base) ** (-2.0 * i / dims)
        c, s = torch.cos(ang)[:, None], torch.sin(ang)[:, None]
        a, b = v[..., i], v[..., i + half]
        out[..., i] = a * c - b * s
        out[..., i + half] = b * c + a * s
    return out


def in_window(pos, size):
    """[T, T] truth table: query i sees key j if 0 <= pos_i - pos_j < size."""
    d = pos[:, None] - pos[None, :]
    return (d >= 0) & (d < size)


def softmax_beside_sink(s, sink, ok):
    """exp(s_j) / (exp(sink) + sum_j exp(s_j)) over the keys a row sees; ``s`` [T, T], ``sink`` a number."""
    s = s.masked_fill(~ok, float("-inf"))
    top = torch.maximum(s.max(dim=-1, keepdim=True).values, sink.reshape(1, 1))
    e = torch.exp(s - top)
    return e / (torch.exp(sink - top) + e.sum(dim=-1, keepdim=True))


def short_conv(z, taps, bias):
    """Causal convolution over time, one filter per channel: z [T, C], taps [C, n] whose last
    column meets the current token; zeros stand before the start."""
    T, C = z.shape
    n = taps.shape[1]
    padded = torch.cat([torch.zeros(n - 1, C, dtype=F64), z], dim=0)
    out = bias[None, :].repeat(T, 1)
    for j in range(n):
        out = out + padded[j:j + T] * taps[:, j][None, :]
    return out


def fading_memory(q, k, v, keep, write):
    """S <- keep_t S + write_t k_t v_t^T from S = 0, o_t = S^T q_t, one head: q, k [T, N], v [T, V], keep and
    write [T]."""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=F64)
    out = []
    for t in range(q.shape[0]):
        S = keep[t] * S + write[t] * torch.outer(k[t], v[t])
        out.append(S.T @ q[t])
    return torch.stack(out)


# ------------------------------------------------------------------------- mixers
def sink_attention(x, W, p, m, pos, eps):
    """Windowed attention with biased projections, turned queries and keys of unit rms per head, and a
    learnt number per head in the softmax's denominator."""
    T = x.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (x @ W[p + "q"].T + W[p + "q.b"]).reshape(T, H, D)
    k = (x @ W[p + "k"].T + W[p + "k.b"]).reshape(T, G, D)
    v = (x @ W[p + "v"].T + W[p + "v.b"]).reshape(T, G, V)
    rot = m["rot"]
    q = unit_rms(turn_halves(q, pos, rot["dims"], rot["base"]), eps)
    k = unit_rms(turn_halves(k, pos, rot["dims"], rot["base"]), eps)
    ok = in_window(pos, m["mask"]["size"])
    heads = []
    for h in range(H):
        g = h // (H // G)
        heads.append(softmax_beside_sink(q[:, h] @ k[:, g].T * m["scale"], W[p + "sink"][h], ok) @ v[:, g])
    return torch.cat(heads, dim=-1) @ W[p + "o"].T + W[p + "o.b"]


def retention(x, W, p, m, pos, eps):
    """A memory per head that fades at a fixed rate; turned queries and keys, the output of every head of
    unit rms and gated."""
    T = x.shape[0]
    H, D, V = m["heads"], m["dim"], m["vdim"]
    rot = m["rot"]
    q = turn_halves((x @ W[p + "q"].T).reshape(T, H, D), pos, rot["dims"], rot["base"])
    k = turn_halves((x @ W[p + "k"].T).reshape(T, H, D), pos, rot["dims"], rot["base"]) * D ** -0.5
    v = (x @ W[p + "v"].T).reshape(T, H, V)
    one = torch.ones(T, dtype=F64)
    o = torch.cat([unit_rms(fading_memory(q[:, h], k[:, h], v[:, h], m["decay"][h] * one, one), eps) for h in range(H)], dim=-1)
    return (o * silu(x @ W[p + "g"].T)) @ W[p + "o"].T


def side_by_side(x, W, p, m, pos, eps):
    left = sink_attention(x, W, p + "left.", m["left"], pos, eps)
    right = retention(x, W, p + "right.", m["right"], pos, eps)
    return m["left_scale"] * left + m["right_scale"] * right


def split_state_input(z, m):
    """The columns of the wide projection: the gate, x, B, C and the step sizes."""
    inner, gn = m["heads"] * m["vdim"], m["groups"] * m["state"]
    return torch.split(z, [inner, inner, gn, gn, m["heads"]], dim=-1)


def state_space(x, W, p, m, eps):
    """A state [N, V] per head that fades by exp(-exp(A_log) dt), dt a number per token and head; what it takes
    in and what reads it come from a short convolution and are shared by the heads of a group."""
    T = x.shape[0]
    H, V, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * V
    z, xs, B, C, dt = split_state_input(x @ W[p + "in"].T, m)
    u = silu(short_conv(torch.cat([xs, B, C], dim=-1), W[p + "conv"], W[p + "conv.b"]))
    xs, B, C = u[:, :inner].reshape(T, H, V), u[:, inner:inner + G * N].reshape(T, G, N), u[:, inner + G * N:].reshape(T, G, N)
    dt = softplus(dt + W[p + "dt_bias"])
    heads = []
    for h in range(H):
        g = h // (H // G)
        keep = torch.exp(-torch.exp(W[p + "A_log"][h]) * dt[:, h])
        heads.append(fading_memory(C[:, g], B[:, g], xs[:, h], keep, dt[:, h]) + W[p + "D"][h] * xs[:, h])
    y = torch.cat(heads, dim=-1) * silu(z)
    parts = m["norm_groups"]
    y = unit_rms(y.reshape(T, parts, inner // parts), eps).reshape(T, inner) * W[p + "norm"]
    return y @ W[p + "o"].T


# ------------------------------------------------------------------- feed-forward
def expert(x, W, p):
    return (silu(x @ W[p + ".gate"].T) * (x @ W[p + ".up"].T)) @ W[p + ".down"].T


def experts_by_token(x, W, p, mlp, tokens):
    """A table row per token id names the experts; their mean is the result."""
    top = mlp["router"]["top"]
    out = []
    for t, tok in enumerate(tokens):
        ids = W[p + "table"][tok].long().tolist()
        assert len(ids) == top
        out.append(sum(expert(x[t:t + 1], W, f"{p}e{e}")[0] for e in ids) / top)
    return torch.stack(out)


# -------------------------------------------------------------------------- model
def weight_layer(cfg, i):
    """The layer whose tensors layer i uses."""
    return cfg["layers"][i].get("weights_of", i)


def forward(cfg, weights, tokens, trail=None):
    """Logits [T, vocab] of a whole sequence; ``trail``: a list that gets the stream after every layer."""
    W = {n: t.to(F64) for n, t in weights.items()}
    eps = cfg["norm"]["eps"]
    pos = torch.arange(len(tokens))
    x = W["embed"][tokens]
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{weight_layer(cfg, i)}.", layer["mixer"]
        y = side_by_side(x, W, p + "mix.", m, pos, eps) if layer["type"] == "parallel" else state_space(x, W, p + "mix.", m, eps)
        x = x + offset_norm(y, W[p + "norm1"], eps)
        if layer.get("mlp") is not None:
            x = x + offset_norm(experts_by_token(x, W, p + "mlp.", layer["mlp"], tokens), W[p + "norm2"], eps)
        if trail is not None:
            trail.append(x)
    return offset_norm(x, W["final.norm"], eps) @ W["embed"].T
