"""Plain implementation of the Vomotar decoder for the tests: whole sequences, no cache, float64 by default,
one function per mechanism, written from the design's equations. It shares no code with the library's parts.

Notation: x is the stream [T, d]; positions count from 0; matrices are stored [out, in] and applied as h @ W.T.
A layer is pre-norm with RMS norms in equal parts of the width:

    x <- x + mixer(part_norm(x, norm1));   x <- x + ffn(part_norm(x, norm2))

Mixers: ``channel_delta`` (a gated delta rule with a decay per head and key channel) and ``parallel`` (softmax
attention inside chunks of the sequence, its scores lowered by a logarithm of the distance, beside a retention with a
fixed decay per head; each result normed over the width, half their sum). The feed-forward is a dense gated one.
"""
import json
import math
import os

import torch

from plain_llama import read_safetensors


def read_model(model_dir):
    with open(os.path.join(model_dir, "config.json")) as fh:
        cfg = json.load(fh)
    return cfg, read_safetensors(os.path.join(model_dir, "model.safetensors"))


# --------------------------------------------------------------------------- small pieces
def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def part_norm(x, gain, eps, parts):
    """The row in ``parts`` equal pieces, each divided by its own root mean square; then the gain over the whole row."""
    T, d = x.shape
    return unit_rms(x.reshape(T, parts, d // parts), eps).reshape(T, d) * gain


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.where(z > 30.0, z, torch.log1p(torch.exp(torch.clamp(z, max=30.0))))


def unit_length(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def short_convolution(u, taps):
    """u [T, C], taps [C, K]: out[t, c] = sum_j taps[c, j] * u[t - (K - 1) + j, c], zeros before the start."""
    T, C = u.shape
    K = taps.shape[1]
    padded = torch.cat([torch.zeros(K - 1, C, dtype=u.dtype), u], dim=0)
    return sum(padded[j:j + T] * taps[:, j] for j in range(K))


def rotate_half(v, positions, base, dims):
    """v [T, heads, n]: feature i (< dims / 2) pairs with i + dims / 2 and turns by position * base^(-2 i / dims)."""
    if not dims:
        return v
    half = dims // 2
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=v.dtype)
    angle = positions.to(v.dtype)[:, None] * f
    cos, sin = torch.cos(angle)[:, None], torch.sin(angle)[:, None]
    a, b = v[..., :half], v[..., half:dims]
    return torch.cat([a * cos - b * sin, b * cos + a * sin, v[..., dims:]], dim=-1)


# --------------------------------------------------------------------------- recurrences
def channel_delta_recurrence(q, k, v, g, beta, S=None):
    """q, k [T, H, dk], v [T, H, dv], g [T, H, dk] (decays of the key channels), beta [T, H]; S [H, dk, dv].
    S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q. Returns (o [T, H, dv], S)."""
    T, H, dk = q.shape
    S = torch.zeros(H, dk, v.shape[-1], dtype=q.dtype) if S is None else S.clone()
    out = []
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hkv,hk->hv", S, q[t]))
    return torch.stack(out), S


def retention_recurrence(q, k, v, decay, S=None):
    """q, k [T, H, dk], v [T, H, dv], decay [H]: S <- decay S + k v^T; o = S^T q. Returns (o, S)."""
    T, H, dk = q.shape
    S = torch.zeros(H, dk, v.shape[-1], dtype=q.dtype) if S is None else S.clone()
    out = []
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hkv,hk->hv", S, q[t]))
    return torch.stack(out), S


# --------------------------------------------------------------------------- mixers
def channel_delta(h, w, p, m, eps):
    T = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = silu(short_convolution(h @ w[p + "q"].T, w[p + "q.conv"])).reshape(T, G, dk)
    k = silu(short_convolution(h @ w[p + "k"].T, w[p + "k.conv"])).reshape(T, G, dk)
    v = silu(short_convolution(h @ w[p + "v"].T, w[p + "v.conv"])).reshape(T, H, dv)
    q = (unit_length(q) * dk ** -0.5).repeat_interleave(H // G, dim=1)
    k = unit_length(k).repeat_interleave(H // G, dim=1)
    beta = torch.sigmoid(h @ w[p + "b"].T)
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]
    g = torch.exp(-torch.exp(w[p + "A_log"])[None, :, None] * softplus(z).reshape(T, H, dk))
    o, _ = channel_delta_recurrence(q, k, v, g, beta)
    gate = torch.sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T).reshape(T, H, dv)
    o = unit_rms(o, eps) * w[p + "norm"] * gate
    return o.reshape(T, H * dv) @ w[p + "o"].T


def chunk_visible(T, size):
    """[T, T] bool (query row, key column): earlier keys in the query's own chunk of ``size`` positions (None: all)."""
    pos = torch.arange(T)
    seen = pos[None, :] <= pos[:, None]
    if size is not None:
        seen = seen & (pos[None, :] // size == pos[:, None] // size)
    return seen


def distance_attention(q, k, v, scale, r1, r2, visible):
    """q [T, H, dk], k [T, H, dk], v [T, H, dv]; the score of key j for query i is (q . k) scale - r1 ln(1 + r2 (i - j))
    with a head's own r1 and r2."""
    pos = torch.arange(q.shape[0])
    gap = (pos[:, None] - pos[None, :]).clamp(min=0).to(q.dtype)
    scores = torch.einsum("thd,shd->hts", q, k) * scale
    if r1 is not None:
        scores = scores - r1[:, None, None] * torch.log(1.0 + r2[:, None, None] * gap)
    scores = scores.masked_fill(~visible[None], -math.inf)
    return torch.einsum("hts,shd->thd", torch.softmax(scores, dim=-1), v)


def chunked_attention(h, w, p, m, eps):
    T = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).reshape(T, H, dk)
    k = (h @ w[p + "k"].T).reshape(T, G, dk).repeat_interleave(H // G, dim=1)
    v = unit_rms((h @ w[p + "v"].T).reshape(T, G, dv), eps).repeat_interleave(H // G, dim=1)
    size = (m.get("mask") or {}).get("size")
    o = distance_attention(q, k, v, m["scale"], w[p + "r1"], w[p + "r2"], chunk_visible(T, size))
    return o.reshape(T, H * dv) @ w[p + "o"].T


def retention(h, w, p, m, eps):
    T = h.shape[0]
    H, dk, dv = m["heads"], m["dim"], m["vdim"]
    positions = torch.arange(T)
    rot = m.get("rot") or {"base": 1.0, "dims": 0}
    q = rotate_half((h @ w[p + "q"].T).reshape(T, H, dk), positions, rot["base"], rot["dims"])
    k = rotate_half((h @ w[p + "k"].T).reshape(T, H, dk), positions, rot["base"], rot["dims"]) * dk ** -0.5
    v = (h @ w[p + "v"].T).reshape(T, H, dv)
    o, _ = retention_recurrence(q, k, v, torch.tensor(m["decay"], dtype=h.dtype))
    return (unit_rms(o, eps).reshape(T, H * dv) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def parallel_mixer(h, w, p, m, eps):
    left = unit_rms(chunked_attention(h, w, p + "left.", m["left"], eps), eps) * w[p + "left.out"]
    right = unit_rms(retention(h, w, p + "right.", m["right"], eps), eps) * w[p + "right.out"]
    return 0.5 * (left + right)


# --------------------------------------------------------------------------- feed-forward and model
def dense_ffn(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def forward(cfg, w, tokens, dtype=torch.float64, rows=None, streams=None):
    """Logits [T (or len(rows)), vocab] of a whole sequence. ``streams``: a list that receives the stream after
    every layer."""
    w = {name: t.to(dtype) for name, t in w.items()}
    eps, parts = cfg["norm"]["eps"], cfg["norm"].get("groups", 1)
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = part_norm(x, w[p + "norm1"], eps, parts)
        mix = {"channel_delta": channel_delta, "parallel": parallel_mixer}[layer["type"]]
        x = x + mix(h, w, p + "mix.", m, eps)
        if layer["mlp"] is not None:
            x = x + dense_ffn(part_norm(x, w[p + "norm2"], eps, parts), w, p + "mlp.")
        if streams is not None:
            streams.append(x.clone())
    if rows is not None:
        x = x[torch.as_tensor(rows, dtype=torch.long)]
    return part_norm(x, w["final.norm"], eps, parts) @ w["head"].T
