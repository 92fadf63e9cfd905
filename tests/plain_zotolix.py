"""Plain implementation of the Zotolix decoder for the tests: whole sequences, no cache, float64 by default,
one function per mechanism, written from the design's equations. It shares no code with the library's parts.

Notation: T tokens; positions count from 0; matrices are stored [out, in] and applied as h @ W.T. There is not one stream
but a bundle X [S, T, d] of S of them, all equal to the embedding's output at the start. A sublayer F (a mixer or a
feed-forward) with the coefficients a [S], b [S], M [S, S] of its connection works on the bundle as

    u = sum_s a_s X_s;   y = F(norm(u));   X'_t = sum_s M[s, t] X_s + m b_t y      (m: one constant of the model)

and the model's norm and head read sum_s X_s.

Mixers: softmax attention inside chunks of the sequence, with additive vectors in the projections, a rotation of part of
a head, values blended with those of the first layer that blends, and either unit-norm heads (``attention``) or one
sigmoid gate per head (``attention_2``). The feed-forward is a mixture of squared-ReLU experts whose sigmoid weight
multiplies the expert's input.
"""
import json
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


def rms_norm(x, gain, eps):
    return unit_rms(x, eps) * gain


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


# --------------------------------------------------------------------------- the bundle of streams
def gather_streams(X, a):
    """X [S, T, d], a [S] -> sum_s a_s X_s [T, d]."""
    return sum(a[s] * X[s] for s in range(X.shape[0]))


def scatter_streams(X, M, b, y, m):
    """X [S, T, d], M [S, S] indexed [from, to], b [S], y [T, d]: stream t becomes sum_s M[s, t] X_s + m b_t y."""
    S = X.shape[0]
    return torch.stack([sum(M[s, t] * X[s] for s in range(S)) + m * b[t] * y for t in range(S)])


# --------------------------------------------------------------------------- attention
def chunk_visible(T, size):
    """[T, T] bool (query row, key column): earlier keys in the query's own chunk of ``size`` positions (None: all)."""
    pos = torch.arange(T)
    seen = pos[None, :] <= pos[:, None]
    if size is not None:
        seen = seen & (pos[None, :] // size == pos[:, None] // size)
    return seen


def softmax_attention(q, k, v, scale, seen):
    """q [T, H, dk], k [T, H, dk], v [T, H, dv], seen [T, T] -> [T, H, dv]."""
    s = torch.einsum("thd,jhd->htj", q, k) * scale
    w = torch.softmax(s.masked_fill(~seen[None], float("-inf")), dim=-1)
    return torch.einsum("htj,jhd->thd", w, v)


def blend_values(v, v_first, lam):
    return (1.0 - lam) * v + lam * v_first


def attention(h, w, p, m, eps, kind, first_values):
    """``first_values``: the dictionary that carries the first blending layer's values to the later ones."""
    T = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T + w[p + "q.b"]).reshape(T, H, dk)
    k = (h @ w[p + "k"].T + w[p + "k.b"]).reshape(T, G, dk)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).reshape(T, G, dv)
    rot = m.get("rot")
    if rot:
        pos = torch.arange(T)
        q, k = rotate_half(q, pos, rot["base"], rot["dims"]), rotate_half(k, pos, rot["base"], rot["dims"])
    if kind == "attention":
        q, k = unit_rms(q, eps), unit_rms(k, eps)
    if m.get("v_mix"):
        if "v" in first_values:
            v = blend_values(v, first_values["v"], w[p + "vmix"])
        else:
            first_values["v"] = v
    mask = m.get("mask") or {}
    o = softmax_attention(q, k.repeat_interleave(H // G, 1), v.repeat_interleave(H // G, 1), m["scale"],
                          chunk_visible(T, mask.get("size")))
    if kind == "attention_2":
        o = o * torch.sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(T, H * dv) @ w[p + "o"].T


# --------------------------------------------------------------------------- feed-forward
def expert_weights(z, top):
    """z [T, E] -> [T, E]: the sigmoid of the ``top`` largest logits, zero elsewhere (no renormalisation)."""
    s = torch.sigmoid(z)
    chosen = torch.zeros_like(s).scatter(-1, z.topk(top, dim=-1).indices, 1.0)
    return s * chosen


def squared_relu_expert(x, up, down):
    return torch.clamp(x @ up.T, min=0.0) ** 2 @ down.T


def routing_gap(z, top):
    """How clearly the choice is made: the smallest distance of a chosen logit from one that is not."""
    if top == z.shape[-1]:
        return float("inf")
    s = z.sort(dim=-1, descending=True).values
    return float((s[:, top - 1] - s[:, top]).min())


def mixture(h, w, p, m, gaps=None):
    z = h @ w[p + "router"].T
    if gaps is not None:
        gaps.append(routing_gap(z, m["router"]["top"]))
    g = expert_weights(z, m["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(m["router"]["experts"]):
        rows = (g[:, e] > 0).nonzero()[:, 0]
        if rows.numel():
            out[rows] += squared_relu_expert(g[rows, e, None] * h[rows], w[p + f"e{e}.up"], w[p + f"e{e}.down"])
    return out


# --------------------------------------------------------------------------- the model
def forward(cfg, weights, tokens, dtype=torch.float64, rows=None, streams=None, gaps=None):
    """Logits [len(rows), vocab] (every position by default). ``streams``: a list that receives the sum of the
    streams after every layer. ``gaps``: a list that receives how clearly every mixture chose."""
    w = {n: t.to(dtype) if t.is_floating_point() else t for n, t in weights.items()}
    eps, m, S = cfg["norm"]["eps"], cfg["residual_mult"], cfg["streams"]
    x = w["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    X = torch.stack([x] * S)
    first_values = {}
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        y = attention(rms_norm(gather_streams(X, w[p + "hc1.in"]), w[p + "norm1"], eps), w, p + "mix.", layer["mixer"], eps,
                      layer["type"], first_values)
        X = scatter_streams(X, w[p + "hc1.mix"], w[p + "hc1.out"], y, m)
        if layer["mlp"] is not None:
            y = mixture(rms_norm(gather_streams(X, w[p + "hc2.in"]), w[p + "norm2"], eps), w, p + "mlp.", layer["mlp"], gaps)
            X = scatter_streams(X, w[p + "hc2.mix"], w[p + "hc2.out"], y, m)
        if streams is not None:
            streams.append(X.sum(0))
    x = X.sum(0)
    if rows is not None:
        x = x[torch.tensor(list(rows), dtype=torch.long)]
    return rms_norm(x, w["final.norm"], eps) @ w["embed"].T
