"""Small Zotolix configurations with sizes of their own, and seeded model folders for them."""
import json
import os

import torch


def _layer(kind, heads, kv_heads, dim, vdim, scale, size=None, dims=0, base=10000.0, v_mix=False, mlp=None):
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": v_mix}
    if size is not None:
        mixer["mask"] = {"size": size}
    if dims:
        mixer["rot"] = {"base": base, "dims": dims}
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def _moe(ff, experts, top):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


UNIT, GATED = "attention", "attention_2"

# Odd sizes: three streams, values wider than keys and narrower, chunks of 9 and of 50, rotations over part of a head and
# none, blended values in layers whose other sizes differ, a first layer that blends nothing and one in between, layers
# without a feed-forward, two of five experts chosen.
SMALL = {
    "architecture": "Zotolix", "vocab": 211, "width": 72, "norm": {"eps": 2e-6}, "embedding": {"scale": 3.0}, "streams": 3,
    "residual_mult": 0.8,
    "layers": [
        _layer(UNIT, 3, 3, 16, 16, 0.25, 50, 8, mlp=_moe(24, 3, 1)),
        _layer(GATED, 4, 2, 24, 40, 0.3, 9, 20, 700.0, v_mix=True, mlp=_moe(40, 5, 2)),
        _layer(UNIT, 6, 2, 20, 40, 0.4, 50, 20, v_mix=True, mlp=None),
        _layer(GATED, 5, 5, 10, 12, 0.3, None, 0, mlp=_moe(20, 4, 4)),
        _layer(GATED, 6, 2, 12, 40, 0.3, 33, 6, v_mix=True, mlp=_moe(36, 6, 3)),
    ],
}
# Sizes the tensor-core kernels take: chunks of exactly one page, of 70 (their borders cross a page's while decoding) and of
# 128 positions, eight query heads on one key head, heads of 128, four streams, top 1 and top 3.
WIDE = {
    "architecture": "Zotolix", "vocab": 384, "width": 128, "norm": {"eps": 1e-5}, "embedding": {"scale": 5.0}, "streams": 4,
    "residual_mult": 0.6,
    "layers": [
        _layer(GATED, 8, 1, 64, 64, 0.2, 64, 32, 50000.0, v_mix=True, mlp=_moe(64, 4, 1)),
        _layer(UNIT, 4, 1, 64, 64, 0.3, 70, 64, 50000.0, v_mix=True, mlp=_moe(96, 6, 3)),
        _layer(GATED, 4, 2, 32, 48, 0.3, 128, 16, mlp=None),
        _layer(UNIT, 2, 1, 128, 64, 0.2, 200, 128, v_mix=True, mlp=_moe(128, 2, 1)),
    ],
}
# A width that is no multiple of 8 (every product leaves the tensor cores, also in bfloat16) nor of 4, one stream, chunks of
# ONE position (a token sees itself alone) and of two, one head, one expert.
RAGGED = {
    "architecture": "Zotolix", "vocab": 131, "width": 53, "norm": {"eps": 3e-5}, "embedding": {"scale": 2.0}, "streams": 1,
    "residual_mult": 1.0,
    "layers": [
        _layer(GATED, 5, 1, 10, 12, 0.4, 1, 2, 100.0, v_mix=True, mlp=_moe(13, 3, 2)),
        _layer(UNIT, 1, 1, 6, 12, 0.4, 2, 6, 100.0, v_mix=True, mlp=_moe(7, 1, 1)),
        _layer(UNIT, 5, 5, 10, 6, 0.4, 65, 10, 100.0, mlp=_moe(22, 5, 5)),
    ],
}
# Nothing but attention over everything: no chunks, no blended values, five streams (a number without a kernel of its own),
# no feed-forward at the end; more experts than a warp has lanes.
OPEN = {
    "architecture": "Zotolix", "vocab": 170, "width": 96, "norm": {"eps": 1e-5}, "embedding": {"scale": 4.0}, "streams": 5,
    "residual_mult": 0.5,
    "layers": [
        _layer(UNIT, 6, 2, 32, 32, 0.2, None, 16, 800.0, mlp=_moe(16, 40, 5)),
        _layer(GATED, 6, 3, 16, 64, 0.3, None, 16, 800.0, mlp=_moe(32, 8, 2)),
        _layer(UNIT, 3, 1, 48, 32, 0.2, 100, 0, mlp=None),
    ],
}
# Two streams and a single blending layer (it shows its values to nobody).
PAIR = {
    "architecture": "Zotolix", "vocab": 150, "width": 64, "norm": {"eps": 1e-5}, "embedding": {"scale": 1.0}, "streams": 2,
    "residual_mult": 0.9,
    "layers": [_layer(GATED, 4, 4, 16, 16, 0.4, 20, 16, mlp=_moe(48, 4, 2)), _layer(UNIT, 2, 1, 64, 64, 0.2, 90, 32, v_mix=True, mlp=_moe(48, 4, 1)),
               _layer(GATED, 4, 2, 32, 16, 0.3, 64, 8, mlp=_moe(40, 3, 1))],
}
CONFIGS = {"small": (SMALL, 61, 0.1), "wide": (WIDE, 62, 0.08), "ragged": (RAGGED, 63, 0.12), "open": (OPEN, 64, 0.1), "pair": (PAIR, 65, 0.12)}

# bfloat16: at most four times the worst error that the comparisons of each configuration achieved on a B200
BFLOAT16_BOUND = {"small": 2.6e-2, "wide": 2.8e-2, "ragged": 2.4e-2, "open": 1.1e-2, "pair": 3.4e-2}     # achieved: 6.6e-3, 7.2e-3, 6.2e-3, 2.9e-3, 8.7e-3


def bound(dtype, name):
    return 2e-5 if dtype == "float32" else BFLOAT16_BOUND[name]


def make_model(tmp_path, name, dtype="bfloat16"):
    """A model folder for configuration ``name``: the library's seeded writer, then the tensors whose random draw would
    switch a mechanism off are drawn again: the connections (streams that differ, each of which every sublayer reads and
    changes, and none of which grows), the share of the first values (also in the first layer that blends, which does not
    use it), additive vectors, gates far from one half.

    The routing is made robust against rounding: the first channels of the stream carry a code per token (distinct levels
    with wide gaps, in the embedding), nothing else writes to these channels (the rows of every matrix that writes to the
    streams are zero there), and every router reads only them, one channel per expert. The streams mix channel by channel,
    so an expert's logit is the token's code times a factor that all experts share, and no choice rests on a close call."""
    from llmplayer_b200.config import config_from_dict
    from llmplayer_b200.weights import write_random_model
    from llmplayer_b200.weights.safetensors_io import write_safetensors
    from plain_llama import read_safetensors
    raw, seed, std = CONFIGS[name]
    out = os.path.join(str(tmp_path), f"zotolix_{name}_{dtype}")
    write_random_model(config_from_dict(raw), seed, out, dtype=dtype, std=std)
    path = os.path.join(out, "model.safetensors")
    tensors = read_safetensors(path)
    gen = torch.Generator().manual_seed(seed + 100)
    store = torch.bfloat16 if dtype == "bfloat16" else torch.float32
    d, S = raw["width"], raw["streams"]
    C = max(layer["mlp"]["router"]["experts"] for layer in raw["layers"] if layer["mlp"] is not None)

    def draw(*shape, scale=1.0, shift=0.0):
        return (shift + scale * torch.randn(*shape, generator=gen)).to(store)

    levels = torch.linspace(-1.9, 1.9, C) + 0.2 / C * torch.sin(torch.arange(C) * 2.4)
    embed = tensors["embed"].to(torch.float32)
    for t in range(raw["vocab"]):
        embed[t, :C] = std * levels[torch.randperm(C, generator=gen)]
    tensors["embed"] = embed.to(store)

    def silent(name_):
        """The matrix does not write to the channels that carry the code."""
        mat = tensors[name_].to(torch.float32)
        mat[:C, :] = 0
        tensors[name_] = mat.to(store)

    for i, layer in enumerate(raw["layers"]):
        p, m = f"l{i}.mix.", layer["mixer"]
        silent(p + "o")
        for q in ("hc1", "hc2"):
            if q == "hc2" and layer["mlp"] is None:
                continue
            tensors[f"l{i}.{q}.in"] = draw(S, scale=0.4, shift=1.0 / S)
            tensors[f"l{i}.{q}.out"] = draw(S, scale=0.5, shift=1.0)
            mix = 0.6 * torch.eye(S) + 0.3 / S + 0.25 * torch.randn(S, S, generator=gen) / S ** 0.5
            tensors[f"l{i}.{q}.mix"] = mix.to(store)
        for n in ("q.b", "k.b", "v.b"):
            tensors[p + n] = draw(*tensors[p + n].shape, scale=0.4)
        if m["v_mix"]:                                             # the first such layer's is in the file and unused
            tensors[p + "vmix"] = (0.3 + 0.4 * torch.rand((), generator=gen)).to(store)
        if layer["type"] == GATED:
            tensors[p + "g"] = draw(m["heads"], d, scale=2.0 * d ** -0.5)
        if layer["mlp"] is not None:
            E = layer["mlp"]["router"]["experts"]
            router = torch.zeros(E, d)
            router[torch.arange(E), torch.arange(E)] = 1.0
            tensors[f"l{i}.mlp.router"] = router.to(store)
            tensors[f"l{i}.norm2"] = torch.cat([torch.ones(C), tensors[f"l{i}.norm2"][C:].to(torch.float32)]).to(store)
            for e in range(E):
                silent(f"l{i}.mlp.e{e}.down")
    write_safetensors(path, tensors, metadata={"format": "pt"})
    with open(os.path.join(out, "config.json"), "w") as fh:
        json.dump(raw, fh, indent=1)
    return out


def plain_logits(model_dir, tokens, rows=None, streams=None, gaps=None):
    import plain_zotolix
    cfg, w = plain_zotolix.read_model(model_dir)
    return plain_zotolix.forward(cfg, w, tokens, dtype=torch.float64, rows=rows, streams=streams, gaps=gaps)
