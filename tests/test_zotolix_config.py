"""Zotolix's configuration: keys, errors, layout, tensors, what the layers keep in the cache, checks across layers; and
that the plain implementation's mechanisms all show in the logits of the tests' models. No GPU."""
import copy

import pytest
import torch

from helpers import random_tokens, relative_error
from zotolix_helpers import CONFIGS, OPEN, PAIR, RAGGED, SMALL, WIDE, bound, make_model


def cfg_of(raw):
    from llmplayer_b200.config import config_from_dict
    return config_from_dict(raw)


def test_round_trip_and_registry():
    from llmplayer_b200.config import known_architectures
    from llmplayer_b200.config.zotolix import ZotolixConfig
    assert "Zotolix" in known_architectures()
    for raw, _, _ in CONFIGS.values():
        cfg = cfg_of(raw)
        assert isinstance(cfg, ZotolixConfig)
        assert cfg_of(cfg.to_dict()) == cfg
        assert cfg.max_positions() >= 65536 and "Zotolix" in cfg.describe()
    bare = copy.deepcopy(SMALL)
    del bare["embedding"], bare["residual_mult"], bare["layers"][0]["mixer"]["v_mix"]
    cfg = cfg_of(bare)
    assert cfg.embedding_scale == 1.0 and cfg.residual_mult == 1.0 and not cfg.layers[0].mixer.v_mix


@pytest.mark.parametrize("path,value", [
    (("layers", 0, "type"), "attention_3"), (("layers", 0, "mixer", "kv_heads"), 2), (("layers", 0, "mixer", "dim"), 0),
    (("layers", 0, "mixer", "dim"), 300), (("layers", 0, "mixer", "vdim"), None), (("layers", 0, "mixer", "scale"), None),
    (("layers", 0, "mixer", "mask", "size"), 0), (("layers", 0, "mixer", "mask", "keep_first"), 3), (("layers", 0, "mixer", "v_mix"), 1),
    (("layers", 0, "mixer", "rot", "dims"), 7), (("layers", 0, "mixer", "rot", "dims"), 18), (("layers", 0, "mixer", "rot", "base"), -1.0),
    (("layers", 4, "mixer", "vdim"), 20), (("layers", 4, "mixer", "kv_heads"), 3), (("layers", 0, "mlp", "kind"), "dense"),
    (("layers", 0, "mlp", "expert", "ff"), 0), (("layers", 0, "mlp", "router", "top"), 4), (("layers", 0, "mlp", "router", "experts"), None),
    (("layers", 0, "mlp"), 5), (("norm", "eps"), 0.0), (("streams",), 0), (("streams",), None), (("embedding", "scale"), "x"),
    (("width",), 0), (("vocab",), -3), (("layers",), []),
])
def test_bad_values_are_refused(path, value):
    from llmplayer_b200.errors import ConfigError
    raw = copy.deepcopy(SMALL)
    at = raw
    for key in path[:-1]:
        at = at[key]
    at[path[-1]] = value
    with pytest.raises(ConfigError):
        cfg_of(raw)


def test_tensors_and_cache_requests():
    from llmplayer_b200.cache.sequence_cache import KVRequest
    from llmplayer_b200.engine.model import Model
    cfg = cfg_of(SMALL)
    model = Model(cfg.layout())
    specs = model.tensor_specs()
    assert specs["embed"].shape == (211, 72) and "head" not in specs and specs["final.norm"].shape == (72,)
    assert specs["l1.mix.q"].shape == (96, 72) and specs["l1.mix.v"].shape == (80, 72) and specs["l1.mix.o"].shape == (72, 160)
    assert specs["l1.mix.v.b"].shape == (80,) and specs["l1.mix.g"].shape == (4, 72) and "l0.mix.g" not in specs
    # the first layer that blends uses no share of its own, later ones do, the one without blending has none
    assert "l1.mix.vmix" not in specs and specs["l2.mix.vmix"].shape == () and "l3.mix.vmix" not in specs and specs["l4.mix.vmix"].shape == ()
    assert specs["l1.mlp.e4.up"].shape == (40, 72) and specs["l1.mlp.e4.down"].shape == (72, 40) and "l1.mlp.e0.gate" not in specs
    assert specs["l1.mlp.router"].shape == (5, 72) and "l1.mlp.e5.up" not in specs
    assert specs["l0.hc1.in"].shape == (3,) and specs["l0.hc2.mix"].shape == (3, 3) and specs["l4.hc2.out"].shape == (3,)
    assert not any(n.startswith(("l2.mlp.", "l2.norm2", "l2.hc2")) for n in specs)
    spare = cfg.ignorable_tensors()
    assert {"l0.mix.vmix", "l1.mix.vmix", "l3.mix.vmix", "l2.norm2", "l2.hc2.mix"} <= set(spare) and "l2.mix.vmix" not in spare
    # keys of 24 and values of 40 are stored in heads of 48, for the positions of the current chunk
    assert model.cache_requests() == [KVRequest(3, 16, None, 0, 50), KVRequest(2, 48, None, 0, 9), KVRequest(2, 48, None, 0, 50),
                                      KVRequest(5, 16), KVRequest(2, 48, None, 0, 33)]
    assert model.capture_safe and Model(cfg_of(WIDE).layout()).capture_safe


def test_layout():
    layout = cfg_of(SMALL).layout()
    assert layout.head.weight == "embed" and layout.embedding.scale == 3.0 and layout.head.logit_scale == 1.0
    assert all(b.streams == 3 and b.residual_scale == 0.8 and b.kind == "bundle" for b in layout.layers)
    m0, m1, m2, m3, m4 = (b.mixer for b in layout.layers)
    assert m0.unit_norm_eps == 2e-6 and m0.head_gate is None and m1.unit_norm_eps is None and m1.head_gate == "l1.mix.g"
    assert [m.shows_values for m in (m0, m1, m2, m3, m4)] == [False, True, False, False, False]
    assert (m0.value_blend, m1.value_blend, m2.value_blend, m4.value_blend) == (None, None, "l2.mix.vmix", "l4.mix.vmix")
    assert m1.chunk == 9 and m3.chunk is None and m3.position.kind == "none" and m1.position.rotary_dim == 20 and m1.position.theta == 700.0
    ffn = layout.layers[1].ffn
    assert ffn.activation == "relu2" and ffn.weight_on == "input" and ffn.routing.scoring == "sigmoid_top" and ffn.routing.top == 2
    assert layout.layers[2].ffn is None and layout.layers[2].ffn_connection is None
    assert cfg_of(PAIR).first_blend() == 1 and cfg_of(OPEN).first_blend() is None and cfg_of(RAGGED).first_blend() == 0


def test_values_must_have_been_shown():
    """The model checks across layers: a layer blends only what a run before it has shown, in its size."""
    from dataclasses import replace
    from llmplayer_b200.engine.model import Model
    from llmplayer_b200.errors import ConfigError
    layout = cfg_of(WIDE).layout()
    Model(layout)
    with pytest.raises(ConfigError):
        Model(replace(layout, schedule=(), layers=layout.layers[1:]))
    first = layout.layers[0]
    with pytest.raises(ConfigError):
        Model(replace(layout, layers=(replace(first, mixer=replace(first.mixer, value_dim=32)),) + layout.layers[1:]))
    with pytest.raises(ConfigError):
        Model(replace(layout, layers=(replace(first, mixer=replace(first.mixer, value_blend="l0.mix.vmix")),) + layout.layers[1:]))


def test_nothing_is_added_between_two_layers_that_share_a_bundle():
    from dataclasses import replace
    from llmplayer_b200.engine.model import Model
    from llmplayer_b200.errors import ConfigError
    layout = cfg_of(WIDE).layout()
    runs = list(layout.schedule)
    Model(replace(layout, schedule=tuple([replace(runs[0], add_embedding=True)] + runs[1:])))
    with pytest.raises(ConfigError):
        Model(replace(layout, schedule=tuple([runs[0], replace(runs[1], add_embedding=True)] + runs[2:])))


def test_parts_refuse_what_does_not_fit_together():
    from dataclasses import replace
    from llmplayer_b200.errors import ConfigError
    from llmplayer_b200.parts import BLOCKS, FEED_FORWARDS
    layout = cfg_of(WIDE).layout()
    block, ffn = layout.layers[0], layout.layers[0].ffn
    for bad in (replace(block, streams=0), replace(block, streams=33), replace(block, ffn_connection=None), replace(block, ffn_norm=None),
                replace(block, mixer_norm=replace(block.mixer_norm, kind="layernorm")), replace(block, mixer_norm=replace(block.mixer_norm, groups=2))):
        with pytest.raises(ConfigError):
            BLOCKS.build(bad)
    for bad in (replace(ffn, activation="silu"), replace(ffn, weight_on="both"), replace(ffn, shared_size=8, shared_prefix="s."),
                replace(ffn, routing=replace(ffn.routing, groups=2))):
        with pytest.raises(ConfigError):
            FEED_FORWARDS.build(bad)
    # the same experts under other rules of choice, weighted on their outputs
    for scoring in ("sigmoid_groups", "softmax_top", "softmax_groups"):
        FEED_FORWARDS.build(replace(ffn, weight_on="output", routing=replace(ffn.routing, scoring=scoring)))


def _variants():
    import plain_zotolix as P

    def mask(grow):
        def change(cfg):
            for layer in cfg["layers"]:
                if layer["mixer"].get("mask"):
                    layer["mixer"]["mask"]["size"] += grow
        return change

    def rot(cfg):
        for layer in cfg["layers"]:
            if layer["mixer"].get("rot"):
                layer["mixer"]["rot"]["base"] *= 1.5

    def no_blend(cfg):
        for layer in cfg["layers"]:
            layer["mixer"]["v_mix"] = False

    def other_kind(cfg):
        for layer in cfg["layers"]:
            layer["type"] = "attention"

    def mult(cfg):
        cfg["residual_mult"] *= 1.15
    return {
        "a chunk one longer": (mask(1), {}), "a chunk one shorter": (mask(-1), {}), "another rotation": (rot, {}),
        "no blended values": (no_blend, {}), "unit-norm heads for gates": (other_kind, {}), "another multiplier": (mult, {}),
        "the mix read the other way round": (None, {"scatter_streams": lambda X, M, b, y, m, f=P.scatter_streams: f(X, M.T, b, y, m)}),
        "one stream read for all": (None, {"gather_streams": lambda X, a, f=P.gather_streams: a.sum() * X[0]}),
        "the weight on the output": (None, {"squared_relu_expert": lambda x, u, d: torch.clamp(x @ u.T, min=0.0) @ d.T}),
        "renormalised weights": (None, {"expert_weights": lambda z, top, f=P.expert_weights: f(z, top) / f(z, top).sum(-1, keepdim=True)}),
    }


@pytest.mark.parametrize("what", list(_variants()))
def test_every_mechanism_shows_in_the_logits(tmp_path, monkeypatch, what):
    """A mistake planted in the plain implementation moves the logits of the tests' model by more than a bfloat16
    comparison forgives."""
    import plain_zotolix
    model_dir = make_model(tmp_path, "wide")
    cfg, w = plain_zotolix.read_model(model_dir)
    tokens = random_tokens(220, cfg["vocab"], seed=9)
    rows = list(range(0, 220, 3)) + [64, 65, 70, 71, 128, 140, 200]
    right = plain_zotolix.forward(cfg, w, tokens, rows=rows)
    change, patches = _variants()[what]
    wrong_cfg = copy.deepcopy(cfg)
    if change is not None:
        change(wrong_cfg)
    for name, fn in patches.items():
        monkeypatch.setattr(plain_zotolix, name, fn)
    wrong = plain_zotolix.forward(wrong_cfg, w, tokens, rows=rows)
    assert relative_error(wrong, right) > 2 * bound("bfloat16", "wide"), what
