"""Vomotar's configuration: keys, errors, layout, tensors, what the layers keep in the cache (pages of the current chunk
beside recurrent states in one layer). No GPU."""
import copy

import pytest
import torch

from vomotar_helpers import ATTENTIVE, CONFIGS, RAGGED, RECURRENT, SMALL, WIDE


def cfg_of(raw):
    from llmplayer_b200.config import config_from_dict
    return config_from_dict(raw)


def test_round_trip_and_registry():
    from llmplayer_b200.config import known_architectures
    from llmplayer_b200.config.vomotar import VomotarConfig
    assert "Vomotar" in known_architectures()
    for raw, _, _ in CONFIGS.values():
        cfg = cfg_of(raw)
        assert isinstance(cfg, VomotarConfig)
        assert cfg_of(cfg.to_dict()) == cfg
        assert cfg.max_positions() >= 65536 and "Vomotar" in cfg.describe()
    cfg = cfg_of(SMALL)
    assert cfg.norm_eps == 2e-6 and cfg.norm_groups == 3
    layout = cfg.layout()
    assert layout.head.norm.groups == 3 and all(b.mixer_norm.groups == 3 for b in layout.layers)
    assert layout.layers[2].ffn is None and layout.layers[2].ffn_norm is None and layout.layers[1].ffn_norm.groups == 3
    bare = copy.deepcopy(SMALL)
    del bare["norm"]["groups"]
    assert cfg_of(bare).norm_groups == 1


@pytest.mark.parametrize("path,value", [
    (("layers", 0, "mixer", "kv_heads"), 3), (("layers", 0, "mixer", "conv"), 0), (("layers", 0, "mixer", "conv"), 9),
    (("layers", 0, "mixer", "dim"), 0), (("layers", 0, "mixer", "dim"), 600), (("layers", 0, "mixer", "vdim"), None),
    (("layers", 0, "type"), "delta"), (("layers", 1, "mixer", "left", "kv_heads"), 3), (("layers", 1, "mixer", "left", "scale"), None),
    (("layers", 1, "mixer", "left", "mask", "size"), 0), (("layers", 1, "mixer", "left", "mask", "size"), -4),
    (("layers", 1, "mixer", "left", "dim"), 300), (("layers", 1, "mixer", "right", "decay"), [0.5, 0.5]),
    (("layers", 1, "mixer", "right", "decay"), 0.5), (("layers", 1, "mixer", "right", "decay"), ["a", 0.5, 0.5]),
    (("layers", 1, "mixer", "right", "rot", "dims"), 7), (("layers", 1, "mixer", "right", "rot", "dims"), 22),
    (("layers", 1, "mixer", "right", "rot", "base"), -1.0), (("layers", 1, "mixer", "right"), None), (("layers", 1, "mlp", "kind"), "moe"),
    (("layers", 1, "mlp", "ff"), 0), (("layers", 1, "mlp"), 5), (("norm", "eps"), 0.0), (("norm", "groups"), 5), (("norm", "groups"), 0),
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
    from llmplayer_b200.cache.sequence_cache import BundleRequest, KVRequest, StateRequest
    from llmplayer_b200.engine.model import Model
    from llmplayer_b200.parts.specs import ANY
    model = Model(cfg_of(SMALL).layout())
    specs = model.tensor_specs()
    assert specs["embed"].shape == (211, 72) and specs["head"].shape == (211, 72) and specs["final.norm"].shape == (72,)
    # the delta rule: fewer query / key heads than value heads, low-rank decays per key channel, a low-rank gate
    assert specs["l0.mix.q"].shape == (40, 72) and specs["l0.mix.k.conv"].shape == (40, 4) and specs["l0.mix.v"].shape == (48, 72)
    assert specs["l0.mix.a1"].shape == (ANY, 72) and specs["l0.mix.a2"].shape == (80, ANY) and specs["l0.mix.dt_bias"].shape == (80,)
    assert specs["l0.mix.g1"].shape == (ANY, 72) and specs["l0.mix.g2"].shape == (48, ANY) and specs["l0.mix.A_log"].shape == (4,)
    assert specs["l0.mix.b"].shape == (4, 72) and specs["l0.mix.norm"].shape == (12,) and specs["l0.mix.o"].shape == (72, 48)
    # the pair: attention without additive vectors, values wider than keys, a distance bias; a retention; two output norms
    assert specs["l1.mix.left.q"].shape == (96, 72) and specs["l1.mix.left.v"].shape == (80, 72) and specs["l1.mix.left.o"].shape == (72, 160)
    assert specs["l1.mix.left.r1"].shape == (4,) and specs["l1.mix.left.r2"].shape == (4,) and "l1.mix.left.q.b" not in specs
    assert specs["l1.mix.right.k"].shape == (60, 72) and specs["l1.mix.right.g"].shape == (36, 72) and specs["l1.mix.right.o"].shape == (72, 36)
    assert specs["l1.mix.left.out"].shape == (72,) and specs["l1.mix.right.out"].shape == (72,)
    assert specs["l1.mlp.gate"].shape == (40, 72) and specs["l1.mlp.down"].shape == (72, 40)
    assert not any(n.startswith(("l2.mlp.", "l2.norm2")) for n in specs)
    reqs = model.cache_requests()
    assert reqs[0] == (StateRequest((4, 12, 20), torch.float32), StateRequest((3, 128), torch.float32))
    # keys of 24 and values of 40 are stored in heads of 48, for the positions of the current chunk
    assert reqs[1] == BundleRequest((KVRequest(2, 48, None, 0, 9), StateRequest((3, 12, 20), torch.float32)))
    assert reqs[3] == BundleRequest((KVRequest(3, 16, None, 0, 50), StateRequest((2, 36, 24), torch.float32)))
    assert reqs[4] == (StateRequest((3, 10, 6), torch.float32), StateRequest((0, 66), torch.float32))
    assert all(isinstance(r, tuple) for r in Model(cfg_of(RECURRENT).layout()).cache_requests())
    assert Model(cfg_of(ATTENTIVE).layout()).cache_requests()[0].members[0] == KVRequest(5, 16)
    assert Model(cfg_of(WIDE).layout()).cache_requests()[0].members[0] == KVRequest(1, 64, None, 0, 64)


def test_a_pair_stacks_its_members_inputs_and_norms_their_results():
    from llmplayer_b200.parts import MIXERS
    layout = cfg_of(WIDE).layout()
    spec = layout.layers[0].mixer
    assert spec.left_scale == spec.right_scale == 0.5 and spec.left_norm.weight == "l0.mix.left.out" and spec.right_norm.groups == 1
    pair = MIXERS.build(spec)
    assert pair.stacked and len(pair.norms) == 2
    assert spec.left.chunk == 64 and spec.left.position.kind == "none" and spec.left.value_norm_eps == 1e-5 and spec.left.general
    assert spec.right.decays == (0.98, 0.99, 0.995, 0.9995) and spec.right.position.pairing == "split_half"
    assert cfg_of(RAGGED).layout().layers[0].mixer.left.chunk == 1


def test_states_inside_a_bundle_are_states():
    """A model whose only states are members of pairs must not run a step twice (captured sampling steps rely on it)."""
    from llmplayer_b200.cache.sequence_cache import BundleRequest, KVRequest, StateRequest, keeps_state
    from llmplayer_b200.engine.model import Model
    assert all(keeps_state(r) for r in Model(cfg_of(ATTENTIVE).layout()).cache_requests())
    assert not keeps_state(BundleRequest((KVRequest(1, 16), None))) and not keeps_state(None) and not keeps_state(KVRequest(1, 16))
    assert keeps_state(StateRequest((2,))) and keeps_state((StateRequest((2,)), StateRequest((3,))))


@pytest.mark.parametrize("chunk", [1, 9, 64, 65, 200, 128])
def test_pages_of_finished_chunks_go_back(chunk):
    """After every length: exactly the pages that hold a position of the next query's chunk (and later ones) are kept."""
    from llmplayer_b200.cache.pages import PageMap
    pages = PageMap(16, chunk=chunk)
    pages.open(0)
    length = 0
    for n in (1, 2, 60, 1, 1, 64, 30, 1, 131, 200, 1):
        pages.extend(0, length + n)
        length += n
        pages.trim(0, length)
        start = length // chunk * chunk
        table = pages.table(0)
        assert len(table) == -(-length // 64)
        for block, page in enumerate(table):
            assert (page >= 0) == ((block + 1) * 64 > start), (length, block)
    pages.close(0)
    assert pages.pool.num_free == 16


def test_cache_serves_both_members_of_a_pair_and_gives_back_clean_states():
    from llmplayer_b200.cache.sequence_cache import BundleView, KVView, SequenceCache, StateView
    from llmplayer_b200.engine.model import Model
    model = Model(cfg_of(SMALL).layout())
    cache = SequenceCache(model.cache_requests(), max_tokens=256, max_slots=3, kv_dtype=torch.float32, device="cpu")
    pair = cache.view(1)
    assert isinstance(pair, BundleView) and isinstance(pair.members[0], KVView) and isinstance(pair.members[1], StateView)
    assert pair.members[0].group_index != cache.view(3).members[0].group_index          # their chunks differ
    a = cache.acquire()
    states = (cache.view(0), pair.members[1], cache.view(2), cache.view(3).members[1], cache.view(4))
    for view in states:
        for block in view.blocks:
            block[a].fill_(3.0)
    cache.release(a)
    b = cache.acquire()
    assert b == a
    for view in states:
        for block in view.blocks:
            assert block[b].numel() == 0 or float(block[b].abs().max()) == 0.0
    cache.reserve([b], [200])
    cache.commit([b], [200])
    assert cache.groups[pair.members[0].group_index].pages.table(b) == [-1, -1, -1, cache.groups[pair.members[0].group_index].pages.table(b)[3]]


def test_norms_in_parts_are_not_fused_into_products():
    """A norm with one factor per row may ride in a product; one with several parts may not."""
    from llmplayer_b200.errors import ConfigError
    from llmplayer_b200.parts import NORMS
    from llmplayer_b200.parts.specs import NormSpec
    whole, parts = NORMS.build(NormSpec(72, 1e-5, "w")), NORMS.build(NormSpec(72, 1e-5, "w", groups=3))
    assert whole.fusable_rms and whole.rms_parts == 1 and not parts.fusable_rms and parts.rms_parts == 3
    with pytest.raises(ConfigError):
        NORMS.build(NormSpec(72, 1e-5, "w", groups=5))


def test_low_rank_maps_must_fit_together():
    from llmplayer_b200.errors import WeightError
    from llmplayer_b200.engine.model import Model
    from llmplayer_b200.parts.base import Runtime
    from llmplayer_b200.weights.random_init import random_tensors
    model = Model(cfg_of(RECURRENT).layout())
    tensors = random_tensors(model.tensor_specs(), 1)
    tensors["l0.mix.a2"] = torch.zeros(128, 7, dtype=torch.bfloat16)
    with pytest.raises(WeightError):
        model.load(tensors, Runtime(device=torch.device("cpu")))
