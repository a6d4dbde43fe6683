"""Ludelorn without a GPU: registry, tensor names and shapes, cache plan, part parameters, distance buckets, refused
configurations."""

import copy
import math

import pytest

import plain_ludelorn as plain
from yalis_b200.cache.manager import CacheManager
from yalis_b200.cache.storage import group_page_bytes, plan_groups
from yalis_b200.config.presets import preset
from yalis_b200.config.registry import ConfigError, load_config, parse_config
from yalis_b200.engine.model import Model
from yalis_b200.parts.base import PagedKV, SlotState, cache_leaves


def spec_of(name):
    arch, cfg = parse_config(preset(name))
    return arch, cfg, arch.model_spec(cfg)


def test_the_registry_knows_the_design_and_round_trips_its_configuration():
    for which in ("tiny-A", "tiny-B", "tiny-C", "tiny-D", "1b", "3b"):
        raw = preset(f"ludelorn-{which}")
        arch, cfg = parse_config(raw)
        assert arch.name == "Ludelorn" and arch.config_to_dict(cfg) == raw


def test_tensor_names_and_shapes_follow_the_layers():
    _, _, spec = spec_of("ludelorn-tiny-A")
    t = {name: tuple(ps.shape) for name, ps in Model(spec).expected_tensors().items()}
    assert t["embed"] == t["head"] == (96, 64) and t["final.norm"] == t["l0.norm1"] == t["l2.norm2"] == ()
    assert t["l0.mix.left.q"] == (64, 64) and t["l0.mix.left.v"] == (48, 64) and t["l0.mix.left.g"] == (96, 64)
    assert t["l0.mix.left.q.norm"] == t["l0.mix.left.k.norm"] == (16,) and t["l0.mix.left.out"] == t["l0.ls1"] == (64,)
    inner, channels = 4 * 12, 4 * 12 + 2 * 2 * 10
    assert t["l0.mix.right.in"] == (inner + channels + 4, 64) and t["l0.mix.right.conv"] == (channels, 3)
    assert t["l0.mix.right.conv.b"] == (channels,) and t["l0.mix.right.dt_bias"] == t["l0.mix.right.D"] == (4,)
    assert t["l0.mix.right.norm"] == (inner,) and t["l0.mix.right.o"] == (64, inner)
    assert t["l1.mix.q.norm"] == (64,) and t["l1.mix.k.norm"] == (32,)                  # over all heads at once
    assert t["l2.mix.rel"] == (8, 4) and t["l2.mix.sink"] == (4,) and t["l2.mix.g"] == (4, 64)
    assert t["l0.mlp.up.b"] == (80,) and t["l0.mlp.down.b"] == (64,)
    assert not {"l2.mix.v", "l2.mix.q.norm", "l1.norm2", "l1.ls2", "l1.mlp.up", "l1.mix.out"} & set(t)


def test_what_the_mixers_keep():
    _, _, spec = spec_of("ludelorn-tiny-A")
    reqs = Model(spec).cache_requests()
    state = reqs[0]["right"]
    assert reqs[0]["left"] == PagedKV(2, 16, 9, v_head_dim=24)
    # per head a matrix [vdim, state rounded up to 4], then the convolution's last two inputs per channel
    assert isinstance(state, SlotState) and state.shape == (4 * 12 * 12 + 88 * 2,)
    # tokens are kept for a block's length where that is more than the window; a mean per block is kept for ever
    assert reqs[1] == {"tokens": PagedKV(2, 16, 7, v_head_dim=8), "blocks": PagedKV(2, 16, None, v_head_dim=8, pool=7)}
    assert reqs[2] == PagedKV(2, 12, 23)
    assert reqs[4]["tokens"].window == 11 and reqs[4]["blocks"].pool == 3


def test_a_group_of_blocks_counts_in_blocks_of_tokens():
    reqs = [{"tokens": PagedKV(2, 16, 44), "blocks": PagedKV(2, 16, None, pool=8)}, PagedKV(1, 8)]
    groups = {g.name: g for g in plan_groups(reqs, 16, 50, 400, max_slots=3, step_tokens=64)}
    blocks = groups["kv_all_pool_8"]
    assert blocks.page_size == 128 and blocks.max_pages_per_request == 4 and blocks.num_pages == 7 + 3
    assert groups["kv_all"].num_pages == 50 and groups["kv_all"].page_size == 16
    size = group_page_bytes(reqs, [None, None], 16, 2)
    assert size["kv_all_pool_8"] == 2 * 16 * 32 * 2 // 8 and size["kv_window_44"] == 2 * 16 * 32 * 2
    # the pool holds any requests that fit the tokens' pool: each takes ceil(length / 128) pages
    m = CacheManager(3, [blocks])
    lengths = [398, 370, 4]
    assert sum(-(-n // 16) for n in lengths) == 50
    slots = [m.acquire() for _ in lengths]
    assert m.reserve_many(slots, lengths)
    m.commit_many(slots, lengths)
    assert m.free_pages("kv_all_pool_8") == 10 - (4 + 3 + 1)
    for s in slots:
        m.release(s)
    m.check()


def test_what_the_design_fixes_reaches_the_parts_as_parameters():
    _, cfg, spec = spec_of("ludelorn-tiny-A")
    par, pooled, biased = (spec.layers[i].parts["mixer"] for i in (0, 1, 2))
    assert par.kind == "sum_of_mixers" and par.params["factor"] == 0.5 and par.params["norm_eps"] == cfg.norm_eps
    left, right = par.params["mixers"]["left"].params, par.params["mixers"]["right"]
    assert right.kind == "state_space" and right.params["conv"] == 3 and right.params["norm_groups"] == 3
    assert left["rotary"]["layout"] == "half" and left["rotary"]["scaling"]["kind"] == "yarn" and left["gate"] is True
    assert left.get("qk_norm_over", "head") == "head" and left["window"] == 9 and left["pool"] is None
    assert pooled.params["qk_norm_over"] == "all" and pooled.params["pool"] == 7 and pooled.params["rotary"]["layout"] == "interleaved"
    assert pooled.params["rotary"]["scaling"] is None
    b = biased.params
    assert b["values_from_keys"] and b["rotary"] is None and not b["qk_norm_weight"] and b["sink"] == "learned" and b["gate"] == "head"
    assert b["distance_bias"] == {"buckets": 8, "max": 20}
    for layer in spec.layers:
        assert layer.block.kind == "pre_norm_connected" and layer.parts["connection_1"].kind == "scaled_sum"
        assert layer.parts["norm_1"].params["scalar"]
    assert spec.layers[0].parts["feed_forward"].params["activation"] == "gelu_tanh" and spec.layers[0].parts["feed_forward"].params["bias"]
    assert "feed_forward" not in spec.layers[1].parts and spec.embedding_scale == 2.5 and spec.head_name == "head"


def test_the_number_of_buckets_is_read_off_a_tensor():
    from ludelorn_models import ludelorn_dir
    _, cfg = load_config(ludelorn_dir("A"))
    assert cfg.layers[2]["mixer"]["buckets"] == 8


def test_distance_buckets_are_exact_where_logarithms_fall_short():
    from yalis_b200.parts.attention import distance_bucket, distance_reach
    for buckets, far in ((2, 3), (4, 9), (8, 20), (10, 160), (16, 300), (20, 320), (32, 128)):
        h = buckets // 2
        values = [distance_bucket(n, buckets, far) for n in range(500)]
        assert values[:h] == list(range(h)) and values == sorted(values) and values[-1] == buckets - 1
        assert values == [plain.distance_bucket(n, buckets, far) for n in range(500)]
        for n in range(h, 500):              # the logarithm, a rounding error aside
            z = math.log(n / h) / math.log(far / h) * (buckets - h)
            assert values[n] in (min(buckets - 1, h + math.floor(z - 1e-9)), min(buckets - 1, h + math.floor(z + 1e-9)))
        reach = distance_reach(buckets, far)
        assert values[reach - 1] == buckets - 1 and (reach == 1 or values[reach - 2] < buckets - 1)
    # 10 / 5 = 2 is the fifth root of 160 / 5 = 32: the bucket changes exactly there
    assert distance_bucket(10, 10, 160) == 6 and distance_bucket(9, 10, 160) == 5
    assert distance_bucket(6, 6, 7.5) == distance_bucket(60, 6, 7.5) == 5          # a limit that is no whole number


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].update(type="mlp"), "type"),
    (lambda c: c["layers"][0]["mixer"].pop("right"), "right"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3), "multiple"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=18), "dims"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].pop("fast"), "fast"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(groups=3), "groups"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(norm_groups=5), "norm_groups"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(pool=0), "pool"),
    (lambda c: c["layers"][2]["mixer"].update(vdim=8), "vdim"),
    (lambda c: c["layers"][2]["mixer"].update(buckets=7), "even"),
    (lambda c: c["layers"][2]["mixer"].update(bias_max=4), "bias_max"),
    (lambda c: c["layers"][2]["mixer"].pop("buckets"), "buckets"),
    (lambda c: c["layers"][0].update(mlp={"kind": "moe"}), "mlp"),
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c.update(layers=[]), "layers")])
def test_configurations_that_are_refused(change, message):
    raw = copy.deepcopy(preset("ludelorn-tiny-A"))
    change(raw)
    with pytest.raises(ConfigError, match=message):
        parse_config(raw)


def test_parts_refuse_what_they_cannot_be():
    from yalis_b200.config.spec import PartSpec
    from yalis_b200.parts.base import make_part
    base = {"hidden_size": 16, "num_heads": 2, "num_kv_heads": 1, "head_dim": 8, "window": 4}
    for extra in ({"pool": 2, "window": None}, {"pool": 2, "window": None, "chunk": 4}, {"values_from_keys": True, "v_head_dim": 4},
                  {"distance_bias": {"buckets": 5, "max": 9}}, {"distance_bias": {"buckets": 4, "max": 2}}):
        with pytest.raises(ValueError):
            make_part("mixer", PartSpec("general_attention", {**base, **extra}))
    attention = PartSpec("general_attention", base)
    with pytest.raises(ValueError):
        make_part("mixer", PartSpec("sum_of_mixers", {"mixers": {"a": attention}, "norm_eps": 1e-5}))
    with pytest.raises(ValueError):
        make_part("mixer", PartSpec("sum_of_mixers", {"mixers": {"a": attention, "b": attention}, "factor": 0.5}))
    with pytest.raises(ValueError):
        make_part("mixer", PartSpec("state_space", {"hidden_size": 8, "heads": 3, "vdim": 4, "state": 4, "groups": 2, "conv": 4,
                                                    "norm_groups": 1, "eps": 1e-5}))


def test_every_preset_plans_its_cache():
    for which in ("tiny-B", "tiny-C", "tiny-D", "1b", "3b"):
        _, _, spec = spec_of(f"ludelorn-{which}")
        model = Model(spec)
        reqs = model.cache_requests()
        groups = plan_groups(reqs, 16, 40, 512, max_slots=4, step_tokens=256)
        assert {g.name for g in groups} and all(leaf is not None for r in reqs for leaf in cache_leaves(r))
