"""Lagulorn without a GPU: registry, layers that run another's tensors, tensor names, caches and states, what reaches the
parts as parameters, refused configurations, and the plain model's own pieces against sums written out by hand."""

import copy
import math

import pytest
import torch

import plain_lagulorn as plain
from lagulorn_models import lagulorn_dir
from yalis_b200.config.presets import preset
from yalis_b200.config.registry import ConfigError, load_config, parse_config
from yalis_b200.config.spec import PartSpec
from yalis_b200.engine.model import Model
from yalis_b200.parts.base import PagedKV, SlotState, make_part


def spec_of(name):
    arch, cfg = parse_config(preset(name))
    return arch, cfg, arch.model_spec(cfg)


def test_the_registry_knows_the_design_and_round_trips_its_configuration():
    for which in "ABCD":
        raw = preset(f"lagulorn-tiny-{which}")
        arch, cfg = parse_config(raw)
        assert arch.name == "Lagulorn" and arch.config_to_dict(cfg) == raw
        assert load_config(lagulorn_dir(which))[1] == cfg


def test_layers_that_run_anothers_tensors_keep_caches_and_states_of_their_own():
    _, _, spec = spec_of("lagulorn-tiny-A")
    assert [e.layer for e in spec.schedule] == [0, 1, 0, 1, 2] and all(e.cache_of is None for e in spec.schedule)
    assert [l.weight_prefix for l in spec.layers] == ["l0.", "l1.", "l4."]
    model = Model(spec)
    state = SlotState((2 * 12 * 16,), torch.float32)
    keys = PagedKV(2, 2 * 12, 9, v_head_dim=20)                       # both maps' keys in one row
    assert model.cache_requests() == [state, keys, state, keys, SlotState((3 * 10 * 8,), torch.float32)]
    names = set(model.expected_tensors())
    assert not any(n.startswith(("l2.", "l3.")) for n in names)
    _, cfg, spec = spec_of("lagulorn-tiny-D")                         # a chain: layer 3 names layer 2, which names layer 0
    assert cfg.owner(3) == 0 and [e.layer for e in spec.schedule] == [0, 1, 0, 0]


def test_tensor_names_and_shapes():
    _, _, spec = spec_of("lagulorn-tiny-A")
    shapes = {n: tuple(p.shape) for n, p in Model(spec).expected_tensors().items()}
    layer0 = {n[3:]: s for n, s in shapes.items() if n.startswith("l0.")}
    assert layer0 == {"norm1": (64,), "norm2": (64,), "mix.q": (32, 64), "mix.k": (32, 64), "mix.v": (24, 64), "mix.g": (24, 64), "mix.o": (64, 24),
                      "mix.norm": (24,), "mlp.up": (80, 64), "mlp.down": (64, 80), "hc1.in": (2,), "hc1.out": (2,), "hc1.mix": (2, 2),
                      "hc2.in": (2,), "hc2.out": (2,), "hc2.mix": (2, 2)}
    layer1 = {n[3:]: s for n, s in shapes.items() if n.startswith("l1.") and ".e" not in n}
    assert layer1 == {"norm1": (64,), "norm2": (64,), "mix.q": (4 * 2 * 12, 64), "mix.k": (2 * 2 * 12, 64), "mix.v": (2 * 20, 64), "mix.o": (64, 80),
                      "mix.q.norm": (12,), "mix.k.norm": (12,), "mix.lq1": (12,), "mix.lk1": (12,), "mix.lq2": (12,), "mix.lk2": (12,),
                      "mlp.router": (8, 64), "mlp.correction": (8,), "hc1.in": (2,), "hc1.out": (2,), "hc1.mix": (2, 2),
                      "hc2.in": (2,), "hc2.out": (2,), "hc2.mix": (2, 2)}
    assert shapes["l1.mlp.e5.gate"] == (16, 64) and "l1.mlp.e6.gate" not in shapes       # identity experts have no tensors
    assert "l4.norm2" not in shapes and "l4.hc2.in" not in shapes                          # a layer without feed-forward
    assert shapes["final.norm"] == (64,) and shapes["head"] == shapes["embed"] == (96, 64)
    plain_sum = {n for n in Model(spec_of("lagulorn-tiny-D")[2]).expected_tensors() if ".hc" in n}
    assert not plain_sum                                                                   # one stream: no mixing weights


def test_constants_reach_the_parts_as_parameters():
    _, _, spec = spec_of("lagulorn-tiny-A")
    lightning, attention = spec.layers[0].parts, spec.layers[1].parts
    assert lightning["mixer"].params["decay"] == [0.5, 0.98] and lightning["norm_1"].params["one_plus"]
    assert lightning["connection_1"].params["factor"] == 0.7
    assert attention["mixer"].params["difference"] == {"offset": 0.2, "eps": 1e-5} and attention["mixer"].params["window"] == 9
    ff = attention["feed_forward"].params
    assert (ff["experts"], ff["identity"], ff["top"], ff["groups"], ff["limit"], ff["renorm"]) == (6, 2, 3, {"count": 4, "keep": 2}, 0.8, False)
    _, _, spec = spec_of("lagulorn-tiny-D")
    assert spec.stream_copies is None and spec.layers[0].parts["connection_1"].params["factor"] == 1.5


def test_refused_configurations():
    base = preset("lagulorn-tiny-A")

    def broken(change, error=ConfigError):
        raw = copy.deepcopy(base)
        change(raw)
        with pytest.raises(error):
            parse_config(raw)

    broken(lambda r: r["layers"][0].update(type="retention"))
    broken(lambda r: r["layers"][0]["mixer"].update(decay=[0.5]))                      # a number per head
    broken(lambda r: r["layers"][0]["mixer"].update(dim=0))
    broken(lambda r: r["layers"][0]["mlp"].update(kind="gated"))
    broken(lambda r: r["layers"][1]["mixer"].update(kv_heads=3))
    broken(lambda r: r["layers"][1]["mixer"].pop("diff"))
    broken(lambda r: r["layers"][1]["mixer"].update(mask={"size": 0}))
    broken(lambda r: r["layers"][1]["mlp"]["router"].update(top=5))                    # two groups of two leave four
    broken(lambda r: r["layers"][1]["mlp"]["router"].update(groups={"count": 3, "keep": 1}))
    broken(lambda r: r["layers"][1]["mlp"]["router"].update(groups={"count": 4, "keep": 5}))
    broken(lambda r: r["layers"][1]["mlp"]["expert"].pop("limit"))
    broken(lambda r: r["layers"][2].update(weights_of=1))                              # another type of layer
    broken(lambda r: r["layers"][2].update(weights_of=9))
    broken(lambda r: r["layers"][0].update(weights_of=2))                              # each names the other
    broken(lambda r: r["layers"][2]["mixer"].update(vdim=13))                          # not the entry of the layer it shares
    broken(lambda r: r.pop("norm"))
    broken(lambda r: r.update(streams=0))
    with pytest.raises(ValueError):
        arch, cfg = parse_config({**copy.deepcopy(base), "streams": 9})
        Model(arch.model_spec(cfg))


def test_parts_refuse_what_they_do_not_combine():
    att = {"hidden_size": 32, "num_heads": 4, "num_kv_heads": 2, "head_dim": 8, "difference": {"offset": 0.1, "eps": 1e-5}}
    make_part("mixer", PartSpec("general_attention", att))
    for extra in ({"sink": True}, {"softcap": 3.0}, {"gate": True}, {"chunk": 4}, {"window": 4, "pool": 2}, {"out_scale": 0.5}):
        with pytest.raises(ValueError):
            make_part("mixer", PartSpec("general_attention", {**att, **extra}))
    moe = {"hidden_size": 32, "experts": 6, "top": 2, "expert_size": 8, "activation": "clamped", "limit": 1.0, "alpha": 1.0, "shift": 0.0, "gated": True,
           "identity": 2}
    make_part("feed_forward", PartSpec("routed_experts", moe))
    for extra in ({"shared_size": 8}, {"weight_on": "input"}, {"groups": {"count": 3, "keep": 1}}, {"groups": {"count": 8, "keep": 1}}, {"limit": 0.0},
                  {"top": 9}):
        with pytest.raises(ValueError):
            make_part("feed_forward", PartSpec("routed_experts", {**moe, **extra}))
    with pytest.raises(ValueError):
        make_part("connection", PartSpec("hyper_connection", {"hidden_size": 8, "mixing": False, "factor": 0.5}))
    with pytest.raises(ValueError):
        make_part("mixer", PartSpec("retention", {"hidden_size": 8, "heads": 1, "dim": 4, "vdim": 4, "decay": [0.5], "eps": 1e-5, "activation": "silu",
                                                  "rotary": {"dims": 4, "theta": 10.0}}))


def test_counts_of_operations():
    model = Model(spec_of("lagulorn-tiny-A")[2])
    assert model.blocks[0].mixer.mixing_flops(3, 100) == 4.0 * 2 * 16 * 12 * 3
    assert model.blocks[1].mixer.mixing_flops(1, 100) == 2.0 * 4 * 2 * (12 + 20) * 9           # two maps, nine keys
    assert model.blocks[1].feed_forward.matrix_flops_per_token() == 2.0 * 64 * (8 + 3 * (3 * 6 / 8) * 16)


# ---- the plain model's pieces against sums by hand ---------------------------------------------------------------

def test_the_plain_pieces_by_hand():
    # the norm's weight lies around zero
    got = plain.layer_norm(torch.tensor([[3.0, 4.0]]), torch.tensor([0.0, 1.0]), 0.0)
    assert got.flatten().tolist() == pytest.approx([3 / math.sqrt(12.5), 8 / math.sqrt(12.5)])
    # a state that halves: the second token reads its own write and half of the first's
    one = torch.ones(2, 1, 1)
    out, last = plain.decaying_state(one, torch.tensor([[[2.0]], [[3.0]]]), torch.tensor([[[5.0]], [[7.0]]]), [0.5])
    assert out.flatten().tolist() == [10.0, 26.0] and last.flatten().tolist() == [26.0]
    # a window of two: position 2 sees positions 1 and 2 with equal scores
    z = torch.zeros(3, 1, 1)
    assert plain.windowed_attention(z, z, torch.tensor([[[9.0]], [[2.0]], [[4.0]]]), 1.0, 2).flatten().tolist() == pytest.approx([9.0, 5.5, 3.0])
    # the balance of the maps, and their difference
    t = {"lq1": torch.tensor([1.0, 2.0]), "lk1": torch.tensor([0.5, 0.25]), "lq2": torch.tensor([1.0, 0.0]), "lk2": torch.tensor([0.0, 3.0])}
    assert plain.map_balance(t, "", 0.25) == pytest.approx(math.e - 1.0 + 0.25)
    o = plain.difference_of_maps(torch.tensor([5.0, 1.0]), torch.tensor([2.0, -1.0]), 1.0, 0.25, 0.0)          # (3, 2)
    assert o.tolist() == pytest.approx([0.75 * 3 / math.sqrt(6.5), 0.75 * 2 / math.sqrt(6.5)])
    # the clamped unit: the gate is bounded from above only
    got = plain.clamped_unit(torch.tensor([5.0, -5.0]), torch.tensor([-9.0, 9.0]), 2.0)
    want = [2 / (1 + math.exp(-3.404)) * -1, -5 / (1 + math.exp(8.51)) * 3]
    assert got.tolist() == pytest.approx(want)
    # two copies: read 1 x_0 + 2 x_1; write with mix [from, to]
    streams = torch.tensor([[[1.0]], [[2.0]]])
    assert plain.read_copies(streams, torch.tensor([1.0, 2.0])).tolist() == [[5.0]]
    new = plain.write_copies(streams, torch.tensor([[1.0, 10.0], [100.0, 1000.0]]), torch.tensor([1.0, -1.0]), torch.tensor([[0.5]]))
    assert new.flatten().tolist() == pytest.approx([1 * 1 + 100 * 2 + 0.5, 10 * 1 + 1000 * 2 - 0.5])


def test_the_plain_choice_by_hand():
    """Four outputs in two groups; scores 0.1, 0.2, 0.3, 0.4.  A correction of -2 on the last two makes every choice score
    of their group negative; masking the group with zero instead of minus infinity would choose them after the first."""
    router = torch.log(torch.tensor([[0.1], [0.2], [0.3], [0.4]]))
    h = torch.tensor([[1.0]])
    chosen, weights = plain.routing(h, router, torch.zeros(4), 2, {"count": 2, "keep": 1})
    assert chosen.tolist() == [[3, 2]] and weights.flatten().tolist() == pytest.approx([0.4, 0.3])
    chosen, weights = plain.routing(h, router, torch.tensor([-1.0, -1.0, -2.0, -2.0]), 2, {"count": 2, "keep": 1})
    assert chosen.tolist() == [[1, 0]] and weights.flatten().tolist() == pytest.approx([0.2, 0.1])
    chosen, _ = plain.routing(h, router, torch.tensor([0.0, 5.0, 0.0, 0.0]), 3, None)
    assert chosen.tolist() == [[1, 3, 2]]
