"""Small Lagulorn model folders for the tests, with weights that make every mechanism show.

The product's random-weights mode draws every matrix from N(0, 0.02) and sets scales, mixing and corrections to neutral
values, under which both maps are nearly uniform, all experts score alike and the copies of the stream do not differ.
The folders made here draw matrices wide enough for peaked attention and decisive routing, mixing matrices and read and
write weights that tell the copies apart, corrections of both signs larger than most scores, and balance vectors that put
the second map's weight away from its constant.  Names and shapes come from the model's own list of expected tensors; the
values are this file's.
"""

import functools
import json
import os
import tempfile

import torch

from yalis_b200.config.presets import preset
from yalis_b200.config.registry import parse_config
from yalis_b200.engine.model import Model
from yalis_b200.weights.safetensors_io import write_safetensors

_ROOT = None


def _root():
    global _ROOT
    if _ROOT is None:
        _ROOT = tempfile.mkdtemp(prefix="yalis_b200_lagulorn_")
    return _ROOT


def lively_tensor(name: str, shape, gen: torch.Generator) -> torch.Tensor:
    def normal(std, mean=0.0):
        return mean + torch.randn(shape, generator=gen) * std

    last = name.split(".")[-1]
    if last in ("norm1", "norm2") or name == "final.norm":
        return normal(0.3)                              # stored around zero
    if last == "norm":
        return normal(0.25, 1.0)                        # plain scales: the read-out's and those of q and k
    if name == "embed":
        return normal(1.0)
    if last in ("lq1", "lk1", "lq2", "lk2"):
        return normal(0.6 / shape[0] ** 0.25)           # dot products of order a third
    if last == "correction":
        return normal(0.25)
    if ".hc" in name and last == "mix":
        return torch.eye(shape[0]) * 0.8 + normal(0.25)
    if ".hc" in name and last == "in":
        return normal(0.3, 1.0 / shape[0] ** 0.5)
    if ".hc" in name and last == "out":
        return normal(0.4, 0.8)
    fan_in = shape[-1]
    if last == "router":
        return normal(3.0 / fan_in ** 0.5)
    if name.endswith((".mix.q", ".mix.k")):
        return normal(2.0 / fan_in ** 0.5)
    if last in ("gate", "up"):
        return normal(1.6 / fan_in ** 0.5)
    return normal(1.3 / fan_in ** 0.5)


def write_model(config: dict, out_dir: str, seed: int, overrides=None) -> str:
    """config.json and model.safetensors (bfloat16) for a Lagulorn configuration; ``overrides`` name -> tensor."""
    arch, cfg = parse_config(config)
    expected = Model(arch.model_spec(cfg)).expected_tensors()
    gen = torch.Generator().manual_seed(seed)
    tensors = {}
    for name, ps in expected.items():
        t = lively_tensor(name, tuple(ps.shape), gen)
        if overrides and name in overrides:
            t = overrides[name].reshape(ps.shape).float()
        tensors[name] = t.to(torch.bfloat16)
    os.makedirs(out_dir, exist_ok=True)
    write_safetensors(os.path.join(out_dir, "model.safetensors"), tensors)
    with open(os.path.join(out_dir, "config.json"), "w") as f:
        json.dump(arch.config_to_dict(cfg), f)
    return out_dir


@functools.lru_cache(maxsize=None)
def lagulorn_dir(which: str, seed: int = 0) -> str:
    return write_model(preset(f"lagulorn-tiny-{which}"), os.path.join(_root(), f"{which}_{seed}"), seed)
