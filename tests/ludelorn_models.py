"""Small Ludelorn model folders for the tests, with weights that make every mechanism show.

The product's random-weights mode draws every matrix from N(0, 0.02) and sets norms, scales and decays to neutral values,
under which attention weights are nearly uniform, a far pooled block hardly counts and a forgotten bias does not show.
The folders made here draw matrices wide enough for peaked attention, norm numbers and layer scales away from one, sinks
and distance biases of both signs, step biases and decay logarithms that let a state live from one token to hundreds.
Names and shapes come from the model's own list of expected tensors; the values are this file's.
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
        _ROOT = tempfile.mkdtemp(prefix="yalis_b200_ludelorn_")
    return _ROOT


def lively_tensor(name: str, shape, gen: torch.Generator) -> torch.Tensor:
    def normal(std, mean=0.0):
        return mean + torch.randn(shape, generator=gen) * std

    last = name.split(".")[-1]
    if last in ("norm1", "norm2", "norm", "out", "D") or last in ("ls1", "ls2"):
        return normal(0.25, 1.0)                       # plain scales, one number or a vector
    if name == "embed":
        return normal(1.0)
    if last == "sink":
        return normal(1.5, 1.0)
    if last == "rel":
        return normal(1.5)
    if last == "dt_bias":
        return normal(1.0, -2.0)                       # step sizes around 0.1
    if last == "A_log":
        return normal(1.0)
    if last == "b":
        return normal(0.4)
    if last == "conv":
        return normal(0.6)
    fan_in = shape[-1]
    if last in ("q", "k"):
        return normal(2.5 / fan_in ** 0.5)
    if last in ("g", "up", "in"):
        return normal(1.6 / fan_in ** 0.5)
    return normal(1.3 / fan_in ** 0.5)


def write_model(config: dict, out_dir: str, seed: int, overrides=None) -> str:
    """config.json and model.safetensors (bfloat16) for a Ludelorn configuration; ``overrides`` name -> tensor.  The
    configuration written names no bucket counts: they are to be read off the tensors."""
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
    written = arch.config_to_dict(cfg)
    for layer in written["layers"]:
        layer["mixer"].pop("buckets", None)
    with open(os.path.join(out_dir, "config.json"), "w") as f:
        json.dump(written, f)
    return out_dir


@functools.lru_cache(maxsize=None)
def ludelorn_dir(which: str, seed: int = 0) -> str:
    return write_model(preset(f"ludelorn-tiny-{which}"), os.path.join(_root(), f"{which}_{seed}"), seed)
