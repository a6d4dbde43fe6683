"""Dense feed-forward without a gate: down(act(up(x))), act a gelu (erf or tanh form) or silu, with or without biases."""

from __future__ import annotations

from typing import Dict, Optional

import torch

from yalis_b200.config.spec import PartSpec
from yalis_b200.ops.elementwise import ACTIVATIONS, activation
from .base import FeedForward, NormedSum, ParamSpec, Projected, register_part


class DenseFeedForward(FeedForward, Projected):
    """Parameters: ``hidden_size``, ``intermediate_size``, ``activation`` (``gelu_erf`` by default,
    ``gelu_tanh`` or ``silu``), ``bias`` (both matrices have one; the inner one is added by the activation's kernel, the
    outer one by the pass that adds the result to the stream).  The activation is computed in float32."""

    def __init__(self, spec: PartSpec):
        super().__init__(spec)
        self.hidden = int(spec.params["hidden_size"])
        self.inter = int(spec.params["intermediate_size"])
        self.act = str(spec.params.get("activation", "gelu_erf"))
        if self.act not in ACTIVATIONS:
            raise ValueError(f"unknown activation {self.act!r} (one of {', '.join(ACTIVATIONS)})")
        self.bias = bool(spec.params.get("bias", False))
        self.shares_projections = not self.bias
        self.hidden_width = self.inter
        self.up_bias: Optional[torch.Tensor] = None
        self.down_bias: Optional[torch.Tensor] = None
        self.w_up: Optional[torch.Tensor] = None
        self.w_down: Optional[torch.Tensor] = None

    def param_specs(self) -> Dict[str, ParamSpec]:
        specs = {"up_proj": ParamSpec((self.inter, self.hidden)), "down_proj": ParamSpec((self.hidden, self.inter))}
        if self.bias:
            specs["up_bias"] = ParamSpec((self.inter,), init="zeros", keep_float32=True)
            specs["down_bias"] = ParamSpec((self.hidden,), init="zeros", keep_float32=True)
        return specs

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.w_up = tensors["up_proj"].contiguous()
        self.w_down = tensors["down_proj"].contiguous()
        if self.bias:
            self.up_bias, self.down_bias = tensors["up_bias"].contiguous(), tensors["down_bias"].contiguous()

    def in_weight(self) -> torch.Tensor:
        return self.w_up

    def out_weight(self) -> torch.Tensor:
        return self.w_down

    def release_projections(self) -> None:
        if self.bias:
            raise ValueError("an arrangement that adds several output products into one cannot carry this part's output bias")
        self.w_up = self.w_down = None

    def mix(self, z: torch.Tensor, ctx, cache, y: torch.Tensor) -> None:
        activation(z, self.act, out=y, bias=self.up_bias)

    def forward(self, x: torch.Tensor, ctx) -> torch.Tensor:
        out = self.project_and_mix(x, ctx, None)
        return NormedSum(out, bias=self.down_bias) if self.bias else out

    def capture_key(self, host):
        return None


register_part("feed_forward", "dense", DenseFeedForward)
