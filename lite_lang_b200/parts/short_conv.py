"""Short causal convolutions over time, one filter of ``taps`` weights a channel (the last one for the token itself), no
bias: conv(u)_t = sum_j w[:, j] u_(t - taps + 1 + j), zeros before the request's start.

``ShortConv`` is a mixer of its own: what a sublayer reads, h, becomes h + conv(h) (tensor ``tensor`` [hidden, taps]
under the prefix).  Behind a norm over a float32 residual it runs in the norm's pass (``after``); behind any other norm
as a kernel of its own (``forward``).

``ConvMemory`` and ``PagedMemory`` are members of a composite mixer that needs two kinds of memory, the pages of its
keys and values and the record of a convolution (``parts/modulated_attention.py``).

A request's last taps - 1 inputs live in its record of the cache manager's state pool (float32, two halves written in
turn, see ``csrc/short_conv.cu``), so a request goes on in a later step from where it stopped.
"""

from __future__ import annotations

from typing import Dict

import torch

from .. import ops
from ..config.spec import PartSpec
from .base import Mixer, PagedKVNeed, StateNeed, TensorDecl, register_part


def filters(w: torch.Tensor, device) -> torch.Tensor:
    """A checkpoint's [channels, taps] as the kernels read it: float32 [taps, channels]."""
    return w.to(torch.float32).t().contiguous().to(device)


class ConvMemory(Mixer):
    """The record of a convolution over ``channels`` channels."""

    def __init__(self, taps: int, channels: int, prefix: str = ""):
        super().__init__(PartSpec("short_conv_memory", {}, prefix))
        self.taps, self.channels = int(taps), int(channels)

    def cache_need(self):
        return StateNeed((ops.conv_record_floats(self.taps, self.channels),), "float32")


class PagedMemory(Mixer):
    """Pages of keys and values."""

    def __init__(self, need: PagedKVNeed, prefix: str = ""):
        super().__init__(PartSpec("paged_memory", {}, prefix))
        self.need = need

    def cache_need(self):
        return self.need


class ShortConv(Mixer):
    def __init__(self, spec: PartSpec):
        super().__init__(spec)
        self.hidden_size = int(spec.params["hidden_size"])
        self.taps = int(spec.params["taps"])
        self.tensor = str(spec.params.get("tensor", "weight"))
        if not (1 <= self.taps <= 64):
            raise ValueError("short_conv: 1 to 64 taps are built")
        self.weight = None

    def tensors(self) -> Dict[str, TensorDecl]:
        return {self.tensor: TensorDecl((self.hidden_size, self.taps), "bias", std=0.3)}

    def load(self, fetch, dtype, device) -> None:
        self.weight = filters(fetch(self.tensor), device)

    def weight_bytes(self) -> int:
        return self.weight.numel() * 4

    def kernel_libraries(self):
        return ("core", "short_conv")

    def cache_need(self):
        return StateNeed((ops.conv_record_floats(self.taps, self.hidden_size),), "float32")

    def forward(self, x, step, cache):
        out = torch.empty((x.shape[0], self.hidden_size), dtype=x.dtype, device=x.device)
        ops.short_conv(out, x, self.weight, cache.state, step, add_input=True, write_state=cache.writable)
        return out

    def after(self, norm, residual, delta, step, cache):
        """(residual rows, h + conv(h)) with h = ``norm`` of the residual and what is pending."""
        if hasattr(norm, "add_conv_forward"):
            return norm.add_conv_forward(residual, delta, self.weight, cache, step)
        return residual, self.forward(norm.add_forward(residual, delta), step, cache)


register_part("mixer", "short_conv", ShortConv)
