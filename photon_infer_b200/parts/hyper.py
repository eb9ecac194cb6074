"""Connections between a layer's sublayers and several parallel residual streams (hyper-connections).

Instead of one residual stream there are ``S`` of them, all equal to the embedding output at the start.  A sublayer has
three small tensors: ``in [S]``, ``out [S]`` and ``mix [S, S]`` (indexed from, to).  It reads ``u = sum_s in[s] X_s`` through its
norm, and with its output ``y`` all streams are replaced at once: ``X_t <- sum_s mix[s, t] X_s + out[t] y``.  At the end
of the model the streams are summed.  With one stream and all weights 1 this is the ordinary residual sum.

The write of one sublayer and the read of the next are one kernel with the norm between them (``csrc/hyper.cu``), so a
token's streams are read and written once per sublayer; the output stays pending (``base.Connected``) until then.
"""
from __future__ import annotations

from typing import Dict, List

import torch

from .base import ConnectionPart, TensorSpec
from .registry import register_connection

#: streams that the kernel holds in registers
MAX_STREAMS = 16


class HyperConnection(ConnectionPart):
    kernel_modules = ("hyper",)

    def __init__(self, streams: int, names=("in", "out", "mix")):
        if not 1 <= streams <= MAX_STREAMS:
            raise ValueError(f"between one and {MAX_STREAMS} residual streams are supported, got {streams}")
        self.streams = int(streams)
        self.names = tuple(names)

    def tensor_specs(self) -> List[TensorSpec]:
        i, o, m = self.names
        S = self.streams
        return [TensorSpec(i, (S,), role="vector", init="norm"), TensorSpec(o, (S,), role="vector", init="norm"),
                TensorSpec(m, (S, S), role="vector", init="eye")]

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.w_in, self.w_out, self.mix = (tensors[n].to(torch.float32).contiguous() for n in self.names)

    def weight_bytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in (self.w_in, self.w_out, self.mix))


register_connection("hyper", HyperConnection)
