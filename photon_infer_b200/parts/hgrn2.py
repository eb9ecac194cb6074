"""Linear attention whose forget gate also decides what is written (the HGRN2 cell): a recurrent mixer with one matrix
of state per head.

``q = silu(W_q h)`` (heads x dim), ``v = W_v h`` (heads x vdim), and per head and channel a forget gate between a lower bound
and 1, ``f = l + (1 - l) sigmoid(W_f h + b)``, ``l`` a stored vector.  Per head

    S_t = diag(f_t) S_(t-1) + (1 - f_t) v_t^T,        o_t = S_t^T q_t,

so every row of the state is a running mean of the values.  Each head's ``o`` is RMS-normed over vdim with a weight that the
heads share; the heads are concatenated and projected by ``W_o``.  The state starts at zero, is 32-bit, and lives in the
request's state slot between steps; everything between the two products is 32-bit.

Kernels of a step: ONE product ``[q | f | v]`` with 32-bit rows; the recurrence over the tokens of the step (``linrec.cu``),
which forms ``silu(q)`` and the gates itself for few tokens and gets them from one pass over all tokens of a long portion; the
norm (``row_norms.cu``); the output product.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..kernels import ops
from .base import LayerCache, Mixer, StateSpec, StepContext, TensorSpec
from .linear import project
from .registry import register_mixer

DEFAULT_NAMES = {"q": "q", "f": "f", "f_bias": "f.b", "lower": "lower", "v": "v", "norm": "norm", "o": "o"}


class Hgrn2Mixer(Mixer):
    kernel_modules = ("linrec", "row_norms")
    state_skips_negative_slots = True

    def __init__(self, hidden_size: int, heads: int, dim: int, vdim: int, eps: float, names: Optional[Dict[str, str]] = None):
        self.hidden_size, self.heads, self.dim, self.vdim = hidden_size, heads, dim, vdim
        self.eps = float(eps)
        self.names = dict(DEFAULT_NAMES, **(names or {}))
        self.w_in = self.w_o = self.f_bias = self.lower = self.norm = None

    def required_kernels(self, dtype):
        return list(self.kernel_modules) + (["gemm_skinny", "gemm_tc", "gemm_tc2"] if dtype == torch.bfloat16 else [])

    def tensor_specs(self) -> List[TensorSpec]:
        n, H = self.names, self.hidden_size
        nd, nv = self.heads * self.dim, self.heads * self.vdim
        vec = lambda name, size, init="normal": TensorSpec(n[name], (size,), role="vector", init=init)
        return [TensorSpec(n["q"], (nd, H)), TensorSpec(n["f"], (nd, H)), TensorSpec(n["v"], (nv, H)), TensorSpec(n["o"], (H, nv)),
                vec("f_bias", nd), vec("lower", nd, "unit"), vec("norm", self.vdim, "norm")]

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        n = self.names
        f32 = lambda name: tensors[n[name]].to(torch.float32).contiguous()
        self.w_in = torch.cat([tensors[n[x]] for x in ("q", "f", "v")], dim=0).contiguous()
        self.w_o = tensors[n["o"]].contiguous()
        self.f_bias, self.lower = f32("f_bias"), f32("lower")
        self.norm = f32("norm").repeat(self.heads)      # the heads share it: one part of the row each

    def weight_bytes(self) -> int:
        return (self.w_in.numel() + self.w_o.numel()) * self.w_in.element_size()

    def state_spec(self) -> Optional[StateSpec]:
        return StateSpec((self.heads * self.dim * self.vdim,), torch.float32)

    def forward(self, h: torch.Tensor, ctx: StepContext, cache: LayerCache) -> torch.Tensor:
        T, H = h.shape[0], self.heads
        nd, nv = H * self.dim, H * self.vdim
        rows = project(h, self.w_in, out_dtype=torch.float32)       # [q | f | v]
        q, k, v = rows[:, :nd], rows[:, nd:2 * nd], rows[:, 2 * nd:]
        bias, lower = self.f_bias, self.lower
        if max(list(ctx.host_query_lens) or [T]) >= GATES_MIN_TOKENS:
            y = torch.empty((T, 2 * nd), dtype=torch.float32, device=h.device)
            ops.linrec_gates(q, k, bias, lower, y[:, :nd], y[:, nd:])
            q, k, bias, lower = y[:, :nd], y[:, nd:], None, None
        o = torch.empty((T, nv), dtype=torch.float32, device=h.device)
        ops.linrec("forget_write", q, k, v, None, None, bias, lower, None, 0.0, 1.0, ctx.cu_tokens, ctx.state_slots, cache.state, o,
                   ctx.num_seqs, H, H, self.dim, self.vdim, ctx.error_flag)
        out = torch.empty((T, nv), dtype=h.dtype, device=h.device)
        ops.group_rmsnorm(o, self.norm, self.eps, H, out=out)
        return project(out, self.w_o)


#: A step in which some request brings at least this many tokens forms the gates in a pass of their own.
GATES_MIN_TOKENS = 32

register_mixer("hgrn2", Hgrn2Mixer)
