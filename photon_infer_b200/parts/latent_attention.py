"""Attention over a cached latent (multi-head latent attention).

Queries go through a latent of their own: ``c_q = rmsnorm(W_dq h)``, ``q = W_uq c_q``, every head laid out as
``[dim unrotated | rot_dim rotated]``.  Keys and values come from ONE latent per token: ``W_dkv h`` has
``kv_rank + rot_dim`` rows, the first ``kv_rank`` (RMS-normed) are the latent ``c``, the last ``rot_dim`` (not
normed, rotated by the token's position) are a key part ``k_r`` that all heads share.  Head ``h`` has the
unrotated key ``W_uk[h] c`` and the value ``W_uv[h] c``; its score against a key is
``(q_u . W_uk[h] c + q_r . k_r) * scale``, softmax over the keys up to the token's own position.

Only ``[c ; k_r]`` is cached, one row of ``kv_rank + rot_dim`` numbers per token and layer, and neither keys nor
values are ever formed: ``q_u . W_uk[h] c = (W_uk[h]^T q_u) . c``, so the queries are taken into the latent space
once per step (``head_linear``), attention runs with ONE key/value head whose key rows are ``[c ; k_r]`` and
whose values are the first ``kv_rank`` numbers of the same rows, and ``W_uv[h]`` is applied to the head's
weighted sum of latents.  Decoded tokens, short portions and the float32 run take this form.  A long bfloat16 portion reads
every cached row many times, so it expands the rows it sees once instead (one product with ``[W_uk; W_uv]``) and attends
with heads of ``dim + rot_dim`` and ``vdim`` numbers on the tcgen05 tensor cores (``csrc/attention_latent_tc.cu``), where
that is the smaller amount of arithmetic.  A step may hold both kinds side by side.

The rotation turns the first ``rot_dims`` numbers of the rotated part by the angle ``position * base^(-2i / rot_dims)``,
feature ``i`` paired with ``i + rot_dims / 2`` or (``rot_interleaved``) feature ``2i`` with ``2i + 1``; the rest passes
unchanged.

Variants, all by parameter.  ``window``: a token sees its own row and the ``window - 1`` before it.  ``output_gate``: the
concatenated heads are multiplied by ``sigmoid(W_g h)`` before ``W_o`` (``head``: ``W_g`` has one row per head, whose gate
multiplies all of the head's output); ``W_g``'s rows ride in the fused down-projection.  ``sink``: the softmax of head ``h``
has one more key with no value and the learned score ``sink[h]``, which is not scaled: ``exp(sink[h])`` joins the denominator.
``rot_scaling`` stretches the rotation's frequencies (``parts/rope.py``).
``own_kv`` False: the layer has no ``W_dkv``; it reads the cached rows of an earlier layer (the run list's ``kv_from``) with
its own queries, ``W_uk``, ``W_uv``, window and everything else.  ``cache_window``: how many rows the cache must keep for
this layer AND the layers that read its pages (``"own"``: this layer's window; None: everything).
"""
from __future__ import annotations

import os
from typing import Dict, List, Optional

import torch

from ..kernels import ops
from .base import LayerCache, Mixer, PagedCacheSpec, StepContext, TensorSpec
from .linear import project
from .registry import register_mixer
from .rope import scaled_frequencies


class LatentAttention(Mixer):
    kernel_modules = ("latent", "attention")

    def __init__(self, hidden_size: int, heads: int, dim: int, rot_dim: int, vdim: int, kv_rank: int, q_rank: int,
                 scale: float, eps: float, rot_base: float, rot_dims: Optional[int] = None, window: Optional[int] = None,
                 rot_interleaved: bool = False, cache_window="own", own_kv: bool = True, output_gate=False, sink: bool = False,
                 rot_scaling: Optional[dict] = None):
        self.hidden_size, self.heads, self.dim, self.rot_dim, self.vdim = hidden_size, heads, dim, rot_dim, vdim
        self.kv_rank, self.q_rank = kv_rank, q_rank
        self.scale, self.eps = float(scale), float(eps)
        self.rot_base = float(rot_base)
        self.rot_dims = rot_dim if rot_dims is None else int(rot_dims)
        if self.rot_dims % 2 or not 0 <= self.rot_dims <= rot_dim:
            raise ValueError("the rotated features must be an even number of at most rot_dim")
        self.rot_interleaved = bool(rot_interleaved)
        self.window = int(window) if window else None
        self.cache_window = self.window if cache_window == "own" else (int(cache_window) if cache_window else None)
        if self.cache_window is not None and (self.window is None or self.window > self.cache_window):
            raise ValueError("the cache must keep at least the rows that this layer's window sees")
        if output_gate not in (False, True, "head"):
            raise ValueError("output_gate is False, True (a number per output) or 'head' (a number per head)")
        self.own_kv, self.output_gate, self.sink = bool(own_kv), output_gate, bool(sink)
        self.gate_width = 0 if not output_gate else heads * (vdim if output_gate is True else 1)
        self.sinks: Optional[torch.Tensor] = None
        self.width = kv_rank + rot_dim          # one cached row
        self.inv_freq_host = scaled_frequencies(self.rot_dims, self.rot_base, rot_scaling).to(torch.float32)
        self.inv_freq: Optional[torch.Tensor] = None
        self.w_down = self.w_uq = self.w_absorb = self.w_uv = self.w_kv = self.w_o = None
        self.q_norm = self.kv_norm = None

    def required_kernels(self, dtype):
        mods = list(self.kernel_modules)
        if dtype == torch.bfloat16:
            mods.extend(["gemm_skinny", "gemm_tc", "gemm_tc2"])
        if self.output_gate:
            mods.append("elementwise")
        defines = self._prompt_defines(dtype)
        if defines is not None:
            mods.append(("attention_latent_tc", defines))
        return mods

    def _prompt_defines(self, dtype):
        return ops.latent_prompt_defines(dtype, self.dim, self.rot_dim, self.vdim, self.kv_rank) if USE_EXPANDED_PROMPTS else None

    def tensor_specs(self) -> List[TensorSpec]:
        H, n, d, r, v = self.hidden_size, self.heads, self.dim, self.rot_dim, self.vdim
        specs = [TensorSpec("dq", (self.q_rank, H)), TensorSpec("dq.norm", (self.q_rank,), role="vector", init="norm"),
                 TensorSpec("uq", (n * (d + r), self.q_rank))]
        if self.own_kv:
            specs += [TensorSpec("dkv", (self.kv_rank + r, H)), TensorSpec("dkv.norm", (self.kv_rank,), role="vector", init="norm")]
        specs += [TensorSpec("uk", (n * d, self.kv_rank)), TensorSpec("uv", (n * v, self.kv_rank))]
        if self.output_gate:
            specs.append(TensorSpec("g", (self.gate_width, H)))
        if self.sink:
            specs.append(TensorSpec("sink", (n,), role="vector", init="normal"))
        return specs + [TensorSpec("o", (H, n * v))]

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        n, d, v = self.heads, self.dim, self.vdim
        down = [tensors["dq"]] + ([tensors["dkv"]] if self.own_kv else []) + ([tensors["g"]] if self.output_gate else [])
        if self.gate_width % 8:                 # rows of the product stay a multiple of 16 bytes
            down.append(torch.zeros((-self.gate_width % 8, self.hidden_size), dtype=down[0].dtype, device=down[0].device))
        self.w_down = torch.cat(down, dim=0).contiguous()                                 # h is read once
        self.sinks = tensors["sink"].to(torch.float32).contiguous() if self.sink else None
        self.q_norm = tensors["dq.norm"].contiguous()
        self.kv_norm = tensors["dkv.norm"].contiguous() if self.own_kv else None
        self.w_uq = tensors["uq"].contiguous()
        # W_uk[h]^T as the [out, in] matrix of the product that takes a head's unrotated query into the latent space
        self.w_absorb = tensors["uk"].view(n, d, self.kv_rank).transpose(1, 2).contiguous()   # [heads, kv_rank, dim]
        self.w_kv = torch.cat([tensors["uk"], tensors["uv"]], dim=0).contiguous()             # expands a latent into keys and values
        self.w_uv = self.w_kv[n * d:].view(n, v, self.kv_rank)                                # [heads, vdim, kv_rank], the same memory
        self.w_o = tensors["o"].contiguous()
        self.inv_freq = self.inv_freq_host.to(self.w_o.device)

    def weight_bytes(self) -> int:
        ws = (self.w_down, self.w_uq, self.w_absorb, self.w_uv, self.w_o)
        return sum(w.numel() * w.element_size() for w in ws)

    def cache_spec(self) -> Optional[PagedCacheSpec]:
        return PagedCacheSpec(1, self.width, self.cache_window, values=False)

    def forward(self, h: torch.Tensor, ctx: StepContext, cache: LayerCache) -> torch.Tensor:
        T = h.shape[0]
        n, d, r, kr = self.heads, self.dim, self.rot_dim, self.kv_rank
        group = ctx.groups[cache.group]
        down = project(h, self.w_down)                                   # [T, q_rank (+ kv_rank + rot) (+ gate)]
        at = self.q_rank + (self.width if self.own_kv else 0)
        gate = down[:, at:at + self.gate_width] if self.output_gate else None
        store = self.own_kv and not cache.shared
        cq = torch.empty((T, self.q_rank), dtype=h.dtype, device=h.device)
        ops.latent_prep(down, self.q_rank, kr, r, self.rot_dims, self.q_norm, self.kv_norm, self.eps, ctx.positions,
                        self.inv_freq, group.slot_mapping if store else None, cq, cache.k if store else None, ctx.error_flag,
                        interleaved=self.rot_interleaved)
        q = project(cq, self.w_uq)                                       # [T, heads * (dim + rot)]
        o = torch.empty((T, n * self.vdim), dtype=h.dtype, device=h.device)
        lens = list(ctx.host_query_lens) or [T]
        expanded = self._expanded_requests(ctx, lens, h.dtype)
        if expanded:
            self._expanded(q, o, gate, ctx, cache, lens, expanded)
        # neighbouring requests that are not expanded run together
        s = t = 0
        while s < len(lens):
            if s in expanded:
                t += lens[s]
                s += 1
                continue
            s0, t0 = s, t
            while s < len(lens) and s not in expanded:
                t += lens[s]
                s += 1
            self._absorbed(q[t0:t], o[t0:t], None if gate is None else gate[t0:t], ctx, cache, s0, s, t0, lens)
        return project(o, self.w_o)

    def _absorbed(self, q, o, gate, ctx: StepContext, cache: LayerCache, s0: int, s1: int, t0: int, lens) -> None:
        """Requests ``s0 .. s1 - 1`` (tokens from ``t0`` on) in the latent space: queries in, weighted latents out."""
        T, n, d, r, kr = q.shape[0], self.heads, self.dim, self.rot_dim, self.kv_rank
        q_lat = torch.empty((T, n, self.width), dtype=q.dtype, device=q.device)
        positions = ctx.positions[t0:t0 + T]
        if ops.latent_absorb_supported(q, d, r):        # few rows: both parts of the queries in one launch
            ops.latent_absorb(q, self.w_absorb, d, r, self.rot_dims, positions, self.inv_freq, q_lat, interleaved=self.rot_interleaved)
        else:
            ops.head_linear(q.view(T, n, d + r)[:, :, :d], self.w_absorb, q_lat[:, :, :kr])
            ops.latent_q_rope(q, n, d, r, self.rot_dims, positions, self.inv_freq, q_lat, kr, interleaved=self.rot_interleaved)
        o_lat = torch.empty((T, n * kr), dtype=q.dtype, device=q.device)
        self.attend(q_lat, o_lat, ctx, cache, s0, s1, t0, lens)
        ops.head_linear(o_lat.view(T, n, kr), self.w_uv, o.view(T, n, self.vdim), gate=gate)

    # ------------------------------------------------------------------ long portions: keys and values formed once
    def _first_seen(self, start: int) -> int:
        return 0 if self.window is None else max(0, start + 1 - self.window)

    def _expanded_requests(self, ctx: StepContext, lens, dtype):
        """The requests of the step whose rows are expanded into keys and values: those for which that is less arithmetic
        than attending to the latents themselves, as long as the expanded rows fit ``EXPANDED_BYTES``."""
        if self._prompt_defines(dtype) is None or not ctx.host_query_lens or max(lens) < LIBRARY_MIN_TOKENS:
            return {}
        n, d, r, v, kr = self.heads, self.dim, self.rot_dim, self.vdim, self.kv_rank
        pad = lambda x: -(-x // 64) * 64
        chosen, total = {}, 0
        for s, m in enumerate(lens):
            if m < LIBRARY_MIN_TOKENS:
                continue
            start = ctx.host_start_positions[s]
            rows = start + m - self._first_seen(start)
            pairs = m * start + m * (m + 1) // 2 if self.window is None else m * min(self.window, start + m)
            expand = rows * kr * (d + v) + pairs * (pad(d) + pad(r) + pad(v))
            if expand > pairs * (self.width + kr) + m * kr * (d + v) or (total + rows) * n * (d + v) * 2 > EXPANDED_BYTES:
                continue
            chosen[s] = (start, rows)
            total += rows
        return chosen

    def _expanded(self, q, o, gate, ctx: StepContext, cache: LayerCache, lens, requests) -> None:
        T, n, d, r, kr = q.shape[0], self.heads, self.dim, self.rot_dim, self.kv_rank
        total = sum(rows for _, rows in requests.values())
        latents = torch.empty((total, self.width), dtype=q.dtype, device=q.device)
        table = ctx.groups[cache.group].block_table
        seqs, t, row = [], 0, 0
        for s, m in enumerate(lens):
            if s in requests:
                start, rows = requests[s]
                base = self._first_seen(start)
                ops.gather_rows(cache.k, table[s], rows, ctx.error_flag, first=base, out=latents[row:row + rows])
                seqs.append((t, m, start, base, row))
                row += rows
            t += m
        kv = project(latents[:, :kr], self.w_kv)                         # [rows, heads * (dim + vdim)]
        q_rot = torch.empty((T, n, r), dtype=q.dtype, device=q.device)
        ops.latent_q_rope(q, n, d, r, self.rot_dims, ctx.positions, self.inv_freq, q_rot, 0, interleaved=self.rot_interleaved)
        # in the epilogue: one number per head, or gates that can be read 16 bytes at a time
        fused = gate is not None and (self.output_gate == "head" or (gate.data_ptr() % 16 == 0 and gate.stride(0) % 8 == 0))
        ops.latent_prompt_attention(q, q_rot, kv, latents[:, kr:], o, seqs, n, d, r, self.vdim, self.window, self.scale,
                                    ctx.error_flag, gate=gate if fused else None, sink=self.sinks)
        if gate is not None and not fused:
            for t, m, *_ in seqs:
                ops.gate_mul(o[t:t + m], gate[t:t + m])

    # ------------------------------------------------------------------ attention over the latents themselves
    def attend(self, q_lat: torch.Tensor, o_lat: torch.Tensor, ctx: StepContext, cache: LayerCache, s0: int = 0,
               s1: Optional[int] = None, t0: int = 0, lens=None) -> None:
        """Requests ``s0 .. s1 - 1`` of the step, whose tokens (from token ``t0`` of the step on) ``q_lat`` and ``o_lat`` hold.
        Decoded tokens, short portions and the float32 run: the paged kernel, whose sums depend only on a token's
        position.  A long bfloat16 portion: the request's cached rows are gathered into one matrix and attention
        is three steps per slab of queries, scores = Q C^T (library product, 32-bit out), a causal softmax over the
        rows, and P C[:, :kv_rank] (library product); a slab starts at the first and ends at the last row its queries
        may see."""
        T = q_lat.shape[0]
        group = ctx.groups[cache.group]
        lens = (list(ctx.host_query_lens) or [T]) if lens is None else lens
        t = 0
        pending = None                                  # a run of neighbouring requests for the paged kernel
        for s in range(s0, len(lens) if s1 is None else s1):
            m = lens[s]
            if q_lat.dtype == torch.bfloat16 and m >= LIBRARY_MIN_TOKENS:
                if pending is not None:
                    self._paged(q_lat, o_lat, ctx, cache, pending, t, t0)
                    pending = None
                self._dense(q_lat[t:t + m], o_lat[t:t + m], ctx.host_start_positions[s], group.block_table[s], cache, ctx)
            elif pending is None:
                pending = t
            t += m
        if pending is not None:
            self._paged(q_lat, o_lat, ctx, cache, pending, T, t0)

    def _paged(self, q_lat, o_lat, ctx, cache, a: int, b: int, t0: int) -> None:
        n = self.heads
        token_seq, positions = ctx.token_seq[t0 + a:t0 + b], ctx.positions[t0 + a:t0 + b]
        group = ctx.groups[cache.group]
        q2 = q_lat[a:b].view(b - a, n * self.width)
        shares = ops.latent_decode_shares(ctx.max_context_len, self.window)
        if ops.latent_decode_supported(q2, self.width, self.kv_rank) \
                and (b - a) * n * shares * (self.kv_rank + 2) * 4 <= DECODE_SHARES_BYTES:
            # bfloat16 with widths that fit the tensor cores' tiles: one block per token and 64 cached rows
            ops.latent_decode_attention(q2, o_lat[a:b], cache.k, group.block_table, token_seq, positions, n,
                                        self.width, self.kv_rank, self.scale, ctx.max_context_len, ctx.error_flag,
                                        window=self.window, sink=self.sinks)
            return
        splits = 1
        if q_lat.dtype == torch.bfloat16:
            # few tokens with long contexts: share every token's key tiles out until the GPU is full (the float32 run keeps
            # one block per token, whose sums depend on the token's position alone)
            chunks = -(-n // max(1, min(n, 4096 // self.width)))
            seen = max(ctx.max_context_len, 1) if self.window is None else min(max(ctx.max_context_len, 1), self.window + 31)
            tiles = -(-seen // 32)
            splits = max(1, min(4 * ops.sm_count(q_lat.device) // max(1, (b - a) * chunks), tiles, 64))
        ops.paged_attention(q_lat[a:b].view(b - a, n * self.width), o_lat[a:b], cache.k, cache.k, group.block_table,
                            token_seq, positions, n, 1, self.width, self.window, self.scale,
                            ctx.error_flag, value_dim=self.kv_rank, splits=splits, sink=self.sinks)

    def _dense(self, q, o, start: int, table: torch.Tensor, cache: LayerCache, ctx: StepContext) -> None:
        m, n, kr = q.shape[0], self.heads, self.kv_rank
        end, w = start + m, self.window
        first_seen = 0 if w is None else max(0, start + 1 - w)       # of the portion's first token
        # the library's products want rows of 16 bytes: the matrix starts and ends at multiples of eight positions (zero
        # rows where no token of the portion sees, which the softmax leaves out)
        base = first_seen // 8 * 8
        rows = ops.gather_rows(cache.k, table, -(-end // 8) * 8 - base, ctx.error_flag, first=base, valid=(first_seen, end))
        # a window: short slabs, so that few of a slab's products fall outside its tokens' windows
        most = m if w is None else max(64, -(-w // 256) * 64)
        t0 = 0
        while t0 < m:
            lo = 0 if w is None else max(0, start + t0 + 1 - w) // 8 * 8       # the first row that the slab's first token sees
            keys = end - lo if w is None else min(end - lo, w + most + 8)
            t1 = min(m, t0 + max(1, min(most, SCORE_BYTES // (4 * n * keys))))
            hi = -(-(start + t1) // 8) * 8                                     # behind the last row that its last token sees
            part = rows[lo - base:hi - base]
            scores = torch.mm(q[t0:t1].view((t1 - t0) * n, self.width), part.t(), out_dtype=torch.float32)
            probs = torch.empty(scores.shape, dtype=q.dtype, device=q.device)
            ops.causal_softmax_rows(scores, probs, n, start + t0, self.scale, first_key=lo, window=w, sink=self.sinks)
            torch.mm(probs, part[:, :kr], out=o[t0:t1].view((t1 - t0) * n, kr))
            t0 = t1


#: The tensor-core decode kernel leaves one share per token, head and 64 rows of the longest context the step allows;
#: beyond this many bytes of shares the step takes the general kernel, which bounds its shares by the GPU's size.
DECODE_SHARES_BYTES = 512 << 20
#: A request that brings at least this many tokens to a bfloat16 step does not take the paged kernel: its rows are expanded
#: or attended to by products and a softmax.
LIBRARY_MIN_TOKENS = 32
#: Bytes of 32-bit scores held at a time on that path (the queries are cut into slabs that fit).
SCORE_BYTES = 64 << 20

#: Long portions over expanded rows (``PHOTON_LATENT_EXPAND=0``: by products and a softmax over the latents).
USE_EXPANDED_PROMPTS = os.environ.get("PHOTON_LATENT_EXPAND", "1") != "0"
#: Most bytes of expanded keys and values a step may form in a layer.
EXPANDED_BYTES = 2 << 30

register_mixer("latent_attention", LatentAttention)
