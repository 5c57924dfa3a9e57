"""Grouped-query softmax attention whose projections pass a short causal convolution over time, within chunks.

``q``, ``k`` and ``v`` have biases; every channel of the three is convolved over time with its own filter of ``taps``
taps (its last ``taps - 1`` inputs are the request's state); every query and key head is RMS-normed with one weight for
all query heads and one for all key heads; then queries and keys are rotated in neighbouring pairs.  A query at position
i sees the keys j <= i of its own chunk of ``chunk`` positions, counted from the sequence's start (None: all keys); the
score is ``(q . k) * scale``.  ``own_kv`` False: the layer has no key and value projections (nor their convolutions and
norms) and attends over the pages of the plan entry it reads (``PlanEntry.reads_cache_of``), with queries and a
convolution state of its own.  One fused product, one kernel that does everything up to the rotated queries and the stored
keys and values (``csrc/conv_qkv.cu``), the paged attention kernels of the plain attention, one output product.
"""

from __future__ import annotations

import torch

from gllm_b200 import ops
from gllm_b200.ops.conv_qkv import MAX_TAPS, conv_qkv
from gllm_b200.parts.attention import stored_head_width
from gllm_b200.parts.base import (
    POSITION_ENCODINGS,
    KVPageRequirement,
    Mixer,
    StateRequirement,
    TensorExpectation,
    build_part,
    register_mixer,
)


@register_mixer("conv_attention")
class ConvAttention(Mixer):
    graph_safe_portions = True
    keeps_own_states = True

    def __init__(self, names, hidden_size: int, heads: int, kv_heads: int, dk: int, dv: int, taps: int, scale: float,
                 eps: float, position=None, chunk: int | None = None, own_kv: bool = True):
        """``names``: ``q``, ``k``, ``v``, their ``*_bias`` and ``*_conv``, ``q_norm``, ``k_norm`` and ``o`` (without
        ``own_kv`` those of ``q`` and ``o`` alone).  ``position``: the PartSpec of an interleaved rotary encoding over
        ``dk`` columns."""
        super().__init__(names)
        if heads % kv_heads:
            raise ValueError("heads must be a multiple of kv_heads")
        if not 1 <= taps <= MAX_TAPS:
            raise ValueError(f"the convolution takes 1 to {MAX_TAPS} taps")
        if chunk is not None and chunk <= 0:
            raise ValueError("chunks have a positive number of positions")
        self.hidden_size, self.heads, self.kv_heads = int(hidden_size), int(heads), int(kv_heads)
        self.dk, self.dv, self.taps = int(dk), int(dv), int(taps)
        self.scale, self.eps = float(scale), float(eps)
        self.chunk = int(chunk) if chunk is not None else None
        self.own_kv = bool(own_kv)
        self.position = build_part(POSITION_ENCODINGS, position) if position is not None else None
        if self.position is not None and not getattr(self.position, "interleaved", False):
            raise ValueError("this attention takes a rotary encoding of neighbouring pairs (or none)")
        # keys and values are stored equally wide, at a width the tensor-core kernels take where there is one
        self.stored_dim = stored_head_width(self.dk, self.dv)
        self.w_in = self.b_in = self.conv_w = self.w_o = self.w_q_norm = self.w_k_norm = None

    def kernel_needs(self):
        return {"attention_head_dims": {self.stored_dim}, "modules": {"conv_qkv"}}

    def kv_requirement(self):
        shape = (self.kv_heads, self.stored_dim)
        return KVPageRequirement((shape, shape), chunks=() if self.chunk is None else (self.chunk,))

    def state_requirement(self):
        return None if self.taps == 1 else StateRequirement((self.taps - 1, sum(r for _, r in self._sections())))

    def _sections(self) -> list[tuple[str, int]]:
        out = [("q", self.heads * self.dk)]
        if self.own_kv:
            out += [("k", self.kv_heads * self.dk), ("v", self.kv_heads * self.dv)]
        return out

    def expected_tensors(self):
        n, exp = self.names, {}
        for s, rows in self._sections():
            exp[n[s]] = TensorExpectation((rows, self.hidden_size))
            exp[n[s + "_bias"]] = TensorExpectation((rows,), "bias")
            exp[n[s + "_conv"]] = TensorExpectation((rows, self.taps), "bias")
        exp[n["q_norm"]] = TensorExpectation((self.dk,), "vector")
        if self.own_kv:
            exp[n["k_norm"]] = TensorExpectation((self.dk,), "vector")
        exp[n["o"]] = TensorExpectation((self.hidden_size, self.heads * self.dv))
        if self.position is not None:
            exp.update(self.position.expected_tensors())
        return exp

    def load(self, get, dtype, device):
        n, sections = self.names, [s for s, _ in self._sections()]
        self.w_in = torch.cat([get(n[s], "matrix") for s in sections], 0).contiguous()
        self.b_in = torch.cat([get(n[s + "_bias"], "bias") for s in sections], 0).contiguous()
        self.conv_w = torch.cat([get(n[s + "_conv"], "bias") for s in sections], 0).t().contiguous()
        self.w_q_norm = get(n["q_norm"], "vector").contiguous()
        if self.own_kv:
            self.w_k_norm = get(n["k_norm"], "vector").contiguous()
        # zero columns for what the stored heads have behind the values' width
        w_o = get(n["o"], "matrix").view(self.hidden_size, self.heads, self.dv)
        self.w_o = torch.nn.functional.pad(w_o, (0, self.stored_dim - self.dv)).reshape(self.hidden_size, -1).contiguous()
        if self.position is not None:
            self.position.load(get, dtype, device)

    def forward(self, x, ctx, cache):
        view, pages = ctx.groups[cache.group], cache.kv_pages()
        inv_freq, rotary_dim, magnitude = None, 0, 1.0
        if self.position is not None:
            (inv_freq, rotary_dim, _), magnitude = self.position.rotary(), self.position.magnitude()
        q = conv_qkv(ops.linear(x, self.w_in, split_ok=True), self.b_in, self.conv_w, cache.state, self.w_q_norm,
                     self.w_k_norm, self.eps, inv_freq, rotary_dim, magnitude,
                     view.slot_mapping if cache.writes else None, pages, self.heads, self.kv_heads, self.dk, self.dv,
                     self.stored_dim, ctx, own_kv=self.own_kv)
        attn = ops.paged_attention(q, pages, view.block_table, ctx.positions, ctx.token_row, self.heads, self.scale,
                                   batch=ctx, chunk=self.chunk)
        return ops.linear(attn, self.w_o, split_ok=True, add_into=getattr(ctx, "residual_sink", None))
