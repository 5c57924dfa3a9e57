"""Grouped-query softmax attention that knows positions only through a learned bias by distance.

``q``, ``k``, ``v`` and the output projection have biases; every query and key head is divided by its root mean square
(no weight, eps inside the root); the score is ``(q . k) * scale + rel[bucket(i - j), head]``; a query at position i sees
the keys j <= i with ``i - j < window`` or ``j < keep_first``; the softmax's denominator also holds ``exp(sink[head])``.
``value_mix``: the values of every layer that mixes but the first such layer are ``(1 - lam) v + lam v_first`` with
``v_first`` that first layer's values of the same token (the mixed ones are cached).  One fused product ``[q | k | v]``,
one kernel that adds biases, norms, mixes and stores, one attention kernel, one output product
(``csrc/attention_distance.cu``, ``csrc/attention_distance_mma.cu``).
"""

from __future__ import annotations

import torch

from gllm_b200 import ops
from gllm_b200.ops import distance
from gllm_b200.parts.base import KVPageRequirement, Mixer, TensorExpectation, register_mixer

# the values of the first layer that mixes, kept for the later ones of the same step
FIRST_VALUES = "first_values"


@register_mixer("distance_attention")
class DistanceAttention(Mixer):
    graph_safe_portions = True

    def __init__(self, names, hidden_size: int, heads: int, kv_heads: int, dk: int, dv: int, scale: float, eps: float,
                 distance_max: float, window: int | None = None, keep_first: int = 0, value_mix: str | None = None,
                 bias_rows: int | None = None):
        """``names``: ``q``, ``k``, ``v``, ``o`` and their biases ``q_bias`` ..., ``rel``, ``sink`` and, with
        ``value_mix`` ("first" or "mixed"), ``mix``.  ``bias_rows``: rows of ``rel``; None takes them from the
        checkpoint's tensor."""
        super().__init__(names)
        if heads % kv_heads:
            raise ValueError("heads must be a multiple of kv_heads")
        if not (0 < dk <= 256 and 0 < dv <= 256):
            raise ValueError("the kernels take query, key and value heads up to 256 wide")
        if value_mix not in (None, "first", "mixed"):
            raise ValueError(f"unknown value mix {value_mix!r}")
        self.hidden_size, self.heads, self.kv_heads = int(hidden_size), int(heads), int(kv_heads)
        self.dk, self.dv = int(dk), int(dv)
        self.scale, self.eps, self.distance_max = float(scale), float(eps), distance_max
        self.window = int(window) if window else None
        self.keep_first = int(keep_first) if self.window else 0
        self.value_mix = value_mix
        self.bias_rows = int(bias_rows) if bias_rows is not None else None
        self.w_qkv = self.w_o = self.b_qkv = self.b_o = None
        self.bias: distance.DistanceBias | None = None
        self.lam = 0.0

    def kernel_needs(self):
        # the second holds the tensor-core kernels of bfloat16 runs, the third the one for longer portions
        wide = {"attention_prefill_tmem"} if self.dk == self.dv and self.dk in (64, 128) else set()
        return {"modules": {"attention_distance", "attention_distance_mma"} | wide}

    def kv_requirement(self):
        return KVPageRequirement(((self.kv_heads, self.dk), (self.kv_heads, self.dv)), self.window, self.keep_first)

    def expected_tensors(self):
        n, w = self.names, self.hidden_size
        rows = {"q": self.heads * self.dk, "k": self.kv_heads * self.dk, "v": self.kv_heads * self.dv}
        exp = {n[k]: TensorExpectation((r, w)) for k, r in rows.items()}
        exp |= {n[k + "_bias"]: TensorExpectation((r,), "bias") for k, r in rows.items()}
        exp[n["rel"]] = TensorExpectation((-1 if self.bias_rows is None else self.bias_rows, self.heads), "bias")
        exp[n["sink"]] = TensorExpectation((self.heads,), "bias")
        if self.value_mix is not None:
            exp[n["mix"]] = TensorExpectation((), "bias")
        exp[n["o"]] = TensorExpectation((w, self.heads * self.dv))
        exp[n["o_bias"]] = TensorExpectation((w,), "bias")
        return exp

    def load(self, get, dtype, device):
        n = self.names
        self.w_qkv = torch.cat([get(n[k], "matrix") for k in ("q", "k", "v")], 0).contiguous()
        self.b_qkv = torch.cat([get(n[k + "_bias"], "bias") for k in ("q", "k", "v")], 0).contiguous()
        self.w_o, self.b_o = get(n["o"], "matrix").contiguous(), get(n["o_bias"], "bias").contiguous()
        self.bias = distance.DistanceBias.build(get(n["rel"], "bias"), self.distance_max, get(n["sink"], "bias"))
        if self.value_mix is not None:
            self.lam = float(get(n["mix"], "bias"))

    def forward(self, x, ctx, cache):
        view = ctx.groups[cache.group]
        mix, first = distance.NO_MIX, None
        if self.value_mix == "first":
            mix = distance.FIRST
            first = torch.empty((x.shape[0], self.kv_heads * self.dv), dtype=x.dtype, device=x.device)
            ctx.shared[FIRST_VALUES] = first
        elif self.value_mix == "mixed":
            mix, first = distance.MIXED, ctx.shared[FIRST_VALUES]
        q = distance.distance_prep(ops.linear(x, self.w_qkv, split_ok=True), self.b_qkv, self.eps,
                                   view.slot_mapping if cache.writes else None, cache.pages, self.heads, self.kv_heads,
                                   self.dk, self.dv, cache.block_size, mix=mix, first=first, lam=self.lam)
        attn = distance.distance_attention(q, cache.pages, view.block_table, ctx.positions, ctx.token_row, self.bias,
                                           self.heads, self.kv_heads, self.dk, self.dv, cache.block_size, self.scale,
                                           window=self.window, keep_first=self.keep_first, batch=ctx)
        if ctx.takes_bias:
            return ops.Biased(ops.linear(attn, self.w_o, split_ok=True), self.b_o)
        return ops.linear(attn, self.w_o, bias=self.b_o)
