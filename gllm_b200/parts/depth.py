"""Parts of layers that norm a sublayer's RESULT: ``x += norm_a(mixer(x + conv_a(x))); x += norm_b(ff(x + conv_b(x)))``,
after which the residual may be replaced by a weighted sum over the embedding output and all layers' results so far.

A sublayer reads the residual itself plus a causal convolution of it over time, one filter per channel
(``causal_conv``); nothing is normed on the way in.  The sublayer's result is not normed and added by a kernel of its own:
it travels on as ``ops.DepthPending`` and the next sublayer's kernel (``csrc/depth_conv.cu``) norms and adds it, averages
over the depth where a layer ends, convolves and rounds, in one pass; the model's final norm takes the last one.
"""

from __future__ import annotations

import dataclasses

from gllm_b200.ops import depth
from gllm_b200.parts.base import (Block, DepthAverage, InputConv, StateRequirement, TensorExpectation, register_block,
                                  register_depth_average, register_input_conv)


@register_input_conv("causal_conv")
class CausalConv(InputConv):
    graph_safe_portions = True

    def __init__(self, names, width: int, taps: int):
        super().__init__(names)
        self.width, self.taps = int(width), int(taps)
        if not 1 <= self.taps <= 16:
            raise ValueError("the convolution takes 1 to 16 taps")

    def kernel_needs(self):
        return {"modules": {"depth_conv"}}

    def state_requirement(self):
        return StateRequirement((self.taps - 1, self.width))

    def expected_tensors(self):
        return {self.names["weight"]: TensorExpectation((self.width, self.taps), "bias")}

    def load(self, get, dtype, device):
        self.weight = get(self.names["weight"], "bias").t().contiguous()


@register_depth_average("depth_average")
class WeightedDepthAverage(DepthAverage):
    """``streams``: how many there are, this layer's own result included."""

    graph_safe_portions = True

    def __init__(self, names, streams: int):
        super().__init__(names)
        self.streams = int(streams)

    def expected_tensors(self):
        return {self.names["weight"]: TensorExpectation((self.streams,), "vector")}

    def load(self, get, dtype, device):
        self.weight = get(self.names["weight"], "vector").contiguous()


@register_block("result_norm")
class ResultNormBlock(Block):
    """Both norms are of a kind that has ``depth_pending`` (the RMS norm).  A layer may have no feed-forward and no
    average over the depth."""

    graph_safe_portions = True
    part_kinds = {"mixer_conv": "input_conv", "mixer": "mixer", "mixer_norm": "norm",
                  "feed_forward_conv": "input_conv", "feed_forward": "feed_forward", "feed_forward_norm": "norm",
                  "depth_average": "depth_average"}
    optional_parts = frozenset({"feed_forward_conv", "feed_forward", "feed_forward_norm", "depth_average"})

    def block_states(self):
        convs = [self.mixer_conv] + ([self.feed_forward_conv] if self.feed_forward is not None else [])
        return tuple(c.state_requirement() for c in convs)

    def _mixer_view(self, cache):
        """``cache`` with the mixer's own states only (they come before the block's)."""
        view = getattr(cache, "mixer_view", None)
        if view is None:
            states = cache.states[:len(cache.states) - len(self.block_states())]
            view = cache.mixer_view = dataclasses.replace(cache, states=states, state=states[0] if states else None)
        return view

    def _input(self, conv, state, branch, resid, ctx):
        return depth.depth_conv(branch, resid, conv.weight, state, ctx.cu_q, ctx.state_slots, ctx.num_requests,
                                ctx.max_q_len, ctx.dtype)

    def forward(self, branch, resid, ctx, cache):
        streams = count = weight = None
        if self.depth_average is not None:
            # the streams before this layer's own: the embedding output and the earlier layers' results
            streams, weight = ctx.depth_streams, self.depth_average.weight
            count = 1 if branch is None else branch.count + 1
        last = dict(streams=streams, count=count or 0, depth_weight=weight)
        ctx.residual_sink, ctx.takes_bias = None, True
        view = self._mixer_view(cache)
        own = cache.states[len(view.states):]
        h, x = self._input(self.mixer_conv, own[0], branch, resid, ctx)
        out = self.mixer.forward(h, ctx, view)
        if self.feed_forward is None:
            out = self.mixer_norm.depth_pending(out, **last)
        else:
            h, x = self._input(self.feed_forward_conv, own[1], self.mixer_norm.depth_pending(out), x, ctx)
            out = self.feed_forward_norm.depth_pending(self.feed_forward.forward(h, ctx), **last)
        ctx.takes_bias = False
        return out, x
