"""Python entry points of ``csrc/depth_conv.cu``: what stands between the sublayers of a layer that norms a sublayer's
result and reads the residual convolved over time, with an average over the depth of the model.  As everywhere in
``gllm_b200.ops``: CUDA tensors only, no CPU path."""

from __future__ import annotations

import torch

from gllm_b200.ops import DepthPending, SplitSum, _check, _cuda, _fn, _parts_args, _ptr, _stream, _suffix

STAGED_BYTES = 200 * 1024         # shared memory for rows that arrive as unsummed splits


def _joined(p: DepthPending, resid: torch.Tensor, dtype: torch.dtype, staged_rows: int):
    """The kernels' common arguments: value, parts ..., depth weights."""
    _cuda(resid, "resid", torch.float32)
    if resid.dim() != 2:
        raise ValueError("resid must be [tokens, width]")
    n, width = resid.shape
    value = p.value
    if isinstance(value, SplitSum) and (value.parts.shape[0] > 16 or 4 * staged_rows * width > STAGED_BYTES):
        value = value.tensor()
    parts_ptr, n_parts, part_stride = _parts_args(value)
    if value is not None:
        if tuple(value.shape) != (n, width) or value.dtype != dtype:
            raise ValueError("the sublayer's result and the residual differ in shape or dtype")
        _cuda(p.post_weight, "post_weight", torch.float32)
        if p.post_weight.numel() != width:
            raise ValueError("the norm of the sublayer's result needs one weight per column")
        if p.value_bias is not None:
            _cuda(p.value_bias, "value_bias", torch.float32)
            if p.value_bias.numel() != width:
                raise ValueError("the bias needs one value per column")
        if not isinstance(value, SplitSum):
            _cuda(value, "value")
    stride = 0
    if p.depth_weight is not None:
        _cuda(p.depth_weight, "depth_weight", torch.float32)
        _cuda(p.streams, "streams", torch.float32)
        if p.depth_weight.numel() != p.count + 1 or p.streams.shape[0] <= p.count or tuple(p.streams.shape[1:]) != (n, width):
            raise ValueError("the depth average needs one weight per stream and a place for its own")
        stride = p.streams.stride(0)
    ptr = None if value is None or isinstance(value, SplitSum) else value.data_ptr()
    return (ptr, parts_ptr, n_parts, part_stride, _ptr(p.value_bias), _ptr(p.post_weight), p.post_eps, resid.data_ptr(),
            _ptr(p.streams) if p.depth_weight is not None else None, stride, p.count, _ptr(p.depth_weight)), value


def depth_conv(pending: DepthPending | None, resid: torch.Tensor, conv_weight: torch.Tensor, conv_state: torch.Tensor,
               cu_q: torch.Tensor, state_slots: torch.Tensor, num_requests: int, max_q_len: int, dtype: torch.dtype):
    """``(h, x)``: ``x`` the residual after ``pending`` (fp32, a new tensor; ``resid`` itself when nothing is pending)
    and ``h = x + conv(x)`` in ``dtype``, the convolution running over each request's own tokens with ``conv_weight
    [taps, width]`` fp32 (last row: the current token) and ``conv_state [slots, taps-1, width]`` fp32 (every request's
    last inputs, oldest first; brought up to date).  With a depth average ``X`` goes into ``pending.streams[count]``."""
    _cuda(conv_weight, "conv_weight", torch.float32)
    _cuda(conv_state, "conv_state", torch.float32)
    n, width = resid.shape
    taps = conv_weight.shape[0]
    if conv_weight.shape[1] != width or tuple(conv_state.shape[1:]) != (taps - 1, width):
        raise ValueError("the convolution's weight or state does not fit the residual")
    rows = 1 if max_q_len == 1 else max(8, taps - 1) + taps - 1
    args, _alive = _joined(pending or DepthPending(), resid, dtype, rows)
    x = resid if pending is None else torch.empty_like(resid)
    out = torch.empty((n, width), dtype=dtype, device=resid.device)
    f = _fn("depth_conv", f"gllm_depth_conv_{_suffix(dtype)}")
    _check(f(*args, x.data_ptr() if pending is not None else None, conv_weight.data_ptr(), conv_state.data_ptr(),
             cu_q.data_ptr(), state_slots.data_ptr(), out.data_ptr(), int(num_requests), int(max_q_len), width, taps,
             _stream()), "depth_conv")
    return out, x


def depth_norm(pending: DepthPending, resid: torch.Tensor, weight: torch.Tensor, eps: float, dtype: torch.dtype,
               rows: torch.Tensor | None = None) -> torch.Tensor:
    """RMS norm of the residual after ``pending``, at ``rows`` (all without); nothing is written back."""
    n, width = resid.shape
    if rows is not None:
        _cuda(rows, "rows", torch.int32)
    n_rows = n if rows is None else rows.numel()
    args, _alive = _joined(pending, resid, dtype, 1)
    out = torch.empty((n_rows, width), dtype=dtype, device=resid.device)
    f = _fn("depth_conv", f"gllm_depth_norm_{_suffix(dtype)}")
    _check(f(*args, _ptr(rows), n_rows, weight.data_ptr(), float(eps), out.data_ptr(), width, _stream()), "depth_norm")
    return out
