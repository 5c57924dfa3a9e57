"""Python entry point of ``csrc/conv_qkv.cu``: bias, short causal convolution, head norm, rotation and cache store of one
attention layer's fused projection.  As everywhere in ``gllm_b200.ops``: CUDA tensors only, no CPU path."""

from __future__ import annotations

import torch

from gllm_b200.ops import SplitSum, _check, _cuda, _fn, _parts_args, _ptr, _stream, _suffix, status_word

MAX_TAPS = 16


def conv_qkv(proj, bias: torch.Tensor | None, conv_w: torch.Tensor, conv_state: torch.Tensor | None, q_norm: torch.Tensor,
             k_norm: torch.Tensor | None, eps: float, inv_freq: torch.Tensor | None, rotary_dim: int, magnitude: float,
             slot_mapping: torch.Tensor | None, cache_layer: torch.Tensor | None, heads: int, kv_heads: int, dk: int,
             dv: int, stored_dim: int, batch, own_kv: bool = True) -> torch.Tensor:
    """``proj [n, channels]`` (a tensor or a SplitSum): ``heads`` query heads and, with ``own_kv``, ``kv_heads`` key heads
    of ``dk`` columns and ``kv_heads`` value heads of ``dv``.  ``bias`` is added; every channel is convolved over time
    with its filter (``conv_w [taps, channels]`` fp32, last row: the current token; ``conv_state [slots, taps - 1,
    channels]`` fp32 holds each request's last inputs and is brought up to date); query and key heads are RMS-normed
    with ``q_norm`` / ``k_norm`` and neighbouring columns below ``rotary_dim`` rotated, sine and cosine times
    ``magnitude``.  Keys and values are stored into ``cache_layer [pages, 2, kv_heads, block_size, stored_dim]`` at
    ``slot_mapping``; the rotated queries ``[n, heads * stored_dim]`` are returned, columns behind a head's width zero."""
    parts_ptr, n_parts, part_stride = _parts_args(proj)
    channels = heads * dk + (kv_heads * (dk + dv) if own_kv else 0)
    if isinstance(proj, SplitSum):
        n, cols, dtype, device, ptr, stride = *proj.shape, proj.dtype, proj.device, None, 0
    else:
        _cuda(proj, "proj", contiguous=False)
        if proj.dim() != 2 or proj.stride(1) != 1:
            raise ValueError("proj must be [tokens, columns] with contiguous columns")
        n, cols, dtype, device, ptr, stride = *proj.shape, proj.dtype, proj.device, proj.data_ptr(), proj.stride(0)
    _cuda(conv_w, "conv_w", torch.float32)
    taps = conv_w.shape[0]
    if cols != channels or tuple(conv_w.shape) != (taps, channels) or not 1 <= taps <= MAX_TAPS:
        raise ValueError(f"the projection has {cols} columns, {channels} were expected, each with up to {MAX_TAPS} taps")
    if bias is not None:
        _cuda(bias, "bias", torch.float32)
        if bias.numel() != channels:
            raise ValueError("one bias value per channel is needed")
    if taps > 1:
        _cuda(conv_state, "conv_state", torch.float32)
        if tuple(conv_state.shape[1:]) != (taps - 1, channels):
            raise ValueError("the convolution's state is [slots, taps - 1, channels]")
    for name, w in (("q_norm", q_norm), ("k_norm", k_norm if own_kv else None)):
        if w is not None:
            _cuda(w, name, torch.float32)
            if w.numel() != dk:
                raise ValueError(f"{name} needs one value per column of a head")
    if q_norm is None or (own_kv and k_norm is None):
        raise ValueError("query and key heads have norm weights")
    if inv_freq is not None:
        _cuda(inv_freq, "inv_freq", torch.float32)
        if inv_freq.numel() != rotary_dim // 2:
            raise ValueError("inv_freq must hold rotary_dim/2 frequencies")
    block_size = num_pages = 0
    if own_kv and slot_mapping is not None:
        _cuda(slot_mapping, "slot_mapping", torch.int32)
        _cuda(cache_layer, "cache_layer", dtype)
        num_pages, two, hkv, block_size, d = cache_layer.shape
        if two != 2 or hkv != kv_heads or d != stored_dim:
            raise ValueError("cache layer shape does not match the mixer's heads")
    else:
        slot_mapping = cache_layer = None
    for name, t in (("positions", batch.positions), ("cu_q", batch.cu_q), ("state_slots", batch.state_slots)):
        _cuda(t, name, torch.int32)
    q = torch.empty((n, heads * stored_dim), dtype=dtype, device=device)
    f = _fn("conv_qkv", f"gllm_conv_qkv_{_suffix(dtype)}")
    _check(f(ptr, stride, parts_ptr, n_parts, part_stride, _ptr(bias), conv_w.data_ptr(),
             _ptr(conv_state) if taps > 1 else None, batch.cu_q.data_ptr(), batch.state_slots.data_ptr(),
             batch.positions.data_ptr(), q_norm.data_ptr(), _ptr(k_norm) if own_kv else None, float(eps), _ptr(inv_freq),
             int(rotary_dim) if inv_freq is not None else 0, float(magnitude), _ptr(slot_mapping), q.data_ptr(),
             _ptr(cache_layer), int(batch.num_requests), int(batch.max_q_len), int(heads), int(kv_heads), int(own_kv),
             int(dk), int(dv), int(stored_dim), int(taps), block_size, num_pages, status_word(device).data_ptr(),
             _stream()), "conv_qkv")
    return q
