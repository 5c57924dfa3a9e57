"""Python entry points of ``csrc/attention_distance.cu`` and ``csrc/attention_distance_mma.cu`` (and of the form with a
bias of ``csrc/attention_prefill_tmem.cu``): softmax attention with a learned bias by distance, a window that keeps the
first tokens, and a sink.  As everywhere in ``gllm_b200.ops``: CUDA
tensors only, no CPU path."""

from __future__ import annotations

import bisect
import math
import os
from dataclasses import dataclass
from fractions import Fraction

import torch

from gllm_b200.ops import _check, _cuda, _fn, _parts_args, _ptr, _stream, _suffix, status_word

# GLLM_B200_DISTANCE_MMA=0: the attention of bf16 models stays on the CUDA-core kernel (for measurements)
USE_TENSOR_CORES = os.environ.get("GLLM_B200_DISTANCE_MMA", "1") != "0"
KEY_TILE = 64             # keys of a tile of portions, and of single tokens
SINGLE_KEY_TILE = 32
SPLIT_TILES = 2           # key tiles per CTA at least when the keys of short portions are cut, and of single tokens
SINGLE_SPLIT_TILES = 4
MAX_SPLITS = 16
# portions shorter than this stay on the mma.sync kernel (its 64-row tiles waste less on short portions)
TMEM_MIN_Q_LEN = 32

NO_MIX, FIRST, MIXED = 0, 1, 2        # what the prep kernel does with the values

_mma = None


def _mma_fns():
    global _mma
    if _mma is None:
        from ctypes import c_float, c_int, c_int64, c_void_p as P

        from gllm_b200.ops.build import load_module

        lib = load_module("attention_distance_mma")
        f = lib.gllm_attention_distance_mma
        f.argtypes = [P, c_int64, P, c_int64, P, P, c_int, P, P, c_int, P, P, P, P, c_int, P, c_int, c_int, c_int, c_int,
                      c_int, c_int, c_int, c_int, c_float, c_int, c_int, c_int, c_int, c_int, P, P]
        f.restype = c_int
        lib.gllm_attention_distance_mma_tokens_per_tile.argtypes = [c_int, c_int]
        lib.gllm_attention_distance_few_tiles.argtypes = [c_int, c_int]
        _mma = (f, lib.gllm_attention_distance_mma_tokens_per_tile, lib.gllm_attention_distance_few_tiles)
    return _mma


_tmem = None


def _tmem_fns():
    global _tmem
    if _tmem is None:
        from ctypes import c_float, c_int, c_int64, c_void_p as P

        from gllm_b200.ops.build import load_module

        lib = load_module("attention_prefill_tmem")
        f = lib.gllm_attention_prefill_distance
        f.argtypes = [P, c_int64, P, c_int64, P, P, c_int, P, P, P, P, c_int, P, c_int, c_int, c_int, c_int, c_int, c_int,
                      c_int, c_int, c_float, c_int, c_int, P, P]
        f.restype = c_int
        lib.gllm_attention_prefill_distance_supports.argtypes = [c_int, c_int, c_int, c_int, c_int]
        _tmem = (f, lib.gllm_attention_prefill_distance_supports)
    return _tmem


def takes_tmem(heads: int, kv_heads: int, dk: int, dv: int, block_size: int, bias_len: int) -> bool:
    """True for the sizes the tcgen05 kernel takes: keys and values both 64 or both 128 wide, pages of a power of two
    of tokens, a bias table that fits shared memory."""
    return (dk == dv and dk in (64, 128)
            and bool(_tmem_fns()[1](heads, kv_heads, dk, block_size, bias_len)))


def takes_tensor_cores(dtype: torch.dtype, dk: int, dv: int) -> bool:
    """True for the widths the tensor-core kernel takes (bf16; multiples of 8 up to 128)."""
    return dtype == torch.bfloat16 and all(0 < d <= 128 and d % 8 == 0 for d in (dk, dv))


# ------------------------------------------------------------------ bias by distance
def distance_buckets(rows: int, distance_max, length: int) -> list[int]:
    """Bucket of every distance 0 .. length-1: the distance itself below half the rows, logarithmic steps up to
    ``distance_max`` above, the last row from there on.  The step of distance n is the largest k with
    ``(n / half)^m >= (distance_max / half)^k``, ``m`` the number of logarithmic rows: compared in integers, so that no
    border depends on how a logarithm is rounded."""
    half = rows // 2
    if half < 1:
        return [0] * length
    m, span = rows - half, Fraction(distance_max) / half
    if span <= 1:
        raise ValueError("the largest distance of the logarithmic rows must exceed half the rows")
    starts = []                            # the first distance of every logarithmic row but the first
    for k in range(1, m):
        lo, hi, bound = half, max(half, math.ceil(distance_max)), span ** k
        while lo < hi:
            mid = (lo + hi) // 2
            lo, hi = (lo, mid) if Fraction(mid, half) ** m >= bound else (mid + 1, hi)
        starts.append(lo)
    return [n if n < half else half + bisect.bisect_right(starts, n) for n in range(length)]


@dataclass
class DistanceBias:
    """A layer's bias by distance, expanded to one value per (head, distance): ``table [heads, length]`` fp32, every
    distance from ``length - 1`` on has the last value; the sink beside it (``[heads]`` or None); both also times
    log2(e) for the kernel that works in base 2."""

    table: torch.Tensor
    sink: torch.Tensor | None
    table_log2: torch.Tensor
    sink_log2: torch.Tensor | None

    @classmethod
    def build(cls, rel: torch.Tensor, distance_max, sink: torch.Tensor | None) -> "DistanceBias":
        """``rel [rows, heads]``: the learned values."""
        buckets = distance_buckets(rel.shape[0], distance_max, max(1, math.ceil(distance_max)) + 1)
        index = torch.tensor(buckets, dtype=torch.long, device=rel.device)
        table = rel.float()[index].t().contiguous()
        log2e = math.log2(math.e)
        return cls(table, None if sink is None else sink.float().contiguous(), (table * log2e).contiguous(),
                   None if sink is None else (sink.float() * log2e).contiguous())


# ------------------------------------------------------------------ prep and attention
def distance_prep(proj, bias: torch.Tensor | None, eps: float, slot_mapping: torch.Tensor | None,
                  pages: torch.Tensor, heads: int, kv_heads: int, dk: int, dv: int, block_size: int,
                  mix: int = NO_MIX, first: torch.Tensor | None = None, lam: float = 0.0) -> torch.Tensor:
    """From the projections ``[q | k | v]`` of a step's tokens (``[n, heads*dk + kv_heads*(dk + dv)]``, a tensor or a
    SplitSum; ``bias`` fp32, one value per column, is added first): every query and key head divided by its root mean
    square (eps inside the root), the values mixed with ``first`` (``[n, kv_heads*dv]``; ``mix`` FIRST writes it, MIXED
    makes ``(1 - lam) v + lam first``), keys and values stored at ``slot_mapping``.  Returns the queries ``[n, heads*dk]``."""
    parts_ptr, n_parts, part_stride = _parts_args(proj)
    total = heads * dk + kv_heads * (dk + dv)
    n, cols = proj.shape
    if cols != total:
        raise ValueError(f"the projection has {cols} columns, {total} were expected")
    if parts_ptr is None:
        _cuda(proj, "proj")
    if n_parts > 16:
        proj = proj.tensor()
        parts_ptr, n_parts, part_stride = None, 0, 0
    dtype = proj.dtype
    if bias is not None:
        _cuda(bias, "bias", torch.float32)
        if bias.numel() != total:
            raise ValueError("one bias value per column is needed")
    if mix != NO_MIX:
        _cuda(first, "first", dtype)
        if tuple(first.shape) != (n, kv_heads * dv):
            raise ValueError("the values to mix with have another shape than this layer's")
    num_pages = 0
    if slot_mapping is not None:
        _cuda(slot_mapping, "slot_mapping", torch.int32)
        _cuda(pages, "pages", dtype)
        num_pages = pages.shape[0]
        if pages.shape[1] != block_size * kv_heads * (dk + dv):
            raise ValueError("the cache pages do not hold keys and values of these widths")
    q = torch.empty((n, heads * dk), dtype=dtype, device=proj.device)
    f = _fn("attention_distance", f"gllm_distance_prep_{_suffix(dtype)}")
    _check(f(None if parts_ptr is not None else proj.data_ptr(), cols, parts_ptr, n_parts, part_stride, _ptr(bias),
             float(eps), q.data_ptr(), _ptr(first) if mix != NO_MIX else None, int(mix), float(lam), _ptr(slot_mapping),
             _ptr(pages) if slot_mapping is not None else None, n, heads, kv_heads, dk, dv, int(block_size), num_pages,
             status_word(q.device).data_ptr(), _stream()), "distance_prep")
    return q


def _ranges(most: int, tiles: int, least: int, per_sm: int, device):
    """(ranges, key tiles per range) for CTAs that visit up to ``most`` key tiles, ``tiles`` of them in all: one range
    unless they do not fill the GPU."""
    sms = torch.cuda.get_device_properties(device).multi_processor_count
    if 2 * tiles > sms * per_sm or most < 2 * least:
        return 1, 0
    want = min(MAX_SPLITS, -(-per_sm * sms // tiles))
    per = max(least, -(-most // want))
    return -(-most // per), per


def _visited(longest: int, tile: int, tokens: int, window: int, keep_first: int) -> int:
    """The most key tiles that ``tokens`` neighbouring tokens visit."""
    most = -(-longest // tile)
    return min(most, -(-keep_first // tile) + -(-(window + tokens) // tile) + 1) if window else most


def _mma_launch(q, out, pages, block_table, bias, heads, kv_heads, dk, dv, block_size, scale, window, keep_first, batch,
                first: int, count: int, single: bool):
    """The mma.sync kernels over requests ``first .. first+count-1`` (``single``: each brings one token)."""
    f, tokens_per_tile, few_tiles = _mma_fns()
    n, longest = q.shape[0], batch.max_seq_len
    if single:
        splits, per = _ranges(_visited(longest, SINGLE_KEY_TILE, 1, window, keep_first), few_tiles(heads, kv_heads) * count,
                              SINGLE_SPLIT_TILES, 2, q.device)
    else:
        # a captured prompt portion is replayed for other contexts: under capture the ranges cover what a block-table
        # row can hold, not just the captured step's longest sequence (single tokens are captured per sequence bucket)
        if torch.cuda.is_current_stream_capturing():
            longest = max(longest, block_table.shape[1] * block_size)
        qt = tokens_per_tile(heads, kv_heads)
        splits, per = _ranges(_visited(longest, KEY_TILE, qt, window, keep_first),
                              -(-batch.max_q_len // qt) * (heads * qt // 64) * count, SPLIT_TILES, 2, q.device)
    partial = stats = None
    if splits > 1:
        partial = batch.workspace.get("distance_attention_partial", splits * n * heads * dv, torch.float32)
        stats = batch.workspace.get("distance_attention_stats", splits * n * heads * 2, torch.float32)
    _check(f(q.data_ptr(), q.stride(0), out.data_ptr(), out.stride(0), _ptr(partial), _ptr(stats), n, pages.data_ptr(),
             block_table.data_ptr(), block_table.stride(0), batch.cu_q[first:].data_ptr(),
             batch.context_lens[first:].data_ptr(), batch.state_slots[first:].data_ptr(), bias.table_log2.data_ptr(),
             bias.table_log2.shape[1], _ptr(bias.sink_log2), count, 1 if single else batch.max_q_len, heads, kv_heads, dk,
             dv, int(block_size), pages.shape[0], float(scale), window, keep_first, int(single), splits, per,
             status_word(q.device).data_ptr(), _stream()), "distance_attention_mma")


def distance_attention(q: torch.Tensor, pages: torch.Tensor, block_table: torch.Tensor, positions: torch.Tensor,
                       token_row: torch.Tensor, bias: DistanceBias, heads: int, kv_heads: int, dk: int, dv: int,
                       block_size: int, scale: float, window: int | None = None, keep_first: int = 0,
                       batch=None) -> torch.Tensor:
    """Per token i and head h, over the request's cached keys j <= i with ``i - j < window`` or ``j < keep_first``
    (no window: all of them): scores ``q . k * scale + bias.table[h, min(i - j, last)]``, softmax whose denominator also
    holds ``exp(sink[h])``; returns ``[n, heads * dv]``.  With ``batch`` (the StepContext: per-request lengths, slots
    and the step's scratch) bf16 inputs of the widths it takes run on the tensor-core kernel, everything else on the
    CUDA cores in fp32."""
    _cuda(q, "q", contiguous=False)
    _cuda(pages, "pages", q.dtype)
    _cuda(block_table, "block_table", torch.int32, contiguous=False)
    if q.dim() != 2 or q.stride(1) != 1 or q.shape[1] < heads * dk:
        raise ValueError("q must be [tokens, >= heads*dk] with contiguous columns")
    if pages.shape[1] != block_size * kv_heads * (dk + dv):
        raise ValueError("the cache pages do not hold keys and values of these widths")
    if bias.table.shape[0] != heads or (bias.sink is not None and bias.sink.numel() != heads):
        raise ValueError("the bias and the sink need one row per head")
    n, win = q.shape[0], int(window or 0)
    out = torch.empty((n, heads * dv), dtype=q.dtype, device=q.device)
    if (batch is not None and USE_TENSOR_CORES and takes_tensor_cores(q.dtype, dk, dv) and q.stride(0) % 8 == 0
            and q.data_ptr() % 16 == 0):
        # the flat batch holds the portions first, then the single tokens: each kind has a kernel of its own
        portions = getattr(batch, "num_prefill_requests", None)
        if portions is None:
            portions = 0 if batch.max_q_len == 1 else batch.num_requests
        args = (bias, heads, kv_heads, dk, dv, block_size, scale, win, int(keep_first), batch)
        if portions and batch.max_q_len >= TMEM_MIN_Q_LEN and takes_tmem(heads, kv_heads, dk, dv, block_size,
                                                                        bias.table.shape[1]):
            _check(_tmem_fns()[0](q.data_ptr(), q.stride(0), out.data_ptr(), out.stride(0), pages.data_ptr(),
                                  block_table.data_ptr(), block_table.stride(0), batch.cu_q.data_ptr(),
                                  batch.context_lens.data_ptr(), batch.state_slots.data_ptr(), bias.table_log2.data_ptr(),
                                  bias.table_log2.shape[1], _ptr(bias.sink_log2), portions, batch.max_q_len, n, heads,
                                  kv_heads, dk, int(block_size), pages.shape[0], float(scale), win, int(keep_first),
                                  status_word(q.device).data_ptr(), _stream()), "distance_attention_tmem")
        elif portions:
            _mma_launch(q, out, pages, block_table, *args, 0, portions, False)
        if portions < batch.num_requests:
            _mma_launch(q, out, pages, block_table, *args, portions, batch.num_requests - portions, True)
        return out
    f = _fn("attention_distance", f"gllm_attention_distance_{_suffix(q.dtype)}")
    _check(f(q.data_ptr(), q.stride(0), out.data_ptr(), out.stride(0), pages.data_ptr(), block_table.data_ptr(),
             block_table.stride(0), positions.data_ptr(), token_row.data_ptr(), bias.table.data_ptr(), bias.table.shape[1],
             _ptr(bias.sink), n, heads, kv_heads, dk, dv, int(block_size), pages.shape[0], float(scale), win,
             int(keep_first), status_word(q.device).data_ptr(), _stream()), "distance_attention")
    return out
