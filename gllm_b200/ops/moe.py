"""Python entry points of the routed-expert kernels (``csrc/moe.cu``).  As everywhere in ``gllm_b200.ops``: CUDA
tensors only, no CPU path; everything that varies between steps of equal shape (which experts were chosen, how
many tiles they fill) stays on the device, so a step can be captured in a CUDA graph."""

from __future__ import annotations

import torch

from gllm_b200.ops import RowSum, SplitSum, _check, _cuda, _fn, _parts_args, _ptr, _stream, _suffix

TILE_ROWS = 16        # rows of one tile of the expert products: an expert's pairs are padded to a multiple of it
PLAIN_GATE = (1.0, 0.0, 0.0)    # slope, limit, offset of a gated expert's activation: silu(gate) * up
TENSOR_CORE_TILE_ROWS = 128     # the same for the tcgen05 products (the rows of one accumulator tile)


def _router_args(logits):
    """(pointer, row stride, parts, part stride, tokens, experts) of fp32 router logits: a tensor or a SplitSum."""
    if isinstance(logits, SplitSum):
        ptr, n_parts, part_stride = _parts_args(logits)
        if logits.dtype != torch.float32:
            raise TypeError("router logits are fp32")
        return ptr, logits.shape[1], n_parts, part_stride, *logits.shape
    _cuda(logits, "logits", torch.float32, contiguous=False)
    if logits.dim() != 2 or logits.stride(1) != 1:
        raise ValueError("router logits must be [tokens, experts] with contiguous columns")
    return logits.data_ptr(), logits.stride(0), 0, 0, *logits.shape


def _rule_args(correction, experts, top, groups, groups_kept, renormalize, score, group_score, renormalize_eps, scale):
    if score not in ("sigmoid", "softmax") or group_score not in ("top2", "max"):
        raise ValueError("router scores are 'sigmoid' or 'softmax', group scores 'top2' or 'max'")
    if correction is not None:
        _cuda(correction, "correction", torch.float32)
        if correction.numel() != experts:
            raise ValueError("one correction value per expert is needed")
    return (experts, int(top), int(groups), int(groups_kept), int(renormalize), int(score == "softmax"),
            int(group_score == "max"), float(renormalize_eps), float(scale))


def route(logits, correction: torch.Tensor | None, top: int, groups: int = 1, groups_kept: int = 1,
          renormalize: bool = False, score: str = "sigmoid", group_score: str = "top2", renormalize_eps: float = 0.0,
          scale: float = 1.0):
    """From fp32 router logits ``[n, experts]`` (a tensor or a SplitSum) to the chosen experts ``[n, top]`` int32 and their
    weights fp32.  Scores ``s = sigmoid(logits)`` (``score`` "softmax": the softmax over all experts); the choice is made
    on ``s + correction`` among the experts of the ``groups_kept`` best of ``groups`` equal groups of neighbours (a
    group's score: the sum of its two largest choice scores, with ``group_score`` "max" its largest); the weights are
    the chosen ``s``, divided by their sum (plus ``renormalize_eps``) with ``renormalize``, times ``scale``."""
    ptr, stride, n_parts, part_stride, n, experts = _router_args(logits)
    rule = _rule_args(correction, experts, top, groups, groups_kept, renormalize, score, group_score, renormalize_eps, scale)
    ids = torch.empty((n, top), dtype=torch.int32, device=logits.device)
    weights = torch.empty((n, top), dtype=torch.float32, device=logits.device)
    _check(_fn("moe", "gllm_moe_route")(ptr, stride, n_parts, part_stride, _ptr(correction), ids.data_ptr(),
                                        weights.data_ptr(), n, *rule, _stream()), "moe_route")
    return ids, weights


def _plan_tensors(pairs: int, experts: int, tile_rows: int, want_sorted: bool, want_rows: bool, device):
    max_tiles = -(-pairs // tile_rows) + min(experts, pairs)
    i32 = lambda n: torch.empty(n, dtype=torch.int32, device=device)
    return (i32(max_tiles * tile_rows) if want_sorted else None, i32(max_tiles), i32(1),
            i32(pairs) if want_rows else None)


def align(ids: torch.Tensor, experts: int, tile_rows: int = TILE_ROWS, want_rows: bool = False):
    """The (token, slot) pairs sorted by expert in tiles of ``tile_rows`` rows: ``(sorted [max_tiles * tile_rows]``
    (pair index or -1), ``tile_expert [max_tiles]``, ``num_tiles [1])``, all int32 on the device; with
    ``want_rows`` also ``row_of_pair [pairs]``, the row each pair got."""
    _cuda(ids, "ids", torch.int32)
    pairs = ids.numel()
    plan = _plan_tensors(pairs, experts, tile_rows, True, want_rows, ids.device)
    _check(_fn("moe", "gllm_moe_align")(ids.data_ptr(), *(_ptr(t) for t in plan), pairs, int(experts), int(tile_rows),
                                        plan[1].numel(), _stream()), "moe_align")
    return plan if want_rows else plan[:3]


# most tokens whose routing and sorting one block does in one launch
ROUTE_ALIGN_TOKENS = 64


def route_and_align(logits, correction, top: int, tile_rows: int, want_sorted: bool, want_rows: bool, groups: int = 1,
                    groups_kept: int = 1, renormalize: bool = False, score: str = "sigmoid", group_score: str = "top2",
                    renormalize_eps: float = 0.0, scale: float = 1.0):
    """``route`` and ``align`` one after the other, in one launch for up to ``ROUTE_ALIGN_TOKENS`` tokens: ``(ids, weights,
    (sorted | None, tile_expert, num_tiles, row_of_pair | None))``."""
    ptr, stride, n_parts, part_stride, n, experts = _router_args(logits)
    if n > ROUTE_ALIGN_TOKENS or 32 * (2 * experts + groups) * 4 + (3 * experts + 1) * 4 > 48 * 1024:
        ids, weights = route(logits, correction, top, groups, groups_kept, renormalize, score, group_score,
                             renormalize_eps, scale)
        plan = align(ids, experts, tile_rows, want_rows=True)
        return ids, weights, plan
    rule = _rule_args(correction, experts, top, groups, groups_kept, renormalize, score, group_score, renormalize_eps, scale)
    ids = torch.empty((n, top), dtype=torch.int32, device=logits.device)
    weights = torch.empty((n, top), dtype=torch.float32, device=logits.device)
    plan = _plan_tensors(n * top, experts, tile_rows, want_sorted, want_rows, logits.device)
    _check(_fn("moe", "gllm_moe_route_align")(ptr, stride, n_parts, part_stride, _ptr(correction), ids.data_ptr(),
                                              weights.data_ptr(), n, *rule, *(_ptr(t) for t in plan), int(tile_rows),
                                              plan[1].numel(), _stream()), "moe_route_align")
    return ids, weights, plan


def gather_rows(x: torch.Tensor, top: int, row_of_pair: torch.Tensor, rows: int, weights: torch.Tensor | None = None):
    """``out[row_of_pair[p]] = x[p // top]`` (bf16, ``[rows, width]``): the tokens' rows in the order of the sorted
    pairs; with ``weights`` (fp32, one per pair) also ``[rows]`` of those in the same order: ``(out, row_scale)``.  Rows
    that no pair owns are left as they are: the products' rows do not mix, and nobody reads theirs."""
    _cuda(x, "x", torch.bfloat16, contiguous=False)
    _cuda(row_of_pair, "row_of_pair", torch.int32)
    out = torch.empty((rows, x.shape[1]), dtype=x.dtype, device=x.device)
    row_scale = None
    if weights is not None:
        _cuda(weights, "weights", torch.float32)
        if weights.numel() != row_of_pair.numel():
            raise ValueError("one weight per (token, slot) pair is needed")
        row_scale = torch.empty(rows, dtype=torch.float32, device=x.device)
    _check(_fn("moe", "gllm_moe_gather_bf16")(x.data_ptr(), x.stride(0), row_of_pair.data_ptr(), out.data_ptr(),
                                              row_of_pair.numel(), int(top), x.shape[1], _ptr(weights), _ptr(row_scale),
                                              _stream()), "moe_gather")
    return out if weights is None else (out, row_scale)


def tensor_cores_take(dtype: torch.dtype, width: int, ff: int, gated: bool = True) -> bool:
    """Whether the experts' products run on the tcgen05 kernel: bf16, rows that start on 16 bytes, and (for gated
    experts) gate and up rows stacked in blocks of 64."""
    return dtype == torch.bfloat16 and width % 8 == 0 and ff % (64 if gated else 8) == 0


def expert_product(a: torch.Tensor, rows_per_input: int, weight: torch.Tensor, plan, n_pairs: int, gated: bool,
                   relu_squared: bool = False, act: tuple = PLAIN_GATE, row_scale: torch.Tensor | None = None):
    """``out[pair] = a[pair // rows_per_input] @ weight[expert of pair].T`` for the pairs of ``plan`` (what
    ``align`` returned).  ``weight [experts, rows, k]``; ``gated``: its rows are gate rows then up rows and the
    result is ``silu(gate) * up`` (or what ``act``, the slope, limit and offset of ``ops.linear_gated``, says) in the
    activation type ``[n_pairs, rows / 2]``; ``row_scale`` (fp32, one number per pair): the products are multiplied by
    it, ahead of the activation; ``relu_squared`` (experts without a
    gate): ``max(result, 0) ** 2`` in the activation type ``[n_pairs, rows]``; otherwise fp32 ``[n_pairs, rows]``."""
    _cuda(a, "a", contiguous=False)
    _cuda(weight, "weight", a.dtype)
    if a.dim() != 2 or a.stride(1) != 1 or weight.dim() != 3 or weight.shape[2] != a.shape[1]:
        raise ValueError("the expert product takes rows of contiguous columns and weights [experts, rows, k]")
    sorted_pairs, tile_expert, num_tiles = plan
    rows, k = weight.shape[1], weight.shape[2]
    if gated and (rows % 2 or relu_squared):
        raise ValueError("gate and up rows come in equal numbers, and the gate is the activation")
    n_cols = rows // 2 if gated else rows
    out = torch.empty((n_pairs, n_cols), dtype=a.dtype if gated or relu_squared else torch.float32, device=a.device)
    f = _fn("moe", f"gllm_moe_gemm_{_suffix(a.dtype)}")
    _check(f(a.data_ptr(), a.stride(0), int(rows_per_input), weight.data_ptr(), weight.stride(0),
             n_cols * k if gated else 0, sorted_pairs.data_ptr(), tile_expert.data_ptr(), num_tiles.data_ptr(),
             out.data_ptr(), tile_expert.numel(), n_cols, k, TILE_ROWS, int(relu_squared), _ptr(row_scale), *act, _stream()),
           "moe_gemm")
    return out


def combine(y: torch.Tensor, weights: torch.Tensor | None, shared: torch.Tensor | None, out_dtype: torch.dtype,
            row_of_pair: torch.Tensor | None = None, shared_gate: torch.Tensor | None = None, tokens: int | None = None,
            top: int | None = None) -> torch.Tensor:
    """``out[t] = sum_s weights[t, s] * y[t * top + s] (+ shared[t])``, summed in slot order in fp32 (``weights`` None: 1
    each; ``tokens`` and ``top`` are then named); ``y`` may be ``[parts, rows, width]``, the parts being added first; with
    ``row_of_pair`` the pair's result is row ``row_of_pair[t * top + s]`` of ``y``; with ``shared_gate`` (fp32, one
    logit per token; may be a column of a wider matrix) the shared result is multiplied by its sigmoid."""
    _cuda(y, "y", torch.float32)
    y = y if y.dim() == 3 else y[None]
    if weights is not None:
        _cuda(weights, "weights", torch.float32)
        tokens, top = weights.shape
    n, width = int(tokens), y.shape[2]
    if row_of_pair is not None:
        _cuda(row_of_pair, "row_of_pair", torch.int32)
    if (y.shape[1] != n * top and row_of_pair is None) or (row_of_pair is not None and row_of_pair.numel() != n * top):
        raise ValueError("one result row per (token, slot) pair is needed")
    if shared is not None:
        _cuda(shared, "shared", out_dtype)
        if tuple(shared.shape) != (n, width):
            raise ValueError("the shared expert's result does not fit")
    gate_stride = 0
    if shared_gate is not None:
        _cuda(shared_gate, "shared_gate", torch.float32, contiguous=False)
        if shared is None or shared_gate.dim() != 1 or shared_gate.numel() != n:
            raise ValueError("the shared expert's gate is one logit per token")
        gate_stride = shared_gate.stride(0)
    out = torch.empty((n, width), dtype=out_dtype, device=y.device)
    _check(_fn("moe", f"gllm_moe_combine_{_suffix(out_dtype)}")(y.data_ptr(), y.shape[0], y.stride(0), _ptr(weights),
                                                               _ptr(shared), out.data_ptr(), _ptr(row_of_pair), n,
                                                               int(top), width, _ptr(shared_gate), gate_stride,
                                                               _stream()), "moe_combine")
    return out


def relu_squared_rows(x: torch.Tensor) -> torch.Tensor:
    """``max(x, 0) ** 2`` of fp32 ``x``, rounded to bf16: between the two tensor-core products of experts without
    a gate."""
    _cuda(x, "x", torch.float32)
    out = torch.empty(x.shape, dtype=torch.bfloat16, device=x.device)
    _check(_fn("moe", "gllm_moe_relu_sq_bf16")(x.data_ptr(), out.data_ptr(), x.numel(), _stream()), "moe_relu_sq")
    return out


def grouped_tile_rows(pairs: int, experts: int) -> int:
    """Rows of a tile of the tensor-core products: small tiles (the weight is then the 128-row operand, and a tile's rows
    cost little) while an expert gets few rows on average."""
    per_expert = pairs / experts
    return 16 if per_expert <= 8 else 32 if per_expert <= 20 else 64 if per_expert <= 40 else TENSOR_CORE_TILE_ROWS


def _down_splits(pairs: int, experts: int, rows: int, k: int, device) -> int:
    """Ranges of K the second product is cut into when its tiles alone would leave most SMs without work."""
    tiles = min(pairs, experts) * -(-rows // 128)
    sms = torch.cuda.get_device_properties(device).multi_processor_count
    blocks = -(-k // 64)
    best = 1
    for s in range(2, 5):
        if tiles * s <= sms and blocks // s >= 4 and -(-blocks // s) * (s - 1) < blocks:
            best = s
    return best


class Choice:
    """Which experts serve which tokens: ids and weights ``[n, top]`` and the (token, slot) pairs sorted by expert."""

    def __init__(self, ids, weights, plan, tile_rows: int):
        self.ids, self.weights, self.plan, self.tile_rows = ids, weights, plan, tile_rows


def choose(logits, correction, top: int, tensor_cores: bool, **rule) -> Choice:
    """Route and sort for ``apply_choice`` (``rule``: the options of ``route``)."""
    n, experts = logits.shape
    tile = grouped_tile_rows(n * top, experts) if tensor_cores else TILE_ROWS
    return Choice(*route_and_align(logits, correction, top, tile, want_sorted=not tensor_cores, want_rows=tensor_cores, **rule),
                  tile)


def apply_experts(x: torch.Tensor, ids: torch.Tensor, weights: torch.Tensor, w_gate_up: torch.Tensor,
                  w_down: torch.Tensor, shared: torch.Tensor | None, tensor_cores: bool, **options) -> torch.Tensor:
    """``apply_choice`` for a choice that is already made: ``ids`` and ``weights`` ``[n, top]``."""
    tile = grouped_tile_rows(ids.numel(), w_gate_up.shape[0]) if tensor_cores else TILE_ROWS
    plan = align(ids, w_gate_up.shape[0], tile, want_rows=True)
    return apply_choice(x, Choice(ids, weights, plan, tile), w_gate_up, w_down, shared, tensor_cores, **options)


def apply_choice(x: torch.Tensor, choice: Choice, w_gate_up: torch.Tensor, w_down: torch.Tensor,
                 shared: torch.Tensor | None, tensor_cores: bool, gated: bool = True,
                 shared_gate: torch.Tensor | None = None, act: tuple = PLAIN_GATE, weight_on_input: bool = False,
                 defer_sum: bool = False):
    """``out[t] = sum_s weights[t, s] * expert_{ids[t, s]}(x[t]) (+ shared[t])`` with ``expert_e(x) = w_down[e]
    (silu(gate) * up)``.  ``tensor_cores``: ``w_gate_up [experts, 2 * ff, width]`` is stacked per expert by
    ``interleave_gate_up``; the tokens' rows are copied into the order of the sorted pairs, both products read and
    write rows in that order on the tcgen05 kernel, and the weighted sum looks every pair's row up.  Otherwise
    ``w_gate_up`` holds an expert's gate rows, then its up rows, and the CUDA-core kernel runs.  ``gated`` False:
    experts without a gate, ``expert_e(x) = w_down[e] relu(w_up[e] x)^2`` with ``w_gate_up [experts, ff, width]`` the
    up weights.  ``shared_gate``: see ``combine``.  ``act``: the slope, limit and offset of the gated activation.
    ``weight_on_input``: ``out[t] = sum_s expert(weights[t, s] * x[t])`` instead; the weight is applied to the first
    product's fp32 sums, which is the same and spares a rounding.  ``defer_sum`` (without a shared expert): the pairs'
    results are returned as an ``ops.RowSum``, for a kernel that adds them up itself."""
    experts, (n, top), pairs = w_gate_up.shape[0], choice.ids.shape, choice.ids.numel()
    weights, (sorted_pairs, tile_expert, num_tiles, row_of_pair) = choice.weights, choice.plan
    if not tensor_cores:
        plan, row_of_pair = (sorted_pairs, tile_expert, num_tiles), None
        hidden = expert_product(x, top, w_gate_up, plan, pairs, gated=gated, relu_squared=not gated, act=act,
                                row_scale=weights if weight_on_input else None)
        y = expert_product(hidden, 1, w_down, plan, pairs, gated=False)
    else:
        from gllm_b200.ops import gemm_bf16

        wide = pairs > 2048
        rows, row_scale = tile_expert.numel() * choice.tile_rows, None
        if weight_on_input:
            if not gated:
                raise ValueError("weights on the input of the tensor-core products are for gated experts")
            xs, row_scale = gather_rows(x, top, row_of_pair, rows, weights)
        else:
            xs = gather_rows(x, top, row_of_pair, rows)
        hidden = gemm_bf16.linear_grouped(xs, w_gate_up, tile_expert, num_tiles, gated=gated, wide=wide, act=act,
                                          row_scale=row_scale, tile_rows=choice.tile_rows)
        if not gated:
            hidden = relu_squared_rows(hidden)
        splits = 1
        if choice.tile_rows != TENSOR_CORE_TILE_ROWS:
            splits = _down_splits(pairs, experts, w_down.shape[1], w_down.shape[2], x.device)
        y = gemm_bf16.linear_grouped(hidden, w_down, tile_expert, num_tiles, gated=False, wide=wide,
                                     tile_rows=choice.tile_rows, splits=splits)
    weights = None if weight_on_input else weights
    if defer_sum and shared is None:
        return RowSum(y if y.dim() == 3 else y[None], row_of_pair, weights, n, top, x.dtype)
    return combine(y, weights, shared, x.dtype, row_of_pair, shared_gate=shared_gate, tokens=n, top=top)
