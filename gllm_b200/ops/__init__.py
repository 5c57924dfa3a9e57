"""Python entry points of the CUDA kernels.

Every function takes CUDA tensors, checks what the kernel assumes (device,
dtype, contiguity, sizes it accepts) and launches on the current stream.
There is no CPU path and no PyTorch fallback: a tensor that is not on a CUDA
device, or a kernel module that cannot be built, raises.

Naming: ``*_f32`` / ``*_bf16`` symbols are the two instantiations of a kernel
for the activation and weight-matrix type.  The residual stream, norm weights,
rotary frequencies, softmax statistics and logits are fp32 in both.
"""

from __future__ import annotations

import os
from ctypes import c_float, c_int, c_int64, c_void_p

import torch

from gllm_b200.ops.build import ExtensionError, build_all, load_module

__all__ = [
    "ExtensionError",
    "build_all",
    "embedding",
    "scale_softcap",
    "scatter_int32",
    "add_rmsnorm",
    "add_cast",
    "silu_mul",
    "rope_store",
    "linear",
    "paged_attention",
    "status_word",
    "check_status",
    "sample",
    "argmax",
    "SplitSum",
    "ADDED",
    "as_tensor",
    "linear_gated",
    "interleave_gate_up",
    "add_bias",
    "rmsnorm_heads",
    "relu_sq",
    "scaled_sum",
    "gated_activation",
    "residual_add",
    "join_rows",
    "qk_rownorm",
    "Pending",
    "rope_norm_store",
    "add_dyt",
    "Biased",
    "DepthPending",
    "RowSum",
]

P = c_void_p
_SIGNATURES = {
    "elementwise": {
        "gllm_embedding_{t}": [P, P, P, P, P, c_int, c_int, c_int, c_float, P, P],
        "gllm_scale_softcap_f32": [P, c_int64, c_float, c_float, P],
        "gllm_scatter_i32": [P, c_int64, P, P, c_int, P, P],
        "gllm_add_bias_{t}": [P, c_int64, P, c_int, c_int, P],
        "gllm_rmsnorm_heads_{t}": [P, c_int64, P, c_int, c_int, c_int, c_int, c_float, c_int, P],
        "gllm_add_rmsnorm_{t}": [P, P, c_int, c_int64, P, P, P, P, c_int, c_int, c_float, c_int, P],
        "gllm_sum_parts_{t}": [P, c_int, c_int64, P, c_int64, P],
        "gllm_silu_mul_{t}": [P, P, c_int, c_int, c_int, P, P],
        "gllm_relu_sq_{t}": [P, P, c_int64, P],
        "gllm_scaled_sum_{t}": [P, P, P, c_float, c_float, c_int64, P],
        "gllm_gated_act_{t}": [P, P, c_int, c_int, c_int, c_float, c_float, c_float, P],
        "gllm_residual_add_{t}": [P, P, c_int, c_int64, P, c_int64, P],
        "gllm_join_rows_{t}": [P, P, c_int, c_int64, P, P, P, c_int64, c_int, P],
        "gllm_qk_rownorm_{t}": [P, c_int64, P, c_int, c_int64, P, P, P, c_int, c_int, c_int, c_int, c_float, P],
        "gllm_rope_store_{t}": [P, P, c_int, c_int64, P, P, P, P, c_int, c_int, c_int, c_int, c_int, c_int, c_int,
                                c_int, P, P],
    },
    "gemm_fp32": {
        "gllm_gemm_f32": [P, P, P, c_int, c_int, c_int, c_int64, c_int64, c_int64, P],
    },
    "sampling": {
        "gllm_sample": [P, c_int64, c_int, c_int, P, P, P, P, P, P, c_int, P, P, P, P, P, P, P],
        "gllm_argmax": [P, c_int64, c_int, c_int, P, P, P],
    },
    "recurrent": {
        "gllm_conv_silu_{t}": [P, c_int64, P, P, P, P, P, P, c_int, c_int, c_int, P],
        "gllm_selective_scan_{t}": [P, P, P, P, P, c_int64, c_int, c_int, P, P, c_int64, c_int, P, P, P, P, P, c_int,
                                    c_int, c_int, c_int, c_int, P],
        "gllm_matrix_recurrence_{t}": [c_int, P, c_int64, P, c_int64, P, c_int64, P, c_int64, P, P, c_float, c_float,
                                       P, P, P, P, P, P, c_int64, c_int, c_int, c_int, c_int, c_int, c_int, P],
        "gllm_gated_group_norm_{t}": [P, c_int64, P, c_int64, P, c_int, P, c_int64, P, P, c_int64, c_int, c_int, c_int,
                                      c_float, P],
        "gllm_conv_state_advance_{t}": [P, c_int64, P, P, P, c_int, c_int, c_int, P],
        "gllm_head_norm_{t}": [P, c_int64, c_int, c_int, c_float, P, c_int, P, c_int64, c_int, P, c_int64, c_int, c_int,
                               c_int, c_float, P],
    },
    "hyper_streams": {
        "gllm_embed_streams_{t}": [P, P, P, P, P, P, P, c_int, c_int, c_int, c_int, c_float, P, P],
        "gllm_stream_mix_norm_{t}": [P, P, P, P, P, P, P, P, P, c_int, c_int, c_int, c_float, P],
    },
    "attention_sigmoid": {
        "gllm_qk_norm_store_{t}": [P, c_int64, P, P, c_float, c_float, c_float, P, P, P, c_int, c_int, c_int, c_int,
                                   c_int, c_int, c_int, P, P],
        "gllm_attention_sigmoid_{t}": [P, c_int64, P, c_int64, P, P, c_int, P, P, P, c_int, c_int, c_int, c_int, c_int,
                                       c_int, c_int, c_float, P, P],
    },
    "attention_latent": {
        "gllm_latent_prep_{t}": [P, c_int64, P, c_int, c_int64, c_int, P, c_float, P, P, P, P, c_int, c_int, c_int, c_int,
                                 c_int, c_int, c_int, c_int, c_int, c_int, c_int, P, P, P, P],
        "gllm_latent_rotate_q_{t}": [P, c_int64, P, P, c_int, c_int, c_int, c_int, c_int, P],
        "gllm_head_linear_{t}": [P, c_int64, c_int, P, P, c_int64, c_int, c_int, c_int, c_int, c_int, P],
        "gllm_attention_latent_{t}": [P, c_int64, c_int, P, c_int64, c_int, P, c_int64, P, c_int64, c_int, P, P, c_int,
                                      P, P, c_int, c_int, c_int, c_int, c_int, c_int, c_float, c_int, P, P],
    },
    "dyt_norm": {
        "gllm_add_dyt_{t}": [P, P, c_int, c_int64, P, P, P, P, P, P, c_int, c_int, P],
    },
    "attention_diff": {
        "gllm_diff_rope_store_{t}": [P, c_int64, P, P, P, P, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int,
                                     c_int, c_int, P, P],
        "gllm_attention_diff_{t}": [P, c_int64, P, c_int64, P, c_int64, P, P, c_int, P, P, c_int, c_int, c_int, c_int,
                                    c_int, c_int, c_int, c_float, c_float, c_float, c_float, c_float, P, P],
    },
    "attention_distance": {
        "gllm_distance_prep_{t}": [P, c_int64, P, c_int, c_int64, P, c_float, P, P, c_int, c_float, P, P, c_int, c_int,
                                   c_int, c_int, c_int, c_int, c_int, P, P],
        "gllm_attention_distance_{t}": [P, c_int64, P, c_int64, P, P, c_int, P, P, P, c_int, P, c_int, c_int, c_int,
                                        c_int, c_int, c_int, c_int, c_float, c_int, c_int, P, P],
    },
    "depth_conv": {
        "gllm_depth_conv_{t}": [P, P, c_int, c_int64, P, P, c_float, P, P, c_int64, c_int, P, P, P, P, P, P, P, c_int,
                                c_int, c_int, c_int, P],
        "gllm_depth_norm_{t}": [P, P, c_int, c_int64, P, P, c_float, P, P, c_int64, c_int, P, P, c_int, P, c_float, P,
                                c_int, P],
    },
    "postnorm": {
        "gllm_postnorm_add_rmsnorm_{t}": [P, P, c_int, c_int64, P, c_float, P, P, P, c_float, P, P, c_int, c_int, P, c_int,
                                          c_int64, P, P, c_int, P],
    },
    "conv_qkv": {
        "gllm_conv_qkv_{t}": [P, c_int64, P, c_int, c_int64, P, P, P, P, P, P, P, P, c_float, P, c_int, c_float, P, P,
                              P, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, P, P],
    },
    "rope_norm": {
        "gllm_rope_norm_store_{t}": [P, P, c_int, c_int64, P, P, c_float, P, P, c_int, c_int, c_int, c_int, c_int,
                                     c_int, c_int, c_float, c_int, c_int, P, P],
    },
    "delta_rule": {
        "gllm_delta_prep_{t}": [P, c_int64, P, P, P, P, P, P, c_int, P, c_int64, P, P, P, c_int64, P, P, P, P, c_int,
                                c_int, c_int, c_int, c_int, c_int, c_float, c_float, c_int, c_int, P],
        "gllm_delta_rule": [P, P, P, P, P, P, P, P, c_int, c_int, c_int, c_int, c_int, c_int, c_int, P],
    },
    "moe": {
        "gllm_moe_route": [P, c_int64, c_int, c_int64, P, P, P, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int,
                           c_float, c_float, P],
        "gllm_moe_route_align": [P, c_int64, c_int, c_int64, P, P, P, c_int, c_int, c_int, c_int, c_int, c_int, c_int,
                                 c_int, c_float, c_float, P, P, P, P, c_int, c_int, P],
        "gllm_moe_align": [P, P, P, P, P, c_int, c_int, c_int, c_int, P],
        "gllm_moe_gemm_{t}": [P, c_int64, c_int, P, c_int64, c_int64, P, P, P, P, c_int, c_int, c_int, c_int, c_int, P,
                              c_float, c_float, c_float, P],
        "gllm_moe_combine_{t}": [P, c_int, c_int64, P, P, P, P, c_int, c_int, c_int, P, c_int64, P],
        "gllm_moe_relu_sq_bf16": [P, P, c_int64, P],
        "gllm_moe_gather_{t}": [P, c_int64, P, P, c_int, c_int, c_int, P, P, P],
    },
    "attention_simt": {
        "gllm_attention_simt_{t}": [P, c_int64, P, c_int64, P, P, c_int, P, P, c_int, c_int, c_int, c_int, c_int,
                                    c_int, c_float, c_int, P, P],
    },
}

_functions: dict[str, object] = {}


def _fn(module: str, name: str):
    f = _functions.get(name)
    if f is not None:
        return f
    lib = load_module(module)
    for pattern, argtypes in _SIGNATURES[module].items():
        for t in ("f32", "bf16"):
            sym = pattern.format(t=t)
            if sym in _functions:
                continue
            try:
                func = getattr(lib, sym)
            except AttributeError:
                continue
            func.argtypes = argtypes
            func.restype = c_int
            _functions[sym] = func
    try:
        return _functions[name]
    except KeyError:
        raise ExtensionError(f"kernel module {module!r} exports no symbol {name!r}") from None


def _error_string(code: int) -> str:
    try:
        return torch.cuda.cudart().cudaGetErrorString(torch.cuda.cudart().cudaError(code))
    except Exception:
        return f"cudaError {code}"


def modules_for(dtype: torch.dtype, head_dims=(), sampling: bool = False, modules=()) -> list[str]:
    """The kernel modules a model of this compute dtype will load: the products and pointwise kernels
    always, the softmax-attention modules when a mixer names a head size (``head_dims``), and whatever
    else its parts name (``modules``: the kernels of mixers with a state, of the streamed residual ...)."""
    if dtype == torch.float32:
        names = ["elementwise", "gemm_fp32"]
        if head_dims:
            names.append("attention_simt")
    else:
        names = ["elementwise", "gemm_bf16", "gemm_bf16_pair"]
        if head_dims:
            names += ["attention_bf16", "attention_prefill_bf16"]
        if any(d in (64, 128) for d in head_dims):
            names += ["attention_prefill_tmem", "attention_decode_tma"]
        if any(d not in (32, 64, 128) for d in head_dims):
            names.append("attention_simt")
    names += [m for m in modules if m not in names]
    if sampling:
        names.append("sampling")
    return names


def prepare(dtype: torch.dtype, head_dims=(), sampling: bool = False, modules=()) -> None:
    """Compile (side by side) whatever of ``modules_for`` is not built yet."""
    from gllm_b200.ops.build import compile_modules

    compile_modules(modules_for(dtype, head_dims, sampling, modules))


# number of kernel launches made through this module (benchmarks read it)
launch_count = 0


def _check(code: int, what: str) -> None:
    global launch_count
    launch_count += 1
    if code != 0:
        raise RuntimeError(f"{what}: launch failed: {_error_string(code)} (code {code})")


def _suffix(dtype: torch.dtype) -> str:
    if dtype == torch.float32:
        return "f32"
    if dtype == torch.bfloat16:
        return "bf16"
    raise TypeError(f"kernels take float32 or bfloat16 activations, not {dtype}")


def _cuda(t: torch.Tensor, name: str, dtype: torch.dtype | None = None, contiguous: bool = True) -> None:
    if not isinstance(t, torch.Tensor) or not t.is_cuda:
        raise RuntimeError(f"{name} must be a CUDA tensor: this engine has no CPU path")
    if dtype is not None and t.dtype != dtype:
        raise TypeError(f"{name} must be {dtype}, is {t.dtype}")
    if contiguous and not t.is_contiguous():
        raise ValueError(f"{name} must be contiguous")


_raw_stream = getattr(torch._C, "_cuda_getCurrentRawStream", None)


def _stream() -> int:
    """The current CUDA stream's handle (every kernel is launched on it).  The raw getter costs a
    fraction of a microsecond; building a ``torch.cuda.Stream`` object for every launch cost 15 us."""
    if _raw_stream is not None:
        return _raw_stream(torch.cuda.current_device())
    return torch.cuda.current_stream().cuda_stream


def _ptr(t: torch.Tensor | None) -> int | None:
    return None if t is None else t.data_ptr()


# ------------------------------------------------------------------- status
_status: dict[int, torch.Tensor] = {}

STATUS_BITS = {
    1: "a token id outside the vocabulary",
    2: "a cache page id outside the pool",
    4: "a bounded wait inside a kernel ran out",
}


def status_word(device: torch.device | int | None = None) -> torch.Tensor:
    """The device's int32 status word that kernels OR error bits into."""
    idx = torch.cuda.current_device() if device is None else torch.device(device).index
    if idx is None:
        idx = torch.cuda.current_device()
    t = _status.get(idx)
    if t is None:
        t = torch.zeros(1, dtype=torch.int32, device=f"cuda:{idx}")
        _status[idx] = t
    return t


def check_status(device=None) -> None:
    """Read the status word (a device sync) and raise if a kernel set a bit."""
    t = status_word(device)
    value = int(t.item())
    if value:
        t.zero_()
        reasons = [text for bit, text in STATUS_BITS.items() if value & bit] or [f"status {value}"]
        raise RuntimeError("a kernel reported: " + "; ".join(reasons))


# ------------------------------------------------------------ unsummed splits
class SplitSum:
    """The result of a product that was cut along K and whose ``splits`` fp32
    partial results ``parts [splits, rows, cols]`` were left unsummed: the
    kernel that consumes it (``add_rmsnorm``, ``rope_store``) adds them in
    ascending order, which saves a reduction pass.  ``parts`` lives in one of
    two scratch buffers that the products take in turn: it survives the next
    product and is overwritten by the one after.  Consume a SplitSum (or call
    ``as_tensor`` on it) before two more products have run; reading it later
    raises."""

    def __init__(self, parts: torch.Tensor, dtype: torch.dtype, generation: int | None = None):
        self.parts = parts
        self.dtype = dtype
        # the count of scratch-taking products on the device when this one ran (None: the parts are
        # the caller's own memory)
        self.generation = generation

    def check_alive(self) -> None:
        if self.generation is None:
            return
        from gllm_b200.ops import gemm_bf16

        now = gemm_bf16.scratch_generation(self.parts.device)
        if now - self.generation > 1:
            raise RuntimeError(
                f"an unsummed product was read after {now - self.generation} further products: its partial sums "
                "have been overwritten (sum it with ops.as_tensor before running two more products)")

    @property
    def shape(self):
        return self.parts.shape[1:]

    @property
    def device(self):
        return self.parts.device

    def tensor(self, out: torch.Tensor | None = None) -> torch.Tensor:
        """The summed result as an ordinary tensor of ``dtype`` (into ``out``, contiguous, when given)."""
        self.check_alive()
        if out is None:
            out = torch.empty(tuple(self.shape), dtype=self.dtype, device=self.parts.device)
        f = _fn("elementwise", f"gllm_sum_parts_{_suffix(self.dtype)}")
        _check(f(self.parts.data_ptr(), self.parts.shape[0], self.parts.stride(0), out.data_ptr(), out.numel(),
                 _stream()), "sum_parts")
        return out


class _Added:
    """What a product returns when it has added its result into the matrix it was given
    (``linear(..., add_into=...)``): there is nothing left to add."""

    def __repr__(self):
        return "ops.ADDED"


ADDED = _Added()


class RowSum:
    """The result of routed experts that has not been added up per token: ``y [parts, rows, width]`` (fp32; the parts are
    added first), of which token ``t``'s row is the sum over its ``top`` slots of rows ``row_of_pair[t * top + s]``
    (without ``row_of_pair``: ``t * top + s``), times ``weights [tokens, top]`` when given.  The kernel that norms and
    adds a sublayer's result (``add_cast``, ``add_rmsnorm`` of a ``Pending``) takes it as it is."""

    def __init__(self, y: torch.Tensor, row_of_pair, weights, tokens: int, top: int, dtype: torch.dtype):
        self.y, self.row_of_pair, self.weights, self.top, self.dtype = y, row_of_pair, weights, int(top), dtype
        self.shape = (int(tokens), y.shape[-1])

    def tensor(self) -> torch.Tensor:
        from gllm_b200.ops import moe

        return moe.combine(self.y, self.weights, None, self.dtype, self.row_of_pair, tokens=self.shape[0], top=self.top)


def as_tensor(x):
    """``x`` itself, or the summed tensor of a SplitSum (or a RowSum)."""
    return x.tensor() if isinstance(x, (SplitSum, RowSum)) else x


class Pending:
    """What is still to be added to the fp32 residual stream when the next norm runs: ``value`` (a tensor of the
    activation type, a SplitSum, or None), first RMS-normed with ``post_weight`` and ``post_eps`` when a weight is
    given (a layer that norms a sublayer's result before it joins the residual), and ``extra``: a second fp32
    stream of the residual's shape that is added as it is.  ``add_rmsnorm`` does all of it in one kernel."""

    def __init__(self, value=None, post_weight: torch.Tensor | None = None, post_eps: float = 0.0,
                 extra: torch.Tensor | None = None):
        self.value, self.post_weight, self.post_eps, self.extra = value, post_weight, float(post_eps), extra

    @classmethod
    def of(cls, branch) -> "Pending":
        """``branch`` as a Pending: itself, or a plain add of a tensor / SplitSum (nothing for None and ADDED)."""
        if isinstance(branch, Pending):
            return branch
        return cls(None if branch is None or branch is ADDED else branch)

    def with_extra(self, extra: torch.Tensor) -> "Pending":
        if self.extra is not None:
            raise ValueError("a second stream is already pending")
        return Pending(self.value, self.post_weight, self.post_eps, extra)


class Biased:
    """The result of a branch's last product (a tensor or a SplitSum) whose bias (fp32, one value per column) has not
    been added yet: for blocks whose next kernel adds it (``StepContext.takes_bias``)."""

    def __init__(self, value, bias: torch.Tensor):
        self.value, self.bias = value, bias


class DepthPending:
    """What is still to be done to the fp32 residual when the next norm runs: ``value`` (a tensor of the activation type
    or a SplitSum, with ``value_bias`` still to be added) is RMS-normed with ``post_weight`` and ``post_eps`` and added;
    with ``depth_weight`` (fp32 ``[count + 1]``) the sum ``X`` is then replaced by the weighted sum over ``streams
    [>= count + 1, n, width]`` (fp32: ``count`` earlier streams and a place for ``X``).  ``value`` None: nothing is
    added."""

    def __init__(self, value=None, value_bias=None, post_weight=None, post_eps: float = 0.0, streams=None,
                 count: int = 0, depth_weight=None):
        self.value, self.value_bias, self.post_weight, self.post_eps = value, value_bias, post_weight, float(post_eps)
        self.streams, self.count, self.depth_weight = streams, int(count), depth_weight


def _parts_args(x):
    if isinstance(x, SplitSum):
        x.check_alive()
        return x.parts.data_ptr(), x.parts.shape[0], x.parts.stride(0)
    return None, 0, 0


# ---------------------------------------------------------------- embedding
def embedding(tokens: torch.Tensor, table: torch.Tensor, out: torch.Tensor | None = None,
              sampled: torch.Tensor | None = None, token_row: torch.Tensor | None = None,
              scale: float = 1.0) -> torch.Tensor:
    """fp32 residual rows ``table[tokens] * scale`` (gllm/model/model.py:175-182; the reference has
    no multiplier).

    With ``sampled`` and ``token_row``: a negative token id stands for
    ``sampled[token_row[i]]``, the token the previous step's argmax left on the
    device for that request, so a decode step can be queued before the host
    has seen the previous step's tokens."""
    _cuda(tokens, "tokens", torch.int32)
    if sampled is not None:
        _cuda(sampled, "sampled", torch.int32)
        _cuda(token_row, "token_row", torch.int32)
    _cuda(table, "table")
    n, (vocab, hidden) = tokens.numel(), table.shape
    if out is None:
        out = torch.empty((n, hidden), dtype=torch.float32, device=table.device)
    else:
        _cuda(out, "out", torch.float32)
    f = _fn("elementwise", f"gllm_embedding_{_suffix(table.dtype)}")
    _check(f(tokens.data_ptr(), _ptr(sampled), _ptr(token_row) if sampled is not None else None, table.data_ptr(),
             out.data_ptr(), n, hidden, vocab, float(scale), status_word(table.device).data_ptr(), _stream()),
           "embedding")
    return out


def scatter_int32(dst: torch.Tensor, index: torch.Tensor, values: torch.Tensor) -> None:
    """``dst.view(-1)[index[i]] = values[i]`` for int32 tensors (indices are distinct); an index
    outside ``dst`` sets a status bit and is skipped."""
    _cuda(dst, "dst", torch.int32)
    _cuda(index, "index", torch.int32)
    _cuda(values, "values", torch.int32)
    if index.numel() != values.numel():
        raise ValueError("index and values differ in length")
    f = _fn("elementwise", "gllm_scatter_i32")
    _check(f(dst.data_ptr(), dst.numel(), index.data_ptr(), values.data_ptr(), index.numel(),
             status_word(dst.device).data_ptr(), _stream()), "scatter_int32")


def scale_softcap(logits: torch.Tensor, scale: float = 1.0, cap: float | None = None) -> torch.Tensor:
    """In place on fp32 ``logits``: multiply by ``scale``, then with ``cap``: ``cap * tanh(x / cap)``."""
    _cuda(logits, "logits", torch.float32)
    f = _fn("elementwise", "gllm_scale_softcap_f32")
    _check(f(logits.data_ptr(), logits.numel(), float(scale), float(cap or 0.0), _stream()), "scale_softcap")
    return logits


# ------------------------------------------------- bias, norm of every head
def add_bias(x: torch.Tensor, bias: torch.Tensor) -> torch.Tensor:
    """``x[r] += bias`` in place (``bias`` fp32, one value per column): the bias of a projection.  The
    reference's projections have none (gllm/model/layers/linear.py:20)."""
    _cuda(x, "x", contiguous=False)
    _cuda(bias, "bias", torch.float32)
    if x.dim() != 2 or x.stride(1) != 1 or bias.numel() != x.shape[1]:
        raise ValueError("add_bias takes rows of contiguous columns and one bias value per column")
    f = _fn("elementwise", f"gllm_add_bias_{_suffix(x.dtype)}")
    _check(f(x.data_ptr(), x.stride(0), bias.data_ptr(), x.shape[0], x.shape[1], _stream()), "add_bias")
    return x


def rmsnorm_heads(x: torch.Tensor, weight: torch.Tensor, eps: float, first_head: int, num_heads: int, head_dim: int,
                  unit_offset: bool = False) -> torch.Tensor:
    """RMSNorm of each of ``num_heads`` heads of ``head_dim`` columns, from head ``first_head`` on, of every row
    of ``x``, in place, with one weight of ``head_dim`` values for all of them; statistics in fp32.  (A norm of
    the queries and keys before their rotation; the reference has none.)"""
    _cuda(x, "x", contiguous=False)
    _cuda(weight, "weight", torch.float32)
    if x.dim() != 2 or x.stride(1) != 1 or (first_head + num_heads) * head_dim > x.shape[1]:
        raise ValueError("the heads do not lie inside the rows of x")
    if weight.numel() != head_dim or head_dim > 256:
        raise ValueError("rmsnorm_heads takes one weight value per column of a head, for heads of up to 256 columns")
    f = _fn("elementwise", f"gllm_rmsnorm_heads_{_suffix(x.dtype)}")
    _check(f(x.data_ptr(), x.stride(0), weight.data_ptr(), x.shape[0], int(first_head), int(num_heads), int(head_dim),
             float(eps), int(unit_offset), _stream()), "rmsnorm_heads")
    return x


# ------------------------------------------------------------- add + RMSNorm
def add_rmsnorm(
    branch: torch.Tensor | None,
    resid: torch.Tensor,
    weight: torch.Tensor,
    eps: float,
    out_dtype: torch.dtype,
    rows: torch.Tensor | None = None,
    unit_offset: bool = False,
    out: torch.Tensor | None = None,
) -> torch.Tensor:
    """``resid += branch`` (fp32, in place) then RMSNorm of the sum.

    With ``rows`` only those rows are normed and ``resid`` is left untouched.
    """
    _cuda(resid, "resid", torch.float32)
    _cuda(weight, "weight", torch.float32)
    hidden = resid.shape[-1]
    if weight.numel() != hidden:
        raise ValueError(f"norm weight has {weight.numel()} elements, rows have {hidden}")
    if isinstance(branch, DepthPending):
        from gllm_b200.ops import depth

        if unit_offset or out is not None:
            raise ValueError("a norm over a depth average takes a plain weight and makes its own result")
        return depth.depth_norm(branch, resid, weight, eps, out_dtype, rows)
    if isinstance(branch, Pending):
        if branch.post_weight is None and branch.extra is None:
            branch = branch.value
        else:
            if unit_offset:
                raise ValueError("a norm whose weight is stored around zero does not take a pending normed branch")
            return _pending_add_rmsnorm(branch, resid, weight, eps, out_dtype, rows, out)
    parts_ptr, n_parts, part_stride = _parts_args(branch)
    if isinstance(branch, SplitSum):
        if tuple(branch.shape) != tuple(resid.shape) or branch.dtype != out_dtype:
            raise ValueError("branch and resid differ in shape or dtype")
        branch = None
    elif branch is not None:
        _cuda(branch, "branch", out_dtype)
        if branch.shape != resid.shape:
            raise ValueError("branch and resid differ in shape")
    if rows is not None:
        _cuda(rows, "rows", torch.int32)
        n_rows = rows.numel()
    else:
        n_rows = resid.numel() // hidden
    if out is None:
        out = torch.empty((n_rows, hidden), dtype=out_dtype, device=resid.device)
    else:
        _cuda(out, "out", out_dtype)
    f = _fn("elementwise", f"gllm_add_rmsnorm_{_suffix(out_dtype)}")
    _check(f(_ptr(branch), parts_ptr, n_parts, part_stride, resid.data_ptr(), weight.data_ptr(), out.data_ptr(),
             _ptr(rows), n_rows, hidden, float(eps), int(unit_offset), _stream()), "add_rmsnorm")
    return out


def add_cast(branch, resid: torch.Tensor, out_dtype: torch.dtype) -> torch.Tensor:
    """``resid += branch`` (fp32, in place; a ``Pending`` is normed first where it says so) and the sum rounded to
    ``out_dtype``: what a sublayer reads that no norm precedes (``csrc/postnorm.cu``)."""
    _cuda(resid, "resid", torch.float32)
    return _pending_add_rmsnorm(Pending.of(branch), resid, None, 0.0, out_dtype, None, None)


def _pending_add_rmsnorm(pending: Pending, resid, weight, eps, out_dtype, rows, out):
    """``resid += rms(value) * post_weight + extra`` and the RMS norm of the sum, or without ``weight`` the sum itself
    (``csrc/postnorm.cu``)."""
    n_total, hidden = resid.numel() // resid.shape[-1], resid.shape[-1]
    value = pending.value
    parts_ptr, n_parts, part_stride = _parts_args(value)
    row_sum = (None, 0, 0, None, None, 0)
    if isinstance(value, RowSum):
        if tuple(value.shape) != tuple(resid.shape) or value.dtype != out_dtype:
            raise ValueError("the pending rows and the residual differ in shape or dtype")
        row_sum = (value.y.data_ptr(), value.y.shape[0], value.y.stride(0), _ptr(value.row_of_pair), _ptr(value.weights),
                   value.top)
        value = None
    elif isinstance(value, SplitSum):
        if tuple(value.shape) != tuple(resid.shape) or value.dtype != out_dtype:
            raise ValueError("the pending value and the residual differ in shape or dtype")
        value = None
    elif value is not None:
        _cuda(value, "value", out_dtype)
        if value.shape != resid.shape:
            raise ValueError("the pending value and the residual differ in shape")
    if pending.post_weight is not None:
        _cuda(pending.post_weight, "post_weight", torch.float32)
        if pending.post_weight.numel() != hidden:
            raise ValueError("the post-norm weight needs one value per column")
    if pending.extra is not None:
        _cuda(pending.extra, "extra", torch.float32)
        if pending.extra.shape != resid.shape:
            raise ValueError("the second stream and the residual differ in shape")
    n_rows = n_total if rows is None else rows.numel()
    if rows is not None:
        _cuda(rows, "rows", torch.int32)
    if out is None:
        out = torch.empty((n_rows, hidden), dtype=out_dtype, device=resid.device)
    else:
        _cuda(out, "out", out_dtype)
    f = _fn("postnorm", f"gllm_postnorm_add_rmsnorm_{_suffix(out_dtype)}")
    _check(f(_ptr(value), parts_ptr, n_parts, part_stride, _ptr(pending.post_weight), pending.post_eps,
             _ptr(pending.extra), resid.data_ptr(), _ptr(weight), float(eps), out.data_ptr(), _ptr(rows), n_rows,
             hidden, *row_sum, _stream()), "postnorm_add_rmsnorm")
    return out


# ------------------------------------------------------- add + a norm without a statistic
def add_dyt(branch, resid: torch.Tensor, alpha: torch.Tensor, weight: torch.Tensor, bias: torch.Tensor | None,
            out_dtype: torch.dtype, rows: torch.Tensor | None = None) -> torch.Tensor:
    """``resid += branch`` (fp32, in place) then ``tanh(alpha * resid) * weight + bias``: a norm that takes no
    statistic of its row.  ``alpha``: one fp32 number on the device.  ``branch``: a tensor of ``out_dtype``, a
    SplitSum, a plain ``Pending`` or None.  With ``rows`` only those rows are computed and ``resid`` is left untouched."""
    _cuda(resid, "resid", torch.float32)
    _cuda(alpha, "alpha", torch.float32)
    _cuda(weight, "weight", torch.float32)
    hidden = resid.shape[-1]
    if weight.numel() != hidden or alpha.numel() != 1 or (bias is not None and bias.numel() != hidden):
        raise ValueError("the norm takes one alpha and one weight (and bias) value per column")
    if bias is not None:
        _cuda(bias, "bias", torch.float32)
    if isinstance(branch, Pending):
        if branch.post_weight is not None or branch.extra is not None:
            raise ValueError("this norm takes a plain pending branch only")
        branch = branch.value
    parts_ptr, n_parts, part_stride = _parts_args(branch)
    if isinstance(branch, SplitSum):
        if tuple(branch.shape) != tuple(resid.shape) or branch.dtype != out_dtype:
            raise ValueError("branch and resid differ in shape or dtype")
        branch = None
    elif branch is not None:
        _cuda(branch, "branch", out_dtype)
        if branch.shape != resid.shape:
            raise ValueError("branch and resid differ in shape")
    if rows is not None:
        _cuda(rows, "rows", torch.int32)
        n_rows = rows.numel()
    else:
        n_rows = resid.numel() // hidden
    out = torch.empty((n_rows, hidden), dtype=out_dtype, device=resid.device)
    f = _fn("dyt_norm", f"gllm_add_dyt_{_suffix(out_dtype)}")
    _check(f(_ptr(branch), parts_ptr, n_parts, part_stride, resid.data_ptr(), alpha.data_ptr(), weight.data_ptr(),
             _ptr(bias), out.data_ptr(), _ptr(rows), n_rows, hidden, _stream()), "add_dyt")
    return out


# ------------------------------------------------------------------ SiLU·up
GATED_BLOCK = 64


def silu_mul(gate_up: torch.Tensor, out: torch.Tensor | None = None, block: int = 0,
             bias: torch.Tensor | None = None) -> torch.Tensor:
    """``silu(gate) * up`` of ``[n, 2*inter]``.  ``block`` 0: gate columns first, up columns after;
    ``block`` b: b gate columns alternate with the b up columns of the same features.  ``bias`` (fp32, one value per
    column of ``gate_up``) is added first, with the rounding a product with a bias gives its result."""
    _cuda(gate_up, "gate_up")
    if bias is not None:
        _cuda(bias, "bias", torch.float32)
        if bias.numel() != gate_up.shape[1]:
            raise ValueError("one bias value per column of gate_up is needed")
    n, two_i = gate_up.shape
    if two_i % 2:
        raise ValueError("gate_up must have an even number of columns")
    inter = two_i // 2
    if out is None:
        out = torch.empty((n, inter), dtype=gate_up.dtype, device=gate_up.device)
    f = _fn("elementwise", f"gllm_silu_mul_{_suffix(gate_up.dtype)}")
    _check(f(gate_up.data_ptr(), out.data_ptr(), n, inter, int(block), _ptr(bias), _stream()), "silu_mul")
    return out


def interleave_gate_up(gate: torch.Tensor, up: torch.Tensor, block: int = GATED_BLOCK) -> torch.Tensor:
    """Stack ``gate`` and ``up`` ``[inter, hidden]`` so that ``block`` gate rows alternate with the
    ``block`` up rows of the same features (``inter`` must be a multiple of ``block``)."""
    inter, hidden = gate.shape
    if inter % block:
        raise ValueError("intermediate size must be a multiple of the block")
    stacked = torch.stack([gate.view(inter // block, block, hidden), up.view(inter // block, block, hidden)], dim=1)
    return stacked.reshape(2 * inter, hidden).contiguous()


def linear_gated(x: torch.Tensor, weight: torch.Tensor, slope: float = 1.0, limit: float | None = None,
                 up_offset: float = 0.0) -> torch.Tensor:
    """``a(x @ Wg.T) * (x @ Wu.T + up_offset)`` for a weight stacked by ``interleave_gate_up``, with
    ``a(g) = g * sigmoid(slope * g)`` and, with ``limit``, the gate capped at ``limit`` and the up product
    clamped to ``[-limit, limit]`` first (the defaults are ``silu(gate) * up``): one kernel with the activation
    in the product's epilogue where the tensor-core kernel takes the operands, the product and the pointwise
    kernel otherwise."""
    _cuda(x, "x")
    _cuda(weight, "weight", x.dtype)
    plain = slope == 1.0 and limit is None and up_offset == 0.0
    if x.dtype == torch.bfloat16:
        from gllm_b200.ops import gemm_bf16

        fused = gemm_bf16.linear_gated(x, weight, slope=slope, limit=limit, up_offset=up_offset)
        if fused is not None:
            return fused
    if plain:
        return silu_mul(linear(x, weight), block=GATED_BLOCK)
    return gated_activation(linear(x, weight), slope=slope, limit=limit, up_offset=up_offset, block=GATED_BLOCK)


def relu_sq(x: torch.Tensor) -> torch.Tensor:
    """``max(x, 0) ** 2``: the activation of a dense feed-forward without a gate."""
    _cuda(x, "x")
    out = torch.empty_like(x)
    f = _fn("elementwise", f"gllm_relu_sq_{_suffix(x.dtype)}")
    _check(f(x.data_ptr(), out.data_ptr(), x.numel(), _stream()), "relu_sq")
    return out


def scaled_sum(x: torch.Tensor, y: torch.Tensor, a: float, b: float) -> torch.Tensor:
    """``a * x + b * y`` (computed in fp32) of two tensors of equal shape and type."""
    _cuda(x, "x")
    _cuda(y, "y", x.dtype)
    if x.shape != y.shape:
        raise ValueError("scaled_sum takes two tensors of equal shape")
    out = torch.empty_like(x)
    f = _fn("elementwise", f"gllm_scaled_sum_{_suffix(x.dtype)}")
    _check(f(x.data_ptr(), y.data_ptr(), out.data_ptr(), float(a), float(b), x.numel(), _stream()), "scaled_sum")
    return out


# ------------------------------- gated activation with clamps; residual add; join; whole-projection norm
def gated_activation(gate_up: torch.Tensor, slope: float = 1.0, limit: float | None = None, up_offset: float = 0.0,
                     block: int = 0, out: torch.Tensor | None = None) -> torch.Tensor:
    """``g * sigmoid(slope * g) * (u + up_offset)`` of ``[n, 2*inter]`` with ``g = min(gate, limit)`` and
    ``u = clamp(up, -limit, limit)`` (no clamps without ``limit``); columns laid out as for ``silu_mul``."""
    _cuda(gate_up, "gate_up")
    n, two_i = gate_up.shape
    if two_i % 2:
        raise ValueError("gate_up must have an even number of columns")
    inter = two_i // 2
    if out is None:
        out = torch.empty((n, inter), dtype=gate_up.dtype, device=gate_up.device)
    f = _fn("elementwise", f"gllm_gated_act_{_suffix(gate_up.dtype)}")
    _check(f(gate_up.data_ptr(), out.data_ptr(), n, inter, int(block), float(slope), float(limit or 0.0),
             float(up_offset), _stream()), "gated_activation")
    return out


def residual_add(resid: torch.Tensor, branch, dtype: torch.dtype | None = None) -> torch.Tensor:
    """``resid += branch`` in place on the fp32 residual stream; ``branch`` is a tensor of the activation type
    or a SplitSum (summed in ascending order and rounded to its type first)."""
    _cuda(resid, "resid", torch.float32)
    parts_ptr, n_parts, part_stride = _parts_args(branch)
    if isinstance(branch, SplitSum):
        if tuple(branch.shape) != tuple(resid.shape):
            raise ValueError("branch and resid differ in shape")
        t, ptr = branch.dtype, None
    else:
        _cuda(branch, "branch")
        if branch.shape != resid.shape:
            raise ValueError("branch and resid differ in shape")
        t, ptr = branch.dtype, branch.data_ptr()
    f = _fn("elementwise", f"gllm_residual_add_{_suffix(t)}")
    _check(f(ptr, parts_ptr, n_parts, part_stride, resid.data_ptr(), resid.numel(), _stream()), "residual_add")
    return resid


def join_rows(branch, resid: torch.Tensor, other: torch.Tensor, out_dtype: torch.dtype) -> torch.Tensor:
    """``[resid (+ branch) ; other]`` as ``[n, 2 * hidden]`` of ``out_dtype``: the residual stream (with a branch
    that has not been added yet: a tensor, a SplitSum or None) beside a second fp32 stream of the same shape."""
    _cuda(resid, "resid", torch.float32)
    _cuda(other, "other", torch.float32)
    if other.shape != resid.shape or resid.dim() != 2:
        raise ValueError("join_rows takes two [n, hidden] streams of equal shape")
    parts_ptr, n_parts, part_stride = _parts_args(branch)
    ptr = None
    if isinstance(branch, SplitSum):
        if tuple(branch.shape) != tuple(resid.shape) or branch.dtype != out_dtype:
            raise ValueError("branch and resid differ in shape or dtype")
    elif branch is not None:
        _cuda(branch, "branch", out_dtype)
        if branch.shape != resid.shape:
            raise ValueError("branch and resid differ in shape")
        ptr = branch.data_ptr()
    n, hidden = resid.shape
    out = torch.empty((n, 2 * hidden), dtype=out_dtype, device=resid.device)
    f = _fn("elementwise", f"gllm_join_rows_{_suffix(out_dtype)}")
    _check(f(ptr, parts_ptr, n_parts, part_stride, resid.data_ptr(), other.data_ptr(), out.data_ptr(), n, hidden,
             _stream()), "join_rows")
    return out


def qk_rownorm(qk, q_weight: torch.Tensor | None, k_weight: torch.Tensor | None, eps: float, q_cols: int, k_cols: int,
               values_from_keys: bool = True) -> torch.Tensor:
    """From the q and k projections ``[n, q_cols + k_cols]`` (a tensor or a SplitSum; with
    ``values_from_keys=False`` a v projection of ``k_cols`` follows) to ``[n, q_cols + 2 * k_cols]``: q and k
    RMS-normed over their WHOLE projection (all heads at once) with one weight per column, values = the keys as
    projected (or the v projection, copied).  A weight of None leaves that projection un-normed."""
    parts_ptr, n_parts, part_stride = _parts_args(qk)
    in_cols = q_cols + k_cols + (0 if values_from_keys else k_cols)
    if isinstance(qk, SplitSum):
        n, cols, t, ptr, stride, device = qk.shape[0], qk.shape[1], qk.dtype, None, 0, qk.device
    else:
        _cuda(qk, "qk", contiguous=False)
        if qk.dim() != 2 or qk.stride(1) != 1:
            raise ValueError("qk must be [tokens, columns] with contiguous columns")
        n, cols, t, ptr, stride, device = qk.shape[0], qk.shape[1], qk.dtype, qk.data_ptr(), qk.stride(0), qk.device
    if cols != in_cols:
        raise ValueError(f"the projection has {cols} columns, {in_cols} were expected")
    for w, size, name in ((q_weight, q_cols, "q_weight"), (k_weight, k_cols, "k_weight")):
        if w is not None:
            _cuda(w, name, torch.float32)
            if w.numel() != size:
                raise ValueError(f"{name} needs one value per column of its projection")
    out = torch.empty((n, q_cols + 2 * k_cols), dtype=t, device=device)
    f = _fn("elementwise", f"gllm_qk_rownorm_{_suffix(t)}")
    _check(f(ptr, stride, parts_ptr, n_parts, part_stride, _ptr(q_weight), _ptr(k_weight), out.data_ptr(), n,
             int(q_cols), int(k_cols), int(values_from_keys), float(eps), _stream()), "qk_rownorm")
    return out


# --------------------------------------------------- rotary + cache store
def rope_store(
    qkv: torch.Tensor,
    positions: torch.Tensor,
    inv_freq: torch.Tensor | None,
    slot_mapping: torch.Tensor | None,
    cache_layer: torch.Tensor | None,
    num_heads: int,
    num_kv_heads: int,
    head_dim: int,
    rotary_dim: int,
    interleaved: bool = False,
) -> torch.Tensor:
    """Rotate q and k of ``qkv`` in place and store k, v into the cache;
    returns ``qkv`` (a SplitSum is summed into a new tensor first, in the same
    kernel).

    ``cache_layer`` is ``[pages, 2, kv_heads, block_size, head_dim]``.
    """
    parts_ptr, n_parts, part_stride = _parts_args(qkv)
    if isinstance(qkv, SplitSum):
        qkv = torch.empty(tuple(qkv.shape), dtype=qkv.dtype, device=qkv.device)
    _cuda(qkv, "qkv")
    _cuda(positions, "positions", torch.int32)
    n = qkv.shape[0]
    if qkv.shape[1] != (num_heads + 2 * num_kv_heads) * head_dim:
        raise ValueError("qkv width does not equal (heads + 2*kv_heads) * head_dim")
    if inv_freq is not None:
        _cuda(inv_freq, "inv_freq", torch.float32)
        if inv_freq.numel() != rotary_dim // 2:
            raise ValueError("inv_freq must hold rotary_dim/2 frequencies")
    block_size = num_pages = 0
    if slot_mapping is not None:
        _cuda(slot_mapping, "slot_mapping", torch.int32)
        _cuda(cache_layer, "cache_layer", qkv.dtype)
        num_pages, two, hkv, block_size, d = cache_layer.shape
        if two != 2 or hkv != num_kv_heads or d != head_dim:
            raise ValueError("cache layer shape does not match the mixer's heads")
    f = _fn("elementwise", f"gllm_rope_store_{_suffix(qkv.dtype)}")
    _check(f(qkv.data_ptr(), parts_ptr, n_parts, part_stride, positions.data_ptr(), _ptr(inv_freq),
             _ptr(slot_mapping), _ptr(cache_layer) if slot_mapping is not None else None, n, num_heads,
             num_kv_heads, head_dim, rotary_dim, int(interleaved), block_size, num_pages,
             status_word(qkv.device).data_ptr(), _stream()), "rope_store")
    return qkv


def rope_norm_store(qkv, positions: torch.Tensor, inv_freq: torch.Tensor | None, magnitude: float,
                    slot_mapping: torch.Tensor | None, cache_layer: torch.Tensor | None, num_heads: int,
                    num_kv_heads: int, head_dim: int, rotary_dim: int, interleaved: bool, norm_dim: int,
                    eps: float) -> torch.Tensor:
    """As ``rope_store`` for layers whose sine and cosine are multiplied by ``magnitude`` and whose query and key
    heads are divided, AFTER the rotation, by ``sqrt(sum(x^2) / norm_dim + eps)`` (``norm_dim`` 0: no norm; it may
    be smaller than ``head_dim`` when heads are stored with zero columns behind them).  Returns ``qkv``."""
    parts_ptr, n_parts, part_stride = _parts_args(qkv)
    if isinstance(qkv, SplitSum):
        qkv = torch.empty(tuple(qkv.shape), dtype=qkv.dtype, device=qkv.device)
    _cuda(qkv, "qkv")
    _cuda(positions, "positions", torch.int32)
    n = qkv.shape[0]
    if qkv.shape[1] != (num_heads + 2 * num_kv_heads) * head_dim:
        raise ValueError("qkv width does not equal (heads + 2*kv_heads) * head_dim")
    if inv_freq is not None:
        _cuda(inv_freq, "inv_freq", torch.float32)
        if inv_freq.numel() != rotary_dim // 2:
            raise ValueError("inv_freq must hold rotary_dim/2 frequencies")
    block_size = num_pages = 0
    if slot_mapping is not None:
        _cuda(slot_mapping, "slot_mapping", torch.int32)
        _cuda(cache_layer, "cache_layer", qkv.dtype)
        num_pages, two, hkv, block_size, d = cache_layer.shape
        if two != 2 or hkv != num_kv_heads or d != head_dim:
            raise ValueError("cache layer shape does not match the mixer's heads")
    f = _fn("rope_norm", f"gllm_rope_norm_store_{_suffix(qkv.dtype)}")
    _check(f(qkv.data_ptr(), parts_ptr, n_parts, part_stride, positions.data_ptr(), _ptr(inv_freq), float(magnitude),
             _ptr(slot_mapping), _ptr(cache_layer) if slot_mapping is not None else None, n, num_heads, num_kv_heads,
             head_dim, rotary_dim if inv_freq is not None else 0, int(interleaved), int(norm_dim), float(eps),
             block_size, num_pages, status_word(qkv.device).data_ptr(), _stream()), "rope_norm_store")
    return qkv


# ------------------------------------------------------------------- linear
# Products of few tokens that end a branch add themselves into the residual stream
# (GLLM_B200_FUSE_ADD=0: they leave their result to the norm kernel after them).
ACCUMULATE_IN_PRODUCT = os.environ.get("GLLM_B200_FUSE_ADD", "1") != "0"


def linear(x: torch.Tensor, weight: torch.Tensor, out_dtype: torch.dtype | None = None,
           out: torch.Tensor | None = None, split_ok: bool = False, add_into: torch.Tensor | None = None,
           bias: torch.Tensor | None = None):
    """``x @ weight.T`` with ``weight`` stored ``[out, in]``
    (gllm/model/layers/linear.py:20).  fp32 inputs run the FFMA kernel (no
    tensor-core mode); bf16 inputs run the tensor-core kernels with fp32
    accumulation.  With ``split_ok`` the result may be a SplitSum (for callers
    that hand it to ``add_rmsnorm`` or ``rope_store``).  With ``add_into``
    (fp32 ``[m, n]``, the residual stream) the product may add itself there
    and return ``ADDED``; when it returns anything else, nothing was added.  With ``bias`` (fp32, one
    value per output column) the result is an ordinary tensor with the bias added."""
    if bias is not None:
        return add_bias(linear(x, weight, out_dtype=out_dtype, out=out), bias)
    _cuda(x, "x", contiguous=False)             # rows may be a slice of wider rows
    _cuda(weight, "weight", x.dtype)
    if x.dim() != 2 or x.stride(1) != 1:
        raise ValueError("x must be [tokens, columns] with contiguous columns")
    m, k = x.shape
    n, k2 = weight.shape
    if k != k2:
        raise ValueError(f"x has {k} columns, weight has {k2}")
    out_dtype = out_dtype or x.dtype
    if add_into is not None and x.dtype == torch.bfloat16 and out is None and ACCUMULATE_IN_PRODUCT:
        from gllm_b200.ops import gemm_bf16

        if gemm_bf16.linear_accumulate(x, weight, add_into):
            return ADDED
    if x.dtype == torch.bfloat16 and split_ok and out is None:
        from gllm_b200.ops import gemm_bf16

        split = gemm_bf16.linear_split(x, weight, out_dtype)
        if split is not None:
            return split
    if out is None:
        out = torch.empty((m, n), dtype=out_dtype, device=x.device)
    else:
        _cuda(out, "out", out_dtype)
    if x.dtype == torch.float32:
        if out_dtype != torch.float32:
            raise TypeError("the fp32 product writes fp32")
        f = _fn("gemm_fp32", "gllm_gemm_f32")
        _check(f(x.data_ptr(), weight.data_ptr(), out.data_ptr(), m, n, k, x.stride(0), k, n, _stream()), "gemm_f32")
        return out
    from gllm_b200.ops import gemm_bf16

    return gemm_bf16.linear_bf16(x, weight, out)


# ---------------------------------------------------------------- attention
def paged_attention_simt(
    q: torch.Tensor,
    q_stride: int,
    cache_layer: torch.Tensor,
    block_table: torch.Tensor,
    positions: torch.Tensor,
    token_row: torch.Tensor,
    num_heads: int,
    scale: float,
    window: int,
    out: torch.Tensor,
) -> torch.Tensor:
    num_pages, _, hkv, block_size, d = cache_layer.shape
    n = positions.numel()
    f = _fn("attention_simt", f"gllm_attention_simt_{_suffix(q.dtype)}")
    _check(f(q.data_ptr(), q_stride, out.data_ptr(), out.shape[1], cache_layer.data_ptr(), block_table.data_ptr(),
             block_table.stride(0), positions.data_ptr(), token_row.data_ptr(), n, num_heads, hkv, d, block_size,
             num_pages, float(scale), int(window), status_word(q.device).data_ptr(), _stream()), "attention_simt")
    return out


def paged_attention(
    qkv: torch.Tensor,
    cache_layer: torch.Tensor,
    block_table: torch.Tensor,
    positions: torch.Tensor,
    token_row: torch.Tensor,
    num_heads: int,
    scale: float,
    window: int | None = None,
    batch=None,
    out: torch.Tensor | None = None,
    chunk: int | None = None,
) -> torch.Tensor:
    """Causal attention of every token of the batch over its request's cache: over all keys, the last ``window``, or
    (``chunk``) those of the query's own chunk of ``chunk`` positions, counted from the sequence's start.

    ``qkv`` is ``[n, (heads + 2*kv_heads) * head_dim]`` with rotated queries in
    its first ``heads * head_dim`` columns, or those columns alone; the keys and values of the batch's
    own tokens are already in ``cache_layer``.  ``token_row[i]`` is the row of
    ``block_table`` that token ``i``'s request uses.  ``batch`` optionally
    carries per-request metadata that the tensor-core kernels need.
    """
    _cuda(qkv, "qkv")
    _cuda(cache_layer, "cache_layer", qkv.dtype)
    _cuda(block_table, "block_table", torch.int32, contiguous=False)
    _cuda(positions, "positions", torch.int32)
    _cuda(token_row, "token_row", torch.int32)
    num_pages, two, hkv, block_size, d = cache_layer.shape
    if two != 2:
        raise ValueError("cache layer must be [pages, 2, kv_heads, block_size, head_dim]")
    if d > 256:
        raise ValueError(f"head_dim {d} is not supported: the attention kernels take head sizes up to 256")
    if num_heads % hkv:
        raise ValueError("the number of query heads must be a multiple of the number of kv heads")
    n = qkv.shape[0]
    if qkv.shape[1] not in ((num_heads + 2 * hkv) * d, num_heads * d):
        raise ValueError("qkv width equals neither (heads + 2*kv_heads) * head_dim nor heads * head_dim")
    if block_table.stride(1) != 1:
        raise ValueError("block_table rows must be contiguous")
    if out is None:
        out = torch.empty((n, num_heads * d), dtype=qkv.dtype, device=qkv.device)
    win = int(window) if window else 0
    if chunk:
        if win:
            raise ValueError("a layer has a window or chunks, not both")
        win = -int(chunk)                 # the kernels' way of saying it (first_visible_key in csrc/common.cuh)
    if qkv.dtype == torch.bfloat16:
        from gllm_b200.ops import attention_bf16

        if attention_bf16.supports(d, block_size) and batch is not None:
            return attention_bf16.paged_attention_bf16(qkv, cache_layer, block_table, positions, token_row,
                                                       num_heads, scale, win, batch, out)
    return paged_attention_simt(qkv, qkv.shape[1], cache_layer, block_table, positions, token_row, num_heads,
                                scale, win, out)


# ----------------------------------------------------------------- sampling
MAX_LOGPROBS = 32


def argmax(logits: torch.Tensor, out: torch.Tensor | None = None,
           scatter_index: torch.Tensor | None = None) -> torch.Tensor:
    """Index of the largest logit of every row (lowest index on ties), int32.
    With ``scatter_index`` row ``r``'s result is written to ``out[scatter_index[r]]``."""
    _cuda(logits, "logits", torch.float32, contiguous=False)
    rows, vocab = logits.shape
    if logits.stride(1) != 1:
        raise ValueError("logit rows must be contiguous")
    if out is None:
        out = torch.empty(rows, dtype=torch.int32, device=logits.device)
    if scatter_index is not None:
        _cuda(scatter_index, "scatter_index", torch.int32)
        if scatter_index.numel() < rows:
            raise ValueError("scatter_index needs one entry per row")
    f = _fn("sampling", "gllm_argmax")
    _check(f(logits.data_ptr(), logits.stride(0), rows, vocab, out.data_ptr(), _ptr(scatter_index), _stream()),
           "argmax")
    return out


def sample(
    logits: torch.Tensor,
    temperature: torch.Tensor,
    top_k: torch.Tensor,
    top_p: torch.Tensor,
    seed: torch.Tensor,
    counter: torch.Tensor,
    num_logprobs: torch.Tensor | None = None,
    max_logprobs: int = 0,
    return_probs: bool = False,
):
    """One token per row from fp32 ``logits [rows, vocab]``.

    Per row: ``temperature`` (0 = greedy), ``top_k`` (0 = whole vocabulary,
    1 = greedy), ``top_p``, ``seed`` (int64) and ``counter`` (int32) of the
    counter-based generator.  Returns a dict with ``tokens`` int32,
    ``logprobs`` (of the sampled tokens), ``num_candidates``, and when
    ``max_logprobs`` > 0 ``top_logprobs`` / ``top_ids`` ``[rows, max_logprobs]``
    of which the first ``min(num_logprobs[row], num_candidates[row])`` are valid;
    with ``return_probs`` also the distribution drawn from, ``[rows, vocab]``.
    """
    _cuda(logits, "logits", torch.float32, contiguous=False)
    rows, vocab = logits.shape
    if logits.stride(1) != 1:
        raise ValueError("logit rows must be contiguous")
    for name, t, dt in (("temperature", temperature, torch.float32), ("top_k", top_k, torch.int32),
                        ("top_p", top_p, torch.float32), ("seed", seed, torch.int64),
                        ("counter", counter, torch.int32)):
        _cuda(t, name, dt)
        if t.numel() != rows:
            raise ValueError(f"{name} must have one entry per row")
    if max_logprobs > MAX_LOGPROBS:
        raise ValueError(f"at most {MAX_LOGPROBS} log-probabilities per token are supported")
    dev = logits.device
    out = {
        "tokens": torch.empty(rows, dtype=torch.int32, device=dev),
        "logprobs": torch.empty(rows, dtype=torch.float32, device=dev),
        "num_candidates": torch.empty(rows, dtype=torch.int32, device=dev),
    }
    top_lp = top_id = None
    if max_logprobs > 0:
        _cuda(num_logprobs, "num_logprobs", torch.int32)
        top_lp = torch.zeros((rows, max_logprobs), dtype=torch.float32, device=dev)
        top_id = torch.full((rows, max_logprobs), -1, dtype=torch.int32, device=dev)
        out["top_logprobs"], out["top_ids"] = top_lp, top_id
    probs = torch.empty((rows, vocab), dtype=torch.float32, device=dev) if return_probs else None
    if probs is not None:
        out["probs"] = probs
    f = _fn("sampling", "gllm_sample")
    _check(f(logits.data_ptr(), logits.stride(0), rows, vocab, temperature.data_ptr(), top_k.data_ptr(),
             top_p.data_ptr(), seed.data_ptr(), counter.data_ptr(),
             _ptr(num_logprobs) if max_logprobs > 0 else None, max_logprobs, out["tokens"].data_ptr(),
             out["logprobs"].data_ptr(), out["num_candidates"].data_ptr(), _ptr(top_lp), _ptr(top_id),
             _ptr(probs), _stream()), "sample")
    return out
