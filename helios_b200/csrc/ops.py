"""Python launchers of the CUDA kernels.

Every function checks its tensors (device, dtype, layout, sizes) and raises a
clear error for a size the kernel does not take; it never computes on the CPU.
Two kinds of matrix product go to the library (cuBLAS through torch), as all of
the reference's do: see ``linear`` and ``GEMM_LIBRARY_TOKEN_RANGE``.  Kernels run
on torch's current stream, so they can be captured into a CUDA graph with the
rest of a step.
"""
from __future__ import annotations

import ctypes
from ctypes import c_float, c_int, c_void_p, c_ulonglong
from typing import Optional

import torch

from .build import load_library

_F32, _BF16 = 0, 1
_STATUS = {1: "a size or option this kernel does not take", 2: "the kernel launch failed"}


class KernelError(RuntimeError):
    pass


def _dt(dtype: torch.dtype) -> int:
    if dtype == torch.float32:
        return _F32
    if dtype == torch.bfloat16:
        return _BF16
    raise KernelError(f"dtype {dtype} is not supported (float32 or bfloat16)")


def _check(t: torch.Tensor, name: str, dtype=None, ndim=None) -> None:
    if not isinstance(t, torch.Tensor):
        raise KernelError(f"{name} must be a tensor")
    if not t.is_cuda:
        raise KernelError(f"{name} must live on a CUDA device (there is no CPU path)")
    if not t.is_contiguous():
        raise KernelError(f"{name} must be contiguous")
    if dtype is not None and t.dtype != dtype:
        raise KernelError(f"{name} must be {dtype}, got {t.dtype}")
    if ndim is not None and t.dim() != ndim:
        raise KernelError(f"{name} must have {ndim} dimensions, got shape {tuple(t.shape)}")


def _stream() -> int:
    # the raw handle of torch's current stream on the current device (capture streams
    # included); the Python-level Stream object costs several microseconds a launch
    return torch._C._cuda_getCurrentRawStream(torch._C._cuda_getDevice())


def _p(t: Optional[torch.Tensor]) -> int:
    # plain integers: ctypes converts them by the declared argument types, which costs less
    # than building a c_void_p object per argument
    return 0 if t is None else t.data_ptr()


#: launches of this package's own kernels since import (library products are not counted)
launch_count = 0


def _run(status: int, what: str) -> None:
    global launch_count
    launch_count += 1
    if status != 0:
        raise KernelError(f"{what}: {_STATUS.get(status, f'status {status}')}")


_fn_cache = {}


def _fn(lib: str, name: str, argtypes):
    key = (lib, name)
    f = _fn_cache.get(key)
    if f is None:
        f = getattr(load_library(lib), name)
        f.argtypes = argtypes
        f.restype = c_int
        _fn_cache[key] = f
    return f


def preload(names) -> None:
    """Compile (in parallel) and load the named libraries, so that the first step does not
    stop at each one in turn.  A library that is not named here is still compiled and loaded
    when an op first asks for it."""
    from .build import build_all

    names = sorted(set(names) | {"elementwise"})
    build_all(names)
    for n in names:
        load_library(n)


def linear_libraries(dtype: torch.dtype, width: int = 0):
    """Libraries the matrix products of a model of this dtype and width run on."""
    if dtype == torch.float32:
        return ("gemm_f32",)
    return ("gemm_bf16",)


def attention_libraries(dtype: torch.dtype, num_heads: int, num_kv_heads: int, head_dim: int):
    """Libraries ``attention`` may choose from at these sizes (whatever the page size)."""
    if dtype != torch.bfloat16 or head_dim not in TILED_HEAD_DIMS:
        return ("attention_generic",)
    names = ["attention_bf16"]
    if ATTENTION_TCGEN05 and tc_attention_supported(num_heads, num_kv_heads, head_dim, 16):
        names += ["attention_tc", "attention_pair"]
    return tuple(names)


def option_attention_libraries(dtype: torch.dtype, num_heads: int, num_kv_heads: int, head_dim: int,
                               value_dim: int, tiled: bool = True):
    """Libraries attention with ``AttentionOptions`` may choose from at these sizes (``tiled`` False:
    options the kernels for sizes of their own do not take)."""
    if dtype != torch.bfloat16 or not ATTENTION_OPTIONS_TILED:
        return ("attention_generic",)
    if head_dim not in TILED_HEAD_DIMS or value_dim != head_dim:
        names = []
        if tiled and pooled_decode_supported(num_heads, num_kv_heads, head_dim, value_dim):
            names.append("attention_pooled")
        if tiled and pooled_tc_supported(num_heads, num_kv_heads, head_dim, value_dim, 16):
            names.append("attention_tc_pooled")
        return tuple(names) if len(names) == 2 else tuple(names + ["attention_generic"])
    names = ["attention_bf16"]
    if ATTENTION_TCGEN05 and tc_attention_supported(num_heads, num_kv_heads, head_dim, 16):
        names.append("attention_tc")
    return tuple(names)


# ------------------------------------------------------------------ embedding
def embedding(ids: torch.Tensor, table: torch.Tensor, scale: float = 1.0) -> torch.Tensor:
    """float32 [T, H] rows of ``table`` ([V, H], float32 or bfloat16) at int32 ``ids``, times
    ``scale`` (a float32 product)."""
    _check(ids, "ids", torch.int32, 1)
    _check(table, "table", None, 2)
    T, (V, H) = ids.numel(), table.shape
    out = torch.empty((T, H), dtype=torch.float32, device=table.device)
    f = _fn("elementwise", "hb_embedding",
            [c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_float, c_void_p])
    _run(f(_p(out), _p(table), _p(ids), T, H, V, _dt(table.dtype), float(scale), _stream()), "embedding")
    return out


# ------------------------------------------------------------------ norms
def add_rmsnorm(residual: torch.Tensor, delta: Optional[torch.Tensor], weight: torch.Tensor,
                eps: float, out_dtype: torch.dtype, rows: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``residual += delta`` (float32, in place) and the RMS-normed rows in ``out_dtype``.

    With ``rows`` (int32) only those rows are normed and the residual is left as it was.
    """
    _check(residual, "residual", torch.float32, 2)
    _check(weight, "weight", torch.float32, 1)
    n, H = residual.shape
    if weight.numel() != H:
        raise KernelError(f"norm weight has {weight.numel()} entries for width {H}")
    if delta is not None:
        _check(delta, "delta", out_dtype, 2)
        if tuple(delta.shape) != (n, H):
            raise KernelError(f"delta {tuple(delta.shape)} does not match residual {(n, H)}")
    n_out = n
    if rows is not None:
        _check(rows, "rows", torch.int32, 1)
        n_out = rows.numel()
    out = torch.empty((n_out, H), dtype=out_dtype, device=residual.device)
    f = _fn("elementwise", "hb_add_rmsnorm",
            [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_float, c_int, c_void_p])
    _run(f(_p(out), _p(residual), _p(delta), _p(weight), _p(rows), n_out, H, float(eps),
           _dt(out_dtype), _stream()), "add_rmsnorm")
    return out


def rmsnorm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    _check(x, "x", None, 2)
    _check(weight, "weight", torch.float32, 1)
    n, H = x.shape
    if weight.numel() != H:
        raise KernelError(f"norm weight has {weight.numel()} entries for width {H}")
    out = torch.empty_like(x)
    f = _fn("elementwise", "hb_rmsnorm",
            [c_void_p, c_void_p, c_void_p, c_int, c_int, c_float, c_int, c_void_p])
    _run(f(_p(out), _p(x), _p(weight), n, H, float(eps), _dt(x.dtype), _stream()), "rmsnorm")
    return out


# ------------------------------------------------------------------ rotary + cache write
def add_rmsnorm_pair(residual: torch.Tensor, a: Optional[torch.Tensor], b: Optional[torch.Tensor],
                     weight1: torch.Tensor, weight2: Optional[torch.Tensor], eps: float,
                     out_dtype: torch.dtype):
    """``residual += a + b`` in float32 and in place (each may be None), then TWO RMS norms of
    the new rows with one 1 / rms: (residual / rms * weight1, residual / rms * weight2) in
    ``out_dtype``; ``weight2`` None: the second is None."""
    _check(residual, "residual", torch.float32, 2)
    T, H = residual.shape
    for name, t in (("a", a), ("b", b)):
        if t is not None:
            _check(t, name, out_dtype, 2)
            if tuple(t.shape) != (T, H):
                raise KernelError(f"{name} {tuple(t.shape)} does not fit the residual {(T, H)}")
    for name, w in (("weight1", weight1), ("weight2", weight2)):
        if w is not None:
            _check(w, name, torch.float32, 1)
            if w.numel() != H:
                raise KernelError(f"{name} has {w.numel()} entries for rows of {H}")
    out1 = torch.empty((T, H), dtype=out_dtype, device=residual.device)
    out2 = torch.empty((T, H), dtype=out_dtype, device=residual.device) if weight2 is not None else None
    f = _fn("elementwise", "hb_add_rmsnorm_pair",
            [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_float,
             c_int, c_void_p])
    _run(f(_p(out1), _p(out2), _p(residual), _p(a), _p(b), _p(weight1), _p(weight2), T, H, float(eps),
           _dt(out_dtype), _stream()), "add_rmsnorm_pair")
    return out1, out2


UNARY_ACTS = {"relu2": 0, "silu": 1, "gelu_tanh": 2}


def unary_act(x: torch.Tensor, kind: str) -> torch.Tensor:
    """act(x) element by element (float32 arithmetic): "relu2" (the square of relu), "silu",
    "gelu_tanh" (0.5 x (1 + tanh(sqrt(2/pi) (x + 0.044715 x^3))))."""
    _check(x, "x", None, 2)
    if kind not in UNARY_ACTS:
        raise KernelError(f"activation {kind!r} is not one of {sorted(UNARY_ACTS)}")
    out = torch.empty_like(x)
    f = _fn("elementwise", "hb_unary_act", [c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_void_p])
    _run(f(_p(out), _p(x), 0, 0, x.shape[0], x.shape[1], UNARY_ACTS[kind], _dt(x.dtype), _stream()), "unary_act")
    return out


def sigmoid_gate(x: torch.Tensor, gate: torch.Tensor) -> torch.Tensor:
    """x * sigmoid(gate), element by element; ``gate`` [T, >= columns of x], a view whose rows
    may be strided."""
    _check(x, "x", None, 2)
    if gate.dim() != 2 or gate.stride(1) != 1 or gate.dtype != x.dtype or gate.shape[0] != x.shape[0] \
            or gate.shape[1] < x.shape[1] or not gate.is_cuda:
        raise KernelError(f"gate {tuple(gate.shape)} does not fit x {tuple(x.shape)}")
    out = torch.empty_like(x)
    f = _fn("elementwise", "hb_unary_act", [c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_void_p])
    _run(f(_p(out), _p(x), _p(gate), gate.stride(0), x.shape[0], x.shape[1], 3, _dt(x.dtype), _stream()),
         "sigmoid_gate")
    return out


def gate_heads(x: torch.Tensor, gate: torch.Tensor, per_head: bool = False) -> torch.Tensor:
    """out[t, h * N + n] = x[t, h, n] * sigmoid(gate[t, h * N + n]), or, ``per_head``, times
    sigmoid(gate[t, h]): ``x`` is a view [T, H, N] whose last dimension is contiguous (the result
    of one small product a head, whatever its token and head strides: no copy is made), ``gate``
    [T, >= H * N] (``per_head``: [T, >= H]) a view whose rows may be strided.  Returns a
    contiguous [T, H * N]."""
    if x.dim() != 3 or x.stride(2) != 1 or not x.is_cuda:
        raise KernelError(f"gate_heads: x {tuple(x.shape)} must be [T, H, N] with a contiguous last dimension")
    T, H, N = x.shape
    if gate.dim() != 2 or gate.stride(1) != 1 or gate.dtype != x.dtype or gate.shape[0] != T \
            or gate.shape[1] < (H if per_head else H * N) or not gate.is_cuda:
        raise KernelError(f"gate {tuple(gate.shape)} does not fit x {tuple(x.shape)}")
    out = torch.empty((T, H * N), dtype=x.dtype, device=x.device)
    f = _fn("elementwise", "hb_gate_heads", [c_void_p, c_void_p, ctypes.c_long, ctypes.c_long, c_void_p, c_int,
                                             c_int, c_int, c_int, c_int, c_int, c_void_p])
    _run(f(_p(out), _p(x), x.stride(0), x.stride(1), _p(gate), gate.stride(0), T, H, N, 1 if per_head else 0,
           _dt(x.dtype), _stream()),
         "gate_heads")
    return out


def rotary_table(positions: torch.Tensor, inv_freq: torch.Tensor, factor: float = 1.0):
    """cos and sin [T, rot/2] (float32) of position * inv_freq, computed in float64 and
    multiplied by ``factor`` (the attention factor of a scaled encoding; 1 for none)."""
    _check(positions, "positions", torch.int32, 1)
    _check(inv_freq, "inv_freq", torch.float64, 1)
    T, half = positions.numel(), inv_freq.numel()
    cos = torch.empty((T, half), dtype=torch.float32, device=positions.device)
    sin = torch.empty_like(cos)
    f = _fn("elementwise", "hb_rotary_table",
            [c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, ctypes.c_double, c_void_p])
    _run(f(_p(cos), _p(sin), _p(positions), _p(inv_freq), T, half, float(factor), _stream()), "rotary_table")
    return cos, sin


def rope_kv_write(qkv: torch.Tensor, cos: Optional[torch.Tensor], sin: Optional[torch.Tensor],
                  positions: torch.Tensor, seq_of_token: torch.Tensor, block_table: torch.Tensor,
                  k_pages: Optional[torch.Tensor], v_pages: Optional[torch.Tensor],
                  num_heads: int, num_kv_heads: int, head_dim: int, page_size: int,
                  write_cache: bool = True) -> None:
    """Rotate q and k of ``qkv`` ([T, (nh + 2 nkv) hd]) by the tokens' cos/sin rows
    ([T, rot/2], float32; None = no rotation); q stays in place, rotated k and v go to the
    tokens' slots of the cache pages ([pages, nkv, page_size, hd])."""
    _check(qkv, "qkv", None, 2)
    T = qkv.shape[0]
    if qkv.shape[1] != (num_heads + 2 * num_kv_heads) * head_dim:
        raise KernelError(f"qkv width {qkv.shape[1]} is not (nh + 2 nkv) * hd = "
                          f"{(num_heads + 2 * num_kv_heads) * head_dim}")
    rot = 0
    if cos is not None:
        _check(cos, "cos", torch.float32, 2)
        _check(sin, "sin", torch.float32, 2)
        if cos.shape != sin.shape or cos.shape[0] != T:
            raise KernelError(f"cos/sin tables {tuple(cos.shape)}/{tuple(sin.shape)} do not "
                              f"match {T} tokens")
        rot = 2 * cos.shape[1]
        if rot > head_dim:
            raise KernelError(f"rotary dimension {rot} exceeds head_dim {head_dim}")
    _check(positions, "positions", torch.int32, 1)
    _check(seq_of_token, "seq_of_token", torch.int32, 1)
    _check(block_table, "block_table", torch.int32, 2)
    if write_cache:
        for name, pages in (("k_pages", k_pages), ("v_pages", v_pages)):
            _check(pages, name, qkv.dtype, 4)
            if tuple(pages.shape[1:]) != (num_kv_heads, page_size, head_dim):
                raise KernelError(f"{name} has shape {tuple(pages.shape)}, expected "
                                  f"[pages, {num_kv_heads}, {page_size}, {head_dim}]")
    f = _fn("elementwise", "hb_rope_kv_write",
            [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_void_p,
             c_void_p, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_void_p])
    _run(f(_p(qkv), _p(cos), _p(sin), _p(positions), _p(seq_of_token), _p(block_table),
           block_table.shape[1], _p(k_pages) if write_cache else 0,
           _p(v_pages) if write_cache else 0, T, num_heads, num_kv_heads, head_dim,
           rot, page_size, 1 if write_cache else 0, _dt(qkv.dtype), _stream()), "rope_kv_write")


# ------------------------------------------------------------------ attention
class AttentionOptions:
    """What an attention kernel may be asked for beyond scaled dot products, a causal mask and
    a window; each is off by default.

    ``slopes``   float32 [heads]: score - slopes[h] * (query position - key position)
    ``bias_table`` float32 [rows, heads]: score + bias_table[min(distance, rows - 1), h]
                 (``distance_bias_rows`` makes one from a table of buckets); ``bias_table_t``,
                 its transpose as a contiguous tensor, is what the tcgen05 kernel reads (made at
                 the call where it is not given)
    ``sink``     the softmax has a key that carries no value: weights
                 exp(s_j) / (exp(sink) + sum_j exp(s_j)); its score is 0, or
                 ``sink_values[h]`` (float32 [heads]) where given
    ``keep_first`` with a window: the first ``keep_first`` keys of a request stay visible to
                 every later token
    ``gate``     [T, >= heads] in the activation dtype, a view whose rows are ``gate_stride``
                 apart: head h's output at token t is multiplied by sigmoid(gate[t, h]); with
                 ``gate_wide`` the view is [T, >= heads * value size] and every output value
                 has a gate of its own
    ``value_dim`` values per head where they differ from the keys' (None: the same)"""

    __slots__ = ("slopes", "sink", "gate", "gate_stride", "value_dim", "bias_table", "sink_values",
                 "keep_first", "gate_wide", "bias_table_t")

    def __init__(self, slopes: Optional[torch.Tensor] = None, sink: bool = False,
                 gate: Optional[torch.Tensor] = None, value_dim: Optional[int] = None,
                 bias_table: Optional[torch.Tensor] = None, sink_values: Optional[torch.Tensor] = None,
                 keep_first: int = 0, gate_wide: bool = False,
                 bias_table_t: Optional[torch.Tensor] = None) -> None:
        self.bias_table_t = bias_table_t
        self.slopes, self.sink, self.gate, self.value_dim = slopes, bool(sink) or sink_values is not None, gate, value_dim
        self.bias_table, self.sink_values = bias_table, sink_values
        self.keep_first, self.gate_wide = int(keep_first or 0), bool(gate_wide)
        self.gate_stride = 0 if gate is None else int(gate.stride(0))

    @property
    def plain(self) -> bool:
        return self.slopes is None and not self.sink and self.gate is None and self.value_dim is None \
            and self.bias_table is None and not self.keep_first

    @property
    def tiled(self) -> bool:
        """Whether the tensor-core kernels (split-context decode, tcgen05 and ``mma.sync``
        prefill) take these options: all of them, as long as values have the keys' size."""
        return self.value_dim is None

    def check(self, tokens: int, num_heads: int, like: torch.Tensor, value_dim: int = 0) -> None:
        if self.slopes is not None:
            _check(self.slopes, "slopes", torch.float32, 1)
            if self.slopes.numel() != num_heads:
                raise KernelError(f"{self.slopes.numel()} slopes for {num_heads} heads")
        if self.sink_values is not None:
            _check(self.sink_values, "sink_values", torch.float32, 1)
            if self.sink_values.numel() != num_heads:
                raise KernelError(f"{self.sink_values.numel()} sink values for {num_heads} heads")
        if self.bias_table is not None:
            _check(self.bias_table, "bias_table", torch.float32, 2)
            if self.bias_table.shape[1] != num_heads or self.bias_table.shape[0] < 1:
                raise KernelError(f"bias table {tuple(self.bias_table.shape)} for {num_heads} heads")
        if self.keep_first < 0:
            raise KernelError("keep_first must not be negative")
        if self.gate is not None:
            g = self.gate
            need = num_heads * value_dim if self.gate_wide else num_heads
            if not g.is_cuda or g.dtype != like.dtype or g.dim() != 2 or g.shape[0] != tokens \
                    or g.shape[1] < need or g.stride(1) != 1:
                raise KernelError(f"gate must be [{tokens}, >= {need}] {like.dtype} with unit column stride")


def distance_bias_rows(table: torch.Tensor, far: float, window: Optional[int] = None) -> torch.Tensor:
    """The bias of every distance 0, 1, 2, ... from a learned table of buckets ([rows, heads]):
    with half = rows // 2, a distance n < half has the row n, a larger one the row
    min(rows - 1, half + floor(ln(n / half) / ln(far / half) * (rows - half))): one row a
    distance close by, rows that grow logarithmically up to ``far``, the last row beyond.
    Returns float32 [distances, heads], long enough that every larger distance has the last
    entry's bias (or ``window`` distances, where nothing beyond is ever asked for): what
    ``AttentionOptions.bias_table`` takes.  The buckets are found on the host in float64."""
    import math
    rows = int(table.shape[0])
    half = rows // 2
    if half < 1 or not far > half:
        raise KernelError(f"a distance-bias table of {rows} rows with far = {far} has no logarithmic part")

    def bucket(n: int) -> int:
        if n < half:
            return n
        return min(rows - 1, half + int(math.floor(math.log(n / half) / math.log(far / half) * (rows - half))))

    last = int(math.ceil(far)) + 1          # from ``far`` on the bucket is the last row
    while bucket(last) != rows - 1:
        last += 1
    if window is not None:
        last = min(last, max(int(window) - 1, 0))
    index = torch.tensor([bucket(n) for n in range(last + 1)], dtype=torch.long, device=table.device)
    return table.float().index_select(0, index).contiguous()


_NO_OPTIONS = AttentionOptions()


def _tiled_options(options: Optional[AttentionOptions], tokens: int, num_heads: int,
                   like: torch.Tensor, head_dim: int = 0) -> AttentionOptions:
    """Checked options for the tensor-core kernels, whose values have the keys' size."""
    if options is None:
        return _NO_OPTIONS
    if options.value_dim is not None:
        raise KernelError("the tensor-core attention kernels take values of the keys' size only")
    options.check(tokens, num_heads, like, head_dim)
    return options


def _option_args(opt: AttentionOptions, window: Optional[int]):
    """The options as the ``mma.sync`` launchers take them, after slopes, sink and gate."""
    return (_p(opt.bias_table), 0 if opt.bias_table is None else int(opt.bias_table.shape[0]),
            _p(opt.sink_values), opt.keep_first if window else 0, 1 if opt.gate_wide else 0)


def attention_generic(qkv: torch.Tensor, k_pages: torch.Tensor, v_pages: torch.Tensor,
                      block_table: torch.Tensor, seq_of_token: torch.Tensor,
                      positions: torch.Tensor, num_heads: int, num_kv_heads: int, head_dim: int,
                      page_size: int, window: Optional[int], scale: float,
                      options: Optional["AttentionOptions"] = None, pooled=None,
                      out: Optional[torch.Tensor] = None, factor: float = 1.0) -> torch.Tensor:
    """Attention of every token of the batch over its request's pages; q is read from the
    first ``nh * hd`` columns of ``qkv``.  Returns [T, nh * vd] in qkv's dtype (vd = hd
    unless ``options`` says otherwise).  ``pooled`` = (key pages, value pages, block table, tokens
    a block): means of whole blocks behind the window.  ``out``: rows to write to (they may be
    strided); ``factor``: a constant on the output."""
    _check(qkv, "qkv", None, 2)
    _check(k_pages, "k_pages", qkv.dtype, 4)
    _check(v_pages, "v_pages", qkv.dtype, 4)
    _check(block_table, "block_table", torch.int32, 2)
    _check(seq_of_token, "seq_of_token", torch.int32, 1)
    _check(positions, "positions", torch.int32, 1)
    if head_dim > 256 or head_dim <= 0:
        raise KernelError(f"head_dim {head_dim} is not supported by the attention kernels (1..256)")
    if num_heads % num_kv_heads != 0:
        raise KernelError(f"{num_heads} query heads are not a multiple of {num_kv_heads} KV heads")
    if tuple(k_pages.shape[1:]) != (num_kv_heads, page_size, head_dim):
        raise KernelError(f"k_pages has shape {tuple(k_pages.shape)}, expected "
                          f"[pages, {num_kv_heads}, {page_size}, {head_dim}]")
    T = qkv.shape[0]
    opt = options or _NO_OPTIONS
    vd = opt.value_dim or head_dim
    opt.check(T, num_heads, qkv, vd)
    if not 0 < vd <= 256 or tuple(v_pages.shape[1:]) != (num_kv_heads, page_size, vd):
        raise KernelError(f"v_pages has shape {tuple(v_pages.shape)}, expected "
                          f"[pages, {num_kv_heads}, {page_size}, {vd}] with at most 256 values a head")
    if out is None:
        out = torch.empty((T, num_heads * vd), dtype=qkv.dtype, device=qkv.device)
    else:
        _check_out_rows(out, T, num_heads * vd, qkv)
    pk = pv = pt = None
    pool = 0
    if pooled is not None:
        pk, pv, pt, pool = _check_pooled(pooled, qkv, num_kv_heads, page_size, head_dim, vd, window)
    f = _fn("attention_generic", "hb_attention_generic",
            [c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_int, c_void_p, c_void_p,
             c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_float, c_void_p, c_int, c_void_p,
             c_int, c_void_p, c_int, c_void_p, c_int, c_int, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int,
             c_float, c_int, c_void_p])
    _run(f(_p(out), _p(qkv), qkv.shape[1], _p(k_pages), _p(v_pages), _p(block_table),
           block_table.shape[1], _p(seq_of_token), _p(positions), T, num_heads, num_kv_heads,
           head_dim, vd, page_size, int(window or 0), float(scale), _p(opt.slopes), int(opt.sink),
           _p(opt.gate), opt.gate_stride, _p(opt.bias_table),
           0 if opt.bias_table is None else opt.bias_table.shape[0], _p(opt.sink_values),
           opt.keep_first if window else 0, 1 if opt.gate_wide else 0, _p(pk), _p(pv), _p(pt),
           0 if pt is None else pt.shape[1], pool, out.stride(0), float(factor), _dt(qkv.dtype), _stream()),
         "attention_generic")
    return out


def _check_out_rows(out: torch.Tensor, tokens: int, columns: int, like: torch.Tensor) -> None:
    if not out.is_cuda or out.dtype != like.dtype or out.dim() != 2 or out.shape[0] != tokens \
            or out.shape[1] < columns or out.stride(1) != 1:
        raise KernelError(f"out must be [{tokens}, >= {columns}] {like.dtype} with unit column stride")


def _check_pooled(pooled, like, num_kv_heads, page_size, head_dim, value_dim, window):
    pk, pv, pt, pool = pooled
    for name, pages, d in (("pooled keys", pk, head_dim), ("pooled values", pv, value_dim)):
        _check(pages, name, like.dtype, 4)
        if tuple(pages.shape[1:]) != (num_kv_heads, page_size, d):
            raise KernelError(f"{name} have shape {tuple(pages.shape)}, expected "
                              f"[pages, {num_kv_heads}, {page_size}, {d}]")
    _check(pt, "pooled block table", torch.int32, 2)
    if not window or pool < 1:
        raise KernelError("pooled blocks lie behind a window and hold at least one token")
    return pk, pv, pt, int(pool)


# ------------------------------------------------------------------ feed-forward gate
def silu_mul(gate_up: torch.Tensor) -> torch.Tensor:
    """silu(gate) * up for ``gate_up`` = [T, 2 I] (gate columns first)."""
    _check(gate_up, "gate_up", None, 2)
    T, two_i = gate_up.shape
    if two_i % 2:
        raise KernelError("gate_up must have an even width")
    out = torch.empty((T, two_i // 2), dtype=gate_up.dtype, device=gate_up.device)
    f = _fn("elementwise", "hb_silu_mul", [c_void_p, c_void_p, c_int, c_int, c_int, c_void_p])
    _run(f(_p(out), _p(gate_up), T, two_i // 2, _dt(gate_up.dtype), _stream()), "silu_mul")
    return out


# ------------------------------------------------------------------ matrix products
def linear_f32(x: torch.Tensor, weight: torch.Tensor, bias: Optional[torch.Tensor] = None) -> torch.Tensor:
    """x [M, K] times weight [N, K] transposed (+ bias [N]) on the float32 FMA pipes."""
    _check(x, "x", torch.float32, 2)
    _check(weight, "weight", torch.float32, 2)
    M, K = x.shape
    N, K2 = weight.shape
    if K != K2:
        raise KernelError(f"x has {K} columns but weight has {K2}")
    if bias is not None:
        _check(bias, "bias", torch.float32, 1)
        if bias.numel() != N:
            raise KernelError(f"bias has {bias.numel()} entries for {N} outputs")
    out = torch.empty((M, N), dtype=torch.float32, device=x.device)
    f = _fn("gemm_f32", "hb_gemm_f32",
            [c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_int, c_void_p])
    _run(f(_p(out), _p(x), _p(weight), _p(bias), M, N, K, K, K, N, _stream()), "gemm_f32")
    return out


# Fixed work space of the tensor-core products on a device: partial sums of split
# reductions, one ticket per output tile (zero between launches), and an error word
# that a kernel sets when one of its bounded waits ran out.  Its addresses never
# change, so captured CUDA graphs stay valid.
#: add the partial sums of a split reduction inside a thread-block cluster (through
#: distributed shared memory) where that is possible, instead of through scratch memory
GEMM_CLUSTER_REDUCE = True
#: prefill-sized products (more than 128 tokens, reduction not split) on pairs of SMs
GEMM_TWO_SM = True
_GEMM_SCRATCH_FLOATS = 16 * 1024 * 1024


def _cluster_fits(bn: int, glu: bool) -> bool:
    """Whether a block's float32 partial sums fit the stage buffers they reuse."""
    if bn == 0:
        stage, budget, cols = 48 * 1024, 196 * 1024, 256
    else:
        a_tiles = 2 if glu else 1
        stage, budget, cols = a_tiles * 16384 + bn * 128, 108 * 1024, bn * a_tiles
    stages = max(2, min(8, budget // stage))
    return cols * 128 * 4 <= stages * stage
_GEMM_TICKETS = 1 << 16
_gemm_ws = {}


def _gemm_workspace(device):
    ws = _gemm_ws.get(device)
    if ws is None:
        ws = (torch.empty(_GEMM_SCRATCH_FLOATS, dtype=torch.float32, device=device),
              torch.zeros(_GEMM_TICKETS, dtype=torch.int32, device=device),
              torch.zeros(1, dtype=torch.int32, device=device))
        _gemm_ws[device] = ws
    return ws


def check_kernel_errors(device=None) -> None:
    """Raise if a kernel of this package gave up a bounded wait (synchronises)."""
    for dev, (_s, _t, err) in _gemm_ws.items():
        if device is not None and dev != torch.device(device):
            continue
        code = int(err.item())
        if code:
            err.zero_()
            role = {1: "the TMA producer", 2: "the MMA issuer", 3: "the epilogue"}.get(code, "a role")
            raise KernelError(f"gemm_bf16: {role} gave up waiting on an mbarrier (code {code}); "
                              "the results of that launch are not valid")


_cluster_capacity = {}


def cluster_capacity(bn: int, glu: bool, size: int) -> int:
    """Clusters of ``size`` blocks of the GEMM variant (bn, glu) the device keeps resident
    at once.  The CUDA occupancy calculator is asked (it knows how the SMs are spread over
    the GPCs, which bounds whole clusters); it counts one block per SM where the swapped
    variants run two, so its figure is doubled for them.  Measured on B200: cluster counts
    up to that doubled figure run in one round, beyond it a second round shows."""
    key = (bn, bool(glu), size)
    if key not in _cluster_capacity:
        lib = load_library("gemm_bf16")
        n = int(lib.hb_gemm_bf16_max_clusters(bn, int(glu), size))
        if n <= 0:
            n = sm_count() // size
        _cluster_capacity[key] = n * (2 if bn else 1)
    return _cluster_capacity[key]


_gemm_plans = {}


def gemm_plan(T: int, N: int, K: int, glu: bool):
    """Cached ``_gemm_plan``."""
    key = (T, N, K, bool(glu), GEMM_CLUSTER_REDUCE, GEMM_TWO_SM)
    plan = _gemm_plans.get(key)
    if plan is None:
        plan = _gemm_plans[key] = _gemm_plan(T, N, K, glu)
    return plan


def _gemm_plan(T: int, N: int, K: int, glu: bool):
    """(swap_bn, k_splits) of the tensor-core product for T tokens, N result features.
    Up to 128 tokens run swapped (features on the MMA M axis).  When the tiles alone do not
    fill the SMs, the reduction is split (at least 2 k-blocks a slice; short reductions of
    small models are bound by latency, and more blocks shorten them): with slices as
    thread-block clusters, the count that keeps the most blocks resident in ONE round of
    clusters; else the count that fills the resident blocks."""
    k_blocks = -(-K // 64)
    if T <= 128:
        bn = 16 if T <= 16 else 32 if T <= 32 else 64 if T <= 64 else 128
        tiles = -(-N // 128) * -(-T // bn)
        cols = bn * (2 if glu else 1)
        slots = 2 * sm_count()
    else:
        bn = 0
        tiles = -(-T // 128) * -(-N // (128 if glu else 256))
        cols = 256
        slots = sm_count()
        if GEMM_TWO_SM:
            # the two-SM kernel takes whole reductions only; even with part of the pairs idle
            # it beats the one-SM kernel with a split reduction (20 against 85 microseconds
            # for 512 tokens x 4096 x 4096)
            return bn, 1
    splits = 1
    if tiles < slots:
        most_k = max(1, k_blocks // 2)
        if GEMM_CLUSTER_REDUCE and _cluster_fits(bn, glu):
            best = 0
            for s in range(1, min(8, most_k) + 1):
                # a few clusters over the figure cost less than a smaller cluster size
                if tiles * 15 <= cluster_capacity(bn, glu, s) * 16 and tiles * s > best + best // 16:
                    splits, best = s, tiles * s
        else:
            splits = _wave_splits(tiles, slots, min(16, most_k))
            while splits > 1 and tiles * splits * 128 * cols > _GEMM_SCRATCH_FLOATS:
                splits -= 1
    return bn, splits


def tc_gemm_supported(x: torch.Tensor, weight: torch.Tensor) -> bool:
    return (x.dtype == torch.bfloat16 and weight.dtype == torch.bfloat16 and x.dim() == 2
            and weight.dim() == 2 and x.shape[1] == weight.shape[1] and x.shape[1] % 8 == 0
            and x.is_contiguous() and weight.is_contiguous()
            and x.data_ptr() % 16 == 0 and weight.data_ptr() % 16 == 0)


#: gated units the tcgen05 products have an epilogue for (``linear_bf16``'s ``glu``)
GLU_EPILOGUES = {False: 0, True: 1, "silu": 1, "gelu_tanh": 2}


def linear_bf16(x: torch.Tensor, weight: torch.Tensor, bias: Optional[torch.Tensor] = None,
                glu=False, out_dtype: torch.dtype = torch.bfloat16,
                plan=None, cluster: Optional[bool] = None, two_sm: Optional[bool] = None,
                sumsq: Optional[torch.Tensor] = None, eps: float = 0.0,
                residual: Optional[torch.Tensor] = None, norm_weight: Optional[torch.Tensor] = None,
                norm_out: Optional[tuple] = None):
    """y = x W^T (+ bias) on tcgen05 tensor cores; bfloat16 operands, float32 accumulate.

    With ``glu`` (True or "silu", or "gelu_tanh") the weight is [gate rows; up rows] ([2 I, K]) and
    the result is act(x gate^T) * (x up^T), [T, I].  ``out_dtype`` bfloat16 or float32.  K must be a
    multiple of 8 (TMA rows are 16-byte aligned); any T and N.

    Up to DEFERRED_NORM_MOST tokens there are two more epilogues.  ``sumsq``
    (float32 [T, slots]): ``x`` is residual * norm weight without the token's 1 / rms;
    the accumulators are multiplied by rsqrt(sum(sumsq[t]) / K + eps) before bias or SwiGLU.
    ``residual`` (float32 [T, N]): the product is added into it and None is returned, or,
    with ``norm_weight`` (float32 [N]), the pair (bfloat16(residual * norm_weight),
    partial sums of squares [T, slots]) that a product with ``sumsq`` takes; ``norm_out``
    gives that pair's tensors to write into."""
    _check(x, "x", torch.bfloat16, 2)
    _check(weight, "weight", torch.bfloat16, 2)
    T, K = x.shape
    rows, K2 = weight.shape
    if K != K2:
        raise KernelError(f"x has {K} columns but weight has {K2}")
    if K % 8:
        raise KernelError(f"the tensor-core product needs K to be a multiple of 8, got {K}")
    if glu and rows % 2:
        raise KernelError("a SwiGLU weight needs an even number of rows")
    glu_code = GLU_EPILOGUES.get(glu)
    if glu_code is None:
        raise KernelError(f"the product has no epilogue for {glu!r}")
    N = rows // 2 if glu else rows
    if bias is not None:
        if glu:
            raise KernelError("the SwiGLU epilogue takes no bias")
        _check(bias, "bias", torch.float32, 1)
        if bias.numel() != N:
            raise KernelError(f"bias has {bias.numel()} entries for {N} outputs")
    if out_dtype not in (torch.bfloat16, torch.float32):
        raise KernelError(f"out_dtype {out_dtype} is not supported")
    few = sumsq is not None or residual is not None
    if few and T > DEFERRED_NORM_MOST:
        raise KernelError(f"the residual and 1 / rms epilogues take at most {DEFERRED_NORM_MOST} tokens, got {T}")
    if sumsq is not None:
        _check(sumsq, "sumsq", torch.float32, 2)
        if sumsq.shape[0] != T or not sumsq.is_contiguous():
            raise KernelError(f"sumsq has shape {tuple(sumsq.shape)} for {T} tokens")
    sumsq_out = None
    if residual is not None:
        _check(residual, "residual", torch.float32, 2)
        if tuple(residual.shape) != (T, N) or not residual.is_contiguous():
            raise KernelError(f"residual has shape {tuple(residual.shape)}, expected ({T}, {N}) contiguous")
        if glu or out_dtype != torch.bfloat16:
            raise KernelError("a product into the residual is a plain bfloat16 one")
        out = None
        if norm_weight is not None:
            _check(norm_weight, "norm_weight", torch.float32, 1)
            if norm_weight.numel() != N:
                raise KernelError(f"norm weight has {norm_weight.numel()} entries for width {N}")
            slots = 8 * -(-N // 128)
            if norm_out is not None:
                out, sumsq_out = norm_out
                _check(out, "norm_out[0]", torch.bfloat16, 2)
                _check(sumsq_out, "norm_out[1]", torch.float32, 2)
                if tuple(out.shape) != (T, N) or tuple(sumsq_out.shape) != (T, slots):
                    raise KernelError("norm_out tensors have the wrong shapes")
            else:
                out = torch.empty((T, N), dtype=torch.bfloat16, device=x.device)
                sumsq_out = torch.empty((T, slots), dtype=torch.float32, device=x.device)
    elif norm_weight is not None:
        raise KernelError("norm_weight goes with residual")
    else:
        out = torch.empty((T, N), dtype=out_dtype, device=x.device)
    if T == 0:
        return out if residual is None else ((out, sumsq_out) if norm_weight is not None else None)
    bn, splits = plan if plan is not None else gemm_plan(T, N, K, bool(glu))
    if few and (bn == 0 or T > bn):
        raise KernelError("the residual and 1 / rms epilogues need the swapped orientation and one token tile")
    if cluster is None:
        cluster = GEMM_CLUSTER_REDUCE
    # slices of a tile as a cluster: at most 8, and the partial sums must fit the stages
    cluster = bool(cluster) and 1 < splits <= 8 and _cluster_fits(bn, bool(glu))
    cluster_arg = 1 if cluster else 0
    if bn == 0 and splits == 1 and (GEMM_TWO_SM if two_sm is None else two_sm):
        cluster_arg = 2                      # prefill tiles on pairs of SMs (cta_group::2)
    scratch, tickets, err = _gemm_workspace(x.device)
    lib = load_library("gemm_bf16")
    if splits > 1 and not cluster:
        lib.hb_gemm_bf16_scratch_floats.restype = ctypes.c_longlong
        need = lib.hb_gemm_bf16_scratch_floats(T, N, bn, glu_code, splits)
        tiles = lib.hb_gemm_bf16_tiles(T, N, bn, glu_code)
        if need > scratch.numel() or tiles > tickets.numel():
            raise KernelError(f"split reduction needs {need} scratch floats and {tiles} tickets; "
                              f"the work space holds {scratch.numel()} and {tickets.numel()}")
    common = [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int,
              c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int]
    args = (_p(out), _p(x), _p(weight), _p(bias), _p(scratch), _p(tickets), _p(err), T, N, K, K, K, N,
            rows, glu_code, N if glu else 0, 1 if out_dtype == torch.float32 else 0, bn, splits, cluster_arg)
    if few:
        f = _fn("gemm_bf16", "hb_gemm_bf16_fused",
                common + [c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_float, c_void_p])
        _run(f(*args, _p(residual), _p(norm_weight), _p(sumsq_out), _p(sumsq),
               0 if sumsq is None else sumsq.shape[1], float(eps), _stream()), "gemm_bf16_fused")
        if residual is not None:
            return (out, sumsq_out) if norm_weight is not None else None
        return out
    f = _fn("gemm_bf16", "hb_gemm_bf16", common + [c_void_p])
    _run(f(*args, _stream()), "gemm_bf16")
    return out


#: Steps of at most this many tokens run a layer's RMS norms inside the products around them
#: (see ``linear_bf16``): the products of such a step run swapped, tokens on one narrow tile,
#: on this package's kernel.  The epilogues take up to DEFERRED_NORM_MOST tokens, but their
#: cost grows with the tokens while a norm launch's does not.  Measured, milliseconds a
#: decode step with the norm launches against without: Llama-3.1-8B sizes 4.01 / 3.89 at 8
#: requests, 4.87 / 4.86 at 16, 5.83 / 5.73 at 24, 6.70 / 6.88 at 32; Qwen2.5-7B sizes 3.38 /
#: 3.22 at 8, 4.52 / 4.58 at 32; Qwen2.5-0.5B sizes 1.06 / 1.08 at 24, 1.12 / 1.14 at 32.
DEFERRED_NORM_TOKENS = 16
DEFERRED_NORM_MOST = 32


def deferred_norm_fits(tokens: int, *weights: torch.Tensor) -> bool:
    """Whether a step of ``tokens`` tokens runs these products with the residual and
    1 / rms epilogues: few tokens, and shapes the tensor-core kernel takes."""
    if not 0 < tokens <= DEFERRED_NORM_TOKENS:
        return False
    return all(w.dtype == torch.bfloat16 and w.dim() == 2 and w.shape[1] % 8 == 0 and w.is_contiguous()
               and w.data_ptr() % 16 == 0 for w in weights)


#: Between the decode kernel's best range (up to 32 tokens: weights streamed once with the
#: tokens on a narrow MMA N axis, a deep ring of weight stages) and the prefill kernel's (pairs
#: of SMs on 256x256 tiles, which need a few hundred tiles to fill 74 pairs) plain products (no
#: bias, bfloat16 out) go to the library (cuBLAS through torch), which the reference uses for
#: every product (python/helios/exec/model.py:170-181).  From 33 tokens on a stage of the decode
#: kernel holds 8-16 KB of tokens beside its 16 KB of weights, the ring gets shallow, and the
#: library is ahead (Llama-3.1-8B sizes at 64 tokens, microseconds in a chain: q|k|v 15.2
#: against 11.5, O 11.1 against 10.0, down 24.3 against 24.2; a decode step of 64 requests
#: 6,300-6,460 against 6,690 tokens/s); from 129 tokens on the two-SM kernel has too few tiles
#: (same sizes, this package's kernel against the library: down 88 / 61 at 513 tokens, 82 / 69
#: at 768, 86 / 83 at 1,024, 171 / 120 at 1,536 with 80 tiles on 74 pairs, 168 / 156 at 2,048,
#: 263 / 271 at 3,072; O 28 / 22, 29 / 22, 30 / 27, 54 / 43, 53 / 50, 84 / 82).  Products with
#: float32 logits, and everything up to 32 tokens, always run on this package's kernels.
#: (0, 0) turns the library off.
GEMM_LIBRARY_TOKEN_RANGE = (33, 1536)
#: gate|up with SwiGLU runs fused on this package's kernels except in these token ranges,
#: where the library's plain product and a gate kernel are ahead (Llama-3.1-8B sizes, fused
#: against library + gate: 73 / 59 at 96 tokens, 82 / 57 at 128; 59 / 67 at 160, 66 / 76 at
#: 256: one full tile of the two-SM kernel; 110 / 93 at 320, 110 / 104 at 384: a second tile
#: that is mostly empty; 111 / 129 at 448, 112 / 141 at 512, 150 / 188 at 640)
GEMM_LIBRARY_GLU_TOKENS = ((33, 128), (257, 383))
#: The library chooses its kernel per shape, which takes about a millisecond of host time
#: the first time a shape is seen; token counts are rounded up to a multiple of this (on a
#: padded copy of the rows) so that a serving run meets a handful of shapes, not hundreds.
#: Up to 128 tokens the step is 8 and up to 256 it is 32 (GEMM_LIBRARY_TOKEN_STEPS_FEW): the
#: padded copy is two launches more per product (the four products of a layer at
#: Llama-3.1-8B sizes and 40 tokens: 105 µs with the copy, 94 without; a decode step of 40
#: requests 7.90 -> 7.60 ms, at Qwen2.5-0.5B sizes 1.26 -> 1.09 ms), and captured steps come
#: in these multiples there anyway.
GEMM_LIBRARY_TOKEN_STEP = 64
GEMM_LIBRARY_TOKEN_STEPS_FEW = ((128, 8), (256, 32))
#: Weight matrices of at most this many bytes (the products of models about 1,000 wide: 2 to
#: 17 MB) go to the library from GEMM_LIBRARY_SMALL_TOKENS[0] tokens on: a product that short
#: is bound by the kernel's own latency, where the tensor-memory kernels (set-up, a cluster for
#: the split reduction) lose to the library's plain ones, and with 896 output features the
#: two-SM kernel has 4 tiles a 256 tokens.  Measured at Qwen2.5-0.5B sizes, microseconds a
#: launch in a chain, this package's kernel against the library, at 24 / 64 / 256 tokens: q|k|v
#: 5.0 / 7.2 / 10.9 against 4.0 / 3.9 / 4.2; down 6.8 / 8.5 / 29.7 against 9.4 / 8.6 / 8.8 (and
#: 30 / 10 at 1,024, 31 / 15 at 2,048, 32 / 27 at 4,096, 64 / 64 at 8,192); gate|up with SwiGLU
#: 14.4 / 18.9 / 16.5 against 8.6 / 8.7 / 12.8 (library product + gate kernel; 26 / 26 at 768,
#: 56 / 58 at 2,048, 96 / 117 at 4,096: GEMM_LIBRARY_SMALL_GLU_TOKENS).  Up to 32 tokens this
#: package's kernels win as a whole (a step of 32 requests: 28,300 against 25,900 tokens/s).
#: 0 bytes turns it off.
GEMM_LIBRARY_SMALL_WEIGHT_BYTES = 20 * 1024 * 1024
GEMM_LIBRARY_SMALL_TOKENS = (33, 4096)
GEMM_LIBRARY_SMALL_GLU_TOKENS = (33, 512)


def _library_range(tokens: int) -> bool:
    lo, hi = GEMM_LIBRARY_TOKEN_RANGE
    return lo <= tokens <= hi


def _small_weight_library(tokens: int, weight: torch.Tensor, glu: bool = False) -> bool:
    lo, hi = GEMM_LIBRARY_SMALL_GLU_TOKENS if glu else GEMM_LIBRARY_SMALL_TOKENS
    return lo <= tokens <= hi and \
        weight.numel() * weight.element_size() <= GEMM_LIBRARY_SMALL_WEIGHT_BYTES


#: Products with a bias take the same way in that range (the library adds the bias, as
#: bfloat16, to its float32 sums before it rounds them): Qwen2.5-7B sizes, 64 requests
#: decoding, 10,550 -> 10,660 tokens/s.
GEMM_LIBRARY_WITH_BIAS = True
_bf16_biases = {}


def _bias_bf16(bias: torch.Tensor) -> torch.Tensor:
    """The bias as bfloat16 for the library, converted once per tensor (a model's biases are
    float32 and do not change)."""
    if bias.dtype == torch.bfloat16:
        return bias
    key = (bias.data_ptr(), bias.numel(), bias.device)
    hit = _bf16_biases.get(key)
    if hit is None or hit[0] is not bias:
        hit = _bf16_biases[key] = (bias, bias.to(torch.bfloat16))
    return hit[1]


def _library_linear(x: torch.Tensor, weight: torch.Tensor, bias: Optional[torch.Tensor]) -> torch.Tensor:
    T = x.shape[0]
    step = next((st for most, st in GEMM_LIBRARY_TOKEN_STEPS_FEW if T <= most), GEMM_LIBRARY_TOKEN_STEP)
    padded = -(-T // step) * step if step > 1 else T
    if padded == T:
        return torch.nn.functional.linear(x, weight, bias)
    rows = x.new_empty((padded, x.shape[1]))
    rows[:T].copy_(x)
    rows[T:].zero_()                              # they reach no result row, but must not hold NaN
    return torch.nn.functional.linear(rows, weight, bias)[:T]


def linear(x: torch.Tensor, weight: torch.Tensor, bias: Optional[torch.Tensor] = None) -> torch.Tensor:
    """y = x W^T + b.  float32: this package's FMA kernel.  bfloat16: the tcgen05 kernels,
    or the library for plain products in the token ranges of GEMM_LIBRARY_TOKEN_RANGE and
    GEMM_LIBRARY_SMALL_TOKENS (small weight matrices); a K that is no multiple of 8 goes to
    the library too, as TMA needs 16-byte rows."""
    if x.dtype == torch.float32:
        return linear_f32(x, weight, bias)
    _check(x, "x", torch.bfloat16, 2)
    _check(weight, "weight", torch.bfloat16, 2)
    T = x.shape[0]
    to_library = ((bias is None or GEMM_LIBRARY_WITH_BIAS) and _library_range(T)) \
        or _small_weight_library(T, weight)
    if tc_gemm_supported(x, weight) and not to_library:
        return linear_bf16(x, weight, bias)
    return _library_linear(x, weight, None if bias is None else _bias_bf16(bias))


def linear_swiglu(x: torch.Tensor, w_gate_up: torch.Tensor) -> torch.Tensor:
    """``linear_glu`` with silu."""
    return linear_glu(x, w_gate_up, "silu")


def linear_glu(x: torch.Tensor, w_gate_up: torch.Tensor, kind: str) -> torch.Tensor:
    """act(x gate^T) * (x up^T) for ``w_gate_up`` = [gate rows; up rows], ``kind`` "silu" or
    "gelu_tanh"; fused into the product's epilogue in bfloat16, two kernels otherwise."""
    def gate(rows):
        return silu_mul(rows) if kind == "silu" else glu_act(rows, kind)

    if x.dtype == torch.bfloat16 and tc_gemm_supported(x, w_gate_up):
        T = x.shape[0]
        if _small_weight_library(T, w_gate_up, glu=True) or \
                any(lo <= T <= hi for lo, hi in GEMM_LIBRARY_GLU_TOKENS):
            return gate(_library_linear(x, w_gate_up, None))
        return linear_bf16(x, w_gate_up, glu=kind)
    return gate(linear(x, w_gate_up))


# ------------------------------------------------------------------ sampling
def sample(logits: torch.Tensor, temperature: torch.Tensor, top_k: torch.Tensor,
           top_p: torch.Tensor, seed: torch.Tensor, offset: torch.Tensor,
           kind: Optional[str] = None) -> torch.Tensor:
    """One token id per row of float32 ``logits`` [R, V]; per-row options as device tensors
    (temperature float32 with 0 = greedy, top_k int32 with 0 = off, top_p float32,
    seed and offset int64).  ``kind``: what the caller knows of the options, which live on
    the device: "greedy" (every row takes the argmax), "draw" (some rows draw, none has a
    top-k or top-p), "narrow" (some have); it chooses between the kernel with one block a row
    and the one with a cluster of blocks a row (``sampling.cu``), as does the number of
    rows.  "one_block" takes the first whatever the rows; None counts as "narrow"."""
    _check(logits, "logits", torch.float32, 2)
    R, V = logits.shape
    _check(temperature, "temperature", torch.float32, 1)
    _check(top_k, "top_k", torch.int32, 1)
    _check(top_p, "top_p", torch.float32, 1)
    _check(seed, "seed", torch.int64, 1)
    _check(offset, "offset", torch.int64, 1)
    for name, t in (("temperature", temperature), ("top_k", top_k), ("top_p", top_p),
                    ("seed", seed), ("offset", offset)):
        if t.numel() != R:
            raise KernelError(f"{name} has {t.numel()} entries for {R} rows")
    out = torch.empty((R,), dtype=torch.int32, device=logits.device)
    f = _fn("sampling", "hb_sample",
            [c_void_p, c_void_p, c_int, c_int, c_int, c_void_p, c_void_p, c_void_p, c_void_p,
             c_void_p, c_int, c_void_p])
    _run(f(_p(out), _p(logits), R, V, V, _p(temperature), _p(top_k), _p(top_p), _p(seed),
           _p(offset), _SAMPLE_KINDS[kind], _stream()), "sample")
    return out


_SAMPLE_KINDS = {None: -1, "greedy": 0, "draw": 1, "narrow": 2, "one_block": 3}


def philox_uniform(seed: int, offset: int) -> float:
    """The uniform in [0, 1) that the sampling kernel draws for (seed, offset)."""
    lib = load_library("sampling")
    lib.hb_philox_uniform.argtypes = [c_ulonglong, c_ulonglong]
    lib.hb_philox_uniform.restype = c_float
    return float(lib.hb_philox_uniform(seed & (2**64 - 1), offset & (2**64 - 1)))


def linear_logits(rows: torch.Tensor, weight: torch.Tensor) -> torch.Tensor:
    """Output head: float32 logits [R, V] of ``rows`` [R, H] against ``weight`` [V, H]."""
    if rows.dtype == torch.float32:
        return linear_f32(rows, weight, None)
    _check(rows, "rows", torch.bfloat16, 2)
    _check(weight, "weight", torch.bfloat16, 2)
    if tc_gemm_supported(rows, weight):
        return linear_bf16(rows, weight, out_dtype=torch.float32)
    return torch.mm(rows, weight.t(), out_dtype=torch.float32)


TILED_HEAD_DIMS = (32, 64, 96, 128)
#: attention with options (bias, sink, gate) on the tensor-core kernels where the sizes allow
ATTENTION_OPTIONS_TILED = True
#: merge the context slices of decode attention inside a thread-block cluster (up to 8 slices)
ATTENTION_CLUSTER_MERGE = True
#: steps of single tokens: rotary position encoding and cache write inside the decode kernel
ATTENTION_DECODE_ROTARY = True
#: use the tcgen05 attention kernel for batches with prompt portions where its sizes fit
ATTENTION_TCGEN05 = True
#: ... with two tiles of query rows per block when a request brings more than one tile of tokens
ATTENTION_TILE_PAIRS = True
#: ... and the step gives at least this many blocks of two tiles: with fewer, the blocks of one
#: tile (twice as many, each about 1/1.5 as long) still fit the 148 SMs in one round
ATTENTION_PAIR_MIN_BLOCKS = 75
_sm_counts = {}


def sm_count(device=None) -> int:
    """Streaming multiprocessors of the (current) device."""
    index = torch.cuda.current_device() if device is None else torch.device(device).index or 0
    n = _sm_counts.get(index)
    if n is None:
        n = _sm_counts[index] = torch.cuda.get_device_properties(index).multi_processor_count
    return n


def _wave_splits(blocks: int, slots: int, most: int) -> int:
    """Number of slices per block so that blocks * slices still fits one round of ``slots``
    resident blocks (at most ``most``)."""
    return max(1, min(most, slots // max(1, blocks)))


_decode_clusters = {}

#: Decode attention blocks have 4 warps, two blocks an SM, or 8 warps, one block an SM, for
#: steps of so few requests that clusters of eight such blocks per (request, KV head) are all
#: resident at once: a warp walks its key tiles one after the other, about 0.8 microseconds
#: each, and with few blocks that chain, not the memory, is what the kernel takes.  Measured,
#: milliseconds a decode step at Llama-3.1-8B sizes, context 4,096 (slices, warps): one request
#: 3.140 (29, 4), 3.129 (8, 4), 3.007 (8, 8), 3.073 (18, 8); two 3.192 (17, 4), 3.164 (8, 8);
#: four 3.365 (9, 4), 3.308 (8, 4), 3.289 (4, 8); eight 3.718 (4, 4), 3.891 (2, 8): once the
#: four-warp blocks fill the SMs they are ahead.  False: always 4.
ATTENTION_DECODE_WIDE_BLOCKS = True


def decode_cluster_capacity(head_dim: int, size: int, warps: int = 4) -> int:
    """Clusters of ``size`` decode-attention blocks of ``warps`` warps the device keeps
    resident at once (the occupancy calculator knows how the SMs are spread over the GPCs,
    which bounds whole clusters: 71 clusters of 4 on a B200 where 74 would fit block by block)."""
    key = (head_dim, size, warps)
    if key not in _decode_clusters:
        n = -1
        if torch.cuda.is_available() and head_dim in TILED_HEAD_DIMS and 1 <= size <= 8:
            n = int(load_library("attention_bf16").hb_attention_decode_max_clusters(head_dim, size, warps))
        _decode_clusters[key] = n if n > 0 else ((2 if warps == 4 else 1) * sm_count()) // size
    return _decode_clusters[key]


#: ... and each of the eight warps still has this many keys (four tiles) of the longest context
#: (Qwen2.5-0.5B sizes at 1,024 tokens, 21 keys a warp: 0.783 against 0.773 ms a step)
ATTENTION_DECODE_WIDE_MIN_KEYS = 64


def decode_warps(blocks: int, n_splits: int, head_dim: int, max_context: int) -> int:
    """Warps per block for ``blocks`` (request, KV head) pairs in ``n_splits`` slices of at most
    ``max_context`` keys together: 8 for slices that run as a cluster in a step small enough
    for clusters of eight, where a warp still has keys enough, else 4."""
    if not (ATTENTION_DECODE_WIDE_BLOCKS and ATTENTION_CLUSTER_MERGE and 1 < n_splits <= 8):
        return 4
    if max_context < ATTENTION_DECODE_WIDE_MIN_KEYS * 8 * n_splits:
        return 4
    fits = min(decode_cluster_capacity(head_dim, n_splits, 8), decode_cluster_capacity(head_dim, 8, 8))
    return 8 if blocks <= fits else 4


def decode_splits(num_seqs: int, num_kv_heads: int, max_context: int, head_dim: int = 128) -> int:
    """Slices of the context per (request, KV head) of the decode attention kernel, by a cost
    model fitted to measurements (64 requests x 8 KV heads of 128 at contexts 1,024 and 4,096;
    it then predicts 40 to 96 requests within 5 %): two blocks of four warps are resident per
    SM, the blocks run in rounds of that many, and a block costs its keys plus a fixed part
    (set-up, merge) worth about 176 keys of 128 values; slices that do not run as a cluster
    need the merge kernel, worth about 300 keys more; a block of eight warps
    (``decode_warps``) walks its keys twice as fast.  A slice has at least 128 keys.  More
    slices are taken when the model gives them 4 % (measured, milliseconds a step at
    Llama-3.1-8B sizes, with the count that a margin of 6 % chose against this one's: 16
    requests x 32,768 keys 15.70 / 14.74, 32 x 16,384 15.91 / 15.06, 64 x 8,192 15.63 / 15.21,
    8 x 32,768 9.23 / 8.98)."""
    blocks = max(1, num_seqs * num_kv_heads)
    slots = 2 * sm_count()
    fixed = 176.0 * 128.0 / max(1, head_dim)
    merge_kernel = 300.0 * 128.0 / max(1, head_dim)
    best, best_cost = 1, None
    for s in range(1, max(1, min(32, max_context // 128)) + 1):
        # 2 to 8 slices run as one cluster per (request, KV head) while all clusters are
        # resident at once; otherwise block by block, with a merge kernel
        if decode_warps(blocks, s, head_dim, max_context) == 8:
            cost = max_context / s / 2 + fixed
        else:
            clustered = 1 < s <= 8 and ATTENTION_CLUSTER_MERGE and blocks <= decode_cluster_capacity(head_dim, s)
            rounds = 1 if clustered else -(-blocks * s // slots)
            cost = rounds * (max_context / s + fixed) + (0.0 if clustered or s == 1 else merge_kernel)
        if best_cost is None or cost < best_cost * 0.96:      # fewer slices unless clearly better
            best, best_cost = s, cost
    return best


def attention_decode_bf16(qkv: torch.Tensor, k_pages: torch.Tensor, v_pages: torch.Tensor,
                          block_table: torch.Tensor, positions: torch.Tensor, num_heads: int,
                          num_kv_heads: int, head_dim: int, page_size: int,
                          window: Optional[int], scale: float, n_splits: int,
                          rotary=None, write_cache: bool = False, warps: Optional[int] = None,
                          options: Optional[AttentionOptions] = None, qk_norm=None) -> torch.Tensor:
    """Decode attention (token i is the one new token of request i) on the tensor cores;
    bfloat16, head_dim in TILED_HEAD_DIMS, at most 16 query heads per KV head.  ``options``:
    a distance bias, a sink, a gate (values of the keys' size only).

    ``rotary`` = (cos, sin), float32 [requests, head_dim / 2]: the rows of ``qkv`` are not
    rotated yet; the kernel rotates the query heads on the way in.  ``write_cache``: the
    requests' new keys (rotated likewise) and values are still in ``qkv`` and the kernel
    stores them in the pages before it attends.  (Without either, ``rope_kv_write`` must have
    run.)  ``qk_norm`` = (q weight, k weight, eps, temperature coefficient, temperature period):
    what ``qk_norm_kv_write`` does to q and k, done on the way in (rows may be wider than q | k | v;
    without ``write_cache`` to q alone, and there is no k weight).  ``qkv`` itself is left as it was.  ``warps``: 4 (the default) or 8 warps a block
    (``decode_warps``)."""
    _check(qkv, "qkv", torch.bfloat16, 2)
    _check(k_pages, "k_pages", torch.bfloat16, 4)
    _check(v_pages, "v_pages", torch.bfloat16, 4)
    _check(block_table, "block_table", torch.int32, 2)
    _check(positions, "positions", torch.int32, 1)
    if head_dim not in TILED_HEAD_DIMS:
        raise KernelError(f"head_dim {head_dim} is not one of {TILED_HEAD_DIMS}")
    if num_heads % num_kv_heads or num_heads // num_kv_heads > 16:
        raise KernelError(f"{num_heads} query heads on {num_kv_heads} KV heads: the decode kernel "
                          "takes groups of at most 16")
    if tuple(k_pages.shape[1:]) != (num_kv_heads, page_size, head_dim) or k_pages.shape != v_pages.shape:
        raise KernelError(f"cache pages have shape {tuple(k_pages.shape)}, expected "
                          f"[pages, {num_kv_heads}, {page_size}, {head_dim}]")
    S = qkv.shape[0]
    if block_table.shape[0] != S or positions.numel() != S:
        raise KernelError("decode attention needs one token per request")
    opt = _tiled_options(options, S, num_heads, qkv, head_dim)
    cos = sin = None
    if rotary is not None and rotary[0] is not None:
        cos, sin = rotary
        _check(cos, "cos", torch.float32, 2)
        _check(sin, "sin", torch.float32, 2)
        if tuple(cos.shape) != (S, head_dim // 2) or cos.shape != sin.shape \
                or not (cos.is_contiguous() and sin.is_contiguous()):
            raise KernelError(f"rotary tables have shape {tuple(cos.shape)}, expected ({S}, {head_dim // 2})")
    wq = wk = None
    n_eps, t_coef, t_every = 0.0, 0.0, 0
    if qk_norm is not None:
        wq, wk, n_eps, t_coef, t_every = qk_norm
        if not write_cache and wk is not None:
            raise KernelError("a key norm inside the decode kernel goes with the cache write")
        for name, w in (("q norm weight", wq), ("k norm weight", wk)):
            if w is not None:
                _check(w, name, torch.float32, 1)
                if w.numel() != head_dim:
                    raise KernelError(f"{name} has {w.numel()} entries for heads of {head_dim}")
        if write_cache and (wq is None) != (wk is None):
            raise KernelError("query and key norm come together")
    exact = qk_norm is None            # rows of a fused projection may carry more columns behind q | k | v
    if (cos is not None or write_cache) and ((qkv.shape[1] != (num_heads + 2 * num_kv_heads) * head_dim if exact
                                              else qkv.shape[1] < (num_heads + 2 * num_kv_heads) * head_dim)
                                             or not qkv.is_contiguous()):
        raise KernelError(f"q|k|v rows have {qkv.shape[1]} entries for {num_heads} + 2 x {num_kv_heads} "
                          f"heads of {head_dim}")
    out = torch.empty((S, num_heads * head_dim), dtype=torch.bfloat16, device=qkv.device)
    part_o = part_ml = None
    # slices as one cluster only while all blocks are resident at once: with several rounds
    # of blocks, clusters (whose blocks must start together) cost more than the merge kernel
    warps = 4 if warps is None else int(warps)
    if warps not in (4, 8):
        raise KernelError(f"decode attention blocks have 4 or 8 warps, not {warps}")
    one_round = n_splits <= 8 and S * num_kv_heads <= decode_cluster_capacity(head_dim, n_splits, warps)
    if n_splits > 8 or (n_splits > 1 and not (ATTENTION_CLUSTER_MERGE and one_round)):
        part_o = torch.empty((S, num_heads, n_splits, head_dim), dtype=torch.float32, device=qkv.device)
        part_ml = torch.empty((S, num_heads, n_splits, 2), dtype=torch.float32, device=qkv.device)
    f = _fn("attention_bf16", "hb_attention_decode_bf16",
            [c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_int,
             c_void_p, c_int, c_int, c_int, c_int, c_int, c_int, c_float, c_int, c_void_p, c_void_p,
             c_int, c_int, c_void_p, c_int, c_void_p, c_int, c_void_p, c_int, c_void_p, c_int, c_int,
             c_void_p, c_void_p, c_float, c_float, c_int, c_void_p])
    _run(f(_p(out), _p(part_o), _p(part_ml), _p(qkv), qkv.shape[1], _p(k_pages), _p(v_pages),
           _p(block_table), block_table.shape[1], _p(positions), S, num_heads, num_kv_heads,
           head_dim, page_size, int(window or 0), float(scale), int(n_splits), _p(cos), _p(sin),
           1 if write_cache else 0, int(warps), _p(opt.slopes), int(opt.sink), _p(opt.gate),
           opt.gate_stride, *_option_args(opt, window), _p(wq), _p(wk), float(n_eps), float(t_coef),
           int(t_every), _stream()),
         "attention_decode_bf16")
    return out


def prefill_tiling(num_heads: int, num_kv_heads: int):
    """(query heads per block, 16-token sub-tiles per block) of the prefill kernel."""
    group = num_heads // num_kv_heads
    heads = min(group, 8)
    return heads, max(1, 8 // heads)


def attention_prefill_bf16(qkv: torch.Tensor, k_pages: torch.Tensor, v_pages: torch.Tensor,
                           block_table: torch.Tensor, q_tiles: torch.Tensor,
                           cu_tokens: torch.Tensor, start_pos: torch.Tensor, num_heads: int,
                           num_kv_heads: int, head_dim: int, page_size: int,
                           window: Optional[int], scale: float,
                           options: Optional[AttentionOptions] = None) -> torch.Tensor:
    """Attention of query-token tiles over the cache, causal by position; ``q_tiles`` is
    int32 [tiles, 2] = (request, first local token) for tiles of
    ``16 * prefill_tiling(...)[1]`` tokens."""
    _check(qkv, "qkv", torch.bfloat16, 2)
    _check(k_pages, "k_pages", torch.bfloat16, 4)
    _check(v_pages, "v_pages", torch.bfloat16, 4)
    _check(block_table, "block_table", torch.int32, 2)
    _check(q_tiles, "q_tiles", torch.int32, 2)
    _check(cu_tokens, "cu_tokens", torch.int32, 1)
    _check(start_pos, "start_pos", torch.int32, 1)
    if head_dim not in TILED_HEAD_DIMS:
        raise KernelError(f"head_dim {head_dim} is not one of {TILED_HEAD_DIMS}")
    if num_heads % num_kv_heads:
        raise KernelError(f"{num_heads} query heads are not a multiple of {num_kv_heads} KV heads")
    if tuple(k_pages.shape[1:]) != (num_kv_heads, page_size, head_dim) or k_pages.shape != v_pages.shape:
        raise KernelError(f"cache pages have shape {tuple(k_pages.shape)}, expected "
                          f"[pages, {num_kv_heads}, {page_size}, {head_dim}]")
    heads, subtiles = prefill_tiling(num_heads, num_kv_heads)
    T = qkv.shape[0]
    opt = _tiled_options(options, T, num_heads, qkv, head_dim)
    out = torch.empty((T, num_heads * head_dim), dtype=torch.bfloat16, device=qkv.device)
    f = _fn("attention_bf16", "hb_attention_prefill_bf16",
            [c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_int, c_void_p, c_int,
             c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_float,
             c_void_p, c_int, c_void_p, c_int, c_void_p, c_int, c_void_p, c_int, c_int, c_void_p])
    _run(f(_p(out), _p(qkv), qkv.shape[1], _p(k_pages), _p(v_pages), _p(block_table),
           block_table.shape[1], _p(q_tiles), q_tiles.shape[0], _p(cu_tokens), _p(start_pos),
           num_heads, num_kv_heads, head_dim, heads, subtiles, page_size, int(window or 0),
           float(scale), _p(opt.slopes), int(opt.sink), _p(opt.gate), opt.gate_stride,
           *_option_args(opt, window), _stream()),
         "attention_prefill_bf16")
    return out


def tc_attention_supported(num_heads: int, num_kv_heads: int, head_dim: int, page_size: int) -> bool:
    """Sizes the tcgen05 prefill attention kernel takes."""
    group = num_heads // max(1, num_kv_heads)
    return (head_dim in (64, 128) and num_heads % num_kv_heads == 0 and group <= 128
            and page_size >= 8 and page_size % 8 == 0 and 128 % page_size == 0)


def attention_prefill_tc(qkv: torch.Tensor, k_pages: torch.Tensor, v_pages: torch.Tensor,
                         block_table: torch.Tensor, q_tiles: torch.Tensor, cu_tokens: torch.Tensor,
                         start_pos: torch.Tensor, num_heads: int, num_kv_heads: int, head_dim: int,
                         page_size: int, window: Optional[int], scale: float, pairs: bool = False,
                         options: Optional[AttentionOptions] = None) -> torch.Tensor:
    """Attention of query tiles over the cache on tcgen05 tensor cores; ``q_tiles`` is int32
    [tiles, 2] = (request, first local token) for tiles of ``128 // (nh // nkv)`` tokens, or
    with ``pairs`` of twice as many: then a block works on two tiles of query rows at a time
    (the softmax of one under the products of the other)."""
    _check(qkv, "qkv", torch.bfloat16, 2)
    _check(k_pages, "k_pages", torch.bfloat16, 4)
    _check(v_pages, "v_pages", torch.bfloat16, 4)
    _check(block_table, "block_table", torch.int32, 2)
    _check(q_tiles, "q_tiles", torch.int32, 2)
    _check(cu_tokens, "cu_tokens", torch.int32, 1)
    _check(start_pos, "start_pos", torch.int32, 1)
    if not tc_attention_supported(num_heads, num_kv_heads, head_dim, page_size):
        raise KernelError(f"the tcgen05 attention kernel does not take {num_heads} heads on "
                          f"{num_kv_heads} KV heads, head_dim {head_dim}, page size {page_size}")
    if tuple(k_pages.shape[1:]) != (num_kv_heads, page_size, head_dim) or k_pages.shape != v_pages.shape:
        raise KernelError(f"cache pages have shape {tuple(k_pages.shape)}, expected "
                          f"[pages, {num_kv_heads}, {page_size}, {head_dim}]")
    T = qkv.shape[0]
    out = torch.empty((T, num_heads * head_dim), dtype=torch.bfloat16, device=qkv.device)
    _scratch, _tickets, err = _gemm_workspace(qkv.device)
    common = [c_void_p, c_void_p, c_int, c_void_p, c_void_p, ctypes.c_longlong, c_void_p, c_int, c_void_p,
              c_int, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_float, c_void_p]
    if pairs:
        if options is not None and not options.plain:
            raise KernelError("the kernel with two query tiles a block takes no attention options")
        f = _fn("attention_pair", "hb_attention_prefill_pair", common + [c_void_p])
        _run(f(_p(out), _p(qkv), qkv.shape[1], _p(k_pages), _p(v_pages), k_pages.shape[0], _p(block_table),
               block_table.shape[1], _p(q_tiles), q_tiles.shape[0], _p(cu_tokens), _p(start_pos), num_heads,
               num_kv_heads, head_dim, page_size, int(window or 0), float(scale), _p(err), _stream()),
             "attention_prefill_pair")
        return out
    opt = _tiled_options(options, T, num_heads, qkv, head_dim)
    bias_t = opt.bias_table_t
    if opt.bias_table is not None and bias_t is None:
        bias_t = opt.bias_table.t().contiguous()
    if bias_t is not None:
        _check(bias_t, "bias_table_t", torch.float32, 2)
        if opt.bias_table is None or tuple(bias_t.shape) != (num_heads, opt.bias_table.shape[0]):
            raise KernelError(f"the transposed bias table {tuple(bias_t.shape)} does not fit")
    f = _fn("attention_tc", "hb_attention_prefill_tc",
            common + [c_void_p, c_int, c_void_p, c_int, c_void_p, c_int, c_void_p, c_int, c_int, c_void_p])
    _run(f(_p(out), _p(qkv), qkv.shape[1], _p(k_pages), _p(v_pages), k_pages.shape[0], _p(block_table),
           block_table.shape[1], _p(q_tiles), q_tiles.shape[0], _p(cu_tokens), _p(start_pos), num_heads,
           num_kv_heads, head_dim, page_size, int(window or 0), float(scale), _p(err), _p(opt.slopes),
           int(opt.sink), _p(opt.gate), opt.gate_stride, _p(bias_t),
           0 if bias_t is None else int(bias_t.shape[1]), _p(opt.sink_values), opt.keep_first if window else 0,
           1 if opt.gate_wide else 0, _stream()),
         "attention_prefill_tc")
    return out


#: first local token of a tile that holds no work (padding of a captured step's tile list)
EMPTY_TILE_TOKEN = 1 << 30


def query_tile_rows(tokens_per_seq, tile: int, start_positions=None):
    """(request, first local token) of every tile of ``tile`` tokens, as a list.  With
    ``start_positions`` the tiles that see the most keys come first (they run longest)."""
    rows = [(i, t0) for i, n in enumerate(tokens_per_seq) for t0 in range(0, n, tile)]
    if start_positions is not None:
        rows.sort(key=lambda r: -(start_positions[r[0]] + r[1]))
    return rows


def query_tiles(tokens_per_seq, tile: int, device, start_positions=None) -> torch.Tensor:
    """int32 [tiles, 2] on ``device``: ``query_tile_rows`` copied over."""
    host = torch.tensor(query_tile_rows(tokens_per_seq, tile, start_positions), dtype=torch.int32).reshape(-1, 2)
    if torch.device(device).type == "cuda":
        host = host.pin_memory()
    return host.to(device, non_blocking=True)


def _step_tiles(ctx, tile: int, longest_first: bool, device) -> torch.Tensor:
    """The step's query tiles of ``tile`` tokens: made once per step and tile size; a step
    that runs as a captured graph hands out buffers that it refills itself
    (``ctx.extras["tile_provider"]``)."""
    key = ("q_tiles", tile, longest_first)
    tiles = ctx.extras.get(key)
    if tiles is None:
        provider = ctx.extras.get("tile_provider")
        if provider is not None:
            tiles = provider(tile, longest_first)
        else:
            tiles = query_tiles([s.num_tokens for s in ctx.seqs], tile, device,
                                [s.start_pos for s in ctx.seqs] if longest_first else None)
        ctx.extras[key] = tiles
    return tiles


def attention(ctx, qkv: torch.Tensor, k_pages: torch.Tensor, v_pages: torch.Tensor,
              block_table: torch.Tensor, num_heads: int, num_kv_heads: int, head_dim: int,
              page_size: int, window: Optional[int], scale: float,
              fresh=None, options: Optional[AttentionOptions] = None, prepare=None) -> torch.Tensor:
    """Attention of the step's tokens over the cache; chooses the kernel by dtype, sizes
    and the shape of the batch described by ``ctx``.  bfloat16 with a tiled head size
    runs on the tensor cores (split-context decode kernel for batches of single tokens,
    tiled kernel otherwise); everything else, and float32, on the generic kernel.

    ``fresh`` = (cos, sin, write_cache): ``qkv`` comes straight from the projection; q and k
    are rotated (tables None: no rotation) and, with ``write_cache``, k and v stored in the
    pages first: inside the decode kernel where that one runs, else by ``rope_kv_write``.

    ``options`` (``AttentionOptions``): a distance bias, a sink, a gate, values of another size.
    ``prepare`` = (q weight, k weight, eps, temperature coefficient, temperature period,
    write_cache), with ``options`` only: ``qkv`` comes straight from a fused projection and still
    wants ``qk_norm_kv_write``: inside the decode kernel where that one runs, else as a launch."""
    if prepare is not None or (options is not None and not options.plain):
        return _attention_with_options(ctx, qkv, k_pages, v_pages, block_table, num_heads, num_kv_heads,
                                       head_dim, page_size, window, scale, options or _NO_OPTIONS, prepare)
    decode = (qkv.dtype == torch.bfloat16 and head_dim in TILED_HEAD_DIMS and ctx.decode_only
              and num_heads // num_kv_heads <= 16)
    rotary, write_cache = None, False
    if fresh is not None:
        cos, sin, write = fresh
        if decode and ATTENTION_DECODE_ROTARY and (cos is None or cos.shape[1] * 2 == head_dim):
            rotary, write_cache = (cos, sin), bool(write)
        else:
            rope_kv_write(qkv, cos, sin, ctx.positions, ctx.seq_of_token, block_table, k_pages, v_pages,
                          num_heads, num_kv_heads, head_dim, page_size, write_cache=write)
    if qkv.dtype == torch.bfloat16 and head_dim in TILED_HEAD_DIMS:
        if decode:
            splits = ctx.extras.get("decode_splits")
            if splits is None:
                splits = decode_splits(ctx.num_seqs, num_kv_heads, ctx.max_context_len, head_dim)
            return attention_decode_bf16(qkv, k_pages, v_pages, block_table, ctx.positions,
                                         num_heads, num_kv_heads, head_dim, page_size, window,
                                         scale, splits, rotary, write_cache,
                                         decode_warps(ctx.num_seqs * num_kv_heads, splits, head_dim,
                                                      ctx.max_context_len))
        if (ATTENTION_TCGEN05 and ctx.max_tokens_per_seq >= 16
                and tc_attention_supported(num_heads, num_kv_heads, head_dim, page_size)):
            tile = 128 // (num_heads // num_kv_heads)
            # two tiles of query rows per block when that still gives most SMs a block: a
            # block of two tiles takes about 1.5 times as long as a block of one
            pairs = (ATTENTION_TILE_PAIRS and ctx.max_tokens_per_seq > tile
                     and -(-ctx.num_tokens // (2 * tile)) * num_kv_heads >= ATTENTION_PAIR_MIN_BLOCKS)
            tiles = _step_tiles(ctx, 2 * tile if pairs else tile, True, qkv.device)
            return attention_prefill_tc(qkv, k_pages, v_pages, block_table, tiles, ctx.cu_tokens,
                                        ctx.start_pos, num_heads, num_kv_heads, head_dim, page_size,
                                        window, scale, pairs)
        _heads, subtiles = prefill_tiling(num_heads, num_kv_heads)
        tiles = _step_tiles(ctx, 16 * subtiles, False, qkv.device)
        return attention_prefill_bf16(qkv, k_pages, v_pages, block_table, tiles, ctx.cu_tokens,
                                      ctx.start_pos, num_heads, num_kv_heads, head_dim, page_size,
                                      window, scale)
    return attention_generic(qkv, k_pages, v_pages, block_table, ctx.seq_of_token, ctx.positions,
                             num_heads, num_kv_heads, head_dim, page_size, window, scale)


#: steps of single tokens: q/k norm, temperature and cache write inside the decode kernel
ATTENTION_DECODE_QK_NORM = True


def _attention_with_options(ctx, qkv, k_pages, v_pages, block_table, num_heads, num_kv_heads, head_dim,
                            page_size, window, scale, options: AttentionOptions, prepare=None) -> torch.Tensor:
    """The kernels that take ``AttentionOptions``.  Without ``prepare`` q is ready and the
    step's keys and values are in the pages; with it (see ``attention``) that is done here first,
    by ``qk_norm_kv_write`` or by the decode kernel itself.  bfloat16 with a tiled head size and values of the
    keys' size runs on the tensor cores as plain attention does: the split-context decode
    kernel for steps of single tokens, the tcgen05 kernel with one tile of query rows a block
    for portions, the ``mma.sync`` kernel for the sizes that one does not take.  Other sizes
    that are multiples of 8, with a sink or a gate as the only options, run on the same two
    kernels compiled for sizes of their own (``sized_attention_supported``).  Everything
    else, and float32, runs one warp a (token, head)."""
    value_dim = options.value_dim or head_dim
    tiled = (ATTENTION_OPTIONS_TILED and qkv.dtype == torch.bfloat16 and head_dim in TILED_HEAD_DIMS
             and options.tiled)
    decode = tiled and ctx.decode_only and num_heads // num_kv_heads <= 16
    sized = None
    if not tiled and ATTENTION_OPTIONS_TILED and qkv.dtype == torch.bfloat16 \
            and qkv.stride(0) % 8 == 0 and qkv.data_ptr() % 16 == 0:
        sized = sized_attention_supported(options, num_heads, num_kv_heads, head_dim, value_dim, page_size,
                                          ctx.decode_only)
    fused = None
    if isinstance(prepare, RotateNormPrepare):
        pr = prepare
        qk_rotate_norm_write(qkv, pr.cos, pr.sin, ctx.positions, ctx.seq_of_token, block_table, k_pages,
                             v_pages, num_heads, num_kv_heads, head_dim, value_dim,
                             page_size, pr.norm, pr.q_weight, pr.k_weight, pr.eps, pr.value_col,
                             write_cache=pr.write, pairing=pr.pairing)
    elif prepare is not None:
        wq, wk, eps, coef, every, write = prepare
        alone = not write and wk is None and wq is not None        # the rows hold queries alone
        if (write or alone) and ATTENTION_DECODE_QK_NORM and qkv.is_contiguous() \
                and (decode or (sized == "decode" and not every)):
            fused = (wq, wk, eps, coef, every)
        else:
            qk_norm_kv_write(qkv, ctx.positions, ctx.seq_of_token, block_table, k_pages, v_pages, num_heads,
                             0 if alone else num_kv_heads, head_dim, value_dim, page_size, wq, wk, eps,
                             coef, every, write_cache=write)
    if tiled:
        if decode:
            splits = ctx.extras.get("decode_splits")
            if splits is None:
                splits = decode_splits(ctx.num_seqs, num_kv_heads, _keys_seen(ctx, window), head_dim)
            return attention_decode_bf16(qkv, k_pages, v_pages, block_table, ctx.positions, num_heads,
                                         num_kv_heads, head_dim, page_size, window, scale, splits,
                                         None, fused is not None and bool(prepare[5]),
                                         decode_warps(ctx.num_seqs * num_kv_heads, splits, head_dim,
                                                      _keys_seen(ctx, window)), options=options, qk_norm=fused)
        if (ATTENTION_TCGEN05 and ctx.max_tokens_per_seq >= 16
                and tc_attention_supported(num_heads, num_kv_heads, head_dim, page_size)):
            tiles = _step_tiles(ctx, 128 // (num_heads // num_kv_heads), True, qkv.device)
            return attention_prefill_tc(qkv, k_pages, v_pages, block_table, tiles, ctx.cu_tokens,
                                        ctx.start_pos, num_heads, num_kv_heads, head_dim, page_size,
                                        window, scale, False, options=options)
        _heads, subtiles = prefill_tiling(num_heads, num_kv_heads)
        tiles = _step_tiles(ctx, 16 * subtiles, False, qkv.device)
        return attention_prefill_bf16(qkv, k_pages, v_pages, block_table, tiles, ctx.cu_tokens,
                                      ctx.start_pos, num_heads, num_kv_heads, head_dim, page_size,
                                      window, scale, options=options)
    if sized is not None:
        out = torch.empty((qkv.shape[0], num_heads * value_dim), dtype=qkv.dtype, device=qkv.device)
        cache = LayerPages(k_pages, v_pages, page_size)
        if sized == "decode":
            splits = ctx.extras.get("decode_splits")
            if splits is None:
                splits = decode_splits(ctx.num_seqs, num_kv_heads, _keys_seen(ctx, window), max(head_dim, value_dim))
            _pooled_decode(ctx, qkv, cache, block_table, None, num_heads, num_kv_heads, head_dim, value_dim,
                           int(window or 0), 0, scale, out, 1.0, int(splits), options,
                           None if fused is None else fused[:3], fused is not None and bool(prepare[5]))
        else:
            _pooled_prefill_tc(ctx, qkv, cache, block_table, None, num_heads, num_kv_heads, head_dim, value_dim,
                               int(window or 0), 0, scale, out, 1.0, options)
        return out
    return attention_generic(qkv, k_pages, v_pages, block_table, ctx.seq_of_token, ctx.positions,
                             num_heads, num_kv_heads, head_dim, page_size, window, scale, options)


def _keys_seen(ctx, window: Optional[int]) -> int:
    """Most keys a token of the step sees."""
    return min(ctx.max_context_len, int(window)) if window else ctx.max_context_len


def sized_attention_supported(options: AttentionOptions, num_heads: int, num_kv_heads: int, head_dim: int,
                              value_dim: int, page_size: int, decode: bool) -> Optional[str]:
    """"decode" or "portions" where the tensor-core kernels compiled for key and value sizes of
    their own take these sizes and options, else None."""
    if options.slopes is not None or options.bias_table is not None or options.keep_first:
        return None
    if decode and pooled_decode_supported(num_heads, num_kv_heads, head_dim, value_dim):
        return "decode"
    return "portions" if pooled_tc_supported(num_heads, num_kv_heads, head_dim, value_dim, page_size) else None


class LayerPages:
    """Key and value pages as the kernels for sizes of their own take them."""

    __slots__ = ("k_pages", "v_pages", "page_size")

    def __init__(self, k_pages: torch.Tensor, v_pages: torch.Tensor, page_size: int) -> None:
        self.k_pages, self.v_pages, self.page_size = k_pages, v_pages, page_size


class RotateNormPrepare:
    """What the rows of a fused projection still want before attention (``attention``'s
    ``prepare``): a rotation of q and k by ``cos`` / ``sin`` ([T, rot/2] float32; None: no
    rotation; ``pairing`` "halves": value i of a head paired with value i + rot/2, "neighbours":
    value 2i with value 2i + 1), then, with ``norm`` True, the division of every q and k head by
    its root mean square (eps inside the root) and optional weights per channel ([head_dim]).
    ``norm`` "row": the RMS norm comes BEFORE the rotation and runs over the whole q row and the
    whole k row (all heads at once) with weights of the rows' sizes.  The keys go to the key
    pages and the values to the value pages: from the columns at ``value_col``, or, with
    ``value_col`` None, the values ARE the keys as projected, before rotation and norm."""

    __slots__ = ("cos", "sin", "norm", "q_weight", "k_weight", "eps", "value_col", "write", "pairing")

    def __init__(self, cos=None, sin=None, norm=True, q_weight=None, k_weight=None,
                 eps: float = 1e-6, value_col: Optional[int] = None, write: bool = True,
                 pairing: str = "halves") -> None:
        self.cos, self.sin = cos, sin
        self.norm = norm if norm == "row" else bool(norm)
        self.q_weight, self.k_weight, self.eps = q_weight, k_weight, float(eps)
        self.value_col, self.write, self.pairing = value_col, bool(write), pairing


ROTARY_PAIRINGS = {"halves": 0, "neighbours": 1}


def qk_rotate_norm_write(rows: torch.Tensor, cos: Optional[torch.Tensor], sin: Optional[torch.Tensor],
                         positions: torch.Tensor, seq_of_token: torch.Tensor, block_table: torch.Tensor,
                         k_pages: Optional[torch.Tensor], v_pages: Optional[torch.Tensor], num_heads: int,
                         num_kv_heads: int, head_dim: int, value_dim: int, page_size: int, norm: bool,
                         q_weight: Optional[torch.Tensor], k_weight: Optional[torch.Tensor], eps: float,
                         value_col: Optional[int], write_cache: bool = True, pairing: str = "halves") -> None:
    """See ``RotateNormPrepare``: rows [T, ld] hold q heads, then k heads, from column 0; q is
    rotated and normed in place, k rotated and normed into the key pages (in place without
    ``write_cache``), the values copied into the value pages.  float32 arithmetic."""
    if pairing not in ROTARY_PAIRINGS:
        raise KernelError(f"pairing {pairing!r} is not one of {sorted(ROTARY_PAIRINGS)}")
    _check(rows, "rows", None, 2)
    T, ld = rows.shape
    _check(positions, "positions", torch.int32, 1)
    _check(seq_of_token, "seq_of_token", torch.int32, 1)
    _check(block_table, "block_table", torch.int32, 2)
    rot = 0
    if cos is not None:
        _check(cos, "cos", torch.float32, 2)
        _check(sin, "sin", torch.float32, 2)
        if cos.shape != sin.shape or cos.shape[0] != T:
            raise KernelError(f"cos/sin tables {tuple(cos.shape)}/{tuple(sin.shape)} do not match {T} tokens")
        rot = 2 * cos.shape[1]
        if rot > head_dim:
            raise KernelError(f"rotary dimension {rot} exceeds head_dim {head_dim}")
    for name, w, heads in (("q_weight", q_weight, num_heads), ("k_weight", k_weight, num_kv_heads)):
        if w is not None:
            _check(w, name, torch.float32, 1)
            want = head_dim * (heads if norm == "row" else 1)
            if w.numel() != want:
                raise KernelError(f"{name} has {w.numel()} entries where the norm runs over {want}")
    if head_dim > 256:
        raise KernelError(f"heads of {head_dim} values are not supported (at most 256)")
    if value_col is None and value_dim != head_dim:
        raise KernelError("values that are the keys have the keys' size")
    if write_cache:
        for name, pages, d in (("k_pages", k_pages, head_dim), ("v_pages", v_pages, value_dim)):
            _check(pages, name, rows.dtype, 4)
            if tuple(pages.shape[1:]) != (num_kv_heads, page_size, d):
                raise KernelError(f"{name} has shape {tuple(pages.shape)}, expected "
                                  f"[pages, {num_kv_heads}, {page_size}, {d}]")
    f = _fn("elementwise", "hb_qk_rotate_norm_write",
            [c_void_p, c_int, c_int, c_void_p, c_void_p, c_int, c_int, c_void_p, c_void_p, c_void_p, c_int,
             c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_int, c_void_p, c_void_p, c_float,
             c_int, c_int, c_int, c_void_p])
    _run(f(_p(rows), ld, -1 if value_col is None else int(value_col), _p(cos), _p(sin), rot,
           ROTARY_PAIRINGS[pairing], _p(positions), _p(seq_of_token), _p(block_table), block_table.shape[1],
           _p(k_pages) if write_cache else 0, _p(v_pages) if write_cache else 0, T, num_heads,
           num_kv_heads, head_dim, value_dim, 2 if norm == "row" else (1 if norm else 0),
           _p(q_weight), _p(k_weight), float(eps),
           page_size, 1 if write_cache else 0, _dt(rows.dtype), _stream()), "qk_rotate_norm_write")


def qk_norm_kv_write(rows: torch.Tensor, positions: torch.Tensor, seq_of_token: torch.Tensor,
                     block_table: torch.Tensor, k_pages: Optional[torch.Tensor],
                     v_pages: Optional[torch.Tensor], num_heads: int, num_kv_heads: int, head_dim: int,
                     value_dim: int, page_size: int, q_weight: Optional[torch.Tensor],
                     k_weight: Optional[torch.Tensor], eps: float, temp_coef: float = 0.0,
                     temp_every: int = 0, write_cache: bool = True) -> None:
    """For the rows of a fused projection ([T, ld]: q heads, k heads, v heads from column 0,
    whatever follows): every q head becomes q / rms(q) * q_weight * (1 + temp_coef *
    ln(floor((p + 1) / temp_every) + 1)) in place (p the token's position; ``temp_every`` 0: no
    such factor; weights None: no norm), every k head k / rms(k) * k_weight at the token's
    place in the key pages, every v head goes to the value pages.  Rows that hold queries alone
    (``num_kv_heads`` 0, no key weight) only norm those.  float32 arithmetic."""
    _check(rows, "rows", None, 2)
    T, ld = rows.shape
    _check(positions, "positions", torch.int32, 1)
    _check(seq_of_token, "seq_of_token", torch.int32, 1)
    _check(block_table, "block_table", torch.int32, 2)
    if num_kv_heads and (q_weight is None) != (k_weight is None):
        raise KernelError("query and key norm come together")
    if not num_kv_heads and write_cache:
        raise KernelError("rows without keys have nothing to store")
    for name, w in (("q_weight", q_weight), ("k_weight", k_weight)):
        if w is not None:
            _check(w, name, torch.float32, 1)
            if w.numel() != head_dim:
                raise KernelError(f"{name} has {w.numel()} entries for heads of {head_dim}")
    if num_heads * head_dim + num_kv_heads * (head_dim + value_dim) > ld:
        raise KernelError(f"rows of {ld} columns do not hold {num_heads} q, {num_kv_heads} k and v heads")
    if write_cache:
        for name, pages, d in (("k_pages", k_pages, head_dim), ("v_pages", v_pages, value_dim)):
            _check(pages, name, rows.dtype, 4)
            if tuple(pages.shape[1:]) != (num_kv_heads, page_size, d):
                raise KernelError(f"{name} has shape {tuple(pages.shape)}, expected "
                                  f"[pages, {num_kv_heads}, {page_size}, {d}]")
    f = _fn("elementwise", "hb_qk_norm_kv_write",
            [c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_int, c_int,
             c_int, c_int, c_int, c_void_p, c_void_p, c_float, c_float, c_int, c_int, c_int, c_int,
             c_void_p])
    _run(f(_p(rows), ld, _p(positions), _p(seq_of_token), _p(block_table), block_table.shape[1],
           _p(k_pages) if write_cache else 0, _p(v_pages) if write_cache else 0, T, num_heads,
           num_kv_heads, head_dim, value_dim, _p(q_weight), _p(k_weight), float(eps), float(temp_coef),
           int(temp_every), page_size, 1 if write_cache else 0, _dt(rows.dtype), _stream()),
         "qk_norm_kv_write")


# ------------------------------------------------------------------ layer norm, learned positions
def add_layernorm(residual: torch.Tensor, weight: Optional[torch.Tensor], bias: Optional[torch.Tensor],
                  eps: float, out_dtype: Optional[torch.dtype], rows: Optional[torch.Tensor] = None,
                  a: Optional[torch.Tensor] = None, scale_a: Optional[torch.Tensor] = None,
                  b: Optional[torch.Tensor] = None, scale_b: Optional[torch.Tensor] = None,
                  mult: float = 1.0) -> Optional[torch.Tensor]:
    """``residual += mult * (scale_a * a + scale_b * b)`` (float32, in place; a, b [n, H] in one
    dtype, the scales float32 [H] or None for 1) and the layer norm of the new rows, (x - mean) /
    sqrt(var + eps) * weight + bias, in ``out_dtype``.  With ``rows`` (int32) only those rows are
    normed and the residual is left as it was.  ``out_dtype`` None: only the add."""
    _check(residual, "residual", torch.float32, 2)
    n, H = residual.shape
    act = None
    for name, t in (("a", a), ("b", b)):
        if t is not None:
            _check(t, name, None, 2)
            if tuple(t.shape) != (n, H) or (act is not None and t.dtype != act):
                raise KernelError(f"{name} {tuple(t.shape)} {t.dtype} does not match residual {(n, H)}")
            act = t.dtype
    for name, t in (("scale_a", scale_a), ("scale_b", scale_b), ("weight", weight), ("bias", bias)):
        if t is not None:
            _check(t, name, torch.float32, 1)
            if t.numel() != H:
                raise KernelError(f"{name} has {t.numel()} entries for width {H}")
    out = None
    n_out = n
    if out_dtype is not None:
        if weight is None:
            raise KernelError("a norm needs its weight")
        if act is not None and act != out_dtype:
            raise KernelError(f"pending tensors are {act}, the norm's output {out_dtype}")
        if rows is not None:
            _check(rows, "rows", torch.int32, 1)
            n_out = rows.numel()
        out = torch.empty((n_out, H), dtype=out_dtype, device=residual.device)
    elif act is None:
        return None
    f = _fn("elementwise", "hb_add_layernorm",
            [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_float, c_void_p, c_void_p,
             c_void_p, c_int, c_int, c_float, c_int, c_void_p])
    _run(f(_p(out), _p(residual), _p(a), _p(scale_a), _p(b), _p(scale_b), float(mult), _p(weight),
           _p(bias), _p(rows) if out is not None else 0, n_out, H, float(eps),
           _dt(out_dtype if out_dtype is not None else act), _stream()), "add_layernorm")
    return out


def add_table_rows(hidden: torch.Tensor, table: torch.Tensor, index: torch.Tensor) -> torch.Tensor:
    """``hidden[t] += table[index[t]]`` in float32 and in place (hidden float32 [T, H], table
    [V, H] float32 or bfloat16, index int32 [T])."""
    _check(hidden, "hidden", torch.float32, 2)
    _check(table, "table", None, 2)
    _check(index, "index", torch.int32, 1)
    T, H = hidden.shape
    if table.shape[1] != H or index.numel() != T:
        raise KernelError(f"table {tuple(table.shape)} / index {index.numel()} do not fit hidden {(T, H)}")
    f = _fn("elementwise", "hb_add_table_rows", [c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_void_p])
    _run(f(_p(hidden), _p(table), _p(index), T, H, table.shape[0], _dt(table.dtype), _stream()), "add_table_rows")
    return hidden


def cast_rows(dst: torch.Tensor, col0: int, src: torch.Tensor) -> None:
    """``dst[:, col0 : col0 + W] = src`` (float32 [T, W]) in dst's dtype; dst [T, ld] contiguous."""
    _check(dst, "dst", None, 2)
    _check(src, "src", torch.float32, 2)
    T, W = src.shape
    if dst.shape[0] != T or col0 < 0 or col0 + W > dst.shape[1]:
        raise KernelError(f"columns {col0}..{col0 + W} of {tuple(dst.shape)} do not take {tuple(src.shape)}")
    f = _fn("elementwise", "hb_cast_rows", [c_void_p, c_int, c_int, c_void_p, c_int, c_int, c_int, c_void_p])
    _run(f(_p(dst), dst.shape[1], col0, _p(src), T, W, _dt(dst.dtype), _stream()), "cast_rows")


# ------------------------------------------------------------------ gated activations, post-norm
GLU_KINDS = {"silu": 0, "gelu_tanh": 1, "clamped_swish": 2}


def glu_act(gate_up: torch.Tensor, kind: str, limit: float = 0.0) -> torch.Tensor:
    """act(gate) * up for ``gate_up`` = [T, 2 I] (gate columns first).  ``kind``: "silu",
    "gelu_tanh" (0.5 g (1 + tanh(sqrt(2/pi) (g + 0.044715 g^3))) * u) or "clamped_swish"
    (g' = min(g, limit), u' = clamp(u, -limit, limit), g' sigmoid(1.702 g') (u' + 1))."""
    _check(gate_up, "gate_up", None, 2)
    if kind not in GLU_KINDS:
        raise KernelError(f"gated activation {kind!r} is not one of {sorted(GLU_KINDS)}")
    T, two_i = gate_up.shape
    if two_i % 2:
        raise KernelError("gate_up must have an even width")
    out = torch.empty((T, two_i // 2), dtype=gate_up.dtype, device=gate_up.device)
    f = _fn("elementwise", "hb_glu_act",
            [c_void_p, c_void_p, c_int, c_int, c_int, c_float, c_int, c_void_p])
    _run(f(_p(out), _p(gate_up), T, two_i // 2, GLU_KINDS[kind], float(limit), _dt(gate_up.dtype),
           _stream()), "glu_act")
    return out


def rmsnorm_add(residual: torch.Tensor, y: Optional[torch.Tensor], weight: Optional[torch.Tensor],
                eps: float, copy_dtype: Optional[torch.dtype]) -> Optional[torch.Tensor]:
    """``residual += y / sqrt(mean(y^2) + eps) * weight`` row by row, in float32 and in place
    (a block that norms a sublayer's OUTPUT).  With ``copy_dtype`` other than float32 the new
    residual is also returned in that dtype (what the next sublayer reads); for float32 the
    residual itself is returned.  ``y`` None: only the copy."""
    _check(residual, "residual", torch.float32, 2)
    n, H = residual.shape
    if y is not None:
        _check(y, "y", None, 2)
        _check(weight, "weight", torch.float32, 1)
        if tuple(y.shape) != (n, H) or weight.numel() != H:
            raise KernelError(f"y {tuple(y.shape)} / weight {weight.numel()} do not match residual {(n, H)}")
    copy = None
    if copy_dtype is not None and copy_dtype != torch.float32:
        copy = torch.empty((n, H), dtype=copy_dtype, device=residual.device)
    if y is not None or copy is not None:
        f = _fn("elementwise", "hb_rmsnorm_add",
                [c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_float, c_int, c_int, c_void_p])
        _run(f(_p(residual), _p(y), _p(weight), _p(copy), n, H, float(eps),
               _dt(y.dtype) if y is not None else _F32, _dt(copy.dtype) if copy is not None else _F32,
               _stream()), "rmsnorm_add")
    if copy_dtype is None:
        return None
    return residual if copy is None else copy


def rmsnorm_add_rmsnorm(residual: torch.Tensor, y: torch.Tensor, weight1: torch.Tensor, eps1: float,
                        weight2: torch.Tensor, eps2: float, rows: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``residual += y / sqrt(mean(y^2) + eps1) * weight1`` row by row, in float32 and in place, and
    the new rows' own norm, x / sqrt(mean(x^2) + eps2) * weight2, in y's dtype (a block that norms
    before AND after a sublayer: the norm after this one and the norm before the next in one
    launch).  With ``rows`` (int32) only those rows are computed, into [len(rows), H], and the
    residual is left as it was."""
    _check(residual, "residual", torch.float32, 2)
    _check(y, "y", None, 2)
    n, H = residual.shape
    for name, w in (("weight1", weight1), ("weight2", weight2)):
        _check(w, name, torch.float32, 1)
        if w.numel() != H:
            raise KernelError(f"{name} has {w.numel()} entries for rows of {H}")
    if tuple(y.shape) != (n, H):
        raise KernelError(f"y {tuple(y.shape)} does not match residual {(n, H)}")
    if rows is not None:
        _check(rows, "rows", torch.int32, 1)
    n_out = n if rows is None else rows.numel()
    out = torch.empty((n_out, H), dtype=y.dtype, device=y.device)
    f = _fn("elementwise", "hb_rmsnorm_add_rmsnorm",
            [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_float, c_float, c_int,
             c_void_p])
    _run(f(_p(out), _p(residual), _p(y), _p(weight1), _p(weight2), _p(rows), n_out, H, float(eps1), float(eps2),
           _dt(y.dtype), _stream()), "rmsnorm_add_rmsnorm")
    return out


def softcap(x: torch.Tensor, cap: float) -> torch.Tensor:
    """``x = cap * tanh(x / cap)`` in place (float32, contiguous); returns x."""
    _check(x, "x", torch.float32)
    f = _fn("elementwise", "hb_softcap", [c_void_p, ctypes.c_long, c_float, c_void_p])
    _run(f(_p(x), x.numel(), float(cap), _stream()), "softcap")
    return x


def scaled_sum_rmsnorm(residual: torch.Tensor, y: torch.Tensor, weight: torch.Tensor, eps: float,
                       factor: float, copy_dtype: Optional[torch.dtype]) -> Optional[torch.Tensor]:
    """``residual <- v / sqrt(mean(v^2) + eps) * weight`` with ``v = factor * residual + y`` row by
    row, in float32 and in place (a block that norms the SUM).  With ``copy_dtype`` other than
    float32 the new stream is also returned in that dtype; for float32 the stream itself is."""
    _check(residual, "residual", torch.float32, 2)
    _check(y, "y", None, 2)
    _check(weight, "weight", torch.float32, 1)
    n, H = residual.shape
    if tuple(y.shape) != (n, H) or weight.numel() != H:
        raise KernelError(f"y {tuple(y.shape)} / weight {weight.numel()} do not match residual {(n, H)}")
    copy = None
    if copy_dtype is not None and copy_dtype != torch.float32:
        copy = torch.empty((n, H), dtype=copy_dtype, device=residual.device)
    f = _fn("elementwise", "hb_scaled_sum_rmsnorm",
            [c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_float, c_float, c_int, c_int, c_void_p])
    _run(f(_p(residual), _p(y), _p(weight), _p(copy), n, H, float(eps), float(factor), _dt(y.dtype),
           _dt(copy.dtype) if copy is not None else _F32, _stream()), "scaled_sum_rmsnorm")
    if copy_dtype is None:
        return None
    return residual if copy is None else copy


# ------------------------------------------------------------------ attention over a latent cache
_LONG = ctypes.c_long


def latent_prepare(proj: torch.Tensor, pages: Optional[torch.Tensor], norm_weight: torch.Tensor,
                   cos: torch.Tensor, sin: torch.Tensor, positions: torch.Tensor,
                   seq_of_token: torch.Tensor, block_table: torch.Tensor, heads: int, nope: int,
                   rot: int, rank: int, page_size: int, eps: float, write_cache: bool = True) -> None:
    """``proj`` [T, heads (nope + rot) + rank + rot] = [q | latent | shared key part], straight
    from the projection.  The latent is RMS-normed (float32 statistics, ``norm_weight``), the
    shared key part rotated (interleaved pairs, cos/sin [T, nrot / 2] over its first nrot
    values) and both stored as one row [rank + rot] of ``pages`` [pages, 1, page_size, rank +
    rot]; the queries' rotated parts are rotated in place."""
    _check(proj, "proj", None, 2)
    nq = heads * (nope + rot)
    if proj.shape[1] != nq + rank + rot:
        raise KernelError(f"proj has {proj.shape[1]} columns, expected {nq + rank + rot}")
    latent_prepare_parts(proj[:, :nq], proj[:, nq:], None, pages, norm_weight, None, cos, sin, positions,
                         seq_of_token, block_table, heads, nope, rot, rank, page_size, eps,
                         write_cache=write_cache, pairing="neighbours")


def latent_prepare_parts(q: Optional[torch.Tensor], latent: Optional[torch.Tensor],
                         query_latent: Optional[torch.Tensor], pages: Optional[torch.Tensor],
                         norm_weight: Optional[torch.Tensor], query_norm_weight: Optional[torch.Tensor],
                         cos: torch.Tensor, sin: torch.Tensor, positions: torch.Tensor,
                         seq_of_token: torch.Tensor, block_table: torch.Tensor, heads: int, nope: int,
                         rot: int, rank: int, page_size: int, eps: float, write_cache: bool = True,
                         pairing: str = "halves", query_latent_out: Optional[torch.Tensor] = None) -> None:
    """``latent_prepare`` piece by piece; each of the three tensors is a view [T, columns] whose
    rows may be strided (last dimension contiguous), or None to leave the piece out:

    ``query_latent`` [T, q_rank]: RMS-normed (``query_norm_weight``) in place, or into
    ``query_latent_out`` (the same shape; contiguous rows suit the product that follows);
    ``latent`` [T, rank + rot] = [latent | shared key part]: the latent RMS-normed
    (``norm_weight``), the shared key part rotated, both stored as the token's row of ``pages``
    (nothing without ``write_cache``: the rows of another layer serve);
    ``q`` [T, heads (nope + rot)]: every head's rotated part rotated in place.

    ``pairing`` "halves": value i of the rotated part is paired with value i + nrot / 2,
    "neighbours": value 2i with value 2i + 1; cos/sin are [T, nrot / 2]."""
    like = next((x for x in (q, latent, query_latent) if x is not None), None)
    if like is None:
        return
    if pairing not in ROTARY_PAIRINGS:
        raise KernelError(f"pairing {pairing!r} is not one of {sorted(ROTARY_PAIRINGS)}")
    T = like.shape[0]
    if query_latent_out is None:
        query_latent_out = query_latent
    elif query_latent is None or query_latent_out.shape != query_latent.shape:
        raise KernelError("latent_prepare: query_latent_out goes with a query_latent of its shape")
    for name, x, cols in (("q", q, heads * (nope + rot)), ("latent", latent, rank + rot),
                          ("query_latent", query_latent, None), ("query_latent_out", query_latent_out, None)):
        if x is None:
            continue
        if not x.is_cuda or x.dim() != 2 or x.stride(1) != 1 or x.shape[0] != T or x.dtype != like.dtype \
                or (cols is not None and x.shape[1] != cols):
            raise KernelError(f"latent_prepare: {name} {tuple(x.shape)} does not fit ({T} rows of {cols} columns)")
    _check(cos, "cos", torch.float32, 2)
    _check(sin, "sin", torch.float32, 2)
    _check(positions, "positions", torch.int32, 1)
    _check(seq_of_token, "seq_of_token", torch.int32, 1)
    _check(block_table, "block_table", torch.int32, 2)
    nrot = 2 * cos.shape[1]
    if cos.shape != sin.shape or cos.shape[0] != T or nrot > rot:
        raise KernelError(f"cos/sin tables {tuple(cos.shape)} do not fit {T} tokens and {rot} rotated values")
    write = bool(write_cache) and latent is not None
    if latent is not None:
        _check(norm_weight, "norm_weight", torch.float32, 1)
        if norm_weight.numel() != rank:
            raise KernelError(f"norm weight has {norm_weight.numel()} entries for rank {rank}")
    if write:
        _check(pages, "pages", like.dtype, 4)
        if tuple(pages.shape[1:]) != (1, page_size, rank + rot):
            raise KernelError(f"pages have shape {tuple(pages.shape)}, expected [pages, 1, {page_size}, {rank + rot}]")
    q_rank = 0
    if query_latent is not None:
        q_rank = query_latent.shape[1]
        _check(query_norm_weight, "query_norm_weight", torch.float32, 1)
        if query_norm_weight.numel() != q_rank:
            raise KernelError(f"query norm weight has {query_norm_weight.numel()} entries for rank {q_rank}")
    f = _fn("latent_attention", "hb_latent_prepare",
            [c_void_p, c_int, c_void_p, c_int, c_void_p, c_int, c_void_p, c_int, c_int, c_void_p, c_void_p,
             c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_int,
             c_int, c_int, c_int, c_float, c_int, c_int, c_void_p])
    _run(f(_p(q), 0 if q is None else q.stride(0), _p(latent), 0 if latent is None else latent.stride(0),
           _p(query_latent), 0 if query_latent is None else query_latent.stride(0),
           _p(query_latent_out), 0 if query_latent_out is None else query_latent_out.stride(0), q_rank,
           _p(query_norm_weight) if query_latent is not None else 0, _p(pages) if write else 0,
           _p(norm_weight) if latent is not None else 0, _p(cos), _p(sin),
           _p(positions), _p(seq_of_token), _p(block_table), block_table.shape[1], T, heads, nope, rot,
           rank, nrot, ROTARY_PAIRINGS[pairing], page_size, float(eps), 1 if write else 0, _dt(like.dtype),
           _stream()), "latent_prepare")


#: from this many tokens on the per-head products of a bfloat16 step go to the library's
#: batched product (tensor cores); below, and in float32, this package's FMA kernel.  Measured,
#: microseconds a launch in a chain, FMA kernel / library: 16 heads of 128 -> 512 10.6 / 2.9 at one
#: token, 11.4 / 3.2 at 32; 512 -> 128 28.9 / 3.7 and 31.0 / 3.5; 8 heads of 64 -> 256 5.0 / 2.7
HEAD_GEMM_LIBRARY_TOKENS = 1


def head_gemm(a: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """out[t, h, n] = sum_k a[t, h, k] w[h, n, k]: one small matrix per head.  ``a`` is a view
    [T, heads, K] whose last dimension is contiguous (a slice of wider rows is fine); ``w``
    [heads, N, K] contiguous.  Returns [T, heads, N] (a view whose last dimension is
    contiguous), float32 sums."""
    if a.dim() != 3 or w.dim() != 3 or a.shape[1] != w.shape[0] or a.shape[2] != w.shape[2]:
        raise KernelError(f"head_gemm: a {tuple(a.shape)} and w {tuple(w.shape)} do not fit")
    if not a.is_cuda or not w.is_cuda or a.dtype != w.dtype or a.stride(2) != 1 or not w.is_contiguous():
        raise KernelError("head_gemm: tensors must be CUDA, of one dtype, rows contiguous")
    T, H, K = a.shape
    N = w.shape[1]
    if a.dtype == torch.bfloat16 and T >= HEAD_GEMM_LIBRARY_TOKENS:
        return torch.bmm(a.transpose(0, 1), w.transpose(1, 2)).transpose(0, 1)
    out = torch.empty((T, H, N), dtype=a.dtype, device=a.device)
    f = _fn("latent_attention", "hb_head_gemm",
            [c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, _LONG, _LONG, _LONG, c_int, _LONG, _LONG,
             _LONG, c_int, c_void_p])
    _run(f(_p(out), _p(a), _p(w), T, N, K, a.stride(0), K, H * N, H, a.stride(1), N * K, N,
           _dt(a.dtype), _stream()), "head_gemm")
    return out


#: bfloat16 steps run attention over the latent cache on the tensor cores where the sizes
#: allow (rank a multiple of 32, rotated part a multiple of 16); float32 and other sizes run
#: the kernel with one warp a row, whose sums have a fixed order
LATENT_ATTENTION_TENSOR_CORES = True


def linear_rows(x: torch.Tensor, weight: torch.Tensor) -> torch.Tensor:
    """``linear`` for rows that are a column slice of wider rows (last dimension contiguous):
    no copy is made.  float32 runs on ``head_gemm`` with one head, bfloat16 on the library, which
    takes the row stride (``HEAD_GEMM_LIBRARY_TOKENS``)."""
    if x.is_contiguous():
        return linear(x, weight)
    if x.dim() != 2 or x.stride(1) != 1:
        raise KernelError("linear_rows: rows must be contiguous in their last dimension")
    if x.dtype == torch.bfloat16 and x.shape[0] >= HEAD_GEMM_LIBRARY_TOKENS:
        return torch.nn.functional.linear(x, weight)
    return head_gemm(x.unsqueeze(1), weight.unsqueeze(0)).view(x.shape[0], weight.shape[0])


def latent_attention(ctx, q_lat: torch.Tensor, q_rot: torch.Tensor, pages: torch.Tensor,
                     block_table: torch.Tensor, rank: int, rot: int, page_size: int,
                     scale: float, window: Optional[int] = None,
                     sink_values: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Causal attention of every token of the step over its request's latent rows, all of them or
    the last ``window``; ``sink_values`` (float32 [heads]): a key of that score without a value.  ``q_lat``
    [T, heads, rank] and ``q_rot`` [T, heads, rot] are views with a contiguous last dimension;
    ``pages`` [pages, 1, page_size, rank + rot].  Returns [T, heads, rank] (softmax-weighted
    sums of the rows' first ``rank`` values).  ``ctx`` gives seq_of_token and positions, and
    for the tensor-core kernel cu_tokens, start_pos, seqs, max_context_len and extras."""
    _check(pages, "pages", q_lat.dtype, 4)
    _check(block_table, "block_table", torch.int32, 2)
    if q_lat.dim() != 3 or q_rot.dim() != 3 or q_lat.stride(2) != 1 or q_rot.stride(2) != 1 \
            or q_lat.shape[:2] != q_rot.shape[:2] or q_lat.shape[2] != rank or q_rot.shape[2] != rot \
            or q_rot.dtype != q_lat.dtype:
        raise KernelError(f"latent_attention: q_lat {tuple(q_lat.shape)} / q_rot {tuple(q_rot.shape)} "
                          f"do not fit rank {rank}, rot {rot}")
    if tuple(pages.shape[1:]) != (1, page_size, rank + rot):
        raise KernelError(f"pages have shape {tuple(pages.shape)}, expected [pages, 1, {page_size}, {rank + rot}]")
    if rank > 512 or rank + rot > 1024:
        raise KernelError(f"latent rank {rank} (at most 512) or row {rank + rot} (at most 1024) is not supported")
    T, H = q_lat.shape[:2]
    window = int(window or 0)
    if sink_values is not None:
        _check(sink_values, "sink_values", torch.float32, 1)
        if sink_values.numel() != H:
            raise KernelError(f"{sink_values.numel()} sink values for {H} heads")
    out = torch.empty((T, H, rank), dtype=q_lat.dtype, device=q_lat.device)
    if LATENT_ATTENTION_TENSOR_CORES and q_lat.dtype == torch.bfloat16 and rank % 32 == 0 and rot % 16 == 0:
        # 32 query rows a block: (token, head) pairs of one request, which share every key
        hpb = min(H, 32)
        tpt = max(1, 32 // hpb)
        tiles = _step_tiles(ctx, tpt, False, q_lat.device)
        blocks = tiles.shape[0] * -(-H // hpb)
        n_splits = 1
        if blocks < sm_count():
            keys = min(ctx.max_context_len, window + tpt - 1) if window else ctx.max_context_len
            # ranges of at least 256 keys, or of 128 where all of those still have an SM each (a range
            # walks its tiles one after the other; 8 requests, 1,024 keys each: 20.6 against 26.3 us)
            least = 128 if blocks * (keys // 128) <= sm_count() else 256
            n_splits = max(1, min(32, keys // least, -(-2 * sm_count() // blocks)))
        part_acc = part_ml = None
        if n_splits > 1:
            part_acc = torch.empty((T * H, n_splits, rank), dtype=torch.float32, device=q_lat.device)
            part_ml = torch.empty((T * H, n_splits, 2), dtype=torch.float32, device=q_lat.device)
        f = _fn("latent_attention", "hb_latent_attention_mma",
                [c_void_p, c_void_p, c_void_p, c_void_p, _LONG, _LONG, c_void_p, _LONG, _LONG, c_void_p,
                 c_void_p, c_int, c_void_p, c_int, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int,
                 c_int, c_int, c_float, c_int, c_int, c_void_p, c_void_p])
        _run(f(_p(out), _p(part_acc), _p(part_ml), _p(q_lat), q_lat.stride(0), q_lat.stride(1), _p(q_rot),
               q_rot.stride(0), q_rot.stride(1), _p(pages), _p(block_table), block_table.shape[1],
               _p(tiles), tiles.shape[0], _p(ctx.cu_tokens), _p(ctx.start_pos), T, H, hpb, tpt, rank, rot,
               page_size, float(scale), n_splits, window, _p(sink_values), _stream()), "latent_attention_mma")
        return out
    f = _fn("latent_attention", "hb_latent_attention",
            [c_void_p, c_void_p, _LONG, _LONG, c_void_p, _LONG, _LONG, c_void_p, c_void_p, c_int, c_void_p,
             c_void_p, c_int, c_int, c_int, c_int, c_int, c_float, c_int, c_void_p, c_int, c_void_p])
    _run(f(_p(out), _p(q_lat), q_lat.stride(0), q_lat.stride(1), _p(q_rot), q_rot.stride(0),
           q_rot.stride(1), _p(pages), _p(block_table), block_table.shape[1], _p(ctx.seq_of_token),
           _p(ctx.positions), T, H, rank, rot, page_size, float(scale), window, _p(sink_values),
           _dt(q_lat.dtype), _stream()), "latent_attention")
    return out


#: portions expand the latent rows they see to keys and values per head where that is estimated to
#: take less time than attention over the rows themselves: None: by the estimate; True / False: always
#: (where the sizes allow) / never
LATENT_EXPAND = None
#: most bytes of expanded keys and values a step may make
LATENT_EXPAND_BYTES = 2 << 30


def latent_expand_supported(dtype: torch.dtype, heads: int, key_dim: int, value_dim: int, rank: int, rot: int,
                            page_size: int) -> bool:
    """Sizes for which latent rows can be expanded and attended as keys and values per head."""
    return (dtype == torch.bfloat16 and rank % 8 == 0 and rot % 8 == 0
            and pooled_tc_supported(heads, heads, key_dim, value_dim, page_size))


def _visible_pages(ctx, page_size: int, window: int) -> int:
    """Pages of rows that the step's requests see, each request's from a page of its own: what a
    step that runs kernel by kernel has, or the most that a captured shape can."""
    if ctx.extras.get("tile_provider") is None:
        total = 0
        for s in ctx.seqs:
            if s.num_tokens:
                first = max(0, s.start_pos - window + 1) // page_size if window else 0
                total += (s.start_pos + s.num_tokens - 1) // page_size - first + 1
        return total
    most = -(-ctx.max_context_len // page_size)
    if not window:
        return ctx.num_seqs * most
    return min(ctx.num_seqs * most, -(-ctx.num_tokens // page_size) + ctx.num_seqs * (-(-(window - 1) // page_size) + 2))


def latent_expand_pages(ctx, heads: int, key_dim: int, value_dim: int, rank: int, rot: int, page_size: int,
                        window: Optional[int]) -> int:
    """Pages to expand in this step, or 0 where attention over the rows themselves is estimated to
    be ahead.  The estimate counts the products over the latents at 95 TFLOP/s (``mma.sync``), the
    expansion at 1,000, attention over heads at 300 (tcgen05), and three trips of the expanded rows
    at 5 TB/s."""
    if LATENT_EXPAND is False or ctx.decode_only or ctx.max_tokens_per_seq < 16:
        return 0
    window = int(window or 0)
    pages = _visible_pages(ctx, page_size, window)
    per_row = heads * (key_dim + value_dim)
    rows = pages * page_size
    if rows * per_row * 2 > LATENT_EXPAND_BYTES:
        return 0
    if LATENT_EXPAND:
        return pages
    pairs = ctx.num_tokens * heads * 2.0 * _keys_seen(ctx, window)
    direct = pairs * (2 * rank + rot) / 95e6
    expanded = 15.0 + rows * 2.0 * (rank + rot) * per_row / 1e9 + rows * per_row * 6.0 / 5e6 \
        + pairs * (key_dim + value_dim) / 300e6
    return pages if expanded < direct else 0


def latent_attention_expanded(ctx, q: torch.Tensor, pages: torch.Tensor, block_table: torch.Tensor,
                              w_expand: torch.Tensor, most_pages: int, heads: int, key_dim: int, value_dim: int,
                              page_size: int, scale: float, window: Optional[int] = None,
                              options: Optional[AttentionOptions] = None) -> torch.Tensor:
    """``latent_attention`` of a step with portions by way of keys and values per head: the rows the
    step's requests see are copied out of their pages, ONE product with ``w_expand`` [heads * (key_dim +
    value_dim), row width] makes every head's keys and values of them, and the tcgen05 prefill kernel
    attends those.  ``q`` [T, heads * key_dim]; ``most_pages``: ``latent_expand_pages``; ``options``: a
    sink, a gate.  Rows of q may be strided.  Returns [T, heads * value_dim], gated."""
    _check(pages, "pages", torch.bfloat16, 4)
    _check(block_table, "block_table", torch.int32, 2)
    _check(w_expand, "w_expand", torch.bfloat16, 2)
    if not q.is_cuda or q.dim() != 2 or q.dtype != torch.bfloat16 or q.stride(1) != 1 or q.stride(0) % 8 \
            or q.data_ptr() % 16:
        raise KernelError("latent_attention_expanded: q must be bfloat16 rows at 16-byte boundaries")
    T, width = q.shape[0], pages.shape[3]
    columns = heads * (key_dim + value_dim)
    if tuple(w_expand.shape) != (columns, width) or pages.shape[1] != 1 or pages.shape[2] != page_size \
            or q.shape[1] < heads * key_dim:
        raise KernelError(f"latent_attention_expanded: q {tuple(q.shape)}, pages {tuple(pages.shape)} and w_expand "
                          f"{tuple(w_expand.shape)} do not fit {heads} heads of {key_dim} / {value_dim}")
    opt = options or _NO_OPTIONS
    rows = torch.empty((most_pages * page_size, width), dtype=torch.bfloat16, device=q.device)
    local = torch.empty_like(block_table)
    f = _fn("latent_attention", "hb_latent_gather",
            [c_void_p, c_int, c_void_p, c_int, c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_int, c_int, c_int, c_int,
             c_void_p])
    _run(f(_p(rows), most_pages, _p(local), local.shape[1], _p(pages), _p(block_table), block_table.shape[1],
           _p(ctx.cu_tokens), _p(ctx.start_pos), ctx.num_seqs, int(window or 0), page_size, width, _stream()),
         "latent_gather")
    kv = linear(rows, w_expand)
    out = torch.empty((T, heads * value_dim), dtype=torch.bfloat16, device=q.device)
    tiles = _step_tiles(ctx, 128, True, q.device)
    _scratch, _tickets, err = _gemm_workspace(q.device)
    f = _fn("attention_tc_pooled", "hb_attention_rows_prefill_tc",
            [c_void_p, c_int, c_void_p, c_int, c_void_p, c_int, ctypes.c_longlong, c_void_p, c_int, c_void_p, c_int,
             c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_float, c_void_p, c_int, c_void_p, c_void_p, c_int,
             c_int, c_void_p])
    _run(f(_p(out), out.stride(0), _p(q), q.stride(0), _p(kv), kv.stride(0), kv.shape[0], _p(local), local.shape[1],
           _p(tiles), tiles.shape[0], _p(ctx.cu_tokens), _p(ctx.start_pos), heads, key_dim, value_dim, page_size,
           int(window or 0), float(scale), _p(err), *_sized_option_args(opt, T, heads, q, value_dim), _stream()),
         "attention_rows_prefill_tc")
    return out


# ------------------------------------------------------------------ gated delta rule
def causal_conv_silu(ctx, x: torch.Tensor, channels: int, weight: torch.Tensor,
                     conv_state: torch.Tensor, bias: Optional[torch.Tensor] = None,
                     col0: int = 0) -> torch.Tensor:
    """silu of a short causal convolution over time, per channel, of the ``channels`` columns
    of ``x`` [T, ld] from column ``col0`` on; ``weight`` [channels, taps] float32 (last column:
    the current token), ``bias`` float32 [channels] or None.  ``conv_state`` [slots, channels *
    (taps - 1)] float32 (rows may be strided) holds every request's last taps - 1 inputs: read
    for the tokens before the step's first, and left holding the step's last ones."""
    _check(x, "x", None, 2)
    _check(weight, "weight", torch.float32, 2)
    taps = weight.shape[1]
    if weight.shape[0] != channels or x.shape[1] < col0 + channels or col0 < 0:
        raise KernelError(f"conv weight {tuple(weight.shape)} / x {tuple(x.shape)} do not fit {channels} "
                          f"channels from column {col0}")
    if bias is not None:
        _check(bias, "bias", torch.float32, 1)
        if bias.numel() != channels:
            raise KernelError(f"conv bias has {bias.numel()} entries for {channels} channels")
    if conv_state.dtype != torch.float32 or conv_state.dim() != 2 or conv_state.stride(1) != 1 \
            or conv_state.shape[1] != channels * (taps - 1):
        raise KernelError(f"conv state {tuple(conv_state.shape)} does not fit {channels} channels x {taps - 1}")
    T = x.shape[0]
    out = torch.empty((T, channels), dtype=x.dtype, device=x.device)
    f = _fn("delta_rule", "hb_causal_conv_silu",
            [c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_void_p, _LONG, c_void_p, c_void_p, c_void_p,
             c_int, c_int, c_int, c_int, c_int, c_void_p])
    _run(f(_p(out), _p(x) + col0 * x.element_size(), x.shape[1], _p(weight), _p(bias), _p(conv_state),
           conv_state.stride(0), _p(ctx.seq_of_token), _p(ctx.cu_tokens), _p(ctx.slots), T, ctx.num_seqs,
           channels, taps, _dt(x.dtype), _stream()), "causal_conv_silu")
    return out


def delta_rule(ctx, qkv: torch.Tensor, offsets, beta_raw: torch.Tensor, a_raw: torch.Tensor,
               a_log: torch.Tensor, dt_bias: torch.Tensor, state: torch.Tensor, heads: int,
               kv_heads: int, dk: int, dv: int) -> torch.Tensor:
    """The gated delta rule over the step's tokens, request by request, from the state each
    request's slot holds (``state`` [slots, heads * dk * dv] float32, rows may be strided;
    left updated).  ``qkv`` [T, .] holds q, k (kv_heads x dk) and v (heads x dv) at the column
    ``offsets`` (q, k, v); ``beta_raw`` [T, .] one column per head before the sigmoid;
    ``a_raw`` [T, heads * dk] before dt_bias and softplus (both views with contiguous rows).
    Returns o [T, heads * dv] float32."""
    _check(qkv, "qkv", None, 2)
    _check(a_log, "a_log", torch.float32, 1)
    _check(dt_bias, "dt_bias", torch.float32, 1)
    for name, t in (("beta_raw", beta_raw), ("a_raw", a_raw)):
        if t.dim() != 2 or t.stride(1) != 1 or t.dtype != qkv.dtype or t.shape[0] != qkv.shape[0]:
            raise KernelError(f"{name} {tuple(t.shape)} does not fit qkv {tuple(qkv.shape)}")
    if state.dtype != torch.float32 or state.dim() != 2 or state.stride(1) != 1 \
            or state.shape[1] != heads * dk * dv:
        raise KernelError(f"state {tuple(state.shape)} does not fit {heads} heads of {dk} x {dv}")
    if a_log.numel() != heads or dt_bias.numel() != heads * dk or beta_raw.shape[1] < heads \
            or a_raw.shape[1] < heads * dk or heads % kv_heads or dk > 256:
        raise KernelError("delta_rule: sizes do not fit (key size at most 256)")
    T = qkv.shape[0]
    o = torch.empty((T, heads * dv), dtype=torch.float32, device=qkv.device)
    # unit-norm k and q, decays and write strengths of every (token, head), float32
    scratch = torch.empty((T * heads * (3 * (-(-dk // 4) * 4) + 2),), dtype=torch.float32, device=qkv.device)
    f = _fn("delta_rule", "hb_delta_rule",
            [c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_void_p, c_int, c_void_p, c_int, c_void_p,
             c_void_p, c_void_p, _LONG, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_void_p])
    _run(f(_p(o), _p(scratch), _p(qkv), qkv.shape[1], offsets[0], offsets[1], offsets[2], _p(beta_raw),
           beta_raw.stride(0), _p(a_raw), a_raw.stride(0), _p(a_log), _p(dt_bias), _p(state),
           state.stride(0), _p(ctx.cu_tokens), _p(ctx.slots), T, ctx.num_seqs, heads, kv_heads, dk, dv,
           _dt(qkv.dtype), _stream()), "delta_rule")
    return o


def gated_rmsnorm(o: torch.Tensor, gate: torch.Tensor, weight: torch.Tensor, heads: int, dv: int,
                  eps: float) -> torch.Tensor:
    """o [T, heads * dv] float32 -> per head o / sqrt(mean(o^2) + eps) * weight[dv] *
    sigmoid(gate), in the dtype of ``gate`` ([T, heads * dv], rows may be strided)."""
    _check(o, "o", torch.float32, 2)
    _check(weight, "weight", torch.float32, 1)
    if gate.dim() != 2 or gate.stride(1) != 1 or tuple(gate.shape) != tuple(o.shape) \
            or o.shape[1] != heads * dv or weight.numel() != dv:
        raise KernelError(f"gated_rmsnorm: o {tuple(o.shape)}, gate {tuple(gate.shape)}, weight "
                          f"{weight.numel()} do not fit {heads} heads of {dv}")
    T = o.shape[0]
    out = torch.empty((T, heads * dv), dtype=gate.dtype, device=o.device)
    f = _fn("delta_rule", "hb_gated_rmsnorm",
            [c_void_p, c_void_p, c_void_p, c_int, c_void_p, c_int, c_int, c_int, c_float, c_int, c_void_p])
    _run(f(_p(out), _p(o), _p(gate), gate.stride(0), _p(weight), T, heads, dv, float(eps),
           _dt(gate.dtype), _stream()), "gated_rmsnorm")
    return out


#: requests with at most this many tokens in a step scan straight from the convolution's rows
SSM_DIRECT_MAX_TOKENS = 4


def ssm_scan(ctx, xbc: torch.Tensor, offsets, dt_raw: torch.Tensor, a_log: torch.Tensor,
             dt_bias: torch.Tensor, d_skip: torch.Tensor, state: torch.Tensor, heads: int, groups: int,
             n_state: int, head_dim: int) -> torch.Tensor:
    """The state-space recurrence over the step's tokens, request by request, from the state
    each request's slot holds (``state`` [slots, heads * n_state * head_dim] float32, rows may be
    strided; left updated): S <- a S + dt B x^T, y = S^T C + D x with dt = softplus(dt_raw +
    dt_bias) and a = exp(-exp(a_log) dt) per head.  ``xbc`` [T, .] holds x (heads x head_dim), B
    and C (groups x n_state each) at the column ``offsets`` (x, B, C); ``dt_raw`` [T, >= heads]
    a view with contiguous rows.  Returns y [T, heads * head_dim] float32."""
    _check(xbc, "xbc", None, 2)
    for name, v in (("a_log", a_log), ("dt_bias", dt_bias), ("d_skip", d_skip)):
        _check(v, name, torch.float32, 1)
        if v.numel() != heads:
            raise KernelError(f"{name} has {v.numel()} entries for {heads} heads")
    if dt_raw.dim() != 2 or dt_raw.stride(1) != 1 or dt_raw.dtype != xbc.dtype or dt_raw.shape[0] != xbc.shape[0] \
            or dt_raw.shape[1] < heads:
        raise KernelError(f"dt_raw {tuple(dt_raw.shape)} does not fit xbc {tuple(xbc.shape)}")
    if state.dtype != torch.float32 or state.dim() != 2 or state.stride(1) != 1 \
            or state.shape[1] != heads * n_state * head_dim:
        raise KernelError(f"state {tuple(state.shape)} does not fit {heads} heads of {n_state} x {head_dim}")
    x_off, b_off, c_off = offsets
    if heads % groups or n_state > 256 or max(x_off + heads * head_dim, b_off + groups * n_state,
                                              c_off + groups * n_state) > xbc.shape[1]:
        raise KernelError("ssm_scan: sizes do not fit (state size at most 256)")
    T = xbc.shape[0]
    y = torch.empty((T, heads * head_dim), dtype=torch.float32, device=xbc.device)
    if getattr(ctx, "max_tokens_per_seq", T) > SSM_DIRECT_MAX_TOKENS:
        # portions of prompts: the inputs as float32 rows first, then the scan that fetches them
        # a chunk ahead (the same arithmetic in the same order as the kernel below)
        sizes = (ctypes.c_int * 3)()
        f = _fn("ssm", "hb_ssm_stage_sizes", [c_int, c_int, c_int, c_int, c_void_p, c_void_p, c_void_p])
        base = ctypes.addressof(sizes)
        _run(f(heads, groups, n_state, head_dim, base, base + 4, base + 8), "ssm_stage_sizes")
        bc = torch.empty((T, sizes[0]), dtype=torch.float32, device=xbc.device)
        xs = torch.empty((T, sizes[1]), dtype=torch.float32, device=xbc.device)
        da = torch.empty((T, sizes[2]), dtype=torch.float32, device=xbc.device)
        f = _fn("ssm", "hb_ssm_scan_staged",
                [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_void_p, c_int,
                 c_void_p, c_void_p, c_void_p, c_void_p, _LONG, c_void_p, c_void_p, c_int, c_int, c_int, c_int,
                 c_int, c_int, c_int, c_void_p])
        _run(f(_p(y), _p(bc), _p(xs), _p(da), _p(xbc), xbc.shape[1], x_off, b_off, c_off, _p(dt_raw),
               dt_raw.stride(0), _p(a_log), _p(dt_bias), _p(d_skip), _p(state), state.stride(0),
               _p(ctx.cu_tokens), _p(ctx.slots), T, ctx.num_seqs, heads, groups, n_state, head_dim,
               _dt(xbc.dtype), _stream()), "ssm_scan_staged")
        return y
    f = _fn("ssm", "hb_ssm_scan",
            [c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_void_p, c_int, c_void_p, c_void_p, c_void_p,
             c_void_p, _LONG, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_void_p])
    _run(f(_p(y), _p(xbc), xbc.shape[1], x_off, b_off, c_off, _p(dt_raw), dt_raw.stride(0), _p(a_log),
           _p(dt_bias), _p(d_skip), _p(state), state.stride(0), _p(ctx.cu_tokens), _p(ctx.slots), T,
           ctx.num_seqs, heads, groups, n_state, head_dim, _dt(xbc.dtype), _stream()), "ssm_scan")
    return y


def gated_group_rmsnorm(y: torch.Tensor, z: torch.Tensor, weight: torch.Tensor, parts: int,
                        eps: float) -> torch.Tensor:
    """v = y * silu(z), then every one of the ``parts`` equal parts of a row divided by its own
    root mean square (eps inside the root), times ``weight``: the gate comes before the norm.
    ``y`` float32 [T, inner]; ``z`` [T, >= inner], a view whose rows may be strided; returns
    [T, inner] in z's dtype."""
    _check(y, "y", torch.float32, 2)
    _check(weight, "weight", torch.float32, 1)
    T, inner = y.shape
    if z.dim() != 2 or z.stride(1) != 1 or z.shape[0] != T or z.shape[1] < inner or weight.numel() != inner \
            or parts <= 0 or inner % parts or not z.is_cuda:
        raise KernelError(f"gated_group_rmsnorm: y {tuple(y.shape)}, z {tuple(z.shape)}, weight "
                          f"{weight.numel()}, {parts} parts do not fit")
    out = torch.empty((T, inner), dtype=z.dtype, device=y.device)
    f = _fn("ssm", "hb_gated_group_rmsnorm",
            [c_void_p, c_void_p, c_void_p, c_int, c_void_p, c_int, c_int, c_int, c_float, c_int, c_void_p])
    _run(f(_p(out), _p(y), _p(z), z.stride(0), _p(weight), T, inner, parts, float(eps), _dt(z.dtype),
           _stream()), "gated_group_rmsnorm")
    return out


# ------------------------------------------------------------------ linear attention, fixed decay
LINEAR_ATTENTION_ACTIVATIONS = {"none": 0, "silu": 1}
LINEAR_ATTENTION_NORMS = ("head", "row")
LINEAR_ATTENTION_GATES = {"silu": 0, "sigmoid": 1}
#: tokens a chunk of the chunked form
LINEAR_ATTENTION_CHUNK = 64
#: steps whose requests bring at most this many tokens each run token by token
LINEAR_ATTENTION_SCAN_TOKENS = 8


def decay_power_table(decay, device) -> torch.Tensor:
    """float32 [heads, chunk + 1]: every head's decay to the power 0 .. chunk, from float64."""
    d = torch.tensor([float(x) for x in decay], dtype=torch.float64)
    n = torch.arange(LINEAR_ATTENTION_CHUNK + 1, dtype=torch.float64)
    return (d[:, None] ** n[None, :]).float().to(device).contiguous()


def linear_attention(ctx, rows: torch.Tensor, offsets, state: torch.Tensor, decay_powers: torch.Tensor,
                     heads: int, dk: int, dv: int, out: torch.Tensor, *, cos=None, sin=None,
                     key_scale: float = 1.0, activation: str = "none", norm: str = "head",
                     norm_weight: Optional[torch.Tensor] = None, gate: str = "silu", eps: float = 1e-6,
                     factor: float = 1.0) -> None:
    """S <- a S + k v^T, o = S^T q per head over the step's tokens, request by request, from the
    state each request's slot holds (``state`` [slots, heads * dk * dv] float32, rows may be
    strided; left updated), then o / rms(o) (``norm`` "head": per head; "row": over all heads,
    times ``norm_weight``) times the gate times ``factor`` into ``out`` [T, heads * dv] (rows may
    be strided).  ``rows`` [T, .] holds q, k (heads x dk), v and the gate (heads x dv) at the
    column ``offsets``; q, k and v may pass silu (``activation``), q and k a rotation by
    ``cos`` / ``sin`` [T, rot / 2] of their first ``rot`` values in halves; k is multiplied by
    ``key_scale``.  ``decay_powers``: ``decay_power_table``.  All of it float32.

    Steps of few tokens a request run token by token, others in chunks of 64 tokens that are
    taken in parallel."""
    _check(rows, "rows", None, 2)
    T = rows.shape[0]
    _check(decay_powers, "decay_powers", torch.float32, 2)
    if tuple(decay_powers.shape) != (heads, LINEAR_ATTENTION_CHUNK + 1):
        raise KernelError(f"decay_powers {tuple(decay_powers.shape)} for {heads} heads")
    if state.dtype != torch.float32 or state.dim() != 2 or state.stride(1) != 1 \
            or state.shape[1] != heads * dk * dv or not state.is_cuda:
        raise KernelError(f"state {tuple(state.shape)} does not fit {heads} heads of {dk} x {dv}")
    if dk > 256 or dv > 256:
        raise KernelError(f"heads of {dk} x {dv} are not supported (at most 256)")
    q_off, k_off, v_off, g_off = (int(o) for o in offsets)
    if min(q_off, k_off, v_off, g_off) < 0 or max(q_off + heads * dk, k_off + heads * dk, v_off + heads * dv,
                                                   g_off + heads * dv) > rows.shape[1]:
        raise KernelError(f"rows of {rows.shape[1]} columns do not hold the columns {tuple(offsets)}")
    rot = 0
    if cos is not None:
        _check(cos, "cos", torch.float32, 2)
        _check(sin, "sin", torch.float32, 2)
        rot = 2 * cos.shape[1]
        if cos.shape != sin.shape or cos.shape[0] != T or rot > dk:
            raise KernelError(f"cos/sin tables {tuple(cos.shape)} do not fit {T} tokens of heads of {dk}")
    if (norm == "row") != (norm_weight is not None) or norm not in LINEAR_ATTENTION_NORMS:
        raise KernelError(f"norm {norm!r} and its weight do not go together")
    if norm_weight is not None:
        _check(norm_weight, "norm_weight", torch.float32, 1)
        if norm_weight.numel() != heads * dv:
            raise KernelError(f"norm weight has {norm_weight.numel()} entries for {heads * dv} columns")
    _check_out_rows(out, T, heads * dv, rows)
    act, gk = LINEAR_ATTENTION_ACTIVATIONS[activation], LINEAR_ATTENTION_GATES[gate]
    most = getattr(ctx, "max_tokens_per_seq", T)
    o = None
    if most > LINEAR_ATTENTION_SCAN_TOKENS:
        tiles = _step_tiles(ctx, LINEAR_ATTENTION_CHUNK, False, rows.device)
        n_tiles = tiles.shape[0]
        sums = torch.empty((n_tiles * heads * dk * dv,), dtype=torch.float32, device=rows.device)
        if norm == "row":
            o = torch.empty((T, heads * dv), dtype=torch.float32, device=rows.device)
        f = _fn("linear_attention", "hb_la_chunked",
                [c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_void_p, c_void_p,
                 c_int, c_int, c_float, c_void_p, _LONG, c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_int, c_int,
                 c_int, c_int, c_int, c_float, c_float, c_int, c_void_p])
        _run(f(_p(o), _p(out), out.stride(0), _p(sums), _p(rows), rows.shape[1], q_off, k_off, v_off, g_off,
               _p(cos), _p(sin), rot, act, float(key_scale), _p(state), state.stride(0), _p(decay_powers), _p(tiles),
               n_tiles, _p(ctx.cu_tokens), _p(ctx.slots), ctx.num_seqs, heads, dk, dv, gk, float(eps), float(factor),
               _dt(rows.dtype), _stream()), "linear_attention_chunked")
        if o is None:
            return
    else:
        fused = norm == "head" and dv <= 128
        if not fused:
            o = torch.empty((T, heads * dv), dtype=torch.float32, device=rows.device)
        f = _fn("linear_attention", "hb_la_scan",
                [c_void_p, c_void_p, c_int, c_void_p, c_int, c_int, c_int, c_int, c_int, c_void_p, c_void_p, c_int, c_int,
                 c_float, c_void_p, _LONG, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_int,
                 c_float, c_float, c_int, c_void_p])
        _run(f(_p(o), _p(out), out.stride(0), _p(rows), rows.shape[1], q_off, k_off, v_off, g_off, _p(cos), _p(sin),
               rot, act, float(key_scale), _p(state), state.stride(0), _p(decay_powers), _p(ctx.cu_tokens),
               _p(ctx.slots), T, ctx.num_seqs, heads, dk, dv, gk, float(eps), float(factor), _dt(rows.dtype),
               _stream()), "linear_attention_scan")
        if fused:
            return
    parts = heads if norm == "head" else 1
    _linear_gate_norm(out, o, rows, g_off, norm_weight, parts, heads * dv // parts, gate, eps, factor)


def _linear_gate_norm(out, o, rows, g_off, weight, parts, width, gate, eps, factor) -> None:
    """``out`` = factor * o / rms(o) (* weight) * gate: ``parts`` norms of ``width`` values a token,
    the gate's argument in the columns of ``rows`` from ``g_off`` on."""
    f = _fn("linear_attention", "hb_la_gate_norm",
            [c_void_p, c_int, c_void_p, c_void_p, c_int, c_void_p, c_int, c_int, c_int, c_int, c_float, c_float,
             c_int, c_void_p])
    _run(f(_p(out), out.stride(0), _p(o), _p(rows) + g_off * rows.element_size(), rows.shape[1], _p(weight),
           out.shape[0], parts, width, LINEAR_ATTENTION_GATES[gate], float(eps), float(factor), _dt(rows.dtype),
           _stream()), "linear_attention_gate_norm")


# ------------------------------------------------------------------ linear attention, decays per channel and token
def gated_linear_attention(ctx, rows: torch.Tensor, offsets, w2: torch.Tensor, bias: torch.Tensor, tau: float,
                           state: torch.Tensor, heads: int, dk: int, dv: int, norm_weight: torch.Tensor, eps: float,
                           out: torch.Tensor, q_scale: float = 1.0, factor: float = 1.0) -> None:
    """S <- diag(a) S + k v^T, o = S^T q per head over the step's tokens, request by request, from
    the state each request's slot holds (``state`` [slots, heads * dk * dv] float32, rows may be
    strided; left updated), with a decay per token and key channel, a = sigmoid(W2 x + bias)^(1 /
    ``tau``) (``w2`` [heads * dk, R] in the rows' dtype, ``bias`` float32), then o / rms(o) *
    ``norm_weight`` per head times silu(gate) times ``factor`` into ``out`` [T, heads * dv] (rows may
    be strided).  ``rows`` [T, .] holds q, k (heads x dk), v and the
    gate (heads x dv) and x (R columns) at the column ``offsets``; q is multiplied by ``q_scale``.
    Float32 in between.

    Steps of few tokens a request run token by token, others in chunks of 64 tokens that are
    taken in parallel."""
    _check(rows, "rows", None, 2)
    T = rows.shape[0]
    if state.dtype != torch.float32 or state.dim() != 2 or state.stride(1) != 1 \
            or state.shape[1] != heads * dk * dv or not state.is_cuda:
        raise KernelError(f"state {tuple(state.shape)} does not fit {heads} heads of {dk} x {dv}")
    if dk > 256 or dv > 256:
        raise KernelError(f"heads of {dk} x {dv} are not supported (at most 256)")
    _check(w2, "w2", rows.dtype, 2)
    _check(bias, "bias", torch.float32, 1)
    _check(norm_weight, "norm_weight", torch.float32, 1)
    rank = w2.shape[1]
    if w2.shape[0] != heads * dk or bias.numel() != heads * dk or norm_weight.numel() != dv or rank > 256:
        raise KernelError(f"w2 {tuple(w2.shape)}, bias {bias.numel()} and norm weight {norm_weight.numel()} do not fit "
                          f"{heads} heads of {dk} x {dv} (a rank of at most 256)")
    offs = tuple(int(o) for o in offsets)
    for o, n in zip(offs, (heads * dk, heads * dk, heads * dv, heads * dv, rank)):
        if o < 0 or o + n > rows.shape[1]:
            raise KernelError(f"rows of {rows.shape[1]} columns do not hold the columns {offs}")
    if not tau > 0:
        raise KernelError(f"tau {tau} must be positive")
    _check_out_rows(out, T, heads * dv, rows)
    f32 = dict(dtype=torch.float32, device=rows.device)
    most = getattr(ctx, "max_tokens_per_seq", T)
    if most > LINEAR_ATTENTION_SCAN_TOKENS:
        tiles = _step_tiles(ctx, LINEAR_ATTENTION_CHUNK, False, rows.device)
        n = tiles.shape[0]
        q, k = torch.empty((T, heads, dk), **f32), torch.empty((T, heads, dk), **f32)
        decays = torch.empty((n, heads, 5, dk), **f32)
        diag = torch.empty((n, heads, LINEAR_ATTENTION_CHUNK, 16), **f32)
        sums = torch.empty((n, heads, dk, dv), **f32)
        f = _fn("gated_linear_attention", "hb_gla_chunked",
                [c_void_p, c_int] + [c_void_p] * 6 + [c_int] * 6 + [c_void_p, c_void_p, c_int, c_float, c_float, c_void_p,
                 _LONG, c_void_p, c_int, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_void_p, c_float, c_float, c_int,
                 c_void_p])
        _run(f(_p(out), out.stride(0), _p(q), _p(k), _p(decays), _p(diag), _p(sums), _p(rows), rows.shape[1], *offs,
               _p(w2), _p(bias), rank, 1.0 / float(tau), float(q_scale), _p(state), state.stride(0), _p(tiles), n,
               _p(ctx.cu_tokens), _p(ctx.slots), ctx.num_seqs, heads, dk, dv, _p(norm_weight), float(eps),
               float(factor), _dt(rows.dtype), _stream()), "gated_linear_attention_chunked")
        return
    o = torch.empty((T, heads * dv), **f32) if dv > 128 else None
    f = _fn("gated_linear_attention", "hb_gla_scan",
            [c_void_p, c_void_p, c_int, c_void_p] + [c_int] * 6 + [c_void_p, c_void_p, c_int, c_float, c_float, c_void_p,
             _LONG, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_void_p, c_float, c_float, c_int, c_void_p])
    _run(f(_p(o), _p(out), out.stride(0), _p(rows), rows.shape[1], *offs, _p(w2), _p(bias), rank, 1.0 / float(tau),
           float(q_scale), _p(state), state.stride(0), _p(ctx.cu_tokens), _p(ctx.slots), T, ctx.num_seqs, heads, dk, dv,
           _p(norm_weight), float(eps), float(factor), _dt(rows.dtype), _stream()), "gated_linear_attention_scan")
    if o is not None:
        _linear_gate_norm(out, o, rows, offs[3], norm_weight, heads, dv, "silu", eps, factor)


# ------------------------------------------------------------------ window attention with pooled blocks
def pooled_attention_libraries(dtype: torch.dtype, num_heads: int, num_kv_heads: int, head_dim: int,
                               value_dim: int):
    """Libraries window attention with pooled blocks runs on at these sizes."""
    names = ["pooled_window"]
    decode = dtype == torch.bfloat16 and pooled_decode_supported(num_heads, num_kv_heads, head_dim, value_dim)
    portions = dtype == torch.bfloat16 and pooled_tc_supported(num_heads, num_kv_heads, head_dim, value_dim, 16)
    if decode:
        names.append("attention_pooled")
    if portions:
        names.append("attention_tc_pooled")
    if not (decode and portions):
        names.append("attention_generic")
    return tuple(names)


def pooled_decode_supported(num_heads: int, num_kv_heads: int, head_dim: int, value_dim: int) -> bool:
    """Sizes the split-context decode kernel with pooled blocks takes."""
    return (head_dim % 8 == 0 and value_dim % 8 == 0 and max(head_dim, value_dim) <= 256
            and num_heads % num_kv_heads == 0 and num_heads // num_kv_heads <= 16)


def pooled_tc_supported(num_heads: int, num_kv_heads: int, head_dim: int, value_dim: int, page_size: int) -> bool:
    """Sizes the tcgen05 prefill kernel with pooled blocks takes: Q, K, V and P tiles of 256-wide keys
    AND values do not fit shared memory together."""
    return (head_dim % 8 == 0 and value_dim % 8 == 0 and max(head_dim, value_dim) <= 256
            and min(head_dim, value_dim) <= 128 and num_heads % num_kv_heads == 0
            and num_heads // num_kv_heads <= 128 and page_size >= 8 and page_size % 8 == 0 and 128 % page_size == 0)


def _check_pages(cache, like: torch.Tensor, num_kv_heads: int, head_dim: int, value_dim: int) -> None:
    for name, pages, d in (("k_pages", cache.k_pages, head_dim), ("v_pages", cache.v_pages, value_dim)):
        _check(pages, name, like.dtype, 4)
        if tuple(pages.shape[1:]) != (num_kv_heads, cache.page_size, d):
            raise KernelError(f"{name} has shape {tuple(pages.shape)}, expected "
                              f"[pages, {num_kv_heads}, {cache.page_size}, {d}]")


def conv_norm_rotate_write(ctx, rows: torch.Tensor, col0: int, conv: Optional[torch.Tensor],
                           state: Optional[torch.Tensor], q_weight: torch.Tensor, k_weight: torch.Tensor,
                           eps: float, cos: torch.Tensor, sin: torch.Tensor, cache, num_heads: int,
                           num_kv_heads: int, head_dim: int, value_dim: int) -> torch.Tensor:
    """From the columns q | k | v of ``rows`` [T, .] at ``col0``: a short causal convolution per
    channel (``conv`` float32 [channels, taps], last column the current token's; None: none; the
    inputs before the step's first token come from ``state`` [slots, channels * (taps - 1)]
    float32, which is left holding the last ones), an RMS norm per q and k head with a weight,
    the rotation of q's and k's first values by ``cos`` / ``sin`` [T, rot / 2] in halves.  k and v
    go to the cache's pages, q is returned [T, heads * head_dim].  Float32 in between."""
    _check(rows, "rows", None, 2)
    T = rows.shape[0]
    channels = num_heads * head_dim + num_kv_heads * (head_dim + value_dim)
    if col0 < 0 or rows.shape[1] < col0 + channels:
        raise KernelError(f"rows of {rows.shape[1]} columns do not hold {channels} from column {col0}")
    taps = 1
    if conv is not None:
        _check(conv, "conv", torch.float32, 2)
        taps = conv.shape[1]
        if conv.shape[0] != channels or taps < 1:
            raise KernelError(f"conv weight {tuple(conv.shape)} does not fit {channels} channels")
        if taps > 1 and (state is None or state.dtype != torch.float32 or state.dim() != 2 or state.stride(1) != 1
                         or state.shape[1] != channels * (taps - 1)):
            raise KernelError(f"the convolution's state does not fit {channels} channels x {taps - 1}")
    for name, w in (("q_weight", q_weight), ("k_weight", k_weight)):
        _check(w, name, torch.float32, 1)
        if w.numel() != head_dim:
            raise KernelError(f"{name} has {w.numel()} entries for heads of {head_dim}")
    _check(cos, "cos", torch.float32, 2)
    _check(sin, "sin", torch.float32, 2)
    rot = 2 * cos.shape[1]
    if cos.shape != sin.shape or cos.shape[0] != T or rot > head_dim:
        raise KernelError(f"cos/sin tables {tuple(cos.shape)} do not fit {T} tokens of heads of {head_dim}")
    _check_pages(cache, rows, num_kv_heads, head_dim, value_dim)
    table = ctx.block_tables[cache.group]
    _check(table, "block_table", torch.int32, 2)
    q = torch.empty((T, num_heads * head_dim), dtype=rows.dtype, device=rows.device)
    moves = taps > 1
    f = _fn("pooled_window", "hb_conv_norm_rotate_write",
            [c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_void_p, c_void_p, _LONG, c_int, c_void_p, c_void_p,
             c_float, c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int,
             c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_void_p])
    _run(f(_p(q), _p(cache.k_pages) if cache.write else 0, _p(cache.v_pages) if cache.write else 0,
           _p(rows) + col0 * rows.element_size(), rows.shape[1], _p(conv), _p(state) if moves else 0,
           state.stride(0) if moves else 0, taps, _p(q_weight), _p(k_weight), float(eps), _p(cos), _p(sin), rot,
           _p(ctx.positions), _p(ctx.seq_of_token), _p(ctx.cu_tokens), _p(ctx.slots), _p(table), table.shape[1], T,
           ctx.num_seqs, num_heads, num_kv_heads, head_dim, value_dim, cache.page_size,
           1 if ctx.decode_only else 0, _dt(rows.dtype), _stream()), "conv_norm_rotate_write")
    return q


def pool_blocks(ctx, cache, pool: int) -> None:
    """For every token of the step that ends a whole block of ``pool`` tokens of its request: the
    means of the block's keys and values, as the pages hold them, into the pooled pages."""
    pooled = cache.pooled
    G, hd = cache.k_pages.shape[1], cache.k_pages.shape[3]
    vd = cache.v_pages.shape[3]
    _check_pages(cache, cache.k_pages, G, hd, vd)
    _check_pages(pooled, cache.k_pages, G, hd, vd)
    table, ptable = ctx.block_tables[cache.group], ctx.block_tables[pooled.group]
    f = _fn("pooled_window", "hb_pool_blocks",
            [c_void_p, c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_int,
             c_int, c_int, c_int, c_int, c_int, c_int, c_void_p])
    _run(f(_p(pooled.k_pages), _p(pooled.v_pages), _p(ptable), ptable.shape[1], _p(cache.k_pages), _p(cache.v_pages),
           _p(table), table.shape[1], _p(ctx.positions), _p(ctx.seq_of_token), ctx.num_tokens, G, hd, vd,
           cache.page_size, int(pool), _dt(cache.k_pages.dtype), _stream()), "pool_blocks")


def pooled_attention(ctx, q: torch.Tensor, cache, num_heads: int, num_kv_heads: int, head_dim: int,
                     value_dim: int, window: int, pool: int, scale: float, out: torch.Tensor,
                     factor: float = 1.0) -> None:
    """Attention of the step's tokens over the last ``window`` tokens of their requests and, with
    ``pool``, one key and value for every whole block of ``pool`` tokens that lies before the
    window, under one softmax; ``factor`` times the result into ``out`` [T, heads * value_dim]
    (rows may be strided)."""
    ptable = ctx.block_tables[cache.pooled.group] if pool else None
    table = ctx.block_tables[cache.group]
    if q.dtype == torch.bfloat16 and POOLED_ATTENTION_TILED and out.stride(0) % 8 == 0 and out.data_ptr() % 16 == 0:
        if ctx.decode_only and pooled_decode_supported(num_heads, num_kv_heads, head_dim, value_dim):
            splits = ctx.extras.get("pooled_splits")
            if splits is None:
                keys = window + (ctx.max_context_len // pool if pool else 0)
                splits = decode_splits(ctx.num_seqs, num_kv_heads, min(keys, max(1, ctx.max_context_len)),
                                       max(head_dim, value_dim))
            _pooled_decode(ctx, q, cache, table, ptable, num_heads, num_kv_heads, head_dim, value_dim, window, pool,
                           scale, out, factor, int(splits))
            return
        if pooled_tc_supported(num_heads, num_kv_heads, head_dim, value_dim, cache.page_size):
            _pooled_prefill_tc(ctx, q, cache, table, ptable, num_heads, num_kv_heads, head_dim, value_dim, window,
                               pool, scale, out, factor)
            return
    pooled = (cache.pooled.k_pages, cache.pooled.v_pages, ptable, pool) if pool else None
    options = None if value_dim == head_dim else AttentionOptions(value_dim=value_dim)
    attention_generic(q, cache.k_pages, cache.v_pages, table, ctx.seq_of_token, ctx.positions, num_heads, num_kv_heads,
                      head_dim, cache.page_size, window, scale, options, pooled=pooled, out=out, factor=factor)


#: window attention with pooled blocks on the tensor-core kernels where the sizes allow
POOLED_ATTENTION_TILED = True
_pooled_clusters = {}


def pooled_cluster_capacity(head_dim: int, value_dim: int, size: int) -> int:
    """Clusters of ``size`` blocks of the decode kernel with pooled blocks that are resident at once."""
    key = (-(-head_dim // 64), -(-value_dim // 64), size)
    if key not in _pooled_clusters:
        f = _fn("attention_pooled", "hb_attention_pooled_max_clusters", [c_int, c_int, c_int])
        _pooled_clusters[key] = max(0, int(f(head_dim, value_dim, size)))
    return _pooled_clusters[key]


def _pooled_args(q, cache, table, ptable, num_kv_heads, head_dim, value_dim, window, pool):
    _check(q, "q", torch.bfloat16, 2)
    _check_pages(cache, q, num_kv_heads, head_dim, value_dim)
    _check(table, "block_table", torch.int32, 2)
    if not pool:
        return (0, 0, 0, 0, 0, 0)
    pk, pv, pt, pool = _check_pooled((cache.pooled.k_pages, cache.pooled.v_pages, ptable, pool), q, num_kv_heads,
                                     cache.page_size, head_dim, value_dim, window)
    return (_p(pk), _p(pv), pk.shape[0], _p(pt), pt.shape[1], pool)


def _sized_option_args(options: AttentionOptions, tokens: int, num_heads: int, like: torch.Tensor, value_dim: int):
    """Sink and gate as the kernels for sizes of their own take them."""
    options.check(tokens, num_heads, like, value_dim)
    return (int(options.sink), _p(options.sink_values), _p(options.gate), options.gate_stride,
            1 if options.gate_wide else 0)


def _pooled_decode(ctx, q, cache, table, ptable, num_heads, num_kv_heads, head_dim, value_dim, window, pool, scale,
                   out, factor, n_splits, options: AttentionOptions = _NO_OPTIONS, qk_norm=None,
                   write_cache: bool = False) -> None:
    """Token i is the one new token of request i; the context in ``n_splits`` slices.
    ``write_cache``: the rows of q hold the token's k and v behind the queries, and the kernel
    stores them; ``qk_norm`` = (q weight, k weight, eps): q (and that k) still lacks its norm."""
    S = q.shape[0]
    pk, pv, _n, pt, pstride, pool = _pooled_args(q, cache, table, ptable, num_kv_heads, head_dim, value_dim, window, pool)
    _check_out_rows(out, S, num_heads * value_dim, q)
    columns = num_heads * head_dim + (num_kv_heads * (head_dim + value_dim) if write_cache else 0)
    if q.shape[1] < columns or table.shape[0] != S:
        raise KernelError(f"decode attention needs one token per request and {num_heads} heads of {head_dim}")
    wq, wk, eps = qk_norm if qk_norm is not None else (None, None, 0.0)
    for name, w in (("q norm weight", wq), ("k norm weight", wk)):
        if w is not None:
            _check(w, name, torch.float32, 1)
            if w.numel() != head_dim:
                raise KernelError(f"{name} has {w.numel()} entries for heads of {head_dim}")
    part_o = part_ml = None
    one_round = n_splits <= 8 and S * num_kv_heads <= pooled_cluster_capacity(head_dim, value_dim, n_splits)
    if n_splits > 8 or (n_splits > 1 and not (ATTENTION_CLUSTER_MERGE and one_round)):
        part_o = torch.empty((S, num_heads, n_splits, value_dim), dtype=torch.float32, device=q.device)
        part_ml = torch.empty((S, num_heads, n_splits, 2), dtype=torch.float32, device=q.device)
    f = _fn("attention_pooled", "hb_attention_pooled_decode",
            [c_void_p, c_int, c_float, c_void_p, c_void_p, c_void_p, c_int, c_void_p, c_void_p, c_void_p, c_int,
             c_void_p, c_void_p, c_void_p, c_int, c_int, c_void_p, c_int, c_int, c_int, c_int, c_int, c_int, c_int,
             c_float, c_int, c_int, c_void_p, c_void_p, c_int, c_int, c_int, c_void_p, c_void_p, c_float, c_void_p])
    _run(f(_p(out), out.stride(0), float(factor), _p(part_o), _p(part_ml), _p(q), q.stride(0), _p(cache.k_pages),
           _p(cache.v_pages), _p(table), table.shape[1], pk, pv, pt, pstride, pool, _p(ctx.positions), S, num_heads,
           num_kv_heads, head_dim, value_dim, cache.page_size, int(window), float(scale), n_splits,
           *_sized_option_args(options, S, num_heads, q, value_dim), 1 if write_cache else 0, _p(wq), _p(wk),
           float(eps), _stream()), "attention_pooled_decode")


def _pooled_prefill_tc(ctx, q, cache, table, ptable, num_heads, num_kv_heads, head_dim, value_dim, window, pool,
                       scale, out, factor, options: AttentionOptions = _NO_OPTIONS) -> None:
    pk, pv, pn, pt, pstride, pool = _pooled_args(q, cache, table, ptable, num_kv_heads, head_dim, value_dim, window, pool)
    _check_out_rows(out, q.shape[0], num_heads * value_dim, q)
    if q.shape[1] < num_heads * head_dim:
        raise KernelError(f"q has {q.shape[1]} columns for {num_heads} heads of {head_dim}")
    tiles = _step_tiles(ctx, 128 // (num_heads // num_kv_heads), True, q.device)
    _scratch, _tickets, err = _gemm_workspace(q.device)
    f = _fn("attention_tc_pooled", "hb_attention_pooled_prefill_tc",
            [c_void_p, c_int, c_float, c_void_p, c_int, c_void_p, c_void_p, ctypes.c_longlong, c_void_p, c_int, c_void_p,
             c_void_p, ctypes.c_longlong, c_void_p, c_int, c_int, c_void_p, c_int, c_void_p, c_void_p, c_int, c_int,
             c_int, c_int, c_int, c_int, c_float, c_void_p, c_int, c_void_p, c_void_p, c_int, c_int, c_void_p])
    _run(f(_p(out), out.stride(0), float(factor), _p(q), q.stride(0), _p(cache.k_pages), _p(cache.v_pages),
           cache.k_pages.shape[0], _p(table), table.shape[1], pk, pv, pn, pt, pstride, pool, _p(tiles), tiles.shape[0],
           _p(ctx.cu_tokens), _p(ctx.start_pos), num_heads, num_kv_heads, head_dim, value_dim, cache.page_size,
           int(window), float(scale), _p(err), *_sized_option_args(options, q.shape[0], num_heads, q, value_dim),
           _stream()), "attention_pooled_prefill_tc")


# ------------------------------------------------------------------ routed experts
ROUTER_KINDS = {"sigmoid": 0, "softmax": 1, "top_softmax": 2}


def moe_topk(logits: torch.Tensor, top: int, kind: str = "sigmoid",
             correction: Optional[torch.Tensor] = None, bias: Optional[torch.Tensor] = None,
             groups=None, normalize: bool = False, scale: float = 1.0):
    """(expert ids int32 [T, top], weights float32 [T, top]) from float32 router ``logits``
    [T, outputs] (+ ``bias``, float32 [outputs], added first).  Kinds "sigmoid" and "softmax":
    scores s = sigmoid(z), or softmax(z) over all outputs; the ``top`` largest s + correction
    (float32 [outputs]; None: s alone) are chosen, lower index on a tie, largest first; the
    weight is s itself.  Kind "top_softmax": the ``top`` largest logits are chosen and the
    weights are the softmax over the chosen logits alone.

    ``groups`` = (count, keep): the router outputs form ``count`` equal runs of neighbours; a
    run scores its largest choice value, and only outputs of the ``keep`` best runs (the lower
    index among equals) can be chosen (rows of at most 256 outputs).  ``normalize``: the weights
    are the chosen scores divided by their sum (+ 1e-20).  ``scale`` multiplies every weight."""
    _check(logits, "logits", torch.float32, 2)
    T, E = logits.shape
    if kind not in ROUTER_KINDS:
        raise KernelError(f"router kind {kind!r} is not one of {sorted(ROUTER_KINDS)}")
    if not 0 < top <= min(E, 16):
        raise KernelError(f"top {top} of {E} experts is not supported (1..16)")
    for name, v in (("correction", correction), ("bias", bias)):
        if v is not None:
            _check(v, name, torch.float32, 1)
            if v.numel() != E:
                raise KernelError(f"{name} has {v.numel()} entries for {E} router outputs")
    count, keep = (int(groups[0]), int(groups[1])) if groups else (1, 1)
    if count > 1 and (E % count or not 0 < keep <= count or top > keep * (E // count) or E > 256):
        raise KernelError(f"{count} groups of which {keep} stay do not fit top {top} of {E} router outputs "
                          "(equal groups, at most 256 outputs)")
    if normalize and kind == "top_softmax":
        raise KernelError("a softmax over the chosen logits is normalised already")
    ids = torch.empty((T, top), dtype=torch.int32, device=logits.device)
    weights = torch.empty((T, top), dtype=torch.float32, device=logits.device)
    biased = torch.empty_like(logits) if bias is not None and E > 256 else None
    f = _fn("moe", "hb_moe_topk", [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int,
                                   c_int, c_int, c_int, c_int, c_int, c_float, c_void_p])
    _run(f(_p(ids), _p(weights), _p(logits), _p(correction), _p(bias), _p(biased), T, E, top,
           ROUTER_KINDS[kind], count, keep, 1 if normalize else 0, float(scale), _stream()), "moe_topk")
    return ids, weights


#: bfloat16 steps of at least this many tokens run the experts as two grouped matrix products
#: of the library (tensor cores; rows sorted by expert on the device, no host round trip, so
#: the step stays capturable): every step, since with one block a (token, choice) pair the
#: streaming kernel took 2 ms a layer for 8 tokens at 16 experts of 2,048 x 1,024 where the
#: grouped path takes 0.1.  Float32, and inner sizes or widths that are no multiple of 8,
#: stream every pair's expert rows.
MOE_GROUPED_MIN_TOKENS = 1
#: gates an expert may have (codes of ``GLU_KINDS``)
MOE_GATES = ("silu", "clamped_swish")
#: activations of an expert WITHOUT a gate, down(act(up x)), whose first matrix has ff rows
MOE_PLAIN_ACTS = ("relu2",)
_MOE_ACT_CODES = {"silu": 0, "clamped_swish": 2, "relu2": 3}


def moe_experts_grouped(h: torch.Tensor, ids: torch.Tensor, weights: torch.Tensor,
                        w_gate_up: torch.Tensor, w_down: torch.Tensor, limit: float,
                        gate: str = "clamped_swish", weight_on: str = "input", identity: int = 0,
                        base: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``moe_experts`` for many tokens: sort the pairs by expert, (scale and) scatter the rows,
    one grouped product for gate|up, the gate, one for down, and a gather that adds a token's
    choices in their order (times their weights where those belong on the output).  Pairs of
    the experts without tensors sort behind all others: the products leave their rows alone
    and the gather takes the token's own row for them."""
    T, width = h.shape
    E, two_ff, _ = w_gate_up.shape
    top = ids.shape[1]
    pairs = T * top
    on_output = weight_on == "output"
    ends = torch.empty((E + identity,), dtype=torch.int32, device=h.device)
    place = torch.empty((pairs,), dtype=torch.int32, device=h.device)
    f = _fn("moe", "hb_moe_sort", [c_void_p, c_void_p, c_void_p, c_int, c_int, c_void_p])
    _run(f(_p(ends), _p(place), _p(ids), pairs, E + identity, _stream()), "moe_sort")
    rows = torch.empty((pairs, width), dtype=h.dtype, device=h.device)
    f = _fn("moe", "hb_moe_scatter_rows",
            [c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_void_p])
    _run(f(_p(rows), _p(h), _p(place), 0 if on_output else _p(weights), T, top, width, _dt(h.dtype),
           _stream()), "moe_scatter_rows")
    offs = ends[:E] if identity else ends
    gate_up = torch._grouped_mm(rows, w_gate_up.transpose(1, 2), offs=offs)
    y = unary_act(gate_up, gate) if gate in MOE_PLAIN_ACTS else glu_act(gate_up, gate, limit)
    down = torch._grouped_mm(y, w_down.transpose(1, 2), offs=offs)
    out = torch.empty((T, width), dtype=h.dtype, device=h.device)
    f = _fn("moe", "hb_moe_gather_sum",
            [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int,
             c_int, c_int, c_void_p])
    _run(f(_p(out), _p(down), _p(place), _p(ids) if identity else 0, _p(weights) if on_output else 0,
           _p(h) if identity else 0, _p(base), E, T, top, width, _dt(h.dtype), _stream()), "moe_gather_sum")
    return out


def moe_experts(h: torch.Tensor, ids: torch.Tensor, weights: torch.Tensor, w_gate_up: torch.Tensor,
                w_down: torch.Tensor, limit: float = 0.0, gate: str = "clamped_swish",
                weight_on: str = "input", identity: int = 0,
                base: Optional[torch.Tensor] = None) -> torch.Tensor:
    """The sum over a token's chosen experts: of expert(weight * h) with ``weight_on`` =
    "input", of weight * expert(h) with "output".  ``w_gate_up`` [experts, 2 ff, width] (gate
    rows, then up rows), ``w_down`` [experts, width, ff]; ``gate``: "clamped_swish" with its
    ``limit`` or "silu" (``glu_act``), or "relu2" for experts without a gate, down(relu(up x)^2),
    whose first matrix is [experts, ff, width].  Expert ids from ``experts`` up to ``experts + identity``
    name experts without tensors, whose output is their input (times the weight).  ``base``
    ([T, width]) is added to the sum.  Returns [T, width] in h's dtype."""
    _check(h, "h", None, 2)
    _check(ids, "ids", torch.int32, 2)
    _check(weights, "weights", torch.float32, 2)
    _check(w_gate_up, "w_gate_up", h.dtype, 3)
    _check(w_down, "w_down", h.dtype, 3)
    T, width = h.shape
    E, two_ff, w2 = w_gate_up.shape
    ff = two_ff if gate in MOE_PLAIN_ACTS else two_ff // 2
    top = ids.shape[1]
    if w2 != width or tuple(w_down.shape) != (E, width, ff) or tuple(ids.shape) != (T, top) \
            or ids.shape != weights.shape:
        raise KernelError("moe_experts: shapes do not fit")
    if gate not in MOE_GATES + MOE_PLAIN_ACTS or weight_on not in ("input", "output") or identity < 0:
        raise KernelError(f"moe_experts: gate {gate!r} / weight_on {weight_on!r} / identity {identity}")
    if base is not None:
        _check(base, "base", h.dtype, 2)
        if tuple(base.shape) != (T, width):
            raise KernelError("moe_experts: base does not fit")
    if h.dtype == torch.bfloat16 and T >= MOE_GROUPED_MIN_TOKENS and width % 8 == 0 and ff % 8 == 0 \
            and hasattr(torch, "_grouped_mm"):
        return moe_experts_grouped(h, ids, weights, w_gate_up, w_down, limit, gate, weight_on, identity, base)
    partial = torch.empty((T * top, width), dtype=torch.float32, device=h.device)
    f = _fn("moe", "hb_moe_expert_rows",
            [c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int,
             c_float, c_int, c_int, c_int, c_int, c_void_p])
    _run(f(_p(partial), _p(h), _p(w_gate_up), _p(w_down), _p(ids), _p(weights), T, top, width, ff,
           float(limit), _MOE_ACT_CODES[gate], 1 if weight_on == "output" else 0, E, _dt(h.dtype), _stream()),
         "moe_expert_rows")
    out = torch.empty((T, width), dtype=h.dtype, device=h.device)
    f = _fn("moe", "hb_moe_combine", [c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_void_p])
    _run(f(_p(out), _p(partial), _p(base), T, width, top, _dt(h.dtype), _stream()), "moe_combine")
    return out
