"""Python faces of the hand-written CUDA kernels.

Each function checks devices, dtypes, shapes and contiguity, then calls the `extern "C"` launcher
through ctypes on the current CUDA stream.  There is no CPU path and no library fallback: on a
machine without the built extension or without a GPU these functions raise.
"""
from __future__ import annotations

import ctypes
import functools
import math
import os
from typing import Optional, Tuple

import torch

from .build import BuildError, build, library

F32, BF16 = 0, 1


class KernelError(RuntimeError):
    pass


def dtype_code(dt: torch.dtype) -> int:
    if dt == torch.float32:
        return F32
    if dt == torch.bfloat16:
        return BF16
    raise KernelError(f"kernels take float32 or bfloat16 operands, not {dt}")


def _ptr(t: Optional[torch.Tensor]):
    return ctypes.c_void_p(0 if t is None else t.data_ptr())


_raw_stream = getattr(torch._C, "_cuda_getCurrentRawStream", None)


def _stream():
    """The current stream's handle (the short way where this torch has it: a launch costs the host a few microseconds)."""
    if _raw_stream is not None:
        return ctypes.c_void_p(_raw_stream(torch.cuda.current_device()))
    return ctypes.c_void_p(torch.cuda.current_stream().cuda_stream)


def _need(t: torch.Tensor, name: str, dtype=None, shape=None):
    if not t.is_cuda:
        raise KernelError(f"{name} is on {t.device}; the kernels run on a CUDA device only")
    if not t.is_contiguous():
        raise KernelError(f"{name} is not contiguous")
    if dtype is not None and t.dtype != dtype:
        raise KernelError(f"{name} has dtype {t.dtype}, expected {dtype}")
    if shape is not None and tuple(t.shape) != tuple(shape):
        raise KernelError(f"{name} has shape {tuple(t.shape)}, expected {tuple(shape)}")


# kernels launched per exported function (for launch accounting in benchmarks)
_LAUNCHES = {"q6k_gated_delta": 1, "q6k_delta_channel": 1, "q6k_attention_flex_mma": 2, "q6k_selective_scan": 1, "q6k_moe_permute": 3, "q6k_moe_plan": 3, "q6k_gemm_tc": 1, "q6k_attention_mma": 2, "q6k_argmax": 2, "q6k_gemm_tc_pairs_scratch": 0}
launch_count = 0


_functions = {}

# Where a step's time goes, without a profiler (the reference times its forward pass op by op the same way and can
# synchronise after every op: crates/engine/src/profile.rs:1-55, crates/engine/src/flint.rs:685-697).
# profile_begin() makes every launcher call stand between two CUDA events; profile_end() adds them up per (tag, launcher).
# Parts name what they are about to launch by setting ops.current_tag (a plain attribute: nothing is paid when no one
# is profiling).  Steps replayed from a CUDA graph run no Python and are not seen: profile eager steps.
# The environment variable Q6K_SYNC=op synchronises after every launcher call and raises where a kernel failed.
current_tag = ""
_profile = None
_sync_each = os.environ.get("Q6K_SYNC", "") == "op"


def profile_begin() -> None:
    global _profile
    _profile = []


def profile_end():
    """{(tag, launcher): (calls, milliseconds)} since profile_begin(), in the order of first use (synchronises)."""
    global _profile
    records, _profile = _profile or [], None
    torch.cuda.synchronize()
    out = {}
    for key, e0, e1 in records:
        calls, ms = out.get(key, (0, 0.0))
        out[key] = (calls + 1, ms + e0.elapsed_time(e1))
    return out


def _call(fn_name: str, *args):
    global launch_count
    launch_count += _LAUNCHES.get(fn_name, 1)
    fn = _functions.get(fn_name)
    if fn is None:
        fn = _functions[fn_name] = getattr(library(), fn_name)
        fn.restype = ctypes.c_int
    if _profile is not None:
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        rc = fn(*args)
        e1.record()
        _profile.append(((current_tag, fn_name), e0, e1))
    else:
        rc = fn(*args)
    if rc != 0:
        lib = library()
        lib.q6k_last_error.restype = ctypes.c_char_p
        raise KernelError(lib.q6k_last_error().decode())
    if _sync_each:
        torch.cuda.synchronize()
        status = tc_status()
        if status:
            raise KernelError(f"{fn_name} ({current_tag}): a bounded wait ran out inside a kernel (status {status})")


_i = ctypes.c_int
_f = ctypes.c_float
_ll = ctypes.c_longlong


# --------------------------------------------------------------------------- elementwise
def embed(tokens: torch.Tensor, table: torch.Tensor, out: Optional[torch.Tensor] = None, fed: Optional[torch.Tensor] = None,
          scale: float = 1.0, copy: Optional[torch.Tensor] = None) -> torch.Tensor:
    """h[t] = float32(table[tokens[t]]) * scale.  With `fed` (int32 on the device), a token id -(i + 1)
    stands for fed[i]: a token the step before has sampled and the host has not read yet.  copy: [T, n D] (rows may lie
    apart, in the table's dtype) that takes the same rows n times side by side."""
    T = tokens.numel()
    V, D = table.shape
    _need(tokens, "tokens", torch.int32)
    _need(table, "table")
    if fed is not None:
        _need(fed, "fed", torch.int32)
    if out is None:
        out = torch.empty((T, D), dtype=torch.float32, device=table.device)
    _need(out, "out", torch.float32, (T, D))
    if copy is not None and (copy.dtype != table.dtype or copy.shape[0] != T or copy.shape[1] % D or copy.stride(1) != 1 or not copy.is_cuda):
        raise KernelError("embed: the second output does not match the table")
    _call("q6k_embed", _ptr(tokens), _ptr(table), _ptr(out), _i(T), _i(D), _i(V), _i(dtype_code(table.dtype)), _ptr(fed),
          _i(fed.numel() if fed is not None else 0), _f(scale), _ptr(copy), _ll(copy.stride(0) if copy is not None else 0),
          _i(copy.shape[1] // D if copy is not None else 0), _stream())
    return out


def embed_pair(h: torch.Tensor, tokens: torch.Tensor, table: torch.Tensor, mul_prev: int, mul_cur: int, positions: torch.Tensor,
               req_of_token: torch.Tensor, q_start: torch.Tensor, slot_ids: torch.Tensor, prev: torch.Tensor,
               fed: Optional[torch.Tensor] = None) -> None:
    """h[t] += float32(table[row]) in place, row = (token before * mul_prev + token * mul_cur) mod buckets with buckets =
    rows of the table - 1, or the table's last row for a request's first token (position 0).  The token before a portion's
    first row is prev[slot] (int32 [slots]), which then takes the portion's last token.  `fed` as in embed."""
    T = tokens.numel()
    _need(h, "h", torch.float32, (T, table.shape[1]))
    _need(tokens, "tokens", torch.int32)
    _need(table, "table")
    _need(prev, "prev", torch.int32)
    if fed is not None:
        _need(fed, "fed", torch.int32)
    if table.shape[0] < 2 or mul_prev < 0 or mul_cur < 0:
        raise KernelError("embed_pair: the table needs a bucket and its last row, the multipliers may not be negative")
    _call("q6k_embed_pair", _ptr(tokens), _ptr(table), _ptr(h), _i(T), _i(table.shape[1]), _i(table.shape[0] - 1), _ll(mul_prev), _ll(mul_cur),
          _ptr(positions), _ptr(req_of_token), _ptr(q_start), _ptr(slot_ids), _ptr(prev), _i(dtype_code(table.dtype)), _ptr(fed),
          _i(fed.numel() if fed is not None else 0), _stream())


def rmsnorm(x: torch.Tensor, w: torch.Tensor, eps: float, out_dtype: torch.dtype, rows: Optional[torch.Tensor] = None,
            out: Optional[torch.Tensor] = None, add: Optional[torch.Tensor] = None, weighted=None) -> torch.Tensor:
    """out[r] = out_dtype(x[row] * rsqrt(mean(x[row]^2) + eps) * w); row = rows[r] if given.
    With `add` (float32, x's shape, or [splits, R, D] partial sums added in order), x += add is
    stored first: the block's residual add, fused.  With `weighted` = (y [pairs, D], pair_row [T, S]
    or None, weights [T, S]), x[t] += sum_s weights[t, s] * y[pair_row[t, s] or t*S + s] is stored
    first: the routed experts' combination (the arithmetic of `combine`)."""
    _need(x, "x", torch.float32)
    D = x.shape[-1]
    _need(w, "w", torch.float32, (D,))
    R = x.shape[0] if rows is None else rows.numel()
    if rows is not None:
        _need(rows, "rows", torch.int32)
    if out is None:
        out = torch.empty((R, D), dtype=out_dtype, device=x.device)
    _need(out, "out", out_dtype, (R, D))
    splits, stride = 1, 0
    if add is not None:
        _need(add, "add", torch.float32)
        if add.dim() == 3:                       # [splits, R, D]: partial sums, added in order
            splits, stride = add.shape[0], add.shape[1] * add.shape[2]
            if tuple(add.shape[1:]) != tuple(x.shape):
                raise KernelError("rmsnorm: the partial sums do not match x")
        elif tuple(add.shape) != tuple(x.shape):
            raise KernelError("rmsnorm: add does not match x")
    y = pair_row = pair_w = None
    S = 0
    if weighted is not None:
        y, pair_row, pair_w = weighted
        T, S = pair_w.shape
        _need(y, "weighted rows", torch.float32)
        _need(pair_w, "weights", torch.float32)
        if pair_row is not None:
            _need(pair_row, "pair_row", torch.int32)
        if T != x.shape[0] or y.shape[1] != D or y.shape[0] < T * S or (pair_row is not None and pair_row.numel() != T * S):
            raise KernelError("rmsnorm: the weighted rows do not match x")
        if not rmsnorm_fuses_weighted(D):
            combine(y, pair_row, pair_w, x)      # widths the register kernel does not take: two passes
            y = pair_row = pair_w = None
    _call("q6k_rmsnorm", _ptr(x), _ptr(add), _i(splits), _ll(stride), _ptr(rows), _ptr(w), _f(eps), _ptr(out), _i(R), _i(D),
          _i(dtype_code(out_dtype)), _ptr(y), _ptr(pair_row), _ptr(pair_w), _i(S), _stream())
    return out


@functools.lru_cache(maxsize=None)          # a question about sizes: asked of the library once
def rmsnorm_fuses_weighted(D: int) -> bool:
    lib = library()
    lib.q6k_rmsnorm_fuses_pairs.restype = ctypes.c_int
    return bool(lib.q6k_rmsnorm_fuses_pairs(_i(D)))


def combine(y: torch.Tensor, pair_row: torch.Tensor, sel_w: torch.Tensor, h: torch.Tensor) -> None:
    """h[t] += sum_s sel_w[t, s] * y[pair_row[t, s]] in slot order."""
    T, S = sel_w.shape
    D = h.shape[1]
    _need(y, "y", torch.float32)
    _need(sel_w, "sel_w", torch.float32)
    _need(h, "h", torch.float32, (T, D))
    if pair_row is not None:
        _need(pair_row, "pair_row", torch.int32)
    if y.shape[1] != D or (pair_row is not None and pair_row.numel() != T * S) or y.shape[0] < T * S:
        raise KernelError("combine: shapes disagree")
    _call("q6k_combine", _ptr(y), _ptr(pair_row), _ptr(sel_w), _i(T), _i(S), _i(D), _ptr(h), _stream())


def swiglu(gu: torch.Tensor, out_dtype: torch.dtype) -> torch.Tensor:
    """act = out_dtype(silu(gu[:, :I]) * gu[:, I:])."""
    _need(gu, "gu", torch.float32)
    rows, two_i = gu.shape
    act = torch.empty((rows, two_i // 2), dtype=out_dtype, device=gu.device)
    _call("q6k_swiglu", _ptr(gu), _ptr(act), _i(rows), _i(two_i // 2), _i(dtype_code(out_dtype)), _stream())
    return act


# --------------------------------------------------------------------------- matrix products (CUDA cores)
EPI_STORE, EPI_ADD, EPI_SWIGLU, EPI_ACT = 0, 1, 2, 4
ACTIVATIONS = {"silu": 0, "gelu_tanh": 1, "relu2": 2}
# A gate that takes a constant is named with it, ("clamped", limit): with g the gate's product and u the other one,
# g' = min(g, limit), u' = clamp(u, -limit, limit), and the result is g' sigmoid(1.702 g') (u' + 1).  Gated epilogues only.
GATES_WITH_LIMIT = {"clamped": 3}


def act_has_param(act) -> bool:
    return isinstance(act, tuple)


def _act_code(act, gated: bool):
    """(code, parameter) of an activation name or a (name, constant) pair."""
    if isinstance(act, tuple):
        name, param = act
        if name not in GATES_WITH_LIMIT or not gated:
            raise KernelError(f"unknown activation {act!r} (with a constant, for gated products: {', '.join(GATES_WITH_LIMIT)})")
        return GATES_WITH_LIMIT[name], float(param)
    if act not in ACTIVATIONS:
        raise KernelError(f"unknown activation {act!r}; known: {', '.join(ACTIVATIONS)}")
    return ACTIVATIONS[act], 0.0


def _epilogue(w2, accumulate: bool, act) -> int:
    """The launchers' epilogue argument: with w2 the gated epilogue act(x w^T) * (x w2^T) (SwiGLU when act is None or
    "silu"); with act alone act(x w^T), stored in the operand dtype; else store or add in FP32.  The activation's code
    rides above bit 8 (its constant, if it has one, is `_act_param(act)`)."""
    code = _act_code(act, w2 is not None)[0] << 8 if act is not None else 0
    if w2 is not None:
        return EPI_SWIGLU | code
    if act is not None:
        if accumulate:
            raise KernelError("an activated product is stored, not added")
        return EPI_ACT | code
    return EPI_ADD if accumulate else EPI_STORE


def _act_param(act) -> float:
    return float(act[1]) if isinstance(act, tuple) else 0.0


def gemm_simt(a: torch.Tensor, w: torch.Tensor, out: Optional[torch.Tensor] = None, accumulate: bool = False,
              w2: Optional[torch.Tensor] = None, a_rows: Optional[torch.Tensor] = None, groups=None,
              rows: Optional[int] = None, act: Optional[str] = None) -> torch.Tensor:
    """out[r] (+)= a[row(r)] @ w_g^T with FP32 fused multiply-adds.  act: the gate's activation when w2 is given (default
    silu); without w2, out = act(a w^T) in a's dtype.

    a: [*, K]; w: [N, K] or, grouped, [G, N, K]; w2 (same shape) switches to the SwiGLU epilogue,
    whose output has a's dtype; otherwise the output is float32.  a_rows: int32 [M] gathers rows of
    a.  groups: (group_offsets [G+1], tile_group, tile_row0, num_tiles) from `tile_list`.
    """
    _need(a, "a")
    _need(w, "w", a.dtype)
    K = a.shape[1]
    grouped = w.dim() == 3
    N = w.shape[-2]
    if w.shape[-1] != K:
        raise KernelError(f"gemm: a has K={K}, w has K={w.shape[-1]}")
    if grouped and groups is None:
        raise KernelError("gemm: a grouped weight needs group offsets and a tile list")
    M = rows if rows is not None else (a_rows.numel() if a_rows is not None else a.shape[0])
    epi = _epilogue(w2, accumulate, act)
    out_dtype = a.dtype if w2 is not None or act is not None else torch.float32
    if out is None:
        if accumulate:
            raise KernelError("gemm: accumulate needs an output")
        out = torch.empty((M, N), dtype=out_dtype, device=a.device)
    _need(out, "out", out_dtype)
    if out.shape[0] < M or out.shape[1] != N:
        raise KernelError(f"gemm: out has shape {tuple(out.shape)}, needs [{M}, {N}]")
    if w2 is not None:
        _need(w2, "w2", a.dtype, w.shape)
    if a_rows is not None:
        _need(a_rows, "a_rows", torch.int32)
    stride = N * K if grouped else 0
    if grouped:
        offsets, tile_group, tile_row0, num_tiles = groups
        max_tiles = tile_group.numel()
    else:
        offsets = tile_group = tile_row0 = num_tiles = None
        max_tiles = 0
    _call("q6k_gemm_simt", _ptr(a), _i(a.stride(0)), _ptr(a_rows), _ptr(w), _ptr(w2), _ll(stride), _ptr(out), _i(out.stride(0)),
          _i(M), _i(N), _i(K), _ptr(tile_group), _ptr(tile_row0), _ptr(offsets), _ptr(num_tiles), _i(max_tiles), _i(epi), _f(_act_param(act)),
          _i(dtype_code(a.dtype)), _stream())
    return out


def simt_tile_rows() -> int:
    lib = library()
    lib.q6k_gemm_tile_rows.restype = ctypes.c_int
    return lib.q6k_gemm_tile_rows()


def tile_list(offsets: torch.Tensor, pairs: int, bm: int):
    """(offsets, tile_group, tile_row0, num_tiles) for the groups' row tiles of bm rows."""
    _need(offsets, "offsets", torch.int32)
    G = offsets.numel() - 1
    max_tiles = pairs // bm + min(pairs, G)          # full tiles plus at most one ragged tile per non-empty group
    tile_group = torch.empty(max_tiles, dtype=torch.int32, device=offsets.device)
    tile_row0 = torch.empty(max_tiles, dtype=torch.int32, device=offsets.device)
    num_tiles = torch.empty(1, dtype=torch.int32, device=offsets.device)
    _call("q6k_tile_list", _ptr(offsets), _i(G), _i(bm), _ptr(tile_group), _ptr(tile_row0), _ptr(num_tiles), _i(max_tiles), _stream())
    return offsets, tile_group, tile_row0, num_tiles


# --------------------------------------------------------------------------- matrix products (tcgen05 tensor cores)
def gather_rows(x: torch.Tensor, idx: torch.Tensor) -> torch.Tensor:
    """out[r] = x[idx[r]] (rows of a multiple of 16 bytes)."""
    _need(x, "x")
    _need(idx, "idx", torch.int32)
    out = torch.empty((idx.numel(), x.shape[1]), dtype=x.dtype, device=x.device)
    _call("q6k_gather_rows", _ptr(x), _ptr(idx), _ptr(out), _i(idx.numel()), _i(x.shape[1] * x.element_size()), _stream())
    return out


def tc_supported(a: torch.Tensor, w: torch.Tensor) -> bool:
    """Whether the tensor-core kernel takes these operands: bfloat16, K a multiple of 8, rows
    starting on 16 bytes."""
    return (a.dtype == torch.bfloat16 and w.dtype == torch.bfloat16 and a.shape[1] % 8 == 0 and a.stride(0) % 8 == 0
            and a.stride(1) == 1 and a.data_ptr() % 16 == 0 and w.data_ptr() % 16 == 0 and w.is_contiguous())


def tc_token_tile(rows: int, dual: bool) -> int:
    lib = library()
    lib.q6k_tc_token_tile.restype = ctypes.c_int
    return lib.q6k_tc_token_tile(_i(rows), _i(1 if dual else 0))


def tc_status() -> int:
    """0, or the code of a bounded wait that ran out inside a tensor-core kernel (synchronises)."""
    lib = library()
    lib.q6k_tc_status.restype = ctypes.c_int
    lib.q6k_attention_status.restype = ctypes.c_int
    lib.q6k_attention_tc_status.restype = ctypes.c_int
    lib.q6k_router_status.restype = ctypes.c_int
    return lib.q6k_tc_status() or lib.q6k_attention_status() or lib.q6k_attention_tc_status() or lib.q6k_router_status()


def selftest_wait_runs_out(limit_cycles: int = 2_000_000):
    """Runs a kernel whose bounded mbarrier wait must run out (nothing ever arrives on its barrier):
    (status, cycles waited); status 1 is the run-out the kernel has to record.  The product kernels'
    waits go through the same routine with a limit of about two seconds."""
    status, waited = ctypes.c_int(-1), ctypes.c_longlong()
    _call("q6k_selftest_wait_runs_out", _ll(limit_cycles), ctypes.byref(status), ctypes.byref(waited), _stream())
    return status.value, waited.value


_workspaces = {}
_retired = []                             # outgrown scratch stays allocated: recorded CUDA graphs still point at it


def _workspace(nbytes: int, device, which: str = "") -> torch.Tensor:
    key = str(device) + which             # one scratch buffer per device and kind: the engine runs on one stream
    ws = _workspaces.get(key)
    if ws is None or ws.numel() * 4 < nbytes:
        if ws is not None:
            _retired.append(ws)
        ws = torch.empty(max(nbytes // 4, 1 << 20), dtype=torch.float32, device=device)
        _workspaces[key] = ws
    return ws


def gemm_tc(a: torch.Tensor, w: torch.Tensor, out: Optional[torch.Tensor] = None, accumulate: bool = False,
            w2: Optional[torch.Tensor] = None, groups=None, bt: int = 0, rows: Optional[int] = None,
            keep_partials: bool = False, act: Optional[str] = None) -> torch.Tensor:
    """The same contract as gemm_simt without the row gather, on tcgen05 tensor cores: bfloat16
    operands, FP32 accumulation in tensor memory.  Grouped calls pass the tile list made for
    token tile `bt` (tile_list(offsets, pairs, bt)).  keep_partials (dense, plain store): when the
    kernel slices K over CTAs the result is the FP32 partial products [slices, M, N], a view of the
    device's scratch buffer that stays valid until the next kernel that uses scratch; the consumer
    sums the slices in order."""
    if not tc_supported(a, w):
        raise KernelError("gemm_tc: operands must be bfloat16 with K a multiple of 8 and 16-byte aligned rows")
    K = a.shape[1]
    grouped = w.dim() == 3
    G = w.shape[0] if grouped else 1
    N = w.shape[-2]
    if w.shape[-1] != K:
        raise KernelError(f"gemm_tc: a has K={K}, w has K={w.shape[-1]}")
    if grouped and groups is None:
        raise KernelError("gemm_tc: a grouped weight needs group offsets and a tile list")
    M = rows if rows is not None else a.shape[0]
    epi = _epilogue(w2, accumulate, act)             # act: the gate's activation with w2; alone (grouped rows only): out = act(a w^T) in bfloat16
    out_dtype = torch.bfloat16 if w2 is not None or act is not None else torch.float32
    lib = library()
    splits = 1
    if keep_partials:
        if grouped or w2 is not None or accumulate or out is not None:
            raise KernelError("gemm_tc: partial products are kept only for a dense product that is stored")
        lib.q6k_gemm_tc_splits.restype = ctypes.c_int
        splits = lib.q6k_gemm_tc_splits(_i(M), _i(N), _i(K))
        keep_partials = splits > 1
    if out is None:
        if accumulate:
            raise KernelError("gemm_tc: accumulate needs an output")
        out = torch.empty((M, N) if not keep_partials else (1, N), dtype=out_dtype, device=a.device)
    _need(out, "out", out_dtype)
    if (out.shape[0] < M and not keep_partials) or out.shape[1] != N:
        raise KernelError(f"gemm_tc: out has shape {tuple(out.shape)}, needs [{M}, {N}]")
    if w2 is not None:
        _need(w2, "w2", torch.bfloat16, w.shape)
    ws = None
    ws_bytes = 0
    if grouped:
        offsets, tile_group, tile_row0, num_tiles = groups
        max_tiles = tile_group.numel()
    else:
        offsets = tile_group = tile_row0 = num_tiles = None
        max_tiles = 0
        if w2 is None and act is None:
            lib.q6k_gemm_tc_workspace.restype = ctypes.c_longlong
            ws_bytes = lib.q6k_gemm_tc_workspace(_i(M), _i(N), _i(K))
            if ws_bytes:
                ws = _workspace(ws_bytes, a.device)
                ws_bytes = ws.numel() * 4
    _call("q6k_gemm_tc", _ptr(a), _ll(a.stride(0)), _i(M), _ptr(w), _ptr(w2), _i(G), _i(N), _i(K), _ptr(out), _i(out.stride(0)),
          _i(epi), _f(_act_param(act)), _ptr(tile_group), _ptr(tile_row0), _ptr(offsets), _ptr(num_tiles), _i(max_tiles), _i(bt), _ptr(ws),
          _ll(ws_bytes), _i(1 if keep_partials else 0), _stream())
    if keep_partials:
        return ws[: splits * M * N].view(splits, M, N)
    return out


# --------------------------------------------------------------------------- matrix-vector products (a step of very few tokens)
@functools.lru_cache(maxsize=None)          # a question about sizes: asked of the library once
def gemv_preferred(tokens: int, N: int, K: int) -> bool:
    """Whether a bfloat16 product of `tokens` rows with an [N, K] matrix should go to the matrix-vector kernel."""
    lib = library()
    lib.q6k_gemv_preferred.restype = ctypes.c_int
    return bool(lib.q6k_gemv_preferred(_i(tokens), _i(N), _i(K)))


def gemv(x: torch.Tensor, w: torch.Tensor, w2: Optional[torch.Tensor] = None, out: Optional[torch.Tensor] = None, accumulate: bool = False,
         pair_expert: Optional[torch.Tensor] = None, pair_div: int = 1, pairs_are_old: bool = False, act: Optional[str] = None) -> torch.Tensor:
    """out[t] (+)= x[t] @ w^T for one to four rows of x (bfloat16, FP32 sums and output); with w2 the SwiGLU epilogue
    silu(x w^T) * (x w2^T) in bfloat16.  With pair_expert (int32 [pairs]) and w [experts, N, K]: pair y multiplies row
    y // pair_div of x with the matrix of expert pair_expert[y] and writes row y (any number of pairs).
    The kernel streams its weights while the kernel launched before it on the stream still runs (only x and out wait
    for that kernel); with a pair list this needs the caller's word (pairs_are_old) that the list was not made by that
    very kernel."""
    if not tc_supported(x, w):
        raise KernelError("gemv: operands must be bfloat16 with K a multiple of 8 and 16-byte aligned rows")
    K = x.shape[1]
    N = w.shape[-2]
    if w.shape[-1] != K or (w.dim() == 3) != (pair_expert is not None):
        raise KernelError(f"gemv: x has K={K}, w has shape {tuple(w.shape)} (three dimensions go with pair_expert)")
    pairs = 0
    if pair_expert is not None:
        _need(pair_expert, "pair_expert", torch.int32)
        pairs = pair_expert.numel()
    rows = pairs if pair_expert is not None else x.shape[0]
    if act is not None and w2 is None:
        raise KernelError("gemv: an activation goes with the gated epilogue")
    epi = _epilogue(w2, accumulate, act)
    out_dtype = torch.bfloat16 if w2 is not None else torch.float32
    if w2 is not None:
        _need(w2, "w2", torch.bfloat16, w.shape)
    if out is None:
        if accumulate:
            raise KernelError("gemv: accumulate needs an output")
        out = torch.empty((rows, N), dtype=out_dtype, device=x.device)
    _need(out, "out", out_dtype)
    if out.shape[0] < rows or out.shape[1] != N:
        raise KernelError(f"gemv: out has shape {tuple(out.shape)}, needs [{rows}, {N}]")
    early = pair_expert is None or pairs_are_old
    _call("q6k_gemv", _ptr(x), _ll(x.stride(0)), _i(x.shape[0]), _ptr(w), _ptr(w2), _i(N), _i(K), _ptr(pair_expert), _i(pairs), _i(pair_div),
          _ptr(out), _ll(out.stride(0)), _i(epi), _i(1 if early else 0), _stream())
    return out


@functools.lru_cache(maxsize=None)          # a question about sizes: asked of the library once
def gemm_skinny_preferred(tokens: int, N: int, K: int) -> bool:
    """Whether a bfloat16 product of `tokens` rows (3 to 16) with an [N, K] matrix should go to the mma.sync kernel for few tokens."""
    lib = library()
    lib.q6k_gemm_skinny_preferred.restype = ctypes.c_int
    return bool(lib.q6k_gemm_skinny_preferred(_i(tokens), _i(N), _i(K)))


@functools.lru_cache(maxsize=None)          # a question about sizes: asked of the library once
def gemm_skinny_slices(tokens: int, N: int, K: int) -> int:
    """Slices of K the mma.sync kernel for few tokens would cut a plain product into when the caller can add partial
    sums itself (a matrix with too few rows to fill the SMs otherwise); 0: the product is not for this kernel."""
    lib = library()
    lib.q6k_gemm_skinny_slices.restype = ctypes.c_int
    return lib.q6k_gemm_skinny_slices(_i(tokens), _i(N), _i(K))


def gemm_skinny(x: torch.Tensor, w: torch.Tensor, w2: Optional[torch.Tensor] = None, out: Optional[torch.Tensor] = None,
                accumulate: bool = False, slices: int = 1, act: Optional[str] = None) -> torch.Tensor:
    """out[t] (+)= x[t] @ w^T for at most 16 rows of x (bfloat16, FP32 sums and output) on mma.sync; with w2 the SwiGLU
    epilogue silu(x w^T) * (x w2^T) in bfloat16.  K is not split over blocks unless slices > 1 (plain products only):
    the result is then [slices, T, N] partial sums, a view of the device's scratch buffer that stays valid until the
    next kernel that uses scratch; the consumer adds the slices in order."""
    if not tc_supported(x, w) or w.dim() != 2:
        raise KernelError("gemm_skinny: operands must be bfloat16 matrices with K a multiple of 8 and 16-byte aligned rows")
    T, K = x.shape
    N = w.shape[0]
    if w.shape[1] != K:
        raise KernelError(f"gemm_skinny: x has K={K}, w has K={w.shape[1]}")
    if act is not None and w2 is None:
        raise KernelError("gemm_skinny: an activation goes with the gated epilogue")
    epi = _epilogue(w2, accumulate, act)
    out_dtype = torch.bfloat16 if w2 is not None else torch.float32
    if w2 is not None:
        _need(w2, "w2", torch.bfloat16, w.shape)
    if slices > 1:
        if out is not None or epi != EPI_STORE:
            raise KernelError("gemm_skinny: slices of K are for plain products into scratch")
        out = _workspace(slices * T * N * 4, x.device)[: slices * T * N].view(slices, T, N)
        _call("q6k_gemm_skinny", _ptr(x), _ll(x.stride(0)), _i(T), _ptr(w), _ptr(w2), _i(N), _i(K), _ptr(out), _ll(N), _i(epi), _f(_act_param(act)),
              _i(slices), _ll(T * N), _stream())
        return out
    if out is None:
        if accumulate:
            raise KernelError("gemm_skinny: accumulate needs an output")
        out = torch.empty((T, N), dtype=out_dtype, device=x.device)
    _need(out, "out", out_dtype)
    if out.shape[0] < T or out.shape[1] != N:
        raise KernelError(f"gemm_skinny: out has shape {tuple(out.shape)}, needs [{T}, {N}]")
    _call("q6k_gemm_skinny", _ptr(x), _ll(x.stride(0)), _i(T), _ptr(w), _ptr(w2), _i(N), _i(K), _ptr(out), _ll(out.stride(0)), _i(epi), _f(_act_param(act)),
          _i(1), _ll(0), _stream())
    return out


# --------------------------------------------------------------------------- attention
def qk_prep(qkv: torch.Tensor, Hq: int, Hkv: int, hd: int, q_norm, k_norm, eps: float, rotary,
            positions: torch.Tensor, req_of_token: torch.Tensor, block_table: Optional[torch.Tensor], page_size: int,
            k_pages: Optional[torch.Tensor], v_pages: Optional[torch.Tensor], out_dtype: torch.dtype, bias: Optional[torch.Tensor] = None,
            values_are_keys: bool = False, value_norm: bool = False) -> torch.Tensor:
    """QK-norm, rotation, q -> out_dtype [T, Hq, hd]; k, v -> their pages (when k_pages is given).
    bias: FP32, one entry per column of a row (q, k, v side by side), added to the summed product first.  values_are_keys:
    the rows hold q and k only, and a key's value is the key as projected (bias included, before norm and rotation).
    value_norm: a head's value is divided by its root mean square (eps, no weight) before it is stored.
    rotary: None, or (inv_freq float32 [rotary_dim / 2] on the device, rotary_dim, neighbours): the
    first rotary_dim dimensions of every q and k head turn by position * inv_freq[pair], paired by
    halves (d with d + rotary_dim / 2) or, neighbours=True, 2i with 2i + 1.
    qkv may be [slices, T, width]: split-K partial products, summed in order first."""
    _need(qkv, "qkv", torch.float32)
    splits, split_stride = 1, 0
    if qkv.dim() == 3:
        splits, split_stride = qkv.shape[0], qkv.shape[1] * qkv.shape[2]
        qkv = qkv[0]
    T = qkv.shape[0]
    if qkv.shape[1] < (Hq + (1 if values_are_keys else 2) * Hkv) * hd and k_pages is not None:
        raise KernelError("qk_prep: qkv rows are too short")
    if bias is not None:
        _need(bias, "bias", torch.float32)
        if bias.numel() < (Hq + (0 if k_pages is None else Hkv if values_are_keys else 2 * Hkv)) * hd:
            raise KernelError("qk_prep: the bias is shorter than a row")
    _need(positions, "positions", torch.int32)
    _need(req_of_token, "req_of_token", torch.int32)
    write = k_pages is not None
    if write:
        _need(k_pages, "k_pages", out_dtype)
        _need(v_pages, "v_pages", out_dtype, k_pages.shape)
        _need(block_table, "block_table", torch.int32)
        if k_pages.dim() != 4 or k_pages.shape[0] != Hkv or tuple(k_pages.shape[2:]) != (page_size, hd):
            raise KernelError(f"qk_prep: pages have shape {tuple(k_pages.shape)}, expected [{Hkv}, *, {page_size}, {hd}]")
    for nm, w in (("q_norm", q_norm), ("k_norm", k_norm)):
        if w is not None:
            _need(w, nm, torch.float32, (hd,))
    inv_freq, rotary_dim, neighbours = rotary if rotary is not None else (None, 0, False)
    if inv_freq is not None:
        if rotary_dim <= 0 or rotary_dim % 2 or rotary_dim > hd:
            raise KernelError(f"qk_prep: {rotary_dim} rotating dimensions of a head of {hd}")
        _need(inv_freq, "inv_freq", torch.float32, (rotary_dim // 2,))
    q = torch.empty((T, Hq, hd), dtype=out_dtype, device=qkv.device)
    max_blocks = block_table.shape[1] if block_table is not None else 1
    _call("q6k_qk_prep", _ptr(qkv), _i(qkv.stride(0)), _i(splits), _ll(split_stride), _i(T), _i(Hq), _i(Hkv), _i(hd), _ptr(q_norm), _ptr(k_norm), _f(eps),
          _ptr(inv_freq), _i(rotary_dim), _i(1 if neighbours else 0), _ptr(positions), _ptr(req_of_token), _ptr(block_table),
          _i(max_blocks), _i(page_size), _i(k_pages.shape[1] if write else 0), _ptr(q), _ptr(k_pages), _ptr(v_pages),
          _i(1 if write else 0), _i(dtype_code(out_dtype)), _ptr(bias), _i(1 if values_are_keys else 0), _i(1 if value_norm else 0), _stream())
    return q


def attention_generic(q: torch.Tensor, k_pages: torch.Tensor, v_pages: torch.Tensor, block_table: torch.Tensor,
                      req_of_token: torch.Tensor, positions: torch.Tensor, window: Optional[int],
                      sinks: Optional[torch.Tensor], scale: Optional[float] = None) -> torch.Tensor:
    """Causal (optionally windowed, optionally with sinks) attention of every row over its request's pages."""
    _need(q, "q")
    T, Hq, hd = q.shape
    _need(k_pages, "k_pages", q.dtype)
    _need(v_pages, "v_pages", q.dtype, k_pages.shape)
    Hkv, num_pages, page_size, hd2 = k_pages.shape
    if hd2 != hd:
        raise KernelError(f"attention: q has head_dim {hd}, the pages {hd2}")
    _need(block_table, "block_table", torch.int32)
    _need(req_of_token, "req_of_token", torch.int32)
    _need(positions, "positions", torch.int32)
    if sinks is not None:
        _need(sinks, "sinks", torch.float32, (Hq,))
    out = torch.empty((T, Hq * hd), dtype=q.dtype, device=q.device)
    _call("q6k_attention_generic", _ptr(q), _ptr(k_pages), _ptr(v_pages), _i(num_pages), _ptr(block_table), _i(block_table.shape[1]),
          _i(page_size), _ptr(req_of_token), _ptr(positions), _i(window or 0), _ptr(sinks),
          _f(scale if scale is not None else 1.0 / math.sqrt(hd)), _ptr(out), _i(T), _i(Hq), _i(Hkv), _i(hd),
          _i(dtype_code(q.dtype)), _stream())
    return out


@functools.lru_cache(maxsize=None)          # a question about sizes: asked of the library once
def attention_tc_supported(hd: int, G: int, page_size: int) -> bool:
    lib = library()
    lib.q6k_attention_tc_supported.restype = ctypes.c_int
    return bool(lib.q6k_attention_tc_supported(_i(hd), _i(G), _i(page_size)))


@functools.lru_cache(maxsize=None)          # a question about sizes: asked of the library once
def attention_tc_tile_tokens(G: int) -> int:
    """Tokens one tile of attention_tc may hold (128 // G: 128 query rows)."""
    lib = library()
    lib.q6k_attention_tc_tile_tokens.restype = ctypes.c_int
    return lib.q6k_attention_tc_tile_tokens(_i(G))


def attention_tc(q: torch.Tensor, k_pages: torch.Tensor, v_pages: torch.Tensor, block_table: torch.Tensor,
                 req_of_token: torch.Tensor, positions: torch.Tensor, tile_tok0: torch.Tensor, tile_ntok: torch.Tensor,
                 window: Optional[int], sinks: Optional[torch.Tensor], scale: Optional[float] = None,
                 out: Optional[torch.Tensor] = None, chunk: Optional[int] = None) -> torch.Tensor:
    """bfloat16 attention for prompt portions with both products on tcgen05 tensor cores
    (accumulators and probabilities in tensor memory, K/V pages by TMA).  Head size 128.
    tile_tok0 / tile_ntok: [n, 2], two tiles of one request per CTA (StepContext.query_tile_pairs),
    each of at most attention_tc_tile_tokens(G) tokens at consecutive positions; the second may be
    empty.  Each tile reads its whole key range; the two share the K/V stream.  Only the rows of
    the listed tiles are written (into `out` [T, Hq*hd] when given).  chunk: a position sees the earlier keys of its own block
    of `chunk` positions only."""
    _need(q, "q", torch.bfloat16)
    T, Hq, hd = q.shape
    _need(k_pages, "k_pages", torch.bfloat16)
    _need(v_pages, "v_pages", torch.bfloat16, k_pages.shape)
    Hkv, num_pages, page_size, hd2 = k_pages.shape
    if hd2 != hd:
        raise KernelError(f"attention: q has head_dim {hd}, the pages {hd2}")
    for nm, t in (("block_table", block_table), ("req_of_token", req_of_token), ("positions", positions),
                  ("tile_tok0", tile_tok0), ("tile_ntok", tile_ntok)):
        _need(t, nm, torch.int32)
    if tile_tok0.dim() != 2 or tile_tok0.shape[1] != 2 or tile_ntok.shape != tile_tok0.shape:
        raise KernelError("attention_tc: tile_tok0 and tile_ntok must be [pairs, 2]")
    if sinks is not None:
        _need(sinks, "sinks", torch.float32, (Hq,))
    if out is None:
        out = torch.empty((T, Hq * hd), dtype=torch.bfloat16, device=q.device)
    else:
        _need(out, "out", torch.bfloat16, (T, Hq * hd))
    _call("q6k_attention_tc", _ptr(q), _ptr(k_pages), _ptr(v_pages), _ll(num_pages), _ptr(block_table),
          _i(block_table.shape[1]), _i(page_size), _ptr(req_of_token), _ptr(positions), _ptr(tile_tok0), _ptr(tile_ntok),
          _i(tile_tok0.shape[0]), _i(window or 0), _i(chunk or 0), _ptr(sinks), _f(scale if scale is not None else 1.0 / math.sqrt(hd)), _ptr(out),
          _i(Hq), _i(Hkv), _i(hd), _stream())
    return out


@functools.lru_cache(maxsize=None)          # a question about sizes: asked of the library once
def attention_mma_supported(hd: int, G: int, wide: bool) -> bool:
    lib = library()
    lib.q6k_attention_mma_supported.restype = ctypes.c_int
    return bool(lib.q6k_attention_mma_supported(_i(hd), _i(G), _i(1 if wide else 0)))


@functools.lru_cache(maxsize=None)          # a question about sizes: asked of the library once
def attention_mma_tile_rows(hd: int, G: int, max_tokens: int) -> int:
    """Query rows of the tiles attention_mma should be given when no request brings more than
    max_tokens tokens to the step: 8, 16 or 128 (a tile holds rows // G tokens); 0 if the kernel
    does not take this head and group size."""
    lib = library()
    lib.q6k_attention_mma_tile_rows.restype = ctypes.c_int
    return lib.q6k_attention_mma_tile_rows(_i(hd), _i(G), _i(max_tokens))


_resident = {}


def attention_mma_resident_ctas(hd: int, rows: int) -> int:
    """CTAs of attention_mma (tiles of `rows` rows) the current device runs at once: the number of
    work items per launch (over all KV heads) that makes exactly one wave."""
    key = (torch.cuda.current_device(), hd, rows)
    if key not in _resident:
        lib = library()
        lib.q6k_attention_mma_resident_ctas.restype = ctypes.c_int
        n = lib.q6k_attention_mma_resident_ctas(_i(hd), _i(rows))
        if n <= 0:
            raise KernelError(f"attention_mma: no resident CTA count for head_dim {hd}, tiles of {rows} rows")
        _resident[key] = n
    return _resident[key]


def attention_plan(positions: torch.Tensor, req_of_token: torch.Tensor, tile_tok0: torch.Tensor, tile_ntok: torch.Tensor,
                   window: Optional[int], n_work: int, min_per: int = 2, into=None, chunk: Optional[int] = None):
    """Which CTA of attention_mma walks which key tiles, made on the device from the step's
    positions: (work int32 [n_work, 8], tile_plan int32 [n_tiles, 4]).  n_work (at least the number
    of tiles) CTAs per KV head share the key tiles about evenly; a tile's keys are split into
    parts of at least min_per key tiles (of 64 keys).  One plan serves every layer with this
    window and chunk; recorded into a CUDA graph it is remade from the positions of each replay.
    into: the pair of tensors of an earlier call with the same sizes, to be filled again."""
    for nm, t in (("req_of_token", req_of_token), ("positions", positions), ("tile_tok0", tile_tok0), ("tile_ntok", tile_ntok)):
        _need(t, nm, torch.int32)
    n_tiles = tile_tok0.numel()
    n_work = max(int(n_work), n_tiles)
    if into is not None:
        work, tile_plan = into
        _need(work, "work", torch.int32, (n_work, 8))
        _need(tile_plan, "tile_plan", torch.int32, (n_tiles, 4))
    else:
        work = torch.empty((n_work, 8), dtype=torch.int32, device=positions.device)
        tile_plan = torch.empty((n_tiles, 4), dtype=torch.int32, device=positions.device)
    _call("q6k_attention_plan", _ptr(positions), _ptr(req_of_token), _ptr(tile_tok0), _ptr(tile_ntok), _i(n_tiles), _i(window or 0), _i(chunk or 0),
          _i(n_work), _i(min_per), _ptr(work), _ptr(tile_plan), _stream())
    return work, tile_plan


@functools.lru_cache(maxsize=None)          # a question about sizes: asked of the library once
def attention_mma_prepares(hd: int, G: int, rows: int, rotary_dim: int, neighbours: bool) -> bool:
    """Whether attention_mma with tiles of `rows` rows can make q and the new keys itself (its `prepare` argument)
    for heads of hd in groups of G with rotary_dim rotating dimensions (0: none)."""
    lib = library()
    lib.q6k_attention_mma_prepares.restype = ctypes.c_int
    return bool(lib.q6k_attention_mma_prepares(_i(hd), _i(G), _i(rows), _i(rotary_dim), _i(1 if neighbours else 0)))


def attention_mma(q: Optional[torch.Tensor], k_pages: torch.Tensor, v_pages: torch.Tensor, block_table: torch.Tensor,
                  req_of_token: torch.Tensor, positions: torch.Tensor, tile_tok0: torch.Tensor, tile_ntok: torch.Tensor,
                  rows: int, window: Optional[int], sinks: Optional[torch.Tensor], max_splits: int = 1, min_tiles: int = 2,
                  scale: Optional[float] = None, out: Optional[torch.Tensor] = None, plan=None, plan_is_old: bool = False,
                  prepare=None, chunk: Optional[int] = None) -> torch.Tensor:
    """bfloat16 tensor-core attention over the pages.  Tiles: tile_tok0[i] is the first row and
    tile_ntok[i] the number of tokens (consecutive positions of one request, at most rows // G;
    rows: 8, 16 or 128, see attention_mma_tile_rows) of tile i.  plan: attention_plan(...) of these tiles, this
    window and chunk; without one it is made here for max_splits CTAs per tile on average, none with fewer
    than min_tiles key tiles.  Only the rows of the listed tiles are written (into `out`
    [T, Hq*hd] when given).  plan_is_old: the caller's word that the plan and the block table were
    made before the kernel launched just before this call (the one that writes this step's q and
    keys); narrow tiles then fetch their older key tiles while that kernel still runs.

    prepare (tiles of 8 or 16 rows, see attention_mma_prepares; q is then None): a dict with what
    qk_prep takes: qkv float32 [T, >= (Hq + 2 Hkv) hd], heads (Hq), q_norm, k_norm, eps, rotary,
    write (bool); qkv may be [slices, T, width] split-K partial products.  The kernel then normalises, rotates and rounds q itself, and with write=True
    makes the tiles' keys and values and puts them into the pages (every token of the step must
    then lie in a tile).  With plan_is_old the plan must be older than the kernel that made qkv
    AND the one before it."""
    _need(k_pages, "k_pages", torch.bfloat16)
    _need(v_pages, "v_pages", torch.bfloat16, k_pages.shape)
    Hkv, num_pages, page_size, hd = k_pages.shape
    qkv = q_norm = k_norm = inv_freq = None
    eps, rotary_dim, write, ld, splits, split_stride = 0.0, 0, False, 0, 1, 0
    if prepare is not None:
        qkv, Hq, write = prepare["qkv"], int(prepare["heads"]), bool(prepare.get("write", False))
        if not qkv.is_cuda or qkv.dtype != torch.float32 or qkv.dim() not in (2, 3) or qkv.stride(-1) != 1:
            raise KernelError("attention_mma: qkv must be float32 rows [T, width] or [slices, T, width] on the device (rows may have a pitch of their own)")
        if qkv.dim() == 3:                   # split-K partial products: summed in order by the kernel
            splits, split_stride = qkv.shape[0], qkv.stride(0)
        T, ld = qkv.shape[-2], qkv.stride(-2)
        if qkv.shape[-1] < (Hq + 2 * Hkv if write else Hq) * hd:
            raise KernelError(f"attention_mma: qkv of shape {tuple(qkv.shape)} for {Hq} + 2 x {Hkv} heads of {hd}")
        q_norm, k_norm, eps = prepare.get("q_norm"), prepare.get("k_norm"), float(prepare.get("eps", 0.0))
        for nm, w in (("q_norm", q_norm), ("k_norm", k_norm)):
            if w is not None:
                _need(w, nm, torch.float32, (hd,))
        if prepare.get("rotary") is not None:
            inv_freq, rotary_dim, neighbours = prepare["rotary"]
            _need(inv_freq, "inv_freq", torch.float32, (rotary_dim // 2,))
            if neighbours:
                raise KernelError("attention_mma: pairs of neighbours are rotated by qk_prep only")
        dev = qkv.device
    else:
        _need(q, "q", torch.bfloat16)
        T, Hq, hd2 = q.shape
        if hd2 != hd:
            raise KernelError(f"attention: q has head_dim {hd2}, the pages {hd}")
        dev = q.device
    _need(block_table, "block_table", torch.int32)
    if sinks is not None:
        _need(sinks, "sinks", torch.float32, (Hq,))
    n_tiles = tile_tok0.numel()
    if plan is None:
        plan_is_old = False
        plan = attention_plan(positions, req_of_token, tile_tok0, tile_ntok, window, n_tiles * max(1, max_splits), min_tiles, chunk=chunk)
    work, tile_plan = plan
    _need(work, "work", torch.int32)
    _need(tile_plan, "tile_plan", torch.int32, (n_tiles, 4))
    n_work = work.shape[0]
    if out is None:
        out = torch.empty((T, Hq * hd), dtype=torch.bfloat16, device=dev)
    else:
        _need(out, "out", torch.bfloat16, (T, Hq * hd))
    part_o = part_ml = None
    if n_work > n_tiles:
        part_rows = n_work * Hkv * rows
        ws = _workspace(part_rows * (hd + 2) * 4, dev, "attention")       # a buffer of its own: qkv may be a view of the common one
        part_o = ws[: part_rows * hd]
        part_ml = ws[part_rows * hd: part_rows * (hd + 2)]
    _call("q6k_attention_mma", _ptr(q), _ptr(k_pages), _ptr(v_pages), _ll(num_pages), _ptr(block_table),
          _i(block_table.shape[1]), _i(page_size), _ptr(work), _ptr(tile_plan), _i(n_work), _i(n_tiles), _i(rows),
          _i(window or 0), _i(chunk or 0), _ptr(sinks), _f(scale if scale is not None else 1.0 / math.sqrt(hd)), _ptr(out), _ptr(part_o), _ptr(part_ml),
          _i(Hq), _i(Hkv), _i(hd), _i(1 if plan_is_old else 0), _ptr(qkv), _i(ld), _i(splits), _ll(split_stride), _ptr(q_norm), _ptr(k_norm), _f(eps),
          _ptr(inv_freq), _i(rotary_dim), _i(1 if write else 0), _stream())
    return out


# --------------------------------------------------------------------------- routing
def route(logits: torch.Tensor, k: int, scoring: str, renorm: bool):
    """(sel_e int32 [T, k], sel_w float32 [T, k]).  logits: [T, E], or [slices, T, E] split-K
    partial products of the router, which are summed in order first."""
    _need(logits, "logits", torch.float32)
    slices = logits.shape[0] if logits.dim() == 3 else 1
    T, E = logits.shape[-2:]
    if scoring not in ("softmax", "sigmoid"):
        raise KernelError(f"route: unknown scoring {scoring!r}")
    sel_e = torch.empty((T, k), dtype=torch.int32, device=logits.device)
    sel_w = torch.empty((T, k), dtype=torch.float32, device=logits.device)
    _call("q6k_route", _ptr(logits), _i(slices), _i(T), _i(E), _i(k), _i(1 if scoring == "sigmoid" else 0), _i(1 if renorm else 0),
          _ptr(sel_e), _ptr(sel_w), _stream())
    return sel_e, sel_w


@functools.lru_cache(maxsize=None)          # a question about sizes: asked of the library once
def router_small_supported(T: int, E: int, D: int, k: int) -> bool:
    """Whether the one-launch decode router (router_small, and with it the per-pair expert products) takes this step."""
    lib = library()
    lib.q6k_router_small_supported.restype = ctypes.c_int
    return bool(lib.q6k_router_small_supported(_i(T), _i(E), _i(D), _i(k)))



def router_small(xn: torch.Tensor, w: torch.Tensor, k: int, scoring: str, renorm: bool, with_logits: bool = False):
    """Router logits, scores and top-k of at most 16 tokens in one launch:
    (sel_e [T, k], sel_w [T, k], order [T*k]: the pairs sorted by expert); with_logits: also the
    FP32 router logits [T, E] the kernel left behind."""
    _need(xn, "xn", torch.bfloat16)
    _need(w, "w", torch.bfloat16)
    T, D = xn.shape
    E = w.shape[0]
    if w.shape[1] != D:
        raise KernelError("router_small: widths disagree")
    dev = xn.device
    logits = torch.empty((T, E), dtype=torch.float32, device=dev)
    sel_e = torch.empty((T, k), dtype=torch.int32, device=dev)
    sel_w = torch.empty((T, k), dtype=torch.float32, device=dev)
    order = torch.empty(T * k, dtype=torch.int32, device=dev)
    _call("q6k_router_small", _ptr(xn), _ptr(w), _i(T), _i(E), _i(D), _i(k), _i(1 if scoring == "sigmoid" else 0),
          _i(1 if renorm else 0), _ptr(logits), _ptr(sel_e), _ptr(sel_w), _ptr(order), _stream())
    return (sel_e, sel_w, order, logits) if with_logits else (sel_e, sel_w, order)


_pair_scratch = {}


def gemm_tc_pairs(a: torch.Tensor, w: torch.Tensor, pair_expert: torch.Tensor, pair_div: int, w2: Optional[torch.Tensor] = None,
                  order: Optional[torch.Tensor] = None, pairs_are_old: bool = False, act: Optional[str] = None) -> torch.Tensor:
    """Expert products of a decode step without a permutation: pair y (= token * slots + slot)
    multiplies row y // pair_div of `a` with expert pair_expert[y]; output row y.  With w2 the
    SwiGLU epilogue (bfloat16 output), else FP32.  A pair whose expert number is beyond the last matrix is skipped (its
    output row is left as it is).  pairs_are_old: the caller's word that
    pair_expert and order were not made by the kernel launched just before this one; the kernel
    then fetches its first weights while that kernel still runs."""
    if not tc_supported(a, w) or w.dim() != 3:
        raise KernelError("gemm_tc_pairs: operands must be bfloat16, K a multiple of 8, weights [experts, N, K]")
    _need(pair_expert, "pair_expert", torch.int32)
    pairs = pair_expert.numel()
    if order is not None:
        _need(order, "order", torch.int32, (pairs,))
    G, N, K = w.shape
    if a.shape[1] != K:
        raise KernelError(f"gemm_tc_pairs: a has K={a.shape[1]}, w has K={K}")
    if w2 is not None:
        _need(w2, "w2", torch.bfloat16, w.shape)
    out = torch.empty((pairs, N), dtype=torch.bfloat16 if w2 is not None or act is not None else torch.float32, device=a.device)
    # a few pairs only: K is sliced over CTAs, which meet through scratch kept per device (one stream uses it at a time)
    floats, counters = ctypes.c_longlong(), ctypes.c_int()
    _call("q6k_gemm_tc_pairs_scratch", _i(pairs), _i(N), _i(K), _i(1 if w2 is not None else 0), ctypes.byref(floats), ctypes.byref(counters))
    partial = tickets = None
    if floats.value:
        key = str(a.device)
        partial, tickets = _pair_scratch.get(key, (None, None))
        if partial is None or partial.numel() < floats.value or tickets.numel() < counters.value:
            _retired.append((partial, tickets))
            partial = torch.empty(max(floats.value, 1 << 18), dtype=torch.float32, device=a.device)
            tickets = torch.zeros(max(counters.value, 1024), dtype=torch.int32, device=a.device)
            _pair_scratch[key] = (partial, tickets)
    _call("q6k_gemm_tc_pairs", _ptr(a), _ll(a.stride(0)), _i(a.shape[0]), _ptr(w), _ptr(w2), _i(G), _i(N), _i(K), _ptr(out),
          _i(out.stride(0)), _i(_epilogue(w2, False, act)), _f(_act_param(act)), _ptr(pair_expert), _ptr(order), _i(pairs), _i(pair_div),
          _ptr(partial), _ll(partial.numel() if partial is not None else 0), _ptr(tickets),
          _i(tickets.numel() if tickets is not None else 0), _i(1 if pairs_are_old else 0), _stream())
    return out


def moe_permute(sel_e: torch.Tensor, E: int):
    """(offsets [E+1], pair_row [T, k], row_token [T*k]): rows sorted by expert, stable in pair order."""
    _need(sel_e, "sel_e", torch.int32)
    T, k = sel_e.shape
    pairs = T * k
    dev = sel_e.device
    lib = library()
    lib.q6k_moe_permute_scratch_ints.restype = ctypes.c_int
    scratch = torch.empty(lib.q6k_moe_permute_scratch_ints(_i(pairs), _i(E)), dtype=torch.int32, device=dev)
    offsets = torch.empty(E + 1, dtype=torch.int32, device=dev)
    pair_row = torch.empty((T, k), dtype=torch.int32, device=dev)
    row_token = torch.empty(pairs, dtype=torch.int32, device=dev)
    _call("q6k_moe_permute", _ptr(sel_e), _i(pairs), _i(k), _i(E), _ptr(scratch), _ptr(offsets), _ptr(pair_row),
          _ptr(row_token), _stream())
    return offsets, pair_row, row_token


def moe_plan(sel_e: torch.Tensor, E: int, bm: int, x: Optional[torch.Tensor] = None, live: Optional[int] = None):
    """The permutation of `moe_permute` and the row tiles of `tile_list(offsets, pairs, bm)` in three
    launches instead of four: (offsets, pair_row, row_token, (offsets, tile_group, tile_row0, num_tiles)).
    With x [T, D] (rows of a multiple of 16 bytes) the last launch also copies each pair's input
    row into its place, and the gathered rows [pairs, D] are returned as a fifth value.  live: only the
    first `live` experts have matrices; the pairs of the others come last and get no tiles and no copies."""
    live = E if live is None else int(live)
    _need(sel_e, "sel_e", torch.int32)
    T, k = sel_e.shape
    pairs = T * k
    dev = sel_e.device
    lib = library()
    lib.q6k_moe_permute_scratch_ints.restype = ctypes.c_int
    scratch = torch.empty(lib.q6k_moe_permute_scratch_ints(_i(pairs), _i(E)), dtype=torch.int32, device=dev)
    offsets = torch.empty(E + 1, dtype=torch.int32, device=dev)
    pair_row = torch.empty((T, k), dtype=torch.int32, device=dev)
    row_token = torch.empty(pairs, dtype=torch.int32, device=dev)
    max_tiles = pairs // bm + min(pairs, live)       # full tiles plus at most one ragged tile per non-empty group
    tile_group = torch.empty(max_tiles, dtype=torch.int32, device=dev)
    tile_row0 = torch.empty(max_tiles, dtype=torch.int32, device=dev)
    num_tiles = torch.empty(1, dtype=torch.int32, device=dev)
    gathered, row_bytes = None, 0
    if x is not None:
        _need(x, "x")
        if x.dim() != 2 or x.shape[0] != T:
            raise KernelError(f"moe_plan: x has shape {tuple(x.shape)}, expected [{T}, D]")
        row_bytes = x.shape[1] * x.element_size()
        if row_bytes % 16:
            raise KernelError(f"moe_plan: rows of {row_bytes} bytes cannot be gathered 16 bytes at a time")
        gathered = torch.empty((pairs, x.shape[1]), dtype=x.dtype, device=dev)
    _call("q6k_moe_plan", _ptr(sel_e), _i(pairs), _i(k), _i(E), _i(live), _ptr(scratch), _ptr(offsets), _ptr(pair_row), _ptr(row_token), _i(bm),
          _ptr(tile_group), _ptr(tile_row0), _ptr(num_tiles), _i(max_tiles), _ptr(x), _ptr(gathered), _i(row_bytes), _stream())
    plan = (offsets, pair_row, row_token, (offsets, tile_group, tile_row0, num_tiles))
    return plan if x is None else plan + (gathered,)


# --------------------------------------------------------------------------- sampling
def argmax(logits: torch.Tensor, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """int32 [rows]; ties go to the lower id.  `out`: an int32 buffer of at least `rows` entries to write into."""
    _need(logits, "logits", torch.float32)
    rows, V = logits.shape
    if out is None:
        out = torch.empty(rows, dtype=torch.int32, device=logits.device)
    else:
        _need(out, "out", torch.int32)
        if out.numel() < rows:
            raise KernelError(f"argmax: the output buffer holds {out.numel()} ids, {rows} rows are asked for")
        out = out[:rows]
    lib = library()
    lib.q6k_argmax_scratch_ints.restype = ctypes.c_int
    scratch = torch.empty(lib.q6k_argmax_scratch_ints(_i(rows), _i(V)), dtype=torch.int32, device=logits.device)
    _call("q6k_argmax", _ptr(logits), _i(rows), _i(V), _ptr(out), _ptr(scratch), _stream())
    return out


def row_logsumexp(logits: torch.Tensor, target: Optional[torch.Tensor] = None):
    """log(sum(exp(row))) of every row, FP32 [rows]; with target (int32 [rows]) also each row's logit at its target."""
    _need(logits, "logits", torch.float32)
    rows, V = logits.shape
    lse = torch.empty(rows, dtype=torch.float32, device=logits.device)
    picked = None
    if target is not None:
        _need(target, "target", torch.int32, (rows,))
        picked = torch.empty(rows, dtype=torch.float32, device=logits.device)
    _call("q6k_row_lse", _ptr(logits), _i(rows), _i(V), _ptr(target), _ptr(lse), _ptr(picked), _stream())
    return lse if target is None else (lse, picked)


def sample_pool(ids: torch.Tensor, vals: torch.Tensor, rows: torch.Tensor, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """One token per row from the sorted pools topk_pool made, chosen on the device with the
    host sampler's arithmetic (no penalties).  rows: int32 [n, 8] on the device, per row the
    32-byte record {int32 candidates, int32 top_k, float32 temperature, top_p, min_p, unused,
    float64 uniform}; a row with no candidates keeps what `out` held."""
    _need(ids, "ids", torch.int32)
    n, K = ids.shape
    _need(vals, "vals", torch.float32, (n, K))
    _need(rows, "rows", torch.int32, (n, 8))
    if out is None:
        out = torch.empty(n, dtype=torch.int32, device=ids.device)
    else:
        _need(out, "out", torch.int32)
        if out.numel() < n:
            raise KernelError(f"sample_pool: out holds {out.numel()} ids, {n} rows are sampled")
    _call("q6k_sample_pool", _ptr(ids), _ptr(vals), _i(n), _i(K), _ptr(rows), _ptr(out), _stream())
    return out[:n]


def topk_pool(logits: torch.Tensor, k: int):
    """(ids int32 [rows, k], vals float32 [rows, k]) sorted by (logit descending, id ascending); k <= 256."""
    _need(logits, "logits", torch.float32)
    rows, V = logits.shape
    ids = torch.empty((rows, k), dtype=torch.int32, device=logits.device)
    vals = torch.empty((rows, k), dtype=torch.float32, device=logits.device)
    _call("q6k_topk_pool", _ptr(logits), _i(rows), _i(V), _i(k), _ptr(ids), _ptr(vals), _stream())
    return ids, vals


# --------------------------------------------------------------------------- layer norm, selective scan, flexible attention
def layernorm(h: torch.Tensor, w: Optional[torch.Tensor], b: Optional[torch.Tensor], eps: float, out_dtype: torch.dtype,
              rows: Optional[torch.Tensor] = None, after=None, extra: Optional[torch.Tensor] = None, mixture=None, replace=None,
              raw: Optional[torch.Tensor] = None) -> Optional[torch.Tensor]:
    """Layer norm with weight and bias on the FP32 stream h [T, D], up to three steps in one pass over each row:
    after = (y, wa, ba): h += LN(u; wa, ba) first (y FP32 [T, D] or [slices, T, D] partial sums added in order, or None), or
    replace = (y, vec): h = u + vec (vec FP32 [D] or None); extra (FP32 like h): h += extra next; w, b: the result LN(h; w, b)
    in out_dtype (None: no result, h is only updated), or raw: a [T, D] buffer in out_dtype (rows may lie apart) that takes the
    stream as it then stands.  u is y, or with mixture = (py, pair_row, pw, x, xw, gate), each but py optional,
    gate[t] * y[t] + sum_s pw[t, s] * py[row] (rows as in `combine`; a row of weight zero is not read) + xw[t] * x[t] (x [T, D] in
    out_dtype).  rows: int32 row numbers whose result is wanted; h then stays as it is."""
    _need(h, "h", torch.float32)
    T, D = h.shape
    R = T if rows is None else rows.numel()
    y = wa = ba = vec = None
    splits, stride = 1, 0
    if after is not None and replace is not None:
        raise KernelError("layernorm: the stream is added to or replaced, not both")
    if after is not None:
        y, wa, ba = after
        _need(wa, "wa", torch.float32, (D,))
        _need(ba, "ba", torch.float32, (D,))
    if replace is not None:
        y, vec = replace
        if vec is not None:
            _need(vec, "vec", torch.float32, (D,))
    if y is not None:
        _need(y, "y", torch.float32)
        if y.dim() == 3:
            splits, stride = y.shape[0], y.shape[1] * y.shape[2]
        if tuple(y.shape[-2:]) != (T, D):
            raise KernelError("layernorm: the sublayer's result does not match h")
    py = pair_row = pw = x = xw = gate = None
    S = 0
    if mixture is not None:
        py, pair_row, pw, x, xw, gate = mixture
        if after is None and replace is None:
            raise KernelError("layernorm: routed rows without the norm they pass")
        if py is not None:
            _need(py, "routed rows", torch.float32)
            _need(pw, "weights", torch.float32)
            S = pw.shape[1]
            if pair_row is not None:
                _need(pair_row, "pair_row", torch.int32)
            if pw.shape[0] != T or py.shape[1] != D or py.shape[0] < T * S or (pair_row is not None and pair_row.numel() != T * S):
                raise KernelError("layernorm: the routed rows do not match h")
        if x is not None:
            _need(x, "x", out_dtype, (T, D))
            _need(xw, "xw", torch.float32, (T,))
        if gate is not None:
            _need(gate, "gate", torch.float32, (T,))
    if extra is not None:
        _need(extra, "extra", torch.float32, (T, D))
    if rows is not None:
        _need(rows, "rows", torch.int32)
    out, ldo = None, D
    if w is not None:
        _need(w, "w", torch.float32, (D,))
        _need(b, "b", torch.float32, (D,))
        out = torch.empty((R, D), dtype=out_dtype, device=h.device)
    elif raw is not None:
        if raw.dtype != out_dtype or tuple(raw.shape) != (R, D) or raw.stride(1) != 1 or not raw.is_cuda:
            raise KernelError(f"layernorm: the buffer for the stream must be [{R}, {D}] in {out_dtype}")
        out, ldo = raw, raw.stride(0)
    _call("q6k_layernorm", _ptr(h), _ptr(y), _i(splits), _ll(stride), _ptr(gate), _ptr(py), _ptr(pair_row), _ptr(pw), _i(S), _ptr(x), _ptr(xw),
          _ptr(wa), _ptr(ba), _i(1 if replace is not None else 0), _ptr(vec), _ptr(extra), _ptr(w), _ptr(b), _ptr(rows), _ptr(out), _ll(ldo), _i(R), _i(D),
          _f(eps), _i(dtype_code(out_dtype)), _stream())
    return out


def conv_silu(x: torch.Tensor, channels: int, w: torch.Tensor, bias: torch.Tensor, tail: torch.Tensor, req_of_token: torch.Tensor,
              q_start: torch.Tensor, slot_ids: torch.Tensor, out_dtype: torch.dtype) -> torch.Tensor:
    """out[t, c] = out_dtype(silu(bias[c] + sum_k w[c, k] * x[t - (taps-1-k), c])) per request; inputs before a portion
    come from tail [slots, taps-1, C] (the last inputs of the request's earlier portions, zeros at its start)."""
    _need(x, "x", torch.float32)
    T = x.shape[0]
    taps = w.shape[1]
    _need(w, "w", torch.float32, (channels, taps))
    _need(bias, "bias", torch.float32, (channels,))
    _need(tail, "tail", torch.float32)
    if tuple(tail.shape[1:]) != (max(taps - 1, 0), channels) or x.shape[1] < channels:
        raise KernelError("conv_silu: shapes disagree")
    out = torch.empty((T, channels), dtype=out_dtype, device=x.device)
    _call("q6k_conv_silu", _ptr(x), _i(x.stride(0)), _ptr(w), _ptr(bias), _ptr(tail), _ptr(req_of_token), _ptr(q_start), _ptr(slot_ids),
          _ptr(out), _i(T), _i(channels), _i(taps), _i(dtype_code(out_dtype)), _stream())
    return out


def cast_columns(src: torch.Tensor, col0: int, n: int, out_dtype: torch.dtype) -> torch.Tensor:
    """out_dtype(src[:, col0:col0 + n]) as a contiguous matrix."""
    _need(src, "src", torch.float32)
    out = torch.empty((src.shape[0], n), dtype=out_dtype, device=src.device)
    _call("q6k_cast_columns", _ptr(src), _i(src.stride(0)), _i(col0), _i(n), _ptr(out), _i(src.shape[0]), _i(dtype_code(out_dtype)), _stream())
    return out


def selective_scan(u: torch.Tensor, dt_raw: torch.Tensor, dt_bias: torch.Tensor, proj: torch.Tensor, b_col: int, c_col: int,
                   A: torch.Tensor, D: torch.Tensor, xz: torch.Tensor, z_col: int, state: torch.Tensor, tail: torch.Tensor,
                   q_start: torch.Tensor, slot_ids: torch.Tensor, R: int, segments=None) -> torch.Tensor:
    """The selective-scan recurrence over each request's tokens in order, from and into the request's state slot:
    dt = softplus(dt_raw + dt_bias); S <- exp(dt A) S + dt u B; y = (S . C + D u) * silu(z).  u [T, C] (operand dtype),
    dt_raw FP32 [T, C], proj FP32 [T, *] holding B and C (N columns each from b_col, c_col), A FP32 [C, N], xz FP32 [T, *]
    holding the convolution's inputs (columns 0..) and z (columns z_col..), state FP32 [slots, C, N], tail FP32
    [slots, taps-1, C] (moved on to the portion's end).  Returns [T, C] in u's dtype.
    segments = (most segments of any request, seg_base int32 [R] on the device, segments in all) from
    selective_scan_segments(q_lens): long portions are then walked by several blocks each (two launches)."""
    _need(u, "u")
    T, C = u.shape
    N = A.shape[1]
    _need(dt_raw, "dt_raw", torch.float32, (T, C))
    _need(dt_bias, "dt_bias", torch.float32, (C,))
    _need(proj, "proj", torch.float32)
    _need(A, "A", torch.float32, (C, N))
    _need(D, "D", torch.float32, (C,))
    _need(xz, "xz", torch.float32)
    _need(state, "state", torch.float32)
    _need(tail, "tail", torch.float32)
    taps = tail.shape[1] + 1
    if tuple(state.shape[1:]) != (C, N) or tail.shape[2] != C or tail.shape[0] != state.shape[0]:
        raise KernelError("selective_scan: state shapes disagree")
    out = torch.empty((T, C), dtype=u.dtype, device=u.device)
    most, seg_base, slots, ws = 1, None, 0, None
    if segments is not None and segments[0] > 1:
        most, seg_base, slots = segments
        lib = library()
        lib.q6k_selective_scan_workspace.restype = ctypes.c_longlong
        ws = _workspace(4 * lib.q6k_selective_scan_workspace(_i(slots), _i(R), _i(C), _i(N)), u.device, "scan")
    _call("q6k_selective_scan", _ptr(u), _ptr(dt_raw), _ptr(dt_bias), _ptr(proj), _i(proj.stride(0)), _i(b_col), _i(c_col), _ptr(A), _ptr(D),
          _ptr(xz), _i(xz.stride(0)), _i(z_col), _ptr(state), _ptr(tail), _ptr(q_start), _ptr(slot_ids), _ptr(out), _i(R), _i(C), _i(N),
          _i(taps), _i(dtype_code(u.dtype)), _i(most), _ptr(seg_base), _i(slots), _ptr(ws), _stream())
    return out


def selective_scan_segments(q_lens, device):
    """(most segments of any request, first segment slot of each request as int32 on the device, segments in all) for a
    step whose requests bring q_lens tokens; (1, None, 0) when no request has more than one segment."""
    lib = library()
    lib.q6k_selective_scan_segment.restype = ctypes.c_int
    seg = lib.q6k_selective_scan_segment()
    counts = [-(-n // seg) for n in q_lens]
    if max(counts, default=0) <= 1:
        return 1, None, 0
    base, at = [], 0
    for n in counts:
        base.append(at)
        at += n
    return max(counts), torch.tensor(base, dtype=torch.int32).to(device, non_blocking=True), at


def qkv_pages(qkv: torch.Tensor, Hq: int, Hkv: int, hd: int, vd: int, q_norm, k_norm, eps: float, rotary, positions: torch.Tensor,
              req_of_token: torch.Tensor, block_table: Optional[torch.Tensor], page_size: int, k_pages: Optional[torch.Tensor],
              v_pages: Optional[torch.Tensor], out_dtype: torch.dtype, v_heads: Optional[int] = None, bias: Optional[torch.Tensor] = None,
              values_are_keys: bool = False, value_norm: bool = False) -> torch.Tensor:
    """qk_prep for keys and values of different widths: qkv FP32 [T, Hq hd + Hkv hd + Hv vd] (or split-K slices of it);
    q -> [T, Hq, hd]; k -> pages [Hkv, P, page, hd]; v -> pages [Hv, P, page, vd].  v_heads: Hv, if it is not Hkv.
    bias: FP32, one entry per column of a row, added to the summed product first.  values_are_keys: the rows hold q and k
    only, and a key's value is the key as projected (bias included, before norm and rotation).  value_norm: a head's value is
    divided by its root mean square (eps, no weight) before it is stored."""
    Hv = v_heads or Hkv
    v_cols = 0 if values_are_keys else Hv * vd
    if bias is not None:
        _need(bias, "bias", torch.float32)
    _need(qkv, "qkv", torch.float32)
    splits, split_stride = 1, 0
    if qkv.dim() == 3:
        splits, split_stride = qkv.shape[0], qkv.shape[1] * qkv.shape[2]
        qkv = qkv[0]
    T = qkv.shape[0]
    write = k_pages is not None
    if write:
        _need(k_pages, "k_pages", out_dtype)
        _need(v_pages, "v_pages", out_dtype)
        _need(block_table, "block_table", torch.int32)
        if (tuple(k_pages.shape[2:]) != (page_size, hd) or tuple(v_pages.shape[2:]) != (page_size, vd) or k_pages.shape[0] != Hkv
                or v_pages.shape[0] != Hv or v_pages.shape[1] != k_pages.shape[1]):
            raise KernelError("qkv_pages: the pages do not match the heads")
    if qkv.shape[1] < Hq * hd + (Hkv * hd + v_cols if write else 0) or (bias is not None and bias.numel() < Hq * hd + (Hkv * hd + v_cols if write else 0)):
        raise KernelError("qkv_pages: qkv rows are too short")
    inv_freq, rotary_dim, neighbours = rotary if rotary is not None else (None, 0, False)
    q = torch.empty((T, Hq, hd), dtype=out_dtype, device=qkv.device)
    _call("q6k_qkv_pages", _ptr(qkv), _i(qkv.stride(0)), _i(splits), _ll(split_stride), _i(T), _i(Hq), _i(Hkv), _i(hd), _i(vd), _ptr(q_norm),
          _ptr(k_norm), _f(eps), _ptr(inv_freq), _i(rotary_dim), _i(1 if neighbours else 0), _ptr(positions), _ptr(req_of_token),
          _ptr(block_table), _i(block_table.shape[1] if block_table is not None else 1), _i(page_size),
          _i(k_pages.shape[1] if write else 0), _ptr(q), _ptr(k_pages), _ptr(v_pages), _i(1 if write else 0),
          _i(dtype_code(out_dtype)), _i(Hv), _ptr(bias), _i(1 if values_are_keys else 0), _i(1 if value_norm else 0), _stream())
    return q


def latent_prep(x: torch.Tensor, H: int, dim: int, rd: int, rank: int, c_weight: Optional[torch.Tensor], eps: float,
                inv_freq: Optional[torch.Tensor], turn: int, positions: torch.Tensor, req_of_token: torch.Tensor, block_table: torch.Tensor,
                page_size: int, pages: torch.Tensor, neighbours: bool = False, write: bool = True, latent=None):
    """x FP32 [T, H (dim + rd) + rank + rd] -> (qn [H, T, dim], qr [H, T, rd]) in the pages' dtype, and the token's row
    [RMS-normed latent | rotated shared key part] into pages [1, P, page, rank + rd].  neighbours: the rotation pairs
    dimension 2i with 2i+1 instead of i with i + turn/2.  write=False: a layer that reads another layer's pages; x then
    holds the queries only and nothing is written.  latent = (rows FP32 [T, *], column): the latent and the shared key part
    are read there; x then holds the queries only."""
    _need(x, "x", torch.float32)
    T = x.shape[0]
    xc, col = latent if latent is not None else (x, H * (dim + rd))
    _need(xc, "latent rows", torch.float32)
    if x.shape[1] < H * (dim + rd) or (write and (xc.shape[0] != T or xc.shape[1] < col + rank + rd)) or tuple(pages.shape[2:]) != (page_size, rank + rd) or pages.shape[0] != 1:
        raise KernelError("latent_prep: shapes disagree")
    _need(pages, "pages")
    if write:
        _need(c_weight, "c_weight", torch.float32, (rank,))
    qn = torch.empty((H, T, dim), dtype=pages.dtype, device=x.device)
    qr = torch.empty((H, T, rd), dtype=pages.dtype, device=x.device)
    _call("q6k_latent_prep", _ptr(x), _i(x.stride(0)), ctypes.c_void_p(xc.data_ptr() + 4 * col if write else 0), _i(xc.stride(0)), _i(T), _i(H), _i(dim), _i(rd), _i(rank), _ptr(c_weight if write else None), _f(eps),
          _ptr(inv_freq), _i(turn), _i(1 if neighbours else 0), _ptr(positions), _ptr(req_of_token), _ptr(block_table), _i(block_table.shape[1]),
          _i(page_size), _ptr(qn), _ptr(qr), _ptr(pages if write else None), _i(dtype_code(pages.dtype)), _stream())
    return qn, qr


def heads_to_rows(src: torch.Tensor, H: int, out_dtype: torch.dtype) -> torch.Tensor:
    """FP32 [H * T, n] (head-major) -> out_dtype [T, H * n]."""
    _need(src, "src", torch.float32)
    T, n = src.shape[0] // H, src.shape[1]
    out = torch.empty((T, H * n), dtype=out_dtype, device=src.device)
    _call("q6k_heads_to_rows", _ptr(src), _ptr(out), _i(H), _i(T), _i(n), _i(dtype_code(out_dtype)), _stream())
    return out


def attention_flex(q_f32: Optional[torch.Tensor], q: Optional[torch.Tensor], head_major: bool, k_pages: torch.Tensor, v_pages: torch.Tensor,
                   block_table: torch.Tensor, req_of_token: torch.Tensor, positions: torch.Tensor, H: int, scale: float,
                   window: Optional[int] = None, chunk: Optional[int] = None, talk: Optional[torch.Tensor] = None,
                   out_head_major: bool = False, tiles=None, max_context: int = 0, sinks: Optional[torch.Tensor] = None,
                   softcap: float = 0.0, maps: int = 1, out_f32: bool = False) -> torch.Tensor:
    """Causal attention of every row over its request's pages, for any key and value widths.  A query row is the FP32
    part q_f32 [H*T or T*H rows, da] followed by q [rows, db] in the pages' dtype (either may be None); rows are head-major
    (h T + t) or token-major.  k_pages [Hkv, P, page, dk]; v_pages [Hkv, P, page, dv], possibly a view into k_pages (the
    last axis contiguous, the others with k's strides).  window: only the last `window` keys; chunk: only keys of the
    position's own block of `chunk` positions; talk FP32 [H, H]: the heads' softmax weights are mixed by it before the
    values; sinks FP32 [H]: exp(sinks[h]) joins head h's softmax denominator (it has no key and no value, is not scaled
    and counts once).  softcap > 0: a scaled score s becomes softcap * tanh(s / softcap).  maps > 1: every head attends
    `maps` times, each time with queries and keys of its own, over the same values: H counts heads x maps query rows per
    token (a head's maps side by side), k_pages holds groups x maps key heads (a group's maps side by side) and v_pages one
    head per group; the result has one row per (head, map).  out_f32: the result leaves as FP32 whatever the pages hold.
    Returns [H, T, dv] (out_head_major) or [T, H dv].
    tiles = (first row, token count, number) of row tiles of attention_flex_tile_tokens(H, Hkv) tokens of one request
    each, with max_context the largest position + 1 of the step: bfloat16 pages then go to the tensor-core kernel where
    it takes the shapes; with few tiles it splits the keys into fixed ranges and merges them."""
    da = q_f32.shape[-1] if q_f32 is not None else 0
    db = q.shape[-1] if q is not None else 0
    rows = (q_f32 if q_f32 is not None else q).numel() // (da if q_f32 is not None else db)
    T = rows // H
    if q_f32 is not None:
        _need(q_f32, "q_f32", torch.float32)
    if q is not None:
        _need(q, "q", k_pages.dtype)
    Hkv, num_pages, page_size, dk = k_pages.shape
    dv = v_pages.shape[-1]
    if maps < 1 or Hkv % maps or (talk is not None and (maps > 1 or softcap or out_f32)):
        raise KernelError(f"attention_flex: {maps} maps over {Hkv} key heads (mixed heads take one map, no cap, no FP32 result)")
    if (da + db != dk or v_pages.dtype != k_pages.dtype or tuple(v_pages.shape[1:3]) != tuple(k_pages.shape[1:3])
            or v_pages.shape[0] * maps != Hkv):
        raise KernelError(f"attention_flex: a query of {da}+{db} against pages {tuple(k_pages.shape)} / {tuple(v_pages.shape)}")
    for nm, p in (("k_pages", k_pages), ("v_pages", v_pages)):
        if not p.is_cuda or p.stride(3) != 1 or p.stride(1) != page_size * p.stride(2):
            raise KernelError(f"attention_flex: {nm} has strides {p.stride()}")
    if talk is not None:
        _need(talk, "talk", torch.float32, (H, H))
    if sinks is not None:
        _need(sinks, "sinks", torch.float32, (H,))
    out = torch.empty((H, T, dv) if out_head_major else (T, H * dv), dtype=torch.float32 if out_f32 else k_pages.dtype, device=k_pages.device)
    as_f32 = out if out_f32 and k_pages.dtype != torch.float32 else None      # FP32 pages: the kernel's own result type
    shared_v = v_pages.data_ptr() == k_pages.data_ptr() and v_pages.stride() == k_pages.stride()
    if (tiles is not None and k_pages.dtype == torch.bfloat16 and not (talk is not None and out_head_major)
            and attention_flex_mma_supported(H, Hkv, dk, dv, k_pages.stride(2), v_pages.stride(2), db, shared_v)):
        tok0, ntok, n_tiles = tiles
        nsplit, split_keys, ws = 1, 0, None
        ctas = n_tiles * Hkv
        if talk is not None:                     # every head's weights against every KV head's values, then the mixture
            lib = library()
            lib.q6k_attention_flex_mma_talk_workspace.restype = ctypes.c_longlong
            ws = _workspace(lib.q6k_attention_flex_mma_talk_workspace(_i(T), _i(H), _i(Hkv), _i(dv)), k_pages.device, "flex")
        elif ctas < 120 and not chunk and max_context > 256:     # few row tiles: fixed key ranges over more CTAs
            want = max(1, 296 // ctas)
            # under a window a tile sees its window and its own tokens: ranges sized for that span (the ranges that lie
            # outside it cost a block that finds no key), and no more than 128 of them
            span = min(max_context, window + attention_flex_tile_tokens(H, Hkv)) if window else max_context
            split_keys = max(256, (-(-span // want) + 63) // 64 * 64, (-(-max_context // 128) + 63) // 64 * 64)
            nsplit = -(-max_context // split_keys)
            if nsplit > 1:
                lib = library()
                lib.q6k_attention_flex_mma_workspace.restype = ctypes.c_longlong
                ws = _workspace(lib.q6k_attention_flex_mma_workspace(_i(T), _i(H), _i(dv), _i(nsplit)), k_pages.device, "flex")
        _call("q6k_attention_flex_mma", _ptr(q_f32), _i(da), _ptr(q), _i(db), _i(1 if head_major else 0), _ptr(k_pages),
              _ll(k_pages.stride(0)), _i(k_pages.stride(2)), _ptr(v_pages), _ll(v_pages.stride(0)), _i(v_pages.stride(2)), _i(dv),
              _ptr(block_table), _i(block_table.shape[1]), _i(page_size), _ptr(req_of_token), _ptr(positions), _ptr(tok0), _ptr(ntok),
              _i(n_tiles), _i(window or 0), _i(chunk or 0), _f(scale), _ptr(out), _i(1 if out_head_major else 0), _i(T), _i(H), _i(Hkv),
              _i(nsplit), _i(split_keys), _ptr(ws), _ptr(talk), _ptr(sinks), _f(softcap), _i(maps), _ptr(as_f32), _stream())
        return out
    _call("q6k_attention_flex", _ptr(q_f32), _i(da), _ptr(q), _i(db), _i(1 if head_major else 0), _ptr(k_pages), _ll(k_pages.stride(0)),
          _i(k_pages.stride(2)), _ptr(v_pages), _ll(v_pages.stride(0)), _i(v_pages.stride(2)), _i(dv), _ptr(block_table),
          _i(block_table.shape[1]), _i(page_size), _ptr(req_of_token), _ptr(positions), _i(window or 0), _i(chunk or 0), _f(scale),
          _ptr(talk), _ptr(sinks), _ptr(out), _i(1 if out_head_major else 0), _i(T), _i(H), _i(Hkv), _i(dtype_code(k_pages.dtype)),
          _f(softcap), _i(maps), _ptr(as_f32), _stream())
    return out


def map_difference(a: torch.Tensor, H: int, dv: int, weight: float, eps: float, mult: float, out_dtype: torch.dtype) -> torch.Tensor:
    """The two maps of every head combined: a FP32 [T, H 2 dv] (a head's maps side by side) -> [T, H dv] in out_dtype,
    o = a1 - weight a2, then o / sqrt(mean(o^2) + eps) * mult over each head's dv values."""
    _need(a, "a", torch.float32)
    T = a.shape[0]
    if a.dim() != 2 or a.shape[1] != H * 2 * dv:
        raise KernelError("map_difference: shapes disagree")
    out = torch.empty((T, H * dv), dtype=out_dtype, device=a.device)
    _call("q6k_map_difference", _ptr(a), _ptr(out), _i(T), _i(H), _i(dv), _f(weight), _f(eps), _f(mult), _i(dtype_code(out_dtype)), _stream())
    return out


@functools.lru_cache(maxsize=None)
def attention_flex_mma_supported(H: int, Hkv: int, dk: int, dv: int, k_ld: int, v_ld: int, db: int, shared_v: bool) -> bool:
    lib = library()
    lib.q6k_attention_flex_mma_supported.restype = ctypes.c_int
    return bool(lib.q6k_attention_flex_mma_supported(_i(H), _i(Hkv), _i(dk), _i(dv), _i(k_ld), _i(v_ld), _i(db), _i(1 if shared_v else 0)))


@functools.lru_cache(maxsize=None)
def attention_flex_tile_tokens(H: int, Hkv: int) -> int:
    """Tokens of one request in a row tile of the tensor-core flexible attention kernel."""
    lib = library()
    lib.q6k_attention_flex_mma_tile_tokens.restype = ctypes.c_int
    return lib.q6k_attention_flex_mma_tile_tokens(_i(H), _i(Hkv))


# --------------------------------------------------------------------------- short convolution, gated delta rule
def _slices_of(x: torch.Tensor):
    """(slices, stride between slices in floats, rows, columns) of an FP32 [T, N] matrix or [slices, T, N] partial sums."""
    if x.dim() == 3:
        return x.shape[0], x.shape[1] * x.shape[2], x.shape[1], x.shape[2]
    return 1, 0, x.shape[0], x.shape[1]


def short_conv(x: torch.Tensor, channels: int, w: torch.Tensor, bias: Optional[torch.Tensor], tail: torch.Tensor, req_of_token: torch.Tensor,
               q_start: torch.Tensor, slot_ids: torch.Tensor, R: int, act: Optional[str] = None, copy_to: Optional[int] = None) -> torch.Tensor:
    """FP32 out[t, c] = act(sum_j w[c, j] * p[t - taps + 1 + j, c]) per request for the first `channels` columns of x, where
    p = x (+ bias) and the rows before a portion come from tail [slots, taps-1, channels] (the last projected values of the
    request's earlier portions, zeros at its start); the tail is then moved on by this step's rows.  x: FP32 [T, N] or
    [slices, T, N] partial sums (added in order).  Columns channels..copy_to of x are copied into the result (summed).
    act: None or "silu"."""
    _need(x, "x", torch.float32)
    slices, stride, T, N = _slices_of(x)
    taps = w.shape[1]
    _need(w, "w", torch.float32, (channels, taps))
    if bias is not None:
        _need(bias, "bias", torch.float32, (channels,))
    _need(tail, "tail", torch.float32)
    copy_to = channels if copy_to is None else copy_to
    if tuple(tail.shape[1:]) != (max(taps - 1, 0), channels) or N < copy_to or copy_to < channels:
        raise KernelError("short_conv: shapes disagree")
    if act not in (None, "silu"):
        raise KernelError(f"short_conv: unknown activation {act!r}")
    out = torch.empty((T, copy_to), dtype=torch.float32, device=x.device)
    _call("q6k_short_conv", _ptr(x), _i(slices), _ll(stride), _i(N), _ptr(bias), _ptr(w), _ptr(tail), _ptr(req_of_token), _ptr(q_start),
          _ptr(slot_ids), _ptr(out), _i(copy_to), _i(T), _i(channels), _i(copy_to), _i(taps), _i(1 if act == "silu" else 0), _stream())
    if taps > 1:
        _call("q6k_short_conv_tail", _ptr(x), _i(slices), _ll(stride), _i(N), _ptr(bias), _ptr(tail), _ptr(q_start), _ptr(slot_ids), _i(R),
              _i(channels), _i(taps), _stream())
    return out


@functools.lru_cache(maxsize=None)
def gated_delta_max_dim() -> int:
    lib = library()
    lib.q6k_gated_delta_max_dim.restype = ctypes.c_int
    return lib.q6k_gated_delta_max_dim()


def gated_delta(u: torch.Tensor, p: torch.Tensor, b_col: int, a_col: int, A_log: torch.Tensor, dt_bias: torch.Tensor, state: torch.Tensor,
                q_start: torch.Tensor, slot_ids: torch.Tensor, R: int, H: int, G: int, dk: int, dv: int, prepare: bool = False) -> torch.Tensor:
    """The gated delta rule over the step's rows, request by request, from and into state [slots, H, dv, dk] (FP32):
    S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q, with unit q (times dk^-1/2) and k.  u: FP32 [T, >= 2 G dk + H dv]
    = [q | k | v]; p: FP32 rows holding the H beta logits at b_col and the H decay inputs at a_col.  Returns FP32 o [T, H dv].
    prepare: a kernel of its own first makes every token's unit vectors (in place over q and k in u), beta, decay and k . q,
    and the recurrence fetches a tile of tokens while it walks the one before (for steps with long portions); else the
    recurrence makes them itself.  The results are the same bit for bit."""
    _need(u, "u", torch.float32)
    _need(p, "p", torch.float32)
    _need(A_log, "A_log", torch.float32, (H,))
    _need(dt_bias, "dt_bias", torch.float32, (H,))
    _need(state, "state", torch.float32)
    T = u.shape[0]
    if tuple(state.shape[1:]) != (H, dv, dk) or u.shape[1] < 2 * G * dk + H * dv or p.shape[0] != T or max(b_col, a_col) + H > p.shape[1]:
        raise KernelError("gated_delta: shapes disagree")
    o = torch.empty((T, H * dv), dtype=torch.float32, device=u.device)
    bg = torch.empty((T, 2 * H + G), dtype=torch.float32, device=u.device) if prepare else None
    _call("q6k_gated_delta", _ptr(u), _i(u.stride(0)), _ptr(p), _i(p.stride(0)), _i(b_col), _i(a_col), _ptr(A_log), _ptr(dt_bias), _ptr(bg),
          _ptr(state), _ptr(q_start), _ptr(slot_ids), _ptr(o), _i(T), _i(R), _i(H), _i(G), _i(dk), _i(dv), _stream())
    return o


OUT_GATES = {"silu": 0, "sigmoid": 1}


def delta_out(o: torch.Tensor, p: torch.Tensor, g_col: int, w: torch.Tensor, eps: float, H: int, dv: int, out_dtype: torch.dtype,
              gate: str = "silu") -> torch.Tensor:
    """out_dtype(o / rms(o) * w * gate(g)) per (row, head): o FP32 [T, H dv], g in p's columns from g_col on; gate: silu or
    sigmoid.  w: FP32 [dv], shared by the heads, or [H, dv].  With H = 1 and dv the width of all heads together, the heads are
    normed as one vector."""
    if gate not in OUT_GATES:
        raise KernelError(f"delta_out: unknown gate {gate!r}; known: {', '.join(OUT_GATES)}")
    _need(o, "o", torch.float32)
    _need(p, "p", torch.float32)
    _need(w, "w", torch.float32, (dv,) if w.dim() == 1 else (H, dv))
    T = o.shape[0]
    if o.shape[1] != H * dv or p.shape[0] != T or g_col + H * dv > p.shape[1]:
        raise KernelError("delta_out: shapes disagree")
    out = torch.empty((T, H * dv), dtype=out_dtype, device=o.device)
    _call("q6k_delta_out", _ptr(o), _ptr(p), _i(p.stride(0)), _i(g_col), _ptr(w), _f(eps), _ptr(out), _i(T), _i(H), _i(dv), _i(dtype_code(out_dtype)),
          _i(OUT_GATES[gate]), _i(dv if w.dim() == 2 else 0), _stream())
    return out


# --------------------------------------------------------------------------- a block of sublayers side by side
def scaled_add_norm(h: torch.Tensor, a: Optional[torch.Tensor], b: Optional[torch.Tensor], weighted, scale: float, w1: Optional[torch.Tensor],
                    w2: Optional[torch.Tensor], eps: float, out_dtype: torch.dtype, rows: Optional[torch.Tensor] = None,
                    bias: Optional[torch.Tensor] = None):
    """h += scale * (a + bias + b + weighted rows) in place (each optional; a and b FP32 [T, D] or [slices, T, D] partial sums,
    bias FP32 [D] the same for every row, weighted = (y, pair_row, weights) as in `combine`), then (out1, out2) = h * rsqrt(mean(h^2) + eps) * (w1, w2) in out_dtype for the
    weights given (None otherwise).  rows: normalise these rows only (no add then)."""
    _need(h, "h", torch.float32)
    T, D = h.shape
    stride = T * D
    counts = []
    for name, t in (("a", a), ("b", b)):
        if t is None:
            counts.append(1)
            continue
        _need(t, name, torch.float32)
        if tuple(t.shape[-2:]) != (T, D):
            raise KernelError(f"scaled_add_norm: {name} does not match h")
        counts.append(t.shape[0] if t.dim() == 3 else 1)
    y = pair_row = pair_w = None
    S = 0
    if weighted is not None:
        y, pair_row, pair_w = weighted
        S = pair_w.shape[1]
        _need(y, "weighted rows", torch.float32)
        _need(pair_w, "weights", torch.float32)
        if pair_row is not None:
            _need(pair_row, "pair_row", torch.int32)
        if pair_w.shape[0] != T or y.shape[1] != D or y.shape[0] < T * S:
            raise KernelError("scaled_add_norm: the weighted rows do not match h")
    R = T if rows is None else rows.numel()
    outs = []
    for w in (w1, w2):
        if w is not None:
            _need(w, "w", torch.float32, (D,))
            outs.append(torch.empty((R, D), dtype=out_dtype, device=h.device))
        else:
            outs.append(None)
    if rows is not None:
        _need(rows, "rows", torch.int32)
    if bias is not None:
        _need(bias, "bias", torch.float32, (D,))
    _call("q6k_scaled_add_norm", _ptr(h), _ptr(a), _i(counts[0]), _ptr(b), _i(counts[1]), _ll(stride), _ptr(y), _ptr(pair_row), _ptr(pair_w), _i(S),
          _f(scale), _ptr(rows), _ptr(w1), _ptr(outs[0]), _ptr(w2), _ptr(outs[1]), _f(eps), _i(R), _i(D), _i(dtype_code(out_dtype)), _ptr(bias), _stream())
    return outs[0], outs[1]


def activate(x: torch.Tensor, I: int, gated: bool, act: str, out_dtype: torch.dtype) -> torch.Tensor:
    """out_dtype(act(x[:, :I]) * x[:, I:2 I]) when gated, else out_dtype(act(x[:, :I])); x FP32 [T, N], or [slices, T, N]
    partial sums (added in order).  act: one of ACTIVATIONS, or "tanh"."""
    _need(x, "x", torch.float32)
    slices, stride, T, N = _slices_of(x)
    if act not in ACTIVATIONS and act != "tanh":
        raise KernelError(f"activate: unknown activation {act!r}")
    out = torch.empty((T, I), dtype=out_dtype, device=x.device)
    _call("q6k_activate", _ptr(x), _i(slices), _ll(stride), _i(N), _ptr(out), _i(T), _i(I), _i(1 if gated else 0), _i(3 if act == "tanh" else ACTIVATIONS[act]),
          _i(dtype_code(out_dtype)), _stream())
    return out


def route_biased(logits: torch.Tensor, k: int, bias: Optional[torch.Tensor], scale: float, renorm: bool = True, groups=None, power: int = 1,
                 scoring: str = "sigmoid", group_worth: str = "two", experts: Optional[int] = None, identity: int = 0, gate: bool = False):
    """(sel_e int32 [T, k], sel_w float32 [T, k]): per row the k experts with the largest score + bias (ties to the
    lower index), a score being sigmoid(logit), or softmax over all experts' logits; weights score / (their sum + 1e-20) * scale,
    or score * scale without renorm.
    groups = (count, keep): the experts form `count` equal groups of neighbours, a group's worth is the sum of its two
    largest choice values (group_worth "two") or its largest one ("best"), and only experts of the `keep` groups of most worth
    can be chosen.  power = 2: the weights leave squared.  logits: [T, N] or [slices, T, N] partial sums; the first `experts`
    columns (default all) are the experts'.  identity: the last `identity` of the experts answer their input: their weights
    leave as zero in sel_w, and the row's sum of them is a third result, float32 [T].  gate: sigmoid of column
    `experts` is one more result, float32 [T]."""
    count, keep = groups if groups is not None else (1, 1)
    _need(logits, "logits", torch.float32)
    slices = logits.shape[0] if logits.dim() == 3 else 1
    T, N = logits.shape[-2:]
    E = N if experts is None else int(experts)
    if scoring not in ("sigmoid", "softmax") or group_worth not in ("two", "best"):
        raise KernelError(f"route_biased: unknown scoring {scoring!r} or worth of a group {group_worth!r}")
    if bias is not None:
        _need(bias, "bias", torch.float32, (E,))
    sel_e = torch.empty((T, k), dtype=torch.int32, device=logits.device)
    sel_w = torch.empty((T, k), dtype=torch.float32, device=logits.device)
    id_w = torch.empty(T, dtype=torch.float32, device=logits.device) if identity else None
    gates = torch.empty(T, dtype=torch.float32, device=logits.device) if gate else None
    _call("q6k_route_biased", _ptr(logits), _i(slices), _i(N), _ptr(bias), _f(scale), _i(T), _i(E), _i(k), _ptr(sel_e), _ptr(sel_w),
          _i(1 if renorm else 0), _i(count), _i(keep), _i(power), _i(1 if scoring == "softmax" else 0), _i(1 if group_worth == "best" else 0), _i(identity),
          _ptr(id_w), _ptr(gates), _stream())
    return (sel_e, sel_w) + ((id_w,) if identity else ()) + ((gates,) if gate else ())


# --------------------------------------------------------------------------- sublayers whose results pass a norm before the stream
def add_normed(h: torch.Tensor, y: Optional[torch.Tensor], w: Optional[torch.Tensor], eps: float, out_dtype: Optional[torch.dtype] = None,
               weighted=None) -> Optional[torch.Tensor]:
    """h += (y + weighted rows) / rms(y + weighted rows) * w in place on the FP32 stream h [T, D]; y FP32 [T, D] or
    [slices, T, D] partial sums added in order (or None), weighted = (rows [pairs, D], pair_row [T, S] or None, weights
    [T, S]) as in `combine` (or None).  With neither, nothing is added.  out_dtype: also return the stream as it then
    stands in that dtype (what the next sublayer reads)."""
    _need(h, "h", torch.float32)
    T, D = h.shape
    slices, stride = 1, 0
    if y is not None:
        _need(y, "y", torch.float32)
        slices, stride, rows, cols = _slices_of(y)
        if (rows, cols) != (T, D):
            raise KernelError("add_normed: the sublayer's result does not match the stream")
    py = pair_row = pw = None
    S = 0
    if weighted is not None:
        py, pair_row, pw = weighted
        _need(py, "weighted rows", torch.float32)
        _need(pw, "weights", torch.float32)
        S = pw.shape[1]
        if pair_row is not None:
            _need(pair_row, "pair_row", torch.int32)
        if pw.shape[0] != T or py.shape[1] != D or py.shape[0] < T * S or (pair_row is not None and pair_row.numel() != T * S):
            raise KernelError("add_normed: the weighted rows do not match the stream")
    if y is None and weighted is None and out_dtype is None:
        return None
    if y is not None or weighted is not None:
        _need(w, "w", torch.float32, (D,))
    out = torch.empty((T, D), dtype=out_dtype, device=h.device) if out_dtype is not None else None
    _call("q6k_add_normed", _ptr(h), _ptr(y), _i(slices), _ll(stride), _ptr(py), _ptr(pair_row), _ptr(pw), _i(S), _ptr(w), _f(eps), _ptr(out),
          _i(T), _i(D), _i(dtype_code(out_dtype or torch.float32)), _stream())
    return out


def side_gate(p: torch.Tensor, e: torch.Tensor, col0: int, out_dtype: torch.dtype) -> torch.Tensor:
    """out_dtype(gelu_tanh(p[t, j]) * e[t, col0 + j]): p FP32 [T, n] (or [slices, T, n] partial sums), e FP32 [T, *]."""
    _need(p, "p", torch.float32)
    _need(e, "e", torch.float32)
    slices, stride, T, n = _slices_of(p)
    if e.shape[0] != T or col0 + n > e.shape[1]:
        raise KernelError("side_gate: shapes disagree")
    out = torch.empty((T, n), dtype=out_dtype, device=p.device)
    _call("q6k_side_gate", _ptr(p), _i(slices), _ll(stride), _ptr(e), _i(e.stride(0)), _i(col0), _ptr(out), _i(T), _i(n), _i(dtype_code(out_dtype)),
          _stream())
    return out


# --------------------------------------------------------------------------- retention
@functools.lru_cache(maxsize=None)
def retention_max_dim() -> int:
    lib = library()
    lib.q6k_retention_max_dim.restype = ctypes.c_int
    return lib.q6k_retention_max_dim()


def retention_prep(p: torch.Tensor, H: int, dk: int, q_col: int, k_col: int, rotary, k_scale: float, positions: torch.Tensor,
                   act_cols: int = 0) -> None:
    """In place on p FP32 [T, N]: the row's first act_cols columns pass through silu; then the first rotary_dim entries of
    every head of q (columns q_col...) and k (k_col...) turn by position * inv_freq[pair]; k is then multiplied by k_scale.
    rotary = (inv_freq, rotary_dim, neighbours) or None."""
    _need(p, "p", torch.float32)
    inv_freq, rd, neighbours = rotary if rotary is not None else (None, 0, False)
    if p.dim() != 2 or max(q_col, k_col) + H * dk > p.shape[1]:
        raise KernelError("retention_prep: shapes disagree")
    _call("q6k_retention_prep", _ptr(p), _i(p.stride(0)), _i(p.shape[0]), _i(H), _i(dk), _i(q_col), _i(k_col), _ptr(inv_freq), _i(rd),
          _i(1 if neighbours else 0), _f(k_scale), _ptr(positions), _i(act_cols), _stream())


def retention(p: torch.Tensor, q_col: int, k_col: int, v_col: int, decay: torch.Tensor, state: torch.Tensor, q_start: torch.Tensor,
              slot_ids: torch.Tensor, R: int, H: int, dk: int, dv: int) -> torch.Tensor:
    """Per request and head, in token order: S <- decay[h] S + k v^T, o = S^T q.  p FP32 [T, N] with q, k (prepared) and v
    at their columns; state FP32 [slots, H, dk, dv], updated in place; returns o FP32 [T, H dv]."""
    _need(p, "p", torch.float32)
    _need(decay, "decay", torch.float32, (H,))
    _need(state, "state", torch.float32)
    if tuple(state.shape[1:]) != (H, dk, dv) or p.dim() != 2 or max(q_col, k_col) + H * dk > p.shape[1] or v_col + H * dv > p.shape[1]:
        raise KernelError("retention: shapes disagree")
    o = torch.empty((p.shape[0], H * dv), dtype=torch.float32, device=p.device)
    _call("q6k_retention", _ptr(p), _i(p.stride(0)), _i(q_col), _i(k_col), _i(v_col), _ptr(decay), _ptr(state), _ptr(q_start), _ptr(slot_ids),
          _i(R), _ptr(o), _i(H), _i(dk), _i(dv), _stream())
    return o


def token_shift(x: torch.Tensor, mu: torch.Tensor, prev: torch.Tensor, req_of_token: torch.Tensor, q_start: torch.Tensor,
                slot_ids: torch.Tensor) -> torch.Tensor:
    """out[j, t] = x + (x' - x) mu[j] in x's dtype, x' the row before t in its request: the n mixes of every token with the one
    before it, [n, T, D].  x: [T, D]; mu: FP32 [n, D]; prev: FP32 [slots, D], the last row of the request's earlier portions
    (zeros at its start), moved on to this portion's last row."""
    _need(x, "x")
    T, D = x.shape
    n = mu.shape[0]
    _need(mu, "mu", torch.float32, (n, D))
    _need(prev, "prev", torch.float32)
    if prev.shape[-1] != D:
        raise KernelError("token_shift: the state does not match the rows")
    out = torch.empty((n, T, D), dtype=x.dtype, device=x.device)
    _call("q6k_token_shift", _ptr(x), _ptr(mu), _i(n), _ptr(prev), _ptr(req_of_token), _ptr(q_start), _ptr(slot_ids), _ptr(out), _i(T), _i(D),
          _i(dtype_code(x.dtype)), _stream())
    return out


def time_mix(r: torch.Tensor, k: torch.Tensor, v: torch.Tensor, w: torch.Tensor, w0: torch.Tensor, u: torch.Tensor, state: torch.Tensor,
             q_start: torch.Tensor, slot_ids: torch.Tensor, R: int) -> torch.Tensor:
    """Per request and head, in token order: o = S^T r + (sum_x u[x] k[x] r[x]) v, then S <- diag(exp(-exp(w + w0))) S + k v^T.
    r, k: FP32 [T, H dk]; v: FP32 [T, H dv]; w: FP32 [T, H dk], overwritten by the decays; w0, u: FP32 [H, dk]; state FP32
    [slots, H, dk, dv], updated in place.  Returns FP32 o [T, H dv]."""
    for nm, t in (("r", r), ("k", k), ("v", v), ("w", w), ("w0", w0), ("u", u), ("state", state)):
        _need(t, nm, torch.float32)
    H, dk = u.shape
    dv = state.shape[-1]
    T = r.shape[0]
    if (tuple(state.shape[1:]) != (H, dk, dv) or tuple(r.shape) != (T, H * dk) or k.shape != r.shape or w.shape != r.shape or w0.numel() != H * dk
            or tuple(v.shape) != (T, H * dv) or dv != dk):
        raise KernelError("time_mix: shapes disagree")
    bonus = torch.empty((T, H), dtype=torch.float32, device=r.device)
    _call("q6k_time_mix_prep", _ptr(r), _ptr(k), _i(H * dk), _ptr(w), _ptr(w0), _ptr(u), _ptr(bonus), _i(T), _i(H), _i(dk), _stream())
    o = torch.empty((T, H * dv), dtype=torch.float32, device=r.device)
    _call("q6k_time_mix", _ptr(r), _ptr(k), _ptr(v), _i(H * dk), _ptr(w), _ptr(bonus), _ptr(state), _ptr(q_start), _ptr(slot_ids), _i(R), _ptr(o), _i(H),
          _i(dk), _i(dv), _stream())
    return o


# --------------------------------------------------------------------------- a delta rule with a decay per key channel
@functools.lru_cache(maxsize=None)
def delta_channel_max_dim() -> int:
    lib = library()
    lib.q6k_delta_channel_max_dim.restype = ctypes.c_int
    return lib.q6k_delta_channel_max_dim()


@functools.lru_cache(maxsize=None)
def _delta_channel_scratch(H: int, dk: int) -> int:
    lib = library()
    lib.q6k_delta_channel_scratch.restype = ctypes.c_longlong
    return lib.q6k_delta_channel_scratch(_i(H), _i(dk))


def delta_channel(u: torch.Tensor, p: torch.Tensor, b_col: int, a: torch.Tensor, a_col: int, A_log: torch.Tensor, dt_bias: torch.Tensor,
                  state: torch.Tensor, req_of_token: torch.Tensor, q_start: torch.Tensor, slot_ids: torch.Tensor, R: int, H: int, G: int, dk: int,
                  dv: int, prepare: bool = False, single: bool = False) -> torch.Tensor:
    """gated_delta with one decay per head and key channel: S <- diag(g) S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q with
    g = exp(-exp(A_log[h]) softplus(a + dt_bias)).  a: FP32 [T, *] with the H dk decay inputs from a_col on, dt_bias: FP32
    [H dk]; the rest as in gated_delta.  prepare: a kernel of its own makes what does not depend on the state (steps with long
    portions); else the recurrence makes it itself, with the same results.  single: the caller's word that no request brings more
    than one token."""
    _need(u, "u", torch.float32)
    _need(p, "p", torch.float32)
    _need(a, "a", torch.float32)
    _need(A_log, "A_log", torch.float32, (H,))
    _need(dt_bias, "dt_bias", torch.float32, (H * dk,))
    _need(state, "state", torch.float32)
    T = u.shape[0]
    if (tuple(state.shape[1:]) != (H, dv, dk) or u.shape[1] < 2 * G * dk + H * dv or p.shape[0] != T or b_col + H > p.shape[1] or a.shape[0] != T
            or a_col + H * dk > a.shape[1]):
        raise KernelError("delta_channel: shapes disagree")
    o = torch.empty((T, H * dv), dtype=torch.float32, device=u.device)
    scratch = torch.empty(T * _delta_channel_scratch(H, dk), dtype=torch.float32, device=u.device) if prepare else None
    _call("q6k_delta_channel", _ptr(u), _i(u.stride(0)), _ptr(p), _i(p.stride(0)), _i(b_col), _ptr(a), _i(a.stride(0)), _i(a_col), _ptr(A_log), _ptr(dt_bias),
          _ptr(scratch), _ptr(state), _ptr(req_of_token), _ptr(q_start), _ptr(slot_ids), _ptr(o), _i(T), _i(R), _i(H), _i(G), _i(dk), _i(dv),
          _i(1 if single else 0), _stream())
    return o


# --------------------------------------------------------------------------- heads' gates, norms of some columns
def gate_heads(a: torch.Tensor, H: int, p: torch.Tensor, col: int) -> None:
    """a[t, h] *= sigmoid(p[t, col + h]) in place: a [T, H n] in either dtype, p FP32 [T, *] or [slices, T, *] partial sums."""
    _need(a, "a")
    _need(p, "p", torch.float32)
    slices, stride, T, N = _slices_of(p)
    if a.shape[0] != T or a.shape[1] % H or col + H > N:
        raise KernelError("gate_heads: shapes disagree")
    _call("q6k_gate_heads", _ptr(a), _ptr(p), _i(slices), _ll(stride), _i(N), _i(col), _i(T), _i(H), _i(a.shape[1] // H), _i(dtype_code(a.dtype)), _stream())


def norm_columns(x: torch.Tensor, col: int, n: int, w: torch.Tensor, eps: float, out_dtype: torch.dtype) -> torch.Tensor:
    """out_dtype(c * rsqrt(mean(c^2) + eps) * w) for the columns c = x[t, col : col + n] of FP32 rows."""
    _need(x, "x", torch.float32)
    _need(w, "w", torch.float32, (n,))
    if col + n > x.shape[1]:
        raise KernelError("norm_columns: shapes disagree")
    out = torch.empty((x.shape[0], n), dtype=out_dtype, device=x.device)
    _call("q6k_norm_columns", _ptr(x), _i(x.stride(0)), _i(col), _i(n), _ptr(w), _f(eps), _ptr(out), _i(x.shape[0]), _i(dtype_code(out_dtype)), _stream())
    return out


# --------------------------------------------------------------------------- a residual of several streams
@functools.lru_cache(maxsize=None)
def hyper_max_streams() -> int:
    lib = library()
    lib.q6k_hyper_max_streams.restype = ctypes.c_int
    return lib.q6k_hyper_max_streams()


def normed_pair(a: torch.Tensor, bias: Optional[torch.Tensor], b: torch.Tensor, wa: torch.Tensor, wb: torch.Tensor, mult: float, eps: float) -> torch.Tensor:
    """FP32 mult * (norm(a + bias) wa + norm(b) wb), each over its root mean square along the row; a, b FP32 [T, D] or
    [slices, T, D] partial sums, bias FP32 [D] or None."""
    _need(a, "a", torch.float32)
    _need(b, "b", torch.float32)
    na, sa, T, D = _slices_of(a)
    nb, sb, T2, D2 = _slices_of(b)
    if (T, D) != (T2, D2):
        raise KernelError("normed_pair: shapes disagree")
    for nm, t in (("bias", bias), ("wa", wa), ("wb", wb)):
        if t is not None:
            _need(t, nm, torch.float32, (D,))
    out = torch.empty((T, D), dtype=torch.float32, device=a.device)
    _call("q6k_normed_pair", _ptr(a), _i(na), _ptr(bias), _ptr(b), _i(nb), _ll(T * D), _ptr(wa), _ptr(wb), _f(mult), _f(eps), _ptr(out), _i(T), _i(D), _stream())
    return out


def hyper_step(x: torch.Tensor, S: int, add=None, read=None, rows: Optional[torch.Tensor] = None, out_dtype: torch.dtype = torch.float32):
    """One pass over a residual of S streams.  x: FP32 [T, S, D], or [T, D] while all streams are equal.
    add = {"a", "bias", "weighted", "pair", "mix", "out"}: x_t <- sum_s mix[s, t] x_s + out[t] y for all streams at once, y = a (FP32
    [T, D] or [slices, T, D] partial sums) + bias (FP32 [D]) + weighted rows (as in `combine`), each optional; or, with pair = (b, wa, wb,
    mult, eps), y = mult (norm(a + bias) wa + norm(b) wb).  mix: FP32 [S, S]; out: FP32 [S].
    read = (weights FP32 [S], norm weight FP32 [D], eps): the norm of sum_t weights[t] x_t in out_dtype.
    rows: read these rows only, and store no streams.  Returns (streams [T, S, D] as they then stand, or x itself when nothing was
    added or rows are picked; the norm or None)."""
    _need(x, "x", torch.float32)
    broadcast = x.dim() == 2
    T, D = x.shape[0], x.shape[-1]
    if not broadcast and x.shape[1] != S:
        raise KernelError(f"hyper_step: {x.shape[1]} streams, expected {S}")
    a = bias = py = pair_row = pw = b = wa = wb = mix = out_w = None
    na = nb = 1
    K, mult, eps = 0, 1.0, read[2] if read is not None else 0.0
    if add is not None:
        a, bias, mix, out_w = add.get("a"), add.get("bias"), add["mix"], add["out"]
        _need(mix, "mix", torch.float32, (S, S))
        _need(out_w, "out", torch.float32, (S,))
        if bias is not None:
            _need(bias, "bias", torch.float32, (D,))
        if a is not None:
            _need(a, "a", torch.float32)
            na, _, ta, da = _slices_of(a)
            if (ta, da) != (T, D):
                raise KernelError("hyper_step: the sublayer's result does not match the streams")
        if add.get("weighted") is not None:
            py, pair_row, pw = add["weighted"]
            _need(py, "weighted rows", torch.float32)
            _need(pw, "weights", torch.float32)
            K = pw.shape[1]
            if pair_row is not None:
                _need(pair_row, "pair_row", torch.int32)
            if pw.shape[0] != T or py.shape[1] != D or py.shape[0] < T * K or (pair_row is not None and pair_row.numel() != T * K):
                raise KernelError("hyper_step: the weighted rows do not match the streams")
        if add.get("pair") is not None:
            b, wa, wb, mult, pair_eps = add["pair"]
            _need(b, "b", torch.float32)
            nb, _, tb, db = _slices_of(b)
            _need(wa, "wa", torch.float32, (D,))
            _need(wb, "wb", torch.float32, (D,))
            if a is None or (tb, db) != (T, D) or py is not None:
                raise KernelError("hyper_step: two normed results of one shape, without routed rows")
            if read is not None and pair_eps != eps:
                raise KernelError("hyper_step: the results' norms and the sublayer's share one eps")
            eps = pair_eps
        if a is None and py is None and bias is None:
            raise KernelError("hyper_step: nothing to add")
    in_w = norm_w = out = None
    R = T if rows is None else rows.numel()
    if read is not None:
        in_w, norm_w = read[0], read[1]
        _need(in_w, "stream weights", torch.float32, (S,))
        _need(norm_w, "norm weight", torch.float32, (D,))
        out = torch.empty((R, D), dtype=out_dtype, device=x.device)
    if rows is not None:
        _need(rows, "rows", torch.int32)
    dst = x if add is None or rows is not None else torch.empty((T, S, D), dtype=torch.float32, device=x.device) if broadcast else x
    if add is None and read is None:
        return x, None
    _call("q6k_hyper_step", _ptr(x), _i(1 if broadcast else 0), _ptr(dst if add is not None and rows is None else None), _ptr(a), _i(na), _ll(T * D), _ptr(bias),
          _ptr(py), _ptr(pair_row), _ptr(pw), _i(K), _ptr(b), _i(nb), _ptr(wa), _ptr(wb), _f(mult), _ptr(mix), _ptr(out_w), _ptr(in_w), _ptr(norm_w), _f(eps),
          _ptr(out), _ptr(rows), _i(R), _i(S), _i(D), _i(dtype_code(out_dtype)), _stream())
    return dst, out
