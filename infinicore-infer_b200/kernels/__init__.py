"""Python bindings of the CUDA kernels in ``csrc``: one thin function per exported symbol.

Arguments are CUDA tensors; each binding checks types, shapes and contiguity, passes raw
device pointers and the current stream to the C function, and raises ``KernelError`` with
the library's message if it returns non-zero.  There is no fallback path: without the
compiled module a call raises.
"""
from __future__ import annotations

import ctypes
from typing import Optional

import torch

from . import build as _build
from . import host as _host

F32, BF16 = 0, 1
_CODE = {torch.float32: F32, torch.bfloat16: BF16}


class KernelError(RuntimeError):
    pass


launch_count = 0      # kernels of this package launched through these bindings (captured ones count once)


def dtype_code(dtype: torch.dtype) -> int:
    try:
        return _CODE[dtype]
    except KeyError:
        raise KernelError(f"kernels take float32 or bfloat16, not {dtype}") from None


def _ptr(t: Optional[torch.Tensor]):
    return ctypes.c_void_p(0 if t is None else t.data_ptr())


def _stream():
    # the raw handle of the current stream of the current device (a Stream object costs microseconds
    # to build, and every launch asks)
    return ctypes.c_void_p(torch._C._cuda_getCurrentRawStream(torch.cuda.current_device()))


def _need(t: torch.Tensor, name: str, dtype=None, contiguous=True):
    if not t.is_cuda:
        raise KernelError(f"{name} must be a CUDA tensor (the engine has no CPU path)")
    if dtype is not None and t.dtype != dtype:
        raise KernelError(f"{name} must be {dtype}, is {t.dtype}")
    if contiguous and not t.is_contiguous():
        raise KernelError(f"{name} must be contiguous")


def _check(module: str, rc: int):
    global launch_count
    launch_count += 1
    if rc:
        lib = _build.load(module)
        fn = getattr(lib, f"jk_{module}_last_error")
        fn.restype = ctypes.c_char_p
        raise KernelError(fn().decode(errors="replace") or f"kernel module {module} returned {rc}")


_c_int, _c_float, _c_ll = ctypes.c_int, ctypes.c_float, ctypes.c_longlong


def embed(tokens: torch.Tensor, table: torch.Tensor, scale: float, out: torch.Tensor) -> torch.Tensor:
    """out[i, :] = scale * table[tokens[i], :], float32."""
    _need(tokens, "tokens", torch.int32); _need(table, "table"); _need(out, "out", torch.float32)
    n, d = tokens.numel(), table.shape[1]
    if out.shape[-1] != d or out.numel() < n * d:
        raise KernelError(f"embed: out {tuple(out.shape)} does not hold {n} rows of {d}")
    lib = _build.load("elementwise")
    _check("elementwise", lib.jk_embed(_ptr(tokens), _c_int(n), _ptr(table), _c_int(dtype_code(table.dtype)),
                                       _c_int(d), _c_float(scale), _ptr(out), _stream()))
    return out


def add_rmsnorm(x: torch.Tensor, delta: Optional[torch.Tensor], delta_scale: float, weight: torch.Tensor,
                eps: float, out: torch.Tensor, out_scale: float = 1.0,
                rows: Optional[torch.Tensor] = None) -> torch.Tensor:
    """x += delta_scale * delta (when rows is None); out = out_scale * rmsnorm(x[rows]) * weight."""
    _need(x, "x", torch.float32); _need(weight, "weight", torch.float32); _need(out, "out")
    d = x.shape[-1]
    if weight.numel() != d or out.shape[-1] != d:
        raise KernelError(f"add_rmsnorm: width {d}, weight {weight.numel()}, out {out.shape[-1]}")
    if delta is not None:
        _need(delta, "delta")
        if delta.shape != x.shape:
            raise KernelError(f"add_rmsnorm: delta {tuple(delta.shape)} vs x {tuple(x.shape)}")
    if rows is not None:
        _need(rows, "rows", torch.int32)
        nout = rows.numel()
    else:
        nout = x.numel() // d
    if out.numel() < nout * d:
        raise KernelError("add_rmsnorm: out is too small")
    lib = _build.load("elementwise")
    _check("elementwise", lib.jk_add_rmsnorm(
        _ptr(x), _ptr(delta), _c_int(dtype_code(delta.dtype) if delta is not None else F32),
        _c_float(delta_scale), _ptr(weight), _c_float(eps), _c_float(out_scale), _ptr(out),
        _c_int(dtype_code(out.dtype)), _ptr(rows), _c_int(nout), _c_int(d), _stream()))
    return out


def residual_add(x: torch.Tensor, delta: torch.Tensor, delta_scale: float) -> torch.Tensor:
    _need(x, "x", torch.float32); _need(delta, "delta")
    if delta.numel() != x.numel():
        raise KernelError("residual_add: sizes differ")
    lib = _build.load("elementwise")
    _check("elementwise", lib.jk_residual_add(_ptr(x), _ptr(delta), _c_int(dtype_code(delta.dtype)),
                                              _c_float(delta_scale), _c_ll(x.numel()), _stream()))
    return x


def swiglu(gate_up: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    """out[t, c] = silu(gate_up[t, c]) * gate_up[t, di + c]."""
    _need(gate_up, "gate_up"); _need(out, "out")
    ntok, di = out.shape
    if gate_up.shape != (ntok, 2 * di):
        raise KernelError(f"swiglu: gate_up {tuple(gate_up.shape)} vs out {tuple(out.shape)}")
    lib = _build.load("elementwise")
    _check("elementwise", lib.jk_swiglu(_ptr(gate_up), _c_int(dtype_code(gate_up.dtype)), _ptr(out),
                                        _c_int(dtype_code(out.dtype)), _c_int(ntok), _c_int(di), _stream()))
    return out


def rope_kv(qkv: torch.Tensor, bias: Optional[torch.Tensor], positions: torch.Tensor, row_req: torch.Tensor,
            block_table: Optional[torch.Tensor], page_size: int, cos: Optional[torch.Tensor],
            sin: Optional[torch.Tensor], interleaved: bool, q_out: torch.Tensor,
            k_pages: Optional[torch.Tensor], v_pages: Optional[torch.Tensor], ntok: int, nh: int, nkvh: int,
            dh: int, write_cache: bool = True) -> None:
    """Rotate query and key heads of ``qkv`` rows; write keys and values into their pages."""
    _need(qkv, "qkv"); _need(positions, "positions", torch.int32); _need(row_req, "row_req", torch.int32)
    _need(q_out, "q_out")
    width = (nh + 2 * nkvh) * dh
    if qkv.shape[-1] != width or qkv.shape[0] < ntok:
        raise KernelError(f"rope_kv: qkv {tuple(qkv.shape)} does not hold {ntok} rows of {width}")
    if q_out.numel() < ntok * nh * dh:
        raise KernelError("rope_kv: q_out is too small")
    max_blocks = 0
    if write_cache:
        _need(block_table, "block_table", torch.int32); _need(k_pages, "k_pages"); _need(v_pages, "v_pages")
        if k_pages.dtype != q_out.dtype or v_pages.dtype != q_out.dtype:
            raise KernelError("rope_kv: pages and q_out must have one type")
        if tuple(k_pages.shape[1:]) != (nkvh, page_size, dh) or k_pages.shape != v_pages.shape:
            raise KernelError(f"rope_kv: pages {tuple(k_pages.shape)} are not [*, {nkvh}, {page_size}, {dh}]")
        max_blocks = block_table.shape[1]
    if cos is not None:
        _need(cos, "cos", torch.float32); _need(sin, "sin", torch.float32)
        if cos.shape[1] != dh // 2 or sin.shape != cos.shape:
            raise KernelError("rope_kv: cos/sin tables must be [positions, head_dim/2]")
    if bias is not None:
        _need(bias, "bias", torch.float32)
    lib = _build.load("elementwise")
    _check("elementwise", lib.jk_rope_kv(
        _ptr(qkv), _c_int(dtype_code(qkv.dtype)), _c_int(width), _ptr(bias), _ptr(positions), _ptr(row_req),
        _ptr(block_table), _c_int(max_blocks), _c_int(page_size), _ptr(cos), _ptr(sin),
        _c_int(1 if interleaved else 0), _ptr(q_out), _ptr(k_pages), _ptr(v_pages),
        _c_int(dtype_code(q_out.dtype)), _c_int(ntok), _c_int(nh), _c_int(nkvh), _c_int(dh),
        _c_int(1 if write_cache else 0), _stream()))


def gemm_f32(a: torch.Tensor, w: torch.Tensor, out: torch.Tensor, bias: Optional[torch.Tensor] = None) -> torch.Tensor:
    """out[M, N] = a[M, K] @ w[N, K]^T (+ bias) in float32 on the CUDA cores (no TF32)."""
    _need(a, "a", torch.float32); _need(w, "w", torch.float32); _need(out, "out", torch.float32)
    m, k = a.shape
    n = w.shape[0]
    if w.shape[1] != k or tuple(out.shape) != (m, n):
        raise KernelError(f"gemm_f32: a {tuple(a.shape)}, w {tuple(w.shape)}, out {tuple(out.shape)}")
    if bias is not None:
        _need(bias, "bias", torch.float32)
    lib = _build.load("elementwise")
    _check("elementwise", lib.jk_gemm_f32(_ptr(a), _c_int(k), _ptr(w), _c_int(k), _ptr(bias), _ptr(out),
                                          _c_int(n), _c_int(m), _c_int(n), _c_int(k), _stream()))
    return out


EPI_F32, EPI_SWIGLU, EPI_RESIDUAL = 0, 1, 3


def linear_small_supports(m: int, n: int, k: int) -> bool:
    """Whether the weight-streaming kernel for steps of few rows takes this product."""
    return bool(_build.load("linear_small").jk_linear_small_supports(_c_int(m), _c_int(n), _c_int(k)))


def linear_small(act: torch.Tensor, w: torch.Tensor, out: torch.Tensor, epilogue: int = EPI_F32) -> torch.Tensor:
    """out = act @ w^T for at most 16 rows of bfloat16 activations.  EPI_F32: float32 out [M, N].
    EPI_SWIGLU: w is [2N, K] (gate rows, then up rows) and out is bfloat16 [M, N] = silu(gate) * up."""
    _need(act, "act", torch.bfloat16); _need(w, "w", torch.bfloat16)
    _need(out, "out", torch.float32 if epilogue == EPI_F32 else torch.bfloat16)
    m, k = act.shape
    n = w.shape[0] // (2 if epilogue == EPI_SWIGLU else 1)
    if w.shape[1] != k or tuple(out.shape) != (m, n):
        raise KernelError(f"linear_small: act {tuple(act.shape)}, w {tuple(w.shape)}, out {tuple(out.shape)}")
    lib = _build.load("linear_small")
    _check("linear_small", lib.jk_linear_small(_ptr(act), _ptr(w), _ptr(out), _c_int(m), _c_int(n), _c_int(k),
                                               _c_int(out.stride(0)), _c_int(epilogue), _c_int(_sm_count(act.device)),
                                               _stream()))
    return out


def linear_small_parts_supports(m: int, n: int, k: int) -> bool:
    """Whether the few-row tile kernel takes several products of ``m`` rows over ``k`` with ``n`` features in all as one launch."""
    return bool(_build.load("linear_small").jk_linear_small_parts_supports(_c_int(m), _c_int(n), _c_int(k)))


def linear_small_parts(acts: torch.Tensor, w: torch.Tensor, ends, out: torch.Tensor) -> torch.Tensor:
    """Several products of at most 16 rows in one launch: ``out[:, ends[p-1]:ends[p]] = acts[p] @ w[ends[p-1]:ends[p]]^T`` for
    bfloat16 ``acts`` [parts, M, K] and ``w`` [N, K], float32 ``out`` [M, N] (rows may be wider: its stride is taken).  Every end
    but the last is a multiple of 16."""
    _need(acts, "acts", torch.bfloat16); _need(w, "w", torch.bfloat16)
    _need(out, "out", torch.float32, contiguous=False)
    parts, m, k = acts.shape
    n = w.shape[0]
    if w.shape[1] != k or tuple(out.shape) != (m, n) or out.stride(1) != 1 or len(ends) != parts or parts > 8:
        raise KernelError(f"linear_small_parts: acts {tuple(acts.shape)}, w {tuple(w.shape)}, out {tuple(out.shape)}, ends {list(ends)}")
    lib = _build.load("linear_small")
    arr = (ctypes.c_int * parts)(*[int(e) for e in ends])
    _check("linear_small", lib.jk_linear_small_parts(_ptr(acts), ctypes.c_longlong(m * k), arr, _c_int(parts), _ptr(w), _ptr(out), _c_int(m),
                                                     _c_int(n), _c_int(k), _c_int(out.stride(0)), _c_int(_sm_count(acts.device)), _stream()))
    return out


def linear_small_qkv_supports(m: int, k: int, dh: int) -> bool:
    """Whether the small-row product can take the fused [q | k | v] projection with rotation and cache
    write in its epilogue."""
    return bool(_build.load("linear_small").jk_linear_small_qkv_supports(_c_int(m), _c_int(k), _c_int(dh)))


def linear_small_qkv(act: torch.Tensor, w: torch.Tensor, q_out: torch.Tensor, k_pages: torch.Tensor,
                     v_pages: torch.Tensor, cos: Optional[torch.Tensor], sin: Optional[torch.Tensor],
                     positions: torch.Tensor, row_req: torch.Tensor, block_table: torch.Tensor, nh: int) -> torch.Tensor:
    """The fused [q | k | v] projection of at most 16 bfloat16 rows: query and key heads rotated
    (rotate-half), queries to ``q_out``, keys and values into their pages, all from the epilogue."""
    _check_qkv_args("linear_small_qkv", act, w, q_out, k_pages, v_pages, cos, sin, positions, row_req, block_table, nh)
    m, k = act.shape
    _, nkvh, page_size, dh = k_pages.shape
    lib = _build.load("linear_small")
    _check("linear_small", lib.jk_linear_small_qkv(
        _ptr(act), _ptr(w), _c_int(m), _c_int(k), _ptr(q_out), _ptr(k_pages), _ptr(v_pages), _ptr(cos), _ptr(sin),
        _ptr(positions), _ptr(row_req), _ptr(block_table), _c_int(block_table.shape[1]), _c_int(page_size), _c_int(nh),
        _c_int(nkvh), _c_int(dh), _c_int(_sm_count(act.device)), _stream()))
    return q_out


SUMSQ_FIXED = float(1 << 26)      # the fixed-point scale of the row sums of squares (csrc/linear_small.cu)


def linear_small_norm_supports(m: int, n: int, k: int) -> bool:
    """Whether the products of a chain without norm kernels take this shape (the tile kernel's reach)."""
    return bool(_build.load("linear_small").jk_linear_small_norm_supports(_c_int(m), _c_int(n), _c_int(k)))


def linear_small_norm(act: torch.Tensor, w: torch.Tensor, out: torch.Tensor, epilogue: int = EPI_F32,
                      in_sumsq: Optional[torch.Tensor] = None, in_eps: float = 0.0, xb: Optional[torch.Tensor] = None,
                      next_w: Optional[torch.Tensor] = None, out_sumsq: Optional[torch.Tensor] = None,
                      scale: float = 1.0) -> torch.Tensor:
    """A few-row product of a chain in which RMSNorm has no kernel of its own.  With ``in_sumsq`` (int64 [M],
    fixed point: sum of squares times ``SUMSQ_FIXED``) the activations are x * norm weight without the 1 / rms,
    which the rows of the product get before the epilogue (EPI_F32 or EPI_SWIGLU).  ``EPI_RESIDUAL``: ``out`` is
    the float32 residual stream, ``out += scale * product``; ``xb`` receives bfloat16(out * next_w) and
    ``out_sumsq`` (zeroed by the caller) this product's sums of squares of the new rows."""
    _need(act, "act", torch.bfloat16); _need(w, "w", torch.bfloat16)
    _need(out, "out", torch.bfloat16 if epilogue == EPI_SWIGLU else torch.float32)
    m, k = act.shape
    n = w.shape[0] // (2 if epilogue == EPI_SWIGLU else 1)
    if w.shape[1] != k or tuple(out.shape) != (m, n):
        raise KernelError(f"linear_small_norm: act {tuple(act.shape)}, w {tuple(w.shape)}, out {tuple(out.shape)}")
    for name, t, dt in (("in_sumsq", in_sumsq, torch.int64), ("out_sumsq", out_sumsq, torch.int64), ("xb", xb, torch.bfloat16),
                        ("next_w", next_w, torch.float32)):
        if t is not None:
            _need(t, name, dt)
    if (in_sumsq is not None and in_sumsq.numel() < m) or (out_sumsq is not None and out_sumsq.numel() < m) \
            or (xb is not None and tuple(xb.shape) != (m, n)) or (next_w is not None and next_w.numel() != n):
        raise KernelError("linear_small_norm: a norm array has the wrong size")
    lib = _build.load("linear_small")
    _check("linear_small", lib.jk_linear_small_norm(
        _ptr(act), _ptr(w), _ptr(out), _c_int(m), _c_int(n), _c_int(k), _c_int(out.stride(0)), _c_int(epilogue),
        _ptr(in_sumsq), _c_float(in_eps), _ptr(xb), _ptr(next_w), _ptr(out_sumsq), _c_float(scale),
        _ptr(gemm_status(act.device)), _c_int(_sm_count(act.device)), _stream()))
    return out


def linear_small_qkv_norm(act: torch.Tensor, w: torch.Tensor, q_out: torch.Tensor, k_pages: torch.Tensor,
                          v_pages: torch.Tensor, cos: Optional[torch.Tensor], sin: Optional[torch.Tensor],
                          positions: torch.Tensor, row_req: torch.Tensor, block_table: torch.Tensor, nh: int,
                          in_sumsq: torch.Tensor, in_eps: float) -> torch.Tensor:
    """``linear_small_qkv`` for activations that came without their norm's 1 / rms (see ``linear_small_norm``)."""
    _check_qkv_args("linear_small_qkv_norm", act, w, q_out, k_pages, v_pages, cos, sin, positions, row_req, block_table, nh)
    _need(in_sumsq, "in_sumsq", torch.int64)
    m, k = act.shape
    _, nkvh, page_size, dh = k_pages.shape
    lib = _build.load("linear_small")
    _check("linear_small", lib.jk_linear_small_qkv_norm(
        _ptr(act), _ptr(w), _c_int(m), _c_int(k), _ptr(q_out), _ptr(k_pages), _ptr(v_pages), _ptr(cos), _ptr(sin),
        _ptr(positions), _ptr(row_req), _ptr(block_table), _c_int(block_table.shape[1]), _c_int(page_size), _c_int(nh),
        _c_int(nkvh), _c_int(dh), _ptr(in_sumsq), _c_float(in_eps), _c_int(_sm_count(act.device)), _stream()))
    return q_out


def _check_qkv_args(what, act, w, q_out, k_pages, v_pages, cos, sin, positions, row_req, block_table, nh) -> None:
    for name, t in (("act", act), ("w", w), ("q_out", q_out), ("k_pages", k_pages), ("v_pages", v_pages)):
        _need(t, name, torch.bfloat16)
    for name, t in (("positions", positions), ("row_req", row_req), ("block_table", block_table)):
        _need(t, name, torch.int32)
    m, k = act.shape
    _, nkvh, page_size, dh = k_pages.shape
    if w.shape != ((nh + 2 * nkvh) * dh, k) or q_out.numel() < m * nh * dh or v_pages.shape != k_pages.shape:
        raise KernelError(f"{what}: act {tuple(act.shape)}, w {tuple(w.shape)}, pages {tuple(k_pages.shape)}")
    if positions.numel() < m or row_req.numel() < m:
        raise KernelError(f"{what}: positions or row_req hold fewer entries than rows")
    if cos is not None:
        _need(cos, "cos", torch.float32); _need(sin, "sin", torch.float32)
        if cos.shape[1] != dh // 2 or sin.shape != cos.shape:
            raise KernelError(f"{what}: cos/sin tables must be [positions, head_dim/2]")


def gemm_tcgen05_qkv_supports(dh: int) -> bool:
    """Head sizes for which the tcgen05 product can rotate and store [q | k | v] in its epilogue."""
    return dh in (64, 128)


def gemm_tcgen05_qkv(act: torch.Tensor, w: torch.Tensor, q_out: torch.Tensor, k_pages: torch.Tensor,
                     v_pages: torch.Tensor, cos: Optional[torch.Tensor], sin: Optional[torch.Tensor],
                     positions: torch.Tensor, row_req: torch.Tensor, block_table: torch.Tensor, nh: int) -> torch.Tensor:
    """The fused [q | k | v] projection of bfloat16 rows: ``act @ w^T`` with query and key heads rotated
    (rotate-half; cos/sin ``[positions, dh/2]`` float32 or None), queries written to ``q_out`` and keys and
    values into their pages through ``block_table``, all from the product's epilogue."""
    _check_qkv_args("gemm_tcgen05_qkv", act, w, q_out, k_pages, v_pages, cos, sin, positions, row_req, block_table, nh)
    m, k = act.shape
    _, nkvh, page_size, dh = k_pages.shape
    lib = _build.load("gemm_tcgen05")
    _check("gemm_tcgen05", lib.jk_gemm_tcgen05_qkv(
        _ptr(act), _ptr(w), _c_int(m), _c_int(k), _ptr(q_out), _ptr(k_pages), _ptr(v_pages), _ptr(cos), _ptr(sin),
        _ptr(positions), _ptr(row_req), _ptr(block_table), _c_int(block_table.shape[1]), _c_int(page_size), _c_int(nh),
        _c_int(nkvh), _c_int(dh), _ptr(gemm_status(act.device)), _c_int(_sm_count(act.device)), _stream()))
    return q_out


TG_F32, TG_BF16, TG_RESIDUAL, TG_SWIGLU = 0, 1, 2, 3
_tg_status = {}


def gemm_status(device) -> torch.Tensor:
    """The word in which a kernel records a wait that ran out (0: none).  It lies in pinned host memory, which the
    device reaches under the same address: a kernel that gives up writes across, and the host reads it without a copy."""
    key = str(device)
    if key not in _tg_status:
        _tg_status[key] = torch.zeros(1, dtype=torch.int32).pin_memory()
    return _tg_status[key]


def check_gemm_status(device) -> None:
    """Wait for the device's work, read the status words; raise if a kernel gave up waiting."""
    torch.cuda.synchronize(device)
    small = _build._loaded.get("linear_small")
    if small is not None:
        fault = small.jk_linear_small_take_fault()
        if fault > 0:
            raise KernelError(f"linear_small: a bounded wait for a tile of weights ran out or shared memory was misaligned "
                              f"(code {fault}); the step's results are not valid")
    key = str(device)
    if key in _tg_status:
        code = int(_tg_status[key].item())
        if code:
            _tg_status[key].zero_()
            if code == 4:
                raise KernelError("linear_small: a row's sum of squares is beyond the range of the fixed-point counters "
                                  "(activations of several thousand on average); the step's results are not valid; "
                                  "JK_NO_FUSED_NORM=1 keeps the norm kernels, which have no such limit")
            raise KernelError(f"gemm_tcgen05: a bounded wait ran out (role {code}: 1 TMA, 2 MMA, 3 epilogue); "
                              "the step's results are not valid")


def gemm_tcgen05_supports(m: int, n: int, k: int) -> bool:
    """K must keep rows 16-byte aligned for TMA; everything else is free (the same rule as the library's
    ``jk_gemm_tcgen05_supports``; answered here so that asking does not compile the module)."""
    return m >= 1 and n >= 1 and k >= 8 and k % 8 == 0


def gemm_tcgen05_pairs(mode: int) -> int:
    """Which products run on pairs of blocks (clusters of two sharing one 256 x 256 tile, ``cta_group::2``):
    0 none, 1 those whose tiles make more than one wave (the default), 2 all of more than 128 rows.  Returns
    the mode before (-1: the environment's or the default had not been read yet)."""
    return _build.load("gemm_tcgen05").jk_gemm_tcgen05_set_pairs(ctypes.c_int(mode))


def gemm_tcgen05(act: torch.Tensor, w: torch.Tensor, out: torch.Tensor, epilogue: int = TG_F32,
                 scale: float = 1.0) -> torch.Tensor:
    """out (op)= act @ w^T on the tcgen05 tensor cores, operands by TMA.  Epilogues: TG_F32 / TG_BF16 store,
    TG_RESIDUAL ``out += scale * product`` (float32, in place), TG_SWIGLU ``w`` is [2N, K] (gate rows, up rows)
    and ``out`` is bfloat16 [M, N] = silu(gate) * up."""
    _need(act, "act", torch.bfloat16); _need(w, "w", torch.bfloat16)
    _need(out, "out", torch.bfloat16 if epilogue in (TG_BF16, TG_SWIGLU) else torch.float32, contiguous=False)
    m, k = act.shape
    n = w.shape[0] // (2 if epilogue == TG_SWIGLU else 1)
    if w.shape[1] != k or tuple(out.shape) != (m, n) or out.stride(1) != 1:
        raise KernelError(f"gemm_tcgen05: act {tuple(act.shape)}, w {tuple(w.shape)}, out {tuple(out.shape)}")
    lib = _build.load("gemm_tcgen05")
    _check("gemm_tcgen05", lib.jk_gemm_tcgen05(_ptr(act), _ptr(w), _ptr(out), _c_int(m), _c_int(n), _c_int(k),
                                               _c_int(out.stride(0)), _c_int(epilogue), _c_float(scale),
                                               _ptr(gemm_status(act.device)), _c_int(_sm_count(act.device)), _stream()))
    return out


def gemm_skinny_supports(m: int, n: int, k: int) -> bool:
    """Up to 128 activation rows; K must keep rows 16-byte aligned for TMA."""
    return 1 <= m <= 128 and n >= 1 and k >= 8 and k % 8 == 0


def gemm_skinny(act: torch.Tensor, w: torch.Tensor, out: torch.Tensor, epilogue: int = TG_F32, scale: float = 1.0) -> torch.Tensor:
    """The product of few activation rows (decode batches, short portions) on the tcgen05 tensor cores with the
    weights on the MMA's M side, so that the kernel streams W once at memory speed: TG_F32 ``out = product``
    (float32), TG_RESIDUAL ``out += scale * product`` (float32, blocks split K and add their partial sums),
    TG_SWIGLU ``w`` is [2N, K] and ``out`` bfloat16 = silu(gate) * up."""
    if epilogue not in (TG_F32, TG_RESIDUAL, TG_SWIGLU):
        raise KernelError(f"gemm_skinny: epilogue {epilogue}")
    _need(act, "act", torch.bfloat16); _need(w, "w", torch.bfloat16)
    _need(out, "out", torch.bfloat16 if epilogue == TG_SWIGLU else torch.float32, contiguous=False)
    m, k = act.shape
    n = w.shape[0] // (2 if epilogue == TG_SWIGLU else 1)
    if w.shape[1] != k or tuple(out.shape) != (m, n) or out.stride(1) != 1:
        raise KernelError(f"gemm_skinny: act {tuple(act.shape)}, w {tuple(w.shape)}, out {tuple(out.shape)}")
    lib = _build.load("gemm_tcgen05")
    _check("gemm_tcgen05", lib.jk_gemm_skinny(_ptr(act), _ptr(w), _ptr(out), _c_int(m), _c_int(n), _c_int(k),
                                              _c_int(out.stride(0)), _c_int(epilogue), _c_float(scale),
                                              _ptr(gemm_status(act.device)), _c_int(_sm_count(act.device)), _stream()))
    return out


_SMS = {}


def _sm_count(device) -> int:
    key = str(device)
    if key not in _SMS:
        _SMS[key] = torch.cuda.get_device_properties(device).multi_processor_count
    return _SMS[key]


def _gate_args(gate: Optional[torch.Tensor], rows: int, nh: int):
    """(pointer, leading dimension) of a float32 gate ``[rows, >= nh]`` (a view of wider rows is fine), or nulls.  ``nh`` counts
    columns: heads, or heads x value size for a gate per element."""
    if gate is None:
        return _ptr(None), _c_int(0)
    _need(gate, "gate", torch.float32, contiguous=False)
    if gate.dim() != 2 or gate.stride(1) != 1 or gate.shape[0] < rows or gate.shape[1] < nh:
        raise KernelError("attention: gate must be [rows, heads] with unit stride along heads")
    return _ptr(gate), _c_int(gate.stride(0))


def attention_rows(q: torch.Tensor, k_pages: torch.Tensor, v_pages: torch.Tensor, out: torch.Tensor,
                   positions: torch.Tensor, row_req: torch.Tensor, block_table: torch.Tensor, ntok: int,
                   nh: int, scale: float, window: int = 0, sink: bool = False,
                   gate: Optional[torch.Tensor] = None, cap: float = 0.0, keep_first: int = 0,
                   sink_w: Optional[torch.Tensor] = None, gate_elem: bool = False) -> torch.Tensor:
    """Causal attention of ``ntok`` query rows over the paged cache, one warp per (row, head).  Values may have
    another size than keys (``v_pages [..., dv]``, ``out [ntok, nh, dv]``); ``sink`` adds a key of score 0 without a
    value; ``gate`` (float32 ``[ntok, >= nh]``, a view of wider rows is fine) multiplies head h's output by
    sigmoid(gate[t, h]); ``cap`` > 0 caps the scores by cap tanh(s / cap); keys at positions below ``keep_first`` stay
    visible when the window has passed them; ``sink_w`` (float32 [nh]): the sinks' scores instead of 0; ``gate_elem``: the gate
    has a column for every output element (``[ntok, >= nh dv]``)."""
    _need(q, "q"); _need(k_pages, "k_pages"); _need(v_pages, "v_pages"); _need(out, "out")
    _need(positions, "positions", torch.int32); _need(row_req, "row_req", torch.int32)
    _need(block_table, "block_table", torch.int32)
    if not (q.dtype == k_pages.dtype == v_pages.dtype == out.dtype):
        raise KernelError("attention: q, pages and out must have one type")
    _, nkvh, page_size, dh = k_pages.shape
    dv = v_pages.shape[-1]
    if q.numel() < ntok * nh * dh or out.numel() < ntok * nh * dv:
        raise KernelError("attention: q or out is too small")
    gate_ld = 0
    if gate is not None:
        _need(gate, "gate", torch.float32, contiguous=False)
        if gate.dim() != 2 or gate.stride(1) != 1 or gate.shape[0] < ntok or gate.shape[1] < nh * (dv if gate_elem else 1):
            raise KernelError("attention: gate must be [rows, heads] with unit stride along heads")
        gate_ld = gate.stride(0)
    lib = _build.load("attention")
    _check("attention", lib.jk_attention_rows(
        _ptr(q), _ptr(k_pages), _ptr(v_pages), _ptr(out), _c_int(dtype_code(q.dtype)), _ptr(positions),
        _ptr(row_req), _ptr(block_table), _c_int(block_table.shape[1]), _c_int(page_size), _c_int(ntok),
        _c_int(nh), _c_int(nkvh), _c_int(dh), _c_float(scale), _c_int(window or 0), _c_int(dv), _c_int(1 if sink else 0),
        _ptr(gate), _c_int(gate_ld), _c_float(cap), _c_int(keep_first), _ptr(sink_w), _c_int(1 if gate_elem else 0), _stream()))
    return out


def attention_decode(q: torch.Tensor, k_pages: torch.Tensor, v_pages: torch.Tensor, out: torch.Tensor,
                     rows: Optional[torch.Tensor], nrows: int, positions: torch.Tensor, row_req: torch.Tensor,
                     block_table: torch.Tensor, nh: int, scale: float, window: int, splits: int,
                     scratch: Optional[torch.Tensor] = None, sink: bool = False, gate: Optional[torch.Tensor] = None,
                     cap: float = 0.0, keep_first: int = 0, sink_w: Optional[torch.Tensor] = None,
                     gate_elem: bool = False) -> torch.Tensor:
    """bfloat16 attention of rows that bring few queries per request (decoded tokens, short portions):
    the key range of every (row, key/value head) is cut into ``splits`` blocks whose partial results
    a second kernel merges.  ``rows`` lists the rows to work on (None: rows 0..nrows-1).  ``cap`` and ``keep_first``
    as ``attention_rows`` takes them: the kept keys that the window has passed are the first of a row's range."""
    for name, t in (("q", q), ("k_pages", k_pages), ("v_pages", v_pages), ("out", out)):
        _need(t, name, torch.bfloat16)
    _need(positions, "positions", torch.int32); _need(row_req, "row_req", torch.int32)
    _need(block_table, "block_table", torch.int32)
    if rows is not None:
        _need(rows, "rows", torch.int32)
    _, nkvh, page_size, dh = k_pages.shape
    dv = v_pages.shape[-1]
    lib = _build.load("attention")
    lib.jk_attention_decode_scratch_floats.restype = ctypes.c_longlong
    need = lib.jk_attention_decode_scratch_floats(_c_int(nrows), _c_int(nh), _c_int(dv), _c_int(splits))
    if need and scratch is None:
        scratch = torch.empty(need, dtype=torch.float32, device=q.device)
    if need:
        _need(scratch, "scratch", torch.float32)
        if scratch.numel() < need:
            raise KernelError(f"attention_decode: scratch holds {scratch.numel()} floats, {need} needed")
    _check("attention", lib.jk_attention_decode(
        _ptr(q), _ptr(k_pages), _ptr(v_pages), _ptr(out), _ptr(scratch if need else None), _ptr(rows), _c_int(nrows),
        _ptr(positions), _ptr(row_req), _ptr(block_table), _c_int(block_table.shape[1]), _c_int(page_size),
        _c_int(nh), _c_int(nkvh), _c_int(dh), _c_float(scale), _c_int(window or 0), _c_int(splits), _c_int(1 if sink else 0),
        *_gate_args(gate, 0, nh * (dv if gate_elem else 1)), _c_float(cap), _c_int(keep_first), _ptr(sink_w), _c_int(1 if gate_elem else 0), _c_int(dv),
        _stream()))
    if need and splits > 1:
        global launch_count
        launch_count += 1          # the merge kernel
    return out


def attention_prefill_supports(dh: int) -> bool:
    return bool(_build.load("attention").jk_attention_prefill_supports(_c_int(dh)))


TILE_ROWS = _host.attention_tile_rows()      # rows of a query tile in the tile lists that the prefill attention kernels take


def attention_prefill(q: torch.Tensor, k_pages: torch.Tensor, v_pages: torch.Tensor, out: torch.Tensor,
                      tiles: torch.Tensor, ntiles: int, req_start: torch.Tensor, req_pos: torch.Tensor,
                      block_table: torch.Tensor, nh: int, scale: float, window: int = 0, sink: bool = False,
                      gate: Optional[torch.Tensor] = None, cap: float = 0.0, keep_first: int = 0,
                      sink_w: Optional[torch.Tensor] = None, gate_elem: bool = False) -> torch.Tensor:
    """bfloat16 tensor-core (mma.sync) attention of requests that bring many rows: ``tiles[i] = (batch
    entry, first row)`` names TILE_ROWS-row tiles of query rows.  ``cap`` and ``keep_first`` as ``attention_rows`` takes
    them: the tiles of keys that hold kept keys and lie before the window's come first."""
    for name, t in (("q", q), ("k_pages", k_pages), ("v_pages", v_pages), ("out", out)):
        _need(t, name, torch.bfloat16)
    for name, t in (("tiles", tiles), ("req_start", req_start), ("req_pos", req_pos), ("block_table", block_table)):
        _need(t, name, torch.int32)
    _, nkvh, page_size, dh = k_pages.shape
    if tiles.numel() < 2 * ntiles:
        raise KernelError("attention_prefill: the tile list is shorter than ntiles")
    lib = _build.load("attention")
    _check("attention", lib.jk_attention_prefill(
        _ptr(q), _ptr(k_pages), _ptr(v_pages), _ptr(out), _ptr(tiles), _c_int(ntiles), _c_int(TILE_ROWS), _ptr(req_start),
        _ptr(req_pos), _ptr(block_table), _c_int(block_table.shape[1]), _c_int(page_size), _c_int(nh), _c_int(nkvh),
        _c_int(dh), _c_float(scale), _c_int(window or 0), _c_int(1 if sink else 0), *_gate_args(gate, 0, nh * (dh if gate_elem else 1)), _c_float(cap),
        _c_int(keep_first), _ptr(sink_w), _c_int(1 if gate_elem else 0), _stream()))
    return out


def attention_tcgen05_supports(dh: int, page_size: int, dv: int = 0) -> bool:
    """Head sizes 64 and 128, or keys and values of unlike sizes up to 128, with pages that divide a tile of 128 keys and fill whole groups of 8 rows
    (``jk::attention_tcgen05_takes`` of csrc/host_rules.h; asking does not compile the kernel's module)."""
    return _host.attention_tcgen05_takes(dh, page_size, dv)


def attention_tcgen05(q: torch.Tensor, k_pages: torch.Tensor, v_pages: torch.Tensor, out: torch.Tensor,
                      tiles: torch.Tensor, ntiles: int, ntok: int, req_start: torch.Tensor, req_pos: torch.Tensor,
                      block_table: torch.Tensor, nh: int, scale: float, window: int = 0, sink: bool = False,
                      gate: Optional[torch.Tensor] = None, cap: float = 0.0, keep_first: int = 0,
                      sink_w: Optional[torch.Tensor] = None, gate_elem: bool = False) -> torch.Tensor:
    """The same attention of TILE_ROWS-row query tiles on the tcgen05 tensor cores (TMA operands, both
    products with accumulators in tensor memory); head sizes 64 and 128, or keys and values of unlike sizes (multiples of 8 up to
    128), pages that divide 128."""
    for name, t in (("q", q), ("k_pages", k_pages), ("v_pages", v_pages), ("out", out)):
        _need(t, name, torch.bfloat16)
    for name, t in (("tiles", tiles), ("req_start", req_start), ("req_pos", req_pos), ("block_table", block_table)):
        _need(t, name, torch.int32)
    num_pages, nkvh, page_size, dh = k_pages.shape
    dv = v_pages.shape[-1]
    if tiles.numel() < 2 * ntiles or q.numel() < ntok * nh * dh:
        raise KernelError("attention_tcgen05: the tile list or q is too short")
    lib = _build.load("attention_tcgen05")
    _check("attention_tcgen05", lib.jk_attention_tcgen05(
        _ptr(q), _ptr(k_pages), _ptr(v_pages), _ptr(out), _ptr(tiles), _c_int(ntiles), _c_int(ntok), _ptr(req_start),
        _ptr(req_pos), _ptr(block_table), _c_int(block_table.shape[1]), _c_int(num_pages), _c_int(page_size), _c_int(nh),
        _c_int(nkvh), _c_int(dh), _c_float(scale), _c_int(window or 0), _ptr(gemm_status(q.device)), _c_int(1 if sink else 0),
        *_gate_args(gate, ntok, nh * (dv if gate_elem else 1)), _c_float(cap), _c_int(keep_first), _ptr(sink_w), _c_int(1 if gate_elem else 0), _c_int(dv),
        _stream()))
    return out


# ---- csrc/mixers.cu ------------------------------------------------------------------------------------------------
ACT_NONE, ACT_SILU, ACT_GELU_TANH, ACT_SIGMOID = 0, 1, 2, 3


def layernorm(src: torch.Tensor, weight: torch.Tensor, bias: Optional[torch.Tensor], eps: float, out: Optional[torch.Tensor] = None,
              rows: Optional[torch.Tensor] = None, add_into: Optional[torch.Tensor] = None) -> Optional[torch.Tensor]:
    """``add_into`` given: add_into += LN(src), and ``out`` (if given) = add_into in its own type.  Otherwise
    out[i] = LN(src[rows[i]]) (all rows without ``rows``).  src and add_into are float32 ``[T, d]``."""
    _need(src, "src", torch.float32); _need(weight, "weight", torch.float32)
    d = src.shape[-1]
    n = rows.numel() if rows is not None else src.numel() // d
    for t, name in ((bias, "bias"), (add_into, "add_into")):
        if t is not None:
            _need(t, name, torch.float32)
    if rows is not None:
        _need(rows, "rows", torch.int32)
    if out is not None:
        _need(out, "out")
        if out.numel() < n * d:
            raise KernelError("layernorm: out is too small")
    lib = _build.load("mixers")
    _check("mixers", lib.jk_layernorm(_ptr(src), _ptr(rows), _c_int(n), _c_int(d), _ptr(weight), _ptr(bias), _c_float(eps), _ptr(add_into),
                                      _ptr(out), _c_int(dtype_code(out.dtype) if out is not None else F32), _stream()))
    return out


def glu(gate_up: torch.Tensor, out: torch.Tensor, act: int, limit: float = 0.0) -> torch.Tensor:
    """out[t, c] = act(gate_up[t, c]) * gate_up[t, di + c]; gate_up float32."""
    _need(gate_up, "gate_up", torch.float32); _need(out, "out")
    ntok, di = out.shape
    if gate_up.shape != (ntok, 2 * di):
        raise KernelError(f"glu: gate_up {tuple(gate_up.shape)} for out {tuple(out.shape)}")
    lib = _build.load("mixers")
    _check("mixers", lib.jk_glu(_ptr(gate_up), _ptr(out), _c_int(dtype_code(out.dtype)), _c_int(ntok), _c_int(di), _c_int(act), _c_float(limit), _stream()))
    return out


def conv_qkv(u: torch.Tensor, offsets, heads: int, kv_heads: int, dk: int, dv: int, has_kv: bool, convs, taps: int, norms, eps: float,
             freq: Optional[torch.Tensor], rot_dims: int, tail: Optional[torch.Tensor], positions, row_req, req_start, slot_ids,
             block_table: Optional[torch.Tensor], page_size: int, q_out: torch.Tensor, k_pages=None, v_pages=None,
             rot_half: bool = False, rot_mag: float = 1.0, head_norm=False, bias: Optional[torch.Tensor] = None,
             temp: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Short convolution, whole-projection RMS norm, pair rotation and cache write of fused float32 projections ``u``
    ``[T, ld]`` (columns ``offsets = (q, k, v)``); ``convs = (q, k, v)`` taps ``[channels, taps]`` or None each;
    ``norms = (q, k)`` weights or None each; ``tail [slots, taps - 1, channels]`` is read and moved forward.  ``rot_half``
    pairs element i of a head with element i + rot_dims / 2, ``rot_mag`` multiplies cos and sin, ``head_norm`` divides each
    head of q and k by its root mean square after the rotation, ``temp`` [heads] multiplies the heads' queries."""
    _need(u, "u", torch.float32); _need(q_out, "q_out")
    T, nreq = u.shape[0], req_start.numel() - 1
    lib = _build.load("mixers")
    _check("mixers", lib.jk_conv_qkv(
        _ptr(u), _c_int(u.shape[1]), _c_int(offsets[0]), _c_int(offsets[1]), _c_int(offsets[2]), _c_int(heads), _c_int(kv_heads),
        _c_int(dk), _c_int(dv), _c_int(1 if has_kv else 0), _ptr(convs[0]), _ptr(convs[1]), _ptr(convs[2]), _c_int(taps),
        _ptr(norms[0]), _ptr(norms[1]), _c_float(eps), _ptr(freq), _c_int(rot_dims), _ptr(tail), _ptr(positions), _ptr(row_req),
        _ptr(req_start), _ptr(slot_ids), _ptr(block_table), _c_int(block_table.shape[1] if block_table is not None else 0),
        _c_int(page_size), _ptr(q_out), _ptr(k_pages), _ptr(v_pages), _c_int(dtype_code(q_out.dtype)), _c_int(T), _c_int(nreq),
        _c_int(1 if rot_half else 0), _c_float(rot_mag), _c_int(int(head_norm)), _ptr(bias), _ptr(temp), _stream()))
    return q_out


def linear_scan(u: torch.Tensor, offsets, heads: int, dk: int, dv: int, qkv_act: int, q_scale: float, decay: Optional[torch.Tensor],
                w2: Optional[torch.Tensor], b2: Optional[torch.Tensor], r_off: int, tau: float, state: torch.Tensor,
                req_start: torch.Tensor, slot_ids: torch.Tensor, out: torch.Tensor, direct: Optional[torch.Tensor] = None,
                n_direct: int = 0, pieces: Optional[torch.Tensor] = None, piece_reqs: Optional[torch.Tensor] = None,
                bonus: Optional[torch.Tensor] = None, decay_form: int = 0, rank_act: int = 0) -> torch.Tensor:
    """S = diag(a) S + k v^T, o = S^T q over each request's rows of the fused float32 projections ``u`` (columns
    ``offsets = (q, k, v)``), from and into ``state [slots, heads, dk, dv]``; ``out`` float32 ``[T, heads * dv]``.
    Without lists every request runs in one go; with them (int32: ``direct`` requests, ``pieces [n, 2]`` (first row, rows),
    ``piece_reqs [m, 3]`` (request, first piece, pieces)) the pieces run side by side and are joined.  ``bonus`` [heads, dk]:
    a row reads the state before its own decay, its own key times the bonus; ``decay_form`` 1: exp(-exp(z)); ``rank_act``: the
    activation on the decay projection's columns."""
    _need(u, "u", torch.float32); _need(state, "state", torch.float32); _need(out, "out", torch.float32)
    T, nreq = u.shape[0], req_start.numel() - 1
    lib = _build.load("mixers")
    n_pieces = pieces.numel() // 2 if pieces is not None else 0
    scratch, floats = None, 0
    if n_pieces:
        _need(pieces, "pieces", torch.int32); _need(piece_reqs, "piece_reqs", torch.int32)
        floats = n_pieces * heads * dk * dv + (T * heads * dk if w2 is not None else 0)
        scratch = torch.empty(floats, dtype=torch.float32, device=u.device)
    if direct is not None:
        _need(direct, "direct", torch.int32)
        n_direct = direct.numel()
    _check("mixers", lib.jk_linear_scan(
        _ptr(u), _c_int(u.shape[1]), _c_int(offsets[0]), _c_int(offsets[1]), _c_int(offsets[2]), _c_int(heads), _c_int(dk), _c_int(dv),
        _c_int(qkv_act), _c_float(q_scale), _ptr(decay), _ptr(w2), _c_int(dtype_code(w2.dtype) if w2 is not None else F32), _ptr(b2),
        _c_int(r_off), _c_int(w2.shape[1] if w2 is not None else 0), _c_float(tau), _ptr(state), _ptr(req_start), _ptr(slot_ids),
        _c_int(nreq), _c_int(T), _ptr(out), _ptr(direct), _c_int(n_direct), _ptr(pieces), _c_int(n_pieces), _ptr(piece_reqs),
        _c_int(piece_reqs.numel() // 3 if piece_reqs is not None else 0), _ptr(scratch), _c_ll(floats), _c_int(_sm_count(u.device)),
        _ptr(bonus), _c_int(decay_form), _c_int(rank_act), _stream()))
    return out


def norm_gate(o: torch.Tensor, u: torch.Tensor, g_off: int, weight: Optional[torch.Tensor], eps: float, heads: int, dv: int, per_head,
              gate_act: int, out: torch.Tensor) -> torch.Tensor:
    """out = rmsnorm(o) * weight * act(u[:, g_off : g_off + heads * dv]); the norm over all heads or head by head (``per_head``
    2: head by head with a weight for every element of every head; ``weight`` None: none)."""
    _need(o, "o", torch.float32); _need(u, "u", torch.float32); _need(out, "out")
    lib = _build.load("mixers")
    _check("mixers", lib.jk_norm_gate(_ptr(o), _ptr(u), _c_int(u.shape[1]), _c_int(g_off), _ptr(weight), _c_float(eps), _c_int(heads),
                                      _c_int(dv), _c_int(int(per_head)), _c_int(gate_act), _ptr(out), _c_int(dtype_code(out.dtype)),
                                      _c_int(o.shape[0]), _stream()))
    return out


def token_shift(h: torch.Tensor, mu: torch.Tensor, last: torch.Tensor, row_req, req_start, slot_ids, out: torch.Tensor) -> torch.Tensor:
    """out[s, t] = h[t] + (h[t - 1] - h[t]) * mu[s]; the row before a request's first row is ``last[slot]`` (float32), which
    then moves on to the request's last row."""
    _need(h, "h"); _need(mu, "mu", torch.float32); _need(last, "last", torch.float32); _need(out, "out")
    lib = _build.load("mixers")
    _check("mixers", lib.jk_token_shift(_ptr(h), _ptr(mu), _ptr(last), _ptr(row_req), _ptr(req_start), _ptr(slot_ids), _ptr(out),
                                        _c_int(dtype_code(h.dtype)), _c_int(h.shape[0]), _c_int(req_start.numel() - 1), _c_int(h.shape[1]),
                                        _c_int(mu.shape[0]), _stream()))
    return out


def act_rows(u: torch.Tensor, out: torch.Tensor, act: int, table: Optional[torch.Tensor] = None, table_off: int = 0,
             tokens: Optional[torch.Tensor] = None) -> torch.Tensor:
    """out = act(u) in the type of ``out``; ``u`` float32 rows (a view of wider rows is fine).  With ``table`` (of ``out``'s type, a
    row per token id): times table[tokens[t], table_off : table_off + n]."""
    _need(u, "u", torch.float32, contiguous=False); _need(out, "out")
    lib = _build.load("mixers")
    _check("mixers", lib.jk_act_rows(_ptr(u), _c_int(u.stride(0)), _ptr(out), _c_int(dtype_code(out.dtype)), _c_int(out.shape[0]),
                                     _c_int(out.shape[1]), _c_int(act), _ptr(table), _c_ll(table.shape[1] if table is not None else 0),
                                     _c_int(table_off), _ptr(tokens), _stream()))
    return out


def rotate_rows(u: torch.Tensor, q_off: int, k_off: int, heads: int, dk: int, freq: torch.Tensor, positions: torch.Tensor, half: bool = True,
                magnitude: float = 1.0) -> torch.Tensor:
    """Rotate, in place, the first 2 * len(freq) elements of ``heads`` heads of ``dk`` at column ``q_off`` of the float32 rows ``u`` and
    of as many at ``k_off`` (< 0: none) by positions * freq."""
    _need(u, "u", torch.float32); _need(freq, "freq", torch.float32)
    lib = _build.load("mixers")
    _check("mixers", lib.jk_rotate_rows(_ptr(u), _c_int(u.shape[1]), _c_int(q_off), _c_int(k_off), _c_int(heads), _c_int(dk), _ptr(freq),
                                        _c_int(2 * freq.numel()), _c_int(1 if half else 0), _c_float(magnitude), _ptr(positions), _c_int(u.shape[0]),
                                        _stream()))
    return u


# ---- csrc/blocks.cu ---------------------------------------------------------------------------------------------------
ACT_RELU, ACT_GELU_ERF, ACT_SWISH_CLAMP, ACT_TANH = 4, 5, 6, 7


def norm_add(delta: torch.Tensor, x: torch.Tensor, weight: torch.Tensor, eps: float, next_weight: Optional[torch.Tensor] = None,
             next_eps: float = 0.0, out: Optional[torch.Tensor] = None, next_weight2: Optional[torch.Tensor] = None,
             out2: Optional[torch.Tensor] = None) -> torch.Tensor:
    """x += rmsnorm(delta) * weight; with ``out``: out = rmsnorm(x) * next_weight (or x itself) in out's type; with ``out2``: the same
    with next_weight2."""
    _need(delta, "delta", torch.float32); _need(x, "x", torch.float32); _need(weight, "weight", torch.float32)
    rows, d = x.shape
    lib = _build.load("blocks")
    _check("blocks", lib.jk_norm_add(_ptr(delta), _ptr(x), _ptr(weight), _c_float(eps), _ptr(next_weight), _c_float(next_eps), _ptr(out),
                                     _ptr(next_weight2), _ptr(out2), _c_int(dtype_code(out.dtype) if out is not None else F32), _c_int(rows), _c_int(d), _stream()))
    return x


def norm_pair_kept_floats(width: int) -> int:
    """Floats of one of the two rows that ``norm_pair`` keeps of a request: the row, and how long the sequence was then."""
    return (width + 3) // 4 * 4 + 4


def norm_pair(x: torch.Tensor, weight: torch.Tensor, eps: float, h: torch.Tensor, mu: Optional[torch.Tensor] = None,
              state: Optional[torch.Tensor] = None, row_req=None, req_start=None, req_pos=None, slot_ids=None, weight2: Optional[torch.Tensor] = None,
              eps2: float = 0.0, h2: Optional[torch.Tensor] = None) -> torch.Tensor:
    """h[t] = n_t + (n_(t-1) - n_t) * mu with n = rmsnorm(x) * weight (``mu`` None: n itself), the row before a request's first
    row being the one that ``state`` ``[slots, 2, norm_pair_kept_floats(width)]`` keeps of it, which then moves on to the n of its
    last row; h2 = rmsnorm(x) * weight2 if given."""
    _need(x, "x", torch.float32); _need(weight, "weight", torch.float32); _need(h, "h")
    lib = _build.load("blocks")
    _check("blocks", lib.jk_norm_pair(_ptr(x), _ptr(weight), _ptr(mu), _c_float(eps), _ptr(weight2), _c_float(eps2), _ptr(state), _ptr(row_req),
                                      _ptr(req_start), _ptr(req_pos), _ptr(slot_ids), _ptr(h), _ptr(h2), _c_int(dtype_code(h.dtype)),
                                      _c_int(x.shape[0]), _c_int(x.shape[1]), _stream()))
    return h


def latent_qkv(u: torch.Tensor, q_off: int, kv_off: int, heads: int, dn: int, dr: int, latent: int, rot_dims: int,
               freq: Optional[torch.Tensor], magnitude: float, norm_weight: torch.Tensor, eps: float, positions, row_req, block_table,
               page_size: int, q_plain: torch.Tensor, q_full: Optional[torch.Tensor], pages: Optional[torch.Tensor],
               q_norm: Optional[torch.Tensor] = None, q_rank: int = 0, rot_half: bool = False) -> None:
    """Queries and cache rows of a latent attention from the fused float32 projection ``u`` (see csrc/blocks.cu); ``kv_off`` < 0: the
    queries only (``norm_weight``, ``block_table`` and ``pages`` may be None)."""
    _need(u, "u", torch.float32); _need(q_plain, "q_plain")
    lib = _build.load("blocks")
    _check("blocks", lib.jk_latent_qkv(
        _ptr(u), _c_int(u.shape[1]), _c_int(q_off), _c_int(kv_off), _c_int(heads), _c_int(dn), _c_int(dr), _c_int(latent), _c_int(rot_dims),
        _ptr(freq), _c_float(magnitude), _ptr(norm_weight), _c_float(eps), _ptr(positions), _ptr(row_req), _ptr(block_table),
        _c_int(block_table.shape[1] if block_table is not None else 1), _c_int(page_size), _ptr(q_plain), _ptr(q_full), _ptr(pages),
        _c_int(dtype_code(q_plain.dtype)), _c_int(u.shape[0]), _ptr(q_norm), _c_int(q_rank), _c_int(1 if rot_half else 0), _stream()))


def head_linear(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor, out_head_stride: int, gate: Optional[torch.Tensor] = None,
                gate_ld: int = 0, gate_head: bool = False) -> torch.Tensor:
    """out[t, h, :n] = x[t, h] w[h]^T for ``w [heads, n, k]``, times sigmoid(gate[t, h n + j]) if given (float32 rows ``gate_ld``
    apart; ``gate_head``: sigmoid(gate[t, h]))."""
    _need(x, "x"); _need(w, "w"); _need(out, "out")
    H, n, k = w.shape
    lib = _build.load("blocks")
    _check("blocks", lib.jk_head_linear(_ptr(x), _ptr(w), _ptr(out), _c_int(dtype_code(x.dtype)), _c_int(x.shape[0]), _c_int(H), _c_int(n),
                                        _c_int(k), _c_int(out_head_stride), _ptr(gate), _c_int(gate_ld), _c_int(1 if gate_head else 0), _stream()))
    return out


def latent_attention(q: torch.Tensor, pages: torch.Tensor, out: torch.Tensor, positions, row_req, block_table, heads: int, latent: int,
                     dr: int, scale: float, splits: int = 1, req_start: Optional[torch.Tensor] = None, window: int = 0,
                     sink_w: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Causal attention of ``heads`` query heads ``[T, heads, latent + dr]`` over the paged rows ``[pages, page, latent + dr]``;
    out ``[T, heads, latent]``.  ``splits`` > 1 cuts each row's keys into that many ranges.  With ``req_start`` (int32, the first
    row of each request and the row count) bfloat16 rows run on the tensor cores.  ``sink_w`` (float32 [heads]): one more key per
    softmax, of that score and without a value."""
    _need(q, "q"); _need(pages, "pages"); _need(out, "out")
    T = q.shape[0]
    lib = _build.load("blocks")
    lib.jk_latent_attention_scratch.restype = ctypes.c_longlong
    floats = lib.jk_latent_attention_scratch(_c_int(T), _c_int(heads), _c_int(latent), _c_int(splits))
    part = torch.empty(max(int(floats), 1), dtype=torch.float32, device=q.device) if splits > 1 else None
    _check("blocks", lib.jk_latent_attention(_ptr(q), _ptr(pages), _ptr(out), _ptr(part), _c_int(dtype_code(q.dtype)), _ptr(positions),
                                             _ptr(row_req), _ptr(block_table), _c_int(block_table.shape[1]), _c_int(pages.shape[-2]),
                                             _c_int(T), _c_int(heads), _c_int(latent), _c_int(dr), _c_float(scale), _c_int(splits), _ptr(req_start),
                                             _c_int(req_start.numel() - 1 if req_start is not None else 0), _c_int(window), _ptr(sink_w), _stream()))
    return out


def causal_conv(u: torch.Tensor, off: int, channels: int, taps: torch.Tensor, bias: Optional[torch.Tensor], act: int,
                tail: Optional[torch.Tensor], row_req, req_start, slot_ids, y32: Optional[torch.Tensor], yT: Optional[torch.Tensor],
                in_bias: Optional[torch.Tensor] = None) -> None:
    """y = act(bias + taps over time of u[:, off : off + channels] (+ in_bias)); the tails ``[slots, taps - 1, channels]`` move forward."""
    _need(u, "u", torch.float32); _need(taps, "taps", torch.float32)
    lib = _build.load("blocks")
    _check("blocks", lib.jk_causal_conv(_ptr(u), _c_int(u.shape[1]), _c_int(off), _c_int(channels), _ptr(taps), _ptr(bias), _c_int(taps.shape[1]),
                                        _c_int(act), _ptr(tail), _ptr(row_req), _ptr(req_start), _ptr(slot_ids), _ptr(y32), _ptr(yT),
                                        _c_int(dtype_code(yT.dtype) if yT is not None else F32), _c_int(u.shape[0]),
                                        _c_int(req_start.numel() - 1), _ptr(in_bias), _stream()))


def selective_scan(x: torch.Tensor, low: torch.Tensor, dt_rank: int, states: int, z: torch.Tensor, z_ld: int, w_dt, dt_bias, A, skip,
                   state: torch.Tensor, req_start, slot_ids, out: torch.Tensor, dt_buf: Optional[torch.Tensor] = None) -> torch.Tensor:
    """The selective scan of csrc/blocks.cu over each request's rows, from and into ``state [slots, channels, states]``.
    ``w_dt`` is of ``out``'s type.  ``dt_buf`` (float32 ``[T, channels]``): room in which the step sizes are made ahead."""
    for t, n in ((x, "x"), (low, "low"), (dt_bias, "dt_bias"), (A, "A"), (skip, "skip"), (state, "state")):
        _need(t, n, torch.float32)
    _need(w_dt, "w_dt", out.dtype)
    _need(z, "z", torch.float32, contiguous=False)
    lib = _build.load("blocks")
    _check("blocks", lib.jk_selective_scan(_ptr(x), _ptr(low), _c_int(low.shape[1]), _c_int(dt_rank), _c_int(states), _c_int(x.shape[1]),
                                           _ptr(z), _c_int(z_ld), _ptr(w_dt), _ptr(dt_bias), _ptr(A), _ptr(skip), _ptr(state), _ptr(req_start),
                                           _ptr(slot_ids), _c_int(req_start.numel() - 1), _ptr(out), _c_int(dtype_code(out.dtype)), _ptr(dt_buf),
                                           _c_int(dt_buf.shape[1] if dt_buf is not None else 0), _c_int(x.shape[0]), _stream()))
    return out


def routed_experts(h: torch.Tensor, router: torch.Tensor, w_gate_up: torch.Tensor, w_down: torch.Tensor, delta: torch.Tensor, add: bool,
                   experts: int, top: int, act: int, score_form: int = 0, limit: float = 0.0, router_bias: Optional[torch.Tensor] = None,
                   gate_w: Optional[torch.Tensor] = None, identity: int = 0, groups=(0, 0), correction: Optional[torch.Tensor] = None,
                   x: Optional[torch.Tensor] = None, x_scale: float = 1.0, pending: Optional[torch.Tensor] = None,
                   pending_scale: float = 1.0, score_scale: float = 1.0) -> torch.Tensor:
    """delta (+)= sum over each row's ``top`` experts of largest sigmoid(router h) of expert(score * h); ``w_gate_up``
    ``[experts * 2 ff, d]`` (an expert's gate rows, then its up rows), ``w_down [experts * d, ff]``.  ``identity``, ``groups``,
    ``correction``: see csrc/blocks.cu (score_form 2).  With ``x`` (float32 ``[T, d]``) the sum goes there instead:
    x += x_scale * sum + pending_scale * pending."""
    _need(h, "h"); _need(router, "router", torch.float32); _need(delta, "delta", torch.float32)
    T, d = h.shape
    ff = w_down.shape[1]
    lib = _build.load("blocks")
    lib.jk_routed_experts_workspace.restype = ctypes.c_longlong
    route = torch.empty(int(lib.jk_routed_experts_workspace(_c_int(T), _c_int(experts + identity), _c_int(top))), dtype=torch.int32, device=h.device)
    act_buf = torch.empty(T * top, ff, dtype=h.dtype, device=h.device)
    y = torch.empty(T * top, d, dtype=torch.float32, device=h.device)
    _check("blocks", lib.jk_routed_experts(_ptr(h), _ptr(router), _ptr(w_gate_up), _ptr(w_down), _ptr(delta), _c_int(1 if add else 0),
                                           _c_int(dtype_code(h.dtype)), _c_int(T), _c_int(d), _c_int(ff), _c_int(experts), _c_int(top),
                                           _c_int(act), _ptr(route), _ptr(act_buf), _ptr(y), _c_int(score_form), _c_float(limit), _ptr(router_bias), _ptr(gate_w),
                                           _c_int(identity), _c_int(groups[0]), _c_int(groups[1]), _ptr(correction), _ptr(x), _c_float(x_scale),
                                           _ptr(pending), _c_float(pending_scale), _c_float(score_scale), _stream()))
    return delta


def softcap(x: torch.Tensor, cap: float) -> torch.Tensor:
    _need(x, "x", torch.float32)
    lib = _build.load("blocks")
    _check("blocks", lib.jk_softcap(_ptr(x), _c_float(cap), _c_ll(x.numel()), _stream()))
    return x


def argmax(logits: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    _need(logits, "logits", torch.float32, contiguous=False); _need(out, "out", torch.int32)
    n, v = logits.shape
    if logits.stride(1) != 1:
        raise KernelError("argmax: rows must be contiguous")
    lib = _build.load("sampling")
    lib.jk_argmax_scratch_bytes.restype = ctypes.c_longlong
    need = lib.jk_argmax_scratch_bytes(_c_int(n), _c_int(v))
    scratch = torch.empty(need, dtype=torch.uint8, device=logits.device) if need else None
    _check("sampling", lib.jk_argmax(_ptr(logits), _c_ll(logits.stride(0)), _c_int(n), _c_int(v), _ptr(out),
                                     _ptr(scratch), _stream()))
    return out


def sample(logits: torch.Tensor, temperature: torch.Tensor, topk: torch.Tensor, topp: torch.Tensor,
           uniform: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    _need(logits, "logits", torch.float32, contiguous=False); _need(out, "out", torch.int32)
    _need(temperature, "temperature", torch.float32); _need(topk, "topk", torch.int32)
    _need(topp, "topp", torch.float32); _need(uniform, "uniform", torch.float32)
    n, v = logits.shape
    if logits.stride(1) != 1:
        raise KernelError("sample: rows must be contiguous")
    if min(temperature.numel(), topk.numel(), topp.numel(), uniform.numel(), out.numel()) < n:
        raise KernelError("sample: a per-row array is shorter than the number of rows")
    lib = _build.load("sampling")
    _check("sampling", lib.jk_sample(_ptr(logits), _c_ll(logits.stride(0)), _c_int(n), _c_int(v), _ptr(temperature),
                                     _ptr(topk), _ptr(topp), _ptr(uniform), _ptr(out), _stream()))
    return out


def build_all(verbose: bool = True):
    return _build.build_all(verbose)


def add_rows(x: torch.Tensor, table: torch.Tensor, index: Optional[torch.Tensor], row: int = -1) -> torch.Tensor:
    """x[t] += table[index[t]] (``index`` int32 per row), or table[row] for every row when ``index`` is None; x float32, the
    table float32 or bfloat16."""
    _need(x, "x", torch.float32); _need(table, "table")
    lib = _build.load("blocks")
    _check("blocks", lib.jk_add_rows(_ptr(x), _ptr(table), _c_int(dtype_code(table.dtype)), _c_int(table.shape[0]), _ptr(index), _c_int(row),
                                     _c_int(x.shape[0]), _c_int(x.shape[1]), _stream()))
    return x


def delta_rule(c: torch.Tensor, offsets, u: torch.Tensor, b_off: int, a_off: int, a_log: torch.Tensor, dt_bias: torch.Tensor, heads: int,
               groups: int, dk: int, dv: int, q_scale: float, unit_eps: float, state: torch.Tensor, req_start: torch.Tensor,
               slot_ids: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    """The gated delta rule over each request's rows (csrc/mixers.cu): ``c`` float32 rows with q, k, v at the columns
    ``offsets`` (after their convolutions), ``u`` float32 rows with the write strength's logits at ``b_off`` and the decay's at
    ``a_off``; from and into ``state [slots, heads, dk, dv]``; ``out`` float32 ``[T, heads * dv]``."""
    for t, n in ((c, "c"), (u, "u"), (a_log, "a_log"), (dt_bias, "dt_bias"), (state, "state"), (out, "out")):
        _need(t, n, torch.float32)
    lib = _build.load("mixers")
    lib.jk_delta_rule_scratch_floats.restype = ctypes.c_longlong
    scratch = torch.empty(int(lib.jk_delta_rule_scratch_floats(_c_int(c.shape[0]), _c_int(heads), _c_int(groups), _c_int(dk))) + 4,
                          dtype=torch.float32, device=c.device)
    _check("mixers", lib.jk_delta_rule(_ptr(c), _c_int(c.shape[1]), _c_int(offsets[0]), _c_int(offsets[1]), _c_int(offsets[2]), _ptr(u),
                                       _c_int(u.shape[1]), _c_int(b_off), _c_int(a_off), _ptr(a_log), _ptr(dt_bias), _c_int(heads), _c_int(groups),
                                       _c_int(dk), _c_int(dv), _c_float(q_scale), _c_float(unit_eps), _ptr(state), _ptr(req_start),
                                       _ptr(slot_ids), _c_int(req_start.numel() - 1), _ptr(out), _ptr(scratch), _c_int(c.shape[0]), _stream()))
    return out


def embed_pair(tokens, positions, row_req, req_start, req_pos, slot_ids, table: torch.Tensor, pairs: Optional[torch.Tensor], mul_prev: int,
               mul_cur: int, scale: float, state: Optional[torch.Tensor], weight: Optional[torch.Tensor], eps: float, x: torch.Tensor) -> torch.Tensor:
    """x = rmsnorm(scale * table[token] + pairs[(previous * mul_prev + token * mul_cur) % buckets]) * weight; ``pairs`` has buckets + 1
    rows, the last one for position 0; ``state`` [slots, 2, 2] of four bytes each keeps the requests' last tokens."""
    _need(table, "table"); _need(x, "x", torch.float32)
    lib = _build.load("blocks")
    _check("blocks", lib.jk_embed_pair(_ptr(tokens), _ptr(positions), _ptr(row_req), _ptr(req_start), _ptr(req_pos), _ptr(slot_ids), _ptr(table),
                                       _ptr(pairs), _c_int(dtype_code(table.dtype)), _c_int(pairs.shape[0] - 1 if pairs is not None else 0),
                                       _c_int(mul_prev), _c_int(mul_cur), _c_float(scale), _ptr(state), _ptr(weight), _c_float(eps), _ptr(x),
                                       _c_int(x.shape[0]), _c_int(x.shape[1]), _stream()))
    return x


def join_parts(x: torch.Tensor, p1: torch.Tensor, w1: Optional[torch.Tensor], eps1: float, p2: Optional[torch.Tensor] = None,
               w2: Optional[torch.Tensor] = None, eps2: float = 0.0, p3: Optional[torch.Tensor] = None, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """x += rmsnorm(p1) * w1 + rmsnorm(p2) * w2 + p3 (a part without a weight as it is); out = x in out's type."""
    _need(x, "x", torch.float32); _need(p1, "p1", torch.float32)
    lib = _build.load("blocks")
    _check("blocks", lib.jk_join_parts(_ptr(x), _ptr(p1), _ptr(w1), _c_float(eps1), _ptr(p2), _ptr(w2), _c_float(eps2), _ptr(p3), _ptr(out),
                                       _c_int(dtype_code(out.dtype) if out is not None else F32), _c_int(x.shape[0]), _c_int(x.shape[1]), _stream()))
    return x


def gated_recurrence(u: torch.Tensor, w_r: torch.Tensor, w_i: torch.Tensor, b_r: torch.Tensor, b_i: torch.Tensor, rate: torch.Tensor, y: torch.Tensor,
                     y_bias: Optional[torch.Tensor], act: int, state: torch.Tensor, req_start, slot_ids, out: torch.Tensor, direct=None,
                     n_direct: int = 0, pieces=None, n_pieces: int = 0, piece_reqs=None, n_piece_reqs: int = 0) -> torch.Tensor:
    """The real-gated recurrence of csrc/blocks.cu over each request's rows ``u [T, C]``, from and into ``state [slots, C]``; ``w_r``,
    ``w_i`` ``[blocks, n, n]`` of ``out``'s type; ``y`` float32 rows (a view of wider ones is fine).  The lists are those of
    ``linear_scan``."""
    for t, n in ((u, "u"), (b_r, "b_r"), (b_i, "b_i"), (rate, "rate"), (state, "state")):
        _need(t, n, torch.float32)
    _need(w_r, "w_r", out.dtype); _need(w_i, "w_i", out.dtype); _need(y, "y", torch.float32, contiguous=False)
    T, C = u.shape
    lib = _build.load("blocks")
    lib.jk_gated_recurrence_scratch_floats.restype = ctypes.c_longlong
    floats = int(lib.jk_gated_recurrence_scratch_floats(_c_int(T), _c_int(C), _c_int(n_pieces)))
    scratch = torch.empty(max(floats, 1), dtype=torch.float32, device=u.device)
    _check("blocks", lib.jk_gated_recurrence(_ptr(u), _ptr(w_r), _ptr(w_i), _ptr(b_r), _ptr(b_i), _ptr(rate), _ptr(y), _c_int(y.stride(0)), _ptr(y_bias),
                                             _c_int(act), _ptr(state), _ptr(req_start), _ptr(slot_ids), _c_int(req_start.numel() - 1), _ptr(out),
                                             _c_int(dtype_code(out.dtype)), _c_int(T), _c_int(C), _c_int(w_r.shape[0]), _ptr(direct), _c_int(n_direct),
                                             _ptr(pieces), _c_int(n_pieces), _ptr(piece_reqs), _c_int(n_piece_reqs), _ptr(scratch), _c_ll(floats),
                                             _stream()))
    return out
