"""Python faces of the CUDA kernels: argument checks, then a ctypes call on the current stream.

Every function works on CUDA tensors only and raises if the kernel library is missing;
nothing here falls back to torch operators.  The dense matrix products of the bfloat16
path go to the library GEMM (cuBLASLt through ``torch``), as the reference's go to
``cublasSgemm`` (kernels/linear.cu:25-27); everything around them is this package's own.
"""
from __future__ import annotations

import ctypes
import weakref
from ctypes import c_float, c_int, c_void_p
from typing import Optional

import torch

from .library import kernels, optional_kernels

F32, BF16 = 0, 1
ACT = {None: 0, "none": 0, "gelu_erf": 1, "gelu_tanh": 2, "silu": 3, "sigmoid": 4, "relu2": 5, "tanh": 6}      # relu2: relu(v)^2

_STATUS = {-1: "unsupported dtype", -2: "a size that the kernel does not take",
           -3: "misaligned pointer or stride", -4: "size too large for this kernel"}


class KernelError(RuntimeError):
    pass


_launches = 0


def launch_count() -> int:
    """Kernel launches of this package since the last reset (captured launches count once, at capture)."""
    return _launches


def reset_launch_count() -> None:
    global _launches
    _launches = 0


def _check(status: int, what: str, detail: str = "", launches: int = 1) -> None:
    global _launches
    if status == 0:
        _launches += launches
        return
    if status < 0:
        raise KernelError(f"{what}: {_STATUS.get(status, 'error %d' % status)}{(' (' + detail + ')') if detail else ''}")
    raise KernelError(f"{what}: CUDA error {status} at launch {detail}")


def dtype_code(dt: torch.dtype) -> int:
    if dt == torch.float32:
        return F32
    if dt == torch.bfloat16:
        return BF16
    raise KernelError(f"dtype {dt} is not supported (float32 or bfloat16)")


def _ptr(t: Optional[torch.Tensor]):
    return c_void_p(t.data_ptr()) if t is not None else None


_raw_stream = getattr(torch._C, "_cuda_getCurrentRawStream", None)
_raw_device = getattr(torch._C, "_cuda_getDevice", None)


def _stream():
    """The current stream of the current device as a raw handle.  torch.cuda.current_stream() builds a Python
    object through several layers (about 5 us, a third of the host's share of a launch); the two calls below are
    what it ends in."""
    if _raw_stream is not None and _raw_device is not None:
        return c_void_p(_raw_stream(_raw_device()))
    return c_void_p(torch.cuda.current_stream().cuda_stream)


def raw_stream_handle():
    """The current stream's raw handle (an int), or None where torch does not offer the fast call."""
    if _raw_stream is not None and _raw_device is not None:
        return _raw_stream(_raw_device())
    return None


def _need_cuda(*ts):
    for t in ts:
        if t is not None and not t.is_cuda:
            raise KernelError("kernels take CUDA tensors only; there is no CPU path")


NORM_MAX_WIDTH = 200 * 1024 // 4 - 33     # the widest row add_layernorm takes (cbis_norm_max_width() says the same)
ATTENTION_MAX_HEAD_DIM = 512             # the general attention kernel's limit; the tiled ones take less and say so


def embed_pos_add(tokens, positions, wte, wpe, out, err, multiplier: float = 1.0):
    """out[r] = wte[tokens[r]] * multiplier + wpe[positions[r]] in 32-bit; err (int32[1]) is set on a bad index."""
    _need_cuda(tokens, positions, wte, wpe, out, err)
    T, d = out.shape
    assert out.dtype == torch.float32 and out.is_contiguous() and wte.is_contiguous()
    assert tokens.dtype == torch.int32 and positions.dtype == torch.int32
    st = kernels().cbis_embed_pos_add(_ptr(tokens), _ptr(positions), _ptr(wte), _ptr(wpe), _ptr(out),
                                      c_int(T), c_int(d), c_int(wte.shape[0]),
                                      c_int(wpe.shape[0] if wpe is not None else 0),
                                      c_int(dtype_code(wte.dtype)), c_float(multiplier), _ptr(err), _stream())
    _check(st, "embed_pos_add", f"T={T} d={d}")


def add_layernorm(x, delta, delta_bias, gamma, beta, eps, out, rows=None):
    """x += delta + delta_bias (32-bit, in place unless ``rows``); out = LayerNorm(x) * gamma + beta.

    ``rows`` (int32[R]) selects source rows: out[r] = LN(x[rows[r]] + ...), x is left as it is.
    ``gamma`` None: no normalisation, out = x + delta + delta_bias in ``out``'s dtype."""
    _need_cuda(x, delta, delta_bias, gamma, beta, out, rows)
    d = x.shape[-1]
    R = rows.shape[0] if rows is not None else x.shape[0]
    assert x.dtype == torch.float32 and x.is_contiguous() and out.is_contiguous() and out.shape[-1] == d
    assert gamma is None or gamma.dtype == torch.float32
    assert beta is None or (gamma is not None and beta.dtype == torch.float32)
    assert delta is None or (delta.is_contiguous() and delta.shape == x.shape)
    assert delta_bias is None or delta_bias.dtype == torch.float32
    assert out.shape[0] >= R
    st = kernels().cbis_add_layernorm(_ptr(x), _ptr(delta), c_int(dtype_code(delta.dtype) if delta is not None else 0),
                                      _ptr(delta_bias), _ptr(gamma), _ptr(beta), c_float(eps), _ptr(out),
                                      c_int(dtype_code(out.dtype)), _ptr(rows), c_int(R), c_int(d), _stream())
    _check(st, "add_layernorm", f"rows={R} width={d}")


def add_delta(x, delta, delta_bias):
    """x += delta + delta_bias (the 32-bit residual stream, in place): what a layer left pending, added without a
    norm for a part that normalises inside its own kernel."""
    add_layernorm(x, delta, delta_bias, None, None, 0.0, torch.empty_like(x, dtype=torch.bfloat16))


def bias_act(x, bias, act):
    """x = act(x + bias) in place, arithmetic in 32-bit."""
    _need_cuda(x, bias)
    M, N = x.shape
    assert x.is_contiguous()
    st = kernels().cbis_bias_act(_ptr(x), _ptr(bias), c_int(ACT[act]), c_int(M), c_int(N),
                                 c_int(dtype_code(x.dtype)), _stream())
    _check(st, "bias_act", f"M={M} N={N}")


def scale_soft_cap(x, scale: float, cap: float):
    """x = cap * tanh(x * scale / cap) if cap > 0 else x * scale, in place on 32-bit values."""
    _need_cuda(x)
    M, N = x.shape
    assert x.dtype == torch.float32 and x.is_contiguous()
    st = kernels().cbis_scale_soft_cap(_ptr(x), c_float(scale), c_float(cap), c_int(M), c_int(N), _stream())
    _check(st, "scale_soft_cap", f"M={M} N={N}")


def bias_act_out(src, bias, act, dst):
    """dst = act(src + bias): 32-bit sums in, activations out with one rounding."""
    _need_cuda(src, bias, dst)
    M, N = src.shape
    assert src.dtype == torch.float32 and src.is_contiguous() and dst.is_contiguous() and dst.shape == src.shape
    st = kernels().cbis_bias_act_out(_ptr(src), _ptr(bias), c_int(ACT[act]), _ptr(dst), c_int(M), c_int(N),
                                     c_int(dtype_code(dst.dtype)), _stream())
    _check(st, "bias_act_out", f"M={M} N={N}")


def linear_f32(x, w, bias, act, out, w_is_nk=False, variant=0):
    """out = act(x @ W + bias) on the FP32 units; W is [K,N], or [N,K] with ``w_is_nk``.  ``variant`` 1 keeps the
    cp.async kernel out (all kernels sum along k in the same order and give the same bits)."""
    _need_cuda(x, w, bias, out)
    M, K = x.shape
    N = w.shape[0] if w_is_nk else w.shape[1]
    assert x.dtype == torch.float32 and w.dtype == torch.float32 and out.dtype == torch.float32
    assert (w.shape[1] if w_is_nk else w.shape[0]) == K and w.is_contiguous()
    assert x.stride(1) == 1 and out.stride(1) == 1 and out.shape[0] >= M and out.shape[1] == N
    st = kernels().cbis_linear_f32(_ptr(x), _ptr(w), _ptr(bias), _ptr(out), c_int(M), c_int(N), c_int(K),
                                   c_int(1 if w_is_nk else 0), c_int(ACT[act]), c_int(x.stride(0)),
                                   c_int(out.stride(0)), c_int(variant), _stream())
    _check(st, "linear_f32", f"M={M} N={N} K={K}")


SMALL_M = int(__import__("os").environ.get("CBIS_SMALL_M", "16"))      # rows up to which the weight-streaming kernel takes a bfloat16 product (it can take 64; measured at batch 32 and 64 of the 1.3B sizes: the library product is 27-33 % faster per step there)


_next_weight = {}      # data_ptr of a weight -> weak reference to the weight used after it
PREFETCH_AHEAD = int(__import__("os").environ.get("CBIS_PREFETCH_AHEAD", "1"))   # products ahead (measured: 1 is best, 6,305 tok/s at batch 8; 0: 6,014, 2: 6,205, 3: 5,975)
PREFETCH_CAP = 64 << 20   # bytes of a successor's weights brought into L2 ahead of time (L2 holds 126 MB)


def add_weight_order(weights) -> None:
    """Tells the few-rows product in which order a decode step uses its weights (a cycle: after the
    last comes the first of the next step), so that each product can prefetch its successor's weights
    into L2 while it runs.  Only weak references are kept: a freed model's entries die with it."""
    import weakref
    ws = [w for w in weights if w is not None and w.is_cuda and w.dtype == torch.bfloat16]
    ahead = PREFETCH_AHEAD % max(1, len(ws))
    for a, b in zip(ws, ws[ahead:] + ws[:ahead]):
        if a.data_ptr() != b.data_ptr():
            _next_weight[a.data_ptr()] = weakref.ref(b)
    for k in [k for k, r in _next_weight.items() if r() is None]:
        del _next_weight[k]


def _next_of(w_nk):
    """(pointer, bytes) of the weight used after ``w_nk``, for the L2 prefetch the weight-streaming kernels issue."""
    ref = _next_weight.get(w_nk.data_ptr())
    nxt = ref() if ref is not None else None
    return _ptr(nxt), ctypes.c_ulonglong(min(nxt.numel() * 2, PREFETCH_CAP) if nxt is not None else 0)


SMALL_WEIGHT = 1 << 20


def gemm_small_m(x, w_nk, bias, act, out, accumulate=False, group_n: int = 0, act_from: int = 0):
    """out = act(x @ w_nk^T + bias) for up to 64 rows of bfloat16, 32-bit accumulation (weight streaming).
    ``accumulate`` (32-bit ``out`` only): the result is added to what ``out`` holds.  ``group_n`` > 0 (a multiple of 16):
    the output's columns come in groups of so many (the last may be narrower), and group i multiplies columns
    i K .. (i + 1) K - 1 of x, K being the weights' width.  With groups the activation is for columns from ``act_from`` on."""
    _need_cuda(x, w_nk, bias, out)
    M = x.shape[0]
    N, K = w_nk.shape
    assert x.dtype == torch.bfloat16 and w_nk.dtype == torch.bfloat16 and w_nk.is_contiguous()
    assert x.shape[1] == (-(-N // group_n) * K if group_n else K)
    assert x.stride(1) == 1 and out.stride(1) == 1 and out.shape == (M, N)
    if accumulate and out.dtype != torch.float32:
        raise KernelError("gemm_small_m: a product is added into a 32-bit matrix only")
    nxt, nbytes = _next_of(w_nk)
    st = kernels().cbis_gemm_small_m_bf16(_ptr(x), c_int(x.stride(0)), _ptr(w_nk), _ptr(bias), _ptr(out),
                                          c_int(out.stride(0)), c_int(M), c_int(N), c_int(K), c_int(ACT[act]),
                                          c_int(dtype_code(out.dtype)), nxt, nbytes, c_int(1 if accumulate else 0), _stream(),
                                          c_int(group_n), c_int(act_from))
    _check(st, "gemm_small_m", f"M={M} N={N} K={K}")


LN_LINEAR_MAX_ROWS = 8


_ln_max_k = []


def ln_linear_max_k() -> int:
    if not _ln_max_k:
        _ln_max_k.append(int(kernels().cbis_gemm_ln_small_m_max_k()))
    return _ln_max_k[0]


# 1: decode steps of up to 8 rows normalise inside the product's kernel and add the layer's results straight into the
# residual stream (5 kernels a layer instead of 7).  Off by default: measured at the 1.3B sizes it is the slower form,
# 0.941 ms against 0.900 per step at batch 1 and 1.258 against 1.220 at batch 8; with programmatic dependent launch the
# separate norm kernel already runs under the next product's first weight loads.
USE_LN_LINEAR = __import__("os").environ.get("CBIS_LN_LINEAR", "0") == "1"


def ln_linear_takes(ctx, norm, w_nk) -> bool:
    """Whether this step's rows can go through ``ln_linear`` with this norm and weight: a bfloat16 step of up to 8
    rows, a LayerNorm with weight and bias over rows the kernel takes."""
    if not USE_LN_LINEAR or ctx.dtype != torch.bfloat16 or not 0 < ctx.n_rows <= LN_LINEAR_MAX_ROWS:
        return False
    if norm.as_layernorm() is None:
        return False
    if w_nk is None or not w_nk.is_cuda or w_nk.dtype != torch.bfloat16:
        return False
    K = w_nk.shape[1]
    return K == norm.as_layernorm()[0].numel() and K % 8 == 0 and K <= ln_linear_max_k()


def ln_linear(x, gamma, beta, eps, w_nk, bias, act, out):
    """out = act(LayerNorm(x) @ w_nk^T + bias) for up to 8 rows: x the 32-bit rows, statistics in 32-bit, the
    normalised rows rounded to bfloat16 (as the separate norm kernel hands them to the product), w_nk bfloat16."""
    _need_cuda(x, gamma, beta, w_nk, bias, out)
    M, K = x.shape
    N = w_nk.shape[0]
    assert x.dtype == torch.float32 and w_nk.dtype == torch.bfloat16 and w_nk.is_contiguous() and w_nk.shape[1] == K
    assert gamma.dtype == torch.float32 and beta.dtype == torch.float32 and gamma.numel() == K and beta.numel() == K
    assert x.stride(1) == 1 and out.stride(1) == 1 and out.shape == (M, N)
    nxt, nbytes = _next_of(w_nk)
    st = kernels().cbis_gemm_ln_small_m(_ptr(x), c_int(x.stride(0)), _ptr(gamma), _ptr(beta), ctypes.c_float(eps),
                                        _ptr(w_nk), _ptr(bias), _ptr(out), c_int(out.stride(0)), c_int(M), c_int(N),
                                        c_int(K), c_int(ACT[act]), c_int(dtype_code(out.dtype)), nxt, nbytes, _stream())
    _check(st, "ln_linear", f"M={M} N={N} K={K}")


def gemm_few_rows(x, w_nk, bias, act, out, ksplit=0):
    """out = act(x @ w_nk^T + bias) for up to 64 rows of bfloat16 on the tcgen05 tensor cores with the operands
    swapped: the weights stream through shared memory by TMA, K split over the blocks of a cluster
    (``ksplit`` 0: the launcher's choice)."""
    _need_cuda(x, w_nk, bias, out)
    M, K = x.shape
    N = w_nk.shape[0]
    assert x.dtype == torch.bfloat16 and w_nk.dtype == torch.bfloat16 and w_nk.is_contiguous() and w_nk.shape[1] == K
    assert x.stride(1) == 1 and out.stride(1) == 1 and out.shape == (M, N)
    ref = _next_weight.get(w_nk.data_ptr())
    nxt = ref() if ref is not None else None
    st = kernels().cbis_gemm_few_rows_tc5(_ptr(x), c_int(x.stride(0)), _ptr(w_nk), _ptr(bias), _ptr(out),
                                          c_int(out.stride(0)), c_int(M), c_int(N), c_int(K), c_int(ACT[act]),
                                          c_int(dtype_code(out.dtype)), c_int(ksplit), _ptr(nxt),
                                          ctypes.c_ulonglong(min(nxt.numel() * 2, PREFETCH_CAP) if nxt is not None else 0),
                                          _ptr(tcgen05_error_flag(x.device)), _stream())
    _check(st, "gemm_few_rows", f"M={M} N={N} K={K} ksplit={ksplit}")


_tc_error = {}
USE_TCGEN05 = __import__("os").environ.get("CBIS_TCGEN05", "1") != "0"
USE_TILED_EXTENDED = __import__("os").environ.get("CBIS_TILED_EXTENDED", "1") != "0"   # 0: attention with a bias, a sink or values of their own width goes to the general kernel for prompts too
USE_KEY_CHUNKS = __import__("os").environ.get("CBIS_KEY_CHUNKS", "1") != "0"   # 0: attention kernels never cut the keys over more blocks
USE_TILED_F32 = __import__("os").environ.get("CBIS_TILED_F32", "1") != "0"   # 0: the general kernel for 32-bit prompts
USE_FEW_ROWS = USE_TCGEN05 and __import__("os").environ.get("CBIS_FEW_ROWS", "1") != "0"


def raise_if_kernel_errors(device="cuda") -> None:
    """Reads the error flag of the tcgen05 product (a 4-byte copy: call it where the host waits anyway)."""
    key = torch.device(device).index or 0
    flag = _tc_error.get(key)
    if flag is not None:
        code = int(flag.item())
        if code:
            flag.zero_()
            _tc_pending.pop(key, None)      # a copy of the flag asked for earlier would report the same event again
            raise KernelError(f"a bounded wait inside a TMA kernel ran out (code {code}: 1-6 and 21-24 the tcgen05 "
                              f"product, 11-19 the prefill attention, 31-34 the persistent decode kernel); the step's "
                              f"results are invalid")



_tc_pending = {}     # device index -> (pinned copy of the flag, event recorded after the copy)


def poll_kernel_errors(device="cuda") -> None:
    """The same check without making the host wait: looks at the copy of the flag that the call before this one
    asked for (if that copy has been made by now) and asks for a new one behind the work queued so far.  A step
    whose wait ran out is therefore reported one or two calls late, but steps keep overlapping with the host."""
    key = torch.device(device).index or 0
    flag = _tc_error.get(key)
    if flag is None:
        return
    pending = _tc_pending.get(key)
    if pending is not None:
        host, event = pending
        if not event.query():
            return                      # the copy asked for earlier has not run yet: ask again next time
        code = int(host[0])
        if code:
            _tc_pending.pop(key, None)
            flag.zero_()
            raise KernelError(f"a bounded wait inside a TMA kernel ran out (code {code}: 1-6 and 21-24 the tcgen05 "
                              f"product, 11-19 the prefill attention, 31-34 the persistent decode kernel); the results "
                              f"of a recent step are invalid")
    else:
        host, event = torch.zeros(1, dtype=torch.int32).pin_memory(), torch.cuda.Event()
    host.copy_(flag, non_blocking=True)
    event.record()
    _tc_pending[key] = (host, event)


def tcgen05_error_flag(device) -> torch.Tensor:
    """int32[1] on the device that the tcgen05 product sets when one of its bounded waits runs out."""
    key = torch.device(device).index or 0
    if key not in _tc_error:
        _tc_error[key] = torch.zeros(1, dtype=torch.int32, device=device)
    return _tc_error[key]


def gemm_tcgen05(x, w_nk, bias, act, out, spin_limit: int = 0, starve: bool = False, accumulate: bool = False):
    """out = act(x @ w_nk^T + bias) on the tcgen05 tensor cores (TMA operands, accumulator in tensor
    memory, bias and activation on the 32-bit sums).  bfloat16, K a multiple of 8.
    ``spin_limit`` (0: the service limit) bounds every wait inside the kernel; ``starve`` (up to 128 rows,
    for the test of the give-up path) makes the kernel request no operands, so that its waits run out:
    it then sets the error flag (``tcgen05_error_flag``), frees its tensor memory and returns.
    ``accumulate`` (32-bit ``out``, more than 128 rows): the result is added into ``out`` (a TMA reduction)."""
    _need_cuda(x, w_nk, bias, out)
    M, K = x.shape
    N = w_nk.shape[0]
    assert x.dtype == torch.bfloat16 and w_nk.dtype == torch.bfloat16 and w_nk.is_contiguous() and w_nk.shape[1] == K
    assert x.stride(1) == 1 and out.stride(1) == 1 and out.shape == (M, N)
    st = kernels().cbis_gemm_tcgen05_bf16_ex(_ptr(x), c_int(x.stride(0)), _ptr(w_nk), _ptr(bias), _ptr(out),
                                             c_int(out.stride(0)), c_int(M), c_int(N), c_int(K), c_int(ACT[act]),
                                             c_int(dtype_code(out.dtype)), _ptr(tcgen05_error_flag(x.device)), _stream(),
                                             ctypes.c_uint(spin_limit), c_int(1 if starve else 0), c_int(1 if accumulate else 0))
    _check(st, "gemm_tcgen05", f"M={M} N={N} K={K}" + (" accumulate" if accumulate else ""))


# 1: products whose result is added to the residual stream (attention output, feed-forward output) add it there
# themselves where the TMA + tcgen05 product has tiles enough (prompts): bias and sum in its epilogue, a TMA reduction
# into the 32-bit rows; 0: the library product writes 32-bit sums and the next norm adds them.
USE_LINEAR_ADD = __import__("os").environ.get("CBIS_LINEAR_ADD", "1") != "0"
USE_TCGEN05_PAIR = __import__("os").environ.get("CBIS_TCGEN05_PAIR", "1") != "0"    # the kernel library reads the same variable


def linear_add_takes(x, w_nk, residual) -> bool:
    """Whether ``linear_add`` takes this product: bfloat16 rows enough for the tcgen05 product's tiles, aligned."""
    if not (USE_LINEAR_ADD and USE_TCGEN05 and USE_TCGEN05_PAIR) or residual is None or x.dtype != torch.bfloat16:
        return False
    M, K = x.shape
    N = w_nk.shape[0]
    return (M > 128 and tc_tiles(M, N) and K % 8 == 0 and x.stride(0) % 8 == 0 and x.data_ptr() % 16 == 0
            and residual.dtype == torch.float32 and residual.stride(0) % 4 == 0 and residual.data_ptr() % 16 == 0 and N >= 16)


def linear_add(x, w_nk, bias, residual) -> None:
    """residual += x @ w_nk^T + bias (32-bit residual rows, bfloat16 operands, 32-bit sums)."""
    gemm_tcgen05(x, w_nk, bias, None, residual, accumulate=True)


def linear(x, w_nk, bias, act=None, out_dtype=None):
    """act(x @ W^T + bias) with W stored [N, K] (K contiguous).

    32-bit inputs: this package's FFMA kernel (no reduced-precision matrix mode).  bfloat16
    inputs: up to 16 rows go to the weight-streaming mma.sync kernel; a head over a vocabulary at
    17..64 rows goes to the TMA + tcgen05 kernel with swapped operands; more rows with a bias or an
    activation go to the TMA + tcgen05 kernel; all apply bias and activation to the 32-bit sums and
    round once.  More rows without an epilogue go to the library GEMM."""
    M, K = x.shape
    N = w_nk.shape[0]
    if x.dtype == torch.float32:
        out = torch.empty((M, N), dtype=torch.float32, device=x.device)
        linear_f32(x, w_nk, bias, act, out, w_is_nk=True)
        return out
    _need_cuda(x, w_nk)
    out_dtype = out_dtype or x.dtype
    aligned = K % 8 == 0 and x.stride(0) % 8 == 0 and x.data_ptr() % 16 == 0
    # up to 16 rows; up to 64 where the weight is small (a million elements: any kernel takes a few microseconds, and the
    # library's call costs the host 15-60 us, this one 6, with the epilogue inside)
    if aligned and (M <= SMALL_M or (M <= 64 and N * K <= SMALL_WEIGHT)):
        out = torch.empty((M, N), dtype=out_dtype, device=x.device)
        gemm_small_m(x, w_nk, bias, act, out)
        return out
    plain = bias is None and not ACT[act]
    if USE_FEW_ROWS and M <= 64 and aligned and plain and (N % 8 != 0 or N >= 32768):
        # a head over a vocabulary at 17..64 rows: the library product is slow when N is no multiple of 8 (212 us at
        # 64 rows of 50,257 x 2,048), the TMA + tcgen05 kernel with swapped operands streams it at 4.9 TB/s (42 us).
        # (Up to 16 rows, and inside a layer, the mma.sync kernel stays: the tcgen05 one is as fast alone and keeps
        # more bytes in flight on large matrices, 5.8 TB/s on 134 MB against 4.4, but its blocks need 90 KB of
        # shared memory each and cannot start beside the blocks of the kernel before them: in the chain of a
        # decode step that costs more than it wins, 1.75 ms per step against 1.29.)
        out = torch.empty((M, N), dtype=out_dtype, device=x.device)
        gemm_few_rows(x, w_nk, bias, act, out)
        return out
    if out_dtype != torch.float32 and plain:
        return torch.mm(x, w_nk.t())
    if USE_LIBRARY_EPILOGUE and out_dtype == torch.bfloat16 and bias is not None and ACT[act] in (0, 2) and not (USE_TCGEN05 and tc_tiles(M, N)):
        # 17 rows up to where the tcgen05 product has tiles enough: the library product with the library's own epilogue
        # (bias, or bias and tanh GELU, applied to its 32-bit sums, rounded once) instead of 32-bit sums and a kernel
        # for the epilogue: 9.1 -> 6.6 us (bias) and 9.2 -> 8.0 us (bias, GELU) on 64 x 6400 x 1600.  It wants the
        # bias in bfloat16: taken only where that copy is exact.  The GELU form only with every operand aligned: on
        # other sizes the library adds the bias, rounds, and then applies the activation to the rounded values.
        b16 = _bias_bf16(bias)
        if b16 is not None:
            if ACT[act] == 0:
                return torch.addmm(b16, x, w_nk.t())
            if aligned and N % 8 == 0 and x.is_contiguous():
                return torch._addmm_activation(b16, x, w_nk.t(), use_gelu=True)
    if (USE_TCGEN05 and tc_tiles(M, N) and out_dtype == torch.bfloat16 and K % 8 == 0 and x.stride(0) % 8 == 0
            and x.data_ptr() % 16 == 0):
        # a product with an epilogue: TMA + tcgen05 with bias and activation applied to the sums in tensor memory
        out = torch.empty((M, N), dtype=out_dtype, device=x.device)
        gemm_tcgen05(x, w_nk, bias, act, out)
        return out
    acc = torch.mm(x, w_nk.t(), out_dtype=torch.float32)
    if out_dtype == torch.float32:
        if not plain:
            bias_act(acc, bias, act)
        return acc
    out = torch.empty((M, N), dtype=out_dtype, device=x.device)
    bias_act_out(acc, bias, act, out)     # one rounding, as in the few-rows kernel
    return out


def tc_tiles(M: int, N: int) -> bool:
    """Whether the 128x256 tiles of the TMA + tcgen05 product cover most of the 148 SMs."""
    return -(-M // 128) * -(-N // 256) >= 96


USE_LIBRARY_EPILOGUE = __import__("os").environ.get("CBIS_LIBRARY_EPILOGUE", "1") != "0"
_bias16 = {}     # data_ptr of a 32-bit bias -> (weak reference to it, its bfloat16 copy or None if the copy is not exact)


def _bias_bf16(bias):
    key = bias.data_ptr()
    hit = _bias16.get(key)
    if hit is not None and hit[0]() is bias:
        return hit[1]
    b16 = bias.to(torch.bfloat16)
    if not torch.equal(b16.float(), bias.float()):
        b16 = None
    if len(_bias16) > 4096:
        for k in [k for k, (r, _) in _bias16.items() if r() is None]:
            del _bias16[k]
    _bias16[key] = (weakref.ref(bias), b16)
    return b16


def kv_write(qkv, k_off, v_off, k_cache, v_cache, slot_mapping, n_kv_head, head_dim, page_size, v_head_dim=0):
    """Rows of this step's K and V (columns k_off.. and v_off.. of qkv) go to their token slots.  ``v_head_dim``: the
    values' width where it is not the keys'; one array given for both takes the rows at k_off only."""
    _need_cuda(qkv, k_cache, v_cache, slot_mapping)
    T = qkv.shape[0]
    assert qkv.stride(1) == 1 and k_cache.dtype == qkv.dtype and v_cache.dtype == qkv.dtype
    assert slot_mapping.dtype == torch.int32 and slot_mapping.shape[0] >= T
    st = kernels().cbis_kv_write(_ptr(qkv), c_int(qkv.stride(0)), c_int(k_off), c_int(v_off), _ptr(k_cache),
                                 _ptr(v_cache), _ptr(slot_mapping), c_int(T), c_int(n_kv_head), c_int(head_dim),
                                 c_int(page_size), c_int(dtype_code(qkv.dtype)), _stream(), c_int(v_head_dim))
    _check(st, "kv_write", f"T={T} kv_heads={n_kv_head} head_dim={head_dim} page={page_size}")


def _need_columns(q, out, n_head, v_heads, head_dim, v_head_dim):
    """The launch's heads have their queries in q and their results in out."""
    if q.shape[1] < n_head // v_heads * head_dim or out.shape[1] < n_head * v_head_dim:
        raise KernelError(f"attention: {n_head} heads ({v_heads} value heads a query head) of {head_dim} and {v_head_dim} do not fit "
                          f"rows of {q.shape[1]} and {out.shape[1]} columns")


def generic_key_chunks(rows: int, n_head: int, max_context: int, head_dim: int):
    """(n_chunks, chunk_keys) for the general attention kernel (a warp per row and head): no cut (1, 0) when rows and
    heads alone give 16 warps to each of the 148 SMs, or the head size is no multiple of 4; else chunks of a power
    of two of keys, at least 256, that do."""
    want = -(-16 * 148 // max(1, rows * n_head))
    if want <= 1 or max_context <= 256 or head_dim % 4 or head_dim > 256 or not USE_KEY_CHUNKS:
        return 1, 0
    chunk = 256
    while chunk * want < max_context:
        chunk *= 2
    n = -(-max_context // chunk)
    return (n, chunk) if n > 1 else (1, 0)


def paged_attention_generic(q, k_cache, v_cache, block_table, row_seq, positions, out, n_head, n_kv_head,
                            head_dim, page_size, scale, window=0, chunks=(1, 0), partial=None, v_head_dim=0,
                            slopes=None, sinks=None, q_temp=None, rates=None, v_heads=1, cap: float = 0.0, keep: int = 0):
    """Attention of every row over its request's pages: keys max(0,p-window+1)..p for the query at p.
    ``window`` is one signed number in every attention kernel: 0 every key up to p; w > 0 a sliding window of w keys;
    w < 0 the keys of p's own block of -w positions, p - p mod (-w) .. p, blocks counted from position 0.
    ``chunks`` = (n, keys) from ``generic_key_chunks`` cuts every row's keys n ways over as many warps (every
    context below n * keys); ``partial`` then holds ``rows * n_head * n * (head_dim + 4)`` floats.
    ``v_head_dim``: the values' width where it differs from the keys' (``out`` is then ``n_head * v_head_dim`` wide);
    the value pages may be the key pages themselves, whose rows' first entries are then the values.  ``slopes`` (32-bit,
    per head): slope * (p - j) is taken off the score of the key at j.  ``sinks`` (32-bit, per head): exp(sink) joins
    the softmax's denominator.  ``q_temp`` = (coef, every): the scores of the query at p are multiplied by
    1 + coef * ln(floor((p + 1) / every) + 1).  ``rates`` (32-bit, per head, with ``slopes``): the bias is
    slope * ln(1 + rate * (p - j)) instead.  ``v_heads`` = n_kv_head: the launch's head h is query head h / v_heads over
    the values of key/value head h % v_heads (``n_head``, and every array per head, counts these pairs; q holds
    n_head / v_heads heads).  ``cap`` > 0: the scaled score s becomes cap * tanh(s / cap) (before a bias).  ``keep`` > 0, with a
    window or blocks: the first ``keep`` keys of a sequence stay visible to every later query."""
    _need_cuda(q, k_cache, v_cache, block_table, row_seq, positions, out, partial)
    T = q.shape[0]
    if head_dim > ATTENTION_MAX_HEAD_DIM:
        raise KernelError(f"attention: head_dim={head_dim} is above the kernel's limit of {ATTENTION_MAX_HEAD_DIM}")
    if n_head % (n_kv_head * v_heads):
        raise KernelError(f"attention: n_head={n_head} is not a multiple of n_kv_head={n_kv_head}")
    assert q.stride(1) == 1 and out.stride(1) == 1 and block_table.dtype == torch.int32
    _need_columns(q, out, n_head, v_heads, head_dim, int(v_head_dim) or head_dim)
    assert block_table.is_contiguous() and row_seq.dtype == torch.int32 and positions.dtype == torch.int32
    n_chunks, chunk_keys = chunks
    vd = int(v_head_dim) or head_dim
    v_row = v_cache.shape[-1]
    if vd > v_row:
        raise KernelError(f"attention: values of {vd} do not fit pages of rows of {v_row}")
    for t in (slopes, sinks, rates):
        assert t is None or (t.dtype == torch.float32 and t.numel() == n_head and t.is_cuda)
    if n_chunks > 1:
        assert partial.dtype == torch.float32 and partial.numel() >= T * n_head * n_chunks * (vd + 4)
        if out.stride(0) % 4 or out.data_ptr() % 16 or vd % 4:
            n_chunks, chunk_keys = 1, 0
    coef, every = q_temp if q_temp else (0.0, 0)
    st = kernels().cbis_paged_attention_generic(
        _ptr(q), c_int(q.stride(0)), _ptr(k_cache), _ptr(v_cache), _ptr(block_table), c_int(block_table.shape[1]),
        _ptr(row_seq), _ptr(positions), _ptr(out), c_int(out.stride(0)), c_int(T), c_int(n_head), c_int(n_kv_head),
        c_int(head_dim), c_int(page_size), c_float(scale), c_int(window), c_int(dtype_code(q.dtype)),
        c_int(n_chunks), c_int(chunk_keys), _ptr(partial), _stream(), c_int(vd), c_int(v_row), _ptr(slopes), _ptr(sinks),
        c_float(coef), c_int(int(every)), _ptr(rates), c_int(v_heads), c_float(cap), c_int(keep))
    _check(st, "paged_attention_generic", f"T={T} heads={n_head}/{n_kv_head} head_dim={head_dim} page={page_size} "
                                          f"chunks={n_chunks}x{chunk_keys}")


def decode_splits(rows: int, n_head: int, max_context: int) -> int:
    """How many ways the decode kernel splits a request's keys.  A block takes (row, head, split) and
    4 blocks fit on each of the 148 SMs: split as far as one round of blocks allows, in pieces of at
    least 32 keys, at most 32 ways; with a round or more of (row, head) pairs there is no split."""
    slots = 4 * 148
    pairs = max(1, rows * n_head)
    return max(1, min(slots // pairs, 32, max(1, max_context // 32)))


def decode_scratch_floats(rows: int, n_head: int, head_dim: int, nsplit: int) -> int:
    """Floats of scratch for the decode kernel's partial results."""
    return rows * n_head * nsplit * (head_dim + 2) if nsplit > 1 else 0


def paged_decode_bf16(qkv, k_off, v_off, k_cache, v_cache, block_table, row_seq, positions, slot_mapping, out,
                      scratch, counters, n_head, n_kv_head, head_dim, page_size, scale, window, nsplit, v_head_dim=0,
                      slopes=None, sinks=None, q_temp=None, rates=None, v_heads=1, cap: float = 0.0, keep: int = 0):
    """Decode attention (one query per row) with the keys split ``nsplit`` ways; with ``k_off >= 0`` the
    current token's key/value are taken from ``qkv`` and stored into the cache by the same kernel.
    ``scratch``: ``decode_scratch_floats`` floats; ``counters``: rows*n_head int32, zero before the
    first launch (every launch leaves them zero).  ``v_head_dim``, ``slopes``, ``sinks``, ``q_temp``, ``rates``, ``v_heads``,
    ``cap``, ``keep``: as in ``paged_attention_generic`` (widths multiples of 8 up to 256; the scratch is then sized by the values' width)."""
    _need_cuda(qkv, k_cache, v_cache, block_table, row_seq, positions, slot_mapping, out, scratch, counters, slopes, sinks)
    rows = qkv.shape[0]
    vd = int(v_head_dim) or head_dim
    if head_dim % 8 or head_dim > 256 or vd % 8 or vd > 256:
        raise KernelError(f"decode attention: widths {head_dim} and {vd} must be multiples of 8, at most 256")
    assert qkv.dtype == torch.bfloat16 and k_cache.dtype == torch.bfloat16 and out.dtype == torch.bfloat16
    for t in (slopes, sinks, rates):
        assert t is None or (t.dtype == torch.float32 and t.numel() == n_head)
    coef, every = q_temp if q_temp else (0.0, 0)
    _need_columns(qkv, out, n_head, v_heads, head_dim, vd)
    if nsplit > 1:
        assert scratch.dtype == torch.float32 and scratch.numel() >= decode_scratch_floats(rows, n_head, vd, nsplit)
        assert counters.dtype == torch.int32 and counters.numel() >= rows * n_head
    st = kernels().cbis_paged_decode_bf16(
        _ptr(qkv), c_int(qkv.stride(0)), c_int(k_off), c_int(v_off), _ptr(k_cache), _ptr(v_cache), _ptr(block_table),
        c_int(block_table.shape[1]), _ptr(row_seq), _ptr(positions), _ptr(slot_mapping), _ptr(out),
        c_int(out.stride(0)), _ptr(scratch), _ptr(counters), c_int(rows), c_int(n_head), c_int(n_kv_head),
        c_int(head_dim), c_int(page_size), c_float(scale), c_int(window), c_int(nsplit), _stream(),
        c_int(int(v_head_dim)), c_int(v_cache.shape[-1]), _ptr(slopes), _ptr(sinks), c_float(coef), c_int(int(every)),
        _ptr(rates), c_int(v_heads), c_float(cap), c_int(keep))
    _check(st, "paged_decode_bf16", f"rows={rows} heads={n_head}/{n_kv_head} head_dim={head_dim} splits={nsplit}")


USE_DECODE_MIX = __import__("os").environ.get("CBIS_DECODE_MIX", "1") != "0"   # 0: decoding rows whose weights are mixed across heads run every head over every value head and mix the results
DECODE_MIX_MAX_SCRATCH = 1 << 29      # the most bytes of scores a decode step may take


def decode_mix_blocks(n_head: int, n_kv_head: int) -> int:
    """Blocks per row and split of the second kernel of ``decode_mix_bf16`` (the counters a row needs)."""
    return int(kernels().cbis_decode_mix_blocks(c_int(n_head), c_int(n_kv_head)))


def decode_mix_splits(rows: int, n_head: int, n_kv_head: int, max_context: int) -> int:
    """How many ways ``decode_mix_bf16`` splits a request's keys: one round of blocks, four of them on an SM, two where
    more than four query heads share a key/value head (a block then holds eight heads' sums)."""
    return decode_splits(rows, decode_mix_blocks(n_head, n_kv_head) * (1 if n_head // n_kv_head <= 4 else 2), max_context)


def decode_mix_scratch_floats(rows: int, n_head: int, v_head_dim: int, cap: int, nsplit: int) -> int:
    fn = kernels().cbis_decode_mix_scratch_floats
    fn.restype = ctypes.c_longlong
    return int(fn(c_int(rows), c_int(n_head), c_int(v_head_dim), c_int(cap), c_int(nsplit)))


def decode_mix_takes(dtype, rows: int, n_head: int, head_dim: int, v_head_dim: int, cap: int) -> bool:
    """Whether ``decode_mix_bf16`` takes these sizes."""
    return (USE_DECODE_MIX and dtype == torch.bfloat16 and head_dim % 8 == 0 and v_head_dim % 8 == 0
            and max(head_dim, v_head_dim) <= 256 and n_head <= 128 and rows * n_head * cap * 4 <= DECODE_MIX_MAX_SCRATCH)


def decode_mix_bf16(qkv, k_off, v_off, k_cache, v_cache, block_table, row_seq, positions, slot_mapping, talk, sinks, gate, out,
                    scratch, counters, cap, n_head, n_kv_head, head_dim, v_head_dim, page_size, scale, window, nsplit):
    """Decode attention (one query per row) whose softmax weights are mixed across heads, w'_h = sum_g talk[h, g] w_g,
    before head h applies them to its own key/value head's values; ``sinks`` (per head, or None) join the denominators
    unmixed; ``gate`` ``[rows, n_head * v_head_dim]`` (or None): the result times sigmoid(gate).  With ``k_off`` / ``v_off``
    >= 0 the current token's key / value are taken from ``qkv`` and stored.  ``cap``: a multiple of 16, no less than the
    longest request; ``scratch``: ``decode_mix_scratch_floats`` floats; ``counters``: rows * ``decode_mix_blocks`` int32,
    zero before the first launch (every launch leaves them zero)."""
    _need_cuda(qkv, k_cache, v_cache, block_table, row_seq, positions, slot_mapping, talk, sinks, gate, out, scratch, counters)
    rows = qkv.shape[0]
    assert qkv.dtype == torch.bfloat16 == out.dtype == k_cache.dtype and qkv.stride(1) == 1 and out.stride(1) == 1
    _need_columns(qkv, out, n_head, 1, head_dim, v_head_dim)
    assert k_cache.shape[1] == n_kv_head == v_cache.shape[1] and k_cache.shape[3] == head_dim and v_cache.shape[3] == v_head_dim
    assert talk.dtype == torch.float32 and talk.shape == (n_head, n_head) and talk.is_contiguous()
    assert sinks is None or (sinks.dtype == torch.float32 and sinks.numel() == n_head)
    assert gate is None or (gate.dtype == torch.bfloat16 and gate.shape == (rows, n_head * v_head_dim) and gate.stride(1) == 1)
    assert scratch.dtype == torch.float32 and scratch.numel() >= decode_mix_scratch_floats(rows, n_head, v_head_dim, cap, nsplit)
    assert nsplit == 1 or (counters.dtype == torch.int32 and counters.numel() >= rows * decode_mix_blocks(n_head, n_kv_head))
    assert block_table.is_contiguous() and block_table.dtype == torch.int32
    st = kernels().cbis_decode_mix_bf16(
        _ptr(qkv), c_int(qkv.stride(0)), c_int(k_off), c_int(v_off), _ptr(k_cache), _ptr(v_cache), _ptr(block_table),
        c_int(block_table.shape[1]), _ptr(row_seq), _ptr(positions), _ptr(slot_mapping), _ptr(talk), _ptr(sinks), _ptr(gate),
        c_int(gate.stride(0) if gate is not None else 0), _ptr(out), c_int(out.stride(0)), _ptr(scratch), _ptr(counters),
        c_int(cap), c_int(rows), c_int(n_head), c_int(n_kv_head), c_int(head_dim), c_int(v_head_dim), c_int(page_size),
        c_float(scale), c_int(window), c_int(nsplit), _stream())
    _check(st, "decode_mix_bf16", f"rows={rows} heads={n_head}/{n_kv_head} widths={head_dim}/{v_head_dim} splits={nsplit}", launches=2)


def paged_prefill_bf16(q, k_cache, v_cache, block_table, cu_rows, seg_start, out, seg0, n_seg, max_seg_rows,
                       n_head, n_kv_head, head_dim, page_size, scale, window=0, chunks=(1, 0), partial=None,
                       positions=None, row0=0, n_rows=0, v_head_dim=0, slopes=None, sinks=None, q_temp=None, rates=None,
                       v_heads=1, cap: float = 0.0, keep: int = 0):
    """Attention of the segments seg0..seg0+n_seg-1 (runs of rows given by ``cu_rows``, first positions
    ``seg_start``) over their pages, on the tensor cores.  Head sizes 16, 32, ... 128, page sizes 2^k.
    With ``v_head_dim`` keys and values may have different widths, multiples of 8 up to 128 (the value pages may be
    the key pages: a row's first entries are then its values); ``slopes``, ``sinks``, ``q_temp``, ``rates``, ``v_heads``, ``cap``,
    ``keep``: as in ``paged_attention_generic``.
    ``chunks`` = (n, keys) from ``prefill_key_chunks`` cuts the keys n ways over more blocks (every context of the
    step below n * keys); ``partial`` then holds ``n_rows * n_head * n * (head_dim + 4)`` floats, ``positions`` the
    position of every row, ``row0`` and ``n_rows`` name the rows of these segments."""
    _need_cuda(q, k_cache, v_cache, block_table, cu_rows, seg_start, out, partial, positions)
    vd = int(v_head_dim) or head_dim
    if not v_head_dim and (head_dim % 16 or not 16 <= head_dim <= 128):
        raise KernelError(f"prefill attention: head_dim={head_dim} is no multiple of 16 up to 128 (the general kernel takes it)")
    if head_dim % 8 or vd % 8 or not 8 <= max(head_dim, vd) <= 128:
        raise KernelError(f"prefill attention: widths {head_dim} and {vd} are no multiples of 8 up to 128 (the general kernel takes them)")
    if page_size & (page_size - 1):
        raise KernelError(f"prefill attention: page_size={page_size} is not a power of two (the general kernel takes it)")
    assert q.dtype == torch.bfloat16 and k_cache.dtype == torch.bfloat16 and out.dtype == torch.bfloat16
    assert q.stride(1) == 1 and out.stride(1) == 1 and block_table.is_contiguous()
    v_row = v_cache.shape[-1]
    _need_columns(q, out, n_head, v_heads, head_dim, vd)
    for t in (slopes, sinks, rates):
        assert t is None or (t.dtype == torch.float32 and t.numel() == n_head and t.is_cuda)
    coef, every = q_temp if q_temp else (0.0, 0)
    n_chunks, chunk_keys = chunks
    if n_chunks > 1:
        assert partial.dtype == torch.float32 and partial.numel() >= n_rows * n_head * n_chunks * (vd + 4)
        assert positions.dtype == torch.int32 and positions.numel() >= row0 + n_rows
    st = kernels().cbis_paged_prefill_bf16(
        _ptr(q), c_int(q.stride(0)), _ptr(k_cache), _ptr(v_cache), _ptr(block_table), c_int(block_table.shape[1]),
        _ptr(cu_rows), _ptr(seg_start), _ptr(out), c_int(out.stride(0)), c_int(seg0), c_int(n_seg),
        c_int(max_seg_rows), c_int(n_head), c_int(n_kv_head), c_int(head_dim), c_int(page_size), c_float(scale),
        c_int(window), c_int(n_chunks), c_int(chunk_keys), _ptr(partial), _ptr(positions), c_int(row0), c_int(n_rows),
        _stream(), c_int(vd), c_int(v_row), _ptr(slopes), _ptr(sinks), c_float(coef), c_int(int(every)), _ptr(rates),
        c_int(v_heads), c_float(cap), c_int(keep))
    _check(st, "paged_prefill_bf16", f"segments={n_seg} heads={n_head}/{n_kv_head} head_dim={head_dim} page={page_size} "
                                     f"chunks={n_chunks}x{chunk_keys}")


def prefill_key_chunks(row_tiles: int, n_head: int, n_seg: int, max_context: int, blocks_per_tile: int = 1,
                       blocks_per_sm: int = 8, min_chunk: int = 256):
    """(n_chunks, chunk_keys) for the tiled prefill attention kernels: no cut (1, 0) when (row tile, head, segment)
    alone give ``blocks_per_sm`` blocks to each of the 148 SMs; else chunks of a power of two of keys, at least
    ``min_chunk``, that do.  The tcgen05 kernel has two blocks per row tile and two per SM, and a block of it costs
    some 8 us before its first tile: it is cut only into chunks of 8,192 keys or more (measured at 512 rows, 16 heads
    of 128: 2,048 keys 32 us whole, 42 us in two chunks; 32,768 keys 385 us whole, 230 us in two, 291 us in eight)."""
    base = max(1, row_tiles * n_head * n_seg * blocks_per_tile)
    want = -(-blocks_per_sm * 148 // base)
    if want <= 1 or max_context <= min_chunk or not USE_KEY_CHUNKS:
        return 1, 0
    chunk = min_chunk
    while chunk * want < max_context:
        chunk *= 2
    n = -(-max_context // chunk)
    return (n, chunk) if n > 1 else (1, 0)


def paged_prefill_f32(q, k_cache, v_cache, block_table, cu_rows, seg_start, out, seg0, n_seg, max_seg_rows,
                      n_head, n_kv_head, head_dim, page_size, scale, window=0, chunks=(1, 0), partial=None,
                      positions=None, row0=0, n_rows=0):
    """The same attention as ``paged_prefill_bf16`` in true 32-bit (no tensor cores): a block takes 64 rows of one
    head and brings keys and values through shared memory once.  Head sizes 16, 32, ... 128, any page size;
    ``q`` and ``out`` in full row numbering.  ``chunks`` = (n, keys) from ``prefill_key_chunks`` cuts the keys n
    ways (every context of the step below n * keys); ``partial`` then holds ``n_rows * n_head * n * (head_dim + 4)``
    floats, ``positions`` the position of every row, ``row0`` and ``n_rows`` name the rows of these segments."""
    _need_cuda(q, k_cache, v_cache, block_table, cu_rows, seg_start, out, partial, positions)
    if head_dim % 16 or not 16 <= head_dim <= 128:
        raise KernelError(f"32-bit prefill attention: head_dim={head_dim} is no multiple of 16 up to 128 (the general kernel takes it)")
    assert q.dtype == torch.float32 and k_cache.dtype == torch.float32 and out.dtype == torch.float32
    assert q.stride(1) == 1 and out.stride(1) == 1 and block_table.is_contiguous() and k_cache.is_contiguous()
    n_chunks, chunk_keys = chunks
    if n_chunks > 1:
        assert partial.dtype == torch.float32 and partial.numel() >= n_rows * n_head * n_chunks * (head_dim + 4)
        assert positions.dtype == torch.int32 and positions.numel() >= row0 + n_rows
    st = kernels().cbis_paged_prefill_f32(
        _ptr(q), c_int(q.stride(0)), _ptr(k_cache), _ptr(v_cache), _ptr(block_table), c_int(block_table.shape[1]),
        _ptr(cu_rows), _ptr(seg_start), _ptr(out), c_int(out.stride(0)), c_int(seg0), c_int(n_seg),
        c_int(max_seg_rows), c_int(n_head), c_int(n_kv_head), c_int(head_dim), c_int(page_size), c_float(scale),
        c_int(window), c_int(n_chunks), c_int(chunk_keys), _ptr(partial), _ptr(positions), c_int(row0), c_int(n_rows),
        _stream())
    _check(st, "paged_prefill_f32", f"segments={n_seg} heads={n_head}/{n_kv_head} head_dim={head_dim} page={page_size} "
                                    f"chunks={n_chunks}x{chunk_keys}")


def paged_prefill_tc5(q, k_cache, v_cache, block_table, cu_rows, seg_start, out, seg0, n_seg, max_seg_rows,
                      n_head, n_kv_head, head_dim, page_size, scale, window=0, chunks=(1, 0), partial=None,
                      positions=None, row0=0, n_rows=0, sinks=None, slopes=None, rates=None, v_heads=1, cap: float = 0.0,
                      keep: int = 0):
    """The same attention as ``paged_prefill_bf16`` on the tcgen05 tensor cores (TMA operands, S and the output in
    tensor memory).  Head size 64 or 128, page sizes 8..128 (powers of two); ``q`` and ``out`` in full row numbering.
    ``chunks``, ``partial``, ``positions``, ``row0``, ``n_rows`` as for ``paged_prefill_bf16`` (chunks from
    ``prefill_key_chunks`` with two blocks per 128-row tile, two per SM and chunks of at least 8,192 keys);
    ``sinks``, ``slopes`` with ``rates``, ``v_heads``, ``cap`` and ``keep`` (not with ``rates``) as in ``paged_attention_generic``."""
    _need_cuda(q, k_cache, v_cache, block_table, cu_rows, seg_start, out, partial, positions)
    if head_dim not in (64, 128):
        raise KernelError(f"tcgen05 prefill attention: head_dim={head_dim} is neither 64 nor 128")
    if page_size & (page_size - 1) or not 8 <= page_size <= 128:
        raise KernelError(f"tcgen05 prefill attention: page_size={page_size} is not a power of two in 8..128")
    assert q.dtype == torch.bfloat16 and k_cache.dtype == torch.bfloat16 and out.dtype == torch.bfloat16
    assert q.stride(1) == 1 and out.stride(1) == 1 and block_table.is_contiguous() and k_cache.is_contiguous()
    _need_columns(q, out, n_head, v_heads, head_dim, head_dim)
    for t in (sinks, slopes, rates):
        assert t is None or (t.dtype == torch.float32 and t.numel() == n_head and t.is_cuda)
    n_chunks, chunk_keys = chunks
    if n_chunks > 1:
        assert partial.dtype == torch.float32 and partial.numel() >= n_rows * n_head * n_chunks * (head_dim + 4)
        assert positions.dtype == torch.int32 and positions.numel() >= row0 + n_rows
    st = kernels().cbis_paged_prefill_tc5(
        _ptr(q), c_int(q.stride(0)), c_int(q.shape[0]), _ptr(k_cache), _ptr(v_cache), c_int(k_cache.shape[0]),
        _ptr(block_table), c_int(block_table.shape[1]), _ptr(cu_rows), _ptr(seg_start), _ptr(out),
        c_int(out.stride(0)), c_int(seg0), c_int(n_seg), c_int(max_seg_rows), c_int(n_head), c_int(n_kv_head),
        c_int(head_dim), c_int(page_size), c_float(scale), c_int(window), c_int(n_chunks), c_int(chunk_keys),
        _ptr(partial), _ptr(positions), c_int(row0), c_int(n_rows), _ptr(tcgen05_error_flag(q.device)), _stream(), _ptr(sinks),
        _ptr(slopes), _ptr(rates), c_int(v_heads), c_float(cap), c_int(keep))
    _check(st, "paged_prefill_tc5", f"segments={n_seg} heads={n_head}/{n_kv_head} page={page_size} chunks={n_chunks}x{chunk_keys}")


def paged_prefill_tc5_blocks_per_sm() -> int:
    """How many blocks of the tcgen05 prefill attention an SM has room for at a time (it is sized for two): from the
    registers, shared memory and tensor memory a block takes as compiled and what the device's SMs have."""
    n = kernels().cbis_paged_prefill_tc5_blocks_per_sm()
    if n < 0:
        raise KernelError(f"paged_prefill_tc5: a device query failed with CUDA error {-n}")
    return n


# 1: decode steps of up to 16 rows run their layers in ONE persistent kernel (csrc/kernels/decode_layers.cu).  Off by
# default: measured at the 1.3B sizes it takes 1.6 ms per step at batch 1 and 2.1 ms at batch 8, the chain of kernels 0.95
# and 1.24 ms (its twelve dependent phases per layer each wait for L2 or for the other blocks while the memory system is
# kept busy by its own weight stream, and eight warps per SM do not hide that).
USE_FUSED_DECODE = __import__("os").environ.get("CBIS_FUSED_DECODE", "0") == "1"
FUSED_DECODE_MAX_ROWS = 16


def decode_layers_blocks(n_min: int) -> int:
    """Blocks the persistent decode kernel runs with: one per SM, fewer when the narrowest product of a layer has
    fewer than 8 columns per block."""
    n = optional_kernels().cbis_decode_layers_blocks(c_int(n_min))
    if n <= 0:
        raise KernelError("decode_layers: the device could not be queried")
    return n


def decode_layers_map(w_nk, blocks: int) -> torch.Tensor:
    """The 128-byte TMA descriptor of a weight matrix ``[N, K]`` for ``blocks`` blocks, as a CPU uint8 tensor."""
    _need_cuda(w_nk)
    assert w_nk.dtype == torch.bfloat16 and w_nk.is_contiguous() and w_nk.dim() == 2
    out = torch.zeros(128, dtype=torch.uint8)
    st = optional_kernels().cbis_decode_layers_map(c_void_p(out.data_ptr()), _ptr(w_nk), c_int(w_nk.shape[0]), c_int(w_nk.shape[1]),
                                          c_int(blocks))
    _check(st, "decode_layers_map", f"N={w_nk.shape[0]} K={w_nk.shape[1]} blocks={blocks}", launches=0)
    return out


def decode_layers_desc_bytes() -> int:
    return int(optional_kernels().cbis_decode_layers_desc_bytes())


def decode_layers_splits(rows: int, n_head: int, max_context: int, blocks: int) -> int:
    """How many ways the persistent decode kernel splits a request's keys: its (row, head, split) items go to the two
    groups of four warps of every block.  An item has a fixed cost (its query, the meeting of its warps, the merge),
    so the items are as long as one round over the groups allows: pieces of 64 keys or more, at most 32 ways."""
    groups, pairs = 2 * blocks, max(1, rows * n_head)
    return max(1, min(32, groups // pairs, max_context // 64))


def decode_layers(maps, layers, n_layers, blocks, M, d, n_head, n_kv_head, head_dim, F, page_size, act, window, scale,
                  nsplit, x, qkv, attn, hidden, block_table, row_seq, positions, slot_mapping, part, counters,
                  grid_counter, trace=None):
    """``n_layers`` pre-norm layers of a decode step of ``M`` <= 16 rows in one persistent kernel (see
    csrc/kernels/decode_layers.cu).  ``grid_counter`` (int32[1]) must be zero; a wait that runs out inside the kernel
    sets the flag that ``raise_if_kernel_errors`` reads.  ``trace`` (int64[256], for measuring): block 0's
    nanosecond timer at every phase boundary, 12 per layer."""
    _need_cuda(maps, layers, x, qkv, attn, hidden, block_table, row_seq, positions, slot_mapping, part, counters, grid_counter)
    assert x.dtype == torch.float32 and x.is_contiguous() and qkv.dtype == torch.bfloat16 and hidden.dtype == torch.bfloat16
    assert block_table.is_contiguous() and block_table.dtype == torch.int32
    st = optional_kernels().cbis_decode_layers(
        _ptr(maps), _ptr(layers), c_int(n_layers), c_int(blocks), c_int(M), c_int(d), c_int(n_head), c_int(n_kv_head),
        c_int(head_dim), c_int(F), c_int(page_size), c_int(ACT[act]), c_int(window), c_float(scale), c_int(nsplit), _ptr(x),
        _ptr(qkv), _ptr(attn), _ptr(hidden), _ptr(block_table), c_int(block_table.shape[1]), _ptr(row_seq), _ptr(positions),
        _ptr(slot_mapping), _ptr(part), _ptr(counters), _ptr(grid_counter), _ptr(tcgen05_error_flag(x.device)), _stream(),
        _ptr(trace))
    _check(st, "decode_layers", f"layers={n_layers} rows={M} width={d} heads={n_head}/{n_kv_head} head_dim={head_dim} inner={F}")


def linear_heads(x, w_hnk, out, x_head_stride: int = 0, out_head_stride: int = 0):
    """Per head h: out[:, h*N:(h+1)*N] = x[:, h*K:(h+1)*K] @ w_hnk[h]^T; ``w_hnk`` is ``[heads, N, K]``, x and out
    are 2-D with unit column stride (views of wider buffers are fine).  With ``x_head_stride`` / ``out_head_stride``
    a head's columns start every so many columns instead of every K / N (a head's part of wider per-head rows).
    32-bit: this package's FFMA product, head by head; bfloat16: one strided batched product of the library."""
    _need_cuda(x, w_hnk, out)
    H, N, K = w_hnk.shape
    T = x.shape[0]
    xs, os_ = int(x_head_stride) or K, int(out_head_stride) or N
    assert x.shape[1] >= (H - 1) * xs + K and out.shape[1] >= (H - 1) * os_ + N and out.shape[0] == T
    assert x.stride(1) == 1 and out.stride(1) == 1
    assert w_hnk.is_contiguous() and x.dtype == w_hnk.dtype == out.dtype
    if T == 0:
        return
    if x.dtype == torch.float32:
        for h in range(H):
            linear_f32(x[:, h * xs:h * xs + K], w_hnk[h], None, None, out[:, h * os_:h * os_ + N], w_is_nk=True)
        return
    xv = x.as_strided((H, T, K), (xs, x.stride(0), 1), x.storage_offset())
    ov = out.as_strided((H, T, N), (os_, out.stride(0), 1), out.storage_offset())
    torch.bmm(xv, w_hnk.transpose(1, 2), out=ov)


def rms_norm(x, weight, eps, out, parts: int = 1, gate=None, gate_act="silu", gate_after: bool = False):
    """out = v / sqrt(mean(v^2) + eps) * weight in ``parts`` equal parts of the row, each by its own mean, with
    v = x * act(gate) if a gate is given (the gate comes BEFORE the norm).  x: 32-bit or ``out``'s type; gate and out:
    the compute type; views with unit column stride are fine.  Arithmetic in 32-bit.  With ``gate_after`` the gate
    stays out of the norm: out = x / sqrt(mean(x^2) + eps) * weight * act(gate)."""
    _need_cuda(x, weight, out, gate)
    rows, n = x.shape
    assert n % parts == 0 and out.shape == x.shape and x.stride(1) == 1 and out.stride(1) == 1
    assert weight is None or (weight.dtype == torch.float32 and weight.numel() == n and weight.is_contiguous())
    assert gate is None or (gate.shape == x.shape and gate.stride(1) == 1 and gate.dtype == out.dtype)
    st = kernels().cbis_rms_norm(_ptr(x), c_int(x.stride(0)), c_int(dtype_code(x.dtype)), _ptr(gate),
                                 c_int(gate.stride(0) if gate is not None else 0), c_int(ACT[gate_act]), _ptr(weight),
                                 c_float(eps), _ptr(out), c_int(out.stride(0)), c_int(dtype_code(out.dtype)), c_int(rows),
                                 c_int(parts), c_int(n // parts), _stream(), c_int(1 if gate_after else 0))
    _check(st, "rms_norm", f"rows={rows} width={n} parts={parts}")


def gate_mul(a, b, act, out, b_rows=None, limit: float = 0.0, beta: float = 1.0, shift: float = 0.0, row_gate=None):
    """out = act(a) * b element by element (32-bit arithmetic, one rounding); a, b, out: ``[rows, n]`` of one type,
    views with unit column stride are fine.  With ``b_rows`` (int32, one per row) b is a table ``[*, n]`` and row r
    takes b[b_rows[r]] (a token's row of a table; an index outside the table reads as zeros).  ``limit`` > 0: a is cut off
    at limit from above and b at -limit and limit first; ``beta``: silu is a * sigmoid(beta a); ``shift`` is added to b;
    ``row_gate`` (32-bit, one per row) multiplies the row."""
    _need_cuda(a, b, out, b_rows)
    rows, n = a.shape
    assert out.shape == a.shape and a.dtype == b.dtype == out.dtype and b.shape[1] == n
    assert b.shape == a.shape if b_rows is None else (b_rows.dtype == torch.int32 and b_rows.shape[0] >= rows)
    assert a.stride(1) == 1 and b.stride(1) == 1 and out.stride(1) == 1
    assert row_gate is None or (row_gate.dtype == torch.float32 and row_gate.is_contiguous() and row_gate.numel() >= rows)
    st = kernels().cbis_gate_mul(_ptr(a), c_int(a.stride(0)), _ptr(b), c_int(b.stride(0)), _ptr(out), c_int(out.stride(0)),
                                 c_int(ACT[act]), c_int(rows), c_int(n), c_int(dtype_code(a.dtype)), _stream(),
                                 _ptr(b_rows), c_int(b.shape[0]), c_float(limit), c_float(beta), c_float(shift),
                                 _ptr(row_gate))
    _check(st, "gate_mul", f"rows={rows} n={n}")


RMS_RESIDUAL_MAX_WIDTH = (200 * 1024 // 4 - 64) // 2     # the widest row add_rmsnorm takes (cbis_rms_residual_max_width() says the same)
MATRIX_MEMORY_MAX_DIM = 512                              # the widest key of the matrix memory (cbis_matrix_memory_max_dim())


def add_rmsnorm(x, delta, delta_bias, post, weight, eps, offset, out, rows=None, delta_scale: float = 1.0,
                x_scale: float = 1.0, stream=None):
    """One pass over the rows of the 32-bit residual stream ``x``: what a part left (``delta``, 32-bit or the compute
    type, plus ``delta_bias`` per column) is, with ``post`` = (weight, eps, offset), first divided by its own root mean
    square and multiplied by (offset + weight); it is added to x in place; and ``out`` takes x / sqrt(mean(x^2) + eps)
    * (offset + weight) (``weight`` None: x itself; ``out`` None: nothing).  With ``rows`` (int32) only those rows
    are produced and x is not changed.  ``delta_scale`` multiplies what is added (after its own norm, if it has one).
    ``x_scale`` multiplies x before the addition, and with ``stream`` = (weight, eps, offset) the SUM is divided by its root
    mean square and multiplied by (offset + weight) before it becomes x (layers whose norm stands after the addition)."""
    _need_cuda(x, delta, delta_bias, weight, out, rows)
    d = x.shape[1]
    assert x.dtype == torch.float32 and x.is_contiguous()
    n = rows.shape[0] if rows is not None else x.shape[0]
    assert out is None or (out.is_contiguous() and out.shape == (n, d))
    assert delta is None or (delta.shape == x.shape and delta.stride(1) == 1)
    pw, peps, poff = post if post is not None else (None, 0.0, 0.0)
    sw, seps, soff = stream if stream is not None else (None, 0.0, 0.0)
    for t in (delta_bias, pw, weight, sw):
        assert t is None or (t.dtype == torch.float32 and t.numel() == d and t.is_contiguous())
    st = kernels().cbis_add_rmsnorm(_ptr(x), _ptr(delta), c_int(delta.stride(0) if delta is not None else 0),
                                    c_int(dtype_code(delta.dtype) if delta is not None else 0), _ptr(delta_bias), _ptr(pw),
                                    c_float(peps), c_float(poff), _ptr(weight), c_float(eps), c_float(offset), _ptr(out),
                                    c_int(dtype_code(out.dtype) if out is not None else 0), _ptr(rows), c_int(n), c_int(d),
                                    _stream(), c_float(delta_scale), c_float(x_scale), _ptr(sw), c_float(seps), c_float(soff))
    _check(st, "add_rmsnorm", f"rows={n} width={d}")


def rope_rows(src, src_col0, src_head_stride, dst, dst_col0, dst_head_stride, positions, heads, width, dims, freqs,
              neighbours: bool = False, length: float = 1.0, keep_col0: int = -1, keep_head0: int = 0):
    """In every row and head, ``width`` entries from column ``col0 + head * head_stride`` of ``src`` go to the like
    place of ``dst``; the first ``dims`` of them rotated in pairs (entry i with entry i + dims/2; with ``neighbours``
    entry 2i with entry 2i + 1) by the angle position * freqs[i] (32-bit), cosine and sine times ``length``, the rest
    as they are.  src and dst may be one buffer.  With ``keep_col0`` >= 0 the heads from ``keep_head0`` on are also
    written UNROTATED to ``dst`` at column keep_col0 + (head - keep_head0) * width (columns nothing else touches)."""
    _need_cuda(src, dst, positions, freqs)
    rows = src.shape[0]
    assert src.dtype == dst.dtype and src.stride(1) == 1 and dst.stride(1) == 1 and dst.shape[0] == rows
    assert positions.dtype == torch.int32 and positions.shape[0] >= rows
    assert dims == 0 or (freqs.dtype == torch.float32 and freqs.numel() >= dims // 2 and freqs.is_contiguous())
    assert src_col0 + (heads - 1) * src_head_stride + width <= src.shape[1]
    assert dst_col0 + (heads - 1) * dst_head_stride + width <= dst.shape[1]
    assert keep_col0 < 0 or (0 <= keep_head0 <= heads and keep_col0 + (heads - keep_head0) * width <= dst.shape[1])
    st = kernels().cbis_rope_rows(_ptr(src), c_int(src.stride(0)), c_int(src_col0), c_int(src_head_stride), _ptr(dst),
                                  c_int(dst.stride(0)), c_int(dst_col0), c_int(dst_head_stride), _ptr(positions),
                                  c_int(rows), c_int(heads), c_int(width), c_int(dims), _ptr(freqs),
                                  c_int(dtype_code(src.dtype)), _stream(), c_int(1 if neighbours else 0), c_float(length),
                                  c_int(keep_col0), c_int(keep_head0))
    _check(st, "rope_rows", f"rows={rows} heads={heads} width={width} dims={dims}")


def head_gate_mul(x, gate, heads, out):
    """out[r, h, :] = x[r, h, :] * sigmoid(gate[r, h]): one gate number per row and head (32-bit or x's type);
    x and out ``[rows, heads * width]``, views with unit column stride are fine."""
    _need_cuda(x, gate, out)
    rows, n = x.shape
    assert n % heads == 0 and out.shape == x.shape and x.dtype == out.dtype and gate.shape == (rows, heads)
    assert x.stride(1) == 1 and out.stride(1) == 1 and gate.stride(1) == 1
    st = kernels().cbis_head_gate_mul(_ptr(x), c_int(x.stride(0)), _ptr(gate), c_int(gate.stride(0)),
                                      c_int(dtype_code(gate.dtype)), _ptr(out), c_int(out.stride(0)), c_int(rows),
                                      c_int(heads), c_int(n // heads), c_int(dtype_code(x.dtype)), _stream())
    _check(st, "head_gate_mul", f"rows={rows} heads={heads} width={n // heads}")


def matrix_memory_state_floats(heads: int, dim: int, v_dim: int) -> int:
    """Floats of one request's state of the matrix memory (the kernel's own layout)."""
    fn = kernels().cbis_matrix_memory_state_floats
    fn.restype = ctypes.c_longlong
    n = int(fn(c_int(heads), c_int(dim), c_int(v_dim)))
    if n < 0:
        raise KernelError(f"matrix_memory: heads={heads} dim={dim} v_dim={v_dim} are sizes the kernel does not take")
    return n


def matrix_memory(qkv, q_off, k_off, v_off, gates, i_bias, f_bias, cap, q_scale, den_eps, state, seg_slot, cu_rows,
                  n_segments, heads, dim, v_dim, y, max_seg_rows: int = 0):
    """The recurrence of a matrix memory with exponential gates over every segment's rows, from and into the requests'
    states: per head m' = max(lf + m, li), S <- exp(lf + m - m') S + exp(li - m') k v^T, n likewise with k alone,
    y = S^T q / (max(|n . q|, exp(-m')) + den_eps), with li = cap tanh((i + i_bias) / cap) and
    lf = logsigmoid(cap tanh((f + f_bias) / cap)).  ``qkv``: the compute type, q | k | v at their column offsets
    (q is multiplied by ``q_scale``); ``gates``: 32-bit ``[T, 2 * heads]``, raw input gates then raw forget gates;
    ``y``: 32-bit ``[T, heads * v_dim]``; ``state``: 32-bit ``[slots, matrix_memory_state_floats]``;
    ``max_seg_rows``: the step's longest segment if known (a step of short segments takes smaller batches of rows)."""
    _need_cuda(qkv, gates, i_bias, f_bias, state, seg_slot, cu_rows, y)
    T = qkv.shape[0]
    assert qkv.stride(1) == 1 and gates.dtype == torch.float32 and gates.stride(1) == 1 and gates.shape == (T, 2 * heads)
    assert y.dtype == torch.float32 and y.stride(1) == 1 and y.shape == (T, heads * v_dim)
    assert state.dtype == torch.float32 and state.stride(1) == 1 and state.shape[1] >= matrix_memory_state_floats(heads, dim, v_dim)
    assert i_bias.dtype == f_bias.dtype == torch.float32 and i_bias.numel() == f_bias.numel() == heads
    st = kernels().cbis_matrix_memory(_ptr(qkv), c_int(qkv.stride(0)), c_int(q_off), c_int(k_off), c_int(v_off), _ptr(gates),
                                      c_int(gates.stride(0)), _ptr(i_bias), _ptr(f_bias), c_float(cap), c_float(q_scale),
                                      c_float(den_eps), _ptr(state), ctypes.c_longlong(state.stride(0)), _ptr(seg_slot),
                                      _ptr(cu_rows), _ptr(y), c_int(y.stride(0)), c_int(n_segments), c_int(heads), c_int(dim),
                                      c_int(v_dim), c_int(dtype_code(qkv.dtype)), _stream(), c_int(int(max_seg_rows)))
    _check(st, "matrix_memory", f"segments={n_segments} heads={heads} dim={dim} v_dim={v_dim}")


RETENTION_MAX_DIM = 512                                  # the widest key of the retention kernel (cbis_retention_max_dim())
QK_PREPARE_MAX_WIDTH = 200 * 1024 // 4 - 64              # q and k of a row together, in entries (cbis_qk_prepare_max_width())
USE_QK_PREPARE = __import__("os").environ.get("CBIS_QK_PREPARE", "1") != "0"   # 0: norm, rotation and blending before attention run as kernels of their own


# A long segment of a retention layer is cut into pieces that run side by side where the step's blocks are few (one
# prompt offers heads x columns / 64 of them, and its rows wait on one another): see ``retention``.
RETENTION_PIECE_UNIT = 32             # a piece's rows are a multiple of this (and of the kernel's batches of 16 rows)
RETENTION_PIECE_SIZES = 16            # piece sizes 32, 64, ... for which a mixer keeps decay^rows
RETENTION_PIECES_FROM = 128           # the longest segment of a step from which segments are cut
RETENTION_PIECES_MAX_BLOCKS = 160     # blocks of the uncut step (segments x heads x column blocks) up to which they are: about one a SM
RETENTION_PIECES_BLOCKS_WANTED = 768  # blocks of the cut step that the piece size aims at
RETENTION_PIECES_MAX_BYTES = 1 << 29  # the most scratch (start states of all pieces) a step may take


def retention_piece_decays(decays):
    """``[RETENTION_PIECE_SIZES, heads]`` 32-bit: row i holds decay^(32 (i + 1)) per head, made in 64-bit and rounded
    once: what a whole piece of a cut segment takes off a state."""
    return torch.tensor([[float(d) ** (RETENTION_PIECE_UNIT * (i + 1)) for d in decays] for i in range(RETENTION_PIECE_SIZES)],
                        dtype=torch.float64).to(torch.float32)


def retention_piece_rows(longest: int, n_segments: int, heads: int, dim: int, v_dim: int, total_rows: int = 0) -> int:
    """Rows of a piece for a step whose longest segment has ``longest`` rows, 0 where segments stay whole: they are cut
    where the uncut step has about a block a SM or fewer, into as many pieces as give RETENTION_PIECES_BLOCKS_WANTED
    blocks (measured: with 32 blocks a segment 16 to 32 pieces are best, with 128 blocks 4 to 8, above 500 none).
    With ``total_rows`` the step counts as no more segments than its rows would fill at the longest one's length: a
    prompt beside a few decoding rows is still one long walk."""
    if total_rows > 0 and longest > 0:
        n_long = min(n_segments, -(-total_rows // longest))
    else:
        n_long = n_segments
    blocks = n_long * heads * -(-v_dim // (64 if dim <= 128 else 32))
    if longest < RETENTION_PIECES_FROM or blocks > RETENTION_PIECES_MAX_BLOCKS:
        return 0
    want = max(2, RETENTION_PIECES_BLOCKS_WANTED // blocks)
    rows = -(-(-(-longest // want)) // RETENTION_PIECE_UNIT) * RETENTION_PIECE_UNIT
    rows = min(rows, RETENTION_PIECE_UNIT * RETENTION_PIECE_SIZES)
    n = -(-longest // rows)
    if n < 2 or n_segments * n > 65535 or n_segments * n * heads * v_dim * dim * 4 > RETENTION_PIECES_MAX_BYTES:
        return 0
    return rows


def retention(qkv, q_off, k_off, v_off, positions, freqs, rot_dims, k_scale, one_minus_decay, state, seg_slot, cu_rows,
              n_segments, heads, dim, v_dim, y, max_seg_rows: int = 0, piece_decays=None, piece_rows=None):
    """Retention over every segment's rows, from and into the requests' states: per head S <- decay S + k v^T,
    y = S^T q, after the first ``rot_dims`` entries of q and k were rotated in pairs (entry i with i + rot_dims/2) by
    position * freqs[i] and k was multiplied by ``k_scale``.  ``qkv``: the compute type, q | k | v at their column
    offsets; ``one_minus_decay``: 32-bit ``[heads]``, 1 - decay per head; ``y``: 32-bit ``[T, heads * v_dim]``;
    ``state``: 32-bit ``[slots, heads * v_dim * dim]``; ``max_seg_rows``: the step's longest segment if known.

    A segment's rows are walked in order.  With ``piece_decays`` (``retention_piece_decays`` of the heads' decays, on
    the device), where the step's longest segment is long and its blocks are few (``retention_piece_rows``), segments
    are cut into pieces that run side by side: every piece's end state from zero, then the start states one after the
    other (start[p + 1] = decay^piece_rows start[p] + end[p]), then every piece again from its start state.  That is
    five thirds of the arithmetic for many times the parallel work; against the walk in one piece the results differ
    by rounding only.  ``piece_rows``: a piece size of one's own (a multiple of 32 up to 512); 0: never cut."""
    _need_cuda(qkv, positions, freqs, one_minus_decay, state, seg_slot, cu_rows, y, piece_decays)
    T = qkv.shape[0]
    assert qkv.stride(1) == 1 and positions.dtype == torch.int32 and positions.shape[0] >= T
    assert y.dtype == torch.float32 and y.stride(1) == 1 and y.shape == (T, heads * v_dim)
    assert state.dtype == torch.float32 and state.stride(1) == 1 and state.shape[1] >= heads * v_dim * dim
    assert one_minus_decay.dtype == torch.float32 and one_minus_decay.numel() == heads and one_minus_decay.is_contiguous()
    assert rot_dims == 0 or (freqs.dtype == torch.float32 and freqs.numel() >= rot_dims // 2 and freqs.is_contiguous())
    longest = int(max_seg_rows or 0)
    n_pieces, rows, starts, decay_piece = 1, 0, None, None
    if piece_decays is not None and piece_rows != 0 and longest > 0:
        assert piece_decays.dtype == torch.float32 and piece_decays.shape == (RETENTION_PIECE_SIZES, heads) and piece_decays.is_contiguous()
        rows = int(piece_rows) if piece_rows is not None else retention_piece_rows(longest, n_segments, heads, dim, v_dim, total_rows=T)
        assert rows >= 0 and rows % RETENTION_PIECE_UNIT == 0 and rows <= RETENTION_PIECE_UNIT * RETENTION_PIECE_SIZES
        if rows and longest > rows:
            n_pieces = -(-longest // rows)
            decay_piece = piece_decays[rows // RETENTION_PIECE_UNIT - 1]
            starts = torch.empty((n_segments * n_pieces, heads * v_dim * dim), dtype=torch.float32, device=qkv.device)
    st = kernels().cbis_retention(_ptr(qkv), c_int(qkv.stride(0)), c_int(q_off), c_int(k_off), c_int(v_off), _ptr(positions),
                                  _ptr(freqs), c_int(rot_dims), c_float(k_scale), _ptr(one_minus_decay), _ptr(state),
                                  ctypes.c_longlong(state.stride(0)), _ptr(seg_slot), _ptr(cu_rows), _ptr(y),
                                  c_int(y.stride(0)), c_int(n_segments), c_int(heads), c_int(dim), c_int(v_dim),
                                  c_int(dtype_code(qkv.dtype)), _stream(), c_int(longest), c_int(n_pieces),
                                  c_int(rows if n_pieces > 1 else 0), _ptr(starts), _ptr(decay_piece))
    _check(st, "retention", f"segments={n_segments} heads={heads} dim={dim} v_dim={v_dim} rot_dims={rot_dims} "
                            f"pieces={n_pieces}", launches=3 if n_pieces > 1 else 1)


def qk_prepare(buf, q_off, q_heads, k_off, k_heads, width, q_weight, k_weight, eps, positions, freqs, rot_dims,
               v_off=0, d_v=0, v_other=None, blend: float = 0.0):
    """What stands between a projection q | k | v (``buf``, the compute type, changed in place) and attention, in
    one pass over a row, 32-bit arithmetic, one rounding: all of q (``q_heads`` x ``width`` from column ``q_off``)
    divided by its root mean square and multiplied by ``q_weight``, the same for all of k (weights None: no norm);
    every head's first ``rot_dims`` entries rotated in pairs (entry i with i + rot_dims/2) by position * freqs[i]; and
    with ``v_other`` (``[rows, d_v]``) the ``d_v`` columns from ``v_off`` become (1 - blend) v + blend v_other."""
    _need_cuda(buf, q_weight, k_weight, positions, freqs, v_other)
    rows = buf.shape[0]
    assert buf.stride(1) == 1 and positions.dtype == torch.int32 and positions.shape[0] >= rows
    assert q_off + q_heads * width <= buf.shape[1] and k_off + k_heads * width <= buf.shape[1]
    for w, n in ((q_weight, q_heads * width), (k_weight, k_heads * width)):
        assert w is None or (w.dtype == torch.float32 and w.numel() == n and w.is_contiguous())
    assert rot_dims == 0 or (freqs.dtype == torch.float32 and freqs.numel() >= rot_dims // 2 and freqs.is_contiguous())
    assert v_other is None or (v_other.dtype == buf.dtype and v_other.stride(1) == 1 and v_other.shape == (rows, d_v)
                               and v_off + d_v <= buf.shape[1])
    st = kernels().cbis_qk_prepare(_ptr(buf), c_int(buf.stride(0)), c_int(q_off), c_int(q_heads), c_int(k_off), c_int(k_heads),
                                   c_int(width), _ptr(q_weight), _ptr(k_weight), c_float(eps), _ptr(positions), _ptr(freqs),
                                   c_int(rot_dims), c_int(v_off), c_int(d_v), _ptr(v_other),
                                   c_int(v_other.stride(0) if v_other is not None else 0), c_float(blend), c_int(rows),
                                   c_int(dtype_code(buf.dtype)), _stream())
    _check(st, "qk_prepare", f"rows={rows} heads={q_heads}/{k_heads} width={width} rot_dims={rot_dims}")


def qk_turn_norm(buf, q_off, q_heads, k_off, k_heads, width, eps, positions, freqs, rot_dims, length: float = 1.0,
                 q_weight=None, k_weight=None):
    """Every head of q (``q_heads`` x ``width`` columns of ``buf`` from ``q_off``, in place) and of k: its first ``rot_dims``
    entries rotated in pairs (entry i with i + rot_dims/2) by position * freqs[i], cosine and sine times ``length``; then
    the head divided by its own root mean square and, with a weight (``width`` numbers, shared by all heads), multiplied by
    it.  32-bit arithmetic, one rounding; heads up to 512 wide."""
    _need_cuda(buf, q_weight, k_weight, positions, freqs)
    rows = buf.shape[0]
    assert buf.stride(1) == 1 and positions.dtype == torch.int32 and positions.shape[0] >= rows
    assert q_off + q_heads * width <= buf.shape[1] and k_off + k_heads * width <= buf.shape[1]
    for w in (q_weight, k_weight):
        assert w is None or (w.dtype == torch.float32 and w.numel() == width and w.is_contiguous())
    assert rot_dims == 0 or (freqs.dtype == torch.float32 and freqs.numel() >= rot_dims // 2 and freqs.is_contiguous())
    st = kernels().cbis_qk_turn_norm(_ptr(buf), c_int(buf.stride(0)), c_int(q_off), c_int(q_heads), c_int(k_off), c_int(k_heads),
                                     c_int(width), _ptr(q_weight), _ptr(k_weight), c_float(eps), _ptr(positions), _ptr(freqs),
                                     c_int(rot_dims), c_float(length), c_int(rows), c_int(dtype_code(buf.dtype)), _stream())
    _check(st, "qk_turn_norm", f"rows={rows} heads={q_heads}/{k_heads} width={width} rot_dims={rot_dims}")


TIME_MIXING_MAX_DIM = 512        # the widest head of the time-mixing kernel (cbis_time_mixing_max_dim())
TOKEN_SHIFT_MOST = 8             # blends token_shift takes


def token_shift(h, state, seg_slot, row_seq, cu_rows, mu, out):
    """out[:, s * W:(s + 1) * W] = h + (h' - h) * mu[s] with h' the row before each row: the row above it in its segment,
    or, for a segment's first row, the request's row of ``state`` (32-bit, ``[slots, >= W]``), which then takes the
    segment's last row.  ``mu`` 32-bit ``[blends, W]``; rows of no segment (``row_seq`` negative) come out as zeros."""
    _need_cuda(h, state, seg_slot, row_seq, cu_rows, mu, out)
    rows, W = h.shape
    n = mu.shape[0]
    assert h.stride(1) == 1 and out.stride(1) == 1 and out.shape == (rows, n * W) and out.dtype == h.dtype
    assert mu.dtype == torch.float32 and mu.is_contiguous() and mu.shape[1] == W
    assert state.dtype == torch.float32 and state.stride(1) == 1 and state.shape[1] >= W
    assert row_seq.dtype == torch.int32 and row_seq.shape[0] >= rows
    st = kernels().cbis_token_shift(_ptr(h), c_int(h.stride(0)), _ptr(state), ctypes.c_longlong(state.stride(0)), _ptr(seg_slot),
                                    _ptr(row_seq), _ptr(cu_rows), _ptr(mu), c_int(n), _ptr(out), c_int(out.stride(0)), c_int(W),
                                    c_int(rows), c_int(dtype_code(h.dtype)), _stream())
    _check(st, "token_shift", f"rows={rows} width={W} blends={n}")


def linear_blends(x, w_all, n_groups, group_n, tail_act=None):
    """Products of blends that lie side by side in x (K columns each, K the weights' width): the first ``n_groups`` with
    ``group_n`` rows of ``w_all`` each, the one after them with the rows left over, through ``tail_act``.  Returns
    (``[T, n_groups * group_n]``, ``[T, rest]``) of x's type.  A few rows of bfloat16: one weight-streaming product."""
    _need_cuda(x, w_all)
    T = x.shape[0]
    N, K = w_all.shape
    n_all = n_groups * group_n
    rest = N - n_all
    if (x.dtype == torch.bfloat16 and 0 < T <= SMALL_M and group_n % 16 == 0 and 0 < rest <= group_n and K % 8 == 0
            and x.stride(0) % 8 == 0 and x.data_ptr() % 16 == 0):
        out = torch.empty((T, N), dtype=x.dtype, device=x.device)
        gemm_small_m(x, w_all, None, tail_act, out, group_n=group_n, act_from=n_all)
        return out[:, :n_all], out[:, n_all:]
    out = torch.empty((T, n_all), dtype=x.dtype, device=x.device)
    linear_heads(x, w_all[:n_all].view(n_groups, group_n, K), out)
    return out, linear(x[:, n_groups * K:], w_all[n_all:], None, tail_act)


TIME_MIXING_ROUND = 4 * 148      # blocks of the walk that run at a time


def time_mixing_piece_rows(longest: int, n_segments: int, heads: int, dim: int, total_rows: int = 0) -> int:
    """Rows of a piece for a step whose longest segment has ``longest`` rows, 0 where segments stay whole: they are cut where
    the uncut step has about a block a SM or fewer, into as many pieces as run in one round.  ``total_rows``: as in
    ``retention_piece_rows``."""
    n_long = min(n_segments, -(-total_rows // longest)) if total_rows > 0 and longest > 0 else n_segments
    blocks = max(1, n_long * heads * -(-dim // (64 if dim <= 128 else 32)))
    if longest < RETENTION_PIECES_FROM or blocks > RETENTION_PIECES_MAX_BLOCKS:
        return 0
    want = max(2, TIME_MIXING_ROUND // blocks)
    rows = max(32, -(-(-(-longest // want)) // 16) * 16)
    n = -(-longest // rows)
    if n < 2 or n_segments * n > 65535 or n_segments * n * heads * dim * dim * 4 > RETENTION_PIECES_MAX_BYTES:
        return 0
    return rows


def time_mixing(x, r_off, k_off, v_off, raw, w0, u, state, seg_slot, cu_rows, n_segments, heads, dim, y, max_seg_rows: int = 0,
                piece_rows=None):
    """The recurrence o = (S + diag(u) k v^T)^T r, S <- diag(w) S + k v^T, w = exp(-exp(raw + w0)), per head over every
    segment's rows, from and into the requests' states.  ``x``: the compute type, r, k and v at their column offsets;
    ``raw``: 32-bit ``[T, heads * dim]``; ``w0``, ``u``: 32-bit, heads * dim numbers; ``y``: 32-bit ``[T, heads * dim]``;
    ``state``: 32-bit ``[slots, >= heads * dim * dim]``; ``max_seg_rows``: the step's longest segment if known.

    A segment's rows are walked in order.  Where the step's longest segment is long and its blocks are few
    (``time_mixing_piece_rows``), segments are cut into pieces that run side by side; against
    the walk in one piece the results differ by rounding only.  ``piece_rows``: a piece size of one's own (a multiple of
    16); 0: never cut."""
    _need_cuda(x, raw, w0, u, state, seg_slot, cu_rows, y)
    T = x.shape[0]
    HD = heads * dim
    assert x.stride(1) == 1 and max(r_off, k_off, v_off) + HD <= x.shape[1]
    assert raw.dtype == torch.float32 and raw.stride(1) == 1 and raw.shape == (T, HD)
    assert y.dtype == torch.float32 and y.stride(1) == 1 and y.shape == (T, HD)
    assert state.dtype == torch.float32 and state.stride(1) == 1 and state.shape[1] >= HD * dim
    for t in (w0, u):
        assert t.dtype == torch.float32 and t.numel() == HD and t.is_contiguous()
    longest = int(max_seg_rows or 0)
    rows = 0
    if piece_rows != 0 and longest > 0:
        rows = int(piece_rows) if piece_rows is not None else time_mixing_piece_rows(longest, n_segments, heads, dim, total_rows=T)
        assert rows >= 0 and rows % 16 == 0
    n_pieces, starts, products = 1, None, None
    if rows and longest > rows:
        n_pieces = -(-longest // rows)
        starts = torch.empty((n_segments * n_pieces, HD * dim), dtype=torch.float32, device=x.device)
        products = torch.empty((n_segments * n_pieces, HD), dtype=torch.float32, device=x.device)
    st = kernels().cbis_time_mixing(_ptr(x), c_int(x.stride(0)), c_int(r_off), c_int(k_off), c_int(v_off), _ptr(raw),
                                    c_int(raw.stride(0)), _ptr(w0), _ptr(u), _ptr(state), ctypes.c_longlong(state.stride(0)),
                                    _ptr(seg_slot), _ptr(cu_rows), _ptr(y), c_int(y.stride(0)), c_int(n_segments), c_int(heads),
                                    c_int(dim), c_int(dtype_code(x.dtype)), _stream(), c_int(longest), c_int(n_pieces),
                                    c_int(rows if n_pieces > 1 else 0), _ptr(starts), _ptr(products))
    _check(st, "time_mixing", f"segments={n_segments} heads={heads} dim={dim} pieces={n_pieces}", launches=3 if n_pieces > 1 else 1)


def qk_head_norm(buf, q_off, q_heads, k_off, k_heads, width, q_weight, k_weight, eps):
    """Every head of q (``q_heads`` x ``width`` columns of ``buf`` from ``q_off``, in place) divided by its own root mean
    square and multiplied by ``q_weight`` (``width`` numbers, shared by all heads); the same for k (``k_heads`` 0: none).
    32-bit arithmetic, one rounding; heads up to 512 wide."""
    _need_cuda(buf, q_weight, k_weight)
    assert buf.stride(1) == 1 and q_off + q_heads * width <= buf.shape[1] and k_off + k_heads * width <= buf.shape[1]
    for w, n in ((q_weight, q_heads), (k_weight, k_heads)):
        assert n == 0 or (w.dtype == torch.float32 and w.numel() == width and w.is_contiguous())
    st = kernels().cbis_qk_head_norm(_ptr(buf), c_int(buf.stride(0)), c_int(q_off), c_int(q_heads), c_int(k_off), c_int(k_heads),
                                     c_int(width), _ptr(q_weight), _ptr(k_weight), c_float(eps), c_int(buf.shape[0]),
                                     c_int(dtype_code(buf.dtype)), _stream())
    _check(st, "qk_head_norm", f"rows={buf.shape[0]} heads={q_heads}/{k_heads} width={width}")


MIX_HEADS_MAX_HEADS = 224        # the most heads mix_heads takes (cbis_mix_heads_max_heads() says the same)


def mix_heads(o, talk, n_head, n_kv_head, v_dim, out, gate=None):
    """out[:, h] = sum over g of talk[h, g] * o[:, g, kv(h)], kv(h) = h // (n_head / n_kv_head), times sigmoid(gate[:, h])
    element by element if a gate is given.  ``o`` ``[rows, n_head * n_kv_head * v_dim]``: what query head g's weights make of
    the values of every key/value head, side by side; talk 32-bit ``[n_head, n_head]``; out and gate
    ``[rows, n_head * v_dim]`` of o's type.  Sums in 32-bit, one rounding."""
    _need_cuda(o, talk, out, gate)
    rows = o.shape[0]
    assert o.shape[1] == n_head * n_kv_head * v_dim and o.stride(1) == 1 and out.stride(1) == 1 and out.dtype == o.dtype
    assert talk.dtype == torch.float32 and talk.shape == (n_head, n_head) and talk.is_contiguous()
    assert out.shape == (rows, n_head * v_dim)
    assert gate is None or (gate.dtype == o.dtype and gate.shape == out.shape and gate.stride(1) == 1)
    st = kernels().cbis_mix_heads(_ptr(o), c_int(o.stride(0)), _ptr(talk), _ptr(gate), c_int(gate.stride(0) if gate is not None else 0),
                                  _ptr(out), c_int(out.stride(0)), c_int(rows), c_int(n_head), c_int(n_kv_head), c_int(v_dim),
                                  c_int(dtype_code(o.dtype)), _stream())
    _check(st, "mix_heads", f"rows={rows} heads={n_head}/{n_kv_head} v_dim={v_dim}")


def blend_rows(a, b, blend: float, out):
    """out = (1 - blend) a + blend b element by element (32-bit arithmetic, one rounding); ``[rows, n]`` of one type,
    views with unit column stride are fine."""
    _need_cuda(a, b, out)
    rows, n = a.shape
    assert b.shape == a.shape and out.shape == a.shape and a.dtype == b.dtype == out.dtype
    assert a.stride(1) == 1 and b.stride(1) == 1 and out.stride(1) == 1
    st = kernels().cbis_blend_rows(_ptr(a), c_int(a.stride(0)), _ptr(b), c_int(b.stride(0)), _ptr(out), c_int(out.stride(0)),
                                   c_float(blend), c_int(rows), c_int(n), c_int(dtype_code(a.dtype)), _stream())
    _check(st, "blend_rows", f"rows={rows} n={n}")


_limits = {}


def conv_max_taps() -> int:
    if "taps" not in _limits:
        _limits["taps"] = int(kernels().cbis_conv_max_taps())
    return _limits["taps"]


def scan_max_state() -> int:
    if "state" not in _limits:
        _limits["state"] = int(kernels().cbis_scan_max_state())
    return _limits["state"]


def conv_rows_per_block() -> int:
    if "conv_rows" not in _limits:
        _limits["conv_rows"] = int(kernels().cbis_conv_rows_per_block())
    return _limits["conv_rows"]


def causal_conv_act(x, c0, channels, weight, bias, state, seg_slot, cu_rows, n_segments, max_seg_rows, act, out,
                    update_state=False):
    """Causal convolution per channel over each segment's rows, bias and activation: the channels are columns
    ``c0 .. c0 + channels - 1`` of x; ``weight`` ``[channels, taps]`` (the last tap meets the current row) and
    ``bias`` 32-bit; ``state`` ``[slots, >= (taps-1)*channels]`` 32-bit holds every request's last taps-1 inputs
    (zeros at a sequence's start) and is NOT changed (``conv_state_update`` does that afterwards), unless
    ``update_state`` is set, which a step may do whose longest segment has at most ``conv_rows_per_block()`` rows (a
    decode step): the same kernel then leaves the state as ``conv_state_update`` would."""
    _need_cuda(x, weight, bias, state, seg_slot, cu_rows, out)
    taps = weight.shape[1]
    assert x.stride(1) == 1 and out.stride(1) == 1 and out.shape == (x.shape[0], channels) and out.dtype == x.dtype
    assert weight.dtype == torch.float32 and weight.is_contiguous() and weight.shape[0] == channels
    assert state.dtype == torch.float32 and state.stride(1) == 1 and state.shape[1] >= (taps - 1) * channels
    st = kernels().cbis_causal_conv_act(_ptr(x), c_int(x.stride(0)), c_int(c0), _ptr(weight), _ptr(bias), _ptr(state),
                                        ctypes.c_longlong(state.stride(0)), _ptr(seg_slot), _ptr(cu_rows), _ptr(out),
                                        c_int(out.stride(0)), c_int(channels), c_int(taps), c_int(ACT[act]),
                                        c_int(n_segments), c_int(max_seg_rows), c_int(1 if update_state else 0),
                                        c_int(dtype_code(x.dtype)), _stream())
    _check(st, "causal_conv_act", f"channels={channels} taps={taps} segments={n_segments}")


def conv_state_update(x, c0, channels, taps, state, seg_slot, cu_rows, n_segments):
    """Every segment's request keeps its last ``taps - 1`` inputs (older ones move up when a segment is shorter)."""
    _need_cuda(x, state, seg_slot, cu_rows)
    st = kernels().cbis_conv_state_update(_ptr(x), c_int(x.stride(0)), c_int(c0), _ptr(state),
                                          ctypes.c_longlong(state.stride(0)), _ptr(seg_slot), _ptr(cu_rows),
                                          c_int(channels), c_int(taps), c_int(n_segments), c_int(dtype_code(x.dtype)),
                                          _stream())
    _check(st, "conv_state_update", f"channels={channels} taps={taps} segments={n_segments}")


# A long segment of a state-space layer is cut into pieces that run side by side where the step's states are few:
# measured on 2,048 rows (us, one piece -> pieces of 128 rows): 18 k state elements (segments x heads x columns x
# states) 293 -> 81, 65 k 300 -> 147, 131 k 438 -> 252, 262 k 546 -> 476 or 473 -> 460, 524 k 578 -> 840: twice the
# arithmetic pays only while one piece leaves most of the machine idle.
SCAN_PIECE_ROWS = 128           # rows of a piece
SCAN_PIECES_FROM = 384          # the longest segment of a step from which segments are cut
SCAN_PIECES_MAX_STATE = 200_000  # state elements of a step up to which they are


def ssm_scan(xbc, proj, dt_off, dt_bias, a_log, d_skip, state, seg_slot, cu_rows, n_segments, heads, head_dim, n_state,
             groups, y, max_seg_rows=None, piece_rows=None):
    """The selective state-space recurrence over each segment's rows, from and into ``state`` ``[slots, >= heads *
    head_dim * n_state]`` (32-bit, laid out ``[head][column][state]``): per head, with dt = softplus(raw + dt_bias),
    S <- exp(-exp(a_log) dt) S + dt B x^T and y = S^T C + d_skip x.  ``xbc`` rows: x | B | C (compute type); the raw
    step sizes are columns ``dt_off ..`` of ``proj``; ``y`` ``[T, heads * head_dim]`` 32-bit.

    A segment's rows are walked in order.  Where the step's longest segment (``max_seg_rows``) is long and the step's
    states are few, segments are cut into pieces of ``piece_rows`` rows that run side by side: every piece's end
    state from zero, then the start states one after the other (S_next = S + expm1(sum of log-decays) S + end), then
    every piece again from its start state.  That is twice the arithmetic for many times the parallel work; against
    the walk in one piece the results differ by rounding only.  ``piece_rows`` names the size (0: never cut)."""
    _need_cuda(xbc, proj, dt_bias, a_log, d_skip, state, seg_slot, cu_rows, y)
    assert xbc.stride(1) == 1 and proj.stride(1) == 1 and y.dtype == torch.float32 and y.stride(1) == 1
    assert xbc.dtype == proj.dtype and state.dtype == torch.float32 and state.stride(1) == 1
    assert state.shape[1] >= heads * head_dim * n_state and xbc.shape[1] == heads * head_dim + 2 * groups * n_state
    assert all(t.dtype == torch.float32 and t.numel() == heads for t in (dt_bias, a_log, d_skip))
    longest = int(max_seg_rows) if max_seg_rows is not None else 0
    if piece_rows is None:
        few = n_segments * heads * head_dim * n_state <= SCAN_PIECES_MAX_STATE
        piece_rows = SCAN_PIECE_ROWS if (few and longest >= SCAN_PIECES_FROM) else 0
    n_pieces = -(-longest // piece_rows) if piece_rows and longest > piece_rows else 1
    ends = logs = None
    if n_pieces > 1:
        ends = torch.empty((n_segments * n_pieces, heads * head_dim * n_state), dtype=torch.float32, device=xbc.device)
        logs = torch.empty((n_segments * n_pieces, heads), dtype=torch.float32, device=xbc.device)
    st = kernels().cbis_ssm_scan(_ptr(xbc), c_int(xbc.stride(0)), _ptr(proj), c_int(proj.stride(0)), c_int(dt_off),
                                 _ptr(dt_bias), _ptr(a_log), _ptr(d_skip), _ptr(state), ctypes.c_longlong(state.stride(0)),
                                 _ptr(seg_slot), _ptr(cu_rows), _ptr(y), c_int(y.stride(0)), c_int(n_segments),
                                 c_int(heads), c_int(head_dim), c_int(n_state), c_int(groups),
                                 c_int(dtype_code(xbc.dtype)), c_int(n_pieces), c_int(piece_rows or 0), _ptr(ends),
                                 _ptr(logs), _stream())
    _check(st, "ssm_scan", f"heads={heads} head_dim={head_dim} state={n_state} groups={groups} segments={n_segments} "
                           f"pieces={n_pieces}", launches=3 if n_pieces > 1 else 1)


ROUTE_SCORE = {"sigmoid": 0, "softmax": 1}


def route_topk(h, router, top, score, renormalize, ids, weights, renorm_eps: float = 0.0, weight_scale: float = 1.0,
               correction=None, side=None):
    """Router logits ``h @ router^T`` in 32-bit, scores by ``score``, the ``top`` largest per row into ``ids``
    (int32 ``[rows, top]``) with their weights (float32; divided by their sum + ``renorm_eps`` with ``renormalize``;
    then times ``weight_scale``).  ``correction`` (32-bit, one per expert) joins the scores for the choice alone, not the
    weights.  ``side`` (32-bit ``[rows]``): the router's last row is no expert's; side takes the sigmoid of its logit."""
    _need_cuda(h, router, ids, weights, correction, side)
    rows, W = h.shape
    E = router.shape[0] - (1 if side is not None else 0)
    assert correction is None or (correction.dtype == torch.float32 and correction.numel() == E and correction.is_contiguous())
    assert side is None or (side.dtype == torch.float32 and side.numel() >= rows and side.is_contiguous())
    assert h.stride(1) == 1 and router.is_contiguous() and router.shape[1] == W and router.dtype == h.dtype
    assert ids.dtype == torch.int32 and weights.dtype == torch.float32 and ids.is_contiguous() and weights.is_contiguous()
    assert ids.shape == (rows, top) and weights.shape == (rows, top)
    st = kernels().cbis_route_topk(_ptr(h), c_int(h.stride(0)), _ptr(router), _ptr(ids), _ptr(weights), c_int(rows),
                                   c_int(W), c_int(E), c_int(top), c_int(ROUTE_SCORE[score]), c_int(1 if renormalize else 0),
                                   c_int(dtype_code(h.dtype)), _stream(), c_float(renorm_eps), c_float(weight_scale),
                                   _ptr(correction), _ptr(side))
    _check(st, "route_topk", f"rows={rows} experts={E} top={top}")


def routed_gate_up(h, gate_up, ids, weights, act, weight_on_input, hidden, limit: float = 0.0, beta: float = 1.0,
                   shift: float = 0.0):
    """hidden[(row, choice)] = act(s * gate_e(h[row])) * (s * up_e(h[row])), e the choice's expert, s its weight if
    the weight multiplies the expert's input, else 1.  ``gate_up`` ``[experts, 2 * inner, width]``; a choice beyond the
    experts is an identity expert and has no hidden row.  ``limit``, ``beta``, ``shift``: as in ``gate_mul``."""
    _need_cuda(h, gate_up, ids, weights, hidden)
    rows, W = h.shape
    E, F2, _ = gate_up.shape
    top = ids.shape[1]
    assert h.stride(1) == 1 and gate_up.is_contiguous() and gate_up.shape[2] == W and hidden.is_contiguous()
    assert hidden.shape == (rows * top, F2 // 2) and hidden.dtype == h.dtype == gate_up.dtype
    st = kernels().cbis_routed_gate_up(_ptr(h), c_int(h.stride(0)), _ptr(gate_up), _ptr(ids), _ptr(weights), _ptr(hidden),
                                       c_int(rows), c_int(W), c_int(F2 // 2), c_int(top), c_int(ACT[act]),
                                       c_int(1 if weight_on_input else 0), c_int(dtype_code(h.dtype)), _stream(), c_int(E),
                                       c_float(limit), c_float(beta), c_float(shift))
    _check(st, "routed_gate_up", f"rows={rows} width={W} inner={F2 // 2} top={top}")


def routed_down(hidden, down, ids, weights, weight_on_input, out, accumulate=False, h=None):
    """out[row] = the sum over the row's choices of down_e(hidden[(row, choice)]) (times the choice's weight unless
    it already multiplied the input); ``down`` ``[experts, width, inner]``; out 32-bit, added to with ``accumulate``.
    ``h``: the feed-forward's input rows; a choice beyond the experts is an identity expert and adds its weight times
    the row (without ``h`` no choice may be one)."""
    _need_cuda(hidden, down, ids, weights, out, h)
    E, W, F = down.shape
    rows, top = ids.shape
    assert hidden.is_contiguous() and hidden.shape == (rows * top, F) and down.is_contiguous() and hidden.dtype == down.dtype
    assert out.dtype == torch.float32 and out.shape == (rows, W) and out.stride(1) == 1
    st = kernels().cbis_routed_down(_ptr(hidden), _ptr(down), _ptr(ids), _ptr(weights), _ptr(out), c_int(out.stride(0)),
                                    c_int(rows), c_int(W), c_int(F), c_int(top), c_int(1 if weight_on_input else 0),
                                    c_int(1 if accumulate else 0), c_int(dtype_code(hidden.dtype)), _stream(),
                                  c_int(E if h is not None else 2 ** 31 - 1), _ptr(h), c_int(h.stride(0) if h is not None else 0))
    _check(st, "routed_down", f"rows={rows} width={W} inner={F} top={top}")


ROUTED_TILES_FROM = 33     # rows from which the routed feed-forward sorts its rows by expert and runs tiles on the tensor cores


def routed_tiles_takes(h, gate_up, down) -> bool:
    """Whether ``routed_tiles`` takes these rows: bfloat16, enough of them, sizes in steps of 8, aligned."""
    W, F = gate_up.shape[2], down.shape[2]
    return (h.dtype == torch.bfloat16 and h.shape[0] >= ROUTED_TILES_FROM and W % 8 == 0 and F % 8 == 0
            and h.stride(0) % 8 == 0 and h.data_ptr() % 16 == 0 and gate_up.shape[0] <= 4096)


def _routed_plan_ints(pairs: int, experts: int) -> int:
    fn = kernels().cbis_routed_plan_ints
    fn.restype = ctypes.c_longlong
    return int(fn(c_int(pairs), c_int(experts)))


def routed_tiles(h, gate_up, down, ids, weights, act, weight_on_input, out, accumulate=False, identity: int = 0,
                 limit: float = 0.0, beta: float = 1.0, shift: float = 0.0):
    """The routed feed-forward for many rows of bfloat16: the (row, choice) pairs are sorted by expert on the device, an
    expert's pairs run in tiles of 128 rows on the tensor cores (gate and up with the gated activation in one kernel,
    then down), and a row's choices are summed in their order.  ``out`` 32-bit ``[rows, width]``, overwritten or, with
    ``accumulate``, added to.  Nothing is read back to the host: it can be captured.  ``identity``: how many choices beyond
    the experts are identity experts (the row itself times the weight); ``limit``, ``beta``, ``shift``: as in ``gate_mul``."""
    _need_cuda(h, gate_up, down, ids, weights, out)
    rows, W = h.shape
    E, F2, _ = gate_up.shape
    F, top = F2 // 2, ids.shape[1]
    assert gate_up.is_contiguous() and down.is_contiguous() and down.shape == (E, W, F) and h.stride(1) == 1
    assert out.dtype == torch.float32 and out.shape == (rows, W) and out.stride(1) == 1
    plan = torch.empty(int(_routed_plan_ints(rows * top, E)), dtype=torch.int32, device=h.device)
    hidden = torch.empty((rows * top, F), dtype=torch.bfloat16, device=h.device)
    y = torch.empty((rows * top, W), dtype=torch.float32, device=h.device) if (top > 1 or accumulate or identity) else None
    st = kernels().cbis_routed_tiles(_ptr(h), c_int(h.stride(0)), _ptr(gate_up), _ptr(down), _ptr(ids), _ptr(weights),
                                     _ptr(plan), _ptr(hidden), _ptr(y), _ptr(out), c_int(out.stride(0)), c_int(rows),
                                     c_int(W), c_int(F), c_int(E), c_int(top), c_int(ACT[act]),
                                     c_int(1 if weight_on_input else 0), c_int(1 if accumulate else 0), _stream(), c_int(identity),
                                     c_float(limit), c_float(beta), c_float(shift))
    _check(st, "routed_tiles", f"rows={rows} width={W} inner={F} experts={E} top={top}", launches=4 if y is not None else 3)


def linear_residual(x, w_nk, residual) -> bool:
    """residual += x @ w_nk^T by a product that adds in place, where one takes these rows (bfloat16: the TMA + tcgen05
    product with its reduction into the 32-bit rows for prompts, the weight-streaming product for a few rows); returns
    whether it did.  After a no the caller computes the product and hands it on to be added."""
    if residual is None or x.dtype != torch.bfloat16 or not x.is_cuda:
        return False
    if linear_add_takes(x, w_nk, residual):
        linear_add(x, w_nk, None, residual)
        return True
    M, K = x.shape
    if (0 < M <= SMALL_M and K % 8 == 0 and x.stride(0) % 8 == 0 and x.data_ptr() % 16 == 0 and x.stride(1) == 1
            and residual.dtype == torch.float32 and residual.stride(1) == 1 and residual.shape == (M, w_nk.shape[0])):
        gemm_small_m(x, w_nk, None, None, residual, accumulate=True)
        return True
    return False


def decode_advance(tokens, positions, seg_start, seg_ctx, sampled, n):
    """tokens <- sampled, positions/seg_start/seg_ctx += 1 for the first n rows (all on the device)."""
    st = kernels().cbis_decode_advance(_ptr(tokens), _ptr(positions), _ptr(seg_start), _ptr(seg_ctx), _ptr(sampled),
                                       c_int(n), _stream())
    _check(st, "decode_advance")


def slots_from_table(positions, row_seq, block_table, page_size, slot_mapping, n):
    """slot_mapping[r] = token slot of positions[r] by the request's block table (-1 for padding rows)."""
    st = kernels().cbis_slots_from_table(_ptr(positions), _ptr(row_seq), _ptr(block_table),
                                         c_int(block_table.shape[1]), c_int(page_size), _ptr(slot_mapping), c_int(n),
                                         _stream())
    _check(st, "slots_from_table")


_sample_scratch = {}
_sample_outgrown = []     # buffers that a later call outgrew: a captured graph may still hold their addresses


def _sample_buffers(device, R: int, chunks: int):
    """Scratch of the sampling kernel, kept per device and grown as needed; counters start at zero
    and every launch leaves them zero."""
    key = device.index     # one scratch per device: launches on different streams must not overlap
    have = _sample_scratch.get(key)
    if have is None or have[0].numel() < R * chunks or have[2].numel() < R:
        if torch.cuda.is_current_stream_capturing():
            raise KernelError("sampling scratch would have to grow during graph capture")
        n = max(R * chunks, 64 * 64)
        if have is not None:
            _sample_outgrown.append(have)
        have = (torch.empty(n, dtype=torch.float32, device=device), torch.empty(n, dtype=torch.int32, device=device),
                torch.zeros(max(R, 1024), dtype=torch.int32, device=device))
        _sample_scratch[key] = have
    return have


def sample(logits, temperature, keys, out):
    """out[r] = argmax_i(logits[r,i]) (temperature[r] <= 0 or None) or the Gumbel-max draw keyed by keys[r]."""
    _need_cuda(logits, temperature, keys, out)
    R, V = logits.shape
    assert logits.dtype == torch.float32 and logits.stride(1) == 1 and out.dtype == torch.int32
    assert temperature is None or temperature.dtype == torch.float32
    assert keys is None or keys.dtype == torch.int64
    chunks = kernels().cbis_sample_chunks(c_int(V))
    pv, pi, cnt = _sample_buffers(logits.device, R, chunks)
    st = kernels().cbis_sample(_ptr(logits), c_int(logits.stride(0)), _ptr(temperature), _ptr(keys), _ptr(out),
                               c_int(R), c_int(V), _ptr(pv), _ptr(pi), _ptr(cnt), _stream())
    _check(st, "sample", f"R={R} V={V}")
