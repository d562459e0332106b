"""Python entry to the tcgen05 GEMM (eb_gemm): C = act(A @ W.T + bias) + residual."""
import torch

from ._lib import lib, check, dtype_code, ptr, stream_ptr, require_cuda, ACT_NONE, ACT_RELU, ACT_GELU_TANH, ACT_GELU_ERF

ACT_CODES = {None: ACT_NONE, "none": ACT_NONE, "relu": ACT_RELU, "gelu_tanh": ACT_GELU_TANH, "gelu": ACT_GELU_ERF}

_workspaces, _outgrown = {}, []


def workspace(device, nbytes):
    """Per-device scratch for the small-M (generation-step) GEMM: zero-filled once, grown on
    demand.  One buffer per device is enough because calls on a device are issued on one stream."""
    key = torch.device(device).index
    ws = _workspaces.get(key)
    if ws is None or ws.numel() < nbytes:
        if ws is not None:
            _outgrown.append(ws)             # captured steps may still hold its address
        ws = torch.zeros(max(nbytes, 1 << 20), dtype=torch.uint8, device=device)
        _workspaces[key] = ws
    return ws


def gemm(a, w, bias=None, act=None, residual=None, out=None, out_dtype=None, out_rows_per_batch=0,
         out_batch_stride=0, out_ld=None, out_row_offset_device=None, out_row_limit=0, static_weight=False, peer=None,
         ln_fold=None):
    """a [M,K] (row stride allowed), w [N,K]; returns out [M,N].

    `out`, if given, receives the result; with out_rows_per_batch > 0 row m is written at
    element (m // rpb) * out_batch_stride + (m % rpb) * out_ld of `out` (a view into a cache);
    out_row_offset_device (int32 device scalar) adds that many rows of out_ld at run time;
    out_row_limit > 0 is the number of rows that offset may address (beyond it the kernel
    stores nothing and raises the device status word).
    static_weight=True promises that `w` is not being written by earlier work still in flight
    on the stream (model weights), which lets the kernel prefetch it early.
    ln_fold=(colsum, bias32, eps), from fold_layernorm(): `a` is the un-normalised input of a
    LayerNorm and `w` the weight with the LayerNorm scale folded in (M <= 32 only).
    (Asking a launch to pull the NEXT launch's weights into L2 was tried and removed: measured on
    B200 it slowed the generation step at every size, 6.50 -> 6.70 / 7.28 ms for 16 / 64 MB on one
    GPU and 2.50 -> 2.57 / 2.63 ms on an 8-way shard.)"""
    require_cuda(a, w, bias, residual, out)
    if a.dim() != 2 or w.dim() != 2 or a.shape[1] != w.shape[1]:
        raise RuntimeError(f"gemm: shapes {tuple(a.shape)} x {tuple(w.shape)}^T do not match")
    if a.dtype != w.dtype or a.dtype not in (torch.float16, torch.bfloat16):
        raise RuntimeError("gemm: fp16 or bf16 operands of one dtype required")
    if a.stride(1) != 1:
        a = a.contiguous()
    if w.stride(1) != 1:
        w = w.contiguous()
    M, K = a.shape
    N = w.shape[0]
    out_dtype = out_dtype or a.dtype
    if out is None:
        out = torch.empty((M, N), dtype=out_dtype, device=a.device)
    if out_ld is None:
        out_ld = out.stride(0) if out.dim() == 2 else N
    if residual is not None and (residual.stride(-1) != 1 or residual.dtype != a.dtype):
        raise RuntimeError("gemm: residual must be row-major and of the operand dtype")
    code = ACT_CODES[act] if not isinstance(act, int) else act
    nbytes = lib().eb_gemm_workspace_bytes(M, N, K)
    ws = workspace(a.device, nbytes) if nbytes else None
    if ln_fold is not None:
        colsum, bias32, eps = ln_fold
        if bias is not None or peer is not None:
            raise RuntimeError("gemm: ln_fold carries the bias and does not combine with the peer exchange")
        if colsum.dtype != torch.float32 or bias32.dtype != torch.float32 or colsum.numel() != N or bias32.numel() != N:
            raise RuntimeError("gemm: ln_fold vectors must be fp32 of length N")
        check(lib().eb_gemm_ln(ptr(a), a.stride(0), ptr(w), w.stride(0), ptr(out), out_ld, ptr(colsum), ptr(bias32), float(eps),
                               ptr(residual), residual.stride(0) if residual is not None else 0, M, N, K,
                               dtype_code(a.dtype), dtype_code(out_dtype), code, out_rows_per_batch, out_batch_stride,
                               ptr(out_row_offset_device), int(out_row_limit), 1 if static_weight else 0, ptr(ws),
                               ws.numel() if ws is not None else 0, stream_ptr()), "gemm_ln")
        return out
    if peer is not None:
        if not peer.fits(M, N):
            raise RuntimeError(f"gemm: {M} x {N} does not fit the peer exchange areas")
        check(lib().eb_gemm_allreduce(ptr(a), a.stride(0), ptr(w), w.stride(0), ptr(out), out_ld, ptr(bias), ptr(residual),
                                      residual.stride(0) if residual is not None else 0, M, N, K, dtype_code(a.dtype),
                                      dtype_code(out_dtype), code, out_rows_per_batch, out_batch_stride,
                                      ptr(out_row_offset_device), int(out_row_limit), 1 if static_weight else 0, ptr(ws),
                                      ws.numel() if ws is not None else 0, peer.handle, stream_ptr()),
              "gemm_allreduce")
        return out
    check(lib().eb_gemm(ptr(a), a.stride(0), ptr(w), w.stride(0), ptr(out), out_ld, ptr(bias), ptr(residual),
                        residual.stride(0) if residual is not None else 0, M, N, K, dtype_code(a.dtype),
                        dtype_code(out_dtype), code, out_rows_per_batch, out_batch_stride,
                        ptr(out_row_offset_device), int(out_row_limit), 1 if static_weight else 0, ptr(ws),
                        ws.numel() if ws is not None else 0, stream_ptr()), "gemm")
    return out


def gemm_parts(a, w, bias=None, xielu=None, tail_col=None, static_weight=False):
    """a [M,K] @ w [N,K].T + bias for stacked weights: xielu = (act_params, act_cols), that activation on
    the columns below act_cols (act_params: device fp32 pair, see xielu_params()); tail_col: the columns
    from there on are returned in fp32.  Returns out, or (out, tail) with tail_col."""
    act_params, act_cols = xielu if xielu is not None else (None, 0)
    require_cuda(a, w, bias, act_params)
    if a.dim() != 2 or w.dim() != 2 or a.shape[1] != w.shape[1] or a.dtype != w.dtype or a.dtype not in (torch.float16, torch.bfloat16):
        raise RuntimeError("gemm_parts: fp16 or bf16 a [M,K] and w [N,K] of one dtype required")
    if act_params is not None and (act_params.dtype != torch.float32 or act_params.numel() != 2):
        raise RuntimeError("gemm_parts: the activation has two fp32 numbers")
    if bias is not None and (bias.dtype != a.dtype or bias.numel() != w.shape[0]):
        raise RuntimeError("gemm_parts: the bias has the operand dtype and one entry per column")
    a, w = (t if t.stride(1) == 1 else t.contiguous() for t in (a, w))
    (M, K), N = a.shape, w.shape[0]
    out = torch.empty((M, N if tail_col is None else tail_col), dtype=a.dtype, device=a.device)
    tail = torch.empty((M, N - tail_col), dtype=torch.float32, device=a.device) if tail_col is not None else None
    nbytes = lib().eb_gemm_workspace_bytes(M, N, K)
    ws = workspace(a.device, nbytes) if nbytes else None
    check(lib().eb_gemm_parts(ptr(a), a.stride(0), ptr(w), w.stride(0), ptr(out), out.shape[1], ptr(bias), M, N, K, int(act_cols),
                              ptr(act_params), tail_col or 0, ptr(tail), tail.shape[1] if tail is not None else 0, dtype_code(a.dtype),
                              1 if static_weight else 0, ptr(ws), ws.numel() if ws is not None else 0, stream_ptr()), "gemm_parts")
    return out if tail is None else (out, tail)


def xielu_params(p, q):
    """(softplus(p), 1/2 + softplus(q)) as the fp32 pair the kernels take."""
    s = torch.nn.functional.softplus(torch.tensor([float(p), float(q)], dtype=torch.float64))
    return torch.stack([s[0], 0.5 + s[1]]).float()


def gemm_f32(a, w, bias=None, xielu=None):
    """a [M,K] @ w [N,K].T (+ bias) in true 32-bit (CUDA cores, no reduced-precision mode); xielu =
    (act_params, act_cols) as in gemm_parts."""
    act_params, act_cols = xielu if xielu is not None else (None, 0)
    require_cuda(a, w, bias, act_params)
    if a.dim() != 2 or w.dim() != 2 or a.shape[1] != w.shape[1] or any(t is not None and t.dtype != torch.float32 for t in (a, w, bias, act_params)):
        raise RuntimeError("gemm_f32: fp32 a [M,K] and w [N,K] required")
    a, w = (t if t.stride(1) == 1 else t.contiguous() for t in (a, w))
    (M, K), N = a.shape, w.shape[0]
    out = torch.empty((M, N), dtype=torch.float32, device=a.device)
    check(lib().eb_gemm_f32(ptr(a), a.stride(0), 0, ptr(w), w.stride(0), 0, ptr(out), out.stride(0), 0, M, N, K, 1, None, None, ptr(bias),
                            int(act_cols), ptr(act_params), stream_ptr()), "gemm_f32")
    return out


def project(x, w, out_dtype=None, bias=None):
    """x @ w.T (+ bias) with a model's weight: the tensor-core GEMM, or the 32-bit one for models run in
    fp32."""
    return gemm_f32(x, w, bias=bias) if w.dtype == torch.float32 else gemm(x, w, bias=bias, out_dtype=out_dtype, static_weight=True)


def project_parts(x, w, bias=None, xielu=None, tail_col=None):
    """gemm_parts with a model's weight, or its 32-bit form."""
    if w.dtype != torch.float32:
        return gemm_parts(x, w, bias, xielu, tail_col, static_weight=True)
    out = gemm_f32(x, w, bias=bias, xielu=xielu)
    return out if tail_col is None else (out[:, :tail_col], out[:, tail_col:])


def project_unit(x, w, unit, out=None):
    """A feed-forward's first product with its unit in the epilogue: "gelu" of x @ w.T, or "geglu", w in blocks of
    8 gate rows and their 8 up rows -> half as many columns (out: rows that receive them, a row stride allowed)."""
    from .moe import UNITS, unit_act
    if out is not None and (out.dtype != x.dtype or out.stride(-1) != 1 or tuple(out.shape) != (x.shape[0], w.shape[0] // (1 if unit == "gelu" else 2))):
        raise RuntimeError("project_unit: the result has another shape")
    if w.dtype == torch.float32:
        return unit_act(gemm_f32(x, w), unit, out=out)
    if unit == "gelu":
        return gemm(x, w, act="gelu", static_weight=True, out=out)
    require_cuda(x, w)
    if x.dim() != 2 or x.stride(1) != 1 or not w.is_contiguous() or x.dtype != w.dtype or x.shape[1] != w.shape[1]:
        raise RuntimeError("project_unit: x [M,K] and contiguous w [N,K] of one dtype required")
    (M, K), N = x.shape, w.shape[0]
    out = torch.empty((M, N // 2), dtype=x.dtype, device=x.device) if out is None else out
    require_cuda(out)
    nbytes = lib().eb_gemm_workspace_bytes(M, N, K)
    ws = workspace(x.device, nbytes) if nbytes else None
    check(lib().eb_gemm_gated(ptr(x), x.stride(0), ptr(w), K, ptr(out), out.stride(0), M, N, K, UNITS[unit], 0.0, 0.0, dtype_code(x.dtype), 1, ptr(ws),
                              ws.numel() if ws is not None else 0, stream_ptr()), "gemm_gated")
    return out


LN_FOLD_MAX_ROWS = 32


def fold_layernorm(weight, bias, gamma, beta):
    """One-time preparation for gemm(..., ln_fold=...): y = LayerNorm(x; gamma, beta) @ weight.T + bias
    equals rstd * (x @ w_folded.T - mean * colsum) + bias32 with
      w_folded = weight * gamma (rounded to the weight dtype), colsum = w_folded.sum(1),
      bias32 = bias + weight @ beta   (fp32).
    Returns (w_folded, colsum, bias32)."""
    with torch.no_grad():
        w32 = weight.detach().float()
        w_folded = (w32 * gamma.detach().float()[None, :]).to(weight.dtype).contiguous()
        colsum = w_folded.float().sum(1).contiguous()
        bias32 = w32 @ beta.detach().float()
        if bias is not None:
            bias32 = bias32 + bias.detach().float()
        return w_folded, colsum, bias32.contiguous()


def device_status(clear=True):
    """(code, where, block, detail) of the current device's bounded-wait status word."""
    import ctypes
    buf = (ctypes.c_int * 4)()
    check(lib().eb_device_status(ctypes.cast(buf, ctypes.c_void_p), 1 if clear else 0), "device_status", launches=0)
    return tuple(buf)
