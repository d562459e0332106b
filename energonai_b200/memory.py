"""Python entry to the matrix-memory kernels (eb_memory_*, eb_head_norm_gate)."""
import torch

from ._lib import lib, check, dtype_code, ptr, stream_ptr, require_cuda


def _row_views(q, k, v, heads, state):
    S, n, m = state
    if any(t.dim() != 2 or t.stride(1) != 1 or t.stride(0) != q.stride(0) or t.dtype != q.dtype for t in (q, k, v)):
        raise RuntimeError("matrix memory: q, k and v are column ranges of one row layout")
    dk, dv = q.shape[1] // heads, v.shape[1] // heads
    B = S.shape[0]
    if q.shape[1] != heads * dk or k.shape[1] != heads * dk or v.shape[1] != heads * dv:
        raise RuntimeError("matrix memory: q, k and v hold whole heads")
    if tuple(S.shape) != (B, heads, dk, dv) or tuple(n.shape) != (B, heads, dk) or tuple(m.shape) != (B, heads) or any(
            t.dtype != torch.float32 or not t.is_contiguous() for t in (S, n, m)):
        raise RuntimeError("matrix memory: the state is fp32 S [batch, heads, dk, dv], n [batch, heads, dk], m [batch, heads]")
    return B, dk, dv


def _gates(gates, bias, heads, rows):
    if gates.dtype != torch.float32 or gates.dim() != 2 or gates.stride(1) != 1 or gates.shape[0] != rows or gates.shape[1] < 2 * heads:
        raise RuntimeError("matrix memory: gates are fp32 [rows, >= 2*heads]")
    if any(b.dtype != torch.float32 or b.numel() != heads or not b.is_contiguous() for b in bias):
        raise RuntimeError("matrix memory: one fp32 bias per head and gate")


MEMORY_KEY_HEADS = (64, 128)      # key head sizes of the chunked tensor-core kernel


def memory_prompt(q, k, v, gates, bias, cap, scale, state, heads, first=None, chunked=False):
    """A prompt through the recurrence, token by token on the CUDA cores, or (chunked: bf16, key heads
    of MEMORY_KEY_HEADS) 128 tokens at a time on the tensor cores: q, k [batch*seq, heads*dk], v [batch*seq,
    heads*dv] (column views of one projection), gates fp32 [batch*seq, >= 2*heads] (input gates, forget
    gates), bias (input, forget) fp32 [heads].  state = (S, n, m) is overwritten with the state behind
    the last token; first [batch] int32: padding rows in front.  Returns [batch*seq, heads*dv]."""
    require_cuda(q, k, v, gates, *state, *bias, first)
    B, dk, dv = _row_views(q, k, v, heads, state)
    T = q.shape[0]
    _gates(gates, bias, heads, T)
    if T % B:
        raise RuntimeError("matrix memory: whole sequences required")
    o = torch.empty((T, heads * dv), dtype=q.dtype, device=q.device)
    run, name = (lib().eb_memory_chunks, "memory_chunks") if chunked else (lib().eb_memory_scan, "memory_scan")
    check(run(ptr(q), ptr(k), ptr(v), q.stride(0), ptr(gates), gates.stride(0), ptr(bias[0]), ptr(bias[1]), float(cap), float(scale),
              ptr(first), ptr(o), o.stride(0), *(ptr(t) for t in state), B, T // B, heads, dk, dv, dtype_code(q.dtype), stream_ptr()), name)
    return o


def memory_step(q, k, v, g, gates, bias, cap, scale, norm, dv_count, eps, state, heads):
    """One token per sequence: the state goes on; returns unit(o_h) * norm * sigmoid(g), [batch, heads*dv]."""
    require_cuda(q, k, v, g, gates, norm, *state, *bias)
    B, dk, dv = _row_views(q, k, v, heads, state)
    _gates(gates, bias, heads, B)
    if q.shape[0] != B or g.shape != v.shape or g.stride() != v.stride() or g.dtype != v.dtype or norm.dtype != v.dtype or norm.numel() != heads * dv:
        raise RuntimeError("matrix memory: one row per sequence; the gate is laid out like v, the norm has one entry per value column")
    out = torch.empty((B, heads * dv), dtype=q.dtype, device=q.device)
    check(lib().eb_memory_step(ptr(q), ptr(k), ptr(v), ptr(g), q.stride(0), ptr(gates), gates.stride(0), ptr(bias[0]), ptr(bias[1]), float(cap),
                               float(scale), ptr(norm), int(dv_count), float(eps), ptr(out), out.stride(0), *(ptr(t) for t in state), B, heads,
                               dk, dv, dtype_code(q.dtype), stream_ptr()), "memory_step")
    return out


def head_norm_gate(o, g, norm, heads, dv_count, eps, silu=False):
    """unit(o_h) * norm * sigmoid(g), or silu(g) instead, for rows o [rows, heads*dv]; unit over the first dv_count of a head."""
    require_cuda(o, g, norm)
    rows, width = o.shape
    if g.shape != o.shape or g.dtype != o.dtype or norm.dtype != o.dtype or norm.numel() != width or o.stride(1) != 1 or g.stride(1) != 1 or width % heads:
        raise RuntimeError("head_norm_gate: o and g are [rows, heads*dv] of one dtype, the norm has one entry per column")
    out = torch.empty((rows, width), dtype=o.dtype, device=o.device)
    check(lib().eb_head_norm_gate_act(ptr(o), o.stride(0), ptr(g), g.stride(0), ptr(norm), float(eps), ptr(out), width, rows, heads, width // heads,
                                  int(dv_count), 1 if silu else 0, dtype_code(o.dtype), stream_ptr()), "head_norm_gate")
    return out
