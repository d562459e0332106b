"""Python entry to the decaying-memory kernels: state-space (eb_short_conv, eb_ssm_*, eb_gate_group_norm) and gated
linear (eb_gla_*) layers, and the state space with a state per channel (eb_selective_*)."""
import torch

from ._lib import lib, check, dtype_code, ptr, stream_ptr, require_cuda


def _rows(t, what):
    if t.dim() != 2 or t.stride(1) != 1:
        raise RuntimeError(f"{what} must be [rows, columns] with contiguous rows")
    return t.stride(0)


def _state(S, heads, dk, dv):
    if S.dim() != 4 or tuple(S.shape[1:]) != (heads, dk, dv) or S.dtype != torch.float32 or not S.is_contiguous():
        raise RuntimeError("decaying memory: the state is fp32 [batch, heads, dk, dv]")
    return S.shape[0]


def _per_head(heads, *vectors):
    if any(v.dtype != torch.float32 or v.numel() != heads or not v.is_contiguous() for v in vectors):
        raise RuntimeError("state space: one fp32 number per head")


KEY_HEADS = (64, 128)            # key head sizes of the chunked tensor-core kernels
PAIRED_VALUE_HEAD = 64           # two value heads of this size share a CTA there


def chunk_heads(dim, vdim, dtype):
    """Padded (key, value) head sizes of the chunked kernels, or None where they do not serve."""
    if dtype != torch.bfloat16 or dim > KEY_HEADS[-1]:
        return None
    return min(n for n in KEY_HEADS if n >= dim), -(-vdim // 8) * 8


def short_conv(x, w, b, ring, batch, first=None):
    """Causal convolution per channel and SiLU of a prompt: x [batch*seq, C] (row stride allowed), w [taps, C], b [C];
    the last inputs go to ring [batch, rows, C].  Returns [batch*seq, C]."""
    require_cuda(x, w, b, ring, first)
    ldx, (n, C) = _rows(x, "short_conv: x"), x.shape
    if w.shape[1] != C or b.numel() != C or not w.is_contiguous() or any(t.dtype != x.dtype for t in (w, b, ring)) or n % batch:
        raise RuntimeError("short_conv: w [taps, C], b [C] of one dtype, whole sequences")
    if ring.dim() != 3 or ring.shape[0] != batch or ring.shape[2] != C or ring.stride(2) != 1:
        raise RuntimeError("short_conv: the ring is [batch, rows, C]")
    out = torch.empty((n, C), dtype=x.dtype, device=x.device)
    check(lib().eb_short_conv(ptr(x), ldx, ptr(w), ptr(b), ptr(out), C, batch, n // batch, C, w.shape[0], ptr(first), ptr(ring), ring.stride(0),
                              ring.stride(1), ring.shape[1], dtype_code(x.dtype), stream_ptr()), "short_conv")
    return out


def ssm_prompt(xbc, dt, dt_bias, a_log, skip, S, heads, groups, dk, dv, first=None, chunked=False):
    """A prompt through the state-space recurrence, token by token on the CUDA cores or (chunked: bf16, dk of KEY_HEADS)
    128 tokens at a time on the tensor cores; xbc [batch*seq, heads*dv + 2*groups*dk] behind the convolution, dt
    fp32 [batch*seq, >= heads].  S is overwritten with the state behind the last token.  Returns [batch*seq, heads*dv]."""
    require_cuda(xbc, dt, dt_bias, a_log, skip, S, first)
    B, n = _state(S, heads, dk, dv), xbc.shape[0]
    _per_head(heads, dt_bias, a_log, skip)
    if xbc.shape[1] != heads * dv + 2 * groups * dk or dt.dtype != torch.float32 or dt.shape[0] != n or dt.shape[1] < heads or n % B:
        raise RuntimeError("state space: rows [x | B | C], dt fp32, whole sequences")
    y = torch.empty((n, heads * dv), dtype=xbc.dtype, device=xbc.device)
    run, name = (lib().eb_ssm_chunks, "ssm_chunks") if chunked else (lib().eb_ssm_scan, "ssm_scan")
    check(run(ptr(xbc), _rows(xbc, "xbc"), ptr(dt), _rows(dt, "dt"), ptr(dt_bias), ptr(a_log), ptr(skip), ptr(first), ptr(y), heads * dv, ptr(S), B, n // B,
              heads, groups, dk, dv, dtype_code(xbc.dtype), stream_ptr()), name)
    return y


def ssm_step(xbc, conv_w, conv_b, ring, pos_device, dt, dt_bias, a_log, skip, S, heads, groups, dk, dv, first=None):
    """One token per sequence, xbc [batch, ...] in front of the convolution; the ring and S go on.  Returns [batch, heads*dv]."""
    require_cuda(xbc, conv_w, conv_b, ring, pos_device, dt, dt_bias, a_log, skip, S, first)
    B = _state(S, heads, dk, dv)
    _per_head(heads, dt_bias, a_log, skip)
    C = heads * dv + 2 * groups * dk
    if tuple(xbc.shape) != (B, C) or dt.dtype != torch.float32 or dt.shape[0] != B or conv_w.shape[1] != C or not conv_w.is_contiguous() or any(
            t.dtype != xbc.dtype for t in (conv_w, conv_b, ring)) or tuple(ring.shape[::2]) != (B, C) or ring.stride(2) != 1:
        raise RuntimeError("state space: one row [x | B | C] per sequence, convolution and ring of its dtype")
    y = torch.empty((B, heads * dv), dtype=xbc.dtype, device=xbc.device)
    check(lib().eb_ssm_step(ptr(xbc), _rows(xbc, "xbc"), ptr(conv_w), ptr(conv_b), conv_w.shape[0], ptr(ring), ring.stride(0), ring.stride(1),
                            ring.shape[1], ptr(pos_device), ptr(first), ptr(dt), _rows(dt, "dt"), ptr(dt_bias), ptr(a_log), ptr(skip), ptr(y),
                            heads * dv, ptr(S), B, heads, groups, dk, dv, dtype_code(xbc.dtype), stream_ptr()), "ssm_step")
    return y


def gate_group_norm(y, z, norm, eps, heads, dv, parts):
    """unit(y * silu(z)) * norm, unit over `parts` equal parts of the heads * dv real columns of y [rows, heads*padded]."""
    require_cuda(y, z, norm)
    rows, width = y.shape
    if z.shape != y.shape or any(t.dtype != y.dtype for t in (z, norm)) or norm.numel() != width or width % heads:
        raise RuntimeError("gate_group_norm: y and z are [rows, heads*dv] of one dtype, the norm has one entry per column")
    pad = width // heads
    out = (torch.empty if pad == dv else torch.zeros)((rows, width), dtype=y.dtype, device=y.device)
    check(lib().eb_gate_group_norm(ptr(y), _rows(y, "y"), ptr(z), _rows(z, "z"), ptr(norm), float(eps), ptr(out), width, rows, heads, int(dv), pad,
                                   int(parts), dtype_code(y.dtype), stream_ptr()), "gate_group_norm")
    return out


def _qkv(q, k, v, heads, S):
    dk, dv = q.shape[1] // heads, v.shape[1] // heads
    if any(t.dim() != 2 or t.stride(1) != 1 or t.stride(0) != q.stride(0) or t.dtype != q.dtype for t in (q, k, v)):
        raise RuntimeError("gated linear: q, k and v are column ranges of one row layout")
    if q.shape[1] != heads * dk or k.shape[1] != heads * dk or v.shape[1] != heads * dv:
        raise RuntimeError("gated linear: q, k and v hold whole heads")
    return _state(S, heads, dk, dv), dk, dv


def gla_prompt(q, k, v, z, tau, scale, S, heads, first=None, chunked=False):
    """A prompt through the gated linear recurrence: q, k [batch*seq, heads*dk], v [batch*seq, heads*dv] (column views of one
    projection), z fp32 [batch*seq, heads*dk]; chunked as in ssm_prompt.  S is overwritten.  Returns [batch*seq,
    heads*dv]."""
    require_cuda(q, k, v, z, S, first)
    B, dk, dv = _qkv(q, k, v, heads, S)
    n = q.shape[0]
    if z.dtype != torch.float32 or tuple(z.shape) != (n, heads * dk) or n % B:
        raise RuntimeError("gated linear: z is fp32 [rows, heads*dk], whole sequences")
    o = torch.empty((n, heads * dv), dtype=q.dtype, device=q.device)
    if chunked:
        nbytes = lib().eb_gla_chunks_workspace_bytes(B, n // B, heads, dk)
        ws = torch.empty(nbytes, dtype=torch.uint8, device=q.device)
        check(lib().eb_gla_chunks(ptr(q), ptr(k), ptr(v), q.stride(0), ptr(z), _rows(z, "z"), float(tau), float(scale), ptr(first), ptr(o), heads * dv, ptr(S),
                                  B, n // B, heads, dk, dv, dtype_code(q.dtype), ptr(ws), nbytes, stream_ptr()), "gla_chunks", launches=2)
        return o
    check(lib().eb_gla_scan(ptr(q), ptr(k), ptr(v), q.stride(0), ptr(z), _rows(z, "z"), float(tau), float(scale), ptr(first), ptr(o), heads * dv, ptr(S),
                            B, n // B, heads, dk, dv, dtype_code(q.dtype), stream_ptr()), "gla_scan")
    return o


def gla_step(q, k, v, g, low, w2, b2, tau, scale, norm, dv_count, eps, S, heads):
    """One token per sequence: z = w2 low + b2, S goes on; returns unit(o_h) * norm * silu(g), [batch, heads*dv]."""
    require_cuda(q, k, v, g, low, w2, b2, norm, S)
    B, dk, dv = _qkv(q, k, v, heads, S)
    rank = w2.shape[1]
    if q.shape[0] != B or g.shape != v.shape or any(t.stride(0) != q.stride(0) or t.dtype != q.dtype for t in (g, low)) or low.shape[1] != rank:
        raise RuntimeError("gated linear: one row per sequence, gate and low-rank part in the same row layout")
    if not w2.is_contiguous() or w2.shape[0] != heads * dk or b2.numel() != heads * dk or norm.numel() != heads * dv or any(
            t.dtype != q.dtype for t in (w2, b2, norm)):
        raise RuntimeError("gated linear: w2 [heads*dk, rank], b2 [heads*dk], norm [heads*dv] of the operand dtype")
    out = torch.empty((B, heads * dv), dtype=q.dtype, device=q.device)
    check(lib().eb_gla_step(ptr(q), ptr(k), ptr(v), ptr(g), ptr(low), q.stride(0), ptr(w2), ptr(b2), rank, float(tau), float(scale), ptr(norm),
                            int(dv_count), float(eps), ptr(out), heads * dv, ptr(S), B, heads, dk, dv, dtype_code(q.dtype), stream_ptr()), "gla_step")
    return out


def short_conv_step(x, w, b, ring, pos_device, first=None):
    """short_conv of one token per sequence, x [batch, C]: earlier inputs from the ring, this one into it."""
    require_cuda(x, w, b, ring, pos_device, first)
    ldx, (n, C) = _rows(x, "short_conv_step: x"), x.shape
    if w.shape[1] != C or b.numel() != C or not w.is_contiguous() or any(t.dtype != x.dtype for t in (w, b, ring)):
        raise RuntimeError("short_conv_step: w [taps, C], b [C] of one dtype")
    if ring.dim() != 3 or ring.shape[0] != n or ring.shape[2] != C or ring.stride(2) != 1:
        raise RuntimeError("short_conv_step: the ring is [batch, rows, C]")
    out = torch.empty((n, C), dtype=x.dtype, device=x.device)
    check(lib().eb_short_conv_step(ptr(x), ldx, ptr(w), ptr(b), ptr(out), C, n, C, w.shape[0], ptr(pos_device), ptr(first), ptr(ring), ring.stride(0),
                                   ring.stride(1), ring.shape[1], dtype_code(x.dtype), stream_ptr()), "short_conv_step")
    return out


def _selective(x, gate, bc, bias, a_log, skip, S, out):
    inner, states = a_log.shape
    if any(t.dtype != torch.float32 or not t.is_contiguous() for t in (bias, a_log, skip, S)) or bias.numel() != inner or skip.numel() != inner or tuple(S.shape[1:]) != (inner, states):
        raise RuntimeError("selective scan: bias, skip [inner], a_log [inner, states] and the state [batch, inner, states] are fp32")
    if x.shape[1] != inner or gate.shape != x.shape or gate.dtype != x.dtype or bc.dtype != torch.float32 or bc.shape[0] != x.shape[0] or bc.shape[1] < 2 * states:
        raise RuntimeError("selective scan: rows x and gate [rows, inner], bc fp32 [rows, 2 * states]")
    out = torch.empty((x.shape[0], inner), dtype=x.dtype, device=x.device) if out is None else out
    if out.shape != x.shape or out.dtype != x.dtype:
        raise RuntimeError("selective scan: the output is laid out like x")
    return inner, states, out, (ptr(x), _rows(x, "x"), ptr(gate), _rows(gate, "gate"))


def selective_scan(x, gate, z, bc, bias, a_log, skip, S, first=None, out=None):
    """A prompt through the recurrence with a state per channel: x [batch*seq, inner] behind the convolution, gate alike, z fp32
    [batch*seq, inner] (projected steps without their bias), bc fp32 [batch*seq, >= 2 * states] (B | C).  S [batch, inner,
    states] is overwritten with the state behind the last token.  Returns (S^T C + skip x) * silu(gate)."""
    require_cuda(x, gate, z, bc, bias, a_log, skip, S, first, out)
    inner, states, out, rows = _selective(x, gate, bc, bias, a_log, skip, S, out)
    B = S.shape[0]
    if z.dtype != torch.float32 or tuple(z.shape) != tuple(x.shape) or x.shape[0] % B:
        raise RuntimeError("selective scan: z is fp32 [rows, inner], whole sequences")
    check(lib().eb_selective_scan(*rows, ptr(z), _rows(z, "z"), ptr(bc), _rows(bc, "bc"), ptr(bias), ptr(a_log), ptr(skip), ptr(first), ptr(out),
                                  _rows(out, "out"), ptr(S), B, x.shape[0] // B, inner, states, dtype_code(x.dtype), stream_ptr()), "selective_scan")
    return out


def selective_step(x, gate, low, w, bc, bias, a_log, skip, S, out=None):
    """One token per sequence: z = low @ w.T (low [batch, rank], w [inner, rank]); S goes on.  Returns as selective_scan."""
    require_cuda(x, gate, low, w, bc, bias, a_log, skip, S, out)
    inner, states, out, rows = _selective(x, gate, bc, bias, a_log, skip, S, out)
    if x.shape[0] != S.shape[0] or not w.is_contiguous() or w.shape[0] != inner or low.shape != (x.shape[0], w.shape[1]) or any(t.dtype != x.dtype for t in (low, w)):
        raise RuntimeError("selective scan: low [batch, rank] and w [inner, rank] of the rows' dtype")
    check(lib().eb_selective_step(*rows, ptr(low), _rows(low, "low"), ptr(w), w.shape[1], ptr(bc), _rows(bc, "bc"), ptr(bias), ptr(a_log), ptr(skip),
                                  ptr(out), _rows(out, "out"), ptr(S), x.shape[0], inner, states, dtype_code(x.dtype), stream_ptr()), "selective_step")
    return out
