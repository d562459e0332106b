"""Python entry to the RMS-norm kernels (eb_rms_norm / eb_rms_residual / eb_stream_update / eb_stream_add /
eb_stream_conv)."""
import torch

from ._lib import lib, check, dtype_code, ptr, stream_ptr, require_cuda


def _rows(t, what):
    if t.dim() != 2 or t.stride(1) != 1:
        raise RuntimeError(f"{what} must be [rows, width] with contiguous rows")
    return t.stride(0)


def rms_norm(x, weight, eps, offset=0.0, count=None, out=None, write_out=True, ring=None, rows_per_batch=1, pos_device=None):
    """y = x / sqrt(mean(x^2) + eps) * (offset + weight) over the rows of x [n1, n2] (fp32 or the
    weight's dtype); the mean is over the first `count` columns (the others are zero padding).
    ring [batch, rows, >= n2]: the rows are also written to a ring cache, row (b, s) at
    (position of the first row + s) mod rows, that position from pos_device (int32 scalar; None: 0).
    Returns y in the weight's dtype (None with write_out=False)."""
    require_cuda(x, weight, out, ring, pos_device)
    ldx = _rows(x, "rms_norm: x")
    n1, n2 = x.shape
    if weight.numel() != n2:
        raise RuntimeError("rms_norm: the weight must have one entry per column")
    if out is None and write_out:
        out = torch.empty((n1, n2), dtype=weight.dtype, device=x.device)
    if ring is not None and (ring.dim() != 3 or ring.stride(2) != 1 or ring.dtype != weight.dtype or ring.shape[0] * rows_per_batch != n1
                             or ring.shape[2] < n2):
        raise RuntimeError("rms_norm: the ring must be [batch, rows, width] of the weight's dtype")
    check(lib().eb_rms_norm(ptr(x), ldx, dtype_code(x.dtype), ptr(weight), float(offset), float(eps), ptr(out),
                            _rows(out, "rms_norm: out") if out is not None else 0, dtype_code(weight.dtype), n1, n2, count or n2,
                            ptr(ring), ring.stride(0) if ring is not None else 0, ring.stride(1) if ring is not None else 0,
                            ring.shape[1] if ring is not None else 0, rows_per_batch, ptr(pos_device), stream_ptr()), "rms_norm")
    return out


def rms_residual(y, weight, eps, x, xt=None, offset=0.0, count=None, mix=None, router=None):
    """x += rms_norm(y) in place, x [n1, n2] fp32; xt (the weight's dtype) receives the new rows.
    mix = (idx, rows, weights) of a mixture of experts (idx / weights [n1, top], rows or None): the
    row of y is then the weighted sum of the token's expert rows.  router = (weight [experts, n2],
    experts, top): also returns (idx, weights) of the mixture that follows."""
    require_cuda(y, weight, x, xt)
    n1, n2 = x.shape
    if x.dtype != torch.float32 or y.dtype != weight.dtype or y.shape[1] != n2 or weight.numel() != n2:
        raise RuntimeError("rms_residual: x is fp32, y and the weight share a dtype, all of one width")
    if mix is None and y.shape[0] != n1:
        raise RuntimeError("rms_residual: one row of y per row of x")
    idx, rows, mw = mix if mix is not None else (None, None, None)
    r_idx = r_w = None
    if router is not None:
        rw, experts, top = router
        if rw.shape[1] != n2 or not rw.is_contiguous() or rw.dtype != weight.dtype or rw.shape[0] < experts:
            raise RuntimeError("rms_residual: the router weight must be contiguous [experts, width]")
        r_idx = torch.empty((n1, top), dtype=torch.int32, device=x.device)
        r_w = torch.empty((n1, top), dtype=torch.float32, device=x.device)
    check(lib().eb_rms_residual(ptr(y), _rows(y, "rms_residual: y"), dtype_code(y.dtype), ptr(idx), ptr(rows), ptr(mw),
                                idx.shape[1] if idx is not None else 0, ptr(weight), float(offset), float(eps), ptr(x),
                                _rows(x, "rms_residual: x"), ptr(xt), _rows(xt, "rms_residual: xt") if xt is not None else 0, n1, n2,
                                count or n2, ptr(router[0]) if router else None, router[1] if router else 0, router[2] if router else 0,
                                ptr(r_idx), ptr(r_w), stream_ptr()), "rms_residual")
    return (r_idx, r_w) if router is not None else None


def stream_update(x, eps, count=None, src=None, src_scale=1.0, y=None, gate=None, w_out=None, w_next=None):
    """The residual step of blocks that normalise in front of and behind a sublayer; x [n1, n2] fp32 in
    place:  x = src_scale * src (if src is given);  x += norm(y * sigmoid(gate)) * w_out (if y is; w_out
    fp32);  returns h = norm(x) * w_next (None without w_next)."""
    require_cuda(x, src, y, gate, w_out, w_next)
    n1, n2 = x.shape
    t = next((a for a in (src, y, w_next) if a is not None), None)
    if t is None or x.dtype != torch.float32 or any(a is not None and a.dtype != t.dtype for a in (src, y, gate, w_next)):
        raise RuntimeError("stream_update: x is fp32, the other rows and weights share a dtype")
    if any(a is not None and tuple(a.shape) != (n1, n2) for a in (src, y, gate)) or any(a is not None and a.shape[-1] != n2 for a in (w_out, w_next)):
        raise RuntimeError("stream_update: everything is [rows, width] of one width")
    if w_out is not None and w_out.dtype != torch.float32:
        raise RuntimeError("stream_update: w_out is fp32")
    h = torch.empty((n1, n2), dtype=t.dtype, device=x.device) if w_next is not None else None
    ld = lambda a, what: _rows(a, f"stream_update: {what}") if a is not None else 0
    check(lib().eb_stream_update(ptr(src), ld(src, "src"), float(src_scale), ptr(y), ld(y, "y"), ptr(gate), ld(gate, "gate"), ptr(w_out), ptr(x),
                                 ld(x, "x"), ptr(w_next), ptr(h), n2, float(eps), n1, n2, count or n2, dtype_code(t.dtype), stream_ptr()),
          "stream_update")
    return h


def stream_add(x, eps, count=None, src=None, src2=None, y=None, w=None, y2=None, w2=None, mix=None, ident=None, experts=0, shared=None, gate=None,
               scale=1.0, w_next=None, next_scale=1.0, router=None):
    """The residual step of blocks with a norm in front of every sublayer only; x [n1, n2] fp32 in place:
      x = src + src2 (if src is given);  x += scale * Y;  returns h = norm(x) * w_next * next_scale (None
      without w_next).
    Y is y; with y2, norm(y) * w + norm(y2) * w2 (w, w2 fp32); with mix = (idx, rows or None, weights), the
    weighted sum of a token's expert rows y, of ident for choices from `experts` on, and gate * shared.
    router = (weight, RouterRule, top, gated): returns (h, (idx, weights, shared gate or None)) of the
    mixture that follows."""
    require_cuda(x, src, src2, y, w, y2, w2, ident, shared, gate, w_next)
    n1, n2 = x.shape
    t = next((a for a in (src, y, w_next) if a is not None), None)
    if t is None or x.dtype != torch.float32 or any(a is not None and a.dtype != t.dtype for a in (src, src2, y, y2, ident, shared, w_next)):
        raise RuntimeError("stream_add: x is fp32, the other rows share a dtype")
    if any(a is not None and tuple(a.shape) != (n1, n2) for a in (src, src2, y if mix is None else None, y2, ident, shared)) or any(
            a is not None and a.shape[-1] != n2 for a in (y, w, w2, w_next)):
        raise RuntimeError("stream_add: everything is [rows, width] of one width")
    if any(a is not None and a.dtype != torch.float32 for a in (w, w2, gate)):
        raise RuntimeError("stream_add: w, w2 and gate are fp32")
    idx, rows, weights = mix if mix is not None else (None, None, None)
    h = torch.empty((n1, n2), dtype=t.dtype, device=x.device) if w_next is not None else None
    ld = lambda a, what: _rows(a, f"stream_add: {what}") if a is not None else 0
    rw = r_idx = r_w = r_gate = rule = None
    top = 0
    if router is not None:
        rw, rule, top, gated = router
        if rw.dtype != t.dtype or not rw.is_contiguous() or rw.shape[1] != n2 or rw.shape[0] < rule.choices + int(gated):
            raise RuntimeError("stream_add: the router weight must be contiguous [choices, width]")
        r_idx = torch.empty((n1, top), dtype=torch.int32, device=x.device)
        r_w = torch.empty((n1, top), dtype=torch.float32, device=x.device)
        r_gate = torch.empty(n1, dtype=torch.float32, device=x.device) if gated else None
    check(lib().eb_stream_add(ptr(src), ld(src, "src"), ptr(src2), ld(src2, "src2"), ptr(y), ld(y, "y"), ptr(w), ptr(y2), ld(y2, "y2"), ptr(w2),
                              ptr(idx), ptr(rows), ptr(weights), idx.shape[1] if idx is not None else 0, int(experts), ptr(ident), ld(ident, "ident"),
                              ptr(shared), ld(shared, "shared"), ptr(gate), float(scale), ptr(x), ld(x, "x"), ptr(w_next), float(next_scale), ptr(h), n2,
                              float(eps), n1, n2, count or n2, ptr(rw), rule.choices if rule else 0, rule.experts if rule else 0, top,
                              ptr(rule.correction) if rule else None, rule.groups if rule else 1, rule.keep if rule else 1, ptr(r_idx), ptr(r_w),
                              ptr(r_gate), dtype_code(t.dtype), stream_ptr()), "stream_add")
    return (h, (r_idx, r_w, r_gate)) if router is not None else h


CONV_TAPS = (2, 3, 4, 8, 16)          # sizes of the tap tables stream_conv takes (pad in front with zero rows)


def stream_conv(x, k1, ring, eps, batch, count=None, src=None, y=None, k2=None, first=None, pos_device=None):
    """The residual step of blocks whose two sublayers read the same stream through a norm and a short causal convolution of
    the normed rows over time; x [rows, n2] fp32 (not read if src, the embedding rows, is given):
      x' = (src or x) + y;  u = x' over its root mean square;  h1_t = sum_j k1[j] u_(t - taps + 1 + j);  h2 with k2
    k1, k2 fp32 [taps, n2] (k2 None: one sublayer).  The last rows u go to ring [batch, rows, n2].  pos_device (int32
    scalar): a step, one row per sequence, earlier rows from the ring.  Returns (x', h1, h2 or None)."""
    require_cuda(x, src, y, k1, k2, ring, first, pos_device)
    t, like = src if src is not None else y, x if x is not None else src
    n1, n2 = like.shape
    taps = k1.shape[0]
    if t is None or ring.dtype != t.dtype or any(a is not None and (a.dtype != t.dtype or tuple(a.shape) != (n1, n2)) for a in (src, y)) or (
            x is not None and (x.dtype != torch.float32 or tuple(x.shape) != (n1, n2))):
        raise RuntimeError("stream_conv: rows [rows, width]; x is fp32, the others and the ring share a dtype")
    if any(k is not None and (k.dtype != torch.float32 or not k.is_contiguous() or tuple(k.shape) != (taps, n2)) for k in (k1, k2)):
        raise RuntimeError("stream_conv: tap tables are contiguous fp32 [taps, width]")
    if n1 % batch or ring.dim() != 3 or ring.shape[0] != batch or ring.shape[2] != n2 or ring.stride(2) != 1 or (pos_device is not None and n1 != batch):
        raise RuntimeError("stream_conv: the ring is [batch, rows, width]; a step has one row per sequence")
    x_out = torch.empty((n1, n2), dtype=torch.float32, device=t.device)
    h1 = torch.empty((n1, n2), dtype=t.dtype, device=t.device)
    h2 = torch.empty_like(h1) if k2 is not None else None
    ld = lambda a, what: _rows(a, f"stream_conv: {what}") if a is not None else n2
    check(lib().eb_stream_conv(ptr(src), ld(src, "src"), ptr(x) if src is None else None, n2, ptr(y), ld(y, "y"), ptr(x_out), ptr(k1), ptr(k2), taps,
                               ptr(h1), ptr(h2), n2, ptr(ring), ring.stride(0), ring.stride(1), ring.shape[1], batch, n1 // batch, n2, count or n2,
                               float(eps), ptr(first), ptr(pos_device), dtype_code(t.dtype), stream_ptr()), "stream_conv")
    return x_out, h1, h2
