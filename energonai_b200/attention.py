"""Python entry to the fused attention kernels (eb_attention_prefill[_tc] / eb_attention_decode)."""
import os

import torch

from ._lib import lib, check, dtype_code, ptr, stream_ptr, require_cuda

_scratch, _outgrown = {}, []
TC_MIN_ROWS = 128        # below this many query rows the 256-row CTAs of the tensor-core kernel are mostly padding


def _get_scratch(device, nbytes):
    key = torch.device(device).index
    buf = _scratch.get(key)
    if buf is None or buf.numel() < nbytes:
        if buf is not None:
            _outgrown.append(buf)            # captured steps may still hold its address
        buf = torch.zeros(max(nbytes, 1 << 20), dtype=torch.uint8, device=device)
        _scratch[key] = buf
    return buf


def _bsh_strides(t, head_dim):
    """(batch_stride, row_stride) of a [B, S, H*D] view whose last dim is contiguous."""
    if t.dim() != 3 or t.stride(2) != 1 or t.shape[2] % head_dim:
        raise RuntimeError("attention: tensors must be [batch, seq, heads*head_dim] views with a contiguous last dim")
    return t.stride(0), t.stride(1)


def attention_prefill(q, k, v, head_dim, mask=None, causal=True, scale=None, out=None, impl=None):
    """q [B,Sq,H*D], k/v [B,Sk,H*D] (strided views allowed), mask [B,Sk] additive or None.
    Returns out [B,Sq,H*D].  impl: "tc" (tcgen05 kernel), "mma" (mma.sync kernel) or None =
    "tc" for prompts of at least TC_MIN_ROWS rows (EB_ATTN_TC=0 keeps "mma")."""
    require_cuda(q, k, v, mask, out)
    B, Sq, HD = q.shape
    Sk = k.shape[1]
    H = HD // head_dim
    if out is None:
        out = torch.empty((B, Sq, HD), dtype=q.dtype, device=q.device)
    if mask is not None:
        if mask.dtype != q.dtype or mask.stride(-1) != 1 or mask.dim() != 2 or mask.shape[1] < Sk:
            raise RuntimeError("attention: mask must be [batch, kv_len] of the tensor dtype")
    qs, ks, vs, os_ = (_bsh_strides(t, head_dim) for t in (q, k, v, out))
    scale = head_dim ** -0.5 if scale is None else scale
    if impl is None:
        impl = "tc" if Sq >= TC_MIN_ROWS and os.environ.get("EB_ATTN_TC", "1") != "0" else "mma"
    if impl == "tc":
        check(lib().eb_attention_prefill_tc(ptr(q), ptr(k), ptr(v), ptr(out), ptr(mask), qs[0], qs[1], ks[0], ks[1], vs[0],
                                            vs[1], os_[0], os_[1], mask.stride(0) if mask is not None else 0, B, H, Sq, Sk,
                                            head_dim, 1 if causal else 0, float(scale), dtype_code(q.dtype), stream_ptr()),
              "attention_prefill_tc")
        return out
    check(lib().eb_attention_prefill(ptr(q), ptr(k), ptr(v), ptr(out), ptr(mask), qs[0], qs[1], ks[0], ks[1], vs[0], vs[1],
                                     os_[0], os_[1], mask.stride(0) if mask is not None else 0, B, H, Sq, Sk, head_dim,
                                     1 if causal else 0, float(scale), dtype_code(q.dtype), stream_ptr()),
          "attention_prefill")
    return out


def pick_nsplit(batch, heads, kv_len, sm_count=148):
    """Key splits per (sequence, head).  Splitting costs a merge and shortens every CTA's stream,
    and was measured to lose whenever a CTA would be left with fewer than about a thousand keys:
    at 576 keys and batch 16, 1 / 2 / 3 / 6 splits take 30.9 / 34.7 / 36.2 / 41.3 us per layer with
    40 heads and 7.9 / 9.1 / 9.7 / 10.0 us with the 5 heads of an 8-way shard (80 CTAs on 148 SMs:
    even an underfilled machine prefers whole streams).  So: one split per 1024 keys, never more
    than gives every SM its three resident CTAs, never more than one per 64-key tile."""
    tiles = max(1, (kv_len + 63) // 64)
    want = -(-3 * sm_count // max(1, batch * heads))
    return max(1, min(want, kv_len // 1024, tiles, 64))


def attention_decode(q, k, v, head_dim, kv_len, mask=None, scale=None, out=None, nsplit=None, kv_len_device=None,
                     q_in_cache=False):
    """q [B, H*D] (one row per sequence), k/v [B, >=kv_len, H*D] cache views, mask [B, >=kv_len].
    With q_in_cache, q is a [B, capacity, H*D] view like k/v and the query is its row kv_len-1.
    Returns out [B, H*D]."""
    require_cuda(q, k, v, mask, out, kv_len_device)
    q_rs = 0
    if q_in_cache:
        q_rs = q.stride(1)
        q = q[:, 0]
    B, HD = q.shape
    H = HD // head_dim
    if q.stride(1) != 1:
        raise RuntimeError("attention_decode: q rows must be contiguous")
    if out is None:
        out = torch.empty((B, HD), dtype=q.dtype, device=q.device)
    ks, vs = _bsh_strides(k, head_dim), _bsh_strides(v, head_dim)
    if mask is not None and (mask.dtype != q.dtype or mask.stride(-1) != 1 or mask.dim() != 2):
        raise RuntimeError("attention: mask must be [batch, kv_len] of the tensor dtype")
    if nsplit is None:
        nsplit = pick_nsplit(B, H, kv_len)
    nbytes = lib().eb_attention_decode_scratch_bytes(B, H, head_dim, nsplit)
    scratch = _get_scratch(q.device, nbytes) if nbytes else None
    scale = head_dim ** -0.5 if scale is None else scale
    check(lib().eb_attention_decode(ptr(q), ptr(k), ptr(v), ptr(out), ptr(mask), q.stride(0), q_rs, ks[0], ks[1], vs[0], vs[1],
                                    out.stride(0), mask.stride(0) if mask is not None else 0, B, H, int(kv_len),
                                    ptr(kv_len_device), head_dim, float(scale), dtype_code(q.dtype), nsplit, ptr(scratch),
                                    scratch.numel() if scratch is not None else 0, stream_ptr()), "attention_decode")
    return out


def attention_prefill_window(q, k, v, head_dim, window, mask=None, scale=None, out=None):
    """attention_prefill (causal, tensor-core kernel) in which row i sees the keys j with
    0 <= i - j < window (window 0: all up to i)."""
    require_cuda(q, k, v, mask, out)
    B, Sq, HD = q.shape
    Sk = k.shape[1]
    if out is None:
        out = torch.empty((B, Sq, HD), dtype=q.dtype, device=q.device)
    if mask is not None and (mask.dtype != q.dtype or mask.stride(-1) != 1 or mask.dim() != 2 or mask.shape[1] < Sk):
        raise RuntimeError("attention: mask must be [batch, kv_len] of the tensor dtype")
    qs, ks, vs, os_ = (_bsh_strides(t, head_dim) for t in (q, k, v, out))
    scale = head_dim ** -0.5 if scale is None else scale
    check(lib().eb_attention_prefill_window_tc(ptr(q), ptr(k), ptr(v), ptr(out), ptr(mask), qs[0], qs[1], ks[0], ks[1], vs[0], vs[1],
                                               os_[0], os_[1], mask.stride(0) if mask is not None else 0, B, HD // head_dim, Sq, Sk,
                                               head_dim, int(window), float(scale), dtype_code(q.dtype), stream_ptr()),
          "attention_prefill_window_tc")
    return out


def _check_sinks(sinks, heads):
    require_cuda(sinks)
    if sinks is not None and (sinks.dtype != torch.float32 or sinks.numel() != heads or not sinks.is_contiguous()):
        raise RuntimeError("attention: one fp32 sink per query head")


def attention_plain(q, k, v, heads, k_dim, v_dim, window=0, scale=1.0, first=None, pos_device=None, shared_kv=False,
                    kv_heads=None, bias=None, sink=False, chunk=None, sinks=None):
    """Windowed causal attention on the CUDA cores, any head sizes, fp32 / fp16 / bf16.  q [B, Sq,
    heads*k_dim]; k / v [B, rows, heads*dim] or, with shared_kv, [B, rows, dim] shared by the heads.
    Query row i holds position pos_device + i (None: i), the key of position j is row j mod rows;
    first [B] int32 is each sequence's first position.  kv_heads: heads of k / v, each shared by
    heads / kv_heads query heads.  bias = (r1, r2), fp32 per query head: r1 * ln(1 + r2 * distance) is
    taken off the scaled score.  sink: one is added to the softmax denominator.  chunk (0: none; instead of
    window and bias): a position sees only its own chunk of so many, counted from first; sinks fp32 [heads] or
    None: exp of it joins the denominator.  Returns [B, Sq, heads*v_dim]."""
    r1, r2 = bias if bias is not None else (None, None)
    require_cuda(q, k, v, first, pos_device, r1, r2)
    if bias is not None and any(r.dtype != torch.float32 or r.numel() != heads or not r.is_contiguous() for r in bias):
        raise RuntimeError("attention: the distance bias has two fp32 numbers per query head")
    B, Sq, _ = q.shape
    out = torch.empty((B, Sq, heads * v_dim), dtype=q.dtype, device=q.device)
    if any(t.stride(2) != 1 for t in (q, k, v)) or k.shape[1] != v.shape[1]:
        raise RuntimeError("attention: contiguous last dims and one number of key / value rows required")
    hk, hv = (0, 0) if shared_kv else (k_dim, v_dim)
    if chunk is not None:
        if bias is not None or window or sink:
            raise RuntimeError("attention: a chunk goes without window, bias and constant sink")
        _check_sinks(sinks, heads)
        check(lib().eb_attention_plain_chunk(ptr(q), ptr(k), ptr(v), ptr(out), q.stride(0), q.stride(1), k_dim, k.stride(0), k.stride(1), hk,
                                             v.stride(0), v.stride(1), hv, out.stride(0), out.stride(1), v_dim, B, heads,
                                             heads // (kv_heads or heads), Sq, k_dim, v_dim, int(chunk), k.shape[1], ptr(pos_device), ptr(first),
                                             ptr(sinks), float(scale), dtype_code(q.dtype), stream_ptr()), "attention_plain_chunk")
        return out
    check(lib().eb_attention_plain(ptr(q), ptr(k), ptr(v), ptr(out), q.stride(0), q.stride(1), k_dim, k.stride(0), k.stride(1), hk,
                                   v.stride(0), v.stride(1), hv, out.stride(0), out.stride(1), v_dim, B, heads,
                                   heads // (kv_heads or heads), Sq, k_dim, v_dim, int(window), k.shape[1], ptr(pos_device), ptr(first),
                                   ptr(r1), ptr(r2), 1 if sink else 0, float(scale), dtype_code(q.dtype), stream_ptr()),
          "attention_plain")
    return out


LATENT_WIDTHS = (64, 128, 256, 384, 512)      # latent widths of the tensor-core generation kernel


def pick_latent_nsplit(batch, heads, keys, sm_count=148):
    """Key splits per (sequence, head tile): what fills the SMs, at least two 64-key tiles each.  2
    and 4 are clusters that merge in shared memory.  (A cluster of 8 CTAs with a whole SM each finds
    room in a GPC so rarely that it ran in two waves: 8 splits took 50 us where 9, merged in a
    second launch, took 33.)"""
    ctas = batch * -(-heads // (32 if heads > 16 else 16))
    tiles = max(1, -(-keys // 64))
    want = max(1, min(sm_count // max(1, ctas), tiles // 2, 64))
    return 4 if 4 <= want < 8 else (2 if 2 <= want < 4 else (9 if want == 8 else want))


def latent_decode(q, cache, rank, heads, window, pos_device, scale, first=None, nsplit=None):
    """Generation step over a latent ring cache: q [B, heads*rank] (absorbed queries), cache [B,
    rows, rank], pos_device int32 scalar (the query's position).  Returns [B, heads*rank]."""
    require_cuda(q, cache, pos_device, first)
    B = q.shape[0]
    rows = cache.shape[1]
    out = torch.empty((B, heads * rank), dtype=q.dtype, device=q.device)
    if nsplit is None:
        nsplit = pick_latent_nsplit(B, heads, min(window, rows) if window > 0 else rows)
    nbytes = lib().eb_latent_decode_scratch_bytes(B, heads, rank, nsplit)
    scratch = torch.empty(nbytes, dtype=torch.uint8, device=q.device) if nbytes else None
    check(lib().eb_latent_decode(ptr(q), q.stride(0), ptr(cache), cache.stride(0), cache.stride(1), rows, ptr(out), out.stride(0), B,
                                 heads, rank, int(window), ptr(pos_device), ptr(first), float(scale), dtype_code(q.dtype), nsplit,
                                 ptr(scratch), nbytes, stream_ptr()), "latent_decode", launches=2 if nbytes else 1)
    return out


def attention_inputs(proj, heads, kv_heads, dk, dv, q_norm, q_count, k_norm, k_count, eps, k_cache, v_cache, rows_per_batch, temp=None,
                     vmix=None, v_first=None, pos_device=None, first=None):
    """Rows [q | k | v | ...] of a projection -> normalised queries [rows, heads*dk]; keys and values go
    to their cache rows.  q and k are normalised over all heads at once (q_count / k_count columns are
    real); temp = (coef, every): q times 1 + coef * ln(floor((p + 1) / every) + 1); vmix (fp32 scalar) and
    v_first (another layer's v_cache): v = (1 - vmix) v + vmix v_first of the same token."""
    require_cuda(proj, q_norm, k_norm, k_cache, v_cache, vmix, v_first, pos_device, first)
    n1 = proj.shape[0]
    if any(t.dtype != proj.dtype for t in (q_norm, k_norm, k_cache, v_cache)) or (v_first is not None and v_first.dtype != proj.dtype):
        raise RuntimeError("attention_inputs: one dtype required")
    if proj.dim() != 2 or proj.stride(1) != 1 or q_norm.numel() != heads * dk or k_norm.numel() != kv_heads * dk:
        raise RuntimeError("attention_inputs: rows [q | k | v], one norm entry per column of q and of k")
    B = n1 // rows_per_batch
    for t, w in ((k_cache, kv_heads * dk), (v_cache, kv_heads * dv), (v_first, kv_heads * dv)):
        if t is not None and (t.dim() != 3 or t.stride(2) != 1 or t.shape[0] != B or t.shape[2] != w or t.shape[1] != k_cache.shape[1]):
            raise RuntimeError("attention_inputs: caches are [batch, rows, kv_heads*dim]")
    if vmix is not None and (vmix.dtype != torch.float32 or v_first is None):
        raise RuntimeError("attention_inputs: vmix is an fp32 scalar and goes with v_first")
    q = torch.empty((n1, heads * dk), dtype=proj.dtype, device=proj.device)
    coef, every = temp if temp is not None else (0.0, 0)
    check(lib().eb_attention_inputs(ptr(proj), proj.stride(0), heads, kv_heads, dk, dv, ptr(q_norm), int(q_count), ptr(k_norm), int(k_count),
                                    float(eps), float(coef), int(every), ptr(vmix), ptr(v_first), v_first.stride(0) if vmix is not None else 0,
                                    v_first.stride(1) if vmix is not None else 0, ptr(q), q.stride(0), ptr(k_cache), k_cache.stride(0),
                                    k_cache.stride(1), ptr(v_cache), v_cache.stride(0), v_cache.stride(1), k_cache.shape[1], n1, rows_per_batch,
                                    ptr(pos_device), ptr(first), dtype_code(proj.dtype), stream_ptr()), "attention_inputs")
    return q


def distance_bias(r1, r2, distances):
    """Table [heads, >= distances] of r1 * log2(1 + r2 * d) for attention_prefill_biased."""
    require_cuda(r1, r2)
    n = distances + 256                              # (rows behind the end of a sequence read on)
    table = torch.empty((r1.numel(), n), dtype=torch.float32, device=r1.device)
    check(lib().eb_distance_bias(ptr(r1), ptr(r2), r1.numel(), n, ptr(table), stream_ptr()), "distance_bias")
    return table


def attention_prefill_biased(q, k, v, head_dim, bias_table, sink=True, window=0, mask=None, scale=None, out=None):
    """attention_prefill_window for q [B, Sq, H*D] and k / v [B, Sk, G*D] (G heads, each shared by H/G
    query heads); the distance bias of bias_table (distance_bias()) is taken off the scores; sink: one is
    added to the softmax denominator."""
    require_cuda(q, k, v, mask, out, bias_table)
    B, Sq, HD = q.shape
    Sk, H, G = k.shape[1], HD // head_dim, k.shape[2] // head_dim
    if out is None:
        out = torch.empty((B, Sq, HD), dtype=q.dtype, device=q.device)
    if mask is not None and (mask.dtype != q.dtype or mask.stride(-1) != 1 or mask.dim() != 2 or mask.shape[1] < Sk):
        raise RuntimeError("attention: mask must be [batch, kv_len] of the tensor dtype")
    if bias_table.dtype != torch.float32 or bias_table.dim() != 2 or not bias_table.is_contiguous() or bias_table.shape[0] != H or H % G:
        raise RuntimeError("attention: a bias table with one row per query head, query heads in equal groups")
    qs, ks, vs, os_ = (_bsh_strides(t, head_dim) for t in (q, k, v, out))
    scale = head_dim ** -0.5 if scale is None else scale
    check(lib().eb_attention_prefill_biased_tc(ptr(q), ptr(k), ptr(v), ptr(out), ptr(mask), qs[0], qs[1], ks[0], ks[1], vs[0], vs[1],
                                               os_[0], os_[1], mask.stride(0) if mask is not None else 0, B, H, H // G, Sq, Sk, head_dim,
                                               int(window), ptr(bias_table), bias_table.shape[1], 1 if sink else 0, float(scale),
                                               dtype_code(q.dtype), stream_ptr()), "attention_prefill_biased_tc")
    return out


def pick_group_nsplit(batch, units, keys, sm_count=148):
    """Key splits per (sequence, group of heads), of at least 256 keys each: enough for two CTAs per SM,
    then what spreads the CTAs over the SMs most evenly, each further split counted as 4 % (its merge)."""
    n, most = max(1, batch * units), max(1, min(keys // 256, 64))
    least = min(most, -(-2 * sm_count // n))
    return min(range(least, most + 1), key=lambda s: -(-n * s // sm_count) / (n * s) * (1 + 0.04 * s))


def attention_group_decode(q, k, v, head_dim, pos_device, scale, first=None, bias=None, sink=True, nsplit=None):
    """Generation step: q [B, H*D], k / v [B, rows, G*D] cache views, pos_device int32 scalar (the query's
    position).  bias = (r1, r2) fp32 per query head.  Returns [B, H*D]."""
    r1, r2 = bias if bias is not None else (None, None)
    require_cuda(q, k, v, pos_device, first, r1, r2)
    B, HD = q.shape
    H, G, rows = HD // head_dim, k.shape[2] // head_dim, k.shape[1]
    if bias is not None and any(r.dtype != torch.float32 or r.numel() != H or not r.is_contiguous() for r in bias):
        raise RuntimeError("attention: the distance bias has two fp32 numbers per query head")
    ks, vs = _bsh_strides(k, head_dim), _bsh_strides(v, head_dim)
    out = torch.empty((B, HD), dtype=q.dtype, device=q.device)
    if nsplit is None:
        nsplit = pick_group_nsplit(B, G * -(-(H // G) // 16), rows)
    nbytes = lib().eb_attention_group_decode_scratch_bytes(B, H, G, head_dim, nsplit)
    scratch = _get_scratch(q.device, nbytes) if nbytes else None
    check(lib().eb_attention_group_decode(ptr(q), ptr(k), ptr(v), ptr(out), q.stride(0), ks[0], ks[1], vs[0], vs[1], out.stride(0), B, H, G,
                                          head_dim, rows, ptr(pos_device), ptr(first), ptr(r1), ptr(r2), 1 if sink else 0, float(scale),
                                          dtype_code(q.dtype), nsplit, ptr(scratch), scratch.numel() if scratch is not None else 0,
                                          stream_ptr()), "attention_group_decode")
    return out


def attention_rotary(proj, heads, kv_heads, dk, dim, q_norm, k_norm, eps, freq, k_cache, v_cache, rows_per_batch, pos_device=None, first=None,
                     keys=False):
    """Rows [q | k | ...] of a projection -> queries [rows, heads*dk], normalised head by head over `dim` columns
    and rotated (freq fp32: angle per position of each leading pair); keys, treated alike, and values, the
    keys as projected, go to the ring caches.  keys: also returns the keys as rows (else None)."""
    require_cuda(proj, q_norm, k_norm, freq, k_cache, v_cache, pos_device, first)
    n1 = proj.shape[0]
    if any(t.dtype != proj.dtype for t in (q_norm, k_norm, k_cache, v_cache)) or freq.dtype != torch.float32 or not freq.is_contiguous():
        raise RuntimeError("attention_rotary: one dtype required, frequencies in fp32")
    if proj.dim() != 2 or proj.stride(1) != 1 or q_norm.numel() != dk or k_norm.numel() != dk:
        raise RuntimeError("attention_rotary: rows [q | k], one norm entry per column of a head")
    B = n1 // rows_per_batch
    for t in (k_cache, v_cache):
        if t.dim() != 3 or t.stride(2) != 1 or t.shape[0] != B or t.shape[2] != kv_heads * dk or t.shape[1] != k_cache.shape[1]:
            raise RuntimeError("attention_rotary: caches are [batch, rows, kv_heads*dk]")
    q = torch.empty((n1, heads * dk), dtype=proj.dtype, device=proj.device)
    k = torch.empty((n1, kv_heads * dk), dtype=proj.dtype, device=proj.device) if keys else None
    check(lib().eb_attention_rotary(ptr(proj), proj.stride(0), heads, kv_heads, dk, int(dim), ptr(q_norm), ptr(k_norm), float(eps), ptr(freq),
                                    freq.numel(), ptr(q), q.stride(0), ptr(k), k.stride(0) if keys else 0, ptr(k_cache), k_cache.stride(0),
                                    k_cache.stride(1), ptr(v_cache), v_cache.stride(0), v_cache.stride(1), k_cache.shape[1], n1, rows_per_batch,
                                    ptr(pos_device), ptr(first), dtype_code(proj.dtype), stream_ptr()), "attention_rotary")
    return q, k


def attention_prefill_chunk(q, k, v, head_dim, chunk, sinks=None, first=None, scale=None, out=None):
    """Prompt attention (tensor-core kernel): q [B, S, H*D], k / v [B, S, G*D]; row i sees the keys up to itself in
    its own chunk (0: no chunks) counted from first[b]; exp(sinks[h]) joins the denominator."""
    require_cuda(q, k, v, first, out)
    B, S, HD = q.shape
    H, G = HD // head_dim, k.shape[2] // head_dim
    if k.shape[1] != S or v.shape != k.shape or H % G:
        raise RuntimeError("attention: a whole prompt with query heads in equal groups")
    _check_sinks(sinks, H)
    if out is None:
        out = torch.empty((B, S, HD), dtype=q.dtype, device=q.device)
    qs, ks, vs, os_ = (_bsh_strides(t, head_dim) for t in (q, k, v, out))
    scale = head_dim ** -0.5 if scale is None else scale
    check(lib().eb_attention_prefill_chunk_tc(ptr(q), ptr(k), ptr(v), ptr(out), *qs, *ks, *vs, *os_, B, H, H // G, S, head_dim, int(chunk),
                                              ptr(first), ptr(sinks), float(scale), dtype_code(q.dtype), stream_ptr()), "attention_prefill_chunk_tc")
    return out


def attention_group_decode_chunk(q, k, v, head_dim, pos_device, scale, chunk, sinks=None, first=None, nsplit=None):
    """Generation step of attention_prefill_chunk: q [B, H*D], k / v [B, rows, G*D] cache views (rings if chunk > 0),
    pos_device int32 scalar (the query's position).  Returns [B, H*D]."""
    require_cuda(q, k, v, pos_device, first)
    B, HD = q.shape
    H, G, rows = HD // head_dim, k.shape[2] // head_dim, k.shape[1]
    _check_sinks(sinks, H)
    ks, vs = _bsh_strides(k, head_dim), _bsh_strides(v, head_dim)
    out = torch.empty((B, HD), dtype=q.dtype, device=q.device)
    if nsplit is None:
        nsplit = pick_group_nsplit(B, G * -(-(H // G) // 16), rows)
    nbytes = lib().eb_attention_group_decode_scratch_bytes(B, H, G, head_dim, nsplit)
    scratch = _get_scratch(q.device, nbytes) if nbytes else None
    check(lib().eb_attention_group_decode_chunk(ptr(q), ptr(k), ptr(v), ptr(out), q.stride(0), ks[0], ks[1], vs[0], vs[1], out.stride(0), B, H, G,
                                                head_dim, rows, int(chunk), ptr(pos_device), ptr(first), ptr(sinks), float(scale),
                                                dtype_code(q.dtype), nsplit, ptr(scratch), scratch.numel() if scratch is not None else 0,
                                                stream_ptr()), "attention_group_decode_chunk")
    return out
