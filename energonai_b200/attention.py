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


LATENT_WIDTHS = (64, 128, 192, 256, 320, 384, 512, 576)      # latent widths of the tensor-core generation kernel


def pick_latent_nsplit(batch, heads, keys, sm_count=148):
    """Key splits per (sequence, head tile): what fills the SMs, at least two 64-key tiles each.  2
    and 4 are clusters that merge in shared memory.  (A cluster of 8 CTAs with a whole SM each finds
    room in a GPC so rarely that it ran in two waves: 8 splits took 50 us where 9, merged in a
    second launch, took 33.)"""
    ctas = batch * -(-heads // (32 if heads > 16 else 16))
    tiles = max(1, -(-keys // 64))
    want = max(1, min(sm_count // max(1, ctas), tiles // 2, 64))
    return 4 if 4 <= want < 8 else (2 if 2 <= want < 4 else (9 if want == 8 else want))


def latent_decode(q, cache, rank, heads, window, pos_device, scale, first=None, sinks=None, nsplit=None):
    """Generation step over a latent ring cache: q [B, heads*rank] (absorbed queries), cache [B,
    rows, rank], pos_device int32 scalar (the query's position); sinks fp32 [heads] or None: exp of it joins the
    softmax denominator.  Returns [B, heads*rank]."""
    require_cuda(q, cache, pos_device, first)
    _check_sinks(sinks, heads)
    B = q.shape[0]
    rows = cache.shape[1]
    out = torch.empty((B, heads * rank), dtype=q.dtype, device=q.device)
    if nsplit is None:
        nsplit = pick_latent_nsplit(B, heads, min(window, rows) if window > 0 else rows)
    nbytes = lib().eb_latent_decode_scratch_bytes(B, heads, rank, nsplit)
    scratch = torch.empty(nbytes, dtype=torch.uint8, device=q.device) if nbytes else None
    check(lib().eb_latent_decode_sink(ptr(q), q.stride(0), ptr(cache), cache.stride(0), cache.stride(1), rows, ptr(out), out.stride(0), B,
                                 heads, rank, int(window), ptr(pos_device), ptr(first), ptr(sinks), float(scale), dtype_code(q.dtype), nsplit,
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


def distance_slopes(heads, device=None):
    """Slopes of a bias linear in the distance: 2^(-8 (h + 1) / heads) for head h, fp32."""
    h = torch.arange(1, heads + 1, dtype=torch.float64)
    return torch.exp2(-8 * h / heads).to(dtype=torch.float32, device=device)


def _check_slopes(slopes, heads):
    require_cuda(slopes)
    if slopes is not None and (slopes.dtype != torch.float32 or slopes.numel() != heads or not slopes.is_contiguous()):
        raise RuntimeError("attention: one fp32 slope per query head")


def _check_gate(gate, out):
    require_cuda(gate)
    if gate is not None and (gate.shape != out.shape or gate.dtype != out.dtype or gate.stride(-1) != 1):
        raise RuntimeError("attention: the gate is laid out like the output")


def attention_values(k, v, kv_heads, dv_count, eps, k_cache, v_cache, keep, rows_per_batch, pos_device=None, first=None):
    """Values v [rows, kv_heads*dv] over their head's root mean square, in place, and keys k [rows, kv_heads*dk] and
    values to a cache [batch, keep + ring rows, ...] (RingCache(keep=...)).  k and v are column views of one
    projection."""
    require_cuda(k, v, k_cache, v_cache, pos_device, first)
    n1 = k.shape[0]
    if k.stride(1) != 1 or v.stride(1) != 1 or k.stride(0) != v.stride(0) or any(t.dtype != k.dtype for t in (v, k_cache, v_cache)):
        raise RuntimeError("attention_values: k and v are column ranges of one row layout, caches of their dtype")
    if n1 % rows_per_batch or k.shape[1] % kv_heads or v.shape[1] % kv_heads:
        raise RuntimeError("attention_values: whole sequences and whole heads")
    for t, x in ((k_cache, k), (v_cache, v)):
        if t.dim() != 3 or t.stride(2) != 1 or t.shape[0] != n1 // rows_per_batch or t.shape[2] != x.shape[1] or t.shape[1] != k_cache.shape[1] or t.shape[1] <= keep:
            raise RuntimeError("attention_values: caches are [batch, keep + ring rows, kv_heads*dim]")
    check(lib().eb_attention_values(ptr(k), ptr(v), k.stride(0), kv_heads, k.shape[1] // kv_heads, v.shape[1] // kv_heads, int(dv_count), float(eps),
                                    ptr(k_cache), k_cache.stride(0), k_cache.stride(1), ptr(v_cache), v_cache.stride(0), v_cache.stride(1), int(keep),
                                    k_cache.shape[1] - keep, n1, rows_per_batch, ptr(pos_device), ptr(first), dtype_code(k.dtype), stream_ptr()),
          "attention_values")


def sigmoid_gate(y, gate, out=None):
    """y * sigmoid(gate), rows [n, columns] (row strides allowed)."""
    out = torch.empty_like(y) if out is None else out
    require_cuda(y, out)
    _check_gate(gate, y)
    if y.dim() != 2 or y.stride(1) != 1 or out.shape != y.shape or out.dtype != y.dtype or out.stride(1) != 1:
        raise RuntimeError("sigmoid_gate: rows of one dtype")
    check(lib().eb_sigmoid_gate(ptr(y), y.stride(0), ptr(gate), gate.stride(0), ptr(out), out.stride(0), y.shape[0], y.shape[1], dtype_code(y.dtype),
                                stream_ptr()), "sigmoid_gate")
    return out


def attention_plain_capped(q, k, v, heads, k_dim, v_dim, window=0, keep=0, kept_rows=0, scale=1.0, first=None, pos_device=None, kv_heads=None, slopes=None,
                           cap=0.0, sink=False):
    """attention_plain with a window that keeps the first `keep` positions visible, scores capped by cap * tanh(score / cap)
    (0: not) and slopes * distance taken off; kept_rows: rows in front of the ring in k / v that hold those
    positions (keep, or 0: position j is row j mod rows)."""
    require_cuda(q, k, v, first, pos_device)
    _check_slopes(slopes, heads)
    B, Sq, _ = q.shape
    out = torch.empty((B, Sq, heads * v_dim), dtype=q.dtype, device=q.device)
    if any(t.stride(2) != 1 for t in (q, k, v)) or k.shape[1] != v.shape[1]:
        raise RuntimeError("attention: contiguous last dims and one number of key / value rows required")
    check(lib().eb_attention_plain_capped(ptr(q), ptr(k), ptr(v), ptr(out), q.stride(0), q.stride(1), k_dim, k.stride(0), k.stride(1), k_dim,
                                          v.stride(0), v.stride(1), v_dim, out.stride(0), out.stride(1), v_dim, B, heads, heads // (kv_heads or heads), Sq,
                                          k_dim, v_dim, int(window), int(keep), int(kept_rows), k.shape[1] - kept_rows, ptr(pos_device), ptr(first),
                                          ptr(slopes), float(cap), 1 if sink else 0, float(scale), dtype_code(q.dtype), stream_ptr()), "attention_plain_capped")
    return out


PROMPT_HEADS = ((64, 64), (128, 64), (128, 128), (192, 64), (192, 128))       # key / value head sizes of attention_prefill_gated


def _prompt_views(q, k, v, k_dim, v_dim, gate, out):
    require_cuda(q, k, v, out)
    B, S, H, G = q.shape[0], q.shape[1], q.shape[2] // k_dim, k.shape[2] // k_dim
    if k.shape[1] != S or v.shape[:2] != k.shape[:2] or v.shape[2] != G * v_dim or H % G:
        raise RuntimeError("attention: a whole prompt with query heads in equal groups")
    if out is None:
        out = torch.empty((B, S, H * v_dim), dtype=q.dtype, device=q.device)
    _check_gate(gate, out)
    strides = [x for t, d in ((q, k_dim), (k, k_dim), (v, v_dim), (out, v_dim)) for x in _bsh_strides(t, d)]
    return B, S, H, G, out, strides + (list(_bsh_strides(gate, v_dim)) if gate is not None else [0, 0])


def attention_prefill_gated(q, k, v, k_dim, v_dim, sinks=None, first=None, gate=None, scale=None, out=None):
    """attention_prefill_chunk without chunks, with heads of k_dim / v_dim (PROMPT_HEADS), the output times sigmoid(gate)."""
    B, S, H, G, out, strides = _prompt_views(q, k, v, k_dim, v_dim, gate, out)
    require_cuda(first)
    _check_sinks(sinks, H)
    scale = k_dim ** -0.5 if scale is None else scale
    check(lib().eb_attention_prefill_gated_tc(ptr(q), ptr(k), ptr(v), ptr(out), ptr(gate), *strides, B, H, H // G, S, k_dim, v_dim, ptr(first), ptr(sinks),
                                              float(scale), dtype_code(q.dtype), stream_ptr()), "attention_prefill_gated_tc")
    return out


def attention_prefill_capped(q, k, v, k_dim, v_dim, window=0, keep=0, slopes=None, cap=0.0, sink=True, first=None, gate=None, scale=None, out=None):
    """Prompt attention (tensor-core kernel) by the rule of attention_plain_capped, the output times sigmoid(gate)."""
    B, S, H, G, out, strides = _prompt_views(q, k, v, k_dim, v_dim, gate, out)
    require_cuda(first)
    _check_slopes(slopes, H)
    scale = k_dim ** -0.5 if scale is None else scale
    check(lib().eb_attention_prefill_capped_tc(ptr(q), ptr(k), ptr(v), ptr(out), ptr(gate), *strides, B, H, H // G, S, k_dim, v_dim, int(window), int(keep),
                                               ptr(first), ptr(slopes), float(cap), 1 if sink else 0, float(scale), dtype_code(q.dtype), stream_ptr()),
          "attention_prefill_capped_tc")
    return out


def attention_group_decode_capped(q, k, v, head_dim, pos_device, scale, window=0, keep=0, slopes=None, cap=0.0, sink=True, first=None, gate=None, out=None,
                                  nsplit=None):
    """Generation step of attention_prefill_capped: q [B, H*D], k / v [B, keep + ring rows, G*D] cache views, pos_device int32
    scalar (the query's position).  Returns [B, H*D]."""
    require_cuda(q, k, v, pos_device, first, out)
    B, HD = q.shape
    H, G, rows = HD // head_dim, k.shape[2] // head_dim, k.shape[1] - keep
    _check_slopes(slopes, H)
    ks, vs = _bsh_strides(k, head_dim), _bsh_strides(v, head_dim)
    if out is None:
        out = torch.empty((B, HD), dtype=q.dtype, device=q.device)
    _check_gate(gate, out)
    if nsplit is None:
        nsplit = pick_group_nsplit(B, G * -(-(H // G) // 16), rows + keep)
    nbytes = lib().eb_attention_group_decode_scratch_bytes(B, H, G, head_dim, nsplit)
    scratch = _get_scratch(q.device, nbytes) if nbytes else None
    check(lib().eb_attention_group_decode_capped(ptr(q), ptr(k), ptr(v), ptr(out), ptr(gate), q.stride(0), ks[0], ks[1], vs[0], vs[1], out.stride(0),
                                                 gate.stride(0) if gate is not None else 0, B, H, G, head_dim, int(keep), rows, int(window),
                                                 ptr(pos_device), ptr(first), ptr(slopes), float(cap), 1 if sink else 0, float(scale),
                                                 dtype_code(q.dtype), nsplit, ptr(scratch), scratch.numel() if scratch is not None else 0,
                                                 stream_ptr()), "attention_group_decode_capped")
    return out


def yarn_rotation(dims, base, scaling=None):
    """(angle per position of each neighbouring pair, fp32 [dims / 2]; factor of sine and cosine).  scaling (YaRN) =
    (factor, original, fast, slow): pairs that turn fewer than `slow` times over `original` positions are slowed
    down by factor, those that turn more than `fast` times are not, with a linear ramp between them."""
    import math
    i = torch.arange(dims // 2, dtype=torch.float64)
    freq = float(base) ** (-2 * i / max(1, dims))
    if scaling is None:
        return freq.float(), 1.0
    factor, original, fast, slow = scaling
    pair_of = lambda turns: dims * math.log(original / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(pair_of(fast)), 0), min(math.ceil(pair_of(slow)), dims - 1)
    ramp = ((i - lo) / max(hi - lo, 1e-3)).clamp(0, 1)
    return (freq / factor * ramp + freq * (1 - ramp)).float(), 0.1 * math.log(factor) + 1


def latent_inputs(proj, q_cols, q_count, q_norm, eps, row=None, rows_per_batch=1, pos_device=None, first=None):
    """Rows [query latent | cached row] of a projection -> the normalised query latent [rows, q_cols] and the rows that go to
    the cache.  row = dict(cols, rot_col, count, norm, freq, factor, ring, keep_rows): the part from rot_col on is
    turned; ring [batch, rows, cols]; keep_rows: also returns the rows themselves (else None).  None: no latent."""
    row = row or {}
    ring, norm, freq = row.get("ring"), row.get("norm"), row.get("freq")
    require_cuda(proj, q_norm, ring, norm, freq, pos_device, first)
    n1, cols = proj.shape[0], row.get("cols", 0)
    if proj.dim() != 2 or proj.stride(1) != 1 or q_norm.numel() != q_cols or any(t is not None and t.dtype != proj.dtype for t in (q_norm, norm, ring)):
        raise RuntimeError("latent_inputs: rows, norms and cache of one dtype")
    if ring is not None and (ring.dim() != 3 or ring.stride(2) != 1 or ring.shape[0] * rows_per_batch != n1 or ring.shape[2] < cols or norm.numel() != row["rot_col"]
                             or freq.dtype != torch.float32 or not freq.is_contiguous()):
        raise RuntimeError("latent_inputs: the cache is [batch, rows, columns], the norm has an entry per column of the latent")
    q = torch.empty((n1, q_cols), dtype=proj.dtype, device=proj.device)
    rows = torch.empty((n1, cols), dtype=proj.dtype, device=proj.device) if row.get("keep_rows") else None
    check(lib().eb_latent_inputs(ptr(proj), proj.stride(0), q_cols, int(q_count), ptr(q_norm), ptr(q), q_cols, cols, row.get("rot_col", 0),
                                 int(row.get("count", 0)), ptr(norm), freq.numel() if freq is not None else 0, ptr(freq), float(row.get("factor", 1.0)),
                                 float(eps), ptr(rows), cols, ptr(ring), ring.stride(0) if ring is not None else 0,
                                 ring.stride(1) if ring is not None else 0, ring.shape[1] if ring is not None else 0, n1, rows_per_batch, ptr(pos_device),
                                 ptr(first), dtype_code(proj.dtype), stream_ptr()), "latent_inputs")
    return q, rows


def rotate_heads(x, heads, head_cols, col, freq, factor, rows_per_batch, pos_device=None, first=None):
    """Turns the pairs from column `col` of every head of rows x, in place."""
    require_cuda(x, freq, pos_device, first)
    if x.dim() != 2 or x.stride(1) != 1 or x.shape[1] != heads * head_cols or freq.dtype != torch.float32 or not freq.is_contiguous() or x.shape[0] % rows_per_batch:
        raise RuntimeError("rotate_heads: rows of whole heads, frequencies in fp32")
    check(lib().eb_rotate_heads(ptr(x), x.stride(0), heads, head_cols, int(col), freq.numel(), ptr(freq), float(factor), x.shape[0], rows_per_batch,
                                ptr(pos_device), ptr(first), dtype_code(x.dtype), stream_ptr()), "rotate_heads")
    return x
