"""Python entry to the mixture-of-experts kernels: routing, the expert-sorted row layout and the
grouped products (eb_moe_*, eb_gemm_grouped, eb_grouped_skinny)."""
import torch

from ._lib import lib, check, dtype_code, ptr, stream_ptr, require_cuda

COUNT_STRIDE = 32        # EB_MOE_COUNT_STRIDE
ROW_TILE = 128           # rows of one expert come in tiles of this many in the sorted layout

SKINNY_MAX_ENTRIES = 10240   # (token, choice) pairs the weight-streaming product sorts in shared memory


UNITS = {None: 0, "clamped": 1, "geglu": 2, "gelu": 3}      # EB_UNIT_*
GATED = ("clamped", "geglu")


def unit_code(unit, gate):
    """(code, limit, alpha, columns per result) of a unit; gate = (limit, alpha) alone names the clamped one."""
    if gate is not None and unit is None:
        unit = "clamped"
    limit, alpha = gate if gate is not None else (0.0, 0.0)
    return UNITS[unit], float(limit), float(alpha), 2 if unit in GATED else 1


class RouterRule:
    """How a router chooses: `choices` softmax scores, those from `experts` on standing for the input itself;
    correction fp32 [choices] or None is added for the choice; of `groups` equal groups the best `keep`
    are open; the weights of the chosen are their scores over their sum."""

    def __init__(self, choices, experts, correction=None, groups=1, keep=1):
        self.choices, self.experts, self.correction, self.groups, self.keep = choices, experts, correction, groups, keep


def route_rule(logits, rule, top, first=None, rows_per_batch=0, counts=None, gated=False):
    """logits [T, >= choices (+ 1 if gated)] fp32 -> (idx, weights, ranks or None, shared gate or None)."""
    require_cuda(logits, first, counts, rule.correction)
    if logits.dim() != 2 or logits.dtype != torch.float32 or logits.stride(1) != 1 or logits.shape[1] < rule.choices + int(gated):
        raise RuntimeError("moe route: logits must be fp32 [tokens, choices]")
    T, dev = logits.shape[0], logits.device
    idx = torch.empty((T, top), dtype=torch.int32, device=dev)
    w = torch.empty((T, top), dtype=torch.float32, device=dev)
    ranks = torch.empty((T, top), dtype=torch.int32, device=dev) if counts is not None else None
    gate = torch.empty(T, dtype=torch.float32, device=dev) if gated else None
    check(lib().eb_moe_route_rule(ptr(logits), logits.stride(0), T, rule.choices, rule.experts, top, ptr(rule.correction), rule.groups, rule.keep,
                                  ptr(first), rows_per_batch, ptr(idx), ptr(w), ptr(counts), ptr(ranks), ptr(gate), stream_ptr()), "moe_route")
    return idx, w, ranks, gate


def new_counts(experts, device):
    """Zeroed row counters of the experts; route() fills them, SortedRows zeroes them again."""
    return torch.zeros(experts * COUNT_STRIDE, dtype=torch.int32, device=device)


def route(logits, experts, top, first=None, rows_per_batch=0, counts=None):
    """logits [T, >= experts] fp32 -> idx [T, top] int32, weights [T, top] fp32 (softmax scores over
    all experts, not renormalised).  first [batch] int32: rows before it in their sequence are
    padding (idx -1).  With counts (new_counts) also ranks [T, top]."""
    require_cuda(logits, first, counts)
    if logits.dim() != 2 or logits.dtype != torch.float32 or logits.stride(1) != 1:
        raise RuntimeError("moe route: logits must be fp32 [tokens, experts]")
    T = logits.shape[0]
    idx = torch.empty((T, top), dtype=torch.int32, device=logits.device)
    w = torch.empty((T, top), dtype=torch.float32, device=logits.device)
    ranks = torch.empty((T, top), dtype=torch.int32, device=logits.device) if counts is not None else None
    check(lib().eb_moe_route(ptr(logits), logits.stride(0), T, experts, top, ptr(first), rows_per_batch, ptr(idx), ptr(w), ptr(counts),
                             ptr(ranks), stream_ptr()), "moe_route")
    return (idx, w, ranks) if counts is not None else (idx, w)


class SortedRows:
    """The rows of a batch in expert order, every expert in whole 128-row tiles."""

    def __init__(self, x, idx, ranks, counts):
        T, top = idx.shape
        experts = counts.numel() // COUNT_STRIDE
        self.max_tiles = (T * top) // ROW_TILE + min(experts, T * top)
        dev = x.device
        i32 = lambda n: torch.empty(n, dtype=torch.int32, device=dev)
        offsets, self.tile_group, self.live_tiles = i32(experts), i32(self.max_tiles), i32(1)
        check(lib().eb_moe_plan(ptr(counts), experts, ptr(offsets), ptr(self.tile_group), self.max_tiles, ptr(self.live_tiles),
                                stream_ptr()), "moe_plan")
        self.rows = torch.empty((T, top), dtype=torch.int32, device=dev)
        n = self.max_tiles * ROW_TILE
        self.x = torch.empty((n, x.shape[1]), dtype=x.dtype, device=dev)
        check(lib().eb_moe_permute(ptr(x), x.stride(0), x.shape[1], dtype_code(x.dtype), T, top, ptr(idx), ptr(ranks), ptr(offsets),
                                   ptr(self.rows), ptr(self.x), self.x.stride(0), n, stream_ptr()), "moe_permute")


def grouped_gemm(a, w, plan, gate=None, unit=None):
    """a [rows of the plan, K], w [experts, N, K] -> [rows, N], or a unit of it: "gelu"; gated ones give
    [rows, N/2] from columns in blocks of 8 gates and their 8 ups ("geglu"; gate = (limit, alpha): the
    clamped one)."""
    require_cuda(a, w)
    E, N, K = w.shape
    M = a.shape[0]
    if not w.is_contiguous() or a.dtype != w.dtype or a.shape[1] != K or a.stride(1) != 1:
        raise RuntimeError("grouped gemm: a [rows, K] and contiguous w [experts, N, K] of one dtype required")
    code, limit, alpha, per = unit_code(unit, gate)
    if a.dtype == torch.float32:
        out = torch.empty((M, N), dtype=a.dtype, device=a.device)
        check(lib().eb_gemm_f32(ptr(a), a.stride(0), 0, ptr(w), K, N * K, ptr(out), N, 0, M, N, K, 1, ptr(plan.tile_group),
                                ptr(plan.live_tiles), None, 0, None, stream_ptr()), "gemm_f32")
        return unit_act(out, unit, gate) if code else out
    out = torch.empty((M, N // per), dtype=a.dtype, device=a.device)
    check(lib().eb_gemm_grouped(ptr(a), a.stride(0), ptr(w), K, ptr(out), out.stride(0), M, N, K, E, ptr(plan.tile_group),
                                ptr(plan.live_tiles), code, limit, alpha, dtype_code(a.dtype), stream_ptr()), "gemm_grouped")
    return out


def unit_act(x, unit=None, gate=None, out=None):
    """A unit alone: [n, N] -> [n, N], or, gated, [n, 2*half] in the 8 + 8 column order -> [n, half]."""
    require_cuda(x, out)
    code, limit, alpha, per = unit_code(unit, gate)
    n = x.shape[1] // per
    y = torch.empty((x.shape[0], n), dtype=x.dtype, device=x.device) if out is None else out
    check(lib().eb_unit_act(ptr(x), x.stride(0), ptr(y), y.stride(0), x.shape[0], n, code, limit, alpha, dtype_code(x.dtype), stream_ptr()), "unit_act")
    return y


def gated_act(x, limit, alpha):
    """[n, 2*half] in the 8 + 8 column order -> [n, half], the clamped unit."""
    return unit_act(x, gate=(limit, alpha))


def skinny_experts(a, w, idx, a_div, gate=None, unit=None):
    """Generation steps: entry i of idx (flattened [T, top]) multiplies row i // a_div of a by the
    weights w [experts, N, K] of expert idx[i] -> [T * top, N or N/2]; rows of unrouted entries are
    not written."""
    require_cuda(a, w, idx)
    E, N, K = w.shape
    n = idx.numel()
    if not w.is_contiguous() or a.dtype != w.dtype or a.shape[1] != K or a.stride(1) != 1 or a.shape[0] * a_div < n:
        raise RuntimeError("skinny product: a [rows, K] and contiguous w [experts, N, K] of one dtype required")
    code, limit, alpha, per = unit_code(unit, gate)
    out = torch.empty((n, N // per), dtype=a.dtype, device=a.device)
    check(lib().eb_grouped_skinny(ptr(a), a.stride(0), 0, a_div, ptr(w), N * K, K, ptr(out), out.stride(0), 0, ptr(idx), n, E, N, K,
                                  code, limit, alpha, dtype_code(a.dtype), stream_ptr()), "grouped_skinny")
    return out


def per_head(a, w):
    """a [B, heads * K] (row stride allowed), w [heads, N, K] -> [B, heads * N]: every head's slice
    times that head's weights."""
    require_cuda(a, w)
    H, N, K = w.shape
    B = a.shape[0]
    if not w.is_contiguous() or a.dtype != w.dtype or a.shape[1] != H * K or a.stride(1) != 1:
        raise RuntimeError("per_head: a [rows, heads*K] and contiguous w [heads, N, K] of one dtype required")
    out = torch.empty((B, H * N), dtype=a.dtype, device=a.device)
    if a.dtype == torch.float32:
        check(lib().eb_gemm_f32(ptr(a), a.stride(0), K, ptr(w), K, N * K, ptr(out), H * N, N, B, N, K, H, None, None, None, 0, None,
                                stream_ptr()), "gemm_f32")
    else:
        check(lib().eb_grouped_skinny(ptr(a), a.stride(0), K, 1, ptr(w), N * K, K, ptr(out), H * N, N, None, B, H, N, K, 0, 0.0, 0.0,
                                      dtype_code(a.dtype), stream_ptr()), "grouped_skinny")
    return out
