"""Feed-forward ops of served layer-plan decoders (``csrc/moe_serve.cu``, ``csrc/router.cu``): activations between strided
matrices, expert choice with the dispatch bookkeeping in the same launch, rows into expert order, and the routed
feed-forward around the grouped GEMM.  CPU tensors run the plain PyTorch definition."""
from __future__ import annotations

import ctypes

import torch

from . import _lib
from .gemm import grouped_gemm, linear_forward
from .router import route_ref

LAUNCHES = {"moe": 0}
SEG = 128               # expert segments are padded to the grouped GEMM's tile height
MAX_EXPERTS, MAX_TOP, MAX_GROUPS = 512, 16, 32
SILU_GATE, RELU2 = 0, 1


def activate(kind: int, src, cols: int, up_off: int, dst, row_logit=None, n_rows=None):
    """``dst = silu(src[:, :cols]) * src[:, up_off:]`` (SILU_GATE) or ``relu(src[:, up_off:])^2`` (RELU2), times
    ``sigmoid(row_logit)`` per row when given.  ``src`` / ``dst`` may have any row stride; ``n_rows``: device count of the
    rows in use."""
    if not src.is_cuda:
        u = src[:, up_off:up_off + cols].float()
        a = torch.nn.functional.silu(src[:, :cols].float()) * u if kind == SILU_GATE else torch.relu(u).square()
        dst.copy_(a if row_logit is None else a * torch.sigmoid(row_logit)[:, None])
        return dst
    ptrs = (ctypes.c_void_p * 4)(*[t.data_ptr() if t is not None else None for t in (src, dst, row_logit, n_rows)])
    lds = (ctypes.c_longlong * 4)(src.stride(0), dst.stride(0), row_logit.stride(0) if row_logit is not None else 0,
                                  src.shape[0])
    dims = (ctypes.c_int * 2)(up_off, cols)
    LAUNCHES["moe"] += 1
    _lib.check(_lib.kernels().gk_ffn_act(kind, int(src.dtype == torch.float32), ptrs, lds, dims, _lib.stream_ptr()), "ffn_act")
    return dst


def choose(logits, experts: int, top: int, correction, counts, sigmoid=False, norm=True, scale=1.0, groups=1, keep=1):
    """Scores of ``logits[:, :experts]`` (32-bit; a softmax or sigmoids), the ``top`` experts by score + ``correction``
    among the best ``keep`` of ``groups`` groups of neighbours, their scores (normalised with ``norm``) times ``scale``.
    Returns ``(expert [T, top] int64, weight [T, top], place [T, top] int32)`` and adds to ``counts`` [experts] int32 how
    many tokens chose each; ``place`` numbers the tokens of one expert."""
    T = logits.shape[0]
    if not logits.is_cuda:
        idx, w = route_ref(logits[:, :experts], correction, None, top, groups, keep, sigmoid, norm, scale)
        place, flat = torch.zeros(T * top, dtype=torch.int32), idx.reshape(-1).tolist()
        for i, e in enumerate(flat):
            place[i] = counts[e]
            counts[e] += 1
        return idx, w, place.view(T, top)
    idx, w, place = _choice_buffers(T, top, logits.device)
    LAUNCHES["moe"] += 1
    _lib.check(_lib.kernels().gk_router_dispatch(
        _lib.ptr(logits), logits.stride(0), _lib.ptr(correction), _lib.ptr(idx), _lib.ptr(w), _lib.ptr(counts),
        _lib.ptr(place), T, experts, top, int(sigmoid), int(norm), float(scale), groups, keep, _lib.stream_ptr()), "router_dispatch")
    return idx, w, place


def _choice_buffers(T, top, device):
    return (torch.empty(T, top, dtype=torch.int64, device=device), torch.empty(T, top, dtype=torch.float32, device=device),
            torch.empty(T, top, dtype=torch.int32, device=device))


FUSED_TOKENS, FUSED_WIDTH = 128, 11264      # up to here a CTA per token computes the logits itself


def route_tokens(h, router, experts: int, top: int, correction, counts, sigmoid=False, norm=True, scale=1.0, groups=1, keep=1):
    """``choose`` on the logits ``h @ router^T``; ``router`` [experts + extra, H] may hold rows that are only projected.
    Returns ``(logits [T, rows], choice)``."""
    T, n = h.shape[0], router.shape[0]
    if not h.is_cuda or T > FUSED_TOKENS or h.shape[1] > FUSED_WIDTH:
        logits = linear_forward(h, router, out_dtype=torch.float32)
        return logits, choose(logits, experts, top, correction, counts, sigmoid, norm, scale, groups, keep)
    logits = torch.empty(T, n, dtype=torch.float32, device=h.device)
    idx, w, place = _choice_buffers(T, top, h.device)
    LAUNCHES["moe"] += 1
    _lib.check(_lib.kernels().gk_router_fused(
        int(h.dtype == torch.float32), _lib.ptr(h), _lib.ptr(router), _lib.ptr(logits), h.shape[1], n, _lib.ptr(correction),
        _lib.ptr(idx), _lib.ptr(w), _lib.ptr(counts), _lib.ptr(place), T, experts, top, int(sigmoid), int(norm), float(scale),
        groups, keep, _lib.stream_ptr()), "router_fused")
    return logits, (idx, w, place)


def expert_rows_bound(tokens: int, top: int, experts: int) -> int:
    """Rows the padded expert segments of ``tokens`` tokens can take."""
    n = tokens * top
    return (n + min(n, experts) * (SEG - 1) + SEG - 1) // SEG * SEG


def expert_rows(h, counts, choice, place):
    """Copies every token's row into its experts' segments.  Returns ``(rows, dest [T, top] int32, offsets int32)``."""
    (T, K), E = choice.shape, counts.numel()
    bound = expert_rows_bound(T, K, E)
    dev = h.device
    out = torch.empty(bound, h.shape[1], dtype=h.dtype, device=dev)
    if not h.is_cuda:
        offsets = torch.zeros(E + 1, dtype=torch.int32)
        offsets[1:] = ((counts + SEG - 1) // SEG * SEG).cumsum(0)
        dest = offsets[choice] + place
        out.zero_()
        out[dest.reshape(-1).long()] = h.repeat_interleave(K, 0)
        return out, dest.to(torch.int32), offsets
    dest = torch.empty(T, K, dtype=torch.int32, device=dev)
    offsets = torch.empty(E + 1, dtype=torch.int32, device=dev)
    LAUNCHES["moe"] += 1
    _lib.check(_lib.kernels().gk_expert_rows(_lib.ptr(h), _lib.ptr(counts), _lib.ptr(choice), _lib.ptr(place),
                                             _lib.ptr(offsets), _lib.ptr(dest), _lib.ptr(out), T, K, E,
                                             h.shape[1] * h.element_size(), _lib.stream_ptr()), "expert_rows")
    return out, dest, offsets


def grouped(x, w, offsets):
    """``y[r] = x[r] @ w[g]^T`` for the rows of segment g; ``w`` [G, N, K]."""
    if x.is_cuda and x.dtype == torch.float32:
        G, N, K = w.shape
        y = torch.empty(x.shape[0], N, dtype=x.dtype, device=x.device)
        LAUNCHES["moe"] += 1
        _lib.check(_lib.kernels().gk_grouped_gemm_f32(_lib.ptr(x), _lib.ptr(w), _lib.ptr(y), _lib.ptr(offsets), G,
                                                      x.shape[0], N, K, _lib.stream_ptr()), "grouped_gemm_f32")
        return y
    return grouped_gemm(x, w, offsets, out_dtype=x.dtype)


def routed_experts(h, choice, up, down, counts, act: int = RELU2):
    """Every token through its chosen experts, ``down(relu(up h)^2)`` (RELU2) or ``down(silu(gate h) * up h)`` (SILU_GATE:
    ``up`` holds the gate rows, then the up rows): returns ``(rows, dest, weight)``, the experts' outputs in expert order and
    where a token finds its own."""
    idx, w, place = choice
    x, dest, offsets = expert_rows(h, counts, idx, place)
    a = grouped(x, up, offsets)
    F = down.shape[2]
    b = a if act == RELU2 else torch.empty(a.shape[0], F, dtype=a.dtype, device=a.device)
    activate(act, a, F, F if act == SILU_GATE else 0, b, n_rows=offsets[-1:])
    return grouped(b, down, offsets), dest, w
