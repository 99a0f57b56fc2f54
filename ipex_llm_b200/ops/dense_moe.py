"""Python front of mixtures of experts on dense banks of decoders with a 32-bit residual stream (``moe_*`` in
``gemv_dense.cu`` / ``stream_ops.cu``, grouped products in ``gemm_stream_tcgen05.cu``): clamped units behind a sigmoid
router, added to the stream, and silu-gated units behind a soft-max router with groups and a gated shared expert.

Every function launches on the current stream; there is no eager substitute.
"""
from __future__ import annotations

import torch

from ..native import cuda_api as api
from ..native.lib import current_stream, ptr, stream_lib
from .cuda_ops import error_flag
from .stream import ACT_GLU, ACT_SILU_GLU, OUT_ACT, OUT_F32, _dt, _tile, gemm, gemm_ok, glu_rows

# ------------------------------------------------------------------------------------------------
# clamped units, sigmoid router
# ------------------------------------------------------------------------------------------------
class ExpertBank:
    """Dense experts with a clamped gated unit: ``gate_up [E, 2 I, W]`` (``interleaved``: gate and up rows alternate in
    16-row tiles), ``down [E, W, I]``, ``router [E, W]``."""

    def __init__(self, router, gate_up, down, top: int, limit: float, alpha: float, interleaved: bool):
        self.router, self.gate_up, self.down = router.contiguous(), gate_up.contiguous(), down.contiguous()
        self.top, self.limit, self.alpha, self.interleaved = top, limit, alpha, interleaved
        self.E, self.I, self.W = gate_up.shape[0], gate_up.shape[1] // 2, gate_up.shape[2]

    def rows_ok(self, tokens: int) -> bool:
        """A few tokens whose rows fit shared memory take the per-slot kernels."""
        size = self.router.element_size()
        return tokens <= 8 and max((self.I + 8) * self.top * size, (self.W + self.E) * 4) <= 200 * 1024


def moe_rows(bank: ExpertBank, x, norm, eps: float, pdl=False):
    """``x += experts(norm(x))`` for a few rows: router with its norm, per-slot hidden units, per-token down product."""
    lib, T, k = stream_lib(), x.shape[0], bank.top
    w = torch.empty(T, k, dtype=torch.float32, device=x.device)
    idx = torch.empty(T, k, dtype=torch.int64, device=x.device)
    y = torch.empty(T * k, bank.I, dtype=bank.router.dtype, device=x.device)
    dt, st = _dt(bank.router), current_stream()
    api.check(lib.ipex_moe_router_sigmoid(ptr(x), x.stride(0), ptr(norm), eps, ptr(bank.router), ptr(w), ptr(idx), T,
                                          bank.W, bank.E, k, dt, int(pdl), st), "moe_router_sigmoid")
    api.check(lib.ipex_moe_glu_rows(ptr(x), x.stride(0), ptr(norm), eps, ptr(bank.gate_up), None, ptr(y), bank.I, ptr(w),
                                    ptr(idx), T, bank.W, bank.I, 0, bank.E, k, ACT_GLU, bank.limit, bank.alpha,
                                    16 if bank.interleaved else 0, 0, dt, int(pdl), st), "moe_glu_rows")
    api.check(lib.ipex_moe_down_rows(ptr(y), bank.I, ptr(bank.down), None, None, ptr(x), x.stride(0), ptr(idx), T, bank.W,
                                     bank.I, 0, bank.E, k, dt, int(pdl), st), "moe_down_rows")
    return x


def sigmoid_topk(logits, k: int):
    """fp32 router logits ``[T, E]`` -> (weights, experts) of the ``k`` largest sigmoid scores, not renormalised."""
    T, E = logits.shape
    w = torch.empty(T, k, dtype=torch.float32, device=logits.device)
    idx = torch.empty(T, k, dtype=torch.int64, device=logits.device)
    rc = stream_lib().ipex_moe_sigmoid_topk(ptr(logits), logits.stride(0), ptr(w), ptr(idx), T, E, k, current_stream())
    api.check(rc, "moe_sigmoid_topk")
    return w, idx


def _group(h, w, idx, E: int):
    """Rows and weights of the (token, choice) slots in the order of their experts, every slot's place, and the experts'
    row ranges."""
    lib, (T, k), W, dev = stream_lib(), idx.shape, h.shape[1], h.device
    S, dt, st = T * k, _dt(h), current_stream()
    order = torch.empty(S, dtype=torch.int32, device=dev)
    inverse = torch.empty(S, dtype=torch.int32, device=dev)
    ranges = torch.empty(E, 2, dtype=torch.int32, device=dev)
    api.check(lib.ipex_moe_group_slots(ptr(idx), S, E, ptr(order), ptr(inverse), ptr(ranges), st), "moe_group_slots")
    hs = torch.empty(S, W, dtype=h.dtype, device=dev)
    ws = torch.empty(S, dtype=torch.float32, device=dev)
    api.check(lib.ipex_moe_gather_slots(ptr(h), ptr(w), ptr(order), ptr(hs), ptr(ws), S, W, k, dt, st), "moe_gather")
    return inverse, ranges, hs, ws


def moe_grouped(bank: ExpertBank, x, h):
    """``x += experts(h)`` for many rows ``h`` (normed): slots grouped by expert on the device, then one grouped GEMM
    per half of the bank."""
    lib, T, k, dev, dtype = stream_lib(), h.shape[0], bank.top, h.device, h.dtype
    S, W, I, E = T * k, bank.W, bank.I, bank.E
    logits = torch.empty(T, E, dtype=torch.float32, device=dev)
    gemm(h, bank.router, logits, OUT_F32)
    w, idx = sigmoid_topk(logits, k)
    dt, st = _dt(h), current_stream()
    inverse, ranges, hs, ws = _group(h, w, idx, E)
    a = torch.empty(S, I, dtype=dtype, device=dev)
    y = torch.empty(S, W, dtype=dtype, device=dev)
    if bank.interleaved and gemm_ok(hs, bank.gate_up) and gemm_ok(a, bank.down):
        err, bt = ptr(error_flag(dev)), _tile(S / E * 1.25)
        api.check(lib.ipex_gemm_stream(ptr(hs), W, ptr(bank.gate_up), W, ptr(a), I, None, None, 0, None, 0, ptr(ws), ptr(ranges), E, S, 2 * I, W,
                                       OUT_ACT, ACT_GLU, bank.limit, bank.alpha, bt, dt, err, st), "gemm_stream(glu)")
        api.check(lib.ipex_gemm_stream(ptr(a), I, ptr(bank.down), I, ptr(y), W, None, None, 0, None, 0, None, ptr(ranges), E, S, W, I, OUT_ACT,
                                       0, 0.0, 0.0, bt, dt, err, st), "gemm_stream(down)")
    else:
        gu = torch.empty(S, 2 * I, dtype=torch.float32, device=dev)
        api.check(lib.ipex_gemm_plain(ptr(hs), ptr(bank.gate_up), ptr(gu), ptr(ranges), E, S, 2 * I, W, 1, dt, st),
                  "gemm_plain")
        api.check(lib.ipex_moe_glu_from_gu(ptr(gu), ptr(ws), ptr(a), S, I, bank.limit, bank.alpha,
                                           int(bank.interleaved), dt, st), "moe_glu")
        api.check(lib.ipex_gemm_plain(ptr(a), ptr(bank.down), ptr(y), ptr(ranges), E, S, W, I, 0, dt, st), "gemm_plain")
    api.check(lib.ipex_moe_combine_slots(ptr(y), ptr(inverse), ptr(x), T, W, k, dt, st), "moe_combine_slots")
    return x


# ------------------------------------------------------------------------------------------------
# silu-gated units, soft-max router over groups, shared expert
# ------------------------------------------------------------------------------------------------
class SoftExpertBank:
    """``gate_up [E, 2 I, W]`` and ``shared_gate_up [2 Is, W]`` (gate and up rows alternating in blocks of eight where the
    hidden size is a multiple of eight, else gate rows first), ``down [E, W, I]``, ``shared_down [W, Is]``, ``router [E, W]``
    and, with a shared expert, its gate's row behind the router's."""

    def __init__(self, router, gate_up, down, top: int, groups: int = 1, keep: int = 1, scale: float = 1.0,
                 shared_gate_up=None, shared_down=None):
        self.router, self.gate_up, self.down = router.contiguous(), gate_up.contiguous(), down.contiguous()
        self.top, self.groups, self.keep, self.scale = top, groups, keep, float(scale)
        self.E, self.I, self.W = gate_up.shape[0], gate_up.shape[1] // 2, gate_up.shape[2]
        self.shared = shared_down is not None
        self.shared_gate_up = shared_gate_up.contiguous() if self.shared else None
        self.shared_down = shared_down.contiguous() if self.shared else None
        self.Is = shared_down.shape[1] if self.shared else 0
        if self.router.shape[0] != self.E + self.shared:
            raise ValueError(f"router of {self.router.shape[0]} rows for {self.E} experts (shared: {self.shared})")

    def rows_ok(self, tokens: int) -> bool:
        """A few tokens whose rows fit shared memory take the per-slot kernels."""
        size = self.router.element_size()
        return tokens <= 8 and max((max(self.I, self.Is) + 8) * (self.top + self.shared) * size,
                                   (self.W + 8) * size + (self.E + self.groups + 1) * 4) <= 200 * 1024


def soft_moe_rows(bank: SoftExpertBank, h, out, pdl=False):
    """``out`` (fp32 rows) = the experts' weighted sum over a few normed rows ``h``: router, per-slot hidden units (the
    shared expert is one more slot), per-token down product."""
    lib, T, k, I, Is = stream_lib(), h.shape[0], bank.top + bank.shared, bank.I, bank.Is
    w = torch.empty(T, k, dtype=torch.float32, device=h.device)
    idx = torch.empty(T, k, dtype=torch.int64, device=h.device)
    ldy = (max(I, Is) + 7) // 8 * 8
    y = torch.empty(T * k, ldy, dtype=h.dtype, device=h.device)
    dt, st = _dt(h), current_stream()
    api.check(lib.ipex_moe_router_softmax(ptr(h), h.stride(0), ptr(bank.router), ptr(w), ptr(idx), T, bank.W, bank.E,
                                          bank.groups, bank.keep, bank.top, int(bank.shared), bank.scale, dt, int(pdl), st),
              "moe_router_softmax")
    api.check(lib.ipex_moe_glu_rows(ptr(h), h.stride(0), None, 0.0, ptr(bank.gate_up), ptr(bank.shared_gate_up), ptr(y), ldy,
                                    ptr(w), ptr(idx), T, bank.W, I, Is, bank.E, k, ACT_SILU_GLU, 0.0, 0.0,
                                    0 if I % 8 else 8, 0 if Is % 8 else 8, dt, int(pdl), st), "moe_glu_rows")
    api.check(lib.ipex_moe_down_rows(ptr(y), ldy, ptr(bank.down), ptr(bank.shared_down), ptr(w), ptr(out), out.stride(0),
                                     ptr(idx), T, bank.W, I, Is, bank.E, k, dt, int(pdl), st), "moe_down_rows")
    return out


def soft_topk(logits, bank: SoftExpertBank):
    """fp32 router logits ``[T, E (+ 1)]`` -> weights and experts ``[T, top]``, and the shared expert's gate ``[T]``."""
    T, dev = logits.shape[0], logits.device
    w = torch.empty(T, bank.top, dtype=torch.float32, device=dev)
    idx = torch.empty(T, bank.top, dtype=torch.int64, device=dev)
    gate = torch.empty(T, dtype=torch.float32, device=dev) if bank.shared else None
    rc = stream_lib().ipex_moe_softmax_grouped_topk(ptr(logits), logits.stride(0), ptr(w), ptr(idx), ptr(gate), T, bank.E,
                                                    bank.groups, bank.keep, bank.top, bank.scale, current_stream())
    api.check(rc, "moe_softmax_grouped_topk")
    return w, idx, gate


def soft_moe_grouped(bank: SoftExpertBank, h, out):
    """``soft_moe_rows`` for many rows: slots grouped by expert on the device, one grouped GEMM per half of the bank, the
    shared expert's products beside them."""
    h = h.contiguous()
    lib, T, dev, dtype = stream_lib(), h.shape[0], h.device, h.dtype
    S, W, I, E = T * bank.top, bank.W, bank.I, bank.E
    w, idx, gate = soft_topk(gemm(h, bank.router, torch.empty(T, E + bank.shared, dtype=torch.float32, device=dev), OUT_F32),
                             bank)
    if bank.shared:
        u = torch.empty(T, (bank.Is + 7) // 8 * 8, dtype=dtype, device=dev)[:, :bank.Is]
        gemm(h, bank.shared_gate_up, u, OUT_ACT, ACT_SILU_GLU, None, bank.Is % 8 == 0)
        gemm(u, bank.shared_down, out, OUT_F32)
    inverse, ranges, hs, _ = _group(h, w, idx, E)
    dt, st = _dt(h), current_stream()
    a = torch.empty(S, I, dtype=dtype, device=dev)
    y = torch.empty(S, W, dtype=dtype, device=dev)
    if I % 8 == 0 and gemm_ok(hs, bank.gate_up) and gemm_ok(a, bank.down):
        err, bt = ptr(error_flag(dev)), _tile(S / E * 1.25)
        api.check(lib.ipex_gemm_stream(ptr(hs), W, ptr(bank.gate_up), W, ptr(a), I, None, None, 0, None, 0, None, ptr(ranges),
                                       E, S, 2 * I, W, OUT_ACT, ACT_SILU_GLU, 0.0, 0.0, bt, dt, err, st), "gemm_stream(glu)")
        api.check(lib.ipex_gemm_stream(ptr(a), I, ptr(bank.down), I, ptr(y), W, None, None, 0, None, 0, None, ptr(ranges), E,
                                       S, W, I, OUT_ACT, 0, 0.0, 0.0, bt, dt, err, st), "gemm_stream(down)")
    else:
        gu = torch.empty(S, 2 * I, dtype=torch.float32, device=dev)
        api.check(lib.ipex_gemm_plain(ptr(hs), ptr(bank.gate_up), ptr(gu), ptr(ranges), E, S, 2 * I, W, 1, dt, st),
                  "gemm_plain")
        glu_rows(gu, None, a, ACT_SILU_GLU, I % 8 == 0)
        api.check(lib.ipex_gemm_plain(ptr(a), ptr(bank.down), ptr(y), ptr(ranges), E, S, W, I, 0, dt, st), "gemm_plain")
    api.check(lib.ipex_moe_combine_weighted(ptr(y), ptr(inverse), ptr(w), ptr(gate), ptr(out), T, W, bank.top, dt, st),
              "moe_combine_weighted")
    return out
