"""Python front of mixtures of experts on dense banks of decoders with a 32-bit residual stream (``moe_*`` in
``gemv_dense.cu`` / ``stream_ops.cu``, grouped products in ``gemm_stream_tcgen05.cu``): clamped units behind a sigmoid
router, added to the stream, and silu-gated or clamped units behind a soft-max router with groups and a shared expert.

Every function launches on the current stream; there is no eager substitute.
"""
from __future__ import annotations

import torch

from ..native import cuda_api as api
from ..native.lib import current_stream, ptr, stream_lib
from .cuda_ops import error_flag
from .stream import (ACT_GLU, ACT_SILU_GLU, OUT_ACT, OUT_ADD, OUT_F32, ActArgs, _dt, _tile, gemm, gemm_ok, gemv_rows, glu_rows)

_NO_TABLE = (0, None, 0, 0, None)        # operands of activations that the grouped products do not have

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
                                    ptr(idx), T, bank.W, bank.I, 0, bank.E, k, ACT_GLU, bank.limit, 0.0, bank.alpha,
                                    16 if bank.interleaved else 0, 0, dt, int(pdl), st), "moe_glu_rows")
    api.check(lib.ipex_moe_down_rows(ptr(y), bank.I, ptr(bank.down), None, None, ptr(x), x.stride(0), ptr(idx), T, bank.W,
                                     bank.I, 0, bank.E, k, 1, dt, int(pdl), st), "moe_down_rows")
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
                                       OUT_ACT, ACT_GLU, bank.limit, bank.alpha, *_NO_TABLE, bt, dt, err, st), "gemm_stream(glu)")
        api.check(lib.ipex_gemm_stream(ptr(a), I, ptr(bank.down), I, ptr(y), W, None, None, 0, None, 0, None, ptr(ranges), E, S, W, I, OUT_ACT,
                                       0, 0.0, 0.0, *_NO_TABLE, bt, dt, err, st), "gemm_stream(down)")
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
# silu-gated or clamped units, soft-max router over groups, shared expert
# ------------------------------------------------------------------------------------------------
class SoftExpertBank:
    """``gate_up [E, 2 I, W]`` and ``shared_gate_up [2 Is, W]`` (gate and up rows alternating in blocks of eight where the
    hidden size is a multiple of eight, else gate rows first), ``down [E, W, I]``, ``shared_down [W, Is]``, ``router [E, W]``
    and, with a gated shared expert, its gate's row behind the router's (not ``shared_gated``: its weight is 1).

    ``act``: ``ACT_SILU_GLU``, or ``ACT_CLAMP_GLU`` with ``limit``, ``alpha`` and the shared expert's ``shared_limit``; ``bias
    [E]`` is added to the router's products."""

    def __init__(self, router, gate_up, down, top: int, groups: int = 1, keep: int = 1, scale: float = 1.0,
                 shared_gate_up=None, shared_down=None, act: int = ACT_SILU_GLU, limit: float = 0.0, alpha: float = 0.0,
                 shared_limit: float = 0.0, bias=None, shared_gated: bool = True):
        self.router, self.gate_up, self.down = router.contiguous(), gate_up.contiguous(), down.contiguous()
        self.top, self.groups, self.keep, self.scale = top, groups, keep, float(scale)
        self.E, self.I, self.W = gate_up.shape[0], gate_up.shape[1] // 2, gate_up.shape[2]
        self.shared = shared_down is not None
        self.shared_gated = self.shared and shared_gated
        self.shared_gate_up = shared_gate_up.contiguous() if self.shared else None
        self.shared_down = shared_down.contiguous() if self.shared else None
        self.Is = shared_down.shape[1] if self.shared else 0
        self.act, self.args = act, ActArgs(limit=float(limit), alpha=float(alpha))
        self.shared_args = ActArgs(limit=float(shared_limit), alpha=float(alpha))
        self.bias = None if bias is None else bias.float().contiguous()
        if self.router.shape[0] != self.E + self.shared_gated:
            raise ValueError(f"router of {self.router.shape[0]} rows for {self.E} experts (shared: {self.shared})")

    def rows_ok(self, tokens: int) -> bool:
        """A few tokens whose rows fit shared memory take the per-slot kernels."""
        size = self.router.element_size()
        return tokens <= 8 and max((max(self.I, self.Is) + 8) * (self.top + self.shared) * size,
                                   (self.W + 8) * size + (self.E + self.groups + 1) * 4) <= 200 * 1024


def soft_moe_rows(bank: SoftExpertBank, h, out, pdl=False, logits=None, add=False):
    """``out`` (fp32 rows) = (with ``add``: +=) the experts' weighted sum over a few normed rows ``h``: router, per-slot hidden
    units (the shared expert is one more slot), per-token down product.  ``logits``: finished products of the router (fp32),
    which banks with a bias or an ungated shared expert need."""
    lib, T, k, I, Is = stream_lib(), h.shape[0], bank.top + bank.shared, bank.I, bank.Is
    w = torch.empty(T, k, dtype=torch.float32, device=h.device)
    idx = torch.empty(T, k, dtype=torch.int64, device=h.device)
    ldy = (max(I, Is) + 7) // 8 * 8
    y = torch.empty(T * k, ldy, dtype=h.dtype, device=h.device)
    dt, st = _dt(h), current_stream()
    if logits is None and bank.bias is None and bank.shared_gated == bank.shared:
        api.check(lib.ipex_moe_router_softmax(ptr(h), h.stride(0), ptr(bank.router), ptr(w), ptr(idx), T, bank.W, bank.E,
                                              bank.groups, bank.keep, bank.top, int(bank.shared), bank.scale, dt, int(pdl),
                                              st), "moe_router_softmax")
    else:
        if logits is None:
            logits = gemv_rows(bank.router, h, torch.empty(T, bank.router.shape[0], dtype=torch.float32, device=h.device),
                               OUT_F32, pdl=pdl)
        if bank.shared_gated:
            raise NotImplementedError("a gated shared expert behind finished router products")
        _soft_topk(logits, bank, w, idx, None, bank.shared, pdl)
    api.check(lib.ipex_moe_glu_rows(ptr(h), h.stride(0), None, 0.0, ptr(bank.gate_up), ptr(bank.shared_gate_up), ptr(y), ldy,
                                    ptr(w), ptr(idx), T, bank.W, I, Is, bank.E, k, bank.act, bank.args.limit,
                                    bank.shared_args.limit, bank.args.alpha, 0 if I % 8 else 8, 0 if Is % 8 else 8, dt,
                                    int(pdl), st), "moe_glu_rows")
    api.check(lib.ipex_moe_down_rows(ptr(y), ldy, ptr(bank.down), ptr(bank.shared_down), ptr(w), ptr(out), out.stride(0),
                                     ptr(idx), T, bank.W, I, Is, bank.E, k, int(add), dt, int(pdl), st), "moe_down_rows")
    return out


def _soft_topk(logits, bank: SoftExpertBank, w, idx, gate, always: bool, pdl=False):
    rc = stream_lib().ipex_moe_softmax_grouped_topk(ptr(logits), logits.stride(0), ptr(bank.bias), ptr(w), ptr(idx), w.shape[1],
                                                    ptr(gate), int(always), logits.shape[0], bank.E, bank.groups, bank.keep,
                                                    bank.top, bank.scale, int(pdl), current_stream())
    api.check(rc, "moe_softmax_grouped_topk")


def soft_topk(logits, bank: SoftExpertBank):
    """fp32 router logits ``[T, E (+ 1)]`` -> weights and experts ``[T, top]``, and a gated shared expert's gate ``[T]``."""
    T, dev = logits.shape[0], logits.device
    w = torch.empty(T, bank.top, dtype=torch.float32, device=dev)
    idx = torch.empty(T, bank.top, dtype=torch.int64, device=dev)
    gate = torch.empty(T, dtype=torch.float32, device=dev) if bank.shared_gated else None
    _soft_topk(logits, bank, w, idx, gate, False)
    return w, idx, gate


def soft_moe_grouped(bank: SoftExpertBank, h, out, logits=None, add=False):
    """``soft_moe_rows`` for many rows: slots grouped by expert on the device, one grouped GEMM per half of the bank, the
    shared expert's products beside them."""
    h = h.contiguous()
    lib, T, dev, dtype = stream_lib(), h.shape[0], h.device, h.dtype
    S, W, I, E = T * bank.top, bank.W, bank.I, bank.E
    if logits is None:
        logits = gemm(h, bank.router, torch.empty(T, bank.router.shape[0], dtype=torch.float32, device=dev), OUT_F32)
    w, idx, gate = soft_topk(logits, bank)
    if bank.shared_gated and add:
        raise NotImplementedError("a gated shared expert added to what is there")
    if bank.shared:
        u = torch.empty(T, (bank.Is + 7) // 8 * 8, dtype=dtype, device=dev)[:, :bank.Is]
        gemm(h, bank.shared_gate_up, u, OUT_ACT, bank.act, None, bank.Is % 8 == 0, args=bank.shared_args)
        gemm(u, bank.shared_down, out, OUT_ADD if add else OUT_F32)
    inverse, ranges, hs, _ = _group(h, w, idx, E)
    dt, st = _dt(h), current_stream()
    a = torch.empty(S, I, dtype=dtype, device=dev)
    y = torch.empty(S, W, dtype=dtype, device=dev)
    if I % 8 == 0 and gemm_ok(hs, bank.gate_up) and gemm_ok(a, bank.down):
        err, bt = ptr(error_flag(dev)), _tile(S / E * 1.25)
        api.check(lib.ipex_gemm_stream(ptr(hs), W, ptr(bank.gate_up), W, ptr(a), I, None, None, 0, None, 0, None, ptr(ranges),
                                       E, S, 2 * I, W, OUT_ACT, bank.act, bank.args.limit, bank.args.alpha, *_NO_TABLE, bt, dt,
                                       err, st), "gemm_stream(glu)")
        api.check(lib.ipex_gemm_stream(ptr(a), I, ptr(bank.down), I, ptr(y), W, None, None, 0, None, 0, None, ptr(ranges), E,
                                       S, W, I, OUT_ACT, 0, 0.0, 0.0, *_NO_TABLE, bt, dt, err, st), "gemm_stream(down)")
    else:
        gu = torch.empty(S, 2 * I, dtype=torch.float32, device=dev)
        api.check(lib.ipex_gemm_plain(ptr(hs), ptr(bank.gate_up), ptr(gu), ptr(ranges), E, S, 2 * I, W, 1, dt, st),
                  "gemm_plain")
        glu_rows(gu, None, a, bank.act, I % 8 == 0, bank.args)
        api.check(lib.ipex_gemm_plain(ptr(a), ptr(bank.down), ptr(y), ptr(ranges), E, S, W, I, 0, dt, st), "gemm_plain")
    api.check(lib.ipex_moe_combine_weighted(ptr(y), ptr(inverse), ptr(w), ptr(gate), ptr(out), T, W, bank.top,
                                            int(add or (bank.shared and not bank.shared_gated)), dt, st),
              "moe_combine_weighted")
    return out
