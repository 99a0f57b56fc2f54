"""Python front of the kernels of latent-attention decoders: a dense expert bank and multi-head latent attention (see
``moe_*`` in ``gemv_dense.cu`` / ``stream_ops.cu`` and the ``latent_*.cu`` files), beside what they share with the other
decoders on a 32-bit residual stream (``ops/stream.py``).

Every function launches on the current stream; there is no eager substitute.
"""
from __future__ import annotations

import torch

from ..native import cuda_api as api
from ..native.lib import current_stream, ptr, stream_lib
from .cuda_ops import error_flag
from .stream import (ACT_GELU_GLU, ACT_GLU, ACT_NONE, ACT_RELU2, OUT_ACT, OUT_ADD, OUT_F32, _dt, _tile, add_stream_,
                     argmax_rows, embed_stream, gemm, gemm_ok, gemv_rows, norm_stream, relu2_, rows_max, softcap_)

__all__ = ["ACT_GELU_GLU", "ACT_GLU", "ACT_NONE", "ACT_RELU2", "OUT_ACT", "OUT_ADD", "OUT_F32", "ExpertBank", "LatentSpec",
           "add_stream_", "argmax_rows", "embed_stream", "gemm", "gemm_ok", "gemv_rows", "latent_prompt", "latent_step",
           "moe_grouped", "moe_rows", "norm_stream", "pick_latent_splits", "relu2_", "rotary_table", "rows_max",
           "sigmoid_topk", "softcap_"]


# ------------------------------------------------------------------------------------------------
# mixture of experts on a dense bank
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
    api.check(lib.ipex_moe_glu_rows(ptr(x), x.stride(0), ptr(norm), eps, ptr(bank.gate_up), ptr(y), ptr(w), ptr(idx), T,
                                    bank.W, bank.I, bank.E, k, bank.limit, bank.alpha, int(bank.interleaved), dt,
                                    int(pdl), st), "moe_glu_rows")
    api.check(lib.ipex_moe_down_rows(ptr(y), ptr(bank.down), ptr(x), x.stride(0), ptr(idx), T, bank.W, bank.I, bank.E, k,
                                     dt, int(pdl), st), "moe_down_rows")
    return x


def sigmoid_topk(logits, k: int):
    """fp32 router logits ``[T, E]`` -> (weights, experts) of the ``k`` largest sigmoid scores, not renormalised."""
    T, E = logits.shape
    w = torch.empty(T, k, dtype=torch.float32, device=logits.device)
    idx = torch.empty(T, k, dtype=torch.int64, device=logits.device)
    rc = stream_lib().ipex_moe_sigmoid_topk(ptr(logits), logits.stride(0), ptr(w), ptr(idx), T, E, k, current_stream())
    api.check(rc, "moe_sigmoid_topk")
    return w, idx


def moe_grouped(bank: ExpertBank, x, h):
    """``x += experts(h)`` for many rows ``h`` (normed): slots grouped by expert on the device, then one grouped GEMM
    per half of the bank."""
    lib, T, k, dev, dtype = stream_lib(), h.shape[0], bank.top, h.device, h.dtype
    S, W, I, E = T * k, bank.W, bank.I, bank.E
    logits = torch.empty(T, E, dtype=torch.float32, device=dev)
    gemm(h, bank.router, logits, OUT_F32)
    w, idx = sigmoid_topk(logits, k)
    order = torch.empty(S, dtype=torch.int32, device=dev)
    inverse = torch.empty(S, dtype=torch.int32, device=dev)
    ranges = torch.empty(E, 2, dtype=torch.int32, device=dev)
    dt, st = _dt(h), current_stream()
    api.check(lib.ipex_moe_group_slots(ptr(idx), S, E, ptr(order), ptr(inverse), ptr(ranges), st), "moe_group_slots")
    hs = torch.empty(S, W, dtype=dtype, device=dev)
    ws = torch.empty(S, dtype=torch.float32, device=dev)
    api.check(lib.ipex_moe_gather_slots(ptr(h), ptr(w), ptr(order), ptr(hs), ptr(ws), S, W, k, dt, st), "moe_gather")
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
# latent attention
# ------------------------------------------------------------------------------------------------
def rotary_table(positions: int, base: float, pairs: int, device):
    """cos / sin of ``position * base^(-2i / (2 pairs))``, angles formed in 64-bit, fp32 ``[positions, pairs]``."""
    f = torch.tensor(base, dtype=torch.float64) ** (-torch.arange(pairs, dtype=torch.float64) / max(pairs, 1))
    a = torch.arange(positions, dtype=torch.float64)[:, None] * f[None, :]
    return a.cos().float().to(device).contiguous(), a.sin().float().to(device).contiguous()


class LatentSpec:
    """Sizes and constants of one latent-attention layer."""

    def __init__(self, heads, dim, rot_dim, v_dim, rank, scale, window, pairs, eps):
        self.heads, self.dim, self.rot_dim, self.v_dim, self.rank = heads, dim, rot_dim, v_dim, rank
        self.scale, self.window, self.pairs, self.eps = scale, window, pairs, eps

    def row(self, dtype) -> int:
        return int(stream_lib("latent").ipex_latent_row(self.rank, self.rot_dim, _dt(dtype)))

    def prefill_ok(self, dtype) -> bool:
        return bool(stream_lib().ipex_packed_prefill_ok(self.dim, self.rot_dim, self.v_dim, self.rank, _dt(dtype)))


def pick_latent_splits(tokens: int, heads: int, visible: int, n_sm: int = 148) -> int:
    """Parts the visible keys of a query token are split into: one CTA per SM in a single wave, at least 64 keys each
    (every part costs the merge a read of its partial output)."""
    groups = -(-heads // 32)
    return max(1, min(n_sm // max(1, tokens * groups), -(-visible // 64), 32))


def latent_step(spec: LatentSpec, qkv, w_uk, w_uv, kv_norm, cos, sin, slot, pos, cache, layer_idx: int, out,
                visible: int, pdl=False, generic=False):
    """Absorbed attention of query tokens against the cache, which gets their own rows first.  ``qkv [M, ...]`` is
    the fused projection (its query parts are rotated in place), ``out [M, H * vd]``; ``visible`` bounds the number of
    keys a token can see (it sizes the split, nothing else)."""
    lib = stream_lib("latent")
    rows = cache.layers[layer_idx]._k
    M, H, R = qkv.shape[0], spec.heads, spec.rank
    dt, st = _dt(qkv), current_stream()
    step = 1024                                  # tokens per attention launch: bounds the scratch of long portions
    qabs = torch.empty(M, H, R, dtype=qkv.dtype, device=qkv.device)
    for s in range(0, M, 65535):
        e = min(M, s + 65535)
        api.check(lib.ipex_latent_prep(ptr(qkv[s:]), qkv.stride(0), ptr(kv_norm), spec.eps, ptr(w_uk), ptr(cos),
                                       ptr(sin), ptr(slot[s:]), ptr(pos[s:]), ptr(cache.start), ptr(rows),
                                       rows.stride(0), rows.stride(2), ptr(qabs[s:]), e - s, H, spec.dim, spec.rot_dim,
                                       R, spec.pairs, dt, int(pdl), st), "latent_prep")
    nsplit = pick_latent_splits(min(M, step), H, visible)
    n = min(M, step)
    o = torch.empty(n, nsplit, H, R, dtype=torch.float32, device=qkv.device)
    ml = torch.empty(n, nsplit, H, 2, dtype=torch.float32, device=qkv.device)
    for s in range(0, M, step):
        m = min(step, M - s)
        api.check(lib.ipex_latent_attn(ptr(qabs[s:]), ptr(qkv[s:]), qkv.stride(0), ptr(rows), rows.stride(0),
                                       rows.stride(2), ptr(slot[s:]), ptr(pos[s:]), ptr(cache.start), ptr(o), ptr(ml),
                                       m, H, spec.dim, spec.rot_dim, R, spec.window, nsplit, spec.scale, int(generic),
                                       dt, int(pdl), st), "latent_attn")
        api.check(lib.ipex_latent_uv(ptr(o), ptr(ml), ptr(w_uv), ptr(out[s:]), out.stride(0), m, H, R, spec.v_dim,
                                     nsplit, dt, int(pdl), st), "latent_uv")
    return out


def latent_prompt(spec: LatentSpec, qkv, w_uk, w_uv, kv_norm, cos, sin, slot, pos, seq_row, seq_len, max_len: int,
                  cache, layer_idx: int, out):
    """Attention of whole prompts, packed one behind the other (``seq_row`` / ``seq_len``: int32, first row and length
    of each): keys and values are expanded from the latents, then the tcgen05 kernel; the cache gets the latents."""
    lib = stream_lib("latent")
    rows = cache.layers[layer_idx]._k
    T, H, R, dev, dtype = qkv.shape[0], spec.heads, spec.rank, qkv.device, qkv.dtype
    dt, st = _dt(qkv), current_stream()
    c = torch.empty(T, R, dtype=dtype, device=dev)
    kr = torch.empty(T, max(8, spec.rot_dim), dtype=dtype, device=dev)
    api.check(lib.ipex_latent_prompt_prep(ptr(qkv), qkv.stride(0), ptr(kv_norm), spec.eps, ptr(cos), ptr(sin), ptr(slot),
                                          ptr(pos), ptr(cache.start), ptr(rows), rows.stride(0), rows.stride(2), ptr(c),
                                          R, ptr(kr), kr.stride(0), T, H, spec.dim, spec.rot_dim, R, spec.pairs, dt, 0,
                                          st), "latent_prompt_prep")
    k = torch.empty(T, H * spec.dim, dtype=dtype, device=dev)
    gemm(c, w_uk, k, OUT_ACT)
    ld = (T + 7) // 8 * 8
    vt = torch.empty(H * spec.v_dim, ld, dtype=dtype, device=dev)
    gemm(w_uv, c, vt, OUT_ACT)                    # V transposed: rows are value dimensions, columns tokens
    rc = stream_lib().ipex_packed_prefill(ptr(qkv), qkv.stride(0), ptr(k), k.stride(0), ptr(kr), kr.stride(0), ptr(vt), ld,
                                          ptr(out), out.stride(0), ptr(seq_row), ptr(seq_len), seq_row.shape[0], H, H, T,
                                          max_len, spec.dim, spec.rot_dim, spec.v_dim, spec.window, 0, spec.scale, dt,
                                          ptr(error_flag(dev)), st)
    if rc == -1:
        raise RuntimeError("ipex_llm_b200: the driver's tensor-map encoder rejected the attention operands")
    api.check(rc, "packed_prefill")
    return out
