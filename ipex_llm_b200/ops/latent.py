"""Python front of the kernels of multi-head latent attention (``latent_attn.cu``), beside what latent-attention decoders
share with the other decoders on a 32-bit residual stream (``ops/stream.py``, ``ops/dense_moe.py``).

Every function launches on the current stream; there is no eager substitute.
"""
from __future__ import annotations

import torch

from ..native import cuda_api as api
from ..native.lib import current_stream, ptr, stream_lib
from .cuda_ops import error_flag
from .dense_moe import ExpertBank, moe_grouped, moe_rows, sigmoid_topk
from .stream import (ACT_GELU_GLU, ACT_GLU, ACT_NONE, ACT_RELU2, OUT_ACT, OUT_ADD, OUT_F32, _dt, add_stream_,
                     argmax_rows, embed_stream, gemm, gemm_ok, gemv_rows, norm_stream, relu2_, rows_max, softcap_)

__all__ = ["ACT_GELU_GLU", "ACT_GLU", "ACT_NONE", "ACT_RELU2", "OUT_ACT", "OUT_ADD", "OUT_F32", "ExpertBank", "LatentSpec",
           "add_stream_", "argmax_rows", "embed_stream", "gemm", "gemm_ok", "gemv_rows", "latent_prompt", "latent_step",
           "moe_grouped", "moe_rows", "norm_stream", "pick_latent_splits", "relu2_", "rotary_table", "rows_max",
           "sigmoid_topk", "softcap_"]


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


BEHIND = object()        # the latent rows follow the queries in the same projection


def _kv_rows(spec: LatentSpec, qkv, kv):
    return qkv[:, spec.heads * (spec.dim + spec.rot_dim):] if kv is BEHIND else kv


def _gate_args(gate, s: int = 0):
    return (None, 0) if gate is None else (gate[s:], gate.stride(0))


def latent_step(spec: LatentSpec, qkv, w_uk, w_uv, kv_norm, cos, sin, slot, pos, cache, layer_idx: int, out,
                visible: int, pdl=False, generic=False, kv=BEHIND, gate=None):
    """Absorbed attention of query tokens against the cache, which gets their own rows first.  ``qkv [M, ...]`` is
    the fused projection (its query parts are rotated in place), ``out [M, H * vd]``; ``visible`` bounds the number of
    keys a token can see (it sizes the split, nothing else).  ``kv``: the latent rows when they are not behind the
    queries; None when cache layer ``layer_idx`` holds them already (rows of an earlier layer).  ``gate [M, H * vd]``:
    outputs times its sigmoid."""
    lib = stream_lib("latent")
    rows = cache.layers[layer_idx]._k
    M, H, R = qkv.shape[0], spec.heads, spec.rank
    kv = _kv_rows(spec, qkv, kv)
    dt, st = _dt(qkv), current_stream()
    step = 1024                                  # tokens per attention launch: bounds the scratch of long portions
    qabs = torch.empty(M, H, R, dtype=qkv.dtype, device=qkv.device)
    for s in range(0, M, 65535):
        e = min(M, s + 65535)
        api.check(lib.ipex_latent_prep(ptr(qkv[s:]), qkv.stride(0), ptr(None if kv is None else kv[s:]),
                                       0 if kv is None else kv.stride(0), ptr(kv_norm), spec.eps, ptr(w_uk), ptr(cos),
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
        g, ldg = _gate_args(gate, s)
        api.check(lib.ipex_latent_uv(ptr(o), ptr(ml), ptr(w_uv), ptr(g), ldg, ptr(out[s:]), out.stride(0), m, H, R, spec.v_dim,
                                     nsplit, dt, int(pdl), st), "latent_uv")
    return out


def prompt_rows(spec: LatentSpec, tokens: int, dtype, device):
    """Room for the latents and rotated key parts of a packed batch of prompts."""
    return (torch.empty(tokens, spec.rank, dtype=dtype, device=device),
            torch.empty(tokens, max(8, spec.rot_dim), dtype=dtype, device=device))


def latent_prompt(spec: LatentSpec, qkv, w_uk, w_uv, kv_norm, cos, sin, slot, pos, seq_row, seq_len, max_len: int,
                  cache, layer_idx: int, out, kv=BEHIND, gate=None, rows_out=None):
    """Attention of whole prompts, packed one behind the other (``seq_row`` / ``seq_len``: int32, first row and length
    of each): keys and values are expanded from the latents, then the tcgen05 kernel; the cache gets the latents.
    ``kv``, ``gate``: see ``latent_step``.  ``rows_out`` (``prompt_rows``): filled with the tokens' latents and key parts,
    or, with ``kv`` None, holding those of the layer whose rows this one uses."""
    lib = stream_lib("latent")
    rows = cache.layers[layer_idx]._k
    T, H, R, dev, dtype = qkv.shape[0], spec.heads, spec.rank, qkv.device, qkv.dtype
    dt, st = _dt(qkv), current_stream()
    kv = _kv_rows(spec, qkv, kv)
    c, kr = prompt_rows(spec, T, dtype, dev) if rows_out is None else rows_out
    api.check(lib.ipex_latent_prompt_prep(ptr(qkv), qkv.stride(0), ptr(kv), 0 if kv is None else kv.stride(0), ptr(kv_norm), spec.eps, ptr(cos), ptr(sin), ptr(slot),
                                          ptr(pos), ptr(cache.start), ptr(rows), rows.stride(0), rows.stride(2), ptr(c),
                                          R, ptr(kr), kr.stride(0), T, H, spec.dim, spec.rot_dim, R, spec.pairs, dt, 0,
                                          st), "latent_prompt_prep")
    k = torch.empty(T, H * spec.dim, dtype=dtype, device=dev)
    gemm(c, w_uk, k, OUT_ACT)
    ld = (T + 7) // 8 * 8
    vt = torch.empty(H * spec.v_dim, ld, dtype=dtype, device=dev)
    gemm(w_uv, c, vt, OUT_ACT)                    # V transposed: rows are value dimensions, columns tokens
    g, ldg = _gate_args(gate)
    rc = stream_lib().ipex_packed_prefill(ptr(qkv), qkv.stride(0), ptr(k), k.stride(0), ptr(kr), kr.stride(0), ptr(vt), ld,
                                          ptr(out), out.stride(0), ptr(seq_row), ptr(seq_len), seq_row.shape[0], H, H, T,
                                          max_len, spec.dim, spec.rot_dim, spec.v_dim, spec.window, 0, 0, None, ptr(g), ldg,
                                          1.0, 0, None, 0, None, 0, None, 0, spec.scale, dt, ptr(error_flag(dev)), st)
    if rc == -1:
        raise RuntimeError("ipex_llm_b200: the driver's tensor-map encoder rejected the attention operands")
    api.check(rc, "packed_prefill")
    return out
