"""Python front of the kernels that decoders with a 32-bit residual stream share: row products and GEMMs that read or
add to the stream, embedding, norms, arg-max (see the ``.cu`` files of the "stream" component).

Every function launches on the current stream; there is no eager substitute.  The stream is ``x [tokens, width]`` fp32;
``dtype`` below is the weight and activation dtype (fp16, bf16 or fp32).
"""
from __future__ import annotations

from contextlib import contextmanager
from dataclasses import dataclass
from typing import Optional

import torch

from ..native import cuda_api as api
from ..native.lib import current_stream, ptr, stream_lib
from .cuda_ops import error_flag

OUT_ACT, OUT_ADD, OUT_F32 = 0, 1, 2        # activation dtype / added to the stream / fp32
ACT_NONE, ACT_RELU2 = 0, 1
ACT_GLU, ACT_GELU_GLU, ACT_SILU_GLU = 2, 3, 4     # grouped GEMM only / gate and up rows in blocks of eight
ACT_CLAMP_GLU, ACT_GELU_MUL = 5, 6               # likewise / gelu_tanh times the token's row of a table
GATED_ACTS = (ACT_GELU_GLU, ACT_SILU_GLU, ACT_CLAMP_GLU)


@dataclass(frozen=True)
class ActArgs:
    """Constants and operands of an activation: ``ACT_RELU2`` from column ``start`` on; ``limit`` and ``alpha`` of
    ``ACT_CLAMP_GLU``; ``table [rows, N]`` (a view) and the tokens' rows ``ids`` (int64) of ``ACT_GELU_MUL``."""
    start: int = 0
    limit: float = 0.0
    alpha: float = 0.0
    table: Optional[torch.Tensor] = None
    ids: Optional[torch.Tensor] = None

    def c_args(self):
        t = self.table
        return (self.start, self.limit, self.alpha, ptr(t), 0 if t is None else t.stride(0), 0 if t is None else t.shape[0],
                ptr(self.ids))


NO_ARGS = ActArgs()


def _dt(t) -> int:
    return api.dtype_code(t if isinstance(t, torch.dtype) else t.dtype)


@contextmanager
def _true_fp32():
    """Library products of 32-bit models in full precision, whatever the process has allowed."""
    m = torch.backends.cuda.matmul
    old = m.allow_tf32
    m.allow_tf32 = False
    try:
        yield
    finally:
        m.allow_tf32 = old


# ------------------------------------------------------------------------------------------------
# products
# ------------------------------------------------------------------------------------------------
def rows_max(K: int, dtype) -> int:
    return int(stream_lib().ipex_gemv_rows_max(K, _dt(dtype)))


def gemv_rows(w, x, out, mode: int, norm=None, eps: float = 0.0, act: int = 0, softcap: float = 0.0, pdl=False, bias=None,
              w2=None, out2=None, interleaved=True, args: ActArgs = NO_ARGS):
    """``act(x @ w.T + bias)`` for a few rows.  ``norm``: ``x`` is the stream and is RMS-normed with this weight on the way
    (inside the product for one or two rows; a CTA would spend longer on the norms of more rows than on its weights); rows
    of the stream without ``norm`` are converted on the way.  ``w2`` / ``out2``: more rows for the same ``x``, with fp32
    results.  ``GATED_ACTS``: ``w`` holds gate and up rows (in blocks of eight, or not ``interleaved``), half as many columns
    come out."""
    M, N, K = x.shape[0], w.shape[0], w.shape[1]
    if norm is not None and M > 2 and w.dtype != torch.float32:
        x, norm = norm_stream(x, norm, eps, pdl=pdl), None
    raw = norm is None and x.dtype != w.dtype
    if raw and (M > 8 or K % 8) and M * (K + 64) * w.element_size() > 160 * 1024:      # more than a CTA can stage
        x, raw = add_sides(x, (), (), None, eps, w.dtype, pdl=pdl), False
    rc = stream_lib().ipex_gemv_rows(ptr(w), w.stride(0), ptr(x), x.stride(0), ptr(norm), eps, ptr(bias), ptr(out),
                                     out.stride(0), ptr(w2), 0 if w2 is None else w2.shape[0], ptr(out2),
                                     0 if out2 is None else out2.stride(0), M, N, K, mode, act, int(interleaved),
                                     softcap, int(raw), *args.c_args(), _dt(w), int(pdl), current_stream())
    api.check(rc, "gemv_rows")
    return out


def gemm_ok(x, w) -> bool:
    return w.dtype in (torch.float16, torch.bfloat16) and x.dtype == w.dtype and w.shape[-1] % 8 == 0 and \
        x.stride(-1) == 1 and x.stride(0) % 8 == 0 and w.stride(-2) % 8 == 0 and \
        x.data_ptr() % 16 == 0 and w.data_ptr() % 16 == 0


def _tile(rows: float, cols: int = 1 << 20) -> int:
    """Token tile of the tcgen05 GEMM: no wider than the rows, and narrower where few columns leave most SMs idle."""
    bt = 32 if rows <= 32 else 64 if rows <= 64 else 128 if rows <= 128 else 256
    while bt > 32 and -(-rows // bt) * -(-cols // 128) < 48:
        bt //= 2
    return bt


def gemm(x, w, out, mode: int, act: int = 0, bias=None, interleaved=True, w2=None, out2=None, args: ActArgs = NO_ARGS):
    """``x [M, K] @ w[N, K].T (+ bias)`` into ``out`` (see ``OUT_*``): the tcgen05 kernel, or the library product for
    32-bit weights and rows that are no multiple of 16 bytes.  Activations, ``w2`` / ``out2``: see ``gemv_rows``."""
    M, (N, K) = x.shape[0], w.shape
    gated = act in GATED_ACTS
    if gemm_ok(x, w) and not (gated and not interleaved):
        both = w2 is not None and gemm_ok(x, w2) and w2.stride(0) == w.stride(0)
        if w2 is not None and not both:
            gemm(x, w2, out2, OUT_F32)
        rc = stream_lib().ipex_gemm_stream(ptr(x), x.stride(0), ptr(w), w.stride(0), ptr(out), out.stride(0), ptr(bias),
                                           ptr(w2 if both else None), w2.shape[0] if both else 0,
                                           ptr(out2 if both else None), out2.stride(0) if both else 0, None, None, 1, M, N,
                                           K, mode, act, args.limit, args.alpha, args.start, *args.c_args()[3:], _tile(M, N),
                                           _dt(w), ptr(error_flag(x.device)), current_stream())
        if rc == -1:
            raise RuntimeError("ipex_llm_b200: the driver's tensor-map encoder rejected the GEMM operands")
        api.check(rc, "gemm_stream")
        return out
    if w2 is not None:
        gemm(x, w2, out2, OUT_F32)
    with _true_fp32():
        if gated:
            return glu_rows(torch.matmul(x.float(), w.float().t()), bias, out, act, interleaved, args)
        if mode == OUT_ACT:
            torch.matmul(x, w.t(), out=out) if out.is_contiguous() else out.copy_(torch.matmul(x, w.t()))
            if bias is not None:
                bias_rows_(out, bias)
            return act_rows_(out, act, args) if act in (ACT_RELU2, ACT_GELU_MUL) else out
        if x.dtype == torch.float32:
            out.addmm_(x, w.t(), beta=1.0 if mode == OUT_ADD else 0.0)
        else:
            y = torch.matmul(x.float(), w.float().t())
            out.add_(y) if mode == OUT_ADD else out.copy_(y)
    return out if bias is None else bias_rows_(out, bias)


def bias_rows_(y, bias):
    """``y [n, N] += bias`` for rows in the bias's dtype or fp32."""
    rc = stream_lib().ipex_bias_rows(ptr(y), y.stride(0), int(y.dtype == torch.float32), ptr(bias), y.shape[0], y.shape[1],
                                     _dt(bias), current_stream())
    api.check(rc, "bias_rows")
    return y


def glu_rows(gu, bias, out, act: int, interleaved=True, args: ActArgs = NO_ARGS):
    """``act(gate + bias) * (up + bias)`` of finished products ``gu [n, 2 I]`` (the dtype of ``out``, or fp32)."""
    rc = stream_lib().ipex_glu_rows(ptr(gu), gu.stride(0), int(gu.dtype == torch.float32), ptr(bias), ptr(out),
                                    out.stride(0), gu.shape[0], gu.shape[1] // 2, int(interleaved), act, args.limit,
                                    args.alpha, _dt(out), current_stream())
    api.check(rc, "glu_rows")
    return out


def act_rows_(y, act: int, args: ActArgs = NO_ARGS):
    """``ACT_RELU2`` or ``ACT_GELU_MUL`` on finished products ``y [n, N]``, in place."""
    start, _, _, *table = args.c_args()
    dtype = y.dtype if args.table is None else args.table.dtype
    rc = stream_lib().ipex_act_rows(ptr(y), y.stride(0), int(y.dtype == torch.float32), y.shape[0], y.shape[1], start, act, *table,
                                    _dt(dtype), current_stream())
    api.check(rc, "act_rows")
    return y


def relu2_(x):
    if not x.is_contiguous():
        raise ValueError("relu2_ wants a contiguous tensor")
    api.check(stream_lib().ipex_relu2_inplace(ptr(x), x.numel(), _dt(x), current_stream()), "relu2")
    return x


def add_stream_(x, y):
    """``x += y`` for the fp32 stream and a contiguous activation."""
    api.check(stream_lib().ipex_add_stream(ptr(x), ptr(y), x.numel(), _dt(y), current_stream()), "add_stream")
    return x


def softcap_(logits, cap: float):
    api.check(stream_lib().ipex_softcap_f32(ptr(logits), logits.numel(), cap, current_stream()), "softcap")
    return logits


# ------------------------------------------------------------------------------------------------
# stream
# ------------------------------------------------------------------------------------------------
def embed_stream(tokens, slot, pos, cache, table, scale: float, bigram=None, buckets=0, mul_prev=0, mul_cur=0, out=None,
                 pdl=False, streams=1):
    """``table[token] * scale (+ bigram row)`` for every entry, ``streams`` times, and the ids filed in
    ``cache.history``."""
    n, (V, W) = tokens.shape[0], table.shape
    if out is None:
        out = torch.empty(n, streams * W, dtype=torch.float32, device=tokens.device)
    rc = stream_lib().ipex_embed_stream(ptr(tokens), ptr(slot), ptr(pos), ptr(cache.start), ptr(cache.history),
                                        cache.capacity, ptr(table), ptr(bigram), ptr(out), n, W, V, scale, buckets,
                                        mul_prev, mul_cur, streams, _dt(table), int(pdl), current_stream())
    api.check(rc, "embed_stream")
    return out


def norm_stream(x, weight, eps: float, rows=None, out=None, pdl=False, dtype=None):
    """RMS norm of the stream (or of its rows ``rows``, int32) in ``dtype``: the weight's own, unless that is fp32 and a
    16-bit one is asked for."""
    n, K = (x.shape[0] if rows is None else rows.shape[0]), x.shape[1]
    dtype = dtype or weight.dtype
    if out is None:
        out = torch.empty(n, K, dtype=dtype, device=x.device)
    rc = stream_lib().ipex_norm_stream(ptr(x), x.stride(0), ptr(weight), int(weight.dtype == torch.float32), ptr(out),
                                       out.stride(0), ptr(rows), n, K, eps, _dt(dtype), int(pdl), current_stream())
    api.check(rc, "norm_stream")
    return out


def add_norm_stream(x, y, w_out, w_in, eps: float, dtype, pdl=False):
    """``x += norm(y) * w_out`` and, unless ``w_in`` is None, ``norm(x) * w_in`` in ``dtype``: the joint between two
    sublayers when a sublayer's output is normed before it joins the stream.  ``y`` and the weights are fp32."""
    h = None if w_in is None else torch.empty(x.shape, dtype=dtype, device=x.device)
    rc = stream_lib().ipex_add_norm_stream(ptr(x), x.stride(0), ptr(y), y.stride(0), ptr(w_out), ptr(w_in), ptr(h),
                                           x.shape[1], x.shape[0], x.shape[1], eps, _dt(dtype), int(pdl), current_stream())
    api.check(rc, "add_norm_stream")
    return h


def add_sides(x, ys, ws, w_in, eps: float, dtype, pdl=False):
    """``x += sum of norm(y) * w`` over up to two fp32 ``ys``, then ``norm(x) * w_in`` in ``dtype``, or ``x`` itself (``w_in``
    None): the joint behind sublayers whose outputs are normed side by side.  The weights are fp32."""
    n, K = x.shape
    h = torch.empty(n, (K + 7) // 8 * 8, dtype=dtype, device=x.device)[:, :K]
    y0, y1 = [*ys, None, None][:2]
    w0, w1 = [*ws, None, None][:2]
    rc = stream_lib().ipex_add_sides(ptr(x), x.stride(0), ptr(y0), ptr(w0), ptr(y1), ptr(w1), 0 if y0 is None else y0.stride(0),
                                     ptr(w_in), ptr(h), h.stride(0), n, K, eps, _dt(dtype), int(pdl), current_stream())
    api.check(rc, "add_sides")
    return h


def hyper_joint(x, y, mix, w_out, w_in, norm, eps: float, dtype, pdl=False):
    """The joint between two sublayers of a decoder with several residual streams ``x [tokens, streams, width]``:
    ``x_t <- sum_s mix[s, t] x_s + w_out[t] y`` (``y`` None: as they are), and the next input ``norm(sum_s w_in[s] x_s)`` in
    ``dtype``.  Everything but the result is fp32."""
    n, S, K = x.shape
    h = torch.empty(n, (K + 7) // 8 * 8, dtype=dtype, device=x.device)[:, :K]
    rc = stream_lib().ipex_hyper_joint(ptr(x), ptr(y), 0 if y is None else y.stride(0), ptr(mix), ptr(w_out), ptr(w_in),
                                       ptr(norm), ptr(h), h.stride(0), n, S, K, eps, _dt(dtype), int(pdl), current_stream())
    api.check(rc, "hyper_joint")
    return h


def argmax_rows(logits, out, pdl=False):
    rc = stream_lib().ipex_argmax(ptr(logits), ptr(out), logits.shape[0], logits.shape[1], logits.stride(0), _dt(logits),
                                  int(pdl), current_stream())
    api.check(rc, "argmax")
    return out
