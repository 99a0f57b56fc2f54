"""Python front of the gated delta rule with short convolutions (``delta_rule.cu``): token by token for decoding, short
portions and 32-bit models, in chunks on the tensor cores for prompts.

Every function launches on the current stream; there is no eager substitute.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

from ..native import cuda_api as api
from ..native.lib import current_stream, ptr, stream_lib
from .cuda_ops import error_flag
from .recurrent import gated_norm, ring_tail
from .stream import _dt

SCRATCH_BYTES = 256 << 20        # of the chunked form; longer prompts run in several passes
CHUNKED_FROM = 17                # tokens of the longest portion from which the chunked form pays


@dataclass(frozen=True)
class DeltaSpec:
    """Sizes of one layer; ``taps``: length of the short convolutions."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int

    @property
    def channels(self) -> int:
        """Convolved columns of the fused projection (queries, keys, values); the output gates follow."""
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim

    @property
    def rows(self) -> int:
        return self.channels + self.heads * self.vdim

    def chunks_ok(self, dtype) -> bool:
        return dtype != torch.float32 and bool(stream_lib("delta").ipex_delta_chunks_ok(self.dim, self.vdim))


class DeltaWeights:
    """What the recurrence needs beside the projections: convolution taps ``[channels, taps]`` and the weight of the
    output norm in the activation dtype, decay constants in fp32."""

    def __init__(self, conv, a_log, dt_bias, norm, eps: float):
        self.conv, self.norm, self.eps = conv.contiguous(), norm.contiguous(), float(eps)
        self.a_log, self.dt_bias = a_log.float().contiguous(), dt_bias.float().contiguous()


def delta_mix(spec: DeltaSpec, w: DeltaWeights, proj, gates, slot, pos, cache, layer_idx: int, out, portions=None, pdl=False,
              chunked=None):
    """Normed and gated outputs ``out [tokens, heads * vdim]`` of the recurrence over ``proj`` (queries, keys, values and
    output gates before their convolutions and activations) and ``gates [tokens, 2 heads]`` (write strengths, decays;
    fp32); the slots' states and convolution inputs move on.  ``portions``: how the tokens belong together, None when
    every token is another sequence's next one.  ``chunked`` overrides the choice of the form."""
    lib, layer = stream_lib("delta"), cache.layers[layer_idx]
    T, dt, st, dev = proj.shape[0], _dt(proj), current_stream(), proj.device
    sizes = (spec.heads, spec.kv_heads, spec.dim, spec.vdim, spec.taps, dt)
    common = (ptr(gates), ptr(w.conv), ptr(w.a_log), ptr(w.dt_bias), ptr(layer._v), ptr(layer._k), ptr(slot), ptr(pos),
              ptr(cache.start))
    gate_at = spec.channels
    if portions is None and lib.ipex_delta_fused_ok(spec.vdim):
        api.check(lib.ipex_delta_step(ptr(proj), proj.stride(0), gate_at, *common, None, None, T, ptr(w.norm), w.eps,
                                      ptr(out), out.stride(0), None, *sizes, int(pdl), st), "delta_step")
        return out
    raw = torch.empty(T, spec.heads, spec.vdim, dtype=torch.float32, device=dev)
    if portions is None:
        api.check(lib.ipex_delta_step(ptr(proj), proj.stride(0), gate_at, *common, None, None, T, None, 0.0, None, 0,
                                      ptr(raw), *sizes, int(pdl), st), "delta_step")
    else:
        row, ln, n = portions.row, portions.length, portions.row.shape[0]
        if chunked is None:
            chunked = portions.longest >= CHUNKED_FROM
        if chunked and spec.chunks_ok(proj.dtype):
            per = spec.heads * lib.ipex_delta_scratch_floats(spec.dim, spec.vdim)
            most = max(1, min(portions.chunks, SCRATCH_BYTES // (4 * per)))
            scratch = torch.empty(most * per, dtype=torch.float32, device=dev)
            for c in range(0, portions.chunks, most):
                api.check(lib.ipex_delta_chunks(ptr(proj), proj.stride(0), *common, ptr(row), ptr(ln), n,
                                                ptr(portions.chunk_seq), ptr(portions.seq_chunk), c,
                                                min(portions.chunks, c + most), ptr(scratch), ptr(raw), *sizes,
                                                ptr(error_flag(dev)), st),
                          "delta_chunks")
        else:
            api.check(lib.ipex_delta_step(ptr(proj), proj.stride(0), gate_at, *common, ptr(row), ptr(ln), n, None, 0.0, None,
                                          0, ptr(raw), *sizes, 0, st), "delta_step")
        ring_tail(proj, layer._v, slot, pos, portions, spec.channels, spec.taps)
    return gated_norm(raw, proj[:, gate_at:], w.norm, out, w.eps)
