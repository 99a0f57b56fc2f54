"""Python front of the generalized delta rule with decays and removal rates per key channel (``general_delta.cu``): token by
token for decoding, short portions and 32-bit models, in chunks on the tensor cores for prompts.

Every function launches on the current stream; there is no eager substitute.
"""
from __future__ import annotations

import math
from dataclasses import dataclass

import torch

from ..native import cuda_api as api
from ..native.lib import current_stream, ptr, stream_lib
from .cuda_ops import error_flag
from .recurrent import gated_norm
from .stream import _dt

SCRATCH_BYTES = 256 << 20        # of the chunked form; longer prompts run in several passes
CHUNKED_FROM = 17                # tokens of the longest portion from which the chunked form pays


@dataclass(frozen=True)
class GeneralDeltaSpec:
    """Sizes and constants of one layer: decays are exp(-decay * sigmoid(.)) of a projection through ``rank`` numbers."""
    heads: int
    dim: int
    vdim: int
    rank: int
    decay: float = math.exp(-0.5)

    @property
    def gate_at(self) -> int:
        """Column of the output gates in the fused projection, behind reads, keys, values and removal rates."""
        return self.heads * (3 * self.dim + self.vdim)

    @property
    def rows(self) -> int:
        return self.gate_at + self.heads * self.vdim

    def chunks_ok(self, dtype) -> bool:
        return dtype != torch.float32 and bool(stream_lib("general_delta").ipex_general_chunks_ok(self.dim, self.vdim, self.rank,
                                                                                                  self.decay))


class GeneralDeltaWeights:
    """What the recurrence needs beside the projections: second half of the decays' projection ``up [heads * dim, rank]`` and
    the weight of the output norm ``[heads * vdim]`` in the activation dtype, biases of decays and rates in fp32."""

    def __init__(self, up, bias, rate_bias, norm, eps: float):
        self.up, self.norm, self.eps = up.contiguous(), norm.contiguous(), float(eps)
        self.bias, self.rate_bias = bias.float().contiguous(), rate_bias.float().contiguous()


def general_delta_mix(spec: GeneralDeltaSpec, w: GeneralDeltaWeights, proj, low, slot, pos, cache, layer_idx: int, out,
                      portions=None, pdl=False, chunked=None):
    """Normed and gated outputs ``out [tokens, heads * vdim]`` of the recurrence over ``proj`` (reads, keys, values, rates and
    output gates, whose place ``out`` may be) and the first ``rank`` columns of ``low`` (fp32, before their tanh); the slots'
    states move on.  ``portions``: how the tokens belong together, None when every token is another sequence's next one.
    ``chunked`` overrides the choice of the form."""
    lib, state = stream_lib("general_delta"), cache.layers[layer_idx]._k
    T, dt, st, dev = proj.shape[0], _dt(proj), current_stream(), proj.device
    sizes = (spec.heads, spec.dim, spec.vdim, spec.rank, spec.decay, dt)
    common = (ptr(low), low.stride(0), ptr(w.up), ptr(w.bias), ptr(w.rate_bias), ptr(state), ptr(slot), ptr(pos),
              ptr(cache.start))
    if portions is None and lib.ipex_general_fused_ok(spec.vdim):
        api.check(lib.ipex_general_step(ptr(proj), proj.stride(0), spec.gate_at, *common, None, None, T, ptr(w.norm), w.eps,
                                        ptr(out), out.stride(0), None, *sizes, int(pdl), st), "general_step")
        return out
    raw = torch.empty(T, spec.heads, spec.vdim, dtype=torch.float32, device=dev)
    row, ln, n = (None, None, T) if portions is None else (portions.row, portions.length, portions.row.shape[0])
    if chunked is None:
        chunked = portions is not None and portions.longest >= CHUNKED_FROM
    if chunked and portions is not None and spec.chunks_ok(proj.dtype):
        per = spec.heads * lib.ipex_general_scratch_floats(spec.dim, spec.vdim)
        most = max(1, min(portions.chunks, SCRATCH_BYTES // (4 * per)))
        scratch = torch.empty(most * per, dtype=torch.float32, device=dev)
        for c in range(0, portions.chunks, most):
            api.check(lib.ipex_general_chunks(ptr(proj), proj.stride(0), *common, ptr(row), ptr(ln), n,
                                              ptr(portions.chunk_seq), ptr(portions.seq_chunk), c,
                                              min(portions.chunks, c + most), ptr(scratch), ptr(raw), *sizes,
                                              ptr(error_flag(dev)), st), "general_chunks")
    else:
        api.check(lib.ipex_general_step(ptr(proj), proj.stride(0), spec.gate_at, *common, ptr(row), ptr(ln), n, None, 0.0, None,
                                        0, ptr(raw), *sizes, int(pdl) if portions is None else 0, st), "general_step")
    return gated_norm(raw, proj[:, spec.gate_at:], w.norm, out, w.eps, sigmoid=True)
