"""Python front of state-space duality, a selective state space with a scalar decay per head behind a short convolution
(``ssd.cu``): token by token for decoding, short portions and 32-bit models, in chunks on the tensor cores for prompts.

Every function launches on the current stream; there is no eager substitute.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

from ..native import cuda_api as api
from ..native.lib import current_stream, ptr, stream_lib
from .cuda_ops import error_flag
from .recurrent import gated_group_norm, ring_tail
from .stream import _dt

SCRATCH_BYTES = 256 << 20        # of the chunked form; longer prompts run in several passes
CHUNKED_FROM = 17                # tokens of the longest portion from which the chunked form pays


@dataclass(frozen=True)
class SSDSpec:
    """Sizes of one layer: ``state`` rows of a head's state, ``groups`` of heads share B and C, ``taps`` of the convolution,
    ``parts`` of the output norm."""
    heads: int
    vdim: int
    state: int
    groups: int
    taps: int
    parts: int

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:
        """Convolved columns of the fused projection (x, B, C); the gates z follow."""
        return self.inner + 2 * self.groups * self.state

    @property
    def rows(self) -> int:
        return self.channels + self.inner

    def chunks_ok(self, dtype) -> bool:
        return dtype != torch.float32 and bool(stream_lib("ssd").ipex_ssd_chunks_ok(self.state, self.vdim, self.taps))


class SSDWeights:
    """What the recurrence needs beside the projections: convolution taps ``[channels, taps]`` and the weight of the output norm
    ``[inner]`` in the activation dtype; biases of convolution and step sizes, decay constants and skip factors in fp32."""

    def __init__(self, conv, conv_bias, dt_bias, a_log, skip, norm, eps: float):
        self.conv, self.norm, self.eps = conv.contiguous(), norm.contiguous(), float(eps)
        self.conv_bias, self.dt_bias, self.a_log, self.skip = (t.float().contiguous() for t in (conv_bias, dt_bias, a_log, skip))


def ssd_mix(spec: SSDSpec, w: SSDWeights, proj, dt, slot, pos, cache, layer_idx: int, out, portions=None, pdl=False,
            chunked=None):
    """Gated and normed outputs ``out [tokens, inner]`` of the recurrence over ``proj`` (x, B and C before their convolution, and
    the gates z) and the first ``heads`` columns of ``dt`` (fp32, before bias and softplus); the slots' states and
    convolution inputs move on.  ``portions``: how the tokens belong together, None when every token is another sequence's
    next one.  ``chunked`` overrides the choice of the form."""
    lib, layer = stream_lib("ssd"), cache.layers[layer_idx]
    T, code, st, dev = proj.shape[0], _dt(proj), current_stream(), proj.device
    sizes = (spec.heads, spec.groups, spec.state, spec.vdim, spec.taps, code)
    common = (ptr(proj), proj.stride(0), ptr(dt), dt.stride(0), ptr(w.conv), ptr(w.conv_bias), ptr(w.dt_bias), ptr(w.a_log),
              ptr(w.skip), ptr(layer._v), ptr(layer._k), ptr(slot), ptr(pos), ptr(cache.start))
    raw = torch.empty(T, spec.inner, dtype=torch.float32, device=dev)
    if portions is None:
        api.check(lib.ipex_ssd_step(*common, None, None, T, ptr(raw), *sizes, int(pdl), st), "ssd_step")
    else:
        row, ln, n = portions.row, portions.length, portions.row.shape[0]
        if chunked is None:
            chunked = portions.longest >= CHUNKED_FROM
        if chunked and spec.chunks_ok(proj.dtype):
            per_g = spec.groups * lib.ipex_ssd_group_floats(spec.state, spec.vdim)
            per_h = spec.heads * lib.ipex_ssd_head_floats(spec.state, spec.vdim)
            most = max(1, min(portions.chunks, SCRATCH_BYTES // (4 * (per_g + per_h))))
            scratch = torch.empty(most * (per_g + per_h), dtype=torch.float32, device=dev)
            for c in range(0, portions.chunks, most):
                api.check(lib.ipex_ssd_chunks(*common, ptr(row), ptr(ln), n, ptr(portions.chunk_seq), ptr(portions.seq_chunk), c,
                                              min(portions.chunks, c + most), ptr(scratch), ptr(scratch[most * per_g:]),
                                              ptr(raw), *sizes, ptr(error_flag(dev)), st), "ssd_chunks")
        else:
            api.check(lib.ipex_ssd_step(*common, ptr(row), ptr(ln), n, ptr(raw), *sizes, 0, st), "ssd_step")
        ring_tail(proj, layer._v, slot, pos, portions, spec.channels, spec.taps)
    return gated_group_norm(raw, proj[:, spec.channels:], w.norm, out, spec.parts, w.eps, pdl=pdl and portions is None)
