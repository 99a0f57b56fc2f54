"""Python front of what recurrent layers share around their recurrences (``recurrent_ops.cu``): the ring of their short
convolutions' inputs and the gated norms of their outputs.

Every function launches on the current stream; there is no eager substitute.
"""
from __future__ import annotations

from ..native import cuda_api as api
from ..native.lib import current_stream, ptr, stream_lib
from .stream import _dt


def ring_tail(proj, ring, slot, pos, portions, channels: int, taps: int):
    """File the last convolution inputs of every portion (the first ``channels`` columns of ``proj``) in the slots' rings."""
    api.check(stream_lib("recurrent").ipex_ring_tail(ptr(proj), proj.stride(0), ptr(ring), ptr(slot), ptr(pos),
                                                     ptr(portions.row), ptr(portions.length), portions.row.shape[0], channels,
                                                     taps, _dt(proj), current_stream()), "ring_tail")


def gated_norm(raw, gate, weight, out, eps: float, scale: float = 1.0, sigmoid=False):
    """``scale * o / rms(o) * weight * act(gate)`` per head of ``raw [tokens, heads, vdim]`` (fp32); ``weight [vdim]``, or
    ``[heads * vdim]``; ``act``: silu or a sigmoid.  ``out`` may be the gates' place."""
    T, heads, vdim = raw.shape
    api.check(stream_lib("recurrent").ipex_gated_norm(ptr(raw), ptr(gate), gate.stride(0), ptr(weight),
                                                      int(weight.numel() == heads * vdim), int(sigmoid), ptr(out),
                                                      out.stride(0), T, heads, vdim, eps, scale, _dt(out), current_stream()),
              "gated_norm")
    return out


def gated_group_norm(raw, z, weight, out, parts: int, eps: float, pdl=False):
    """``norm(raw * silu(z)) * weight`` over ``parts`` equal parts of the columns of ``raw [tokens, width]`` (fp32)."""
    T, width = raw.shape
    api.check(stream_lib("recurrent").ipex_gated_group_norm(ptr(raw), ptr(z), z.stride(0), ptr(weight), ptr(out), out.stride(0),
                                                            T, width, parts, eps, _dt(out), int(pdl), current_stream()),
              "gated_group_norm")
    return out
