"""Python front of gated linear attention with a decay per key channel (``linear_attn.cu``): token by token for decoding,
short portions and 32-bit models, in chunks on the tensor cores for prompts.

Every function launches on the current stream; there is no eager substitute.
"""
from __future__ import annotations

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
class LinearSpec:
    """Sizes and constants of one layer: decays are sigmoid(.)^(1 / tau) of a projection through ``rank`` numbers, outputs
    are multiplied by ``out_scale``."""
    heads: int
    dim: int
    vdim: int
    rank: int
    tau: float
    out_scale: float = 1.0

    @property
    def gate_at(self) -> int:
        """Column of the output gates in the fused projection, behind queries, keys and values."""
        return self.heads * (2 * self.dim + self.vdim)

    @property
    def rows(self) -> int:
        return self.gate_at + self.heads * self.vdim

    def chunks_ok(self, dtype) -> bool:
        return dtype != torch.float32 and bool(stream_lib("linear").ipex_linear_chunks_ok(self.dim, self.vdim, self.rank))


class LinearWeights:
    """What the recurrence needs beside the projections: second half of the decays' projection ``up [heads * dim, rank]``
    and the weight of the output norm in the activation dtype, its bias in fp32."""

    def __init__(self, up, bias, norm, eps: float):
        self.up, self.norm, self.eps = up.contiguous(), norm.contiguous(), float(eps)
        self.bias = bias.float().contiguous()


def linear_mix(spec: LinearSpec, w: LinearWeights, proj, low, slot, pos, cache, layer_idx: int, out, portions=None,
               pdl=False, chunked=None):
    """Normed and gated outputs ``out [tokens, heads * vdim]`` of the recurrence over ``proj`` (queries, keys, values and
    output gates) and ``low [tokens, rank]`` (fp32); the slots' states move on.  ``portions``: how the tokens belong
    together, None when every token is another sequence's next one.  ``chunked`` overrides the choice of the form."""
    lib, state = stream_lib("linear"), cache.layers[layer_idx]._k
    T, dt, st, dev = proj.shape[0], _dt(proj), current_stream(), proj.device
    sizes = (spec.heads, spec.dim, spec.vdim, spec.rank, spec.tau, dt)
    common = (ptr(low), ptr(w.up), ptr(w.bias), ptr(state), ptr(slot), ptr(pos), ptr(cache.start))
    if portions is None and lib.ipex_linear_fused_ok(spec.vdim):
        api.check(lib.ipex_linear_step(ptr(proj), proj.stride(0), spec.gate_at, *common, None, None, T, ptr(w.norm), w.eps,
                                       spec.out_scale, ptr(out), out.stride(0), None, *sizes, int(pdl), st), "linear_step")
        return out
    raw = torch.empty(T, spec.heads, spec.vdim, dtype=torch.float32, device=dev)
    row, ln, n = (None, None, T) if portions is None else (portions.row, portions.length, portions.row.shape[0])
    if chunked is None:
        chunked = portions is not None and portions.longest >= CHUNKED_FROM
    if chunked and portions is not None and spec.chunks_ok(proj.dtype):
        per = spec.heads * lib.ipex_linear_scratch_floats(spec.dim, spec.vdim)
        most = max(1, min(portions.chunks, SCRATCH_BYTES // (4 * per)))
        scratch = torch.empty(most * per, dtype=torch.float32, device=dev)
        for c in range(0, portions.chunks, most):
            api.check(lib.ipex_linear_chunks(ptr(proj), proj.stride(0), *common, ptr(row), ptr(ln), n,
                                             ptr(portions.chunk_seq), ptr(portions.seq_chunk), c,
                                             min(portions.chunks, c + most), ptr(scratch), ptr(raw), *sizes,
                                             ptr(error_flag(dev)), st), "linear_chunks")
    else:
        api.check(lib.ipex_linear_step(ptr(proj), proj.stride(0), spec.gate_at, *common, ptr(row), ptr(ln), n, None, 0.0,
                                       0.0, None, 0, ptr(raw), *sizes, int(pdl) if portions is None else 0, st), "linear_step")
    return gated_norm(raw, proj[:, spec.gate_at:], w.norm, out, w.eps, spec.out_scale)
