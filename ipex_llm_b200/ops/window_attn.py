"""Python front of the attention over cached keys and values of different sizes (``kv_attn.cu``, and the packed tcgen05
prompt kernel of ``packed_prefill_tcgen05.cu``): grouped query heads, sliding window (alone or beside pooled blocks of what has
left it) or chunks, optional sink in the soft-max, rotated and normed queries and keys, gated outputs, values mixed with those
of an earlier layer.

Every function launches on the current stream; there is no eager substitute.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from ..native import cuda_api as api
from ..native.lib import current_stream, ptr, stream_lib
from .cuda_ops import error_flag
from .stream import _dt


@dataclass(frozen=True)
class AttnSpec:
    """Sizes and constants of one layer.  ``window`` 0: every earlier key; ``chunk``: only those of the query's own chunk of
    this many positions.  ``sink``: one more score without a value, 0 or a number per head (``AttnTables.sinks``).
    ``rot_pairs``: pairs (i, i + rot_pairs) of queries and keys turn with the position; ``unit_eps``: they are divided by
    sqrt(mean square + unit_eps), and times the weights of ``AttnTables``.  ``pool``: beside the window, a key and a value for every
    block of this many tokens that lies wholly before it, their means.  ``gated``: the projection ends with gate columns, outputs are multiplied by
    ``gate_scale`` times their sigmoid."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int = 0
    sink: bool = False
    chunk: int = 0
    rot_pairs: int = 0
    unit_eps: Optional[float] = None
    gated: bool = False
    gate_scale: float = 1.0
    pool: int = 0

    @property
    def k_at(self) -> int:
        """Column of the keys in the fused projection (queries come first)."""
        return self.heads * self.dim

    @property
    def v_at(self) -> int:
        return (self.heads + self.kv_heads) * self.dim

    @property
    def gate_at(self) -> int:
        return self.v_at + self.kv_heads * self.vdim

    @property
    def rows(self) -> int:
        return self.gate_at + (self.heads * self.vdim if self.gated else 0)

    @property
    def prepared(self) -> bool:
        """Queries and keys are not used as they are projected."""
        return self.rot_pairs > 0 or self.unit_eps is not None

    def seen(self, visible: int) -> int:
        """Upper bound of the keys a token sees when ``visible`` bounds its position."""
        seen = min(visible, self.window or visible, self.chunk or visible)
        return seen + (visible - seen) // self.pool if self.pool else seen

    def prefill_ok(self, dtype) -> bool:
        """Does the tcgen05 prompt kernel take these sizes?"""
        return bool(stream_lib().ipex_packed_prefill_ok(self.dim, 0, self.vdim, 8, _dt(dtype)))


@dataclass
class ValueMix:
    """Values of an earlier layer (a ``[tokens, kv_heads * vdim]`` view) and their share."""
    first: torch.Tensor
    share: float


@dataclass
class AttnTables:
    """What a layer's attention reads beside the projection: sink scores ``[heads]``, rotation tables ``[positions, rot_pairs]``
    and weights of the queries' and keys' norms ``[dim]``, fp32."""
    sinks: Optional[torch.Tensor] = None
    cos: Optional[torch.Tensor] = None
    sin: Optional[torch.Tensor] = None
    q_weight: Optional[torch.Tensor] = None
    k_weight: Optional[torch.Tensor] = None


NO_TABLES = AttnTables()


def _prepare_args(spec: AttnSpec, tables: AttnTables):
    return (ptr(tables.cos), ptr(tables.sin), spec.rot_pairs, int(spec.unit_eps is not None), spec.unit_eps or 0.0,
            ptr(tables.q_weight), ptr(tables.k_weight))


def prepare_heads(spec: AttnSpec, qkv, slot, pos, cache, tables: AttnTables):
    """Norm and rotation of all query and key heads in place."""
    api.check(stream_lib("attention").ipex_qk_prepare(ptr(qkv), qkv.stride(0), ptr(slot), ptr(pos), ptr(cache.start),
                                                      *_prepare_args(spec, tables), spec.heads, qkv.shape[0],
                                                      spec.heads + spec.kv_heads, spec.dim, _dt(qkv), 0, current_stream()),
              "qk_prepare")


def _rows_args(t):
    return (None, 0, 0) if t is None else (ptr(t), t.stride(0), t.stride(1))


def pool_blocks(spec: AttnSpec, portions, slot, pos, cache, layer_idx: int, pooled: int, packed=None):
    """Keys and values of the blocks that the portions complete, from the rows of cache layer ``layer_idx`` into those of
    ``pooled``; ``packed``: keys, transposed values and first rows (``pool_rows``) for the prompt kernel as well."""
    layer, blocks = cache.layers[layer_idx], cache.layers[pooled]
    kp, vt, rows = (None, None, None) if packed is None else packed
    api.check(stream_lib("attention").ipex_kv_pool(*_rows_args(layer._k), *_rows_args(layer._v), *_rows_args(blocks._k),
                                                   *_rows_args(blocks._v), ptr(kp), 0 if kp is None else kp.stride(0), ptr(vt),
                                                   0 if vt is None else vt.stride(0), ptr(rows), ptr(slot), ptr(pos),
                                                   ptr(cache.start), ptr(portions.row), ptr(portions.length),
                                                   portions.row.shape[0], portions.longest, spec.kv_heads, spec.dim, spec.vdim,
                                                   spec.pool, _dt(layer._k), current_stream()), "kv_pool")


def pick_splits(tokens: int, spec: AttnSpec, visible: int, n_sm: int = 148) -> int:
    """CTAs that share the keys of a query token: up to a cluster of eight, at least 64 keys each, about two waves."""
    group = spec.heads // spec.kv_heads
    ctas = tokens * spec.kv_heads * -(-group // 8)
    n = 1
    while n < 8 and visible >= 128 * n and ctas * n < n_sm:
        n *= 2
    return n


def _mix_args(mix: Optional[ValueMix], at: int = 0):
    return (None, 0, 0.0) if mix is None else (mix.first[at:], mix.first.stride(0), mix.share)


def attend_step(spec: AttnSpec, qkv, mix: Optional[ValueMix], slot, pos, cache, layer_idx: int, out, visible: int,
                single: bool, pdl=False, nsplit: Optional[int] = None, tables: AttnTables = NO_TABLES, portions=None,
                pooled: Optional[int] = None):
    """Attention of query tokens against the cache, which gets their own rows first.  ``single``: every token is another
    sequence's next one (preparation and append are then part of the attention kernel).  ``visible`` bounds the number of keys a
    token can see (it sizes the split, nothing else).  ``pooled``: the cache layer of the blocks (``spec.pool``), with
    ``portions`` saying how the tokens belong together unless ``single``."""
    lib, layer = stream_lib("attention"), cache.layers[layer_idx]
    blocks = cache.layers[pooled] if spec.pool else None
    k, v = layer._k, layer._v
    M, dt, st = qkv.shape[0], _dt(qkv), current_stream()
    cols = (qkv[:, spec.k_at:], qkv[:, spec.v_at:])
    if not single:
        if spec.prepared:
            prepare_heads(spec, qkv, slot, pos, cache, tables)
        first, ld_vf, share = _mix_args(mix)
        api.check(lib.ipex_kv_append(ptr(cols[0]), ptr(cols[1]), qkv.stride(0), ptr(first), ld_vf, share, ptr(k), k.stride(0),
                                     k.stride(1), ptr(v), v.stride(0), v.stride(1), None, 0, ptr(slot), ptr(pos), M,
                                     spec.kv_heads, spec.dim, spec.vdim, dt, int(pdl), st), "kv_append")
        if spec.pool:
            pool_blocks(spec, portions, slot, pos, cache, layer_idx, pooled)
    step = 65535
    for s in range(0, M, step):
        m = min(step, M - s)
        first, ld_vf, share = _mix_args(mix, s)
        api.check(lib.ipex_kv_attn(ptr(qkv[s:]), ptr(cols[0][s:]), ptr(cols[1][s:]), qkv.stride(0), ptr(first), ld_vf, share,
                                   ptr(k), k.stride(0), k.stride(1), ptr(v), v.stride(0), v.stride(1), ptr(out[s:]),
                                   out.stride(0), ptr(slot[s:]), ptr(pos[s:]), ptr(cache.start), m, spec.heads,
                                   spec.kv_heads, spec.dim, spec.vdim, spec.window, spec.chunk, int(spec.sink),
                                   ptr(tables.sinks), ptr(qkv[s:, spec.gate_at:] if spec.gated else None), qkv.stride(0),
                                   spec.gate_scale, int(single), int(single and spec.prepared),
                                   *_prepare_args(spec, tables), spec.pool, *_rows_args(blocks and blocks._k),
                                   *_rows_args(blocks and blocks._v), nsplit or pick_splits(m, spec, visible), spec.scale,
                                   dt, int(pdl), st), "kv_attn")
    return out


def attend_prompt(spec: AttnSpec, qkv, mix: Optional[ValueMix], slot, pos, seq_row, seq_len, max_len: int, cache,
                  layer_idx: int, out, tables: AttnTables = NO_TABLES, portions=None, pooled: Optional[int] = None):
    """Attention of whole prompts, packed one behind the other (``seq_row`` / ``seq_len``: int32, first row and length of
    each), on the tensor cores; the cache gets keys and mixed values, and with ``spec.pool`` cache layer ``pooled`` the blocks
    (``portions``: the prompts)."""
    lib, layer = stream_lib("attention"), cache.layers[layer_idx]
    k, v = layer._k, layer._v
    T, dt, st, dev = qkv.shape[0], _dt(qkv), current_stream(), qkv.device
    ld = (T + 7) // 8 * 8
    vt = torch.empty(spec.kv_heads * spec.vdim, ld, dtype=qkv.dtype, device=dev)
    first, ld_vf, share = _mix_args(mix)
    keys = qkv[:, spec.k_at:]
    if spec.prepared:
        prepare_heads(spec, qkv, slot, pos, cache, tables)
    api.check(lib.ipex_kv_append(ptr(keys), ptr(qkv[:, spec.v_at:]), qkv.stride(0), ptr(first), ld_vf, share, ptr(k),
                                 k.stride(0), k.stride(1), ptr(v), v.stride(0), v.stride(1), ptr(vt), ld, ptr(slot),
                                 ptr(pos), T, spec.kv_heads, spec.dim, spec.vdim, dt, 0, st), "kv_append")
    pool = (0, None, 0, None, 0, None, 0)
    if spec.pool:
        rows, n = portions.pool_rows(spec.pool)
        # rows between the sequences' blocks are read and not used: they have to be numbers
        kp = torch.zeros(n, (spec.kv_heads * spec.dim + 7) // 8 * 8, dtype=qkv.dtype, device=dev)
        vp = torch.zeros(spec.kv_heads * spec.vdim, n, dtype=qkv.dtype, device=dev)
        pool_blocks(spec, portions, slot, pos, cache, layer_idx, pooled, (kp, vp, rows))
        pool = (spec.pool, ptr(kp), kp.stride(0), ptr(vp), n, ptr(rows), n)
    rc = stream_lib().ipex_packed_prefill(ptr(qkv), qkv.stride(0), ptr(keys), qkv.stride(0), None, 0, ptr(vt), ld, ptr(out),
                                          out.stride(0), ptr(seq_row), ptr(seq_len), seq_row.shape[0], spec.heads,
                                          spec.kv_heads, T, max_len, spec.dim, 0, spec.vdim, spec.window, spec.chunk,
                                          int(spec.sink), ptr(tables.sinks), ptr(qkv[:, spec.gate_at:] if spec.gated else None),
                                          qkv.stride(0), spec.gate_scale, *pool, spec.scale, dt, ptr(error_flag(dev)), st)
    if rc == -1:
        raise RuntimeError("ipex_llm_b200: the driver's tensor-map encoder rejected the attention operands")
    api.check(rc, "packed_prefill")
    return out
