"""Engine for decoders whose mixer and feed-forward read one norm side by side and whose layers add an embedding of the token
of their own (family engine ``parallel_block``), on the base of ``stream_engine.py``.  Mixers: a generalized delta rule, or
attention over a window and pooled blocks beside a state-space recurrence.

Kernels of a decode step, per layer (up to sixteen sequences):
    delta     1. fused projection (the feed-forward's squared hidden units included; decays' first half and router in fp32)
              2. decays, rates, recurrence, norm and gate, into the gates' place beside the hidden units  3. both output
              projections in one product, added to the stream
    parallel  1. fused projection of both sides (likewise; step sizes and router in fp32)  2. norms, rotation, append, attention
              over window and blocks, the block's means  3. convolution and recurrence  4. gate and grouped norm  5., 6. output
              projections  7. down product, added to the stream  8. both sides normed and added
    experts   choice, hidden units of the chosen and the shared experts, weighted down product added to the stream (up to eight
              sequences)
    both      token side: 1. gate product, gelu and the token's row  2. projection  3. norm, addition and the next layer's norm
then lm_head and arg-max.  More sequences, and prompts, replace the row products by GEMMs; prompts run the tcgen05 attention
and the chunked forms of the recurrences.
"""
from __future__ import annotations

from typing import Optional

import torch

from ..models.gegorax import SIDE_SHARE, UNIT_ALPHA
from ..ops import dense_moe as X, general_delta as R, ssd as S, stream as K, window_attn as A
from ..ops.kv_cache import DeltaStateShape, KeyValueShape, PooledShape, SlotCache
from .stream_engine import Portions, StreamEngine, StreamStack, _Layer, _Proj

_COMPONENTS = {"general_delta": ("recurrent", "general_delta"), "parallel": ("attention", "recurrent", "ssd")}


def _f32(t, factor: float = 1.0):
    return (t.data.float() * factor).contiguous()


class ParallelBlockStack(StreamStack):
    def __init__(self, model):
        base = model.model
        used = dict.fromkeys(c for blk in base.layers for c in _COMPONENTS[blk.kind])
        self.components = ("stream", *used)
        super().__init__(model, [blk.in_proj for blk in base.layers])
        dt = self.dtype
        self.final_norm = _f32(base.norm.weight)
        table = None if base.side_table is None else base.side_table.data.to(dt).contiguous()
        self.kernel_launches_per_step = 4
        for i, blk in enumerate(base.layers):
            L, m = _Layer(), blk.mixer
            L.layer_idx, L.kind, L.dense_ff = i, blk.kind, blk.dense_ff
            L.norm1 = _f32(blk.norm1.weight)
            L.in_proj, L.low_proj = _Proj(blk.in_proj, dt), blk.low_proj.weight.data.to(dt).contiguous()
            L.out_proj = None if blk.out_proj is None else _Proj(blk.out_proj, dt)
            L.up_at, L.low_rows = m.rows, m.low_rows
            (self._parallel_layer if blk.kind == "parallel" else self._delta_layer)(L, m)
            L.bank = None if blk.moe is None else self._experts_of(L, blk)
            L.side = None
            if blk.side is not None:
                n = blk.side.gate.weight.shape[0]
                L.side = (_Proj(blk.side.gate, dt), _Proj(blk.side.proj, dt), _f32(blk.side.norm.weight),
                          table[:, i * n:(i + 1) * n])
            self.kernel_launches_per_step += (3 if L.bank is not None else 0) + \
                (3 if L.side is not None else 0 if blk.kind == "parallel" else 1)
            self.layers.append(L)

    def _delta_layer(self, L, m):
        dt = self.dtype
        L.spec = s = m.spec
        L.weights = R.GeneralDeltaWeights(m.decay_up.data.to(dt), m.decay_bias.data, m.rate_bias.data, m.head_norm.data.to(dt),
                                          self.eps)
        L.state = self._store(DeltaStateShape(s.heads, s.dim, s.vdim, 0, 0))
        self.kernel_launches_per_step += 3

    def _parallel_layer(self, L, m):
        dt = self.dtype
        s, r = m.left, m.right
        L.spec, L.ssd = s, r
        L.rot_key = (m.rot_base, s.rot_pairs)
        L.head_norms = _f32(m.q_norm.weight), _f32(m.k_norm.weight)
        L.sides = [(_Proj(m.o_left, dt), _f32(m.left_out.weight, SIDE_SHARE)),
                   (_Proj(m.o_right, dt), _f32(m.right_out.weight, SIDE_SHARE))]
        L.weights = S.SSDWeights(m.conv.data.to(dt), m.conv_bias.data, m.dt_bias.data, m.A_log.data, m.skip.data,
                                 m.inner_norm.weight.data.to(dt), self.eps)
        L.prefill_fast = s.prefill_ok(dt)
        L.store = self._store(KeyValueShape(s.kv_heads, s.dim, s.vdim))
        L.pooled = self._store(PooledShape(s.kv_heads, s.dim, s.vdim, s.pool)) if s.pool else None
        L.state = self._store(DeltaStateShape(r.heads, r.state, r.vdim, r.taps, r.channels))
        self.kernel_launches_per_step += 7 + (L.dense_ff > 0)

    def _experts_of(self, L, blk):
        f, dt = blk.moe, self.dtype
        sh = f.shared
        return X.SoftExpertBank(L.low_proj[L.low_rows:], f.experts.gate_up_rows.data.to(dt), f.experts.down_rows.data.to(dt),
                                f.top_k, shared_gate_up=None if sh is None else sh.gate_up_rows.data.to(dt),
                                shared_down=None if sh is None else sh.down_rows.data.to(dt), act=K.ACT_CLAMP_GLU,
                                limit=f.limit, alpha=UNIT_ALPHA, shared_limit=f.shared_limit, bias=f.router_bias.data,
                                shared_gated=False)

    # -- mixers ---------------------------------------------------------------------------------------
    def _delta(self, L, proj, low, x, slot, pos, cache, portions, pdl):
        """Adds the mixer's output, and that of a dense feed-forward, to the stream."""
        s = L.spec
        R.general_delta_mix(s, L.weights, proj, low, slot, pos, cache, L.state, proj[:, s.gate_at:s.rows], portions, pdl=pdl)
        self._linear(L.out_proj, proj[:, s.gate_at:], x, K.OUT_ADD, pdl=pdl)      # mixed columns, hidden units

    def _parallel(self, L, proj, low, x, slot, pos, cache, visible, portions, pdl):
        """The sides' outputs, before their norms; adds that of a dense feed-forward to the stream."""
        s, r, T = L.spec, L.ssd, x.shape[0]
        left, right = proj[:, :s.rows], proj[:, s.rows:s.rows + r.rows]
        a, b = self._rows(T, s.heads * s.vdim), self._rows(T, r.inner)
        tables = A.AttnTables(None, *self._rot[L.rot_key], *L.head_norms)
        if portions is not None and portions.whole and T > 8 and L.prefill_fast:
            A.attend_prompt(s, left, None, slot, pos, portions.row, portions.length, portions.longest, cache, L.store, a, tables,
                            portions, L.pooled)
        else:
            A.attend_step(s, left, None, slot, pos, cache, L.store, a, s.seen(visible), portions is None, pdl=pdl,
                          tables=tables, portions=portions, pooled=L.pooled)
        S.ssd_mix(r, L.weights, right, low, slot, pos, cache, L.state, b, portions, pdl=pdl)
        ys = []
        for h, (o, _) in zip((a, b), L.sides):
            ys.append(self._linear(o, h, torch.empty(T, self.W, dtype=torch.float32, device=self.device), K.OUT_F32, pdl=pdl))
        if L.dense_ff:
            self._linear(L.out_proj, proj[:, L.up_at:], x, K.OUT_ADD, pdl=pdl)
        return ys

    def _token_side(self, L, x, sides, after, tokens, pdl):
        """Adds the sides and the layer's embedding of the tokens to the stream; returns the next input."""
        gate, proj, norm, table = L.side
        T = x.shape[0]
        h = x
        if sides[0] or not self._few(gate, T):
            h = K.add_sides(x, *sides, None, self.eps, self.dtype, pdl=pdl)
        g = self._rows(T, gate.N)
        self._linear(gate, h, g, K.OUT_ACT, act=K.ACT_GELU_MUL, pdl=pdl, args=K.ActArgs(table=table, ids=tokens))
        y = torch.empty(T, self.W, dtype=torch.float32, device=self.device)
        self._linear(proj, g, y, K.OUT_F32, pdl=pdl)
        return K.add_norm_stream(x, y, norm, after, self.eps, self.dtype, pdl=pdl)

    # -- pass -----------------------------------------------------------------------------------------
    def run(self, tokens, slot, pos, cache: SlotCache, visible: int, portions: Optional[Portions] = None, pdl=False,
            collect=None):
        T, dev, dt, eps = tokens.shape[0], self.device, self.dtype, self.eps
        x = K.embed_stream(tokens, slot, pos, cache, self.embed, 1.0, pdl=pdl)
        h = K.norm_stream(x, self.layers[0].norm1 if self.layers else self.final_norm, eps, pdl=pdl, dtype=dt)
        for L, nxt in zip(self.layers, self.layers[1:] + [None]):
            after = self.final_norm if nxt is None else nxt.norm1
            proj = self._rows(T, L.in_proj.N)
            low = torch.empty(T, L.low_proj.shape[0], dtype=torch.float32, device=dev)
            self._linear(L.in_proj, h, proj, K.OUT_ACT, act=K.ACT_RELU2 if L.dense_ff else K.ACT_NONE, pdl=pdl, w2=L.low_proj,
                         out2=low, args=K.ActArgs(start=L.up_at))
            sides = ((), ())
            if L.kind == "parallel":
                sides = self._parallel(L, proj, low, x, slot, pos, cache, visible, portions, pdl), [w for _, w in L.sides]
            else:
                self._delta(L, proj, low, x, slot, pos, cache, portions, pdl)
            if L.bank is not None:
                experts = X.soft_moe_rows if L.bank.rows_ok(T) else X.soft_moe_grouped
                kw = {"pdl": pdl} if experts is X.soft_moe_rows else {}
                experts(L.bank, h, x, logits=low[:, L.low_rows:], add=True, **kw)
            if L.side is not None:
                h = self._token_side(L, x, sides, after, tokens, pdl)
            else:
                h = K.add_sides(x, *sides, after, eps, dt, pdl=pdl)
            if collect is not None:
                collect.append(x.clone())
        return x, h


class ParallelBlockEngine(StreamEngine):
    stack_cls = ParallelBlockStack
