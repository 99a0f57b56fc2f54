"""Engine for decoders that mix windowed attention and recurrent (gated delta rule) layers on a 32-bit residual stream, with
norms before and after every sublayer (family engine ``hybrid``), on the base of ``stream_engine.py``.

Kernels of a decode step, per layer (up to sixteen sequences):
    attention  1. fused q / k / v projection with biases      2. value mixing, cache append and windowed attention
    delta      1. fused projection, its gates in fp32         2. convolutions, recurrence and gated norm
    both       3. output projection    4. norm of the output, added to the stream, and the next sublayer's norm
    and, with a feed-forward, 5. gate / up products, gelu and product    6. down product    7. like 4.
then lm_head and arg-max.  More sequences, and prompts, replace the row products by GEMMs; prompts run the tcgen05 attention
and the chunked form of the recurrence.
"""
from __future__ import annotations

from typing import Optional

import torch

from ..ops import delta as R, stream as K, window_attn as A
from ..ops.kv_cache import DeltaStateShape, KeyValueShape, SlotCache
from .stream_engine import Portions, StreamEngine, StreamStack, _Layer, _Proj


def _one_plus(norm):
    """fp32 factors of a norm whose weight is stored as its distance from one."""
    return (1.0 + norm.weight.data.float()).contiguous()


class HybridStack(StreamStack):
    components = ("stream", "attention", "recurrent", "delta")

    def __init__(self, model):
        base = model.model
        super().__init__(model, [blk.mixer.in_proj for blk in base.layers])
        dt = self.dtype
        self.final_norm = _one_plus(base.norm)
        self.kernel_launches_per_step = 4
        for i, blk in enumerate(base.layers):
            L, m = _Layer(), blk.mixer
            L.layer_idx, L.kind = i, blk.kind
            L.in_proj, L.o = _Proj(m.in_proj, dt), _Proj(m.o_proj, dt)
            L.norm1, L.norm1b = _one_plus(blk.norm1), _one_plus(blk.norm1b)
            if blk.kind == "attention":
                L.spec = m.spec
                L.mix_role, L.share = m.mix_role, float(m.value_share) if m.value_share is not None else 0.0
                L.prefill_fast = m.spec.prefill_ok(dt)
                self.shapes.append(KeyValueShape(m.spec.kv_heads, m.spec.dim, m.spec.vdim))
            else:
                L.spec = s = m.spec
                L.gates = m.gate_proj.weight.data.to(dt).contiguous()
                L.weights = R.DeltaWeights(m.conv.data.to(dt), m.A_log.data, m.dt_bias.data, m.norm.weight.data.to(dt),
                                           self.eps)
                self.shapes.append(DeltaStateShape(s.heads, s.dim, s.vdim, s.taps, s.channels))
            L.gate_up = L.down = None
            if blk.mlp is not None:
                L.gate_up, L.down, L.interleaved = _Proj(blk.mlp.gate_up_proj, dt), _Proj(blk.mlp.down_proj, dt), \
                    blk.mlp.interleaved
                L.norm2, L.norm2b = _one_plus(blk.norm2), _one_plus(blk.norm2b)
            self.kernel_launches_per_step += 4 if blk.mlp is None else 7
            self.layers.append(L)

    # -- mixers ---------------------------------------------------------------------------------------
    def _attention(self, L, h, first, slot, pos, cache, visible, portions, pdl):
        """The heads' outputs and, from the layer whose values the later ones mix in, those values."""
        s, T = L.spec, h.shape[0]
        qkv = torch.empty(T, (s.rows + 7) // 8 * 8, dtype=self.dtype, device=self.device)[:, :s.rows]
        self._linear(L.in_proj, h, qkv, K.OUT_ACT, pdl=pdl)
        a = torch.empty(T, s.heads * s.vdim, dtype=self.dtype, device=self.device)
        mix = A.ValueMix(first, L.share) if L.mix_role == "mixed" else None
        if portions is not None and portions.whole and T > 8 and L.prefill_fast:
            A.attend_prompt(s, qkv, mix, slot, pos, portions.row, portions.length, portions.longest, cache, L.layer_idx, a)
        else:
            A.attend_step(s, qkv, mix, slot, pos, cache, L.layer_idx, a, min(visible, s.window or visible),
                          portions is None, pdl=pdl)
        return a, qkv[:, s.v_at:] if L.mix_role == "first" else first

    def _delta(self, L, h, slot, pos, cache, portions, pdl):
        s, T = L.spec, h.shape[0]
        proj = torch.empty(T, (s.rows + 7) // 8 * 8, dtype=self.dtype, device=self.device)[:, :s.rows]
        gates = torch.empty(T, 2 * s.heads, dtype=torch.float32, device=self.device)
        self._linear(L.in_proj, h, proj, K.OUT_ACT, pdl=pdl, w2=L.gates, out2=gates)
        a = torch.empty(T, s.heads * s.vdim, dtype=self.dtype, device=self.device)
        return R.delta_mix(s, L.weights, proj, gates, slot, pos, cache, L.layer_idx, a, portions, pdl=pdl)

    def _feed_forward(self, L, h, y, pdl):
        u = torch.empty(h.shape[0], L.gate_up.N // 2, dtype=self.dtype, device=self.device)
        self._linear(L.gate_up, h, u, K.OUT_ACT, act=K.ACT_GELU_GLU, pdl=pdl, interleaved=L.interleaved)
        return self._linear(L.down, u, y, K.OUT_F32, pdl=pdl)

    # -- pass -----------------------------------------------------------------------------------------
    def run(self, tokens, slot, pos, cache: SlotCache, visible: int, portions: Optional[Portions] = None, pdl=False,
            collect=None):
        T, dev, dt, eps = tokens.shape[0], self.device, self.dtype, self.eps
        x = K.embed_stream(tokens, slot, pos, cache, self.embed, 1.0, pdl=pdl)
        y = torch.empty(T, self.W, dtype=torch.float32, device=dev)
        h = K.norm_stream(x, self.layers[0].norm1 if self.layers else self.final_norm, eps, pdl=pdl, dtype=dt)
        first = None
        for L, nxt in zip(self.layers, self.layers[1:] + [None]):
            after = self.final_norm if nxt is None else nxt.norm1
            if L.kind == "attention":
                a, first = self._attention(L, h, first, slot, pos, cache, visible, portions, pdl)
            else:
                a = self._delta(L, h, slot, pos, cache, portions, pdl)
            self._linear(L.o, a, y, K.OUT_F32, pdl=pdl)
            h = K.add_norm_stream(x, y, L.norm1b, after if L.down is None else L.norm2, eps, dt, pdl=pdl)
            if L.down is not None:
                self._feed_forward(L, h, y, pdl)
                h = K.add_norm_stream(x, y, L.norm2b, after, eps, dt, pdl=pdl)
            if collect is not None:
                collect.append(x.clone())
        return x, h


class HybridEngine(StreamEngine):
    stack_cls = HybridStack
