"""Engine for decoders with multi-head latent attention and a 32-bit residual stream (family engine ``latent``), on the
base of ``stream_engine.py``.

Kernels of a decode step, per layer (up to eight sequences):
    1. norm + fused query / latent projection          2. q absorption, rotation, cache append
    3. latent attention over the visible rows           4. split merge + value up-projection
    5. o_proj, added to the stream                      6. norm + up_proj + squared ReLU     7. down_proj, added
  with, for a mixture-of-experts layer, 6. norm + router + top-k, 7. expert hidden units, 8. expert down product, added;
then norm + lm_head + soft-cap and the arg-max.  More sequences, and prompts, replace the row products by GEMMs, and
prompts the absorbed attention by the tcgen05 attention on expanded keys and values.
"""
from __future__ import annotations

import os
from typing import Optional

import torch

from ..ops import latent as K
from ..ops.kv_cache import LatentCache
from .stream_engine import Portions, StreamEngine, StreamStack, _Layer, _Proj


class LatentStack(StreamStack):
    cache_cls = LatentCache
    components = ("stream", "latent")

    def __init__(self, model):
        cfg, base = model.config, model.model
        super().__init__(model, [blk.mixer.qkv_a_proj for blk in base.layers])
        dt = self.dtype
        self.softcap = float(cfg.logit_softcap or 0.0)
        emb = cfg.embedding
        self.embed_scale = float(emb.get("scale", 1.0))
        self.bigram = base.bigram.weight.data.to(dt).contiguous() if base.bigram is not None else None
        b = emb.get("bigram") or {}
        self.bigram_args = (int(b.get("buckets", 0)), int(b.get("mul_prev", 0)), int(b.get("mul_cur", 0)))
        self.final_norm = base.norm.weight.data.to(dt)
        for i, blk in enumerate(base.layers):
            L, m = _Layer(), blk.mixer
            L.layer_idx = i
            L.spec = K.LatentSpec(m.heads, m.dim, m.rot_dim, m.v_dim, m.kv_rank, m.scale, m.window, m.rot_pairs, self.eps)
            L.rot_key = (m.rot_base, m.rot_pairs)
            L.qkv, L.o = _Proj(m.qkv_a_proj, dt), _Proj(m.o_proj, dt)
            L.w_uk, L.w_uv = m.k_up.data.to(dt).contiguous(), m.v_up.data.to(dt).contiguous()
            L.kv_norm = m.kv_norm.weight.data.to(dt)
            L.norm1 = blk.norm1.weight.data.to(dt)
            L.norm2 = blk.norm2.weight.data.to(dt) if blk.norm2 is not None else None
            L.up = L.down = L.bank = None
            if blk.mlp is not None and hasattr(blk.mlp, "experts"):
                ex = blk.mlp.experts
                L.bank = K.ExpertBank(blk.mlp.router.weight.data.to(dt), ex.gate_up_rows.data.to(dt),
                                      ex.down_rows.data.to(dt), blk.mlp.top_k, blk.mlp.limit, blk.mlp.gate_alpha,
                                      ex.interleaved)
            elif blk.mlp is not None:
                L.up, L.down = _Proj(blk.mlp.up_proj, dt), _Proj(blk.mlp.down_proj, dt)
            L.prefill_fast = L.spec.prefill_ok(dt) and os.environ.get("IPEX_LLM_LATENT_PREFILL", "1") != "0"
            self.layers.append(L)
        self.shapes = [L.spec.row(dt) for L in self.layers]
        self._rot = {}           # (base, pairs) -> (positions, cos, sin)
        self._rot_retired = []   # tables a captured graph may still read
        self._positions = 0
        self.kernel_launches_per_step = 3 + sum(5 + (3 if L.bank is not None else 2 if L.up is not None else 0)
                                                for L in self.layers)

    def ensure_positions(self, n: int):
        if n <= self._positions and self._rot:
            return
        n = max(2048, (n + 1023) // 1024 * 1024)
        self._rot_retired.append(self._rot)
        self._rot = {L.rot_key: K.rotary_table(n, *L.rot_key, self.device) for L in self.layers}
        self._positions = n

    def run(self, tokens, slot, pos, cache: LatentCache, visible: int, portions: Optional[Portions] = None, pdl=False,
            collect=None):
        T, dev, dt = tokens.shape[0], self.device, self.dtype
        # few tokens (or continued sequences) go through the absorbed attention, whole prompts through the expanded one
        prompts = portions is not None and portions.whole and T > 8
        x = K.embed_stream(tokens, slot, pos, cache, self.embed, self.embed_scale, self.bigram, *self.bigram_args,
                           pdl=pdl)
        for L in self.layers:
            s = L.spec
            cos, sin = self._rot[L.rot_key]
            qkv = torch.empty(T, (L.qkv.N + 7) // 8 * 8, dtype=dt, device=dev)[:, :L.qkv.N]
            a = torch.empty(T, s.heads * s.v_dim, dtype=dt, device=dev)
            self._from_stream(L.qkv, x, L.norm1, qkv, pdl=pdl)
            args = (s, qkv, L.w_uk, L.w_uv, L.kv_norm, cos, sin, slot, pos)
            if prompts and L.prefill_fast:
                K.latent_prompt(*args, portions.row, portions.length, portions.longest, cache, L.layer_idx, a)
            else:
                K.latent_step(*args, cache, L.layer_idx, a, min(visible, s.window or visible), pdl=pdl)
            self._to_stream(L.o, a, x, pdl=pdl)
            if L.bank is not None:
                if L.bank.rows_ok(T):
                    K.moe_rows(L.bank, x, L.norm2, self.eps, pdl=pdl)
                else:
                    K.moe_grouped(L.bank, x, K.norm_stream(x, L.norm2, self.eps))
            elif L.up is not None:
                u = torch.empty(T, L.up.N, dtype=dt, device=dev)
                self._from_stream(L.up, x, L.norm2, u, act=K.ACT_RELU2, pdl=pdl)
                self._to_stream(L.down, u, x, pdl=pdl)
            if collect is not None:
                collect.append(x.clone())
        return x, None


class LatentEngine(StreamEngine):
    stack_cls = LatentStack
