"""Engine for decoders with several 32-bit residual streams (hyper-connections) whose layers are latent attention - with a
latent of its own or with the rows of an earlier layer - or chunked attention beside gated linear attention (family engine
``multistream``), on the base of ``stream_engine.py``.

Kernels of a decode step, per layer (up to sixteen sequences):
    latent    1. fused projection (latent and key rows, output gates; the queries' latent in fp32)  2. its norm and the query
              projection  3. q absorption, rotation, cache append  4. latent attention  5. split merge, value
              up-projection and gate
    parallel  1. fused projection of both sides (the decays' first half in fp32)  2. rotation, unit norm, append, chunked
              attention and gate  3. decays, linear recurrence, norm and gate; both sides write one activation
    both      output projection, then one joint: streams mixed, next input gathered and normed
    and, with a feed-forward, gate / up products and silu, down product; or router, hidden units of the chosen and the shared
    experts, weighted down product (up to eight sequences); then a joint again
then lm_head and arg-max.  More sequences, and prompts, replace the row products by GEMMs; prompts run the tcgen05 attention
and the chunked form of the recurrence.
"""
from __future__ import annotations

import os
from dataclasses import dataclass
from typing import Optional

import torch

from ..ops import dense_moe as X, latent as N, linear_attn as R, stream as K, window_attn as A
from ..ops.kv_cache import DeltaStateShape, KeyValueShape, SlotCache
from .stream_engine import Portions, StreamEngine, StreamStack, _Layer, _Proj


@dataclass
class Joint:
    """How a sublayer meets the streams: their mixture behind it (``mix``, ``w_out``), the weights its input is gathered with
    (``w_in``) and the norm of that input; all fp32."""
    mix: Optional[torch.Tensor]
    w_out: Optional[torch.Tensor]
    w_in: torch.Tensor
    norm: torch.Tensor

    @classmethod
    def of(cls, hyper, norm):
        f = lambda t: t.data.float().contiguous()      # noqa: E731
        return cls(f(hyper.mix), f(hyper.w_out), f(hyper.w_in), f(norm.weight))


class MultiStreamStack(StreamStack):
    components = ("stream", "latent", "attention", "recurrent", "linear")

    def __init__(self, model):
        cfg, base = model.config, model.model
        super().__init__(model, [blk.mixer.in_proj for blk in base.layers])
        dt = self.dtype
        self.streams = int(cfg.streams)
        self.embed_scale = float(cfg.embedding.get("scale", 1.0))
        # the factor of the logits is part of the last norm's weight
        self.final_norm = (base.norm.weight.data.float() * float(cfg.logit_scale)).contiguous()
        self.last = Joint(None, None, torch.ones(self.streams, device=self.device), self.final_norm)
        self.kernel_launches_per_step = 4
        for i, blk in enumerate(base.layers):
            L, m = _Layer(), blk.mixer
            L.layer_idx, L.kind = i, blk.kind
            L.in_proj, L.o = _Proj(m.in_proj, dt), _Proj(m.o_proj, dt)
            L.joint1 = Joint.of(blk.hyper1, blk.norm1)
            (self._latent_layer if blk.kind == "latent_attention" else self._parallel_layer)(L, m)
            self._feed_forward_layer(L, blk)
            self.layers.append(L)
        self.lenders = {L.lender for L in self.layers if getattr(L, "lender", None) is not None}

    def _latent_layer(self, L, m):
        dt = self.dtype
        L.spec = s = N.LatentSpec(m.heads, m.dim, m.rot_dim, m.v_dim, m.kv_rank, m.scale, 0, m.rot_pairs, self.eps)
        L.rot_key, L.lender = (m.rot_base, m.rot_pairs), m.kv_from
        L.q_down, L.q_up = m.q_down.weight.data.to(dt).contiguous(), _Proj(m.q_up, dt)
        L.q_norm = m.q_norm.weight.data.to(dt)
        L.kv_norm = m.kv_norm.weight.data.to(dt) if m.kv_from is None else None
        L.w_uk, L.w_uv = m.k_up.data.to(dt).contiguous(), m.v_up.data.to(dt).contiguous()
        L.kv_rows = m.kv_rows
        L.prefill_fast = s.prefill_ok(dt) and os.environ.get("IPEX_LLM_LATENT_PREFILL", "1") != "0"
        L.store = self._store(s.row(dt)) if m.kv_from is None else self.layers[m.kv_from].store
        self.kernel_launches_per_step += 7

    def _parallel_layer(self, L, m):
        dt = self.dtype
        L.spec, L.linear = m.left, m.right
        L.rot_key = (m.rot_base, m.left.rot_pairs)
        L.sinks = m.sink.data.float().contiguous()
        L.decay_down = m.decay_down.weight.data.to(dt).contiguous()
        L.weights = R.LinearWeights(m.decay_up.data.to(dt), m.decay_bias.data, m.head_norm.weight.data.to(dt), self.eps)
        L.prefill_fast = m.left.prefill_ok(dt)
        L.store = self._store(KeyValueShape(m.left.kv_heads, m.left.dim, m.left.vdim))
        L.state = self._store(DeltaStateShape(m.right.heads, m.right.dim, m.right.vdim, 0, 0))
        self.kernel_launches_per_step += 5

    def _feed_forward_layer(self, L, blk):
        dt, f = self.dtype, blk.mlp
        L.gate_up = L.down = L.bank = L.joint2 = None
        if f is None:
            return
        L.joint2 = Joint.of(blk.hyper2, blk.norm2)
        if not hasattr(f, "experts"):
            L.gate_up, L.down, L.interleaved = _Proj(f.gate_up_proj, dt), _Proj(f.down_proj, dt), f.interleaved
            self.kernel_launches_per_step += 3
            return
        sh = f.shared
        L.bank = X.SoftExpertBank(f.router.weight.data.to(dt), f.experts.gate_up_rows.data.to(dt),
                                  f.experts.down_rows.data.to(dt), f.top_k, f.groups, f.keep, f.scale,
                                  None if sh is None else sh.gate_up_rows.data.to(dt),
                                  None if sh is None else sh.down_rows.data.to(dt))
        self.kernel_launches_per_step += 4

    # -- mixers ---------------------------------------------------------------------------------------
    def _latent(self, L, h, slot, pos, cache, visible, portions, borrowed, pdl):
        s, T = L.spec, h.shape[0]
        proj = self._rows(T, L.in_proj.N)
        cq = torch.empty(T, L.q_down.shape[0], dtype=torch.float32, device=self.device)
        self._linear(L.in_proj, h, proj, K.OUT_ACT, pdl=pdl, w2=L.q_down, out2=cq)
        q = self._rows(T, L.q_up.N)
        self._from_stream(L.q_up, cq, L.q_norm, q, pdl=pdl)
        a = self._rows(T, s.heads * s.v_dim)
        kv = proj[:, :L.kv_rows] if L.lender is None else None
        cos, sin = self._rot[L.rot_key]
        args = (s, q, L.w_uk, L.w_uv, L.kv_norm, cos, sin, slot, pos)
        prompts = portions is not None and portions.whole and T > 8 and L.prefill_fast and \
            (L.lender is None or L.lender in borrowed)
        if prompts:
            rows = N.prompt_rows(s, T, self.dtype, self.device) if L.lender is None else borrowed[L.lender]
            N.latent_prompt(*args, portions.row, portions.length, portions.longest, cache, L.store, a, kv=kv,
                            gate=proj[:, L.kv_rows:], rows_out=rows)
            if L.layer_idx in self.lenders:
                borrowed[L.layer_idx] = rows
        else:
            N.latent_step(*args, cache, L.store, a, visible, pdl=pdl, kv=kv, gate=proj[:, L.kv_rows:])
        return a

    def _parallel(self, L, h, slot, pos, cache, visible, portions, pdl):
        s, r, T = L.spec, L.linear, h.shape[0]
        proj = self._rows(T, s.rows + r.rows)
        low = torch.empty(T, r.rank, dtype=torch.float32, device=self.device)
        self._linear(L.in_proj, h, proj, K.OUT_ACT, pdl=pdl, w2=L.decay_down, out2=low)
        left, right = proj[:, :s.rows], proj[:, s.rows:]
        n = s.heads * s.vdim
        a = self._rows(T, n + r.heads * r.vdim)
        tables = A.AttnTables(L.sinks, *self._rot[L.rot_key])
        if portions is not None and portions.whole and T > 8 and L.prefill_fast:
            A.attend_prompt(s, left, None, slot, pos, portions.row, portions.length, portions.longest, cache, L.store,
                            a[:, :n], tables)
        else:
            A.attend_step(s, left, None, slot, pos, cache, L.store, a[:, :n], s.seen(visible), portions is None, pdl=pdl,
                          tables=tables)
        R.linear_mix(r, L.weights, right, low, slot, pos, cache, L.state, a[:, n:], portions, pdl=pdl)
        return a

    def _feed_forward(self, L, h, y, pdl):
        if L.bank is not None:
            if L.bank.rows_ok(h.shape[0]):
                return X.soft_moe_rows(L.bank, h, y, pdl=pdl)
            return X.soft_moe_grouped(L.bank, h, y)
        u = self._rows(h.shape[0], L.gate_up.N // 2)
        self._linear(L.gate_up, h, u, K.OUT_ACT, act=K.ACT_SILU_GLU, pdl=pdl, interleaved=L.interleaved)
        return self._linear(L.down, u, y, K.OUT_F32, pdl=pdl)

    # -- pass -----------------------------------------------------------------------------------------
    def _join(self, x, y, behind: Optional[Joint], before: Joint, pdl=False):
        mix, out = (None, None) if behind is None else (behind.mix, behind.w_out)
        return K.hyper_joint(x, y, mix, out, before.w_in, before.norm, self.eps, self.dtype, pdl=pdl)

    def run(self, tokens, slot, pos, cache: SlotCache, visible: int, portions: Optional[Portions] = None, pdl=False,
            collect=None):
        """As ``StreamStack.run``; the streams are ``[T, streams, width]``, ``collect`` receives their sum."""
        T, S, W = tokens.shape[0], self.streams, self.W
        x = K.embed_stream(tokens, slot, pos, cache, self.embed, self.embed_scale, pdl=pdl, streams=S).view(T, S, W)
        y = torch.empty(T, W, dtype=torch.float32, device=self.device)
        h = self._join(x, None, None, self.layers[0].joint1 if self.layers else self.last, pdl)
        borrowed = {}            # latents and key parts of this pass's prompts, by the layer they belong to
        for L, nxt in zip(self.layers, self.layers[1:] + [None]):
            after = self.last if nxt is None else nxt.joint1
            if L.kind == "latent_attention":
                a = self._latent(L, h, slot, pos, cache, visible, portions, borrowed, pdl)
            else:
                a = self._parallel(L, h, slot, pos, cache, visible, portions, pdl)
            self._linear(L.o, a, y, K.OUT_F32, pdl=pdl)
            h = self._join(x, y, L.joint1, L.joint2 or after, pdl)
            if L.joint2 is not None:
                self._feed_forward(L, h, y, pdl)
                h = self._join(x, y, L.joint2, after, pdl)
            if collect is not None:
                collect.append(x.sum(1))
        return x, h

    def logits(self, x, rows=None, out=None, pdl=False, h=None):
        if h is None:
            x = x if rows is None else x[rows.long()]
            h, rows = self._join(x, None, None, self.last, pdl), None
        return super().logits(x, rows, out, pdl, h)


class MultiStreamEngine(StreamEngine):
    stack_cls = MultiStreamStack
