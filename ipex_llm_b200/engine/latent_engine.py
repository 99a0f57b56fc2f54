"""Engine for decoders with multi-head latent attention and a 32-bit residual stream (family engine ``latent``).

``LatentStack`` is the flattened model: it runs any set of sequence portions - whole prompts, one token each, or
anything between - as one packed batch of tokens, without padding rows, against a ``LatentCache``.  ``LatentEngine``
puts the framework's decode loop around it (static buffers, one CUDA-graph replay per token, the interface of
``DecoderEngine``).

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
from typing import List, Optional, Sequence, Tuple

import torch

from ..ops import cuda_ops, latent as K
from ..ops.kv_cache import LatentCache
from ..ops.linear import LowBitLinear
from .decoder_engine import DecoderEngine, _W


class _Proj:
    """One linear of the stack: a dense matrix in the stack's dtype, or packed low-bit tiles."""

    def __init__(self, mod, dtype):
        self.packed = _W.from_module(mod, dtype) if isinstance(mod, LowBitLinear) else None
        w = None if self.packed is not None else mod.weight.data
        self.w = None if w is None else w.to(dtype).contiguous()
        self.N, self.K = (self.packed.N, self.packed.K) if self.packed is not None else self.w.shape
        self.tp = None


class _Layer:
    pass


def stack_for(model) -> "LatentStack":
    stack = getattr(model, "_ipex_stack", None)
    dev = next(model.parameters()).device
    if stack is None or stack.device != dev:
        stack = LatentStack(model)
        model._ipex_stack = stack
    return stack


class LatentStack:
    def __init__(self, model):
        cfg, base = model.config, model.model
        self.device = next(model.parameters()).device
        if self.device.type != "cuda":
            raise RuntimeError("latent-attention decoders run on CUDA only: call model.to('cuda')")
        self.config = cfg
        self.dtype = dt = self._dtype(model)
        self.eps = float(cfg.norm["eps"])
        self.W, self.vocab = int(cfg.width), int(cfg.vocab)
        self.softcap = float(cfg.logit_softcap or 0.0)
        emb = cfg.embedding
        self.embed_scale = float(emb.get("scale", 1.0))
        self.embed = base.embed_tokens.weight.data.to(dt).contiguous()
        self.bigram = base.bigram.weight.data.to(dt).contiguous() if base.bigram is not None else None
        b = emb.get("bigram") or {}
        self.bigram_args = (int(b.get("buckets", 0)), int(b.get("mul_prev", 0)), int(b.get("mul_cur", 0)))
        self.final_norm = base.norm.weight.data.to(dt)
        self.lm_head = _Proj(model.lm_head, dt)
        self.layers: List[_Layer] = []
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
        self.row_widths = [L.spec.row(dt) for L in self.layers]
        self._rot = {}           # (base, pairs) -> (positions, cos, sin)
        self._rot_retired = []   # tables a captured graph may still read
        self._positions = 0

    @staticmethod
    def _dtype(model):
        """The dtype of the projections: what a bf16 / fp16 / plain linear holds, bf16 around packed weights."""
        mods = [blk.mixer.qkv_a_proj for blk in model.model.layers] + [model.lm_head]
        for mod in mods:
            if not isinstance(mod, LowBitLinear):
                return mod.weight.dtype if mod.weight.dtype != torch.float64 else torch.float32
        return torch.bfloat16

    # ------------------------------------------------------------------------------------------------
    def ensure_positions(self, n: int):
        if n <= self._positions and self._rot:
            return
        n = max(2048, (n + 1023) // 1024 * 1024)
        self._rot_retired.append(self._rot)
        self._rot = {L.rot_key: K.rotary_table(n, *L.rot_key, self.device) for L in self.layers}
        self._positions = n

    # ------------------------------------------------------------------------------------------------
    # products
    # ------------------------------------------------------------------------------------------------
    def _few(self, P: _Proj, M: int) -> bool:
        return P.packed is None and M <= K.rows_max(P.K, self.dtype)

    def _from_stream(self, P: _Proj, x, norm, out, act=0, h=None, pdl=False):
        """``out = act(norm(x) @ w.T)`` in the activation dtype."""
        if self._few(P, x.shape[0]):
            return K.gemv_rows(P.w, x, out, K.OUT_ACT, norm=norm, eps=self.eps, act=act, pdl=pdl)
        h = K.norm_stream(x, norm, self.eps) if h is None else h
        return self._product(P, h, out, K.OUT_ACT, act)

    def _to_stream(self, P: _Proj, a, x, pdl=False):
        """``x += a @ w.T``."""
        if self._few(P, x.shape[0]):
            return K.gemv_rows(P.w, a, x, K.OUT_ADD, pdl=pdl)
        return self._product(P, a, x, K.OUT_ADD)

    def _product(self, P: _Proj, h, out, mode, act=0):
        if P.packed is None:
            return K.gemm(h, P.w, out, mode, act)
        w, M = P.packed, h.shape[0]
        y = out if mode == K.OUT_ACT else torch.empty(M, w.N, dtype=h.dtype, device=h.device)
        if M <= cuda_ops.GEMV_MAX_M:
            per = cuda_ops._gemv_rows_per_call(w.K)
            for s in range(0, M, per):
                cuda_ops.gemv_lowbit(h[s:s + per], w.data, w.qtype, w.N, w.K, out=y[s:s + per], wf=w.wf)
        else:
            cuda_ops.gemm_lowbit(h, w.data, w.qtype, w.N, w.K, out=y)
        if mode == K.OUT_ACT:
            return K.relu2_(y) if act == K.ACT_RELU2 else y
        return K.add_stream_(out, y) if mode == K.OUT_ADD else out.copy_(y)

    # ------------------------------------------------------------------------------------------------
    # one pass over packed tokens
    # ------------------------------------------------------------------------------------------------
    def run(self, tokens, slot, pos, cache: LatentCache, visible: int, prompts: Optional[tuple] = None, pdl=False,
            collect=None):
        """The residual stream ``[T, width]`` after the last layer for ``tokens`` (int64) at cache rows ``slot`` and
        positions ``pos`` (int32).  Tokens of a sequence are in order.  ``visible``: an upper bound of the keys a token
        can see.  ``prompts = (seq_row, seq_len, longest)`` says that the tokens are whole sequences from their first
        token on, packed in that order.  ``collect``: a list that receives the stream after every layer."""
        T, dev, dt = tokens.shape[0], self.device, self.dtype
        x = K.embed_stream(tokens, slot, pos, cache, self.embed, self.embed_scale, self.bigram, *self.bigram_args,
                           pdl=pdl)
        for L in self.layers:
            s = L.spec
            cos, sin = self._rot[L.rot_key]
            qkv = torch.empty(T, (L.qkv.N + 7) // 8 * 8, dtype=dt, device=dev)[:, :L.qkv.N]
            a = torch.empty(T, s.heads * s.v_dim, dtype=dt, device=dev)
            self._from_stream(L.qkv, x, L.norm1, qkv, pdl=pdl)
            args = (s, qkv, L.w_uk, L.w_uv, L.kv_norm, cos, sin, slot, pos)
            if prompts is not None and L.prefill_fast:
                K.latent_prompt(*args, *prompts, cache, L.layer_idx, a)
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
        return x

    def logits(self, x, rows=None, out=None, pdl=False):
        """Soft-capped fp32 logits of the stream's rows (of ``rows``, int32, when given)."""
        n = x.shape[0] if rows is None else rows.shape[0]
        if out is None:
            out = torch.empty(n, self.vocab, dtype=torch.float32, device=self.device)
        if rows is None and self._few(self.lm_head, n):
            return K.gemv_rows(self.lm_head.w, x, out, K.OUT_F32, norm=self.final_norm, eps=self.eps,
                               softcap=self.softcap, pdl=pdl)
        h = K.norm_stream(x, self.final_norm, self.eps, rows=rows)
        if self._few(self.lm_head, n):
            return K.gemv_rows(self.lm_head.w, h, out, K.OUT_F32, softcap=self.softcap)
        self._product(self.lm_head, h, out, K.OUT_F32)
        return K.softcap_(out, self.softcap) if self.softcap > 0 else out

    def run_portions(self, portions: Sequence[Tuple[int, int, Sequence[int]]], cache: LatentCache, collect=None):
        """Run ``(slot, first position, token ids)`` portions as one packed batch; returns the stream.  Token ids may be
        lists or int64 tensors on the device.  Positions count from the cache's first row of the slot."""
        lens = [len(p[2]) for p in portions]
        T, dev = sum(lens), self.device
        meta = torch.empty(2 * T + 2 * len(portions), dtype=torch.int32)
        slot, pos, row, ln = meta.split([T, T, len(portions), len(portions)])
        at = 0
        for i, ((s, p0, _), n) in enumerate(zip(portions, lens)):
            slot[at:at + n] = s
            pos[at:at + n] = torch.arange(p0, p0 + n, dtype=torch.int32)
            row[i], ln[i] = at, n
            at += n
        if isinstance(portions[0][2], torch.Tensor):
            tokens = torch.cat([p[2].to(dev) for p in portions])
        else:
            tokens = torch.tensor([t for p in portions for t in p[2]], dtype=torch.int64).to(dev)
        slot, pos, row, ln = meta.to(dev).split([T, T, len(portions), len(portions)])
        longest = max(p0 + n for (_, p0, _), n in zip(portions, lens))
        self.ensure_positions(longest)
        # few tokens (or continued sequences) go through the absorbed attention, whole prompts through the expanded one
        whole = T > 8 and all(p0 == cache.first_row(s) for s, p0, _ in portions)
        return self.run(tokens, slot, pos, cache, longest, prompts=(row, ln, max(lens)) if whole else None,
                        collect=collect)

    # ------------------------------------------------------------------------------------------------
    # the transformers calling convention: padded batch, growing cache
    # ------------------------------------------------------------------------------------------------
    def forward_padded(self, input_ids, attention_mask, cache: LatentCache, logits_to_keep=0):
        B, S = input_ids.shape
        past = cache.get_seq_length()
        if cache.layers and (cache.layers[0]._k.dtype != self.dtype or cache.slots != B or
                             [layer._k.shape[-1] for layer in cache.layers] != self.row_widths):
            raise TypeError(f"the cache was filled by another model or batch: {cache.slots} x {cache.layers[0]._k.dtype}"
                            f", this call needs {B} x {self.dtype} of the same row widths")
        cache.allocate(B, self._grown(cache, past + S), self.row_widths, self.dtype, self.device)
        if past == 0:
            pads = [0] * B
            if attention_mask is not None:
                seen = (attention_mask[:, :S] != 0).int().cummax(dim=1).values
                pads = (S - seen.sum(dim=1)).tolist()
            cache.set_first_rows(pads)
        portions, place = [], []
        for b in range(B):
            skip = min(max(0, cache.first_row(b) - past), S)
            if skip < S:
                portions.append((b, past + skip, input_ids[b, skip:]))
                place.append((b, skip))
        cache.advance_all(past + S)
        keep = torch.arange(S)
        if isinstance(logits_to_keep, torch.Tensor):
            keep = keep[logits_to_keep.cpu()]
        elif logits_to_keep:
            keep = keep[-int(logits_to_keep):]
        out = torch.zeros(B, keep.numel(), self.vocab, dtype=torch.float32, device=self.device)
        if not portions:
            return out
        x = self.run_portions(portions, cache)
        rows, dest, at = [], [], 0
        for b, skip in place:
            for j, p in enumerate(keep.tolist()):
                if p >= skip:
                    rows.append(at + p - skip)
                    dest.append(b * keep.numel() + j)
            at += S - skip
        if rows:
            lg = self.logits(x, torch.tensor(rows, dtype=torch.int32, device=self.device))
            out.view(-1, self.vocab)[torch.tensor(dest, device=self.device)] = lg
        return out

    @staticmethod
    def _grown(cache, need: int) -> int:
        from ..ops.kv_cache import KV_CACHE_ALLOC_BLOCK_LENGTH
        return cache.capacity if need <= cache.capacity else need + KV_CACHE_ALLOC_BLOCK_LENGTH


class LatentEngine(DecoderEngine):
    """``DecoderEngine``'s interface (prefill, graph-replayed decode steps, caches) over a ``LatentStack``.  Batches may
    be ragged: rows carry their own lengths, so padded prompts stay on the engine."""

    ragged = True

    def __init__(self, model, max_batch: int = 1, max_len: int = 2048):
        self.model, self.cfg = model, model.config
        self.stack = stack = stack_for(model)
        self.device, self.dtype, self.vocab = stack.device, stack.dtype, stack.vocab
        self.layers = stack.layers
        self.max_batch, self.max_len = max_batch, max_len
        self.first_stage = self.last_stage = True
        self.lm_gather = None
        self.use_pdl = os.environ.get("IPEX_LLM_PDL", "1") != "0"
        B, dev = max_batch, self.device
        self.tokens = torch.zeros(B, dtype=torch.int64, device=dev)
        self.past_len = torch.zeros(B, dtype=torch.int32, device=dev)      # position of each row's next token
        self.row_slot = torch.zeros(B, dtype=torch.int32, device=dev)
        self.logits = torch.zeros(B, self.vocab, dtype=torch.float32, device=dev)
        self.cache: Optional[LatentCache] = None
        self.batch = 0
        self._slots: List[int] = []          # host copy of row_slot[:batch]
        self._bound_lengths = None           # ... and of past_len[:batch], None when it is not known
        self._graphs = {}
        self._nsplit = None
        self._visible = max_len
        self._mega = False
        stack.ensure_positions(max_len)

    @property
    def kernel_launches_per_step(self) -> int:
        return 3 + sum(5 + (3 if L.bank is not None else 2 if L.up is not None else 0) for L in self.layers)

    def mega_step(self, B: int):
        return None

    # -- cache ----------------------------------------------------------------------------------------
    def new_cache(self, batch: int):
        """The engine's cache, emptied; it grows to ``batch`` slots when it has fewer."""
        self.open_cache(batch)
        self.cache.release_all()
        return self.cache

    def open_cache(self, slots: int):
        if self.cache is None:
            self.cache = LatentCache(self.cfg)
        if self.cache.allocate(slots, self.max_len, self.stack.row_widths, self.dtype, self.device):
            self._graphs = {}

    def bind_rows(self, slots: Sequence[int], lengths: Sequence[int]):
        """Rows ``0 .. len(slots)`` of the decode batch are the sequences in these cache slots, which hold ``lengths``
        tokens; a batch from which sequences have left is bound again with the remaining ones."""
        n = len(slots)
        self.batch, self._slots, self._bound_lengths = n, list(slots), list(lengths)
        self.row_slot[:n] = torch.tensor(self._slots, dtype=torch.int32, device=self.device)
        self.past_len[:n] = torch.tensor(self._bound_lengths, dtype=torch.int32, device=self.device)

    def sync_cache_length(self, n: int):
        for layer in self.cache.layers:
            layer.set_length(n)

    # -- prompts and portions -------------------------------------------------------------------------
    @torch.no_grad()
    def prefill(self, input_ids: torch.Tensor, attention_mask=None):
        B, S = input_ids.shape
        if S + 1 > self.max_len:
            raise ValueError(f"prompt of {S} tokens does not fit max_len={self.max_len}")
        self.new_cache(B)
        pads = [0] * B
        if attention_mask is not None:
            seen = (attention_mask != 0).int().cummax(dim=1).values
            pads = (S - seen.sum(dim=1)).tolist()
        slots = [self.cache.acquire() for _ in range(B)]
        portions = [(s, 0, input_ids[b, pads[b]:]) for b, s in enumerate(slots) if pads[b] < S]
        if len(portions) < B:
            raise ValueError("a row of the batch holds no token")
        x = self.stack.run_portions(portions, self.cache)
        lens = [S - p for p in pads]
        for s, n in zip(slots, lens):
            self.cache.lengths[s] = n
        self.bind_rows(slots, lens)
        self._visible = S
        last = torch.tensor(lens).cumsum(0).sub(1).to(torch.int32).to(self.device)
        return self.stack.logits(x, last)

    @torch.no_grad()
    def step_rows(self, entries, use_graph: bool = True):
        """Feed given tokens: ``entries`` is a list of ``(slot, token ids, wanted places)``, one per sequence.  Runs the
        whole step as one batch from what the slots hold and returns the fp32 logits ``[wanted, vocab]`` in that
        order (None when nothing is wanted).  Steps of one token per started sequence go through ``decode_step``."""
        cache = self.cache
        lengths = [cache.lengths[s] for s, _, _ in entries]
        for (s, toks, _), n in zip(entries, lengths):
            if n + len(toks) > cache.capacity:
                raise ValueError(f"slot {s} would hold {n + len(toks)} tokens, the cache has room for {cache.capacity}")
        if all(len(t) == 1 and n > 0 for (_, t, _), n in zip(entries, lengths)) and len(entries) <= self.max_batch:
            slots = [s for s, _, _ in entries]
            if slots != self._slots or self._bound_lengths != lengths:
                self.bind_rows(slots, lengths)
            self.tokens[:len(slots)] = torch.tensor([t[0] for _, t, _ in entries], device=self.device)
            self._visible = max(lengths) + 1
            self.decode_step(len(slots), use_graph=use_graph)
            self._bound_lengths = [n + 1 for n in lengths]
            rows = [i for i, (_, _, w) in enumerate(entries) for _ in w]
            out = self.logits[rows] if rows else None
        else:
            self._bound_lengths = None
            x = self.stack.run_portions([(s, n, list(t)) for (s, t, _), n in zip(entries, lengths)], cache)
            rows, at = [], 0
            for _, t, w in entries:
                rows += [at + j for j in w]
                at += len(t)
            out = self.stack.logits(x, torch.tensor(rows, dtype=torch.int32, device=self.device)) if rows else None
        for s, t, _ in entries:
            cache.lengths[s] += len(t)
        return out

    # -- decode ---------------------------------------------------------------------------------------
    def decode_step(self, B: int, use_graph: bool = True):
        self._bound_lengths = None
        super().decode_step(B, use_graph)

    def _pick_splits(self, B: int) -> int:
        """Bound of the visible keys the attention splits are sized for: the next power of two above the context this
        generation reaches soon (part of the graph key)."""
        target = 512
        while target < min(self._visible + 256, self.max_len):
            target *= 2
        return target

    def _step_kernels(self, B: int):
        pdl = self.use_pdl
        x = self.stack.run(self.tokens[:B], self.row_slot[:B], self.past_len[:B], self.cache, self._nsplit, pdl=pdl)
        self.stack.logits(x, out=self.logits[:B], pdl=pdl)
        K.argmax_rows(self.logits[:B], self.tokens[:B], pdl=pdl)
        self.past_len[:B].add_(1)

    def _tp_comm(self):
        return None

    def verify_step(self, S: int, use_graph: bool = True):
        raise NotImplementedError("self-speculative decoding is not wired up for latent attention")

    def clone_for_microbatch(self):
        raise NotImplementedError("pipeline stages are not wired up for latent attention")

    def prefill_stage(self, x):
        raise NotImplementedError("pipeline stages are not wired up for latent attention")
