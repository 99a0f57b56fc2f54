"""What the engines of decoders with a 32-bit residual stream share.

``StreamStack`` is the base of a flattened model: it runs any set of sequence portions - whole prompts, one token each, or
anything between - as one packed batch of tokens, without padding rows, against a ``SlotCache``.  A family's stack adds
its layers and the pass over them (``run``).  ``StreamEngine`` puts the framework's decode loop around a stack (static
buffers, one CUDA-graph replay per token, the interface of ``DecoderEngine``).
"""
from __future__ import annotations

import os
from dataclasses import dataclass, field
from typing import List, Optional, Sequence, Tuple

import torch

from ..native.lib import prepare_components
from ..ops import cuda_ops, stream as K
from ..ops.latent import rotary_table
from ..ops.kv_cache import SlotCache
from ..ops.linear import LowBitLinear
from .decoder_engine import DecoderEngine, _W


class _Proj:
    """One linear of the stack: a dense matrix in the stack's dtype, or packed low-bit tiles."""

    def __init__(self, mod, dtype):
        self.packed = _W.from_module(mod, dtype) if isinstance(mod, LowBitLinear) else None
        w = None if self.packed is not None else mod.weight.data
        self.w = None if w is None else w.to(dtype).contiguous()
        self.bias = mod.bias.data.to(dtype).contiguous() if getattr(mod, "bias", None) is not None else None
        self.N, self.K = (self.packed.N, self.packed.K) if self.packed is not None else self.w.shape
        self.tp = None


class _Layer:
    pass


@dataclass
class Portions:
    """Sequence portions behind one another in a packed batch: device tables (int32) and what the host knows of them."""
    row: torch.Tensor            # [n] first packed token of every portion
    length: torch.Tensor         # [n]
    longest: int
    whole: bool                  # every portion starts with its sequence's first token
    chunk_seq: torch.Tensor      # [chunks] portion of every chunk of CHUNK tokens
    seq_chunk: torch.Tensor      # [n + 1] first chunk of every portion
    chunks: int
    lengths: Optional[List[int]] = None      # ``length`` on the host
    _pool_rows: dict = field(default_factory=dict)

    CHUNK = 32

    def pool_rows(self, pool: int):
        """Where the blocks of ``pool`` tokens of every (whole) portion go when they are packed: first rows, multiples of eight
        (int32, device), and the number of all rows."""
        if pool not in self._pool_rows:
            lengths = self.length.tolist() if self.lengths is None else self.lengths
            first, n = [], 0
            for m in lengths:
                first.append(n)
                n += (m // pool + 7) // 8 * 8
            self._pool_rows[pool] = torch.tensor(first, dtype=torch.int32, device=self.row.device), max(n, 8)
        return self._pool_rows[pool]


def stack_for(model, cls) -> "StreamStack":
    stack = getattr(model, "_ipex_stack", None)
    dev = next(model.parameters()).device
    if stack is None or stack.device != dev:
        stack = cls(model)
        model._ipex_stack = stack
    return stack


class StreamStack:
    cache_cls = SlotCache
    components = ("stream",)         # parts of the kernel library the family needs (native/build.py)
    softcap = 0.0
    kernel_launches_per_step = 0

    def __init__(self, model, linears):
        """``linears``: the modules whose dtype is the stack's."""
        cfg, base = model.config, model.model
        self.device = next(model.parameters()).device
        if self.device.type != "cuda":
            raise RuntimeError(f"{type(model).__name__} runs on CUDA only: call model.to('cuda')")
        prepare_components(*self.components)
        self.config = cfg
        self.dtype = dt = self._dtype([*linears, model.lm_head])
        self.eps = float(cfg.norm["eps"])
        self.W, self.vocab = int(cfg.width), int(cfg.vocab)
        self.embed = base.embed_tokens.weight.data.to(dt).contiguous()
        self.lm_head = _Proj(model.lm_head, dt)
        self.layers: List[_Layer] = []
        self.shapes = []             # of the layers' cache storage
        self.final_norm = None
        self._rot = {}               # (base, pairs) -> (cos, sin), of the layers' ``rot_key``
        self._rot_retired = []       # tables a captured graph may still read
        self._positions = 0

    @staticmethod
    def _dtype(mods):
        """The dtype of the projections: what a bf16 / fp16 / plain linear holds, bf16 around packed weights."""
        for mod in mods:
            if not isinstance(mod, LowBitLinear):
                return mod.weight.dtype if mod.weight.dtype != torch.float64 else torch.float32
        return torch.bfloat16

    def ensure_positions(self, n: int):
        """Rotation tables for positions below ``n`` (families whose layers have none need nothing)."""
        keys = {L.rot_key for L in self.layers if getattr(L, "rot_key", None) is not None}
        if not keys or (n <= self._positions and self._rot):
            return
        n = max(2048, (n + 1023) // 1024 * 1024)
        self._rot_retired.append(self._rot)
        self._rot = {key: rotary_table(n, *key, self.device) for key in keys}
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
        return self._linear(P, a, x, K.OUT_ADD, pdl=pdl)

    def _rows(self, T: int, n: int):
        """An activation of ``n`` columns whose rows start on 16-byte boundaries."""
        return torch.empty(T, (n + 7) // 8 * 8, dtype=self.dtype, device=self.device)[:, :n]

    def _store(self, shape) -> int:
        """Add storage to the cache's layers; returns its index."""
        self.shapes.append(shape)
        return len(self.shapes) - 1

    def _linear(self, P: _Proj, h, out, mode, act=0, pdl=False, interleaved=True, w2=None, out2=None, args=K.NO_ARGS):
        """``act(h @ w.T + bias)`` into ``out`` (see ``OUT_*``); ``w2`` / ``out2``: further dense rows with fp32 results."""
        # (the tensor-core row product, which takes up to sixteen rows, wants gate and up rows in blocks)
        if self._few(P, h.shape[0]) and (interleaved or h.shape[0] <= 8):
            return K.gemv_rows(P.w, h, out, mode, act=act, pdl=pdl, bias=P.bias, w2=w2, out2=out2, interleaved=interleaved,
                               args=args)
        if w2 is not None and P.packed is None:
            return K.gemm(h, P.w, out, mode, act, P.bias, interleaved, w2, out2, args)
        if w2 is not None:
            if h.shape[0] <= K.rows_max(w2.shape[1], self.dtype):
                K.gemv_rows(w2, h, out2, K.OUT_F32)
            else:
                K.gemm(h, w2, out2, K.OUT_F32)
        return self._product(P, h, out, mode, act, interleaved, args)

    def _product(self, P: _Proj, h, out, mode, act=0, interleaved=True, args=K.NO_ARGS):
        if P.packed is None:
            return K.gemm(h, P.w, out, mode, act, P.bias, interleaved, args=args)
        w, M, h = P.packed, h.shape[0], h.contiguous()
        glu = act in K.GATED_ACTS
        y = out if mode == K.OUT_ACT and not glu and out.is_contiguous() else torch.empty(M, w.N, dtype=h.dtype, device=h.device)
        if M <= cuda_ops.GEMV_MAX_M:
            per = cuda_ops._gemv_rows_per_call(w.K)
            for s in range(0, M, per):
                cuda_ops.gemv_lowbit(h[s:s + per], w.data, w.qtype, w.N, w.K, out=y[s:s + per], wf=w.wf)
        else:
            cuda_ops.gemm_lowbit(h, w.data, w.qtype, w.N, w.K, out=y)
        if glu:
            return K.glu_rows(y, P.bias, out, act, interleaved, args)
        if P.bias is not None:
            K.bias_rows_(y, P.bias)
        if mode == K.OUT_ACT:
            out = y if y is out else out.copy_(y)
            return K.act_rows_(out, act, args) if act in (K.ACT_RELU2, K.ACT_GELU_MUL) else out
        return K.add_stream_(out, y) if mode == K.OUT_ADD else out.copy_(y)

    # ------------------------------------------------------------------------------------------------
    # one pass over packed tokens
    # ------------------------------------------------------------------------------------------------
    def run(self, tokens, slot, pos, cache: SlotCache, visible: int, portions: Optional[Portions] = None, pdl=False,
            collect=None):
        """The residual stream ``[T, width]`` after the last layer for ``tokens`` (int64) at cache rows ``slot`` and
        positions ``pos`` (int32), and the same behind the final norm (None when the pass does not produce it).  Tokens
        of a sequence are in order.  ``visible``: an upper bound of the keys a token can see.  ``portions``: how the
        tokens belong together; without it every token is a sequence's next one.  ``collect``: a list that receives the
        stream after every layer."""
        raise NotImplementedError

    def logits(self, x, rows=None, out=None, pdl=False, h=None):
        """Soft-capped fp32 logits of the stream's rows (of ``rows``, int32, when given); ``h``: the stream behind the
        final norm, when it is at hand."""
        n = x.shape[0] if rows is None else rows.shape[0]
        if out is None:
            out = torch.empty(n, self.vocab, dtype=torch.float32, device=self.device)
        few = self._few(self.lm_head, n)
        if h is None and rows is None and few and self.final_norm.dtype == self.dtype:
            return K.gemv_rows(self.lm_head.w, x, out, K.OUT_F32, norm=self.final_norm, eps=self.eps,
                               softcap=self.softcap, pdl=pdl)
        if h is None:
            h = K.norm_stream(x, self.final_norm, self.eps, rows=rows, pdl=pdl, dtype=self.dtype)
        elif rows is not None:
            h = h[rows.long()]
        if few:
            return K.gemv_rows(self.lm_head.w, h, out, K.OUT_F32, softcap=self.softcap, pdl=pdl)
        self._product(self.lm_head, h, out, K.OUT_F32)
        return K.softcap_(out, self.softcap) if self.softcap > 0 else out

    def run_portions(self, portions: Sequence[Tuple[int, int, Sequence[int]]], cache: SlotCache, collect=None):
        """Run ``(slot, first position, token ids)`` portions as one packed batch; returns the stream.  Token ids may be
        lists or int64 tensors on the device.  Positions count from the cache's first row of the slot."""
        lens = [len(p[2]) for p in portions]
        n, T, dev = len(portions), sum(lens), self.device
        per = [-(-m // Portions.CHUNK) for m in lens]
        sizes = [T, T, n, n, n + 1, sum(per)]
        meta = torch.empty(sum(sizes), dtype=torch.int32)
        slot, pos, row, ln, first_chunk, owner = meta.split(sizes)
        first_chunk[0] = 0
        at = c = 0
        for i, ((s, p0, _), m) in enumerate(zip(portions, lens)):
            slot[at:at + m] = s
            pos[at:at + m] = torch.arange(p0, p0 + m, dtype=torch.int32)
            row[i], ln[i] = at, m
            owner[c:c + per[i]] = i
            at, c = at + m, c + per[i]
            first_chunk[i + 1] = c
        if isinstance(portions[0][2], torch.Tensor):
            tokens = torch.cat([p[2].to(dev) for p in portions])
        else:
            tokens = torch.tensor([t for p in portions for t in p[2]], dtype=torch.int64).to(dev)
        slot, pos, row, ln, first_chunk, owner = meta.to(dev).split(sizes)
        longest = max(p0 + m for (_, p0, _), m in zip(portions, lens))
        self.ensure_positions(longest)
        whole = all(p0 == cache.first_row(s) for s, p0, _ in portions)
        where = Portions(row, ln, max(lens), whole, owner, first_chunk, sum(per), lens)
        return self.run(tokens, slot, pos, cache, longest, portions=where, collect=collect)[0]

    # ------------------------------------------------------------------------------------------------
    # the transformers calling convention: padded batch, growing cache
    # ------------------------------------------------------------------------------------------------
    def forward_padded(self, input_ids, attention_mask, cache: SlotCache, logits_to_keep=0):
        B, S = input_ids.shape
        past = cache.get_seq_length()
        if cache.layers and (cache.dtype != self.dtype or cache.slots != B or cache.shapes != self.shapes):
            raise TypeError(f"the cache was filled by another model or batch: {cache.slots} x {cache.dtype}, this call "
                            f"needs {B} x {self.dtype} of the same layer shapes")
        cache.allocate(B, self._grown(cache, past + S), self.shapes, self.dtype, self.device)
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


class StreamEngine(DecoderEngine):
    """``DecoderEngine``'s interface (prefill, graph-replayed decode steps, caches) over a ``StreamStack``.  Batches may
    be ragged: rows carry their own lengths, so padded prompts stay on the engine."""

    stack_cls = StreamStack

    ragged = True

    def __init__(self, model, max_batch: int = 1, max_len: int = 2048):
        self.model, self.cfg = model, model.config
        self.stack = stack = stack_for(model, self.stack_cls)
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
        self.cache: Optional[SlotCache] = None
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
        return self.stack.kernel_launches_per_step

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
            self.cache = self.stack.cache_cls(self.cfg)
        if self.cache.allocate(slots, self.max_len, self.stack.shapes, self.dtype, self.device):
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
        x, h = self.stack.run(self.tokens[:B], self.row_slot[:B], self.past_len[:B], self.cache, self._nsplit, pdl=pdl)
        self.stack.logits(x, out=self.logits[:B], pdl=pdl, h=h)
        K.argmax_rows(self.logits[:B], self.tokens[:B], pdl=pdl)
        self.past_len[:B].add_(1)

    def _step_state(self):
        return self.cache.step_state()

    def _tp_comm(self):
        return None

    def verify_step(self, S: int, use_graph: bool = True):
        raise NotImplementedError("self-speculative decoding is not wired up for this family")

    def clone_for_microbatch(self):
        raise NotImplementedError("pipeline stages are not wired up for this family")

    def prefill_stage(self, x):
        raise NotImplementedError("pipeline stages are not wired up for this family")
