"""Letarax on the GPU: every kernel against the float64 oracle (``tests/letarax_oracle.py``), then the engine with whole
prompts, portions, ragged batches, slot reuse, long decoding and generation."""
import json
import os

import pytest
import torch

import letarax_oracle as O

pytestmark = pytest.mark.gpu

F32, BF16, F16 = torch.float32, torch.bfloat16, torch.float16
TOL = {F32: 2e-5, F16: 4e-3, BF16: 2.5e-2}          # relative to the size of the compared values


@pytest.fixture(autouse=True)
def _no_expired_wait():
    yield
    from ipex_llm_b200.ops.cuda_ops import check_error_flag
    check_error_flag(torch.device("cuda", 0))


def close(got, want, dtype, what="", factor=1.0):
    got, want = got.double().cpu(), want.double().cpu()
    assert torch.isfinite(got).all(), what
    err = (got - want).abs().max().item() / max(want.abs().max().item(), 1e-3)
    assert err < TOL[dtype] * factor, f"{what}: {err}"


def gen(seed):
    return torch.Generator().manual_seed(seed)


def rnd(*shape, seed=0, dtype=F32, gain=1.0):
    """Random values that the dtype can hold, as float64."""
    return (torch.randn(*shape, generator=gen(seed)) * gain).to(dtype).double()


def i32(v):
    return torch.tensor(v, dtype=torch.int32, device="cuda")


# ------------------------------------------------------------------------------------------------
# products with biases and gated units, the joint between two sublayers
# ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF16, F16])
@pytest.mark.parametrize("M,ff,K", [(1, 24, 40), (2, 2400, 136), (7, 32, 72), (13, 520, 64), (3, 21, 60), (40, 72, 200),
                                    (150, 136, 520), (33, 19, 72)])
def test_gated_unit_with_biases(dtype, M, ff, K):
    from ipex_llm_b200.models.letarax import interleave_gate_up
    from ipex_llm_b200.ops import stream as S
    g, u = rnd(ff, K, seed=1, dtype=dtype, gain=K ** -0.5), rnd(ff, K, seed=2, dtype=dtype, gain=K ** -0.5)
    bg, bu = rnd(ff, seed=3, dtype=dtype), rnd(ff, seed=4, dtype=dtype)
    x = rnd(M, K, seed=5, dtype=dtype, gain=2.0)
    want = O.gelu_tanh(x @ g.T + bg) * (x @ u.T + bu)
    W, B = interleave_gate_up(g, u).to("cuda", dtype), interleave_gate_up(bg, bu).to("cuda", dtype)
    X = x.to("cuda", dtype)
    out = torch.empty(M, ff, dtype=dtype, device="cuda")
    il = ff % 8 == 0
    if M <= S.rows_max(K, dtype):
        close(S.gemv_rows(W, X, out, S.OUT_ACT, act=S.ACT_GELU_GLU, bias=B, interleaved=il), want, dtype, "rows")
    close(S.gemm(X, W, torch.empty_like(out), S.OUT_ACT, S.ACT_GELU_GLU, B, il), want, dtype, "gemm")
    gu = (X.float() @ W.float().t()).to(dtype)
    close(S.glu_rows(gu, B, torch.empty_like(out), S.ACT_GELU_GLU, il), want, dtype, "from finished products", 2)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("M,N,K,N2", [(1, 97, 136, 5), (3, 40, 60, 12), (11, 2500, 520, 64), (2, 33, 7, 1), (7, 136, 1536, 4), (40, 120, 64, 6), (300, 257, 136, 150),
                                      (9, 64, 30, 10)])
def test_bias_and_second_matrix(dtype, M, N, K, N2):
    from ipex_llm_b200.ops import stream as S
    w, w2 = rnd(N, K, seed=1, dtype=dtype, gain=K ** -0.5), rnd(N2, K, seed=2, dtype=dtype, gain=K ** -0.5)
    b, x, res = rnd(N, seed=3, dtype=dtype), rnd(M, K, seed=4, dtype=dtype), rnd(M, N, seed=5)
    W, W2, B, X = (t.to("cuda", dtype) for t in (w, w2, b, x))
    want = x @ w.T + b
    out, f, R = (torch.empty(M, N, dtype=d, device="cuda") for d in (dtype, F32, F32))
    R.copy_(res)
    if M <= S.rows_max(K, dtype):
        o2 = torch.empty(M, N2, dtype=F32, device="cuda")
        close(S.gemv_rows(W, X, out, S.OUT_ACT, bias=B, w2=W2, out2=o2), want, dtype)
        close(o2, x @ w2.T, F32, "second matrix", 5)              # never rounded to 16 bits
        close(S.gemv_rows(W, X, f, S.OUT_F32, bias=B), want, F32, "fp32", 5)
        close(S.gemv_rows(W, X, R, S.OUT_ADD, bias=B), res + want, F32, "stream", 5)
        R.copy_(res)
    g2 = torch.full((M, N2 + 3), 7.0, dtype=F32, device="cuda")
    close(S.gemm(X, W, torch.empty_like(out), S.OUT_ACT, bias=B, w2=W2, out2=g2[:, :N2]), want, dtype, "gemm")
    close(g2[:, :N2], x @ w2.T, F32, "gemm, second matrix", 5)
    assert bool((g2[:, N2:] == 7.0).all())
    close(S.gemm(X, W, torch.empty_like(out), S.OUT_ACT, bias=B), want, dtype, "gemm")
    close(S.gemm(X, W, torch.empty_like(f), S.OUT_F32, bias=B), want, F32, "gemm fp32", 5)
    close(S.gemm(X, W, R, S.OUT_ADD, bias=B), res + want, F32, "gemm stream", 5)
    close(S.bias_rows_(torch.zeros_like(f), B), b.expand(M, N), F32)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("M,K", [(1, 48), (5, 75), (3, 2052), (2, 5000), (1, 17000), (200, 256)])
def test_norms_around_the_addition(dtype, M, K):
    from ipex_llm_b200.ops import stream as S
    x, y = rnd(M, K, seed=1, gain=3.0), rnd(M, K, seed=2, gain=0.1)
    a, b = rnd(K, seed=3, gain=0.3), rnd(K, seed=4, gain=0.3)
    X, Y, A, B = (t.to("cuda", F32) for t in (x, y, 1 + a, 1 + b))
    h = S.add_norm_stream(X, Y, A, B, 1e-3, dtype)
    want = x + O.rms_norm(y, a, 1e-3)
    close(X, want, F32, "stream")
    close(h, O.rms_norm(want, b, 1e-3), dtype, "next input")
    assert h.dtype == dtype and S.add_norm_stream(X, Y, A, None, 1e-3, dtype) is None
    close(X, want + O.rms_norm(y, a, 1e-3), F32, "twice")
    rows = i32([M - 1, 0])
    close(S.norm_stream(X, B, 1e-3, rows=rows, dtype=dtype), O.rms_norm(X.double().cpu()[[M - 1, 0]], b, 1e-3), dtype)


# ------------------------------------------------------------------------------------------------
# windowed attention alone
# ------------------------------------------------------------------------------------------------
class Attention:
    """One attention layer behind its projection, on the kernels and on the oracle, with keys that stand out."""

    def __init__(self, dtype, heads, kv_heads, dim, vdim, window, n, standout=(), scale=None, share=0.375, seed=0):
        from ipex_llm_b200.ops import window_attn as A
        from ipex_llm_b200.ops.kv_cache import KeyValueShape, SlotCache
        self.A, self.dtype, self.n, self.share = A, dtype, n, share
        scale = dim ** -0.5 if scale is None else scale
        self.spec = A.AttnSpec(heads, kv_heads, dim, vdim, scale, window or 0, True)
        q, k = rnd(n, heads, dim, seed=seed + 1), rnd(n, kv_heads, dim, seed=seed + 2)
        if len(standout):
            # the queries of a group share a direction, and the stand-out keys point along it
            d = rnd(kv_heads, dim, seed=seed + 3)
            q = 0.4 * q + 1.8 * d.repeat_interleave(heads // kv_heads, 0)
            for i, p in enumerate(standout):
                k[p] = d * (2.0 + i)
        self.q, self.k, self.v, self.vf = (t.to(dtype).double() for t in (
            q, k, rnd(n, kv_heads, vdim, seed=seed + 4), rnd(n, kv_heads, vdim, seed=seed + 5)))
        self.cache = SlotCache()
        self.cache.allocate(4, n + 64, [KeyValueShape(kv_heads, dim, vdim)], dtype, "cuda")

    def want(self, faults=(), a=0, b=None):
        """Outputs of rows a .. b taken as a sequence of its own."""
        q, k, v, vf = (t[a:b] for t in (self.q, self.k, self.v, self.vf))
        if self.share is not None:
            v = O.mix_values(v, vf, self.share)
            if self.dtype != F32:
                v = v.float().to(self.dtype).double()             # mixed values are kept in the cache's format
        return O.attend(q, k, v, self.spec.scale, self.spec.window, faults).flatten(1)

    def operands(self, idx):
        s, N = self.spec, self.spec.rows
        t = torch.zeros(len(idx), (N + 7) // 8 * 8, dtype=self.dtype, device="cuda")
        t[:, :N] = torch.cat([x[idx].flatten(1) for x in (self.q, self.k, self.v)], 1).to(self.dtype)
        vf = torch.zeros(len(idx), s.kv_heads * s.vdim + 8, dtype=self.dtype, device="cuda")
        vf[:, 8:] = self.vf[idx].flatten(1).to(self.dtype)
        return t[:, :N], None if self.share is None else self.A.ValueMix(vf[:, 8:], self.share)

    def step(self, cuts, slot=2, first=0, visible=None, nsplit=None):
        """Portions [cuts[i], cuts[i + 1]); portions of one token append on the way."""
        self.cache.set_first_rows([first if s == slot else 0 for s in range(4)])
        outs = []
        for a, b in zip(cuts, cuts[1:]):
            qkv, mix = self.operands(list(range(a, b)))
            out = torch.empty(b - a, self.spec.heads * self.spec.vdim, dtype=self.dtype, device="cuda")
            self.A.attend_step(self.spec, qkv, mix, i32([slot] * (b - a)), i32(list(range(first + a, first + b))), self.cache,
                               0, out, visible or (self.spec.window or b), b - a == 1, nsplit=nsplit)
            outs.append(out)
        return torch.cat(outs)

    def prompt(self, lens, slots):
        """Sequences cut out of the rows 0.., packed; every one restarts at position 0."""
        T = sum(lens)
        self.cache.set_first_rows([0] * 4)
        row, sl, pos, at = [], [], [], 0
        for n, s in zip(lens, slots):
            row.append(at)
            sl += [s] * n
            pos += list(range(n))
            at += n
        qkv, mix = self.operands(list(range(T)))
        out = torch.empty(T, self.spec.heads * self.spec.vdim, dtype=self.dtype, device="cuda")
        return self.A.attend_prompt(self.spec, qkv, mix, i32(sl), i32(pos), i32(row), i32(lens), max(lens), self.cache, 0, out)


ATTN_SIZES = [  # heads, kv_heads, dim, vdim
    (4, 2, 32, 24), (6, 6, 48, 40), (16, 1, 16, 8), (3, 3, 10, 7), (20, 2, 128, 128), (5, 1, 64, 96), (24, 8, 256, 16),
    (2, 1, 8, 200)]


@pytest.mark.parametrize("dtype", [F32, BF16, F16])
@pytest.mark.parametrize("size", ATTN_SIZES)
@pytest.mark.parametrize("window", [None, 1, 37])
def test_attention_step_kernel(dtype, size, window):
    n = 75
    at = Attention(dtype, *size, window, n)
    want = at.want()
    close(at.step([0, 1, 2, 40, 42, 75]), want, dtype, "portions")
    close(at.step([0, 30] + list(range(31, 76)), nsplit=4), want, dtype, "one by one")
    close(at.step([0, 64, 65, 75], slot=1, first=9, nsplit=8), want, dtype, "first row 9")


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_sink_value_mixing_and_head_groups_show(dtype):
    at = Attention(dtype, 6, 3, 24, 16, 9, 40, scale=0.05)
    want = at.want()
    for fault in ("no_sink", "heads_interleaved"):
        assert (at.want((fault,)) - want).abs().max() > 8 * TOL[dtype] * want.abs().max()
    plain = Attention(dtype, 6, 3, 24, 16, 9, 40, scale=0.05, share=None)
    assert (plain.want() - want).abs().max() > 8 * TOL[dtype] * want.abs().max()
    close(plain.step([0, 20] + list(range(21, 41))), plain.want(), dtype, "values of the layer alone")
    for low in (Attention(dtype, 2, 1, 8, 8, 20, 60, scale=-3.0), Attention(dtype, 2, 1, 8, 8, 20, 60, scale=4.0)):
        close(low.step([0, 30] + list(range(31, 61))), low.want(), dtype, "scores far from the sink's")
        if dtype != F32:
            close(low.prompt([60], [0]), low.want(), dtype, "prompt, scores far from the sink's")


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("window", [16, 100, 128, 129, 300])
def test_window_edges_with_a_key_that_stands_out(dtype, window):
    """The stand-out key at p decides every query that sees it, and none past p + window - 1; decoding one by one, in
    portions and (16-bit) as a prompt."""
    p, n = 13, 13 + window + 6
    at = Attention(dtype, 6, 2, 48, 32, window, n, standout=(p,))
    want = at.want()
    i, o = p + window - 1, p + window
    for fault, row in (("window_plus_one", o), ("window_minus_one", i)):
        assert (at.want((fault,))[row] - want[row]).abs().max() > 8 * TOL[dtype] * want.abs().max()
    runs = {"portions": at.step([0, 30, n]), "one by one": at.step([0, 10] + list(range(11, n + 1))),
            "one by one, split": at.step([0, 10] + list(range(11, n + 1)), nsplit=8)}
    if dtype == BF16:
        runs["prompt"] = at.prompt([n], [0])
    for name, got in runs.items():
        close(got[[i, o]], want[[i, o]], dtype, f"{name} edge")
        close(got, want, dtype, name)


@pytest.mark.parametrize("dtype", [BF16, F16])
@pytest.mark.parametrize("size", [(4, 2, 32, 24), (2, 2, 64, 64), (6, 1, 128, 96), (4, 4, 192, 128), (3, 3, 72, 104),
                                  (8, 4, 256, 8)])
@pytest.mark.parametrize("window", [None, 50, 128, 200])
def test_prompt_kernel_on_packed_sequences(dtype, size, window):
    """Sequences of different lengths behind one another (tiles that start inside a sequence's 8-token boundary, lengths
    around the 128-query tile, one single token), keys far away that stand out; what the prompt filed serves the steps
    that follow."""
    lens = [130, 1, 257, 64, 5]
    at = Attention(dtype, *size, window, sum(lens) + 1, standout=(2, 140, 141, 260))
    assert at.spec.prefill_ok(dtype)
    got, row = at.prompt(lens, [0, 1, 2, 3, 0]), 0
    for n in lens:
        close(got[row:row + n], at.want(a=row, b=row + n), dtype, f"rows {row}..{row + n}")
        row += n
    n = lens[2]                                       # slot 2 goes on by one token behind its prompt
    idx = list(range(131, 131 + n)) + [sum(lens)]
    qkv, mix = at.operands(idx[-1:])
    out = torch.empty(1, at.spec.heads * at.spec.vdim, dtype=dtype, device="cuda")
    at.A.attend_step(at.spec, qkv, mix, i32([2]), i32([n]), at.cache, 0, out, n + 1, True)
    at.q, at.k, at.v, at.vf = (t[idx] for t in (at.q, at.k, at.v, at.vf))
    close(out[0], at.want()[-1], dtype, "next token")


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_far_key_among_many_and_split_counts(dtype):
    """Without a window one early key must be found among a thousand, however the visible keys are split."""
    n = 1100
    at = Attention(dtype, 4, 2, 32, 24, None, n, standout=(3,))
    want = at.want()
    at.step([0, 1000])
    for nsplit in (1, 2, 4, 8):
        close(at.step([1000, 1001, 1003, 1100], nsplit=nsplit), want[1000:], dtype, f"nsplit={nsplit}")


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_unequal_sequences_in_one_step(dtype):
    """One new token each for sequences of different lengths in different slots, one of them at its very first token."""
    at = Attention(dtype, 8, 2, 40, 16, 33, 90)
    spans = {3: (0, 50), 0: (50, 80), 1: (80, 81)}     # slot -> rows that make up its sequence
    for s, (a, b) in spans.items():
        if b - a > 1:
            qkv, mix = at.operands(list(range(a, b - 1)))
            at.A.attend_step(at.spec, qkv, mix, i32([s] * (b - a - 1)), i32(list(range(b - a - 1))), at.cache, 0,
                             torch.empty(b - a - 1, 8 * 16, dtype=dtype, device="cuda"), 60, False)
    qkv, mix = at.operands([b - 1 for _, b in spans.values()])
    out = torch.empty(3, 8 * 16, dtype=dtype, device="cuda")
    at.A.attend_step(at.spec, qkv, mix, i32(list(spans)), i32([b - a - 1 for a, b in spans.values()]), at.cache, 0, out, 60, True)
    for i, (a, b) in enumerate(spans.values()):
        close(out[i], at.want(a=a, b=b)[-1], dtype, f"sequence {i}")


# ------------------------------------------------------------------------------------------------
# gated delta rule alone
# ------------------------------------------------------------------------------------------------
class Delta:
    """One delta layer behind its projections, on the kernels and on the oracle."""

    def __init__(self, dtype, heads, kv_heads, dim, vdim, taps, n, decay=0.0, seed=0):
        from ipex_llm_b200.engine.stream_engine import Portions
        from ipex_llm_b200.ops import delta as R
        from ipex_llm_b200.ops.kv_cache import DeltaStateShape, SlotCache
        self.R, self.Portions, self.dtype, self.n = R, Portions, dtype, n
        self.spec = s = R.DeltaSpec(heads, kv_heads, dim, vdim, taps)
        self.x = rnd(n, s.rows, seed=seed + 1, dtype=dtype)
        self.gates = rnd(n, 2 * heads, seed=seed + 2, gain=1.5)
        self.conv = rnd(s.channels, taps, seed=seed + 3, dtype=dtype, gain=1.5 * taps ** -0.5)
        self.a_log, self.dt_bias = rnd(heads, seed=seed + 4, gain=0.7) + decay, rnd(heads, seed=seed + 5)
        self.norm = (1 + 0.2 * rnd(vdim, seed=seed + 6)).to(dtype).double()
        self.weights = R.DeltaWeights(self.conv.to("cuda", dtype), self.a_log.cuda(), self.dt_bias.cuda(),
                                      self.norm.to("cuda", dtype), 1e-5)
        self.cache = SlotCache()
        self.cache.allocate(4, n + 64, [DeltaStateShape(heads, dim, vdim, taps, s.channels)], dtype, "cuda")

    def want(self, a=0, b=None, faults=()):
        s, n = self.spec, len(self.x[a:b])
        qk = s.kv_heads * s.dim
        y = O.silu(O.short_conv(self.x[a:b, :s.channels], self.conv))
        head = torch.arange(s.heads) // (s.heads // s.kv_heads)
        q = O.unit(y[:, :qk].view(n, s.kv_heads, s.dim))[:, head] * s.dim ** -0.5
        k = O.unit(y[:, qk:2 * qk].view(n, s.kv_heads, s.dim))[:, head]
        v = y[:, 2 * qk:].view(n, s.heads, s.vdim)
        g = self.gates[a:b]
        beta, dec = O.delta_gates(g[:, :s.heads], g[:, s.heads:], self.a_log, self.dt_bias)
        o, state = O.delta_rule(q, k, v, beta, dec, faults=faults)
        return O.gated_head_norm(o, self.x[a:b, s.channels:].view(n, s.heads, s.vdim), self.norm, 1e-5).flatten(1), state

    def portions(self, lens):
        row, c, owner, first = 0, 0, [], [0]
        rows = []
        for i, n in enumerate(lens):
            rows.append(row)
            k = -(-n // 32)
            owner += [i] * k
            row, c = row + n, c + k
            first.append(c)
        return self.Portions(i32(rows), i32(lens), max(lens), False, i32(owner), i32(first), c)

    def run(self, idx, slots, pos, lens=None, chunked=None):
        """One call over the rows ``idx``; ``lens``: portions they make up, None: one token each."""
        s = self.spec
        pad = (s.rows + 7) // 8 * 8
        proj = torch.zeros(len(idx), pad, dtype=self.dtype, device="cuda")
        proj[:, :s.rows] = self.x[idx].to(self.dtype)
        out = torch.empty(len(idx), s.heads * s.vdim, dtype=self.dtype, device="cuda")
        return self.R.delta_mix(s, self.weights, proj[:, :s.rows], self.gates[idx].to("cuda", F32), i32(slots), i32(pos),
                                self.cache, 0, out, None if lens is None else self.portions(lens), chunked=chunked)

    def step(self, cuts, slot=2, first=0, chunked=None):
        self.cache.set_first_rows([first if s == slot else 0 for s in range(4)])
        return torch.cat([self.run(list(range(a, b)), [slot] * (b - a), list(range(first + a, first + b)),
                                   None if b - a == 1 else [b - a], chunked) for a, b in zip(cuts, cuts[1:])])

    def state(self, slot):
        return self.cache.layers[0]._k[slot]


DELTA_SIZES = [  # heads, kv_heads, dim, vdim, taps
    (4, 2, 16, 24, 4), (3, 3, 32, 32, 4), (2, 1, 128, 128, 4), (6, 1, 24, 40, 3), (2, 2, 10, 7, 2), (1, 1, 200, 96, 1),
    (2, 2, 256, 64, 5), (2, 1, 48, 300, 4), (4, 4, 8, 16, 9)]


@pytest.mark.parametrize("dtype", [F32, BF16, F16])
@pytest.mark.parametrize("size", DELTA_SIZES)
def test_delta_token_by_token_and_in_portions(dtype, size):
    n = 70
    d = Delta(dtype, *size, n)
    want, state = d.want()
    for name, cuts, kw in (("one by one", list(range(n + 1)), {}), ("portions", [0, 1, 3, 5, 40, 41, 70], {"chunked": False}),
                           ("portions from row 9", [0, 2, 33, 70], {"chunked": False, "first": 9, "slot": 1})):
        close(d.step(cuts, **kw), want, dtype, name)
        close(d.state(kw.get("slot", 2)), state, F32, name + ", state", 5)


@pytest.mark.parametrize("dtype", [BF16, F16])
@pytest.mark.parametrize("size", DELTA_SIZES)
@pytest.mark.parametrize("decay", [-4.0, 0.0, 2.5])
def test_delta_in_chunks(dtype, size, decay):
    """Chunk borders everywhere, portions that go on from a state, decays from hundreds of tokens down to less than one;
    the state agrees to 32-bit accuracy."""
    n = 150
    d = Delta(dtype, *size, n, decay=decay)
    assert d.spec.chunks_ok(dtype)
    want, state = d.want()
    for cuts in ([0, n], [0, 33, 65, 129, 150], [0, 1, 2, 34, 66, 149, 150], [0, 96, 150]):
        close(d.step(cuts, chunked=True), want, dtype, f"cuts {cuts}")
        close(d.state(2), state, F32, f"state, cuts {cuts}", 5)
    close(d.step([0, 40, 150], slot=0, first=7, chunked=True), want, dtype, "first row 7")


def test_delta_chunks_in_several_passes():
    """A prompt longer than the scratch runs in passes; sequences then start and end in the middle of a pass."""
    d = Delta(BF16, 4, 2, 16, 24, 4, 300)
    lens, at = [70, 1, 130, 99], 0
    old = d.R.SCRATCH_BYTES
    per = 4 * 4 * int(__import__("ipex_llm_b200.native.lib", fromlist=["x"]).stream_lib().ipex_delta_scratch_floats(16, 24))
    try:
        for chunks in (1, 2, 3):
            d.R.SCRATCH_BYTES = chunks * per
            got = d.run(list(range(300)), sum(([s] * n for s, n in zip((3, 0, 1, 2), lens)), []),
                        sum((list(range(n)) for n in lens), []), lens, True)
            at = 0
            for s, n in zip((3, 0, 1, 2), lens):
                want, state = d.want(at, at + n)
                close(got[at:at + n], want, BF16, f"{chunks} chunks a pass")
                close(d.state(s), state, F32, "state", 5)
                at += n
    finally:
        d.R.SCRATCH_BYTES = old


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_delta_unequal_sequences_and_used_slots(dtype):
    """Prompts of several lengths in one call, then one token each; then the slots go to other sequences without being
    cleared, among them one that starts with a single token."""
    d = Delta(dtype, 4, 2, 32, 40, 4, 240)
    for rounds, spans in enumerate(({1: (0, 40), 3: (40, 43), 0: (43, 141)}, {0: (150, 190), 1: (190, 240), 3: (141, 149)})):
        idx, slots, pos, lens = [], [], [], []
        for s, (a, b) in spans.items():
            idx += range(a, b - 2)
            slots += [s] * (b - a - 2)
            pos += range(b - a - 2)
            lens.append(b - a - 2)
        got = d.run(idx, slots, pos, lens)
        at = 0
        for (a, b), n in zip(spans.values(), lens):
            close(got[at:at + n], d.want(a, b)[0][:-2], dtype, f"prompts, round {rounds}")
            at += n
        for back in (2, 1):
            got = d.run([b - back for _, b in spans.values()], list(spans), [b - a - back for a, b in spans.values()])
            for i, (a, b) in enumerate(spans.values()):
                close(got[i], d.want(a, b)[0][-back], dtype, f"decoding, round {rounds}")
    got = [d.run([t], [3], [t]) for t in range(6)]
    close(torch.cat(got), d.want(0, 6)[0], dtype, "first token alone in a used slot")


def test_delta_far_write_is_found_again():
    """One write with a key of its own direction is read by a far query through a slowly decaying state; the read-out sees
    the current token's write."""
    n = 400
    d = Delta(F32, 2, 1, 16, 16, 2, n, decay=-9.0)
    d.conv[:] = torch.tensor([0.0, 1.0])              # the taps pass the current token through
    d.weights.conv.copy_(d.conv)
    d.x[:, 16:32] = 0.0
    d.x[:, 16:24] = rnd(n, 8, seed=8).abs()           # keys of the others live in the first half
    d.x[5, 16:32], d.x[5, 28] = 0.0, 6.0
    d.x[n - 1, :16], d.x[n - 1, 12] = 0.0, 6.0
    d.x[:, :4] += 1.0
    want, _ = d.want()
    assert (want[n - 1] - d.want(6)[0][-1]).abs().max() > 0.1
    assert (want - d.want(faults=("read_before_write",))[0]).abs().max() > 0.1
    close(d.step([0, 300] + list(range(301, n + 1)), chunked=False), want, F32, factor=5)
    half = Delta(BF16, 2, 1, 16, 16, 2, n, decay=-9.0)
    for name in ("x", "conv"):
        setattr(half, name, getattr(d, name).to(BF16).double())
    half.weights.conv.copy_(half.conv)
    close(half.step([0, n], chunked=True), half.want()[0], BF16)


# ------------------------------------------------------------------------------------------------
# whole models
# ------------------------------------------------------------------------------------------------
def cfg_a():
    return {"architecture": "Letarax", "vocab": 150, "width": 96, "norm": {"eps": 1e-5},
            "layers": [O.attention_layer(4, 2, 32, 24, window=20, ff=160),
                       O.delta_layer(4, 2, 16, 40, conv=4),
                       O.attention_layer(6, 2, 24, 24, window=33, ff=None, scale=0.3),
                       O.delta_layer(3, 1, 32, 16, conv=3, ff=64),
                       O.attention_layer(8, 2, 16, 24, window=7, ff=96)]}


def cfg_odd():
    """Nothing a multiple of anything: the generic kernels; layers that mix no values between layers that do."""
    return {"architecture": "Letarax", "vocab": 101, "width": 50, "norm": {"eps": 1e-3},
            "layers": [O.delta_layer(3, 3, 10, 7, conv=2, ff=33),
                       O.attention_layer(3, 1, 10, 9, window=4, v_mix=False, ff=11),
                       O.attention_layer(2, 1, 13, 5, window=1, ff=None),
                       O.attention_layer(3, 1, 6, 5, window=90, ff=21),
                       O.delta_layer(1, 1, 5, 3, conv=1)]}


def cfg_attention():
    """Attention only; a window of 64 at a tile edge."""
    return {"architecture": "Letarax", "vocab": 120, "width": 64, "norm": {"eps": 1e-6},
            "layers": [O.attention_layer(2, 2, 64, 64, window=64, ff=128), O.attention_layer(4, 2, 32, 64, window=64, ff=64)]}


def cfg_delta():
    """Recurrent layers only."""
    return {"architecture": "Letarax", "vocab": 120, "width": 64, "norm": {"eps": 1e-6},
            "layers": [O.delta_layer(2, 2, 32, 32, conv=4, ff=128), O.delta_layer(4, 2, 16, 32, conv=4)]}


def cfg_ff20():
    """A hidden size that is no multiple of eight in a model whose other sizes are."""
    return {"architecture": "Letarax", "vocab": 90, "width": 64, "norm": {"eps": 1e-6},
            "layers": [O.attention_layer(2, 1, 16, 32, window=30, ff=20), O.delta_layer(2, 1, 16, 32, conv=4, ff=20)]}


CFGS = {"a": cfg_a, "odd": cfg_odd, "attention": cfg_attention, "delta": cfg_delta, "ff 20": cfg_ff20}
_models, _want = {}, {}


def make(name, dtype):
    from ipex_llm_b200.models import letarax
    from ipex_llm_b200.transformers.model import _attach_api
    key = (name, dtype)
    if key not in _models:
        cfg = CFGS[name]()
        w = O.random_weights(cfg, seed=len(name))
        model = _attach_api(letarax.build(cfg, w, dtype).to("cuda"))
        _models[key] = (model, cfg, {k: v.double() for k, v in w.items()})
    return _models[key]


def tokens(n, V, seed):
    return torch.randint(0, V, (n,), generator=gen(seed)).tolist()


def oracle(name, toks):
    key = (name, tuple(toks))
    if key not in _want:
        _, cfg, w = make(name, F32)
        _want[key] = O.forward(w, cfg, toks)
    return _want[key]


def engine(model, batch=4, length=400):
    from ipex_llm_b200.engine import get_engine
    eng = get_engine(model, batch, length)
    eng.new_cache(batch)
    return eng


# logits through several layers: rounding adds up, and a sharp soft-max amplifies it
MODEL_TOL = {F32: 3.0, BF16: 4.0}


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", list(CFGS))
def test_prompt_portions_and_decoding_agree(name, dtype):
    model, cfg, _ = make(name, dtype)
    toks = tokens(150, cfg["vocab"], 5)
    want, n = oracle(name, toks), len(toks)
    for cuts in ([0, n], [0, 75, n], list(range(0, n, 13)) + [n], list(range(0, n, 2)) + [n], [0, 1, 9, 20, 148, n]):
        eng = engine(model)
        s = eng.cache.acquire()
        got = [eng.step_rows([(s, toks[a:b], list(range(b - a)))]).clone() for a, b in zip(cuts, cuts[1:])]
        close(torch.cat(got), want, dtype, f"cuts {cuts[:4]}", MODEL_TOL[dtype])
    for graph in (True, False):
        eng = engine(model)
        s = eng.cache.acquire()
        got = [eng.step_rows([(s, toks[:3], [0, 1, 2])])]
        got += [eng.step_rows([(s, [t], [0])], use_graph=graph).clone() for t in toks[3:]]
        close(torch.cat(got), want, dtype, f"token by token, graph={graph}", MODEL_TOL[dtype])


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", ["a", "odd"])
def test_residual_after_every_layer(name, dtype):
    model, cfg, w = make(name, dtype)
    toks = tokens(41, cfg["vocab"], 7)
    trace, got = [], []
    O.forward(w, cfg, toks, trace=trace)
    eng = engine(model)
    eng.stack.run_portions([(eng.cache.acquire(), 0, toks)], eng.cache, collect=got)
    for i, (g, t) in enumerate(zip(got, trace)):
        close(g, t, dtype, f"layer {i}", 2)
        assert g.dtype == F32


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_ragged_batches_against_each_alone(dtype):
    """Unequal prompts in one batch, decoded together while the shorter ones leave; slots handed to new sequences."""
    model, cfg, _ = make("a", dtype)
    V, tol = cfg["vocab"], MODEL_TOL[dtype]
    seqs = [tokens(n, V, 20 + n) for n in (1, 9, 130, 70)]
    tails = [3, 12, 5, 9]
    want = [oracle("a", s) for s in seqs]
    eng = engine(model)
    slots = [eng.cache.acquire() for _ in seqs]
    split = [max(1, len(s) - t) for s, t in zip(seqs, tails)]
    got = [[] for _ in seqs]
    lg = eng.step_rows([(sl, s[:k], list(range(k))) for sl, s, k in zip(slots, seqs, split)])
    at = 0
    for i, k in enumerate(split):
        got[i].append(lg[at:at + k])
        at += k
    pos = list(split)
    while any(p < len(s) for p, s in zip(pos, seqs)):
        live = [i for i in range(4) if pos[i] < len(seqs[i])]
        lg = eng.step_rows([(slots[i], [seqs[i][pos[i]]], [0]) for i in live])
        for j, i in enumerate(live):
            got[i].append(lg[j:j + 1].clone())
            pos[i] += 1
            if pos[i] == len(seqs[i]):
                eng.cache.release(slots[i])
    eng.cache.release(slots[0])                      # one token: it was finished after the first step
    for i in range(4):
        close(torch.cat(got[i]), want[i], dtype, f"sequence {i}", tol)
    # all slots are free again: other sequences, other lengths, in another order
    again = [seqs[2], seqs[1], seqs[3], seqs[2][:40]]
    slots = [eng.cache.acquire() for _ in again]
    lg = eng.step_rows([(sl, s, list(range(len(s)))) for sl, s in zip(slots, again)])
    close(lg, torch.cat([want[2], want[1], want[3], want[2][:40]]), dtype, "reused slots", tol)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_mixed_portions_in_one_batch(dtype):
    """A prompt, a continued portion and a decoded token in the same step."""
    model, cfg, _ = make("a", dtype)
    a, b, c = (tokens(n, cfg["vocab"], 50 + n) for n in (40, 90, 33))
    wa, wb, wc = (oracle("a", t) for t in (a, b, c))
    eng = engine(model)
    sa, sb, sc = (eng.cache.acquire() for _ in range(3))
    eng.step_rows([(sa, a[:39], []), (sb, b[:30], [])])
    lg = eng.step_rows([(sb, b[30:], list(range(60))), (sa, a[39:], [0]), (sc, c, list(range(33)))])
    close(lg, torch.cat([wb[30:], wa[39:], wc]), dtype, factor=MODEL_TOL[dtype])


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name,count", [("a", 19), ("a", 12), ("odd", 11), ("ff 20", 12)])
def test_many_sequences_decode_together(name, count, dtype):
    """More rows than the small row products take, then more than any of them does: GEMMs in the decode graph."""
    model, cfg, _ = make(name, dtype)
    seqs = [tokens(20 + 3 * i, cfg["vocab"], 80 + i) for i in range(count)]
    want = [oracle(name, s) for s in seqs]
    eng = engine(model, count)
    slots = [eng.cache.acquire() for _ in seqs]
    eng.step_rows([(sl, s[:-4], []) for sl, s in zip(slots, seqs)])
    for k in range(4, 0, -1):
        lg = eng.step_rows([(sl, [s[-k]], [0]) for sl, s in zip(slots, seqs)])
        close(lg, torch.stack([w[-k] for w in want]), dtype, f"{k} from the end", MODEL_TOL[dtype])


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_long_decoding(dtype):
    """Several windows and graphs past the prompt, one token at a time."""
    model, cfg, _ = make("a", dtype)
    toks = tokens(330, cfg["vocab"], 3)
    want = oracle("a", toks)
    eng = engine(model)
    s = eng.cache.acquire()
    got = [eng.step_rows([(s, toks[:11], [10])])]
    got += [eng.step_rows([(s, [t], [0])]).clone() for t in toks[11:]]
    close(torch.cat(got), want[10:], dtype, factor=MODEL_TOL[dtype])


# ------------------------------------------------------------------------------------------------
# the framework's entry points
# ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", ["a", "odd", "delta"])
def test_greedy_generate(name):
    model, cfg, w = make(name, F32)
    prompts = [tokens(n, cfg["vocab"], n) for n in (23, 6, 14)]
    want = [O.greedy(w, cfg, p, 12) for p in prompts]
    for p, e in zip(prompts, want):
        out = model.generate(torch.tensor([p], device="cuda"), max_new_tokens=12, do_sample=False)
        assert out[0, len(p):].tolist() == e
        assert type(model._ipex_engine).__name__ == "HybridEngine"
    # left-padded batch: stays on the engine, rows keep their own positions
    S = max(map(len, prompts))
    ids = torch.tensor([[0] * (S - len(p)) + p for p in prompts], device="cuda")
    mask = torch.tensor([[0] * (S - len(p)) + [1] * len(p) for p in prompts], device="cuda")
    out = model.generate(ids, attention_mask=mask, max_new_tokens=12, do_sample=False)
    assert out[:, S:].tolist() == want
    # ... and the transformers loop over the module's forward gives the same
    out = model._hf_generate(ids, attention_mask=mask, max_new_tokens=12, do_sample=False, pad_token_id=0)
    assert out[:, S:].tolist() == want


def test_sampling_stays_on_the_engine():
    model, cfg, _ = make("a", F32)
    ids = torch.tensor([tokens(12, cfg["vocab"], 2)] * 3, device="cuda")
    torch.manual_seed(0)
    out = model.generate(ids, max_new_tokens=9, do_sample=True, temperature=60.0, top_k=40, top_p=0.95)
    assert out.shape == (3, 21) and len({tuple(r) for r in out[:, 12:].tolist()}) > 1
    one = model.generate(ids, max_new_tokens=9, do_sample=True, top_k=1)
    assert torch.equal(one, model.generate(ids, max_new_tokens=9, do_sample=False))


def test_forward_logits_and_beam_search():
    model, cfg, w = make("a", F32)
    p = tokens(19, cfg["vocab"], 4)
    ids = torch.tensor([p, p[::-1]], device="cuda")
    out = model(ids)
    for b in range(2):
        close(out.logits[b], O.forward(w, cfg, ids[b].tolist()), F32, factor=MODEL_TOL[F32])
    more = model(torch.tensor([[5], [6]], device="cuda"), past_key_values=out.past_key_values)
    close(more.logits[1, -1], O.forward(w, cfg, p[::-1] + [6])[-1], F32, factor=MODEL_TOL[F32])
    assert model(ids, logits_to_keep=2).logits.shape == (2, 2, cfg["vocab"])
    beams = model.generate(ids[:1], max_new_tokens=5, num_beams=3, do_sample=False, pad_token_id=0)
    full = torch.log_softmax(O.forward(w, cfg, beams[0].tolist()), -1)
    lp = sum(full[18 + i, beams[0, 19 + i]].item() for i in range(5))
    g = O.greedy(w, cfg, p, 5)
    fg = torch.log_softmax(O.forward(w, cfg, p + g), -1)
    assert lp >= sum(fg[18 + i, t].item() for i, t in enumerate(g)) - 1e-6      # never worse than greedy


def test_prefill_and_decode_step_api():
    model, cfg, w = make("a", F32)
    p = tokens(17, cfg["vocab"], 8)
    want = O.greedy(w, cfg, p, 5)
    t = model.prefill(torch.tensor([p]), max_new_tokens=8)
    got = [int(t[0])]
    for _ in range(4):
        t = model.decode_step(t.clone().pin_memory())
        got.append(int(t[0]))
    assert got == want


def write_checkpoint(path, cfg, w):
    from safetensors.torch import save_file
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.bfloat16().contiguous() for k, v in w.items()}, os.path.join(path, "model.safetensors"))


def test_low_bit_projections_run(tmp_path):
    """Packed projections with biases and gated units: logits close to those of the dense weights."""
    from ipex_llm_b200.models import letarax
    from ipex_llm_b200.transformers import AutoModelForCausalLM
    cfg = {"architecture": "Letarax", "vocab": 128, "width": 128, "norm": {"eps": 1e-6},
           "layers": [O.attention_layer(4, 2, 32, 32, window=30, ff=256), O.delta_layer(4, 2, 32, 32, ff=128)]}
    w = O.random_weights(cfg, sharp=1.0)
    write_checkpoint(str(tmp_path), cfg, w)
    m8 = AutoModelForCausalLM.from_pretrained(str(tmp_path), load_in_low_bit="sym_int8").to("cuda")
    ref = letarax.build(cfg, w, BF16).to("cuda")
    toks = torch.tensor([tokens(40, cfg["vocab"], 2)], device="cuda")
    a, b = m8(toks).logits, ref(toks).logits
    assert torch.nn.functional.cosine_similarity(a[0], b[0], dim=-1).median() > 0.99
    out = m8.generate(toks, max_new_tokens=4, do_sample=False)
    assert out.shape == (1, 44)


def test_served_batch_runs_on_the_engine():
    """``ModelWorker``: unequal prompts, stop after different lengths, same tokens as alone."""
    from tokenizers import Tokenizer, models, pre_tokenizers
    from transformers import PreTrainedTokenizerFast
    from ipex_llm_b200.serving import ModelWorker, SamplingParams
    from ipex_llm_b200.serving.model_worker import ServingRequest
    model, cfg, w = make("a", F32)
    words = ["<pad>", "<s>", "</s>", "<unk>"] + [f"w{i}" for i in range(cfg["vocab"] - 4)]
    tk = Tokenizer(models.WordLevel({x: i for i, x in enumerate(words)}, unk_token="<unk>"))
    tk.pre_tokenizer = pre_tokenizers.Whitespace()
    tok = PreTrainedTokenizerFast(tokenizer_object=tk, pad_token="<pad>", bos_token="<s>", unk_token="<unk>",
                                  padding_side="left")
    worker = ModelWorker(model=model, tokenizer=tok, max_num_seqs=4)
    ids = [[10, 20, 30, 40, 50, 60], [7, 8], [99, 5, 140]]
    news = [6, 9, 3]
    reqs = [ServingRequest(prompt=" ".join(words[i] for i in p), params=SamplingParams(max_new_tokens=n))
            for p, n in zip(ids, news)]
    calls = []
    eng_cls = type(engine(model))
    orig = eng_cls.decode_step
    try:
        eng_cls.decode_step = lambda self, B, use_graph=True: (calls.append(B), orig(self, B, use_graph))[1]
        worker._run_batch(reqs)
    finally:
        eng_cls.decode_step = orig
    assert calls and set(calls) == {3}
    for r, p, n in zip(reqs, ids, news):
        want = [words[t] for t in O.greedy(w, cfg, p, n)]
        want = [x for x in want if x not in ("<pad>", "<s>", "<unk>")]
        assert r.generated_tokens == n and r.text.split() == want


def test_command_line_on_token_ids(tmp_path, capsys):
    from ipex_llm_b200.cli import llm_cli
    from ipex_llm_b200.transformers import AutoModelForCausalLM
    cfg = cfg_a()
    write_checkpoint(str(tmp_path), cfg, O.random_weights(cfg, seed=4))
    assert llm_cli.main(["-m", str(tmp_path), "-t", "bf16", "--token-ids", "3 9 4, 77", "-n", "6"]) == 0
    got = [int(t) for t in capsys.readouterr().out.split()]
    model = AutoModelForCausalLM.from_pretrained(str(tmp_path), load_in_low_bit="bf16", torch_dtype=BF16).to("cuda")
    out = model.generate(torch.tensor([[3, 9, 4, 77]], device="cuda"), max_new_tokens=6, do_sample=False)
    assert got == out[0, 4:].tolist() and len(got) == 6


def test_trace_replay(tmp_path):
    """The replay program on a checkpoint: a batch that starts together and thins out, then another request."""
    import subprocess
    import sys
    import numpy as np
    cfg = cfg_a()
    w = O.random_weights(cfg, seed=4)
    d, out = str(tmp_path / "m"), str(tmp_path / "o")
    write_checkpoint(d, cfg, w)
    V = cfg["vocab"]
    x, y, z = tokens(12, V, 1), tokens(70, V, 2), tokens(9, V, 3)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": x[:10], "want": [9]}, {"id": "y", "tokens": y[:68], "want": []}]},
             {"step": 1, "entries": [{"id": "x", "tokens": x[10:11], "want": []}, {"id": "y", "tokens": y[68:69], "want": []}],
              "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": x[11:], "want": [0]}, {"id": "y", "tokens": y[69:], "want": [0]}],
              "end": ["x", "y"]},
             {"step": 3, "entries": [{"id": "z", "tokens": z, "want": [0, 8]}], "end": ["z"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", d, "--dtype", "float32", "--out",
                        out, "--max-tokens", "90"], input="".join(json.dumps(s) + "\n" for s in steps), text=True,
                       capture_output=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == [f"done {i}" for i in range(4)]
    w64 = {k: v.double() for k, v in w.items()}
    fx, fy, fz = (O.forward(w64, cfg, t) for t in (x, y, z))
    for step, want in ((0, fx[9:10]), (2, torch.stack([fx[11], fy[69]])), (3, fz[[0, 8]])):
        got = torch.from_numpy(np.fromfile(os.path.join(out, f"{step}.f32"), dtype="<f4").reshape(-1, V))
        close(got, want, F32, f"step {step}", MODEL_TOL[F32])
    assert not os.path.exists(os.path.join(out, "1.f32"))
