"""Dodilix on the GPU: every kernel against the float64 oracle (``tests/dodilix_oracle.py``), then the engine with whole
prompts, portions, ragged batches, slot reuse, long decoding and generation."""
import json
import os

import pytest
import torch

import dodilix_oracle as O

pytestmark = pytest.mark.gpu

F32, BF16, F16 = torch.float32, torch.bfloat16, torch.float16
TOL = {F32: 2e-5, F16: 4e-3, BF16: 2.5e-2}          # relative to the size of the compared values
EPS = 1e-5


@pytest.fixture(autouse=True)
def _no_expired_wait():
    yield
    from ipex_llm_b200.ops.cuda_ops import check_error_flag
    check_error_flag(torch.device("cuda", 0))


def close(got, want, dtype, what="", factor=1.0):
    got, want = got.double().cpu(), want.double().cpu()
    assert got.shape == want.shape, (what, got.shape, want.shape)
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


def padded(x, dtype, extra=0):
    """``x`` in rows that start on 16-byte boundaries."""
    n = x.shape[1]
    t = torch.zeros(x.shape[0], (n + 7) // 8 * 8 + extra, dtype=dtype, device="cuda")
    t[:, :n] = x.to(dtype)
    return t[:, :n]


# ------------------------------------------------------------------------------------------------
# streams
# ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF16, F16])
@pytest.mark.parametrize("n,S,K", [(1, 1, 64), (3, 2, 208), (2, 3, 1028), (5, 4, 4096), (2, 4, 8192), (2, 2, 2060), (7, 5, 96),
                                   (2, 2, 75), (1, 16, 40), (200, 2, 256), (2, 3, 9000)])
def test_joint_between_sublayers(dtype, n, S, K):
    from ipex_llm_b200.ops import stream as St
    x, y = rnd(n, S, K, seed=1, gain=3.0), rnd(n, K, seed=2)
    mix, out, w_in, norm = rnd(S, S, seed=3, gain=0.6), rnd(S, seed=4), rnd(S, seed=5), 1 + rnd(K, seed=6, gain=0.2)
    X, Y, M, B, A, N = (t.to("cuda", F32).contiguous() for t in (x, y, mix, out, w_in, norm))
    h = St.hyper_joint(X, None, None, None, A, N, 1e-3, dtype)
    assert h.dtype == dtype
    close(h, O.rms(O.gather_streams(x, w_in), 1e-3) * norm, dtype, "gathered")
    close(X, x, F32, "untouched", 1e-3)
    h = St.hyper_joint(X, Y, M, B, A, N, 1e-3, dtype)
    want = O.spread_streams(x, y, mix, out)
    close(X, want, F32, "streams")
    close(h, O.rms(O.gather_streams(want, w_in), 1e-3) * norm, dtype, "next input")
    if S > 1:
        wrong = O.spread_streams(x, y, mix, out, ("mix_transposed",))
        assert (wrong - want).abs().max() > 0.05 * want.abs().max()


@pytest.mark.parametrize("copies", [1, 2, 5])
def test_embedding_into_several_streams(copies):
    from ipex_llm_b200.ops import stream as St
    from ipex_llm_b200.ops.kv_cache import KeyValueShape, SlotCache
    cache = SlotCache()
    cache.allocate(2, 8, [KeyValueShape(1, 8, 8)], BF16, "cuda")
    table = rnd(30, 44, seed=1, dtype=BF16)
    toks = torch.tensor([3, 29, 3], device="cuda")
    x = St.embed_stream(toks, i32([1, 1, 0]), i32([0, 1, 0]), cache, table.to("cuda", BF16), 2.5, streams=copies)
    close(x.view(3, copies, 44), (table[[3, 29, 3]] * 2.5).unsqueeze(1).expand(3, copies, 44), F32)
    assert cache.history[1, :2].tolist() == [3, 29]


# ------------------------------------------------------------------------------------------------
# silu-gated units and experts
# ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF16, F16])
@pytest.mark.parametrize("M,ff,K", [(1, 24, 40), (2, 2400, 136), (7, 32, 72), (13, 520, 64), (3, 21, 60), (40, 72, 200),
                                    (150, 136, 520), (33, 19, 72)])
def test_silu_gated_unit(dtype, M, ff, K):
    from ipex_llm_b200.models.letarax import interleave_gate_up
    from ipex_llm_b200.ops import stream as St
    g, u = rnd(ff, K, seed=1, dtype=dtype, gain=2 * K ** -0.5), rnd(ff, K, seed=2, dtype=dtype, gain=K ** -0.5)
    x = rnd(M, K, seed=5, dtype=dtype, gain=2.0)
    want = O.silu(x @ g.T) * (x @ u.T)
    W, X = interleave_gate_up(g, u).to("cuda", dtype), x.to("cuda", dtype)
    out = torch.empty(M, ff, dtype=dtype, device="cuda")
    il = ff % 8 == 0
    if M <= St.rows_max(K, dtype) and (il or M <= 8):
        close(St.gemv_rows(W, X, out, St.OUT_ACT, act=St.ACT_SILU_GLU, interleaved=il), want, dtype, "rows")
    close(St.gemm(X, W, torch.empty_like(out), St.OUT_ACT, St.ACT_SILU_GLU, None, il), want, dtype, "gemm")
    close(St.glu_rows((X.float() @ W.float().t()).to(dtype), None, torch.empty_like(out), St.ACT_SILU_GLU, il), want, dtype,
          "from finished products", 2)


@pytest.mark.parametrize("E,groups,keep,top,scale", [(8, 1, 1, 2, 1.0), (15, 5, 3, 5, 1.25), (16, 4, 1, 4, 0.7), (6, 6, 2, 2, 2.0),
                                                     (64, 8, 3, 6, 2.5), (5, 1, 1, 5, 1.0), (10, 5, 5, 1, 1.0), (256, 8, 4, 8, 1.0)])
def test_choice_of_experts(E, groups, keep, top, scale):
    """Soft-max scores, groups by their best expert, renormalised weights; group limits and renormalisation show."""
    from ipex_llm_b200.ops import dense_moe as X
    T = 70
    z = rnd(T, E + 1, seed=E, gain=2.0)
    for t in range(T):                          # apart from one another, so that rounding decides nothing
        z[t, :E] = z[t, :E].sort().values.add(torch.arange(E) * 1e-3)[torch.randperm(E, generator=gen(t))]
    r = {"experts": E, "top": top, "groups": {"count": groups, "keep": keep}, "scale": scale}
    val, idx = O.route(z[:, :E], r)
    bank = X.SoftExpertBank(torch.zeros(E + 1, 8), torch.zeros(E, 16, 8), torch.zeros(E, 8, 8), top, groups, keep, scale,
                            torch.zeros(16, 8), torch.zeros(8, 8))
    w, i, g = X.soft_topk(z.to("cuda", F32).contiguous(), bank)
    assert torch.equal(i.cpu(), idx)
    close(w, val, F32)
    close(g, torch.sigmoid(z[:, E]), F32)
    if keep < groups < E and top > 1:
        assert not torch.equal(O.route(z[:, :E], r, ("no_groups",))[1], idx)


MOE = [  # width, ff, experts, top, groups, keep, scale, shared ff
    (64, 32, 8, 2, 1, 1, 1.0, None), (176, 80, 15, 5, 5, 3, 1.25, 112), (96, 24, 6, 3, 3, 2, 0.7, 24), (40, 20, 4, 2, 2, 1, 2.0, 13),
    (50, 7, 5, 1, 1, 1, 1.0, 9), (128, 64, 16, 6, 4, 2, 2.5, 200), (256, 40, 4, 4, 1, 1, 1.0, 64)]


@pytest.mark.parametrize("dtype", [F32, BF16, F16])
@pytest.mark.parametrize("size", MOE)
def test_experts_with_a_shared_one(dtype, size):
    from ipex_llm_b200.models.letarax import interleave_gate_up
    from ipex_llm_b200.ops import dense_moe as X
    W, ff, E, top, groups, keep, scale, shared = size
    cfg = {"vocab": 4, "width": W, "streams": 1, "layers": [O.parallel_layer(mlp=O.moe(ff, E, top, (groups, keep), scale, shared))]}
    w = {k: v.to(dtype).double() for k, v in O.random_weights(cfg, seed=E).items()}
    p, pre = cfg["layers"][0]["mlp"], "l0.mlp."
    T = 60
    h = rnd(T, W, seed=3, dtype=dtype)
    # rows whose choice rounding could change are left out
    z = torch.softmax(h @ w[pre + "router"].T, -1).sort(-1, descending=True).values
    gap = (z[:, :-1] - z[:, 1:]).min(-1).values if E > 1 else torch.ones(T)
    h = h[gap > 1e-4][:40]
    want = O.experts(w, pre, p, h)
    dev = lambda t: t.to("cuda", dtype)                                                          # noqa: E731
    unit = lambda q: interleave_gate_up(w[q + "gate"], w[q + "up"])                              # noqa: E731
    router = torch.cat([w[pre + "router"], w[pre + "shared.sg"]]) if shared else w[pre + "router"]
    bank = X.SoftExpertBank(dev(router), dev(torch.stack([unit(f"{pre}e{e}.") for e in range(E)])),
                            dev(torch.stack([w[f"{pre}e{e}.down"] for e in range(E)])), top, groups, keep, scale,
                            dev(unit(pre + "shared.")) if shared else None, dev(w[pre + "shared.down"]) if shared else None)
    H = padded(h, dtype, 8)
    out = torch.full((len(h), W), 7.0, device="cuda")
    close(X.soft_moe_grouped(bank, H, out), want, dtype, "grouped", 1.5)
    for n in (1, 2, 5, 8):
        assert bank.rows_ok(n)
        out = torch.full((n, W), 7.0, device="cuda")
        close(X.soft_moe_rows(bank, H[:n], out), want[:n], dtype, f"{n} rows", 1.5)
    faults = ["not_renormalized"] + (["shared_ungated"] if shared else [])
    for f in faults:
        if top < E or f != "not_renormalized" or scale != 1.0:
            assert (O.experts(w, pre, p, h, (f,)) - want).abs().max() > 0.02 * want.abs().max(), f


# ------------------------------------------------------------------------------------------------
# chunked attention alone
# ------------------------------------------------------------------------------------------------
class Attention:
    """The left side of a layer behind its projection, on the kernels and on the oracle, with keys that stand out."""

    def __init__(self, dtype, heads, kv_heads, dim, vdim, chunk, n, rot, standout=(), scale=None, gate_scale=0.75, seed=0):
        from ipex_llm_b200.ops import latent as N, window_attn as A
        from ipex_llm_b200.ops.kv_cache import KeyValueShape, SlotCache
        self.A, self.dtype, self.n = A, dtype, n
        scale = (2.0 if len(standout) else 1.0) * dim ** -0.5 if scale is None else scale
        self.m = {"mask": {"size": chunk}, "rot": {"base": 700.0, "dims": rot}, "scale": scale}
        self.spec = A.AttnSpec(heads, kv_heads, dim, vdim, scale, sink=True, chunk=chunk, rot_pairs=rot // 2, unit_eps=EPS,
                               gated=True, gate_scale=gate_scale)
        q, k = rnd(n, heads, dim, seed=seed + 1, gain=2.0), rnd(n, kv_heads, dim, seed=seed + 2)
        if len(standout):
            # queries of a group share a direction among the entries that do not turn; the stand-out keys point along it
            d = rnd(kv_heads, dim, seed=seed + 3)
            d[:, :rot] = 0.0
            q = 0.3 * q + 2.0 * d.repeat_interleave(heads // kv_heads, 0)
            for i, p in enumerate(standout):
                k[p] = d * (2.0 + i)
        self.q, self.k, self.v, self.g = (t.to(dtype).double() for t in (
            q, k, rnd(n, kv_heads, vdim, seed=seed + 4), rnd(n, heads * vdim, seed=seed + 5)))
        self.sink = rnd(heads, seed=seed + 6) + 1.0
        cos, sin = N.rotary_table(n + 64, 700.0, rot // 2, "cuda")
        self.tables = A.AttnTables(self.sink.to("cuda", F32), cos, sin)
        self.cache = SlotCache()
        self.cache.allocate(4, n + 64, [KeyValueShape(kv_heads, dim, vdim)], dtype, "cuda")

    def want(self, faults=(), a=0, b=None):
        """Outputs of rows a .. b taken as a sequence of its own."""
        q, k, v, g = (t[a:b] for t in (self.q, self.k, self.v, self.g))
        o = O.chunk_attend(q, k, v, self.m, self.sink, EPS, faults).flatten(1)
        return o if "no_gate" in faults else o * torch.sigmoid(g) * self.spec.gate_scale

    def operands(self, idx):
        return padded(torch.cat([x[idx].flatten(1) for x in (self.q, self.k, self.v, self.g)], 1), self.dtype)

    def out(self, n):
        w = self.spec.heads * self.spec.vdim
        return torch.empty(n, (w + 7) // 8 * 8, dtype=self.dtype, device="cuda")[:, :w]

    def step(self, cuts, slot=2, first=0, nsplit=None):
        """Portions [cuts[i], cuts[i + 1]); portions of one token prepare and append on the way."""
        self.cache.set_first_rows([first if s == slot else 0 for s in range(4)])
        outs = []
        for a, b in zip(cuts, cuts[1:]):
            outs.append(self.A.attend_step(self.spec, self.operands(list(range(a, b))), None, i32([slot] * (b - a)),
                                           i32(list(range(first + a, first + b))), self.cache, 0, self.out(b - a),
                                           self.spec.seen(b), b - a == 1, nsplit=nsplit, tables=self.tables))
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
        return self.A.attend_prompt(self.spec, self.operands(list(range(T))), None, i32(sl), i32(pos), i32(row), i32(lens),
                                    max(lens), self.cache, 0, self.out(T), self.tables)


ATTN_SIZES = [  # heads, kv_heads, dim, vdim, rotated
    (4, 2, 32, 24, 16), (6, 6, 48, 40, 48), (16, 1, 16, 8, 4), (3, 3, 10, 7, 6), (20, 2, 128, 128, 64), (5, 1, 64, 96, 32),
    (24, 8, 256, 16, 128), (2, 1, 8, 200, 2)]


@pytest.mark.parametrize("dtype", [F32, BF16, F16])
@pytest.mark.parametrize("size", ATTN_SIZES)
@pytest.mark.parametrize("chunk", [1, 13, 64])
def test_attention_step_kernel(dtype, size, chunk):
    n = 75
    at = Attention(dtype, *size[:4], chunk, n, size[4])
    want = at.want()
    close(at.step([0, 1, 3, 40, 42, 75]), want, dtype, "portions")
    close(at.step([0, 30] + list(range(31, 76)), nsplit=4), want, dtype, "one by one")
    close(at.step([0, 64, 65, 75], slot=1, first=9, nsplit=8), want, dtype, "first row 9")


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_sink_rotation_norm_gate_and_head_groups_show(dtype):
    at = Attention(dtype, 6, 3, 24, 16, 9, 40, 16)
    want = at.want()
    for fault in ("no_sink", "heads_interleaved", "no_rotation", "other_pairs", "no_unit_norm", "no_gate"):
        assert (at.want((fault,)) - want).abs().max() > 6 * TOL[dtype] * want.abs().max(), fault
    for scale in (-3.0, 4.0):
        far = Attention(dtype, 2, 1, 8, 8, 20, 60, 4, scale=scale)
        close(far.step([0, 30] + list(range(31, 61))), far.want(), dtype, "scores far from the sink's")
        if dtype != F32:
            close(far.prompt([60], [0]), far.want(), dtype, "prompt, scores far from the sink's")


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("chunk", [16, 100, 128, 129, 300])
def test_chunk_edges_with_a_key_that_stands_out(dtype, chunk):
    """The stand-out keys decide every query of their own chunk behind them, the last position of it included, and none of the
    next chunk; decoding one by one, in portions and (16-bit) as a prompt."""
    p, n = chunk - 3, 2 * chunk + 7
    at = Attention(dtype, 6, 2, 48, 32, chunk, n, 16, standout=(p, 2 * chunk - 1))
    want = at.want()
    inside, outside = [chunk - 1, 2 * chunk - 1], [chunk, chunk + 1, 2 * chunk]
    for fault, row in (("chunk_plus_one", chunk), ("chunk_minus_one", chunk - 1)):
        assert (at.want((fault,))[row] - want[row]).abs().max() > 8 * TOL[dtype] * want.abs().max()
    runs = {"portions": at.step([0, 9, chunk - 1, chunk + 1, n]), "one by one": at.step([0, 10] + list(range(11, n + 1))),
            "one by one, split": at.step([0, 10] + list(range(11, n + 1)), nsplit=8)}
    if dtype == BF16:
        runs["prompt"] = at.prompt([n], [0])
    for name, got in runs.items():
        close(got[inside + outside], want[inside + outside], dtype, f"{name} edge")
        close(got, want, dtype, name)


@pytest.mark.parametrize("dtype", [BF16, F16])
@pytest.mark.parametrize("size", [(4, 2, 32, 24, 16), (2, 2, 64, 64, 64), (6, 1, 128, 96, 32), (4, 4, 192, 128, 128), (3, 3, 72, 104, 8),
                                  (8, 4, 256, 8, 64)])
@pytest.mark.parametrize("chunk", [50, 128, 200, 1000])
def test_prompt_kernel_on_packed_sequences(dtype, size, chunk):
    """Sequences of different lengths behind one another, chunks counted from each one's own start; what the prompt filed
    serves the steps that follow."""
    lens = [130, 1, 257, 64, 5]
    at = Attention(dtype, *size[:4], chunk, sum(lens) + 1, size[4], standout=() if size[2] == size[4] else (2, 140, 141, 260))
    assert at.spec.prefill_ok(dtype)
    got, row = at.prompt(lens, [0, 1, 2, 3, 0]), 0
    for n in lens:
        close(got[row:row + n], at.want(a=row, b=row + n), dtype, f"rows {row}..{row + n}")
        row += n
    n = lens[2]                                       # slot 2 goes on by one token behind its prompt
    idx = list(range(131, 131 + n)) + [sum(lens)]
    out = at.A.attend_step(at.spec, at.operands(idx[-1:]), None, i32([2]), i32([n]), at.cache, 0, at.out(1), n + 1, True,
                           tables=at.tables)
    at.q, at.k, at.v, at.g = (t[idx] for t in (at.q, at.k, at.v, at.g))
    close(out[0], at.want()[-1], dtype, "next token")


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_unequal_sequences_in_one_step(dtype):
    """One new token each for sequences of different lengths in different slots, one of them at its very first token."""
    at = Attention(dtype, 8, 2, 40, 16, 33, 90, 24)
    spans = {3: (0, 50), 0: (50, 80), 1: (80, 81)}     # slot -> rows that make up its sequence
    for s, (a, b) in spans.items():
        if b - a > 1:
            at.A.attend_step(at.spec, at.operands(list(range(a, b - 1))), None, i32([s] * (b - a - 1)), i32(list(range(b - a - 1))),
                             at.cache, 0, at.out(b - a - 1), 60, False, tables=at.tables)
    out = at.A.attend_step(at.spec, at.operands([b - 1 for _, b in spans.values()]), None, i32(list(spans)),
                           i32([b - a - 1 for a, b in spans.values()]), at.cache, 0, at.out(3), 60, True, tables=at.tables)
    for i, (a, b) in enumerate(spans.values()):
        close(out[i], at.want(a=a, b=b)[-1], dtype, f"sequence {i}")


# ------------------------------------------------------------------------------------------------
# gated linear attention alone
# ------------------------------------------------------------------------------------------------
class Linear:
    """The right side of a layer behind its projections, on the kernels and on the oracle."""

    def __init__(self, dtype, heads, dim, vdim, rank, n, bias=1.0, tau=8.0, scale=0.625, seed=0):
        from ipex_llm_b200.engine.stream_engine import Portions
        from ipex_llm_b200.ops import linear_attn as R
        from ipex_llm_b200.ops.kv_cache import DeltaStateShape, SlotCache
        self.R, self.Portions, self.dtype, self.n = R, Portions, dtype, n
        self.spec = s = R.LinearSpec(heads, dim, vdim, rank, tau, scale)
        self.x = rnd(n, s.rows, seed=seed + 1, dtype=dtype)
        self.low = rnd(n, rank, seed=seed + 2)
        self.up = rnd(heads * dim, rank, seed=seed + 3, dtype=dtype, gain=1.5 * rank ** -0.5)
        self.bias = rnd(heads * dim, seed=seed + 4, gain=1.5) + bias
        self.norm = (1 + 0.2 * rnd(vdim, seed=seed + 5)).to(dtype).double()
        self.refresh()
        self.cache = SlotCache()
        self.cache.allocate(4, n + 64, [DeltaStateShape(heads, dim, vdim, 0, 0)], dtype, "cuda")

    def refresh(self):
        self.weights = self.R.LinearWeights(self.up.to("cuda", self.dtype), self.bias.cuda(), self.norm.to("cuda", self.dtype),
                                            EPS)

    def want(self, a=0, b=None, faults=()):
        s, n = self.spec, len(self.x[a:b])
        H, D, V = s.heads, s.dim, s.vdim
        q, k, v, g = self.x[a:b].split([H * D, H * D, H * V, H * V], 1)
        alpha = O.channel_decay((self.low[a:b] @ self.up.T + self.bias).view(n, H, D), s.tau)
        if "one_decay_per_head" in faults:
            alpha = alpha.mean(-1, keepdim=True).expand_as(alpha)
        o, state = O.linear_rule(q.view(n, H, D) * D ** -0.5, k.view(n, H, D), v.view(n, H, V), alpha, faults=faults)
        o = (O.rms(o, EPS) * self.norm).flatten(1) * O.silu(g) * s.out_scale
        return o, state

    def portions(self, lens):
        row, c, owner, first, rows = 0, 0, [], [0], []
        for i, n in enumerate(lens):
            rows.append(row)
            k = -(-n // 32)
            owner += [i] * k
            row, c = row + n, c + k
            first.append(c)
        return self.Portions(i32(rows), i32(lens), max(lens), False, i32(owner), i32(first), c)

    def run(self, idx, slots, pos, lens=None, chunked=None):
        """One call over the rows ``idx``; ``lens``: portions they make up, None: one token each."""
        w = self.spec.heads * self.spec.vdim
        out = torch.empty(len(idx), (w + 7) // 8 * 8 + 8, dtype=self.dtype, device="cuda")[:, 8:8 + w]
        return self.R.linear_mix(self.spec, self.weights, padded(self.x[idx], self.dtype), self.low[idx].to("cuda", F32),
                                 i32(slots), i32(pos), self.cache, 0, out, None if lens is None else self.portions(lens),
                                 chunked=chunked)

    def step(self, cuts, slot=2, first=0, chunked=None):
        self.cache.set_first_rows([first if s == slot else 0 for s in range(4)])
        return torch.cat([self.run(list(range(a, b)), [slot] * (b - a), list(range(first + a, first + b)),
                                   None if b - a == 1 else [b - a], chunked) for a, b in zip(cuts, cuts[1:])])

    def state(self, slot):
        return self.cache.layers[0]._k[slot]


LINEAR_SIZES = [  # heads, dim, vdim, rank
    (4, 16, 24, 6), (3, 32, 32, 16), (2, 128, 128, 16), (6, 24, 40, 5), (2, 10, 7, 1), (1, 200, 96, 33), (2, 256, 64, 64),
    (2, 48, 300, 16), (4, 8, 16, 7), (5, 56, 72, 24), (1, 64, 256, 128)]


@pytest.mark.parametrize("dtype", [F32, BF16, F16])
@pytest.mark.parametrize("size", LINEAR_SIZES + [(1, 300, 24, 3)])
def test_linear_token_by_token_and_in_portions(dtype, size):
    n = 70
    d = Linear(dtype, *size, n)
    want, state = d.want()
    for name, cuts, kw in (("one by one", list(range(n + 1)), {}), ("portions", [0, 1, 3, 5, 40, 41, 70], {"chunked": False}),
                           ("portions from row 9", [0, 2, 33, 70], {"chunked": False, "first": 9, "slot": 1})):
        close(d.step(cuts, **kw), want, dtype, name)
        close(d.state(kw.get("slot", 2)), state, F32, name + ", state", 5)


@pytest.mark.parametrize("dtype", [BF16, F16])
@pytest.mark.parametrize("size", LINEAR_SIZES)
@pytest.mark.parametrize("bias,tau", [(4.0, 16.0), (0.0, 4.0), (-3.0, 1.0), (-40.0, 1.0)])
def test_linear_in_chunks(dtype, size, bias, tau):
    """Chunk borders everywhere, portions that go on from a state, decays from hundreds of tokens down to nothing at once
    (products that underflow, not differences that overflow); the state agrees to 32-bit accuracy."""
    n = 150
    d = Linear(dtype, *size, n, bias=bias, tau=tau)
    if bias < -10:                                       # channels that forget everything beside some that keep it
        d.bias[::3] = 5.0
        d.refresh()
    assert d.spec.chunks_ok(dtype)
    want, state = d.want()
    for cuts in ([0, n], [0, 33, 65, 129, 150], [0, 1, 2, 34, 66, 149, 150], [0, 96, 150]):
        close(d.step(cuts, chunked=True), want, dtype, f"cuts {cuts}")
        close(d.state(2), state, F32, f"state, cuts {cuts}", 5)
    close(d.step([0, 40, 150], slot=0, first=7, chunked=True), want, dtype, "first row 7")


def test_linear_chunks_in_several_passes():
    """A prompt longer than the scratch runs in passes; sequences then start and end in the middle of a pass."""
    from ipex_llm_b200.native.lib import stream_lib
    d = Linear(BF16, 4, 16, 24, 6, 300)
    lens, old = [70, 1, 130, 99], d.R.SCRATCH_BYTES
    per = 4 * 4 * int(stream_lib("linear").ipex_linear_scratch_floats(16, 24))
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
def test_linear_unequal_sequences_and_used_slots(dtype):
    """Prompts of several lengths in one call, then one token each; then the slots go to other sequences without being
    cleared, among them one that starts with a single token."""
    d = Linear(dtype, 4, 32, 40, 16, 240)
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


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_linear_far_write_is_found_again(dtype):
    """A key far back of its own direction is read through channels that hardly forget, past channels that do; the order of
    decay, write and read-out and the decay per channel show."""
    n = 400
    d = Linear(dtype, 2, 16, 16, 4, n, tau=16.0)
    d.bias[:] = 0.0
    d.bias[12::16], d.bias[28::16] = 9.0, 9.0           # one channel per head remembers
    d.low[:] *= 0.1
    d.refresh()
    d.x[:, 32 + 12:64:16] = 0.0                         # only token 5 writes there
    d.x[5, 32 + 12:64:16] = 4.0
    d.x[n - 1, :32] = 0.0
    d.x[n - 1, 12:32:16] = 4.0
    want, _ = d.want()
    assert (want[n - 1] - d.want(6)[0][-1]).abs().max() > 0.1
    for fault in ("read_before_write", "decay_after_write", "one_decay_per_head"):
        assert (want - d.want(faults=(fault,))[0]).abs().max() > 0.05, fault
    close(d.step([0, 300] + list(range(301, n + 1)), chunked=False), want, dtype, factor=5 if dtype == F32 else 1)
    if dtype == BF16:
        close(d.step([0, n], chunked=True), want, dtype)


# ------------------------------------------------------------------------------------------------
# latent attention with borrowed rows and gates
# ------------------------------------------------------------------------------------------------
class Latent:
    """Two layers behind their projections on one store of latents: the second reads what the first filed."""

    def __init__(self, dtype, heads, dim, rd, vd, R, n, heads2, standout=None):
        from ipex_llm_b200.models.dodilix import split_pairs
        from ipex_llm_b200.ops import latent as N
        from ipex_llm_b200.ops.kv_cache import SlotCache
        self.N, self.dtype, self.R, self.rd = N, dtype, R, rd
        self.m = [{"heads": h, "dim": dim, "rot_dim": rd, "vdim": vd, "kv_rank": R, "scale": (dim + rd) ** -0.5,
                   "rot": {"base": 900.0, "dims": rd}} for h in (heads, heads2)]
        self.specs = [N.LatentSpec(m["heads"], dim, rd, vd, R, m["scale"], 0, rd // 2, EPS) for m in self.m]
        self.kv = rnd(n, R + rd, seed=1, dtype=dtype)
        if standout is not None:
            self.kv[standout] *= 3.0
            self.kv[standout, R:] = self.kv[standout, R:] * 2
        self.norm = (1 + 0.2 * rnd(R, seed=2)).to(dtype).double()
        self.q = [rnd(n, m["heads"], dim + rd, seed=3 + i, dtype=dtype, gain=2.0) for i, m in enumerate(self.m)]
        self.uk = [rnd(m["heads"] * dim, R, seed=5 + i, dtype=dtype, gain=R ** -0.5) for i, m in enumerate(self.m)]
        self.uv = [rnd(m["heads"] * vd, R, seed=7 + i, dtype=dtype, gain=R ** -0.5) for i, m in enumerate(self.m)]
        self.g = [rnd(n, m["heads"] * vd, seed=9 + i, dtype=dtype) for i, m in enumerate(self.m)]
        pairs = lambda t: split_pairs(t.transpose(-1, -2), rd // 2).transpose(-1, -2)            # noqa: E731
        self.kv_dev = torch.cat([self.kv[:, :R], pairs(self.kv[:, R:])], 1)
        self.q_dev = [torch.cat([q[..., :dim], pairs(q[..., dim:])], -1) for q in self.q]
        self.cos, self.sin = N.rotary_table(n + 64, 900.0, rd // 2, "cuda")
        self.cache = SlotCache()
        self.cache.allocate(3, n + 64, [self.specs[0].row(dtype)], dtype, "cuda")

    def want(self, i, a=0, b=None, faults=()):
        kv = self.kv[a:b]
        c = O.rms(kv[:, :self.R], EPS) * self.norm
        kr = O.turn_neighbours(kv[:, self.R:], torch.arange(len(kv)), 900.0, self.rd)
        o = O.latent_attend(self.q[i][a:b], c, kr, self.uk[i], self.uv[i], self.m[i], faults).flatten(1)
        return o * torch.sigmoid(self.g[i][a:b])

    def call(self, i, idx, slots, pos, prompt=None, rows=None):
        dev = lambda t: t.to("cuda", self.dtype).contiguous()                                    # noqa: E731
        out = padded(torch.zeros(len(idx), self.uv[i].shape[0]), self.dtype)
        args = (self.specs[i], padded(self.q_dev[i][idx].flatten(1), self.dtype), dev(self.uk[i]), dev(self.uv[i]),
                dev(self.norm) if i == 0 else None, self.cos, self.sin, i32(slots), i32(pos))
        kw = {"kv": padded(self.kv_dev[idx], self.dtype, 8) if i == 0 else None, "gate": padded(self.g[i][idx], self.dtype)}
        if prompt is not None:
            return self.N.latent_prompt(*args, *prompt, self.cache, 0, out, rows_out=rows, **kw)
        return self.N.latent_step(*args, self.cache, 0, out, max(pos) + 1, **kw)


LATENT_SIZES = [  # heads, dim, rot_dim, vdim, rank, n, heads of the borrower
    (4, 24, 16, 32, 64, 70, 3), (3, 10, 6, 7, 33, 50, 5), (20, 128, 64, 128, 512, 40, 16), (2, 16, 8, 80, 96, 300, 4)]


@pytest.mark.parametrize("dtype", [F32, BF16, F16])
@pytest.mark.parametrize("size", LATENT_SIZES)
def test_latent_rows_are_lent(dtype, size):
    d, n = Latent(dtype, *size), size[5]
    want = [d.want(0), d.want(1)]
    assert (d.want(0, faults=("other_latent_pairs",)) - want[0]).abs().max() > 6 * TOL[dtype] * want[0].abs().max()
    for cuts, slot in (([0, n - 20] + list(range(n - 19, n + 1)), 1), ([0, 2, 3, 20, n], 2)):
        got = [[], []]
        for a, b in zip(cuts, cuts[1:]):
            for i in (0, 1):                             # the lender files its rows first
                got[i].append(d.call(i, list(range(a, b)), [slot] * (b - a), list(range(a, b))))
        for i in (0, 1):
            close(torch.cat(got[i]), want[i], dtype, f"layer {i}, {cuts[:4]}", 2)
    if dtype != F32 and d.specs[0].prefill_ok(dtype):
        lens = [n - 9, 9]
        pos = list(range(n - 9)) + list(range(9))
        prompt = (i32([0, n - 9]), i32(lens), n - 9)
        rows = d.N.prompt_rows(d.specs[0], n, dtype, "cuda")
        for i in (0, 1):
            got = d.call(i, list(range(n)), [0] * (n - 9) + [1] * 9, pos, prompt, rows)
            close(got, torch.cat([d.want(i, 0, n - 9), d.want(i, n - 9, n)]), dtype, f"prompt, layer {i}", 2)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_latent_far_key(dtype):
    """An early key that stands out decides the outputs a thousand tokens later, decoded or in a portion."""
    n = 1100
    d = Latent(dtype, 4, 24, 16, 32, 64, n, 3, standout=3)
    for i in (0, 1):
        want = d.want(i)
        assert (want[-1] - d.want(i, 4)[-1]).abs().max() > 4 * TOL[dtype] * want.abs().max()
        d.call(i, list(range(n - 3)), [1] * (n - 3), list(range(n - 3)))
        got = [d.call(i, [t], [1], [t]) for t in (n - 3, n - 2)] + [d.call(i, [n - 1], [1], [n - 1])]
        close(torch.cat(got), want[-3:], dtype, f"layer {i}", 2)


# ------------------------------------------------------------------------------------------------
# whole models
# ------------------------------------------------------------------------------------------------
def cfg_a():
    return {"architecture": "Dodilix", "vocab": 150, "width": 96, "norm": {"eps": 1e-5}, "streams": 3, "logit_scale": 0.75,
            "embedding": {"scale": 1.5},
            "layers": [O.latent_layer(4, 24, 16, 32, 40, 64, mlp=O.dense(160)),
                       O.parallel_layer(4, 2, 32, 24, 21, 16, lheads=3, ldim=16, lvdim=24,
                                        mlp=O.moe(24, 6, 3, (3, 2), 1.5, 40)),
                       O.latent_layer(3, 16, 16, 24, 24, 64, kv_from=0, mlp=O.moe(32, 8, 2, None, 1.0, None)),
                       O.parallel_layer(6, 3, 16, 32, 64, 8, lheads=2, ldim=32, lvdim=40, tau=2.0, mlp=None),
                       O.latent_layer(5, 8, 8, 16, 32, 48, base=300.0, mlp=None)]}


def cfg_odd():
    """Nothing a multiple of anything: the generic kernels."""
    return {"architecture": "Dodilix", "vocab": 101, "width": 50, "norm": {"eps": 1e-3}, "streams": 5, "logit_scale": 1.25,
            "embedding": {"scale": 0.5},
            "layers": [O.parallel_layer(3, 1, 10, 9, 17, 6, lheads=3, ldim=10, lvdim=7, tau=1.0, left_scale=1.0,
                                        right_scale=1.0, mlp=O.dense(33)),
                       O.latent_layer(3, 10, 6, 7, 13, 33, mlp=O.moe(11, 5, 2, None, 0.6, 9)),
                       O.latent_layer(2, 5, 6, 9, 21, 33, kv_from=1, mlp=O.dense(21))]}


def cfg_one():
    """One stream, one head here and there, one expert chosen; every position its own chunk."""
    return {"architecture": "Dodilix", "vocab": 64, "width": 64, "norm": {"eps": 1e-6}, "streams": 1, "logit_scale": 1.0,
            "embedding": {"scale": 1.0},
            "layers": [O.parallel_layer(1, 1, 64, 64, 1, 64, lheads=1, ldim=64, lvdim=64, mlp=O.moe(16, 4, 1, (4, 1), 1.0, 16)),
                       O.latent_layer(1, 32, 32, 64, 16, 32, mlp=O.dense(128))]}


def cfg_latent():
    """Latent attention only, two lenders."""
    return {"architecture": "Dodilix", "vocab": 120, "width": 64, "norm": {"eps": 1e-6}, "streams": 2, "logit_scale": 2.0,
            "embedding": {"scale": 1.0},
            "layers": [O.latent_layer(2, 32, 32, 64, 24, 64, mlp=O.dense(128)),
                       O.latent_layer(4, 16, 8, 32, 24, 32, base=50.0, mlp=O.dense(64)),
                       O.latent_layer(3, 24, 32, 16, 24, 64, kv_from=0, mlp=O.dense(64)),
                       O.latent_layer(2, 16, 8, 32, 24, 32, base=50.0, kv_from=1, mlp=O.dense(64))]}


def cfg_parallel():
    """Layers of two sides only; chunks of a tile."""
    return {"architecture": "Dodilix", "vocab": 120, "width": 64, "norm": {"eps": 1e-6}, "streams": 4, "logit_scale": 1.0,
            "embedding": {"scale": 1.0},
            "layers": [O.parallel_layer(2, 2, 64, 64, 64, 32, lheads=2, ldim=32, lvdim=32, mlp=O.dense(128)),
                       O.parallel_layer(4, 1, 32, 16, 128, 32, lheads=4, ldim=16, lvdim=32, mlp=O.moe(32, 4, 2, (2, 1), 1.0, 64))]}


CFGS = {"a": cfg_a, "odd": cfg_odd, "one": cfg_one, "latent": cfg_latent, "parallel": cfg_parallel}
_models, _want = {}, {}


def make(name, dtype):
    from ipex_llm_b200.models import dodilix
    from ipex_llm_b200.transformers.model import _attach_api
    key = (name, dtype)
    if key not in _models:
        cfg = CFGS[name]()
        w = O.random_weights(cfg, seed=len(name), sharp=2.0, rank=5 if name == "odd" else 16, spread=0.3)
        model = _attach_api(dodilix.build(cfg, w, dtype).to("cuda"))
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


# logits through several layers: rounding adds up and a sharp soft-max amplifies it; a 16-bit input may also turn the choice
# of an expert around, which a few rows then show
MODEL_TOL = {F32: 4.0, BF16: 5.0}


def agree(got, want, dtype, what=""):
    got, want = got.double().cpu(), want.double().cpu()
    if dtype == F32:
        return close(got, want, dtype, what, MODEL_TOL[dtype])
    assert torch.isfinite(got).all(), what
    err = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    worst = err.sort().values
    assert worst[int(0.9 * (len(worst) - 1))] < 0.06 and err.median() < 0.04, f"{what}: {worst[-5:].tolist()}"


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
        agree(torch.cat(got), want, dtype, f"cuts {cuts[:4]}")
    for graph in (True, False):
        eng = engine(model)
        s = eng.cache.acquire()
        got = [eng.step_rows([(s, toks[:3], [0, 1, 2])])]
        got += [eng.step_rows([(s, [t], [0])], use_graph=graph).clone() for t in toks[3:]]
        agree(torch.cat(got), want, dtype, f"token by token, graph={graph}")


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", ["a", "odd"])
def test_streams_after_every_layer(name, dtype):
    model, cfg, w = make(name, dtype)
    toks = tokens(41, cfg["vocab"], 7)
    trace, got = [], []
    O.forward(w, cfg, toks, trace=trace)
    eng = engine(model)
    eng.stack.run_portions([(eng.cache.acquire(), 0, toks)], eng.cache, collect=got)
    for i, (g, t) in enumerate(zip(got, trace)):
        agree(g, t, dtype, f"layer {i}")
        assert g.dtype == F32


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_ragged_batches_against_each_alone(dtype):
    """Unequal prompts in one batch, decoded together while the shorter ones leave; slots handed to new sequences."""
    model, cfg, _ = make("a", dtype)
    V = cfg["vocab"]
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
    agree(torch.cat([torch.cat(g) for g in got]), torch.cat(want), dtype, "together")
    # all slots are free again: other sequences, other lengths, in another order
    again = [seqs[2], seqs[1], seqs[3], seqs[2][:40]]
    slots = [eng.cache.acquire() for _ in again]
    lg = eng.step_rows([(sl, s, list(range(len(s)))) for sl, s in zip(slots, again)])
    agree(lg, torch.cat([want[2], want[1], want[3], want[2][:40]]), dtype, "reused slots")


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
    agree(lg, torch.cat([wb[30:], wa[39:], wc]), dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name,count", [("a", 19), ("a", 12), ("odd", 11)])
def test_many_sequences_decode_together(name, count, dtype):
    """More rows than the small row products take, then more than any of them does: GEMMs in the decode graph."""
    model, cfg, _ = make(name, dtype)
    seqs = [tokens(20 + 3 * i, cfg["vocab"], 80 + i) for i in range(count)]
    want = [oracle(name, s) for s in seqs]
    eng = engine(model, count)
    slots = [eng.cache.acquire() for _ in seqs]
    eng.step_rows([(sl, s[:-4], []) for sl, s in zip(slots, seqs)])
    got = [eng.step_rows([(sl, [s[-k]], [0]) for sl, s in zip(slots, seqs)]).clone() for k in range(4, 0, -1)]
    agree(torch.cat(got), torch.cat([torch.stack([w[-k] for w in want]) for k in range(4, 0, -1)]), dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_long_decoding(dtype):
    """Many chunks and graphs past the prompt, one token at a time."""
    model, cfg, _ = make("a", dtype)
    toks = tokens(330, cfg["vocab"], 3)
    want = oracle("a", toks)
    eng = engine(model)
    s = eng.cache.acquire()
    got = [eng.step_rows([(s, toks[:11], [10])])]
    got += [eng.step_rows([(s, [t], [0])]).clone() for t in toks[11:]]
    agree(torch.cat(got), want[10:], dtype)


# ------------------------------------------------------------------------------------------------
# the framework's entry points
# ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", ["a", "odd", "one"])
def test_greedy_generate(name):
    model, cfg, w = make(name, F32)
    prompts = [tokens(n, cfg["vocab"], n) for n in (23, 6, 14)]
    want = [O.greedy(w, cfg, p, 12) for p in prompts]
    for p, e in zip(prompts, want):
        out = model.generate(torch.tensor([p], device="cuda"), max_new_tokens=12, do_sample=False)
        assert out[0, len(p):].tolist() == e
        assert type(model._ipex_engine).__name__ == "MultiStreamEngine"
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
        agree(out.logits[b], O.forward(w, cfg, ids[b].tolist()), F32)
    more = model(torch.tensor([[5], [6]], device="cuda"), past_key_values=out.past_key_values)
    agree(more.logits[1, -1:], O.forward(w, cfg, p[::-1] + [6])[-1:], F32)
    assert model(ids, logits_to_keep=2).logits.shape == (2, 2, cfg["vocab"])
    beams = model.generate(ids[:1], max_new_tokens=5, num_beams=3, do_sample=False, pad_token_id=0)
    full = torch.log_softmax(O.forward(w, cfg, beams[0].tolist()), -1)
    lp = sum(full[18 + i, beams[0, 19 + i]].item() for i in range(5))
    g = O.greedy(w, cfg, p, 5)
    fg = torch.log_softmax(O.forward(w, cfg, p + g), -1)
    assert lp >= sum(fg[18 + i, t].item() for i, t in enumerate(g)) - 1e-6      # never worse than greedy


def test_prompt_lookup_on_latents_alone():
    """Without a recurrent side drafts may be taken back: lookup gives the greedy tokens."""
    model, cfg, w = make("latent", F32)
    p = tokens(9, cfg["vocab"], 6) * 3
    out = model.generate(torch.tensor([p], device="cuda"), max_new_tokens=8, do_sample=False, lookahead=2)
    assert out[0, len(p):].tolist()[:8] == O.greedy(w, cfg, p, 8)


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
    """Packed projections beside dense experts and up-projections: logits close to those of the dense weights."""
    from ipex_llm_b200.models import dodilix
    from ipex_llm_b200.transformers import AutoModelForCausalLM
    cfg = {"architecture": "Dodilix", "vocab": 128, "width": 128, "norm": {"eps": 1e-6}, "streams": 2, "logit_scale": 1.0,
           "embedding": {"scale": 1.0},
           "layers": [O.parallel_layer(4, 2, 32, 32, 30, 32, lheads=4, ldim=32, lvdim=32, mlp=O.dense(256)),
                      O.latent_layer(4, 32, 32, 32, 64, 64, mlp=O.moe(64, 4, 2, None, 1.0, 64))]}
    w = O.random_weights(cfg, sharp=1.0)
    write_checkpoint(str(tmp_path), cfg, w)
    m8 = AutoModelForCausalLM.from_pretrained(str(tmp_path), load_in_low_bit="sym_int8").to("cuda")
    ref = dodilix.build(cfg, w, BF16).to("cuda")
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
    model = AutoModelForCausalLM.from_pretrained(str(tmp_path), load_in_low_bit="bf16", torch_dtype=BF16, device="cuda")
    out = model.generate(torch.tensor([[3, 9, 4, 77]], device="cuda"), max_new_tokens=6, do_sample=False)
    assert got == out[0, 4:].tolist() and len(got) == 6


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay(tmp_path, dtype):
    """The replay program on a checkpoint: a batch that starts together and thins out, then another request."""
    import subprocess
    import sys
    import numpy as np
    cfg = cfg_a()
    w = O.random_weights(cfg, seed=4, sharp=2.0, spread=0.3)
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
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", d, "--dtype", dtype, "--out",
                        out, "--max-tokens", "90"], input="".join(json.dumps(s) + "\n" for s in steps), text=True,
                       capture_output=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == [f"done {i}" for i in range(4)]
    w64 = {k: v.double() for k, v in w.items()}
    fx, fy, fz = (O.forward(w64, cfg, t) for t in (x, y, z))
    got = [torch.from_numpy(np.fromfile(os.path.join(out, f"{s}.f32"), dtype="<f4").reshape(-1, V)) for s in (0, 2, 3)]
    agree(torch.cat(got), torch.cat([fx[9:10], torch.stack([fx[11], fy[69]]), fz[[0, 8]]]), getattr(torch, dtype))
    assert not os.path.exists(os.path.join(out, "1.f32"))
