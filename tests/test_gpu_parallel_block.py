"""Gegorax on the GPU: every kernel against the float64 oracle (``tests/gegorax_oracle.py``), then the engine with whole
prompts, portions, ragged batches, slot reuse, long decoding and generation."""
import json
import os

import pytest
import torch

import gegorax_oracle as O

pytestmark = pytest.mark.gpu

F32, BF16, F16 = torch.float32, torch.bfloat16, torch.float16
TOL = {F32: 2e-5, F16: 4e-3, BF16: 2.5e-2}          # relative to the size of the compared values
EPS = 1e-5
CUDA = "cuda"


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
    return torch.tensor(v, dtype=torch.int32, device=CUDA)


def padded(x, dtype, extra=0):
    """``x`` in rows that start on 16-byte boundaries."""
    n = x.shape[1]
    t = torch.zeros(x.shape[0], (n + 7) // 8 * 8 + extra, dtype=dtype, device=CUDA)
    t[:, :n] = x.to(dtype)
    return t[:, :n]


def portions_of(lens, whole=False):
    from ipex_llm_b200.engine.stream_engine import Portions
    row, c, owner, first, rows = 0, 0, [], [0], []
    for i, n in enumerate(lens):
        rows.append(row)
        k = -(-n // 32)
        owner += [i] * k
        row, c = row + n, c + k
        first.append(c)
    return Portions(i32(rows), i32(lens), max(lens), whole, i32(owner), i32(first), c, list(lens))


# ------------------------------------------------------------------------------------------------
# products and joints
# ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF16, F16])
@pytest.mark.parametrize("M,ff,K", [(1, 24, 40), (2, 2400, 136), (7, 32, 72), (13, 520, 64), (3, 21, 60), (40, 72, 200),
                                    (150, 136, 520), (33, 19, 72)])
def test_clamped_unit(dtype, M, ff, K):
    from ipex_llm_b200.models.letarax import interleave_gate_up
    from ipex_llm_b200.ops import stream as St
    g, u = rnd(ff, K, seed=1, dtype=dtype, gain=2 * K ** -0.5), rnd(ff, K, seed=2, dtype=dtype, gain=K ** -0.5)
    x = rnd(M, K, seed=5, dtype=dtype, gain=2.0)
    args = St.ActArgs(limit=0.9, alpha=1.7)
    a, b = (x @ g.T).clamp(max=0.9), (x @ u.T).clamp(-0.9, 0.9)
    want = a * torch.sigmoid(1.7 * a) * (b + 1.0)
    W, X = interleave_gate_up(g, u).to(CUDA, dtype), x.to(CUDA, dtype)
    out = torch.empty(M, ff, dtype=dtype, device=CUDA)
    il = ff % 8 == 0
    if M <= St.rows_max(K, dtype) and (il or M <= 8):
        close(St.gemv_rows(W, X, out, St.OUT_ACT, act=St.ACT_CLAMP_GLU, interleaved=il, args=args), want, dtype, "rows")
    close(St.gemm(X, W, torch.empty_like(out), St.OUT_ACT, St.ACT_CLAMP_GLU, None, il, args=args), want, dtype, "gemm")
    close(St.glu_rows((X.float() @ W.float().t()).to(dtype), None, torch.empty_like(out), St.ACT_CLAMP_GLU, il, args), want,
          dtype, "from finished products", 2)


@pytest.mark.parametrize("dtype", [F32, BF16, F16])
@pytest.mark.parametrize("M,N,K", [(1, 16, 320), (3, 20, 60), (16, 130, 64), (8, 7, 50), (17, 16, 136), (200, 72, 264), (40, 11, 48)])
def test_gelu_times_the_tokens_row(dtype, M, N, K):
    """From activations, and (few rows) from the 32-bit stream as it is; a token id outside the table takes an end row."""
    from ipex_llm_b200.ops import stream as St
    w, x = rnd(N, K, seed=1, dtype=dtype, gain=K ** -0.5), rnd(M, K, seed=2, dtype=dtype, gain=2.0)
    table = rnd(30, 3 * N, seed=3, dtype=dtype)
    ids = torch.randint(0, 30, (M,), generator=gen(4))
    args = St.ActArgs(table=table.to(CUDA, dtype)[:, N:2 * N], ids=ids.cuda())
    want = O.gelu_tanh(x @ w.T) * table[ids, N:2 * N]
    W, X = w.to(CUDA, dtype), x.to(CUDA, dtype)
    out = torch.empty(M, (N + 7) // 8 * 8, dtype=dtype, device=CUDA)[:, :N]
    if M <= St.rows_max(K, dtype):
        for src in (X, x.to(CUDA, F32)):
            close(St.gemv_rows(W, src, out.zero_(), St.OUT_ACT, act=St.ACT_GELU_MUL, args=args), want, dtype, "rows")
    close(St.gemm(X, W, out.zero_(), St.OUT_ACT, St.ACT_GELU_MUL, args=args), want, dtype, "gemm")
    ids2 = ids.clone()
    ids2[0] = 1 << 40
    args = St.ActArgs(table=args.table, ids=ids2.cuda())
    got = St.gemm(X, W, out.zero_(), St.OUT_ACT, St.ACT_GELU_MUL, args=args)
    close(got[:1], O.gelu_tanh(x[:1] @ w.T) * table[29:, N:2 * N], dtype, "outside")


@pytest.mark.parametrize("dtype", [F32, BF16, F16])
@pytest.mark.parametrize("M,N,start,K", [(1, 96, 64, 40), (5, 37, 20, 60), (16, 200, 130, 64), (30, 264, 64, 72), (140, 77, 13, 50)])
def test_squared_relu_from_a_column_on_beside_a_second_matrix(dtype, M, N, start, K):
    from ipex_llm_b200.ops import stream as St
    w, w2, x = rnd(N, K, seed=1, dtype=dtype, gain=K ** -0.5), rnd(9, K, seed=2, dtype=dtype), rnd(M, K, seed=3, dtype=dtype, gain=2.0)
    want = x @ w.T
    want[:, start:] = torch.relu(want[:, start:]) ** 2
    W, W2, X = w.to(CUDA, dtype), w2.to(CUDA, dtype), x.to(CUDA, dtype)
    args = St.ActArgs(start=start)
    for name in ("rows", "gemm"):
        if name == "rows" and M > St.rows_max(K, dtype):
            continue
        out = torch.zeros(M, (N + 7) // 8 * 8, dtype=dtype, device=CUDA)[:, :N]
        out2 = torch.zeros(M, 9, device=CUDA)
        if name == "rows":
            St.gemv_rows(W, X, out, St.OUT_ACT, act=St.ACT_RELU2, w2=W2, out2=out2, args=args)
        else:
            St.gemm(X, W, out, St.OUT_ACT, St.ACT_RELU2, w2=W2, out2=out2, args=args)
        close(out, want, dtype, name)
        close(out2, x @ w2.T, F32, name + ", second matrix")


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("n,K", [(1, 64), (3, 320), (2, 2052), (5, 75), (200, 256), (2, 6000)])
def test_joint_of_sides_normed_side_by_side(dtype, n, K):
    from ipex_llm_b200.ops import stream as St
    x, a, b = rnd(n, K, seed=1, gain=3.0), rnd(n, K, seed=2), rnd(n, K, seed=3, gain=0.1)
    wa, wb, wi = (1 + rnd(K, seed=s, gain=0.2) for s in (4, 5, 6))
    dev = lambda t: t.to(CUDA, F32).contiguous()                                                 # noqa: E731
    for ys, ws, add in (((a, b), (wa, wb), O.rms(a, 1e-3) * wa + O.rms(b, 1e-3) * wb), ((a,), (wa,), O.rms(a, 1e-3) * wa),
                        ((), (), 0.0 * x)):
        for w_in in (None, wi):
            X = dev(x)
            h = St.add_sides(X, [dev(y) for y in ys], [dev(w) for w in ws], None if w_in is None else dev(w_in), 1e-3, dtype)
            close(X, x + add, F32, "stream")
            close(h, x + add if w_in is None else O.rms(x + add, 1e-3) * wi, dtype, "next input")


# ------------------------------------------------------------------------------------------------
# experts
# ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("E,top", [(8, 2), (5, 5), (64, 6), (1, 1), (40, 1), (256, 8)])
def test_choice_of_experts_with_a_bias(E, top):
    from ipex_llm_b200.ops import dense_moe as X
    T = 70
    z, bias = rnd(T, E, seed=E, gain=2.0), rnd(E, seed=E + 1)
    for t in range(T):                          # apart from one another, so that rounding decides nothing
        z[t] = z[t].sort().values.add(torch.arange(E) * 1e-3)[torch.randperm(E, generator=gen(t))]
    val, idx = O.route(z, top)
    bank = X.SoftExpertBank(torch.zeros(E, 8), torch.zeros(E, 16, 8), torch.zeros(E, 8, 8), top, shared_gate_up=torch.zeros(16, 8),
                            shared_down=torch.zeros(8, 8), bias=bias.to(CUDA), shared_gated=False)
    wide = torch.zeros(T, E + 3, device=CUDA)
    wide[:, 2:2 + E] = (z - bias).to(CUDA, F32)
    w, i, g = X.soft_topk(wide[:, 2:2 + E], bank)
    assert torch.equal(i.cpu(), idx) and g is None
    close(w, val, F32)


MOE = [  # width, ff, experts, top, limit, shared ff, shared limit
    (64, 32, 8, 2, 0.7, None, 0.0), (176, 80, 15, 5, 1.5, 112, 0.4), (96, 24, 6, 3, 0.5, 24, 2.0), (40, 20, 4, 2, 1.0, 13, 0.6),
    (50, 7, 5, 1, 0.8, 9, 1.1), (128, 64, 16, 6, 3.0, 200, 1.0), (256, 40, 4, 4, 0.3, 64, 5.0)]


@pytest.mark.parametrize("dtype", [F32, BF16, F16])
@pytest.mark.parametrize("size", MOE)
def test_clamped_experts_with_a_shared_one(dtype, size):
    from ipex_llm_b200.models.letarax import interleave_gate_up
    from ipex_llm_b200.ops import dense_moe as X, stream as St
    W, ff, E, top, limit, shared, sl = size
    cfg = {"vocab": 4, "width": W, "layers": [O.delta_layer(1, 8, mlp=O.moe(ff, E, top, limit, shared, sl))]}
    w = {k: v.to(dtype).double() for k, v in O.random_weights(cfg, seed=E).items()}
    p, pre = cfg["layers"][0]["mlp"], "l0.mlp."
    h = rnd(60, W, seed=3, dtype=dtype)
    # rows whose choice rounding could change are left out
    z = (h @ w[pre + "router"].T + w[pre + "router.b"]).sort(-1, descending=True).values
    gap = (z[:, :-1] - z[:, 1:]).min(-1).values
    h = h[gap > 1e-3][:40]
    want = O.experts(w, pre, p, h)
    dev = lambda t: t.to(CUDA, dtype)                                                            # noqa: E731
    unit = lambda q: interleave_gate_up(w[q + "gate"], w[q + "up"])                              # noqa: E731
    bank = X.SoftExpertBank(dev(w[pre + "router"]), dev(torch.stack([unit(f"{pre}e{e}.") for e in range(E)])),
                            dev(torch.stack([w[f"{pre}e{e}.down"] for e in range(E)])), top,
                            shared_gate_up=dev(unit(pre + "shared.")) if shared else None,
                            shared_down=dev(w[pre + "shared.down"]) if shared else None, act=St.ACT_CLAMP_GLU, limit=limit,
                            alpha=1.702, shared_limit=sl, bias=w[pre + "router.b"].cuda(), shared_gated=False)
    H = padded(h, dtype, 8)
    x = rnd(len(h), W, seed=9)
    logits = (h @ w[pre + "router"].T).to(CUDA, F32)
    for kw in ({}, {"logits": logits}, {"logits": logits, "add": True}):
        base = x if "add" in kw else 0 * x
        out = x.to(CUDA, F32).contiguous()
        close(X.soft_moe_grouped(bank, H, out, **kw) - base.cuda(), want, dtype, "grouped", 1.5)
        for n in (1, 2, 5, 8):
            assert bank.rows_ok(n)
            k2 = {k: v[:n] if k == "logits" else v for k, v in kw.items()}
            out = x[:n].to(CUDA, F32).contiguous()
            close(X.soft_moe_rows(bank, H[:n], out, **k2) - base[:n].cuda(), want[:n], dtype, f"{n} rows", 1.5)
    for f in ["no_clamp", "no_plus_one", "no_router_bias"] + (["no_shared", "shared_limit"] if shared else []):
        if f != "no_router_bias" or top < E:
            if f != "no_clamp" or limit < 2:
                assert (O.experts(w, pre, p, h, (f,)) - want).abs().max() > 0.02 * want.abs().max(), f


# ------------------------------------------------------------------------------------------------
# attention over a window and pooled blocks
# ------------------------------------------------------------------------------------------------
class Attention:
    """The left side of a layer behind its projection, on the kernels and on the oracle, with keys that stand out."""

    def __init__(self, dtype, heads, kv_heads, dim, vdim, size, pool, n, rot, standout=(), scale=None, seed=0):
        from ipex_llm_b200.models.dodilix import split_pairs
        from ipex_llm_b200.ops import latent as N, window_attn as A
        from ipex_llm_b200.ops.kv_cache import KeyValueShape, PooledShape, SlotCache
        self.A, self.dtype, self.n = A, dtype, n
        scale = (2.0 if len(standout) else 1.0) * dim ** -0.5 if scale is None else scale
        self.m = {"mask": {"size": size, "pool": pool}, "rot": {"base": 700.0, "dims": rot}, "scale": scale}
        self.spec = A.AttnSpec(heads, kv_heads, dim, vdim, scale, window=size, pool=pool, rot_pairs=rot // 2, unit_eps=EPS)
        self.wq, self.wk = 1.5 + rnd(dim, seed=seed + 6, gain=0.3), 1.0 + rnd(dim, seed=seed + 7, gain=0.3)
        q, k = rnd(n, heads, dim, seed=seed + 1, gain=2.0), rnd(n, kv_heads, dim, seed=seed + 2)
        if len(standout):
            # queries of a group share a direction among the entries that do not turn; the stand-out keys point along it,
            # the others lean away from it
            d = rnd(kv_heads, dim, seed=seed + 3)
            d[:, :rot] = 0.0
            d = d * (dim / (dim - rot)) ** 0.5
            q = 0.3 * q + 2.0 * d.repeat_interleave(heads // kv_heads, 0)
            k = 0.7 * k - 0.5 * d
            for p in standout:
                k[p] = 3.0 * d + 0.1 * k[p]
        self.q, self.k, self.v = (t.to(dtype).double() for t in (q, k, rnd(n, kv_heads, vdim, seed=seed + 4)))
        for p in standout:
            self.v[p] = torch.sign(self.v[standout[0]]) * (-3.0 if p == standout[-1] else 3.0)
        turn = lambda t: split_pairs(t.transpose(-1, -2), rot // 2).transpose(-1, -2)            # noqa: E731
        self.q_dev, self.k_dev = turn(self.q), turn(self.k)
        cos, sin = N.rotary_table(n + 64, 700.0, rot // 2, CUDA)
        w = [split_pairs(t.view(-1, 1), rot // 2).flatten().to(CUDA, F32).contiguous() for t in (self.wq, self.wk)]
        self.tables = A.AttnTables(None, cos, sin, *w)
        self.cache = SlotCache()
        self.shapes = [KeyValueShape(kv_heads, dim, vdim)] + ([PooledShape(kv_heads, dim, vdim, pool)] if pool else [])
        self.cache.allocate(5, n + 64, self.shapes, dtype, CUDA)
        self.pooled = 1 if pool else None

    def want(self, faults=(), a=0, b=None):
        """Outputs of rows a .. b taken as a sequence of its own."""
        return O.pooled_attend(self.q[a:b], self.k[a:b], self.v[a:b], self.m, self.wq, self.wk, EPS, faults).flatten(1)

    def operands(self, idx):
        return padded(torch.cat([x[idx].flatten(1) for x in (self.q_dev, self.k_dev, self.v)], 1), self.dtype)

    def out(self, n):
        w = self.spec.heads * self.spec.vdim
        return torch.empty(n, (w + 7) // 8 * 8, dtype=self.dtype, device=CUDA)[:, :w]

    def call(self, idx, slots, pos, lens=None, nsplit=None):
        return self.A.attend_step(self.spec, self.operands(idx), None, i32(slots), i32(pos), self.cache, 0, self.out(len(idx)),
                                  self.spec.seen(max(pos) + 1), lens is None, nsplit=nsplit, tables=self.tables,
                                  portions=None if lens is None else portions_of(lens), pooled=self.pooled)

    def step(self, cuts, slot=2, first=0, nsplit=None):
        """Portions [cuts[i], cuts[i + 1]); portions of one token prepare and append on the way."""
        self.cache.set_first_rows([first if s == slot else 0 for s in range(5)])
        return torch.cat([self.call(list(range(a, b)), [slot] * (b - a), list(range(first + a, first + b)),
                                    None if b - a == 1 else [b - a], nsplit) for a, b in zip(cuts, cuts[1:])])

    def prompt(self, lens, slots):
        """Sequences cut out of the rows 0.., packed; every one restarts at position 0."""
        T = sum(lens)
        self.cache.set_first_rows([0] * 5)
        sl, pos, where = [], [], portions_of(lens, True)
        for n, s in zip(lens, slots):
            sl += [s] * n
            pos += list(range(n))
        return self.A.attend_prompt(self.spec, self.operands(list(range(T))), None, i32(sl), i32(pos), where.row, where.length,
                                    max(lens), self.cache, 0, self.out(T), self.tables, where, self.pooled)


ATTN_SIZES = [  # heads, kv_heads, dim, vdim, rotated
    (4, 2, 32, 24, 16), (6, 6, 48, 40, 48), (16, 1, 16, 8, 4), (3, 3, 10, 7, 6), (20, 2, 128, 128, 64), (5, 1, 64, 96, 32),
    (24, 8, 256, 16, 128), (2, 1, 8, 200, 2)]


@pytest.mark.parametrize("dtype", [F32, BF16, F16])
@pytest.mark.parametrize("size", ATTN_SIZES)
@pytest.mark.parametrize("window,pool", [(1, 1), (13, 4), (20, 33), (64, 0), (9, 2)])
def test_attention_step_kernel(dtype, size, window, pool):
    n = 75
    at = Attention(dtype, *size[:4], window, pool, n, size[4])
    want = at.want()
    close(at.step([0, 1, 3, 40, 42, 75]), want, dtype, "portions")
    close(at.step([0, 30] + list(range(31, 76)), nsplit=4), want, dtype, "one by one")
    close(at.step(list(range(76)), slot=0), want, dtype, "one by one from the first token")
    close(at.step([0, 64, 65, 75], slot=1, first=9, nsplit=8), want, dtype, "first row 9")


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_blocks_rotation_norms_and_head_groups_show(dtype):
    at = Attention(dtype, 6, 3, 24, 16, 9, 4, 40, 16)
    want = at.want()
    for fault in ("heads_interleaved", "no_rotation", "other_pairs", "no_norm", "norm_after_rotation", "no_blocks", "block_sums"):
        assert (at.want((fault,)) - want).abs().max() > 4 * TOL[dtype] * want.abs().max(), fault
    for scale in (-1.0, 2.0):
        far = Attention(dtype, 2, 1, 8, 8, 20, 3, 60, 4, scale=scale)
        close(far.step([0, 30] + list(range(31, 61))), far.want(), dtype, "sharp scores", 2)
        if dtype != F32:
            close(far.prompt([60], [0]), far.want(), dtype, "prompt, sharp scores", 2)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("window,pool", [(16, 4), (100, 7), (128, 16), (129, 32), (61, 64), (5, 1), (130, 130), (33, 2)])
def test_edges_with_a_block_that_stands_out(dtype, window, pool):
    """The keys of block 2 stand out, its last token with values of its own.  They decide a query as long as the window holds
    them - the last of them alone in the end -, and then their mean does; decoding one by one, in portions and (16-bit) as a
    prompt."""
    first, last = 2 * pool, 3 * pool - 1
    edge = last + window                             # the first position that sees the block
    n = edge + pool + 9
    at = Attention(dtype, 6, 2, 48, 32, window, pool, n, 16, standout=range(first, last + 1))
    want = at.want()
    for fault, row in (("window_plus_one", edge), ("window_minus_one", edge - 1), ("block_early", edge - 1), ("block_late", edge),
                       ("partial_blocks", edge - 1), ("no_blocks", edge)):
        if pool > 1 or fault in ("block_late", "no_blocks"):                  # (a block of one token takes over at once)
            assert (at.want((fault,))[row] - want[row]).abs().max() > 3 * TOL[dtype] * want.abs().max(), fault
    runs = {"portions": at.step(sorted({0, 9, first + window, edge - 1, edge + 1, n})),
            "one by one": at.step([0, 10] + list(range(11, n + 1))), "portions of two": at.step(list(range(0, n, 2)) + [n]),
            "one by one, split": at.step([0, 10] + list(range(11, n + 1)), nsplit=8)}
    if dtype == BF16:
        runs["prompt"] = at.prompt([n], [0])
    for name, got in runs.items():
        close(got[edge - 1:edge + 1], want[edge - 1:edge + 1], dtype, f"{name} edge")
        close(got, want, dtype, name)


@pytest.mark.parametrize("dtype", [BF16, F16])
@pytest.mark.parametrize("size", [(4, 2, 32, 24, 16), (2, 2, 64, 64, 64), (6, 1, 128, 96, 32), (4, 4, 192, 128, 128), (3, 3, 72, 104, 8),
                                  (8, 4, 256, 8, 64)])
@pytest.mark.parametrize("window,pool", [(50, 3), (128, 16), (200, 1), (20, 64), (1000, 8)])
def test_prompt_kernel_on_packed_sequences(dtype, size, window, pool):
    """Sequences of different lengths behind one another, blocks counted from each one's own start, more than a tile of them;
    what the prompt filed serves the steps that follow."""
    lens = [130, 1, 357, 64, 5]
    at = Attention(dtype, *size[:4], window, pool, sum(lens) + 1, size[4], standout=() if size[2] == size[4] else (2, 140, 141, 260))
    assert at.spec.prefill_ok(dtype)
    got, row = at.prompt(lens, [0, 1, 2, 3, 4]), 0
    for n in lens:
        close(got[row:row + n], at.want(a=row, b=row + n), dtype, f"rows {row}..{row + n}")
        row += n
    n = lens[2]                                       # slot 2 goes on by one token behind its prompt
    idx = list(range(131, 131 + n)) + [sum(lens)]
    out = at.call(idx[-1:], [2], [n])
    for t in ("q", "k", "v"):
        setattr(at, t, getattr(at, t)[idx])
    close(out[0], at.want()[-1], dtype, "next token", 2)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_unequal_sequences_and_used_slots(dtype):
    """One new token each for sequences of different lengths in different slots, one of them at its very first token; then
    other sequences in the same slots, whose rows and blocks still hold the old ones."""
    at = Attention(dtype, 8, 2, 40, 16, 23, 4, 190, 24)
    for spans in ({3: (0, 60), 0: (60, 90), 1: (90, 91)}, {0: (91, 150), 1: (150, 180), 3: (180, 190)}):
        before = [(s, a, b - 1) for s, (a, b) in spans.items() if b - a > 1]
        got = at.call(sum((list(range(a, b)) for _, a, b in before), []), sum(([s] * (b - a) for s, a, b in before), []),
                      sum((list(range(b - a)) for _, a, b in before), []), [b - a for _, a, b in before])
        row = 0
        for s, a, b in before:
            close(got[row:row + b - a], at.want(a=a, b=b), dtype, f"slot {s}")
            row += b - a
        out = at.call([b - 1 for _, b in spans.values()], list(spans), [b - a - 1 for a, b in spans.values()])
        for i, (a, b) in enumerate(spans.values()):
            close(out[i], at.want(a=a, b=b)[-1], dtype, f"sequence {i}")


# ------------------------------------------------------------------------------------------------
# recurrences alone
# ------------------------------------------------------------------------------------------------
class Recurrence:
    """A recurrence behind its projections, on the kernels and on the oracle."""

    def run(self, idx, slots, pos, lens=None, chunked=None):
        """One call over the rows ``idx``; ``lens``: portions they make up, None: one token each."""
        w = self.width
        out = torch.empty(len(idx), (w + 7) // 8 * 8 + 8, dtype=self.dtype, device=CUDA)[:, 8:8 + w]
        return self.mix(self.spec, self.weights, padded(self.x[idx], self.dtype), self.low[idx].to(CUDA, F32), i32(slots),
                        i32(pos), self.cache, 0, out, None if lens is None else portions_of(lens), chunked=chunked)

    def step(self, cuts, slot=2, first=0, chunked=None):
        self.cache.set_first_rows([first if s == slot else 0 for s in range(4)])
        return torch.cat([self.run(list(range(a, b)), [slot] * (b - a), list(range(first + a, first + b)),
                                   None if b - a == 1 else [b - a], chunked) for a, b in zip(cuts, cuts[1:])])

    def state(self, slot):
        return self.cache.layers[0]._k[slot]


class SSD(Recurrence):
    def __init__(self, dtype, heads, vdim, state, groups, taps, parts, n, speed=0.0, seed=0):
        from ipex_llm_b200.ops import ssd as S
        from ipex_llm_b200.ops.kv_cache import DeltaStateShape, SlotCache
        self.S, self.mix, self.dtype = S, S.ssd_mix, dtype
        self.spec = s = S.SSDSpec(heads, vdim, state, groups, taps, parts)
        self.width = s.inner
        self.x = rnd(n, s.rows, seed=seed + 1, dtype=dtype)
        self.low = rnd(n, heads + 3, seed=seed + 2)              # (columns behind the step sizes belong to others)
        self.conv, self.conv_b = rnd(s.channels, taps, seed=seed + 3, dtype=dtype, gain=taps ** -0.5), rnd(s.channels, seed=seed + 4, gain=0.3)
        self.dt_bias, self.a_log = rnd(heads, seed=seed + 5) - 1.0, rnd(heads, seed=seed + 6) + speed
        self.skip, self.norm = 1 + rnd(heads, seed=seed + 7, gain=0.5), (1 + 0.2 * rnd(s.inner, seed=seed + 8)).to(dtype).double()
        self.refresh()
        self.cache = SlotCache()
        self.cache.allocate(4, n + 64, [DeltaStateShape(heads, state, vdim, taps, s.channels)], dtype, CUDA)

    def refresh(self):
        self.weights = self.S.SSDWeights(self.conv.to(CUDA, self.dtype), *(t.cuda() for t in (self.conv_b, self.dt_bias, self.a_log,
                                                                                             self.skip)),
                                         self.norm.to(CUDA, self.dtype), EPS)

    def want(self, a=0, b=None, faults=()):
        s, x = self.spec, self.x[a:b]
        n = len(x)
        xbc, z = x.split([s.channels, s.inner], 1)
        bias = 0 * self.conv_b if "no_conv_bias" in faults else self.conv_b
        u, B, C = O.silu(O.short_conv(xbc, self.conv, bias)).split([s.inner, s.groups * s.state, s.groups * s.state], 1)
        dt = torch.nn.functional.softplus(self.low[a:b, :s.heads] + self.dt_bias, threshold=1e9)
        u = u.to(self.dtype).double()                            # 16-bit models keep x in 16 bits
        y, state = O.ssd_rule(u.view(n, s.heads, s.vdim), B.view(n, s.groups, s.state), C.view(n, s.groups, s.state), dt,
                              self.a_log, self.skip, faults=faults)
        return O.gated_group_norm(y.flatten(1), z, self.norm, s.parts, EPS, faults), state


class General(Recurrence):
    def __init__(self, dtype, heads, dim, vdim, rank, n, bias=-1.0, rate=0.0, seed=0):
        from ipex_llm_b200.ops import general_delta as R
        from ipex_llm_b200.ops.kv_cache import DeltaStateShape, SlotCache
        self.R, self.mix, self.dtype = R, R.general_delta_mix, dtype
        self.spec = s = R.GeneralDeltaSpec(heads, dim, vdim, rank)
        self.width = heads * vdim
        self.x = rnd(n, s.rows, seed=seed + 1, dtype=dtype)
        self.low = rnd(n, rank + 2, seed=seed + 2)
        self.up = rnd(heads * dim, rank, seed=seed + 3, dtype=dtype, gain=1.5 * rank ** -0.5)
        self.bias, self.rate_bias = rnd(heads * dim, seed=seed + 4, gain=1.5) + bias, rnd(heads * dim, seed=seed + 5) + rate
        self.norm = (1 + 0.2 * rnd(heads * vdim, seed=seed + 6)).to(dtype).double()
        self.refresh()
        self.cache = SlotCache()
        self.cache.allocate(4, n + 64, [DeltaStateShape(heads, dim, vdim, 0, 0)], dtype, CUDA)

    def refresh(self):
        self.weights = self.R.GeneralDeltaWeights(self.up.to(CUDA, self.dtype), self.bias.cuda(), self.rate_bias.cuda(),
                                                  self.norm.to(CUDA, self.dtype), EPS)

    def want(self, a=0, b=None, faults=()):
        s, n = self.spec, len(self.x[a:b])
        H, D, V = s.heads, s.dim, s.vdim
        r, k, v, rate, g = self.x[a:b].split([H * D, H * D, H * V, H * D, H * V], 1)
        w = O.channel_decay(torch.tanh(self.low[a:b, :s.rank]) @ self.up.T + self.bias).view(n, H, D)
        if "one_decay_per_head" in faults:
            w = w.mean(-1, keepdim=True).expand_as(w)
        o, state = O.general_delta_rule(r.view(n, H, D), k.view(n, H, D), v.view(n, H, V), w,
                                        torch.sigmoid(rate + self.rate_bias).view(n, H, D), faults=faults)
        return O.rms(o, EPS).flatten(1) * self.norm * torch.sigmoid(g), state


SSD_SIZES = [  # heads, vdim, state, groups, taps, parts
    (4, 24, 16, 2, 4, 2), (6, 32, 32, 3, 3, 1), (2, 128, 128, 1, 4, 2), (6, 40, 24, 6, 2, 4), (4, 7, 10, 2, 1, 7), (1, 96, 200, 1, 5, 3),
    (2, 64, 256, 2, 4, 16), (4, 300, 48, 4, 4, 2), (8, 16, 8, 1, 7, 8), (2, 256, 64, 1, 4, 1)]
GENERAL_SIZES = [  # heads, dim, vdim, rank
    (4, 24, 24, 6), (3, 32, 32, 16), (2, 128, 128, 16), (6, 40, 40, 5), (2, 10, 10, 1), (1, 96, 96, 33), (2, 64, 64, 64), (2, 16, 300, 4),
    (4, 8, 16, 7), (5, 56, 72, 24), (1, 160, 48, 9), (1, 256, 256, 8)]


def build(kind, dtype, size, n, **kw):
    return (SSD if kind == "ssd" else General)(dtype, *size, n, **kw)


CASES = [("ssd", s) for s in SSD_SIZES] + [("general", s) for s in GENERAL_SIZES]


@pytest.mark.parametrize("dtype", [F32, BF16, F16])
@pytest.mark.parametrize("kind,size", CASES + [("ssd", (1, 24, 300, 1, 4, 1)), ("general", (1, 300, 24, 3))])
def test_token_by_token_and_in_portions(kind, dtype, size):
    n = 70
    d = build(kind, dtype, size, n)
    want, state = d.want()
    loose = 1.0 if dtype == F32 else 5.0
    for name, cuts, kw in (("one by one", list(range(n + 1)), {}), ("portions", [0, 1, 3, 5, 40, 41, 70], {"chunked": False}),
                           ("portions of two", list(range(0, 71, 2)), {"chunked": False}),
                           ("portions from row 9", [0, 2, 33, 70], {"chunked": False, "first": 9, "slot": 1})):
        close(d.step(cuts, **kw), want, dtype, name, 1.0 if dtype != F32 else 2.0)
        if kind == "general" or dtype == F32:
            close(d.state(kw.get("slot", 2)), state, F32, name + ", state", 2 * loose)
        else:                                                    # x is rounded on the way in
            close(d.state(kw.get("slot", 2)), state, dtype, name + ", state", 0.2)


@pytest.mark.parametrize("dtype", [BF16, F16])
@pytest.mark.parametrize("size", GENERAL_SIZES)
@pytest.mark.parametrize("bias,rate", [(-1.0, 0.0), (-8.0, 3.0), (8.0, -3.0), (0.0, 12.0)])
def test_general_delta_in_chunks(dtype, size, bias, rate):
    """Chunk borders everywhere, portions that go on from a state, channels that keep everything or decay as fast as the rule
    allows, rates up to one; the state agrees to 32-bit accuracy."""
    n = 150
    d = General(dtype, *size, n, bias=bias, rate=rate)
    if not d.spec.chunks_ok(dtype):
        assert d.spec.dim > 200
        return
    want, state = d.want()
    for cuts in ([0, n], [0, 33, 65, 129, 150], [0, 1, 2, 34, 66, 149, 150], [0, 96, 150]):
        close(d.step(cuts, chunked=True), want, dtype, f"cuts {cuts}")
        close(d.state(2), state, F32, f"state, cuts {cuts}", 10)
    close(d.step([0, 40, 150], slot=0, first=7, chunked=True), want, dtype, "first row 7")


@pytest.mark.parametrize("dtype", [BF16, F16])
@pytest.mark.parametrize("size", SSD_SIZES)
@pytest.mark.parametrize("speed", [-4.0, 0.0, 3.0, 9.0])
def test_ssd_in_chunks(dtype, size, speed):
    """Chunk borders everywhere, portions that go on from a state and from convolution inputs, decays from hundreds of tokens
    down to nothing at once."""
    n = 150
    d = SSD(dtype, *size, n, speed=speed)
    if speed == 9.0:                                     # heads that forget everything beside some that keep it
        d.a_log[::2] = -3.0
        d.refresh()
    assert d.spec.chunks_ok(dtype)
    want, state = d.want()
    for cuts in ([0, n], [0, 33, 65, 129, 150], [0, 1, 2, 34, 66, 149, 150], [0, 96, 150]):
        close(d.step(cuts, chunked=True), want, dtype, f"cuts {cuts}")
        close(d.state(2), state, dtype, f"state, cuts {cuts}", 0.2)
    close(d.step([0, 40, 150], slot=0, first=7, chunked=True), want, dtype, "first row 7")


@pytest.mark.parametrize("kind,size", [("ssd", (4, 24, 16, 2, 4, 2)), ("general", (4, 24, 24, 6))])
def test_chunks_in_several_passes(kind, size):
    """A prompt longer than the scratch runs in passes; sequences then start and end in the middle of a pass."""
    from ipex_llm_b200.native.lib import stream_lib
    d = build(kind, BF16, size, 300)
    mod = d.S if kind == "ssd" else d.R
    lens, old = [70, 1, 130, 99], mod.SCRATCH_BYTES
    if kind == "ssd":
        lib = stream_lib("ssd")
        per = 4 * (2 * int(lib.ipex_ssd_group_floats(16, 24)) + 4 * int(lib.ipex_ssd_head_floats(16, 24)))
    else:
        per = 4 * 4 * int(stream_lib("general_delta").ipex_general_scratch_floats(24, 24))
    try:
        for chunks in (1, 2, 3):
            mod.SCRATCH_BYTES = chunks * per
            got = d.run(list(range(300)), sum(([s] * n for s, n in zip((3, 0, 1, 2), lens)), []),
                        sum((list(range(n)) for n in lens), []), lens, True)
            at = 0
            for s, n in zip((3, 0, 1, 2), lens):
                want, state = d.want(at, at + n)
                close(got[at:at + n], want, BF16, f"{chunks} chunks a pass")
                close(d.state(s), state, BF16, "state", 0.2)
                at += n
    finally:
        mod.SCRATCH_BYTES = old


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("kind,size", [("ssd", (4, 40, 32, 2, 4, 4)), ("general", (4, 32, 40, 16))])
def test_unequal_recurrences_and_used_slots(kind, dtype, size):
    """Prompts of several lengths in one call, then one token each; then the slots go to other sequences without being
    cleared, among them one that starts with a single token."""
    d = build(kind, dtype, size, 240)
    loose = 2.0 if dtype == F32 else 1.0
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
            close(got[at:at + n], d.want(a, b)[0][:-2], dtype, f"prompts, round {rounds}", loose)
            at += n
        for back in (2, 1):
            got = d.run([b - back for _, b in spans.values()], list(spans), [b - a - back for a, b in spans.values()])
            for i, (a, b) in enumerate(spans.values()):
                close(got[i], d.want(a, b)[0][-back], dtype, f"decoding, round {rounds}", loose)
    got = [d.run([t], [3], [t]) for t in range(6)]
    close(torch.cat(got), d.want(0, 6)[0], dtype, "first token alone in a used slot", loose)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_general_delta_far_write_is_found_again(dtype):
    """A key far back of its own direction is read through channels that hardly forget, past hundreds of others; what makes
    the rule what it is shows."""
    n = 400
    d = General(dtype, 2, 16, 16, 4, n, bias=0.0)
    d.bias[12::16], d.rate_bias[12::16] = -30.0, -30.0      # one channel per head keeps what it holds
    d.low[:] *= 0.1
    d.refresh()
    d.x[:, 32 + 12:64:16] = 0.0                             # only token 5 writes there
    d.x[5, 32:64] = 0.0
    d.x[5, 32 + 12:64:16] = 4.0
    d.x[:, 96:128][:, 12::16] = 0.0
    d.x[n - 1, :32] = 0.0
    d.x[n - 1, 12:32:16] = 4.0
    want, _ = d.want()
    assert (want[n - 1] - d.want(6)[0][-1]).abs().max() > 0.1
    for fault in ("read_before_write", "no_removal", "removal_after_decay", "one_decay_per_head", "one_rate_per_head", "unit_write",
                  "no_unit_key"):
        got = d.want(faults=(fault,))[0]
        assert not torch.isfinite(got).all() or (want - got).abs().max() > 0.05, fault
    close(d.step([0, 300] + list(range(301, n + 1)), chunked=False), want, dtype, factor=5 if dtype == F32 else 1)
    if dtype == BF16:
        close(d.step([0, n], chunked=True), want, dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_ssd_far_write_is_found_again(dtype):
    n = 400
    d = SSD(dtype, 4, 16, 8, 2, 3, 2, n)
    d.a_log[:] = -9.0
    d.skip[:] = 0.0
    s = d.spec
    d.conv[:], d.conv_b[:] = 0.0, 0.0
    d.conv[:, -1] = 1.0
    B, C = slice(s.inner, s.inner + 16), slice(s.inner + 16, s.inner + 32)
    d.x[:, B][:, 3::8] = -30.0                              # silu of it is nothing: only token 5 writes row 3 ...
    d.x[5, B] = -30.0
    d.x[5, B][3::8] = 6.0
    d.x[n - 1, C] = -30.0                                   # ... and the last one reads it alone
    d.x[n - 1, C][3::8] = 3.0
    d.refresh()
    want, _ = d.want()
    assert (want[n - 1] - d.want(6)[0][-1]).abs().max() > 0.1
    for fault in ("groups_interleaved", "unscaled_input", "read_before_write", "gate_after_norm", "one_norm_group"):
        assert (want - d.want(faults=(fault,))[0]).abs().max() > 0.05, fault
    close(d.step([0, 300] + list(range(301, n + 1)), chunked=False), want, dtype, factor=5 if dtype == F32 else 1)
    if dtype == BF16:
        close(d.step([0, n], chunked=True), want, dtype)


def test_convolution_bias_taps_and_skip_show():
    d = SSD(F32, 4, 24, 16, 2, 4, 2, 40)
    want = d.want()[0]
    for fault in ("no_conv_bias", "no_skip"):
        assert (d.want(faults=(fault,))[0] - want).abs().max() > 0.1, fault
    keep = d.conv.clone()
    for tap in range(4):
        d.conv[:, tap] = 0.0
        assert (d.want()[0] - want).abs().max() > 0.1
        d.conv = keep.clone()


# ------------------------------------------------------------------------------------------------
# whole models
# ------------------------------------------------------------------------------------------------
def base(**kw):
    return {"architecture": "Gegorax", "norm": {"eps": 1e-5}} | kw


def cfg_a():
    return base(vocab=150, width=96, token_side={"dim": 24},
                layers=[O.parallel_layer(4, 2, 32, 24, 21, 5, 16, rheads=6, rvdim=16, state=24, groups=3, conv=4, norm_groups=2,
                                         mlp=O.dense(160)),
                        O.delta_layer(3, 32, mlp=O.moe(24, 6, 3, 0.9, 40, 1.4)),
                        O.delta_layer(4, 16, mlp=O.dense(72)),
                        O.parallel_layer(6, 3, 16, 40, 64, 16, 8, rheads=2, rvdim=40, state=40, groups=1, conv=3, norm_groups=8,
                                         mlp=O.moe(32, 8, 2, 1.2, None)),
                        O.delta_layer(2, 48, mlp=None), O.parallel_layer(2, 1, 64, 64, 7, 3, 64, rheads=4, rvdim=32, state=16,
                                                                         groups=4, conv=2, norm_groups=1, mlp=None)])


def cfg_odd():
    """Nothing a multiple of anything: the generic kernels."""
    return base(vocab=101, width=50, norm={"eps": 1e-3}, token_side={"dim": 5},
                layers=[O.delta_layer(3, 10, mlp=O.dense(33)),
                        O.parallel_layer(3, 1, 10, 9, 17, 7, 6, rheads=3, rvdim=7, state=9, groups=1, conv=5, norm_groups=7,
                                         mlp=O.moe(11, 5, 2, 0.6, 9, 2.0)),
                        O.delta_layer(1, 21, mlp=O.moe(9, 3, 3, 1.0, None))])


def cfg_one():
    """One head, one expert chosen, a window of one token and blocks of one."""
    return base(vocab=64, width=64, norm={"eps": 1e-6}, token_side={"dim": 1},
                layers=[O.parallel_layer(1, 1, 64, 64, 1, 1, 64, rheads=1, rvdim=64, state=64, groups=1, conv=1, norm_groups=1,
                                         mlp=O.moe(16, 4, 1, 0.5, 16, 0.5)),
                        O.delta_layer(1, 64, mlp=O.dense(128))])


def cfg_delta():
    """The generalized delta rule only, no embedding per layer."""
    return base(vocab=120, width=64, layers=[O.delta_layer(2, 32, mlp=O.dense(128)), O.delta_layer(4, 24, mlp=None),
                                             O.delta_layer(1, 128, mlp=O.moe(32, 4, 2, 1.0, 32))])


def cfg_parallel():
    """Layers of two sides only; windows of a tile, blocks longer than the window; no rotation in one of them."""
    return base(vocab=120, width=64, token_side={"dim": 32},
                layers=[O.parallel_layer(2, 2, 64, 64, 128, 16, 32, rheads=2, rvdim=64, state=64, groups=1, norm_groups=1,
                                         mlp=O.dense(128)),
                        O.parallel_layer(4, 1, 32, 16, 24, 40, 0, rheads=4, rvdim=32, state=16, groups=2, norm_groups=4,
                                         mlp=O.moe(32, 4, 2, 2.0, 64))])


CFGS = {"a": cfg_a, "odd": cfg_odd, "one": cfg_one, "delta": cfg_delta, "parallel": cfg_parallel}
_models, _want = {}, {}


def make(name, dtype):
    from ipex_llm_b200.models import gegorax
    from ipex_llm_b200.transformers.model import _attach_api
    key = (name, dtype)
    if key not in _models:
        cfg = CFGS[name]()
        w = O.random_weights(cfg, seed=len(name), rank=5 if name == "odd" else 16, spread=0.3)
        model = _attach_api(gegorax.build(cfg, w, dtype).to(CUDA))
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
def test_stream_after_every_layer(name, dtype):
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
    """Many blocks and graphs past the prompt, one token at a time."""
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
@pytest.mark.parametrize("name", ["a", "odd", "one", "delta"])
def test_greedy_generate(name):
    model, cfg, w = make(name, F32)
    prompts = [tokens(n, cfg["vocab"], n) for n in (23, 6, 14)]
    want = [O.greedy(w, cfg, p, 12) for p in prompts]
    for p, e in zip(prompts, want):
        out = model.generate(torch.tensor([p], device=CUDA), max_new_tokens=12, do_sample=False)
        assert out[0, len(p):].tolist() == e
        assert type(model._ipex_engine).__name__ == "ParallelBlockEngine"
    # left-padded batch: stays on the engine, rows keep their own positions
    S = max(map(len, prompts))
    ids = torch.tensor([[0] * (S - len(p)) + p for p in prompts], device=CUDA)
    mask = torch.tensor([[0] * (S - len(p)) + [1] * len(p) for p in prompts], device=CUDA)
    out = model.generate(ids, attention_mask=mask, max_new_tokens=12, do_sample=False)
    assert out[:, S:].tolist() == want
    # ... and the transformers loop over the module's forward gives the same
    out = model._hf_generate(ids, attention_mask=mask, max_new_tokens=12, do_sample=False, pad_token_id=0)
    assert out[:, S:].tolist() == want


def test_sampling_stays_on_the_engine():
    model, cfg, _ = make("a", F32)
    ids = torch.tensor([tokens(12, cfg["vocab"], 2)] * 3, device=CUDA)
    torch.manual_seed(0)
    out = model.generate(ids, max_new_tokens=9, do_sample=True, temperature=60.0, top_k=40, top_p=0.95)
    assert out.shape == (3, 21) and len({tuple(r) for r in out[:, 12:].tolist()}) > 1
    one = model.generate(ids, max_new_tokens=9, do_sample=True, top_k=1)
    assert torch.equal(one, model.generate(ids, max_new_tokens=9, do_sample=False))


def test_forward_logits_and_beam_search():
    model, cfg, w = make("a", F32)
    p = tokens(19, cfg["vocab"], 4)
    ids = torch.tensor([p, p[::-1]], device=CUDA)
    out = model(ids)
    for b in range(2):
        agree(out.logits[b], O.forward(w, cfg, ids[b].tolist()), F32)
    more = model(torch.tensor([[5], [6]], device=CUDA), past_key_values=out.past_key_values)
    agree(more.logits[1, -1:], O.forward(w, cfg, p[::-1] + [6])[-1:], F32)
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
    """Packed projections (the fused ones with hidden units included) beside dense experts and token sides: logits close to
    those of the dense weights."""
    from ipex_llm_b200.models import gegorax
    from ipex_llm_b200.transformers import AutoModelForCausalLM
    cfg = base(vocab=128, width=128, token_side={"dim": 16},
               layers=[O.delta_layer(4, 32, mlp=O.dense(256)),
                       O.parallel_layer(4, 2, 32, 32, 30, 4, 32, rheads=4, rvdim=32, state=32, groups=2, mlp=O.dense(128)),
                       O.delta_layer(2, 64, mlp=O.moe(64, 4, 2, 1.5, 64))])
    w = O.random_weights(cfg, sharp=1.0)
    write_checkpoint(str(tmp_path), cfg, w)
    m8 = AutoModelForCausalLM.from_pretrained(str(tmp_path), load_in_low_bit="sym_int8").to(CUDA)
    assert type(m8.model.layers[0].in_proj).__name__ == "LowBitLinear" and type(m8.model.layers[0].out_proj).__name__ == "LowBitLinear"
    ref = gegorax.build(cfg, w, BF16).to(CUDA)
    toks = torch.tensor([tokens(40, cfg["vocab"], 2)], device=CUDA)
    a, b = m8(toks).logits, ref(toks).logits
    assert torch.nn.functional.cosine_similarity(a[0], b[0], dim=-1).median() > 0.99
    a = m8(toks[:, :3]).logits                                   # few rows
    assert torch.nn.functional.cosine_similarity(a[0], b[0, :3], dim=-1).median() > 0.99
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
    model = AutoModelForCausalLM.from_pretrained(str(tmp_path), load_in_low_bit="bf16", torch_dtype=BF16, device=CUDA)
    out = model.generate(torch.tensor([[3, 9, 4, 77]], device=CUDA), max_new_tokens=6, do_sample=False)
    assert got == out[0, 4:].tolist() and len(got) == 6


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay(tmp_path, dtype):
    """The replay program on a checkpoint: a batch that starts together and thins out, then another request."""
    import subprocess
    import sys
    import numpy as np
    cfg = cfg_a()
    w = O.random_weights(cfg, seed=4, spread=0.3)
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
