"""Latent-attention decoders on the GPU: every kernel against the float64 oracle (``tests/dobetar_oracle.py``), then the
engine with whole prompts, portions, ragged batches, slot reuse, long decoding and generation."""
import pytest
import torch

import dobetar_oracle as O

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
    err = (got - want).abs().max().item() / max(want.abs().max().item(), 1e-3)
    assert err < TOL[dtype] * factor, f"{what}: {err}"


def gen(seed):
    return torch.Generator().manual_seed(seed)


def rnd(*shape, seed=0, dtype=F32, gain=1.0):
    """Random values that the dtype can hold, as float64."""
    return (torch.randn(*shape, generator=gen(seed)) * gain).to(dtype).double()


# ------------------------------------------------------------------------------------------------
# row products, GEMMs, stream
# ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF16, F16])
@pytest.mark.parametrize("M,N,K", [(1, 97, 136), (3, 40, 60), (8, 2500, 520), (5, 9600, 256), (2, 33, 7)])
def test_gemv_rows(dtype, M, N, K):
    from ipex_llm_b200.ops import latent as L
    w, x = rnd(N, K, seed=1, dtype=dtype, gain=K ** -0.5), rnd(M, K, seed=2)
    nw = 1 + 0.2 * rnd(K, seed=3, dtype=dtype)
    nw = nw.to(dtype).double()
    W, X, NW = w.to("cuda", dtype), x.to("cuda", F32), nw.to("cuda", dtype)
    ref = O.rms_norm(x, nw, 1e-5) @ w.T
    out = torch.empty(M, N, dtype=dtype, device="cuda")
    close(L.gemv_rows(W, X, out, L.OUT_ACT, norm=NW, eps=1e-5), ref, dtype, "norm")
    close(L.gemv_rows(W, X, out, L.OUT_ACT, norm=NW, eps=1e-5, act=L.ACT_RELU2), torch.relu(ref) ** 2, dtype, "relu2", 2)
    lg = torch.empty(M, N, dtype=F32, device="cuda")
    close(L.gemv_rows(W, X, lg, L.OUT_F32, norm=NW, eps=1e-5, softcap=1.5), O.softcap(ref, 1.5), dtype, "softcap")
    a = rnd(M, K, seed=4, dtype=dtype)
    res = rnd(M, N, seed=5)
    R = res.to("cuda", F32)
    L.gemv_rows(W, a.to("cuda", dtype), R, L.OUT_ADD)
    close(R, res + a @ w.T, F32, "stream", 1.0 if dtype == F32 else 5.0)       # the sum itself is never rounded to 16 bits


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("M,N,K", [(9, 40, 72), (33, 200, 64), (70, 129, 136), (300, 257, 520), (12, 30, 50)])
def test_gemm_modes(dtype, M, N, K):
    from ipex_llm_b200.ops import latent as L
    w, x = rnd(N, K, seed=1, dtype=dtype, gain=K ** -0.5), rnd(M, K, seed=2, dtype=dtype)
    W, X = w.to("cuda", dtype), x.to("cuda", dtype)
    ref = x @ w.T
    wide = torch.full((M, N + 8), 7.0, dtype=dtype, device="cuda")
    close(L.gemm(X, W, wide[:, :N], L.OUT_ACT), ref, dtype)
    assert bool((wide[:, N:] == 7.0).all())
    out = torch.empty(M, N, dtype=dtype, device="cuda")
    close(L.gemm(X, W, out, L.OUT_ACT, L.ACT_RELU2), torch.relu(ref) ** 2, dtype, "relu2", 2)
    f = torch.empty(M, N, dtype=F32, device="cuda")
    close(L.gemm(X, W, f, L.OUT_F32), ref, F32, "fp32", 5)
    res = rnd(M, N, seed=5)
    R = res.to("cuda", F32)
    close(L.gemm(X, W, R, L.OUT_ADD), res + ref, F32, "stream", 5)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("bigram", [True, False])
def test_embedding_takes_the_previous_token_from_the_batch_or_the_history(dtype, bigram):
    from ipex_llm_b200.ops import latent as L
    from ipex_llm_b200.ops.kv_cache import LatentCache
    V, W, nb = 50, 36, 23
    w = {"embed": rnd(V, W, seed=1, dtype=dtype), "bigram": rnd(nb + 1, W, seed=2, dtype=dtype)}
    cfg = {"embedding": {"scale": 3.0, "bigram": {"buckets": nb, "mul_prev": 1000003, "mul_cur": 70001} if bigram
                         else None}}
    c = LatentCache()
    c.allocate(3, 16, [8], dtype, "cuda")
    c.set_first_rows([0, 3, 0])
    table = w["embed"].to("cuda", dtype)
    big = w["bigram"].to("cuda", dtype) if bigram else None
    seqs = {2: [4, 49, 7, 7, 0], 1: [9, 9, 30]}
    first = {2: 0, 1: 3}
    want = {s: O.embed(w, cfg, t) for s, t in seqs.items()}
    got = {2: [], 1: []}
    # a portion of each, then the rest: tokens of slot 2 and 1 in one launch
    for part in ({2: (0, 3), 1: (0, 1)}, {1: (1, 3), 2: (3, 4)}, {2: (4, 5)}):
        tok, slot, pos = [], [], []
        for s, (a, b) in part.items():
            tok += seqs[s][a:b]
            slot += [s] * (b - a)
            pos += [first[s] + i for i in range(a, b)]
        x = L.embed_stream(torch.tensor(tok, device="cuda"), torch.tensor(slot, dtype=torch.int32, device="cuda"),
                           torch.tensor(pos, dtype=torch.int32, device="cuda"), c, table, 3.0, big, nb, 1000003, 70001)
        at = 0
        for s, (a, b) in part.items():
            got[s].append(x[at:at + b - a])
            at += b - a
    for s in seqs:
        close(torch.cat(got[s]), want[s], F32)
    assert c.history[2, :5].tolist() == seqs[2] and c.history[1, 3:6].tolist() == seqs[1]


def test_norm_stream_rows_and_softcap():
    from ipex_llm_b200.ops import latent as L
    for K in (64, 75):
        x, w = rnd(6, K, seed=1), rnd(K, seed=2, dtype=BF16)
        X, Wb = x.to("cuda", F32), w.to("cuda", BF16)
        close(L.norm_stream(X, Wb, 1e-3), O.rms_norm(x, w, 1e-3), BF16)
        rows = torch.tensor([4, 0], dtype=torch.int32, device="cuda")
        close(L.norm_stream(X, Wb, 1e-3, rows=rows), O.rms_norm(x[[4, 0]], w, 1e-3), BF16)
        close(L.norm_stream(X, w.to("cuda", F32), 1e-3), O.rms_norm(x, w, 1e-3), F32)
        close(L.softcap_(X.clone() * 9, 4.0), O.softcap(x * 9, 4.0), F32)


# ------------------------------------------------------------------------------------------------
# mixture of experts
# ------------------------------------------------------------------------------------------------
def bank_and_weights(dtype, W, I, E, top, limit, seed=0):
    from ipex_llm_b200.models.dobetar import interleave_gate_up
    from ipex_llm_b200.ops import latent as L
    w = {"router": rnd(E, W, seed=seed, dtype=dtype, gain=2 * W ** -0.5)}
    for e in range(E):
        w[f"e{e}.gate"] = rnd(I, W, seed=seed + 10 + e, dtype=dtype, gain=3 * W ** -0.5)
        w[f"e{e}.up"] = rnd(I, W, seed=seed + 50 + e, dtype=dtype, gain=3 * W ** -0.5)
        w[f"e{e}.down"] = rnd(W, I, seed=seed + 90 + e, dtype=dtype, gain=I ** -0.5)
    gu = torch.stack([interleave_gate_up(w[f"e{e}.gate"], w[f"e{e}.up"]) for e in range(E)])
    dn = torch.stack([w[f"e{e}.down"] for e in range(E)])
    bank = L.ExpertBank(w["router"].to("cuda", dtype), gu.to("cuda", dtype), dn.to("cuda", dtype), top, limit, 1.702,
                        I % 16 == 0)
    return bank, w, {"router": {"top": top}, "expert": {"limit": limit}}


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("W,I,E,top", [(64, 32, 6, 1), (72, 24, 5, 3), (50, 10, 4, 4), (128, 48, 40, 2)])
def test_experts_both_paths(dtype, W, I, E, top):
    """Experts read scaled inputs (scaling outputs instead would show); the clamps bind: the limit is below the typical
    gate."""
    from ipex_llm_b200.ops import latent as L
    bank, w, p = bank_and_weights(dtype, W, I, E, top, limit=0.8)
    nw = (1 + 0.2 * rnd(W, seed=7)).to(dtype).double()
    for T in (1, 6, 41, 150):
        x = rnd(T, W, seed=T)
        h = O.rms_norm(x, nw, 1e-6)
        if dtype == BF16:
            # a rounded h may flip a near tie: keep rows whose choice is clear
            s = torch.sort(torch.sigmoid(h @ w["router"].T), dim=-1, descending=True).values
            clear = torch.ones(T, dtype=torch.bool) if top == E else (s[:, top - 1] - s[:, top]) > 0.02
        else:
            clear = torch.ones(T, dtype=torch.bool)
        want = x + O.moe_mlp(w, "", p, h)
        wrong = x + O.moe_mlp(w, "", p, h, faults=("weight_on_output",))
        X = x.to("cuda", F32)
        if bank.rows_ok(T):
            L.moe_rows(bank, X, nw.to("cuda", dtype), 1e-6)
        else:
            L.moe_grouped(bank, X, L.norm_stream(X, nw.to("cuda", dtype), 1e-6))
        if clear.any():
            close(X.cpu()[clear], want[clear], dtype, f"T={T}")
        if dtype == F32:
            assert (want - wrong).abs().max() > 3 * TOL[dtype] * want.abs().max()


def test_experts_that_get_no_token_or_all_of_them():
    from ipex_llm_b200.ops import latent as L
    bank, w, p = bank_and_weights(F32, 64, 32, 8, 1, limit=2.0)
    x = rnd(70, 64, seed=3)
    h = O.rms_norm(x, torch.ones(64).double(), 1e-6)
    # a router that sends every row to expert 5: scores follow one strong common direction
    d = rnd(64, seed=9)
    h = h * 0.05 + d
    bank.router.copy_((w["router"] * 0.01).to("cuda", F32))
    bank.router[5] = (d / d.norm() * 0.5).to("cuda", F32)
    w["router"] = bank.router.double().cpu()
    X = x.to("cuda", F32)
    L.moe_grouped(bank, X, h.to("cuda", F32))
    assert bool((O.route(w, "", h, 1)[1] == 5).all())
    close(X, x + O.moe_mlp(w, "", p, h), F32, factor=3)


@pytest.mark.parametrize("E,k", [(3, 1), (12, 12), (70, 5)])
def test_sigmoid_topk(E, k):
    from ipex_llm_b200.ops import latent as L
    z = torch.randn(33, E, generator=gen(E)).cuda()
    w, idx = L.sigmoid_topk(z, k)
    rw, ri = torch.topk(torch.sigmoid(z), k, dim=-1)
    assert torch.equal(idx, ri) and torch.allclose(w, rw, atol=1e-6)


# ------------------------------------------------------------------------------------------------
# latent attention alone
# ------------------------------------------------------------------------------------------------
class Mixer:
    """One latent-attention layer between its projections, on the kernels and on the oracle, with a stand-out key."""

    def __init__(self, dtype, heads, dim, rd, vd, R, window, n, base=1000.0, standout=(), scale=None, pairs=None, seed=0):
        from ipex_llm_b200.ops import latent as L
        from ipex_llm_b200.ops.kv_cache import LatentCache
        self.dtype, self.n = dtype, n
        scale = (dim + rd) ** -0.5 if scale is None else scale
        pairs = rd // 2 if pairs is None else pairs
        self.m = {"heads": heads, "dim": dim, "rot_dim": rd, "vdim": vd, "kv_rank": R, "mask": {"size": window},
                  "rot": {"base": base, "dims": 2 * pairs}, "scale": scale}
        self.uk = rnd(heads * dim, R, seed=seed + 1, dtype=dtype, gain=R ** -0.5)
        self.uv = rnd(heads * vd, R, seed=seed + 2, dtype=dtype, gain=R ** -0.5)
        self.nw = (1 + 0.2 * rnd(R, seed=seed + 3)).to(dtype).double()
        q = rnd(n, heads, dim + rd, seed=seed + 4)
        kv = rnd(n, R + rd, seed=seed + 5)
        if len(standout):
            # every query shares a direction per head, and the stand-out rows' latents point along it for all heads
            d = rnd(heads, dim, seed=seed + 6)
            q[:, :, :dim] = 0.4 * q[:, :, :dim] + 1.8 * d
            pull = torch.einsum("hd,hdr->r", d, self.uk.view(heads, dim, R))
            for i, p in enumerate(standout):
                kv[p, :R] = 0.4 * kv[p, :R] + pull / pull.std() * (2.0 + i)
        self.q, self.kv = q.to(dtype).double(), kv.to(dtype).double()
        self.spec = L.LatentSpec(heads, dim, rd, vd, R, scale, window or 0, pairs, 1e-6)
        self.cos, self.sin = L.rotary_table(n + 64, base, pairs, "cuda")
        self.L, self.cache = L, LatentCache()
        self.cache.allocate(4, n + 64, [self.spec.row(dtype)], dtype, "cuda")

    def want(self, faults=()):
        return O.latent_mix(self.q, self.kv, self.nw, self.uk, self.uv, self.m, 1e-6, faults).flatten(1)

    def qkv(self, a, b):
        N = self.q[0].numel() + self.kv.shape[1]
        t = torch.zeros(b - a, (N + 7) // 8 * 8, dtype=self.dtype, device="cuda")
        t[:, :N] = torch.cat([self.q[a:b].flatten(1), self.kv[a:b]], 1).to(self.dtype)
        return t[:, :N]

    def args(self):
        return [t.to("cuda", self.dtype) for t in (self.uk, self.uv, self.nw)] + [self.cos, self.sin]

    def step(self, cuts, slot=2, first=0, generic=False, visible=None):
        """Portions [cuts[i], cuts[i + 1]) through the absorbed kernels."""
        self.cache.set_first_rows([first if s == slot else 0 for s in range(4)])
        outs = []
        for a, b in zip(cuts, cuts[1:]):
            out = torch.empty(b - a, self.spec.heads * self.spec.v_dim, dtype=self.dtype, device="cuda")
            sl = torch.full((b - a,), slot, dtype=torch.int32, device="cuda")
            pos = torch.arange(first + a, first + b, dtype=torch.int32, device="cuda")
            self.L.latent_step(self.spec, self.qkv(a, b), *self.args(), sl, pos, self.cache, 0, out,
                               visible or (self.spec.window or b), generic=generic)
            outs.append(out)
        return torch.cat(outs)

    def prompt(self, lens, slots):
        """Sequences cut out of the rows 0.., packed; every one restarts at position 0."""
        T = sum(lens)
        self.cache.set_first_rows([0] * 4)
        row, ln, sl, pos, at = [], [], [], [], 0
        for n, s in zip(lens, slots):
            row.append(at)
            ln.append(n)
            sl += [s] * n
            pos += list(range(n))
            at += n

        def i32(v):
            return torch.tensor(v, dtype=torch.int32, device="cuda")
        out = torch.empty(T, self.spec.heads * self.spec.v_dim, dtype=self.dtype, device="cuda")
        return self.L.latent_prompt(self.spec, self.qkv(0, T), *self.args(), i32(sl), i32(pos), i32(row), i32(ln),
                                    max(lens), self.cache, 0, out)


SIZES = [  # heads, dim, rd, vd, R
    (4, 32, 16, 24, 64), (16, 48, 8, 40, 96), (3, 20, 6, 12, 36), (20, 128, 64, 128, 512), (1, 8, 2, 8, 8),
    (33, 64, 32, 64, 256)]


@pytest.mark.parametrize("dtype", [F32, BF16, F16])
@pytest.mark.parametrize("size", SIZES)
@pytest.mark.parametrize("window", [None, 1, 37])
def test_latent_step_kernels(dtype, size, window):
    n = 75
    mx = Mixer(dtype, *size, window, n)
    want = mx.want()
    close(mx.step([0, 1, 2, 40, 42, 75]), want, dtype, "portions")
    close(mx.step(list(range(0, 75, 25)) + [75], generic=True), want, dtype, "generic")
    close(mx.step([0, 64, 75], slot=1, first=9), want, dtype, "first row 9")


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("window", [16, 100, 129])
def test_window_edges_with_a_key_that_stands_out(dtype, window):
    """The stand-out key at p decides every query that sees it, and none past p + window - 1; decoding one by one, in
    portions and (16-bit) as a prompt."""
    p, n = 13, 13 + window + 6
    mx = Mixer(dtype, 6, 48, 24, 32, 80, window, n, standout=(p,))
    want = mx.want()
    i, o = p + window - 1, p + window
    for fault, at in (("window_plus_one", o), ("window_minus_one", i)):
        assert (mx.want((fault,))[at] - want[at]).abs().max() > 8 * TOL[dtype] * want.abs().max()
    runs = {"portions": mx.step([0, 30, n]), "one by one": mx.step([0, 10] + list(range(11, n + 1))),
            "generic": mx.step([0, n], generic=True)}
    if dtype == BF16:
        runs["prompt"] = mx.prompt([n], [0])
    for name, got in runs.items():
        close(got[[i, o]], want[[i, o]], dtype, f"{name} edge")
        close(got, want, dtype, name)


@pytest.mark.parametrize("dtype", [BF16, F16])
@pytest.mark.parametrize("size", [(4, 32, 16, 24, 64), (2, 64, 64, 64, 128), (3, 128, 64, 128, 96), (2, 192, 64, 128, 64),
                                  (2, 72, 8, 104, 40), (2, 64, 0, 128, 64)])
@pytest.mark.parametrize("window", [None, 50, 128, 200])
def test_prompt_kernel_on_packed_sequences(dtype, size, window):
    """Sequences of different lengths behind one another (tiles that start inside a sequence's 8-token boundary, lengths
    around the 128-query tile, one single token), keys far away that stand out."""
    lens = [130, 1, 257, 64, 5]
    mx = Mixer(dtype, *size, window, sum(lens), standout=(2, 140, 141, 260))
    assert mx.spec.prefill_ok(dtype)
    got = mx.prompt(lens, [0, 1, 2, 3, 0])
    at = 0
    q, kv = mx.q, mx.kv
    for n in lens:
        mx.q, mx.kv = q[at:at + n], kv[at:at + n]
        close(got[at:at + n], mx.want(), dtype, f"rows {at}..{at + n}")
        at += n


def test_prompt_kernel_negative_scale_and_partial_rotation():
    mx = Mixer(BF16, 2, 32, 32, 32, 64, 70, 150, scale=-0.2, pairs=4)
    close(mx.prompt([150], [0]), mx.want(), BF16)
    close(mx.step([0, 150]), mx.want(), BF16)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_far_key_among_many_and_split_counts(dtype):
    """Without a window one early key must be found among a thousand, however the visible keys are split."""
    n = 1100
    mx = Mixer(dtype, 4, 32, 16, 24, 64, None, n, standout=(3,))
    want = mx.want()
    mx.step([0, 1000])
    for visible in (1, 64, 700, 1100, 5000):
        close(mx.step([1000, 1003, 1100], visible=visible), want[1000:], dtype, f"visible={visible}")


# ------------------------------------------------------------------------------------------------
# whole models
# ------------------------------------------------------------------------------------------------
def cfg_a():
    return {"architecture": "Dobetar", "vocab": 150, "width": 96,
            "embedding": {"scale": 1.5, "bigram": {"buckets": 61, "mul_prev": 31, "mul_cur": 17}},
            "layers": [O.latent_layer(4, 32, 16, 24, 64, window=20, mlp=O.dense(160)),
                       O.latent_layer(6, 24, 8, 32, 48, window=33, base=300.0, mlp=O.moe(32, 6, 2, 0.9)),
                       O.latent_layer(4, 32, 16, 24, 64, window=7, mlp=O.moe(48, 5, 1))],
            "logit_softcap": 9.0, "norm": {"eps": 1e-5}}


def cfg_odd():
    """Nothing a multiple of anything: the generic kernels; a layer without feed-forward, top = all experts."""
    return {"architecture": "Dobetar", "vocab": 101, "width": 50,
            "embedding": {"scale": 0.7, "bigram": {"buckets": 7, "mul_prev": 1, "mul_cur": 1}},
            "layers": [O.latent_layer(3, 10, 6, 9, 21, window=4, base=50.0, mlp=O.moe(11, 3, 3, 0.5)),
                       O.latent_layer(1, 13, 2, 5, 17, window=1, mlp=None),
                       O.latent_layer(2, 10, 6, 9, 21, window=90, mlp=O.dense(33))],
            "logit_softcap": 30.0, "norm": {"eps": 1e-3}}


def cfg_plain():
    """No bigram, no soft-cap, one expert of one, window of 64 at a tile edge."""
    return {"architecture": "Dobetar", "vocab": 120, "width": 64, "embedding": {"scale": 1.0},
            "layers": [O.latent_layer(2, 64, 32, 64, 32, window=64, mlp=O.moe(64, 1, 1, 3.0)),
                       O.latent_layer(2, 64, 32, 64, 32, window=64, mlp=O.dense(64))],
            "logit_softcap": None, "norm": {"eps": 1e-6}}


CFGS = {"a": cfg_a, "odd": cfg_odd, "plain": cfg_plain}
_models = {}


def make(name, dtype):
    from ipex_llm_b200.models import dobetar
    from ipex_llm_b200.transformers.model import _attach_api
    key = (name, dtype)
    if key not in _models:
        cfg = CFGS[name]()
        w = O.random_weights(cfg, seed=len(name))
        model = _attach_api(dobetar.build(cfg, w, dtype).to("cuda"))
        _models[key] = (model, cfg, {k: v.double() for k, v in w.items()})
    return _models[key]


def tokens(n, V, seed):
    return torch.randint(0, V, (n,), generator=gen(seed)).tolist()


_want = {}


def oracle(name, dtype, toks):
    key = (name, tuple(toks))
    if key not in _want:
        _, cfg, w = make(name, dtype)
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
    want = oracle(name, F32, toks)
    if name != "plain" and dtype == BF16:
        # the oracle's routing without near ties is checked per mechanism; here the median row must agree
        def cmp(got, what):
            e = (got.double().cpu() - want).abs().amax(-1) / want.abs().max()
            assert e.median() < TOL[dtype] * 2 and e.quantile(0.9) < TOL[dtype] * 8, (what, e.median(), e.max())
    else:
        def cmp(got, what):
            close(got, want, dtype, what, MODEL_TOL[dtype])
    n = len(toks)
    for cuts in ([0, n], [0, 75, n], list(range(0, n, 13)) + [n], list(range(0, n, 2)) + [n], [0, 1, 9, 20, 148, n]):
        eng = engine(model)
        s = eng.cache.acquire()
        got = [eng.step_rows([(s, toks[a:b], list(range(b - a)))]) for a, b in zip(cuts, cuts[1:])]
        cmp(torch.cat(got), f"cuts {cuts[:4]}")
    for graph in (True, False):
        eng = engine(model)
        s = eng.cache.acquire()
        got = [eng.step_rows([(s, toks[:3], [0, 1, 2])])]
        got += [eng.step_rows([(s, [t], [0])], use_graph=graph) for t in toks[3:]]
        cmp(torch.cat(got), f"token by token, graph={graph}")


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_ragged_batches_against_each_alone(dtype):
    """Unequal prompts in one batch, decoded together while the shorter ones leave; slots handed to new sequences."""
    model, cfg, _ = make("plain", dtype)
    V = cfg["vocab"]
    seqs = [tokens(n, V, 20 + n) for n in (1, 9, 130, 70)]
    tails = [3, 12, 5, 9]
    want = [oracle("plain", F32, s) for s in seqs]
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
            got[i].append(lg[j:j + 1])
            pos[i] += 1
            if pos[i] == len(seqs[i]):
                eng.cache.release(slots[i])
    eng.cache.release(slots[0])                      # one token: it was finished after the first step
    for i in range(4):
        close(torch.cat(got[i]), want[i], dtype, f"sequence {i}", MODEL_TOL[dtype])
    # all slots are free again: other sequences, other lengths, in another order
    again = [seqs[2], seqs[1], seqs[3], seqs[2][:40]]
    slots = [eng.cache.acquire() for _ in again]
    lg = eng.step_rows([(sl, s, list(range(len(s)))) for sl, s in zip(slots, again)])
    close(lg, torch.cat([want[2], want[1], want[3], want[2][:40]]), dtype, "reused slots", MODEL_TOL[dtype])


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_mixed_portions_in_one_batch(dtype):
    """A prompt, a continued portion and a decoded token in the same step."""
    model, cfg, _ = make("plain", dtype)
    a, b, c = (tokens(n, cfg["vocab"], 50 + n) for n in (40, 90, 33))
    wa, wb, wc = (oracle("plain", F32, t) for t in (a, b, c))
    eng = engine(model)
    sa, sb, sc = (eng.cache.acquire() for _ in range(3))
    eng.step_rows([(sa, a[:39], []), (sb, b[:30], [])])
    lg = eng.step_rows([(sb, b[30:], list(range(60))), (sa, a[39:], [0]), (sc, c, list(range(33)))])
    close(lg, torch.cat([wb[30:], wa[39:], wc]), dtype, factor=MODEL_TOL[dtype])


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_many_sequences_decode_through_the_gemms(dtype):
    """More rows than the row products take: GEMMs, grouped experts and the batched attention in the decode graph."""
    model, cfg, _ = make("plain", dtype)
    seqs = [tokens(20 + 3 * i, cfg["vocab"], 80 + i) for i in range(12)]
    want = [oracle("plain", F32, s) for s in seqs]
    eng = engine(model, 12)
    slots = [eng.cache.acquire() for _ in seqs]
    eng.step_rows([(sl, s[:-4], []) for sl, s in zip(slots, seqs)])
    for k in range(4, 0, -1):
        lg = eng.step_rows([(sl, [s[-k]], [0]) for sl, s in zip(slots, seqs)])
        close(lg, torch.stack([w[-k] for w in want]), dtype, f"{k} from the end", MODEL_TOL[dtype])


def test_long_decoding_in_32_bit():
    """Several windows and split sizes past the prompt, one token at a time."""
    model, cfg, _ = make("a", F32)
    toks = tokens(330, cfg["vocab"], 3)
    want = oracle("a", F32, toks)
    eng = engine(model)
    s = eng.cache.acquire()
    got = [eng.step_rows([(s, toks[:11], [10])])]
    got += [eng.step_rows([(s, [t], [0])]).clone() for t in toks[11:]]
    close(torch.cat(got), want[10:], F32, factor=MODEL_TOL[F32])


# ------------------------------------------------------------------------------------------------
# the framework's entry points
# ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", ["a", "odd"])
def test_greedy_generate(name):
    model, cfg, w = make(name, F32)
    prompts = [tokens(n, cfg["vocab"], n) for n in (23, 6, 14)]
    want = [O.greedy(w, cfg, p, 12) for p in prompts]
    for p, e in zip(prompts, want):
        out = model.generate(torch.tensor([p], device="cuda"), max_new_tokens=12, do_sample=False)
        assert out[0, len(p):].tolist() == e
        assert type(model._ipex_engine).__name__ == "LatentEngine"
    # left-padded batch: stays on the engine, rows keep their own positions
    S = max(map(len, prompts))
    ids = torch.tensor([[0] * (S - len(p)) + p for p in prompts], device="cuda")
    mask = torch.tensor([[0] * (S - len(p)) + [1] * len(p) for p in prompts], device="cuda")
    out = model.generate(ids, attention_mask=mask, max_new_tokens=12, do_sample=False)
    assert out[:, S:].tolist() == want
    # ... and the transformers loop over the module's forward gives the same
    out = model._hf_generate(ids, attention_mask=mask, max_new_tokens=12, do_sample=False, pad_token_id=0)
    assert out[:, S:].tolist() == want


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
    lp = 0.0
    full = torch.log_softmax(O.forward(w, cfg, beams[0].tolist()), -1)
    for i in range(5):
        lp += full[18 + i, beams[0, 19 + i]].item()
    g = O.greedy(w, cfg, p, 5)
    fg = torch.log_softmax(O.forward(w, cfg, p + g), -1)
    assert lp >= sum(fg[18 + i, t].item() for i, t in enumerate(g)) - 1e-6      # never worse than greedy


def test_prompt_lookup_and_speculative_decoding():
    """Drafted tokens are verified in one call and rejected ones cropped from the cache: greedy output is unchanged."""
    from ipex_llm_b200.models import dobetar
    from ipex_llm_b200.transformers.model import _attach_api
    from ipex_llm_b200.transformers.speculative import attach_draft_model
    model, cfg, w = make("a", F32)
    p = tokens(9, cfg["vocab"], 6)
    p = p + p + p[:4]
    want = O.greedy(w, cfg, p, 14)
    ids = torch.tensor([p], device="cuda")
    assert model.generate(ids, max_new_tokens=14, lookahead=3)[0, len(p):].tolist() == want
    src = {k: v.float() for k, v in w.items()}
    other = dict(src, head=src["head"] + 0.04 * torch.randn(src["head"].shape, generator=gen(1)))     # right now and then
    target, draft = (_attach_api(dobetar.build(cfg, x, F32).to("cuda")) for x in (src, other))
    attach_draft_model(target, draft)
    assert target.generate(ids, max_new_tokens=14, do_sample=False)[0, len(p):].tolist() == want
    assert sum(target.draft_num) > sum(target.accept_num) > 0
    half = dobetar.build(cfg, src, BF16).to("cuda")
    with pytest.raises(TypeError):
        half(ids[:, :1], past_key_values=target(ids).past_key_values)


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


def test_low_bit_projections_run():
    """Packed projections beside dense experts: logits close to those of the dequantized weights' size of error."""
    from ipex_llm_b200.transformers import AutoModelForCausalLM
    from ipex_llm_b200.models import dobetar
    cfg = cfg_plain()
    cfg["width"] = 128
    cfg["layers"][1]["mlp"] = O.dense(256)
    w = O.random_weights(cfg, sharp=1.0)
    import json
    import os
    import tempfile
    from safetensors.torch import save_file
    with tempfile.TemporaryDirectory() as d:
        with open(os.path.join(d, "config.json"), "w") as f:
            json.dump(cfg, f)
        save_file({k: v.bfloat16().contiguous() for k, v in w.items()}, os.path.join(d, "model.safetensors"))
        m8 = AutoModelForCausalLM.from_pretrained(d, load_in_low_bit="sym_int8").to("cuda")
    ref = dobetar.build(cfg, w, torch.bfloat16).to("cuda")
    toks = torch.tensor([tokens(40, cfg["vocab"], 2)], device="cuda")
    a, b = m8(toks).logits, ref(toks).logits
    cos = torch.nn.functional.cosine_similarity(a[0], b[0], dim=-1)
    assert cos.median() > 0.99
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
    import json
    from safetensors.torch import save_file
    from ipex_llm_b200.cli import llm_cli
    from ipex_llm_b200.transformers import AutoModelForCausalLM
    cfg = cfg_plain()
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_file({k: v.bfloat16().contiguous() for k, v in O.random_weights(cfg, seed=4).items()},
              str(tmp_path / "model.safetensors"))
    assert llm_cli.main(["-m", str(tmp_path), "-t", "bf16", "--token-ids", "3 9 4, 77", "-n", "6"]) == 0
    got = [int(t) for t in capsys.readouterr().out.split()]
    model = AutoModelForCausalLM.from_pretrained(str(tmp_path), load_in_low_bit="bf16", torch_dtype=BF16).to("cuda")
    out = model.generate(torch.tensor([[3, 9, 4, 77]], device="cuda"), max_new_tokens=6, do_sample=False)
    assert got == out[0, 4:].tolist() and len(got) == 6


def test_trace_replay(tmp_path):
    """The replay program on a checkpoint: a batch that starts together and thins out, then another request."""
    import json
    import os
    import subprocess
    import sys
    import numpy as np
    from safetensors.torch import save_file
    cfg = cfg_plain()
    w = O.random_weights(cfg, seed=4)
    d, out = str(tmp_path / "m"), str(tmp_path / "o")
    os.makedirs(d)
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.bfloat16().contiguous() for k, v in w.items()}, os.path.join(d, "model.safetensors"))
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
