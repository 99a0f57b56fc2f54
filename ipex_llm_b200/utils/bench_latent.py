"""Latent-attention decoder (Dobetar, bf16, random weights) against the closest model of the framework at equal size.

    python -m ipex_llm_b200.utils.bench_latent [--sizes mid,large] [--kernels] [--json OUT]

Model runs: prompt throughput (one prompt of ``--prompt`` tokens, device-timed) and decode latency (graph replay) of the
new design and of a Llama-architecture model in bf16 with the same width, depth, heads and feed-forward size (dense
layers), both through ``AutoModelForCausalLM.from_config`` and the engine; the design's own mixture-of-experts variant is
timed beside them.  ``--kernels`` times every kernel of the new design alone, next to the like kernel of the closest
model on the same shape, with its distance from the roofline (measured copy bandwidth and GEMM rate of
``MEASURED_PEAKS.json`` when that file is in the working directory).  Inputs rotate through more than the L2.
"""
from __future__ import annotations

import argparse
import gc
import json

import torch

SIZES = {
    # width, layers, heads, dim, rot_dim, vdim, kv_rank, window, ff, experts, top, expert ff
    "small": dict(W=1024, layers=8, H=16, dim=64, rd=32, vd=64, R=256, window=512, ff=4096, E=8, top=2, eff=2048),
    "mid": dict(W=2048, layers=8, H=16, dim=128, rd=64, vd=128, R=512, window=1024, ff=8192, E=16, top=2, eff=2048),
    "large": dict(W=4096, layers=8, H=32, dim=128, rd=64, vd=128, R=512, window=2048, ff=16384, E=32, top=2, eff=4096),
}
VOCAB = 32000


def dobetar_config(z, moe: bool):
    from ..models.dobetar import DobetarConfig
    mixer = {"heads": z["H"], "dim": z["dim"], "rot_dim": z["rd"], "vdim": z["vd"], "kv_rank": z["R"],
             "mask": {"size": z["window"]}, "rot": {"base": 10000.0, "dims": z["rd"]},
             "scale": (z["dim"] + z["rd"]) ** -0.5}
    dense = {"kind": "dense", "ff": z["ff"]}
    sparse = {"kind": "moe", "expert": {"ff": z["eff"], "limit": 7.0}, "router": {"experts": z["E"], "top": z["top"]}}
    return DobetarConfig(vocab=VOCAB, width=z["W"], logit_softcap=30.0, norm={"eps": 1e-6},
                         embedding={"scale": 1.0, "bigram": {"buckets": 50021, "mul_prev": 31, "mul_cur": 7}},
                         layers=[{"type": "latent_attention", "mixer": mixer, "mlp": sparse if moe and i % 2 else dense}
                                 for i in range(z["layers"])])


def llama_config(z):
    from transformers import LlamaConfig
    # a gated MLP has three matrices: two thirds of ff gives the same weight bytes
    ff = z["ff"] * 2 // 3 // 64 * 64
    return LlamaConfig(hidden_size=z["W"], intermediate_size=ff, num_hidden_layers=z["layers"],
                       num_attention_heads=z["H"], num_key_value_heads=z["H"], head_dim=z["vd"], vocab_size=VOCAB,
                       max_position_embeddings=8192, tie_word_embeddings=False)


def _events(fn, iters, warmup):
    for _ in range(warmup):
        fn()
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    for _ in range(iters):
        fn()
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) / iters


def run_model(cfg, prompt: int, batches, iters: int):
    from ..engine import get_engine
    from ..transformers import AutoModelForCausalLM
    model = AutoModelForCausalLM.from_config(cfg, load_in_low_bit="bf16", torch_dtype=torch.bfloat16, device="cuda")
    params = sum(p.numel() for p in model.parameters())
    g = torch.Generator().manual_seed(0)
    out = {"params_m": round(params / 1e6, 1), "decode_ms": {}}
    with torch.no_grad():
        eng = get_engine(model, max(batches), prompt + 512)
        ids = torch.randint(0, VOCAB, (1, prompt), generator=g).cuda()
        ms = _events(lambda: eng.prefill(ids), max(3, iters // 8), 3)
        out["prefill_ms"], out["prefill_tok_s"] = round(ms, 3), round(prompt / ms * 1e3)
        for B in batches:
            ids = torch.randint(0, VOCAB, (B, prompt // 2 if B > 8 else prompt), generator=g).cuda()
            eng.prefill(ids)
            eng.tokens[:B] = 1
            out["decode_ms"][B] = round(_events(lambda: eng.decode_step(B), iters, 8), 4)
    out["decode_tok_s"] = {B: round(B / ms * 1e3) for B, ms in out["decode_ms"].items()}
    from ..ops.cuda_ops import check_error_flag
    check_error_flag(torch.device("cuda", torch.cuda.current_device()))
    del eng, model
    gc.collect()            # model and engine refer to each other: their graphs must not be freed during a later capture
    torch.cuda.empty_cache()
    return out


# ------------------------------------------------------------------------------------------------
# kernels alone
# ------------------------------------------------------------------------------------------------
def _graph_us(fn, n_sets: int, launches: int = 24):
    """Microseconds per call: one graph of ``launches`` calls over rotating inputs, replayed a few times."""
    for i in range(min(n_sets, 3)):
        fn(i)
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g):
        for i in range(launches):
            fn(i % n_sets)
    return _events(g.replay, 5, 2) / launches * 1e3


def _sets(nbytes: float) -> int:
    return int(min(48, max(2, 300e6 // max(nbytes, 1) + 1)))


def _fp8_bank(E: int, I: int, W: int):
    from ..ops.moe import convert_fused_experts
    from ..quant import qtypes as qt
    m = torch.nn.Module()
    m.gate_up_proj = torch.nn.Parameter(torch.randn(E, 2 * I, W, device="cuda", dtype=torch.bfloat16) * 0.02, False)
    m.down_proj = torch.nn.Parameter(torch.randn(E, W, I, device="cuda", dtype=torch.bfloat16) * 0.02, False)
    return convert_fused_experts(m, qt.FP8E4, device="cuda")


def kernels(z, prompt: int, peaks):
    """Rows ``{kernel, us, roofline_us, frac}`` and the like kernel's ``frac`` on the same shape."""
    from ..ops import cuda_ops, latent as L, tcgen05_gemm
    from ..ops.kv_cache import LatentCache
    hbm, tf = peaks.get("hbm_gbs", 6650.0) * 1e3, peaks.get("bf16_tflops", 1590.0) * 1e6     # bytes / us, flop / us
    dev, bf = "cuda", torch.bfloat16
    W, H, R, rows = z["W"], z["H"], z["R"], []

    def mat(*shape, s=0.02):
        return torch.randn(*shape, device=dev, dtype=bf) * s

    def add(name, us, nbytes=0.0, flops=0.0, like=None, like_frac=None):
        roof = max(nbytes / hbm, flops / tf)
        rows.append({"kernel": name, "us": round(us, 2), "roofline_us": round(roof, 2), "frac": round(roof / us, 3),
                     "like": like, "like_frac": None if like_frac is None else round(like_frac, 3)})

    # --- few-row products: qkv (norm in front), o (added to the stream), up, lm_head
    for name, N, K, mode, norm in (("gemv qkv", H * (z["dim"] + z["rd"]) + R + z["rd"], W, 0, True),
                                   ("gemv o_proj", W, H * z["vd"], 1, False), ("gemv up", z["ff"], W, 0, True),
                                   ("gemv down", W, z["ff"], 1, False), ("gemv lm_head", VOCAB, W, 2, True)):
        n = _sets(2 * N * K)
        ws = [mat(N, K) for _ in range(n)]
        for M in (m for m in (1, 8) if m <= L.rows_max(K, bf)):
            x = torch.randn(M, K, device=dev) if norm else mat(M, K, s=1.0)
            out = torch.zeros(M, N, device=dev, dtype=bf if mode == 0 else torch.float32)
            nw = torch.ones(K, device=dev, dtype=bf) if norm else None
            us = _graph_us(lambda i: L.gemv_rows(ws[i], x, out, mode, norm=nw, eps=1e-6, pdl=True), n)
            xb, ob = mat(M, K, s=1.0), torch.empty(M, N, device=dev, dtype=bf)
            like = _graph_us(lambda i: cuda_ops.gemv_lowbit(xb, ws[i], None, N, K, out=ob, wf=7, pdl=True,
                                                            norm_weight=nw), n) \
                if K % 64 == 0 and N % 16 == 0 and M <= cuda_ops._gemv_rows_per_call(K) else None
            add(f"{name} M={M} {N}x{K}", us, 2 * N * K, 2.0 * M * N * K, "gemv_lowbit bf16",
                2 * N * K / hbm / like if like else None)
        del ws
    # --- decode attention
    spec = L.LatentSpec(H, z["dim"], z["rd"], z["vd"], R, 0.1, z["window"], z["rd"] // 2, 1e-6)
    cos, sin = L.rotary_table(4096, 1e4, z["rd"] // 2, dev)
    uk, uv, kn = mat(H * z["dim"], R), mat(H * z["vd"], R), torch.ones(R, device=dev, dtype=bf)
    lib, st = L.stream_lib("latent"), L.current_stream
    for B in (1, 8, 32):
        ctx = z["window"]
        n = _sets(B * ctx * (R + z["rd"]) * 2)
        n = min(n, 32)
        cache = LatentCache()
        cache.allocate(B, ctx + 8, [spec.row(bf)] * n, bf, dev)
        for layer in cache.layers:
            layer._k.normal_()
        qkv = mat(B, H * (z["dim"] + z["rd"]) + R + z["rd"], s=1.0)
        slot = torch.arange(B, device=dev, dtype=torch.int32)
        pos = torch.full((B,), ctx - 1, device=dev, dtype=torch.int32)
        qabs = mat(B, H, R, s=1.0)
        ns = L.pick_latent_splits(B, H, ctx)
        o = torch.empty(B, ns, H, R, device=dev)
        ml = torch.empty(B, ns, H, 2, device=dev)
        out = torch.empty(B, H * z["vd"], device=dev, dtype=bf)
        p = L.ptr

        def prep(i):
            k = cache.layers[i]._k
            lib.ipex_latent_prep(p(qkv), qkv.stride(0), p(qkv[:, -(R + z["rd"]):]), qkv.stride(0), p(kn), 1e-6, p(uk), p(cos), p(sin), p(slot), p(pos),
                                 p(cache.start), p(k), k.stride(0), k.stride(2), p(qabs), B, H, z["dim"], z["rd"], R,
                                 z["rd"] // 2, 1, 1, st())

        def attn(i):
            k = cache.layers[i]._k
            lib.ipex_latent_attn(p(qabs), p(qkv), qkv.stride(0), p(k), k.stride(0), k.stride(2), p(slot), p(pos),
                                 p(cache.start), p(o), p(ml), B, H, z["dim"], z["rd"], R, z["window"], ns, 0.1, 0, 1, 1,
                                 st())

        def up(i):
            lib.ipex_latent_uv(p(o), p(ml), p(uv), None, 0, p(out), out.stride(0), B, H, R, z["vd"], ns, 1, 1, st())
        wb = 2.0 * H * z["dim"] * R
        add(f"latent_prep B={B}", _graph_us(prep, n), wb, 2.0 * B * H * z["dim"] * R)
        kvb = 2.0 * B * ctx * (R + z["rd"])
        us = _graph_us(attn, n)
        # the like kernel: split-KV decode attention of the same heads over the same context, 16-bit keys and values
        D = z["vd"]
        nk = min(16, _sets(4.0 * B * H * ctx * D))
        q = mat(B, H, 1, D, s=1.0)
        ks = [mat(B, H, ctx, D, s=1.0) for _ in range(nk + 1)]
        like = _graph_us(lambda i: cuda_ops.sdpa_decode(q, ks[i % nk], ks[i % nk + 1], None, 0.1, None, None), nk)
        lb = 4.0 * B * H * ctx * D
        add(f"latent_attn B={B} ctx={ctx}", us, kvb, 2.0 * B * H * ctx * (2 * R + z["rd"]),
            f"attn_decode {like:.1f} us for {lb / 1e6:.0f} MB", lb / hbm / like)
        parts = 4.0 * B * ns * H * R                        # partial outputs of the splits
        add(f"latent_uv B={B} splits={ns}", _graph_us(up, n), 2.0 * H * z["vd"] * R + parts, 2.0 * B * H * z["vd"] * R)
        del cache, ks
    # --- experts, few rows
    E, k, I = z["E"], z["top"], z["eff"]
    n = max(2, min(6, _sets(6.0 * E * I * W)))
    banks = [L.ExpertBank(mat(E, W), mat(E, 2 * I, W), mat(E, W, I), k, 7.0, 1.702, True) for _ in range(n)]
    nw = torch.ones(W, device=dev, dtype=bf)
    fp8 = _fp8_bank(E, I, W)
    router = mat(E, W)

    def like_moe(T):
        """(us, roofline fraction) of the framework's packed expert bank (fp8) on the same shape."""
        xb = mat(T, W, s=1.0)

        def fn(i):
            _, w, idx = cuda_ops.moe_softmax_topk(torch.matmul(xb, router.t()), k, True)
            cuda_ops.moe_forward(fp8, xb, idx, w)
        # (its prompt path allocates host tensors: timed eagerly)
        us = _graph_us(fn, 1, launches=6) if T <= 8 else _events(lambda: fn(0), 5, 3) * 1e3
        hit = E * (1 - (1 - k / E) ** T)
        return us, max(3.0 * hit * I * W * 1.03 / hbm, 6.0 * T * k * I * W / tf) / us
    for B in (1, 8):
        x = torch.randn(B, W, device=dev)
        hit = E * (1 - (1 - k / E) ** B)                   # experts that expect a token
        us = _graph_us(lambda i: L.moe_rows(banks[i], x, nw, 1e-6, pdl=True), n)
        lu, lf = like_moe(B)
        add(f"moe_rows (3 kernels) B={B}", us, 6.0 * hit * I * W + 2.0 * E * W, 6.0 * B * k * I * W,
            f"fp8 bank {lu:.1f} us", lf)
    # --- prompt GEMMs
    T = prompt
    xs = [mat(T, W, s=1.0) for _ in range(_sets(2 * T * W))]
    for name, N, K, mode in (("gemm qkv", H * (z["dim"] + z["rd"]) + R + z["rd"], W, 0), ("gemm up relu2", z["ff"], W, 0),
                             ("gemm o_proj += stream", W, H * z["vd"], 1), ("gemm down += stream", W, z["ff"], 1)):
        n = _sets(2.0 * (N * K + T * K))
        ws, xk = [mat(N, K) for _ in range(n)], [mat(T, K, s=1.0) for _ in range(n)]
        out = torch.zeros(T, N, device=dev, dtype=bf if mode == 0 else torch.float32)
        act = L.ACT_RELU2 if "relu2" in name else 0
        us = _graph_us(lambda i: L.gemm(xk[i], ws[i], out, mode, act), n)
        ob = torch.empty(T, N, device=dev, dtype=bf)
        res = mat(T, N) if mode == 1 else None
        like = _graph_us(lambda i: tcgen05_gemm.gemm_dense(xk[i], ws[i], residual=res, out=ob), n)
        fl = 2.0 * T * N * K
        add(f"{name} {T}x{N}x{K}", us, 0, fl, f"gemm_dense {like:.1f} us", fl / tf / like)
        del ws, xk
    # --- prompt attention
    spec2 = L.LatentSpec(H, z["dim"], z["rd"], z["vd"], R, 0.05, z["window"], z["rd"] // 2, 1e-6)
    ldq = H * (z["dim"] + z["rd"]) + R + z["rd"]
    n = 6
    qs, ks = [mat(T, ldq, s=1.0) for _ in range(n)], [mat(T, H * z["dim"], s=1.0) for _ in range(n)]
    kr, vt = mat(T, z["rd"], s=1.0), mat(H * z["vd"], T, s=1.0)
    out = torch.empty(T, H * z["vd"], device=dev, dtype=bf)
    i32 = dict(device=dev, dtype=torch.int32)
    row, ln, err = torch.zeros(1, **i32), torch.full((1,), T, **i32), cuda_ops.error_flag(torch.device("cuda", 0))
    for win in (z["window"], 0):
        us = _graph_us(lambda i: L.stream_lib().ipex_packed_prefill(
            L.ptr(qs[i]), ldq, L.ptr(ks[i]), H * z["dim"], L.ptr(kr), z["rd"], L.ptr(vt), T, L.ptr(out), H * z["vd"],
            L.ptr(row), L.ptr(ln), 1, H, H, T, T, z["dim"], z["rd"], z["vd"], win, 0, 0, None, None, 0,
            1.0, 0, None, 0, None, 0, None, 0, 0.05, 1, L.ptr(err),
            L.current_stream()), n)
        w = win or T
        pairs = T * min(w, T) - min(w, T) * (min(w, T) - 1) / 2
        fl = 2.0 * H * pairs * (z["dim"] + z["rd"] + z["vd"])
        D = z["vd"]
        qkv = [mat(1, T, 3 * H, D, s=1.0) for _ in range(n)]

        def like_fn(i):
            t = qkv[i]
            cuda_ops.attn_prefill_tcgen05(t[:, :, :H].transpose(1, 2), t[:, :, H:2 * H].transpose(1, 2),
                                          t[:, :, 2 * H:].transpose(1, 2), 0.05, True, window=win)
        like = _graph_us(like_fn, n)
        lf = 4.0 * H * pairs * D
        add(f"latent_prefill T={T} window={win}", us, 0, fl, f"attn_prefill_tcgen05 {like:.1f} us (+ transpose)",
            lf / tf / like)
    # --- grouped experts
    h = [mat(T, W, s=1.0) for _ in range(2)]
    x = torch.zeros(T, W, device=dev)
    us = _graph_us(lambda i: L.moe_grouped(banks[i % len(banks)], x, h[i % 2]), 2, launches=6)
    lu, lf = like_moe(T)
    add(f"moe_grouped (8 kernels) T={T}", us, 6.0 * E * I * W, 6.0 * T * k * I * W, f"fp8 bank {lu:.1f} us", lf)
    cuda_ops.check_error_flag(torch.device("cuda", 0))
    return rows


def run(argv=None, timed=None):
    ap = argparse.ArgumentParser(description=__doc__.split("\n")[0])
    ap.add_argument("--sizes", default="small,mid,large")
    ap.add_argument("--prompt", type=int, default=2048)
    ap.add_argument("--iters", type=int, default=64)
    ap.add_argument("--kernels", action="store_true")
    ap.add_argument("--no-models", action="store_true")
    ap.add_argument("--json", default=None)
    a = ap.parse_args(argv)
    try:
        with open("MEASURED_PEAKS.json") as f:
            peaks = json.load(f)
    except OSError:
        peaks = {}
    res = {"prompt": a.prompt, "sizes": {}}
    if timed is not None:
        timed[0]()
    for name in a.sizes.split(","):
        z, r = SIZES[name], {"shape": SIZES[name]}
        if not a.no_models:
            batches = (1, 8, 32)
            r["dobetar_dense"] = run_model(dobetar_config(z, False), a.prompt, batches, a.iters)
            r["dobetar_moe"] = run_model(dobetar_config(z, True), a.prompt, batches, a.iters)
            r["llama"] = run_model(llama_config(z), a.prompt, batches, a.iters)
        if a.kernels:
            r["kernels"] = kernels(z, a.prompt, peaks)
        res["sizes"][name] = r
    if timed is not None:
        timed[1]()
    last = res["sizes"][a.sizes.split(",")[-1]]
    if "dobetar_moe" in last:
        m = last["dobetar_moe"]
        res.update(model=f"dobetar-{a.sizes.split(',')[-1]} ({m['params_m']:.0f} M, 8 layers)", unit="tokens/s",
                   value=m["decode_tok_s"][1], ms_per_step=m["decode_ms"][1])
    if a.json:
        with open(a.json, "w") as f:
            json.dump(res, f, indent=1)
    return res


if __name__ == "__main__":
    print(json.dumps(run(), indent=1))
