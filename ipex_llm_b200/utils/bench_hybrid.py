"""Hybrid decoder (Letarax, bf16, random weights) against the closest model of the framework at equal size.

    python -m ipex_llm_b200.utils.bench_hybrid [--sizes mid,large] [--kernels] [--json OUT]

Model runs: prompt throughput (one prompt of ``--prompt`` tokens, device-timed) and decode latency (graph replay) of the
design with attention and recurrent layers taking turns, of attention layers alone and of recurrent layers alone, and of a
Llama-architecture model in bf16 with the same width, depth, heads, key / value heads and feed-forward size, all through
``AutoModelForCausalLM.from_config`` and the engine.  ``--kernels`` times every kernel of the new design alone, next to the
like kernel of the closest model (for the recurrence: the RWKV-5 kernel) on the same shape, with its distance from the
roofline (measured copy bandwidth and GEMM rate of ``MEASURED_PEAKS.json`` when that file is in the working directory).
Inputs rotate through more than the L2.
"""
from __future__ import annotations

import argparse
import json

import torch

from .bench_latent import VOCAB, _events, _graph_us, _sets, run_model

SIZES = {
    # width, layers, heads, key / value heads, dim (= vdim), window, ff, recurrent layers: heads, key heads, dim, vdim
    "small": dict(W=1024, layers=8, H=16, G=4, dim=64, window=512, ff=2816, dH=16, dG=8, dD=64, dV=64),
    "mid": dict(W=2048, layers=8, H=16, G=4, dim=128, window=1024, ff=5504, dH=16, dG=8, dD=128, dV=128),
    "large": dict(W=4096, layers=8, H=32, G=8, dim=128, window=2048, ff=11008, dH=32, dG=16, dD=128, dV=128),
}
TAPS = 4


def letarax_config(z, kinds: str):
    """``kinds``: layer types in turn, ``a`` attention and ``d`` recurrent."""
    from ..models.letarax import LetaraxConfig
    mlp = {"kind": "dense", "ff": z["ff"]}
    layers = []
    for i in range(z["layers"]):
        if kinds[i % len(kinds)] == "a":
            layers.append({"type": "attention", "mlp": mlp,
                           "mixer": {"heads": z["H"], "kv_heads": z["G"], "dim": z["dim"], "vdim": z["dim"],
                                     "mask": {"size": z["window"]}, "scale": z["dim"] ** -0.5, "v_mix": True}})
        else:
            layers.append({"type": "delta", "mlp": mlp,
                           "mixer": {"heads": z["dH"], "kv_heads": z["dG"], "dim": z["dD"], "vdim": z["dV"], "conv": TAPS}})
    return LetaraxConfig(vocab=VOCAB, width=z["W"], norm={"eps": 1e-6}, layers=layers)


def llama_config(z):
    from transformers import LlamaConfig
    return LlamaConfig(hidden_size=z["W"], intermediate_size=z["ff"], num_hidden_layers=z["layers"],
                       num_attention_heads=z["H"], num_key_value_heads=z["G"], head_dim=z["dim"], vocab_size=VOCAB,
                       max_position_embeddings=8192, tie_word_embeddings=False)


def kernels(z, prompt: int, peaks):
    """Rows ``{kernel, us, roofline_us, frac}`` and the like kernel's ``frac`` on the same shape."""
    from ..engine.stream_engine import Portions
    from ..ops import cuda_ops, delta as R, stream as S, tcgen05_gemm, window_attn as A
    from ..ops.kv_cache import DeltaStateShape, KeyValueShape, SlotCache
    from ..ops.rwkv import rwkv_linear_attention_v5
    hbm, tf = peaks.get("hbm_gbs", 6650.0) * 1e3, peaks.get("bf16_tflops", 1590.0) * 1e6     # bytes / us, flop / us
    dev, bf = "cuda", torch.bfloat16
    W, H, G, D, ff, rows = z["W"], z["H"], z["G"], z["dim"], z["ff"], []
    dH, dG, dD, dV = z["dH"], z["dG"], z["dD"], z["dV"]

    def mat(*shape, s=0.02):
        return torch.randn(*shape, device=dev, dtype=bf) * s

    def ints(v):
        return torch.tensor(v, device=dev, dtype=torch.int32)

    def add(name, us, nbytes=0.0, flops=0.0, like=None, like_frac=None):
        roof = max(nbytes / hbm, flops / tf)
        rows.append({"kernel": name, "us": round(us, 2), "roofline_us": round(roof, 2), "frac": round(roof / us, 3),
                     "like": like, "like_frac": None if like_frac is None else round(like_frac, 3)})

    att = A.AttnSpec(H, G, D, D, D ** -0.5, z["window"], True)
    dl = R.DeltaSpec(dH, dG, dD, dV, TAPS)
    # --- few-row products
    gate_rows = mat(2 * dH, W)
    for name, N, K, mode, act, two in (("gemv q/k/v + bias", att.rows, W, 0, 0, False),
                                       ("gemv recurrent projections + gates", dl.rows, W, 0, 0, True),
                                       ("gemv o_proj", W, H * D, 2, 0, False),
                                       ("gemv gate / up, gelu", 2 * ff, W, 0, S.ACT_GELU_GLU, False),
                                       ("gemv down + bias", W, ff, 2, 0, False), ("gemv lm_head", VOCAB, W, 2, 0, False)):
        n = _sets(2 * N * K)
        ws, bias = [mat(N, K) for _ in range(n)], mat(N)
        for M in (1, 8):
            x = mat(M, K, s=1.0)
            out = torch.zeros(M, N // 2 if act else N, device=dev, dtype=bf if mode == 0 else torch.float32)
            o2 = torch.empty(M, 2 * dH, device=dev) if two else None
            us = _graph_us(lambda i: S.gemv_rows(ws[i], x, out, mode, act=act, bias=bias, w2=gate_rows if two else None,
                                                 out2=o2, pdl=True), n)
            ob = torch.empty(M, N // 2 if act else N, device=dev, dtype=bf)
            like = _graph_us(lambda i: cuda_ops.gemv_lowbit(x, ws[i], None, N, K, out=ob, wf=7, pdl=True,
                                                            act=2 if act else 0), n) \
                if K % 64 == 0 and N % 16 == 0 and M <= cuda_ops._gemv_rows_per_call(K) else None
            add(f"{name} M={M} {N}x{K}", us, 2 * N * K, 2.0 * M * N * K, "gemv_lowbit bf16",
                2 * N * K / hbm / like if like else None)
        del ws
    # --- the joint between two sublayers
    w1 = torch.ones(W, device=dev)
    for M in (1, 8, prompt):
        n = _sets(8.0 * M * W)
        xs, ys = [torch.randn(M, W, device=dev) for _ in range(n)], [torch.randn(M, W, device=dev) for _ in range(n)]
        us = _graph_us(lambda i: S.add_norm_stream(xs[i], ys[i], w1, w1, 1e-6, bf, pdl=True), n)
        xb, wb = [mat(M, W) for _ in range(n)], torch.ones(W, device=dev, dtype=bf)
        ro = torch.empty_like(xb[0])
        like = _graph_us(lambda i: cuda_ops.rms_norm(xb[i], wb, 1e-6, residual=xb[(i + 1) % n], residual_out=ro), n)
        add(f"norm, add, norm M={M}", us, 14.0 * M * W, 0, f"rms_norm + residual {like:.1f} us", 8.0 * M * W / hbm / like)
        del xs, ys, xb
    # --- decode attention
    ctx = z["window"]
    for B in (1, 8, 32):
        n = min(32, _sets(4.0 * B * ctx * G * D))
        cache = SlotCache()
        cache.allocate(B, ctx + 8, [KeyValueShape(G, D, D)] * n, bf, dev)
        for layer in cache.layers:
            layer._k.normal_()
            layer._v.normal_()
        qkv, slot, pos = mat(B, att.rows, s=1.0), ints(list(range(B))), ints([ctx - 1] * B)
        mix = A.ValueMix(mat(B, G * D, s=1.0), 0.5)
        out = torch.empty(B, H * D, device=dev, dtype=bf)
        us = _graph_us(lambda i: A.attend_step(att, qkv, mix, slot, pos, cache, i, out, ctx, True, pdl=True), n)
        q, ks, vs = mat(B, H, 1, D, s=1.0), [c._k[:, :, :ctx] for c in cache.layers], [c._v[:, :, :ctx] for c in cache.layers]
        like = _graph_us(lambda i: cuda_ops.sdpa_decode(q, ks[i], vs[i], None, D ** -0.5, None, None), n)
        nb = 4.0 * B * ctx * G * D
        add(f"kv_attn B={B} ctx={ctx} splits={A.pick_splits(B, att, ctx)}", us, nb, 4.0 * B * ctx * H * D,
            f"attn_decode {like:.1f} us", nb / hbm / like)
        del cache, ks, vs
    # --- recurrence, one token each
    w = R.DeltaWeights(mat(dl.channels, TAPS, s=0.5), torch.zeros(dH, device=dev), torch.zeros(dH, device=dev),
                       torch.ones(dV, device=dev, dtype=bf), 1e-6)
    for B in (1, 8, 32):
        n = min(48, _sets(4.0 * B * dH * dD * dV))
        cache = SlotCache()
        cache.allocate(B, 64, [DeltaStateShape(dH, dD, dV, TAPS, dl.channels)] * n, bf, dev)
        proj, gates = mat(B, dl.rows, s=1.0), torch.randn(B, 2 * dH, device=dev)
        slot, pos = ints(list(range(B))), ints([9] * B)
        out = torch.empty(B, dH * dV, device=dev, dtype=bf)
        us = _graph_us(lambda i: R.delta_mix(dl, w, proj, gates, slot, pos, cache, i, out, pdl=True), n)
        st = [torch.zeros(B, dH, dV, dV, device=dev) for _ in range(n)]
        r = torch.randn(B, dH, 1, dV, device=dev)
        dec = torch.full((dH * dV,), 0.9, device=dev)
        like = _graph_us(lambda i: rwkv_linear_attention_v5(dec, dec, r, r, r, st[i]), n)
        nb = 8.0 * B * dH * dD * dV
        add(f"delta_step B={B}", us, nb, 6.0 * B * dH * dD * dV, f"rwkv5 {like:.1f} us", 8.0 * B * dH * dV * dV / hbm / like)
        del cache, st
    # --- prompt GEMMs
    T = prompt
    for name, N, K, mode, act in (("gemm q/k/v + bias", att.rows, W, 0, 0), ("gemm recurrent projections + gates", dl.rows, W, 0, 0),
                                  ("gemm o_proj, fp32", W, H * D, 2, 0),
                                  ("gemm gate / up, gelu", 2 * ff, W, 0, S.ACT_GELU_GLU),
                                  ("gemm down + bias, fp32", W, ff, 2, 0)):
        n = _sets(2.0 * (N * K + T * K))
        ws, xk, bias = [mat(N, K) for _ in range(n)], [mat(T, K, s=1.0) for _ in range(n)], mat(N)
        No = N // 2 if act else N
        out = torch.zeros(T, No, device=dev, dtype=bf if mode == 0 else torch.float32)
        two = (gate_rows, torch.empty(T, 2 * dH, device=dev)) if "gates" in name else (None, None)
        us = _graph_us(lambda i: S.gemm(xk[i], ws[i], out, mode, act, bias, True, *two), n)
        ob, res = torch.empty(T, No, device=dev, dtype=bf), mat(T, N) if mode == 2 else None
        like = _graph_us(lambda i: tcgen05_gemm.gemm_dense(xk[i], ws[i], residual=res, out=ob, act=2 if act else 0), n)
        fl, nb = 2.0 * T * N * K, 2.0 * (T * K + N * K)
        add(f"{name} {T}x{N}x{K}", us, nb, fl, f"gemm_dense {like:.1f} us", max(fl / tf, nb / hbm) / like)
        del ws, xk
    # --- prompt attention
    cache = SlotCache()
    cache.allocate(1, T + 8, [KeyValueShape(G, D, D)], bf, dev)
    n = 6
    qkv, mix = [mat(T, att.rows, s=1.0) for _ in range(n)], A.ValueMix(mat(T, G * D, s=1.0), 0.5)
    slot, pos, row, ln = ints([0] * T), ints(list(range(T))), ints([0]), ints([T])
    out = torch.empty(T, H * D, device=dev, dtype=bf)
    full = A.AttnSpec(H, G, D, D, D ** -0.5, 0, True)
    for spec in (att, full):
        us = _graph_us(lambda i: A.attend_prompt(spec, qkv[i], mix, slot, pos, row, ln, T, cache, 0, out), n)
        w_ = min(spec.window or T, T)
        pairs = T * w_ - w_ * (w_ - 1) / 2
        fl = 4.0 * H * pairs * D
        t = [q.view(1, T, H + 2 * G, D) for q in qkv]
        like = _graph_us(lambda i: cuda_ops.attn_prefill_tcgen05(
            t[i][:, :, :H].transpose(1, 2), t[i][:, :, H:H + G].transpose(1, 2), t[i][:, :, H + G:].transpose(1, 2),
            D ** -0.5, True, window=spec.window), n)
        add(f"kv_append + packed_prefill T={T} window={spec.window}", us, 0, fl,
            f"attn_prefill_tcgen05 {like:.1f} us (transposes V, appends nothing)", fl / tf / like)
    # --- recurrence over a prompt
    cache = SlotCache()
    cache.allocate(1, T + 8, [DeltaStateShape(dH, dD, dV, TAPS, dl.channels)], bf, dev)
    nc = -(-T // Portions.CHUNK)
    where = Portions(row, ln, T, True, ints([0] * nc), ints([0, nc]), nc)
    projs, gates = [mat(T, dl.rows, s=1.0) for _ in range(4)], torch.randn(T, 2 * dH, device=dev)
    out = torch.empty(T, dH * dV, device=dev, dtype=bf)
    nb, fl = 2.0 * T * (dl.rows + dH * dV), 6.0 * T * dH * dD * dV
    us = _graph_us(lambda i: R.delta_mix(dl, w, projs[i], gates, slot, pos, cache, 0, out, where), 4)
    r = torch.randn(1, dH, T, dV, device=dev)
    st, dec = torch.zeros(1, dH, dV, dV, device=dev), torch.full((dH * dV,), 0.9, device=dev)
    like = _events(lambda: rwkv_linear_attention_v5(dec, dec, r, r, r, st), 3, 2) * 1e3
    add(f"delta_chunks (4 kernels) T={T}", us, nb, fl, f"rwkv5 {like:.1f} us",
        max(16.0 * T * dH * dV / hbm, 4.0 * T * dH * dV * dV / tf) / like)
    from ..native.lib import ptr, stream_lib
    lib = stream_lib("recurrent")
    per = dH * stream_lib("delta").ipex_delta_scratch_floats(dD, dV)
    rows.append({"kernel": f"delta scratch, MB for T={T}", "us": round(nc * per * 4 / 1e6, 1)})
    raw = torch.empty(T, dH, dV, device=dev)
    us = _graph_us(lambda i: lib.ipex_gated_norm(ptr(raw), ptr(projs[i][:, dl.channels:]), dl.rows, ptr(w.norm), 0, 0, ptr(out),
                                                 out.stride(0), T, dH, dV, 1e-6, 1.0, 1, S.current_stream()), 4)
    add(f"gated_norm T={T}", us, 8.0 * T * dH * dV)
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
            for label, cfg in (("letarax", letarax_config(z, "da")), ("letarax_attention", letarax_config(z, "a")),
                               ("letarax_recurrent", letarax_config(z, "d")), ("llama", llama_config(z))):
                r[label] = run_model(cfg, a.prompt, batches, a.iters)
        if a.kernels:
            r["kernels"] = kernels(z, a.prompt, peaks)
        res["sizes"][name] = r
    if timed is not None:
        timed[1]()
    last = a.sizes.split(",")[-1]
    if "letarax" in res["sizes"][last]:
        m = res["sizes"][last]["letarax"]
        res.update(model=f"letarax-{last} ({m['params_m']:.0f} M, {SIZES[last]['layers']} layers)", unit="tokens/s",
                   value=m["decode_tok_s"][1], ms_per_step=m["decode_ms"][1])
    if a.json:
        with open(a.json, "w") as f:
            json.dump(res, f, indent=1)
    return res


if __name__ == "__main__":
    print(json.dumps(run(), indent=1))
