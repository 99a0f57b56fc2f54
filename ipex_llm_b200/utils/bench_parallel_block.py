"""Parallel-block decoder (Gegorax, bf16, random weights) against the closest models of the framework at equal size.

    python -m ipex_llm_b200.utils.bench_parallel_block [--sizes mid,large] [--kernels] [--json OUT]

Model runs: prompt throughput (one prompt of ``--prompt`` tokens, device-timed) and decode latency (graph replay) of the
design with generalized-delta layers alone, with two-sided layers alone, and with both and experts; beside them an attention
+ recurrence decoder and a decoder with several streams (Letarax, Dodilix) of the same width, heads and feed-forward bytes,
all through ``AutoModelForCausalLM.from_config`` and the engine.  ``--kernels`` times every kernel that is new or does more
than before, next to the like kernel of those models on the same shape, with its distance from the roofline (measured copy
bandwidth and GEMM rate of ``MEASURED_PEAKS.json`` when that file is in the working directory).  Inputs rotate through more
than the L2.
"""
from __future__ import annotations

import argparse
import json

import torch

from .bench_latent import VOCAB, _graph_us, _sets, run_model

SIZES = {
    # width, layers; generalized delta: heads, dim, rank; left: heads, key / value heads, dim (= vdim), window, pool; right:
    # heads, vdim, state, groups; feed-forward (two matrices), experts, chosen, expert and shared hidden size; token side
    "small": dict(W=1024, layers=8, dH=16, dD=64, rank=64, H=16, G=4, ad=64, window=512, pool=16, sH=32, sV=64, N=64, sG=1,
                  ff=4096, E=16, top=2, eff=512, sff=512, side=64),
    "mid": dict(W=2048, layers=8, dH=32, dD=64, rank=64, H=16, G=4, ad=128, window=1024, pool=16, sH=64, sV=64, N=128, sG=2,
                ff=8192, E=16, top=2, eff=1024, sff=1024, side=128),
    "large": dict(W=4096, layers=8, dH=32, dD=128, rank=128, H=32, G=8, ad=128, window=1024, pool=16, sH=128, sV=64, N=128, sG=8,
                  ff=16384, E=32, top=2, eff=2048, sff=2048, side=256),
}
TAPS = 4


def gegorax_config(z, kinds: str, moe: bool = False):
    """``kinds``: a letter per layer in turn: ``d`` generalized delta, ``p`` two-sided."""
    from ..models.gegorax import GegoraxConfig
    dense = {"kind": "dense", "ff": z["ff"]}
    sparse = {"kind": "moe", "expert": {"ff": z["eff"], "limit": 7.0}, "router": {"experts": z["E"], "top": z["top"]},
              "shared": {"ff": z["sff"], "limit": 7.0}}
    layers = []
    for i in range(z["layers"]):
        if kinds[i % len(kinds)] == "p":
            m = {"left": {"heads": z["H"], "kv_heads": z["G"], "dim": z["ad"], "vdim": z["ad"],
                          "mask": {"size": z["window"], "pool": z["pool"]}, "rot": {"base": 1e4, "dims": z["ad"]},
                          "scale": z["ad"] ** -0.5},
                 "right": {"heads": z["sH"], "vdim": z["sV"], "state": z["N"], "groups": z["sG"], "conv": TAPS,
                           "norm_groups": z["sG"]}}
        else:
            m = {"heads": z["dH"], "dim": z["dD"], "rank": z["rank"]}
        layers.append({"type": "parallel" if kinds[i % len(kinds)] == "p" else "general_delta", "mixer": m,
                       "mlp": sparse if moe and i else dense})
    return GegoraxConfig(vocab=VOCAB, width=z["W"], norm={"eps": 1e-6}, token_side={"dim": z["side"]}, layers=layers)


def letarax_config(z):
    from .bench_hybrid import letarax_config as make
    return make(dict(W=z["W"], layers=z["layers"], H=z["H"], G=z["G"], dim=z["ad"], window=z["window"], ff=z["ff"] * 2 // 3 // 64 * 64,
                     dH=z["dH"], dG=z["dH"], dD=z["dD"], dV=z["dD"]), "da")


def dodilix_config(z):
    from .bench_multistream import dodilix_config as make
    return make(dict(W=z["W"], layers=z["layers"], S=2, H=z["H"], G=z["G"], ad=z["ad"], chunk=z["window"], lH=z["dH"], lD=z["dD"],
                     lV=z["dD"], rank=16, ff=z["ff"] * 2 // 3 // 64 * 64, E=z["E"], top=z["top"], groups=1, keep=1, eff=z["eff"],
                     sff=z["sff"], dim=z["ad"], rd=64, vd=z["ad"], Rq=512, R=512), "p")


def kernels(z, prompt: int, peaks):
    """Rows ``{kernel, us, roofline_us, frac}`` and the like kernel's ``frac`` on the same shape."""
    from ..engine.stream_engine import Portions
    from ..ops import cuda_ops, delta as D, dense_moe as X, general_delta as R, latent as N, linear_attn as Li, ssd as Ss, \
        stream as K, window_attn as A
    from ..ops.kv_cache import DeltaStateShape, KeyValueShape, PooledShape, SlotCache
    from ..ops.recurrent import gated_group_norm, gated_norm
    hbm, tf = peaks.get("hbm_gbs", 6650.0) * 1e3, peaks.get("bf16_tflops", 1590.0) * 1e6     # bytes / us, flop / us
    dev, bf = "cuda", torch.bfloat16
    W, H, G, ad, T, P, win, rows = z["W"], z["H"], z["G"], z["ad"], prompt, z["pool"], z["window"], []

    def mat(*shape, s=0.02):
        return torch.randn(*shape, device=dev, dtype=bf) * s

    def f32(*shape):
        return torch.randn(*shape, device=dev)

    def ints(v):
        return torch.tensor(v, device=dev, dtype=torch.int32)

    def add(name, us, nbytes=0.0, flops=0.0, like=None, like_us=None, like_bytes=None, like_flops=None):
        roof = max(nbytes / hbm, flops / tf)
        lf = None if like_us is None else max((nbytes if like_bytes is None else like_bytes) / hbm,
                                              (flops if like_flops is None else like_flops) / tf) / like_us
        rows.append({"kernel": name, "us": round(us, 2), "roofline_us": round(roof, 2), "frac": round(roof / us, 3),
                     "like": like, "like_us": None if like_us is None else round(like_us, 2),
                     "like_frac": None if lf is None else round(lf, 3)})

    # --- joints
    ones = torch.ones(W, device=dev)
    for M in (1, 8, T):
        n = _sets(16.0 * M * W)
        xs, ys, y2 = ([f32(M, W) for _ in range(n)] for _ in range(3))
        like = _graph_us(lambda i: K.add_norm_stream(xs[i], ys[i], ones, ones, 1e-6, bf, pdl=True), n)
        us = _graph_us(lambda i: K.add_sides(xs[i], (ys[i], y2[i]), (ones, ones), None, 1e-6, bf, pdl=True), n)
        add(f"add_sides M={M}", us, 18.0 * M * W, 0, "add_norm_stream", like, 14.0 * M * W)
        del xs, ys, y2
    # --- few-row products
    dn = z["dH"] * z["dD"]
    sr = 2 * z["sH"] * z["sV"] + 2 * z["sG"] * z["N"]
    for name, Nr, two, act, start in (("gemv delta projection, hidden units, low rank", 5 * dn + z["ff"], z["rank"], K.ACT_RELU2, 5 * dn),
                                      ("gemv two-sided projection, hidden units, step sizes", (H + 2 * G) * ad + sr + z["ff"], z["sH"],
                                       K.ACT_RELU2, (H + 2 * G) * ad + sr)):
        n = _sets(2.0 * (Nr + two) * W)
        ws, w2 = [mat(Nr, W) for _ in range(n)], [mat(two, W) for _ in range(n)]
        for M in (1, 8):
            x, out, o2 = mat(M, W, s=1.0), torch.empty(M, Nr, device=dev, dtype=bf), torch.empty(M, two, device=dev)
            us = _graph_us(lambda i: K.gemv_rows(ws[i], x, out, 0, act=act, w2=w2[i], out2=o2, pdl=True,
                                                 args=K.ActArgs(start=start)), n)
            like = _graph_us(lambda i: K.gemv_rows(ws[i], x, out, 0, pdl=True), n)
            add(f"{name} M={M} {Nr + two}x{W}", us, 2.0 * (Nr + two) * W, 0, "plain product", like, 2.0 * Nr * W)
        del ws, w2
    sd = z["side"]
    n = 48
    ws, table = [mat(sd, W) for _ in range(n)], mat(1000, sd, s=1.0)
    for M in (1, 8):
        xs, ids = [f32(M, W) for _ in range(n)], torch.zeros(M, dtype=torch.int64, device=dev)
        out = torch.empty(M, sd, device=dev, dtype=bf)
        xb = [x.to(bf) for x in xs]
        us = _graph_us(lambda i: K.gemv_rows(ws[i], xs[i], out, 0, act=K.ACT_GELU_MUL, pdl=True,
                                             args=K.ActArgs(table=table, ids=ids)), n)
        like = _graph_us(lambda i: K.gemv_rows(ws[i], xb[i], out, 0, pdl=True), n)
        add(f"gemv side gate from the stream, gelu, token row M={M} {sd}x{W}", us, 2.0 * sd * W, 0, "plain product", like)
    # --- experts
    E, k, I, Is = z["E"], z["top"], z["eff"], z["sff"]
    n = max(2, min(6, _sets(6.0 * E * I * W)))
    gu, dw = [mat(E, 2 * I, W) for _ in range(n)], [mat(E, W, I) for _ in range(n)]
    sgu, sdw, bias = mat(2 * Is, W), mat(W, Is), torch.zeros(E, device=dev)
    clamp = [X.SoftExpertBank(mat(E, W), gu[i], dw[i], k, shared_gate_up=sgu, shared_down=sdw, act=K.ACT_CLAMP_GLU, limit=7.0,
                              alpha=1.702, shared_limit=7.0, bias=bias, shared_gated=False) for i in range(n)]
    soft = [X.SoftExpertBank(mat(E + 1, W), gu[i], dw[i], k, shared_gate_up=sgu, shared_down=sdw) for i in range(n)]
    for B in (1, 8):
        h, out, logits = mat(B, W, s=1.0), torch.zeros(B, W, device=dev), f32(B, E)
        hit = E * (1 - (1 - k / E) ** B)                   # experts that expect a token
        nb = 6.0 * (hit * I + Is) * W
        us = _graph_us(lambda i: X.soft_moe_rows(clamp[i], h, out, pdl=True, logits=logits, add=True), n)
        like = _graph_us(lambda i: X.soft_moe_rows(soft[i], h, out, pdl=True), n)
        add(f"clamped experts, rows (3 kernels) B={B}", us, nb, 0, "silu experts, rows", like, nb + 2.0 * E * W)
    h, out, logits = [mat(T, W, s=1.0) for _ in range(2)], torch.zeros(T, W, device=dev), f32(T, E)
    fl = 6.0 * T * (k * I + Is) * W
    us = _graph_us(lambda i: X.soft_moe_grouped(clamp[i % n], h[i % 2], out, logits=logits, add=True), 2, launches=6)
    like = _graph_us(lambda i: X.soft_moe_grouped(soft[i % n], h[i % 2], out), 2, launches=6)
    add(f"clamped experts, grouped T={T}", us, 6.0 * (E * I + Is) * W, fl, "silu experts, grouped", like)
    del clamp, soft, gu, dw, sgu, sdw
    # --- attention over window and blocks, one token each
    cos, sin = N.rotary_table(16384, 1e4, ad // 2, dev)
    tab = A.AttnTables(None, cos, sin, torch.ones(ad, device=dev), torch.ones(ad, device=dev))
    pooled = A.AttnSpec(H, G, ad, ad, ad ** -0.5, window=win, pool=P, rot_pairs=ad // 2, unit_eps=1e-6)
    plain = A.AttnSpec(H, G, ad, ad, ad ** -0.5, win, True)
    for B, ctx in ((1, 4 * win), (8, 4 * win), (32, 4 * win)):
        seen = win + (ctx - win) // P
        n = min(32, _sets(4.0 * B * seen * G * ad))
        cache = SlotCache()
        cache.allocate(B, ctx + 8, [KeyValueShape(G, ad, ad), PooledShape(G, ad, ad, P)] * n, bf, dev)
        for layer in cache.layers:
            layer._k.normal_()
            layer._v.normal_()
        qkv, slot, pos = mat(B, pooled.rows, s=1.0), ints(list(range(B))), ints([ctx - 1] * B)
        out = torch.empty(B, H * ad, device=dev, dtype=bf)
        us = _graph_us(lambda i: A.attend_step(pooled, qkv, None, slot, pos, cache, 2 * i, out, pooled.seen(ctx), True, pdl=True,
                                               tables=tab, pooled=2 * i + 1), n)
        like = _graph_us(lambda i: A.attend_step(plain, qkv, None, slot, pos, cache, 2 * i, out, win, True, pdl=True), n)
        add(f"kv_attn pooled, completing a block B={B} ctx={ctx}", us, 4.0 * B * (seen + P) * G * ad, 0, "kv_attn window", like,
            4.0 * B * win * G * ad)
        pos = ints([ctx - 2] * B)
        us = _graph_us(lambda i: A.attend_step(pooled, qkv, None, slot, pos, cache, 2 * i, out, pooled.seen(ctx), True, pdl=True,
                                               tables=tab, pooled=2 * i + 1), n)
        add(f"kv_attn pooled B={B} ctx={ctx}", us, 4.0 * B * seen * G * ad, 0, "kv_attn window", like, 4.0 * B * win * G * ad)
        del cache
    # --- recurrences, one token each
    dH, dD, rank, sH, sV, sN, sG = z["dH"], z["dD"], z["rank"], z["sH"], z["sV"], z["N"], z["sG"]
    gs, ds, ls = R.GeneralDeltaSpec(dH, dD, dD, rank), D.DeltaSpec(dH, dH, dD, dD, TAPS), Li.LinearSpec(dH, dD, dD, 16, 16.0)
    ss = Ss.SSDSpec(sH, sV, sN, sG, TAPS, sG)
    es = D.DeltaSpec(sH, sG, sN, sV, TAPS)               # the delta rule on the state space's sizes
    gw = R.GeneralDeltaWeights(mat(dn, rank), f32(dn), f32(dn), torch.ones(dn, device=dev, dtype=bf), 1e-6)

    def delta_weights(s):
        return D.DeltaWeights(mat(s.channels, TAPS, s=0.5), torch.zeros(s.heads, device=dev), torch.zeros(s.heads, device=dev),
                              torch.ones(s.vdim, device=dev, dtype=bf), 1e-6)
    dwt, ewt = delta_weights(ds), delta_weights(es)
    lw = Li.LinearWeights(mat(dn, 16), f32(dn), torch.ones(dD, device=dev, dtype=bf), 1e-6)
    zeros = torch.zeros(sH, device=dev)
    sw = Ss.SSDWeights(mat(ss.channels, TAPS, s=0.5), torch.zeros(ss.channels, device=dev), zeros, zeros, zeros,
                       torch.ones(ss.inner, device=dev, dtype=bf), 1e-6)
    width = max(gs.rows, ds.rows, ss.rows, es.rows, ls.rows)
    for B in (1, 8, 32):
        slot, pos = ints(list(range(B))), ints([9] * B)
        proj, low, gates = mat(B, width, s=1.0), f32(B, max(rank, sH)), f32(B, 2 * max(dH, sH))
        for name, fn, st, like_name, like_fn, like_st, nb in (
                ("general_step", lambda c, i: R.general_delta_mix(gs, gw, proj[:, :gs.rows], low, slot, pos, c, i, proj[:, gs.gate_at:gs.rows],
                                                                  pdl=True), DeltaStateShape(dH, dD, dD, 0, 0),
                 "delta_step", lambda c, i: D.delta_mix(ds, dwt, proj[:, :ds.rows], gates[:, :2 * dH].contiguous(), slot, pos, c, i, out1, pdl=True),
                 DeltaStateShape(dH, dD, dD, TAPS, ds.channels), 8.0 * B * dH * dD * dD),
                ("ssd_step + grouped norm (2 kernels)", lambda c, i: Ss.ssd_mix(ss, sw, proj[:, :ss.rows], low, slot, pos, c, i, out2, pdl=True),
                 DeltaStateShape(sH, sN, sV, TAPS, ss.channels),
                 "delta_step", lambda c, i: D.delta_mix(es, ewt, proj[:, :es.rows], g2, slot, pos, c, i, out2, pdl=True),
                 DeltaStateShape(sH, sN, sV, TAPS, es.channels), 8.0 * B * sH * sN * sV)):
            n = min(48, _sets(nb / 2))
            cache, other = SlotCache(), SlotCache()
            cache.allocate(B, 64, [st] * n, bf, dev)
            other.allocate(B, 64, [like_st] * n, bf, dev)
            out1, out2 = torch.empty(B, dn, device=dev, dtype=bf), torch.empty(B, ss.inner, device=dev, dtype=bf)
            g2 = gates[:, :2 * sH].contiguous()
            us = _graph_us(lambda i: fn(cache, i), n)
            like = _graph_us(lambda i: like_fn(other, i), n)
            add(f"{name} B={B}", us, nb, 0, like_name, like)
            del cache, other
    # --- prompts
    slot, pos = ints([0] * T), ints(list(range(T)))
    nc = -(-T // Portions.CHUNK)
    where = Portions(ints([0]), ints([T]), T, True, ints([0] * nc), ints([0, nc]), nc, [T])
    cache = SlotCache()
    cache.allocate(1, T + 8, [KeyValueShape(G, ad, ad), PooledShape(G, ad, ad, P), DeltaStateShape(dH, dD, dD, 0, 0),
                              DeltaStateShape(dH, dD, dD, TAPS, ds.channels), DeltaStateShape(sH, sN, sV, TAPS, ss.channels),
                              DeltaStateShape(sH, sN, sV, TAPS, es.channels)], bf, dev)
    n = 6
    qkv, out = [mat(T, pooled.rows, s=1.0) for _ in range(n)], torch.empty(T, H * ad, device=dev, dtype=bf)
    unweighted = A.AttnTables(None, cos, sin)
    for w in (win, win // 4):
        f = A.AttnSpec(H, G, ad, ad, ad ** -0.5, window=w, pool=P, rot_pairs=ad // 2, unit_eps=1e-6)
        p = A.AttnSpec(H, G, ad, ad, ad ** -0.5, window=w, rot_pairs=ad // 2, unit_eps=1e-6)
        us = _graph_us(lambda i: A.attend_prompt(f, qkv[i], None, slot, pos, where.row, where.length, T, cache, 0, out, tab, where, 1), n)
        like = _graph_us(lambda i: A.attend_prompt(p, qkv[i], None, slot, pos, where.row, where.length, T, cache, 0, out, unweighted), n)
        pairs = T * min(w, T) - min(w, T) * (min(w, T) - 1) / 2
        blocks = sum(max(0, i - w + 1) // P for i in range(T))
        add(f"qk_prepare + kv_append + kv_pool + packed_prefill T={T} window={w}", us, 0, 4.0 * H * (pairs + blocks) * ad,
            "the same without blocks", like, 0, 4.0 * H * pairs * ad)
    us = _graph_us(lambda i: A.prepare_heads(pooled, qkv[i], slot, pos, cache, tab), n)
    like = _graph_us(lambda i: A.prepare_heads(pooled, qkv[i], slot, pos, cache, unweighted), n)
    add(f"qk_prepare, weighted norms T={T}", us, 4.0 * T * (H + G) * ad, 0, "unit norms", like)
    us = _graph_us(lambda i: A.pool_blocks(pooled, where, slot, pos, cache, 0, 1), 2)
    add(f"kv_pool T={T}", us, 4.0 * T * G * ad)
    del qkv
    projs = [mat(T, width, s=1.0) for _ in range(4)]
    low, gates = f32(T, max(rank, sH)), f32(T, 2 * max(dH, sH))
    g1, g2 = gates[:, :2 * dH].contiguous(), gates[:, :2 * sH].contiguous()
    out, out2 = torch.empty(T, dn, device=dev, dtype=bf), torch.empty(T, ss.inner, device=dev, dtype=bf)
    l2 = f32(T, 16)
    us = _graph_us(lambda i: R.general_delta_mix(gs, gw, projs[i][:, :gs.rows], low, slot, pos, cache, 2, out, where), 4)
    like = _graph_us(lambda i: D.delta_mix(ds, dwt, projs[i][:, :ds.rows], g1, slot, pos, cache, 3, out, where), 4)
    like2 = _graph_us(lambda i: Li.linear_mix(ls, lw, projs[i][:, :ls.rows], l2, slot, pos, cache, 2, out, where), 4)
    add(f"general_chunks + norm (3 kernels) T={T}", us, 2.0 * T * (gs.rows + dn), 8.0 * T * dH * dD * dD, "delta_chunks", like,
        2.0 * T * (ds.rows + dn), 6.0 * T * dH * dD * dD)
    rows[-1]["linear_chunks_us"] = round(like2, 2)
    us = _graph_us(lambda i: Ss.ssd_mix(ss, sw, projs[i][:, :ss.rows], low, slot, pos, cache, 4, out2, where), 4)
    like = _graph_us(lambda i: D.delta_mix(es, ewt, projs[i][:, :es.rows], g2, slot, pos, cache, 5, out2, where), 4)
    add(f"ssd_chunks + norm (5 kernels) T={T}", us, 2.0 * T * (ss.rows + ss.inner), 4.0 * T * sH * sN * sV, "delta_chunks", like,
        2.0 * T * (es.rows + es.heads * es.vdim), 6.0 * T * sH * sN * sV)
    raw = f32(T, ss.inner)
    us = _graph_us(lambda i: gated_group_norm(raw, projs[i][:, ss.channels:ss.rows], sw.norm, out2, sG, 1e-6), 4)
    like = _graph_us(lambda i: gated_norm(raw.view(T, sH, sV), projs[i][:, ss.channels:ss.rows], torch.ones(sV, device=dev, dtype=bf), out2, 1e-6), 4)
    add(f"gated_group_norm T={T}", us, 8.0 * T * ss.inner, 0, "gated_norm", like)
    nf = 5 * dn + z["ff"]
    n = _sets(2.0 * (nf + T) * W)
    ws, xk = [mat(nf, W) for _ in range(n)], [mat(T, W, s=1.0) for _ in range(n)]
    out, w2, o2 = torch.empty(T, nf, device=dev, dtype=bf), mat(rank, W), torch.empty(T, rank, device=dev)
    us = _graph_us(lambda i: K.gemm(xk[i], ws[i], out, 0, K.ACT_RELU2, w2=w2, out2=o2, args=K.ActArgs(start=5 * dn)), n)
    like = _graph_us(lambda i: K.gemm(xk[i], ws[i], out, 0), n)
    add(f"gemm delta projection, hidden units, low rank {T}x{nf + rank}x{W}", us, 0, 2.0 * T * (nf + rank) * W, "plain product", like, 0,
        2.0 * T * nf * W)
    sg, ids = mat(sd, W), torch.zeros(T, dtype=torch.int64, device=dev)
    out = torch.empty(T, sd, device=dev, dtype=bf)
    us = _graph_us(lambda i: K.gemm(xk[i], sg, out, 0, K.ACT_GELU_MUL, args=K.ActArgs(table=table, ids=ids)), n)
    like = _graph_us(lambda i: K.gemm(xk[i], sg, out, 0), n)
    add(f"gemm side gate, gelu, token row {T}x{sd}x{W}", us, 2.0 * T * W, 2.0 * T * sd * W, "plain product", like)
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
            for label, cfg in (("gegorax", gegorax_config(z, "dp", True)), ("gegorax_delta", gegorax_config(z, "d")),
                               ("gegorax_two_sided", gegorax_config(z, "p")), ("letarax", letarax_config(z)),
                               ("dodilix_two_sided", dodilix_config(z))):
                r[label] = run_model(cfg, a.prompt, (1, 8, 32), a.iters)
        if a.kernels:
            r["kernels"] = kernels(z, a.prompt, peaks)
        res["sizes"][name] = r
    if timed is not None:
        timed[1]()
    last = a.sizes.split(",")[-1]
    if "gegorax" in res["sizes"][last]:
        m = res["sizes"][last]["gegorax"]
        res.update(model=f"gegorax-{last} ({m['params_m']:.0f} M, {SIZES[last]['layers']} layers)", unit="tokens/s",
                   value=m["decode_tok_s"][1], ms_per_step=m["decode_ms"][1])
    if a.json:
        with open(a.json, "w") as f:
            json.dump(res, f, indent=1)
    return res


if __name__ == "__main__":
    print(json.dumps(run(), indent=1))
