"""Multi-stream decoder (Dodilix, bf16, random weights) against the closest models of the framework at equal size.

    python -m ipex_llm_b200.utils.bench_multistream [--sizes mid,large] [--kernels] [--json OUT]

Model runs: prompt throughput (one prompt of ``--prompt`` tokens, device-timed) and decode latency (graph replay) of the
design with latent layers alone (the second half borrows the first half's rows), with two-sided layers alone, and with
both and routed experts; beside them a latent-attention decoder and an attention + recurrence decoder (Dobetar, Letarax) of
the same width, heads and feed-forward bytes, all through ``AutoModelForCausalLM.from_config`` and the engine.  ``--kernels``
times every kernel that is new or does more than before, next to the like kernel of those models on the same shape, with its
distance from the roofline (measured copy bandwidth and GEMM rate of ``MEASURED_PEAKS.json`` when that file is in the
working directory).  Inputs rotate through more than the L2.
"""
from __future__ import annotations

import argparse
import json

import torch

from .bench_latent import VOCAB, _graph_us, _sets, run_model

SIZES = {
    # width, layers, streams; latent: heads, dim, rot_dim, vdim, query and key ranks; two-sided: heads, key / value heads,
    # dim (= vdim), chunk, then heads, dim, vdim of the linear side and its decays' rank; feed-forward, experts, groups, kept
    # groups, chosen experts, expert and shared hidden size
    "small": dict(W=1024, layers=8, S=2, H=16, dim=64, rd=32, vd=64, Rq=384, R=256, G=4, ad=64, chunk=512, lH=16, lD=64, lV=64,
                  rank=16, ff=2816, E=16, groups=4, keep=2, top=2, eff=512, sff=512),
    "mid": dict(W=2048, layers=8, S=2, H=16, dim=128, rd=64, vd=128, Rq=768, R=512, G=4, ad=128, chunk=1024, lH=16, lD=128,
                lV=128, rank=16, ff=5504, E=16, groups=4, keep=2, top=2, eff=1024, sff=1024),
    "large": dict(W=4096, layers=8, S=4, H=32, dim=128, rd=64, vd=128, Rq=1536, R=512, G=8, ad=128, chunk=2048, lH=32, lD=128,
                  lV=128, rank=16, ff=11008, E=32, groups=8, keep=4, top=2, eff=2048, sff=2048),
}


def dodilix_config(z, kinds: str, moe: bool = False):
    """``kinds``: a letter per layer in turn: ``l`` latent, ``b`` latent on the rows of the last ``l``, ``p`` two-sided."""
    from ..models.dodilix import DodilixConfig
    dense = {"kind": "dense", "ff": z["ff"]}
    sparse = {"kind": "moe", "expert": {"ff": z["eff"]}, "shared": {"ff": z["sff"]},
              "router": {"experts": z["E"], "top": z["top"], "scale": 1.0, "groups": {"count": z["groups"], "keep": z["keep"]}}}
    layers, own = [], None
    for i in range(z["layers"]):
        k = kinds[i % len(kinds)]
        if k == "p":
            m = {"left": {"heads": z["H"], "kv_heads": z["G"], "dim": z["ad"], "vdim": z["ad"], "mask": {"size": z["chunk"]},
                          "rot": {"base": 1e4, "dims": z["ad"] // 2}, "scale": z["ad"] ** -0.5},
                 "right": {"heads": z["lH"], "dim": z["lD"], "vdim": z["lV"], "tau": 16.0, "rank": z["rank"]},
                 "left_scale": 0.5, "right_scale": 0.5}
        else:
            m = {"heads": z["H"], "dim": z["dim"], "rot_dim": z["rd"], "vdim": z["vd"], "q_rank": z["Rq"], "kv_rank": z["R"],
                 "rot": {"base": 1e4, "dims": z["rd"]}, "scale": (z["dim"] + z["rd"]) ** -0.5}
            if k == "b":
                m["kv_from"] = own
            else:
                own = i
        layers.append({"type": "parallel" if k == "p" else "latent_attention", "mixer": m, "mlp": sparse if moe and i else dense})
    return DodilixConfig(vocab=VOCAB, width=z["W"], streams=z["S"], norm={"eps": 1e-6}, layers=layers)


def dobetar_config(z):
    """Latent attention with the same feed-forward bytes in two matrices."""
    from ..models.dobetar import DobetarConfig
    mixer = {"heads": z["H"], "dim": z["dim"], "rot_dim": z["rd"], "vdim": z["vd"], "kv_rank": z["R"], "mask": {"size": 0},
             "rot": {"base": 1e4, "dims": z["rd"]}, "scale": (z["dim"] + z["rd"]) ** -0.5}
    return DobetarConfig(vocab=VOCAB, width=z["W"], norm={"eps": 1e-6}, embedding={"scale": 1.0},
                         layers=[{"type": "latent_attention", "mixer": mixer,
                                  "mlp": {"kind": "dense", "ff": z["ff"] * 3 // 2 // 64 * 64}} for _ in range(z["layers"])])


def letarax_config(z):
    from .bench_hybrid import letarax_config as make
    return make(dict(W=z["W"], layers=z["layers"], H=z["H"], G=z["G"], dim=z["ad"], window=z["chunk"], ff=z["ff"], dH=z["lH"],
                     dG=z["lH"], dD=z["lD"], dV=z["lV"]), "da")


def kernels(z, prompt: int, peaks):
    """Rows ``{kernel, us, roofline_us, frac}`` and the like kernel's ``frac`` on the same shape."""
    from ..engine.stream_engine import Portions
    from ..ops import cuda_ops, delta as D, dense_moe as X, latent as N, linear_attn as R, stream as K, window_attn as A
    from ..ops.kv_cache import DeltaStateShape, KeyValueShape, SlotCache
    hbm, tf = peaks.get("hbm_gbs", 6650.0) * 1e3, peaks.get("bf16_tflops", 1590.0) * 1e6     # bytes / us, flop / us
    dev, bf = "cuda", torch.bfloat16
    W, S, H, G, ad, T, rows = z["W"], z["S"], z["H"], z["G"], z["ad"], prompt, []

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

    # --- the joint between two sublayers
    norm, w = torch.ones(W, device=dev), torch.ones(S, device=dev)
    mix = torch.eye(S, device=dev)
    for M in (1, 8, T):
        n = _sets(4.0 * S * M * W)
        xs, ys = [f32(M, S, W) for _ in range(n)], [f32(M, W) for _ in range(n)]
        us = _graph_us(lambda i: K.hyper_joint(xs[i], ys[i], mix, w, w, norm, 1e-6, bf, pdl=True), n)
        like = _graph_us(lambda i: K.add_norm_stream(xs[i][:, 0], ys[i], norm, norm, 1e-6, bf, pdl=True), n)
        add(f"hyper_joint M={M} streams={S}", us, (8.0 * S + 6.0) * M * W, 0, "add_norm_stream", like, 14.0 * M * W)
        del xs, ys
    # --- few-row products with a gated unit, and with fp32 rows riding along
    for name, Nr, two, act, la in (("gemv gate / up, silu", 2 * z["ff"], 0, K.ACT_SILU_GLU, K.ACT_GELU_GLU),
                                   ("gemv two-sided projection + decays", 2 * (H + G) * ad + z["lH"] * 2 * (z["lD"] + z["lV"]),
                                    z["rank"], 0, 0),
                                   ("gemv latent projection + query latent", z["R"] + z["rd"] + H * z["vd"], z["Rq"], 0, 0)):
        n = _sets(2.0 * (Nr + two) * W)
        ws, w2 = [mat(Nr, W) for _ in range(n)], [mat(two, W) for _ in range(n)] if two else [None] * n
        for M in (1, 8):
            x, out = mat(M, W, s=1.0), torch.empty(M, Nr // 2 if act else Nr, device=dev, dtype=bf)
            o2 = torch.empty(M, two, device=dev) if two else None
            us = _graph_us(lambda i: K.gemv_rows(ws[i], x, out, 0, act=act, w2=w2[i], out2=o2, pdl=True), n)
            like = _graph_us(lambda i: K.gemv_rows(ws[i], x, out, 0, act=la, pdl=True), n)
            add(f"{name} M={M} {Nr + two}x{W}", us, 2.0 * (Nr + two) * W, 0, "gelu unit" if act else "without them", like,
                2.0 * Nr * W)
        del ws, w2
    # --- experts
    E, k, I, Is = z["E"], z["top"], z["eff"], z["sff"]
    n = max(2, min(6, _sets(6.0 * E * I * W)))
    gu, dn = [mat(E, 2 * I, W) for _ in range(n)], [mat(E, W, I) for _ in range(n)]
    soft = [X.SoftExpertBank(mat(E + 1, W), gu[i], dn[i], k, z["groups"], z["keep"], 1.0, mat(2 * Is, W), mat(W, Is))
            for i in range(n)]
    hard = [X.ExpertBank(mat(E, W), gu[i], dn[i], k, 7.0, 1.702, True) for i in range(n)]
    nw = torch.ones(W, device=dev, dtype=bf)
    for B in (1, 8):
        h, x, out = mat(B, W, s=1.0), f32(B, W), torch.empty(B, W, device=dev)
        hit = E * (1 - (1 - k / E) ** B)                   # experts that expect a token
        us = _graph_us(lambda i: X.soft_moe_rows(soft[i], h, out, pdl=True), n)
        like = _graph_us(lambda i: X.moe_rows(hard[i], x, nw, 1e-6, pdl=True), n)
        add(f"soft_moe_rows (3 kernels) B={B}", us, 6.0 * (hit * I + Is) * W + 2.0 * E * W, 0, "moe_rows", like,
            6.0 * hit * I * W + 2.0 * E * W)
    h, x, out = [mat(T, W, s=1.0) for _ in range(2)], torch.zeros(T, W, device=dev), torch.empty(T, W, device=dev)
    us = _graph_us(lambda i: X.soft_moe_grouped(soft[i % n], h[i % 2], out), 2, launches=6)
    like = _graph_us(lambda i: X.moe_grouped(hard[i % n], x, h[i % 2]), 2, launches=6)
    add(f"soft_moe_grouped T={T}", us, 6.0 * (E * I + Is) * W, 6.0 * T * (k * I + Is) * W, "moe_grouped", like, 6.0 * E * I * W,
        6.0 * T * k * I * W)
    del soft, hard, gu, dn
    # --- chunked attention, one token each
    cos, sin = N.rotary_table(8192, 1e4, ad // 4, dev)
    tab = A.AttnTables(f32(H), cos, sin)
    full = A.AttnSpec(H, G, ad, ad, ad ** -0.5, sink=True, chunk=z["chunk"], rot_pairs=ad // 4, unit_eps=1e-6, gated=True)
    plain = A.AttnSpec(H, G, ad, ad, ad ** -0.5, z["chunk"], True)
    ctx = z["chunk"]
    for B in (1, 8, 32):
        n = min(32, _sets(4.0 * B * ctx * G * ad))
        cache = SlotCache()
        cache.allocate(B, ctx + 8, [KeyValueShape(G, ad, ad)] * n, bf, dev)
        for layer in cache.layers:
            layer._k.normal_()
            layer._v.normal_()
        qkv, slot, pos = mat(B, full.rows, s=1.0), ints(list(range(B))), ints([ctx - 1] * B)
        out = torch.empty(B, H * ad, device=dev, dtype=bf)
        us = _graph_us(lambda i: A.attend_step(full, qkv, None, slot, pos, cache, i, out, ctx, True, pdl=True, tables=tab), n)
        like = _graph_us(lambda i: A.attend_step(plain, qkv, None, slot, pos, cache, i, out, ctx, True, pdl=True), n)
        add(f"kv_attn rotated, normed, gated B={B} ctx={ctx}", us, 4.0 * B * ctx * G * ad, 0, "kv_attn", like)
        del cache
    # --- linear recurrence, one token each
    lH, lD, lV, rank = z["lH"], z["lD"], z["lV"], z["rank"]
    ls, ds = R.LinearSpec(lH, lD, lV, rank, 16.0), D.DeltaSpec(lH, lH, lD, lV, 4)
    lw = R.LinearWeights(mat(lH * lD, rank), f32(lH * lD), torch.ones(lV, device=dev, dtype=bf), 1e-6)
    dw = D.DeltaWeights(mat(ds.channels, 4, s=0.5), torch.zeros(lH, device=dev), torch.zeros(lH, device=dev),
                        torch.ones(lV, device=dev, dtype=bf), 1e-6)
    for B in (1, 8, 32):
        n = min(48, _sets(4.0 * B * lH * lD * lV))
        cache, other = SlotCache(), SlotCache()
        cache.allocate(B, 64, [DeltaStateShape(lH, lD, lV, 0, 0)] * n, bf, dev)
        other.allocate(B, 64, [DeltaStateShape(lH, lD, lV, 4, ds.channels)] * n, bf, dev)
        proj, low, gates = mat(B, max(ls.rows, ds.rows), s=1.0), f32(B, rank), f32(B, 2 * lH)
        slot, pos = ints(list(range(B))), ints([9] * B)
        out = torch.empty(B, lH * lV, device=dev, dtype=bf)
        us = _graph_us(lambda i: R.linear_mix(ls, lw, proj[:, :ls.rows], low, slot, pos, cache, i, out, pdl=True), n)
        like = _graph_us(lambda i: D.delta_mix(ds, dw, proj[:, :ds.rows], gates, slot, pos, other, i, out, pdl=True), n)
        add(f"linear_step B={B}", us, 8.0 * B * lH * lD * lV, 0, "delta_step", like)
        del cache, other
    # --- latent attention, one token each: gated, and on rows that are there already
    rd, vd, Rk, dim = z["rd"], z["vd"], z["R"], z["dim"]
    spec = N.LatentSpec(H, dim, rd, vd, Rk, 0.1, 0, rd // 2, 1e-6)
    cos, sin = N.rotary_table(8192, 1e4, rd // 2, dev)
    uk, uv, kn = mat(H * dim, Rk), mat(H * vd, Rk), torch.ones(Rk, device=dev, dtype=bf)
    for B in (1, 8, 32):
        n = min(32, _sets(2.0 * B * ctx * (Rk + rd)))
        cache = SlotCache()
        cache.allocate(B, ctx + 8, [spec.row(bf)] * n, bf, dev)
        for layer in cache.layers:
            layer._k.normal_()
        q, kv, g = mat(B, H * (dim + rd), s=1.0), mat(B, Rk + rd, s=1.0), mat(B, H * vd, s=1.0)
        slot, pos = ints(list(range(B))), ints([ctx - 1] * B)
        out = torch.empty(B, H * vd, device=dev, dtype=bf)
        nb = 2.0 * B * ctx * (Rk + rd) + 2.0 * H * (dim + vd) * Rk
        args = (spec, q, uk, uv, kn, cos, sin, slot, pos, cache)
        like = _graph_us(lambda i: N.latent_step(*args, i, out, ctx, pdl=True, kv=kv), n)
        for name, kw in (("gated", {"kv": kv, "gate": g}), ("gated, borrowed rows", {"kv": None, "gate": g})):
            us = _graph_us(lambda i: N.latent_step(*args, i, out, ctx, pdl=True, **kw), n)
            add(f"latent_step (3 kernels) {name} B={B} ctx={ctx}", us, nb, 0, "latent_step", like)
        del cache
    # --- prompts
    slot, pos, row, ln = ints([0] * T), ints(list(range(T))), ints([0]), ints([T])
    cache = SlotCache()
    cache.allocate(1, T + 8, [KeyValueShape(G, ad, ad), spec.row(bf), DeltaStateShape(lH, lD, lV, 0, 0),
                              DeltaStateShape(lH, lD, lV, 4, ds.channels)], bf, dev)
    n = 6
    qkv, out = [mat(T, full.rows, s=1.0) for _ in range(n)], torch.empty(T, H * ad, device=dev, dtype=bf)
    cos, sin = N.rotary_table(8192, 1e4, ad // 4, dev)
    tab = A.AttnTables(tab.sinks, cos, sin)
    for c in (z["chunk"], z["chunk"] // 4):
        f = A.AttnSpec(H, G, ad, ad, ad ** -0.5, sink=True, chunk=c, rot_pairs=ad // 4, unit_eps=1e-6, gated=True)
        p = A.AttnSpec(H, G, ad, ad, ad ** -0.5, c, True)
        us = _graph_us(lambda i: A.attend_prompt(f, qkv[i], None, slot, pos, row, ln, T, cache, 0, out, tab), n)
        like = _graph_us(lambda i: A.attend_prompt(p, qkv[i], None, slot, pos, row, ln, T, cache, 0, out), n)
        wn, whole = min(c, T), T // c
        chunks = whole * c * (c + 1) / 2 + (T - whole * c) * (T - whole * c + 1) / 2
        add(f"qk_prepare + kv_append + packed_prefill T={T} chunk={c}", us, 0, 4.0 * H * chunks * ad,
            "kv_append + packed_prefill, window", like, 0, 4.0 * H * (T * wn - wn * (wn - 1) / 2) * ad)
    us = _graph_us(lambda i: A.prepare_heads(full, qkv[i], slot, pos, cache, tab), n)
    add(f"qk_prepare T={T}", us, 4.0 * T * (H + G) * ad)
    q, kv, g = mat(T, H * (dim + rd), s=1.0), mat(T, Rk + rd, s=1.0), mat(T, H * vd, s=1.0)
    cos, sin = N.rotary_table(8192, 1e4, rd // 2, dev)
    rows_out, out = N.prompt_rows(spec, T, bf, dev), torch.empty(T, H * vd, device=dev, dtype=bf)
    fl = H * T * T * (dim + rd + vd) + 2.0 * T * H * (dim + vd) * Rk
    args = (spec, q, uk, uv, kn, cos, sin, slot, pos, row, ln, T, cache, 1, out)
    like = _graph_us(lambda i: N.latent_prompt(*args, kv=kv, rows_out=rows_out), 2)
    for name, kw in (("gated", {"kv": kv, "gate": g}), ("gated, borrowed rows", {"kv": None, "gate": g})):
        us = _graph_us(lambda i: N.latent_prompt(*args, rows_out=rows_out, **kw), 2)
        add(f"latent_prompt {name} T={T}", us, 0, fl, "latent_prompt", like)
    nc = -(-T // Portions.CHUNK)
    where = Portions(row, ln, T, True, ints([0] * nc), ints([0, nc]), nc)
    projs, low, gates = [mat(T, max(ls.rows, ds.rows), s=1.0) for _ in range(4)], f32(T, rank), f32(T, 2 * lH)
    out = torch.empty(T, lH * lV, device=dev, dtype=bf)
    us = _graph_us(lambda i: R.linear_mix(ls, lw, projs[i][:, :ls.rows], low, slot, pos, cache, 2, out, where), 4)
    like = _graph_us(lambda i: D.delta_mix(ds, dw, projs[i][:, :ds.rows], gates, slot, pos, cache, 3, out, where), 4)
    add(f"linear_chunks + norm (3 kernels) T={T}", us, 2.0 * T * (ls.rows + lH * lV), 4.0 * T * lH * lD * lV, "delta_chunks", like,
        2.0 * T * (ds.rows + lH * lV), 6.0 * T * lH * lD * lV)
    n = _sets(2.0 * (2 * z["ff"] + T) * W)
    ws, xk = [mat(2 * z["ff"], W) for _ in range(n)], [mat(T, W, s=1.0) for _ in range(n)]
    out = torch.empty(T, z["ff"], device=dev, dtype=bf)
    us = _graph_us(lambda i: K.gemm(xk[i], ws[i], out, 0, K.ACT_SILU_GLU), n)
    like = _graph_us(lambda i: K.gemm(xk[i], ws[i], out, 0, K.ACT_GELU_GLU), n)
    add(f"gemm gate / up, silu {T}x{2 * z['ff']}x{W}", us, 0, 4.0 * T * z["ff"] * W, "gelu unit", like)
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
            for label, cfg in (("dodilix", dodilix_config(z, "lppb", True)), ("dodilix_latent", dodilix_config(z, "lb")),
                               ("dodilix_two_sided", dodilix_config(z, "p")), ("dobetar", dobetar_config(z)),
                               ("letarax", letarax_config(z))):
                r[label] = run_model(cfg, a.prompt, (1, 8, 32), a.iters)
        if a.kernels:
            r["kernels"] = kernels(z, a.prompt, peaks)
        res["sizes"][name] = r
    if timed is not None:
        timed[1]()
    last = a.sizes.split(",")[-1]
    if "dodilix" in res["sizes"][last]:
        m = res["sizes"][last]["dodilix"]
        res.update(model=f"dodilix-{last} ({m['params_m']:.0f} M, {SIZES[last]['layers']} layers)", unit="tokens/s",
                   value=m["decode_tok_s"][1], ms_per_step=m["decode_ms"][1])
    if a.json:
        with open(a.json, "w") as f:
            json.dump(res, f, indent=1)
    return res


if __name__ == "__main__":
    print(json.dumps(run(), indent=1))
