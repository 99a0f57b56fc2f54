"""Plain, slow, float64 implementation of the Dodilix decoder, one function per mechanism.

It shares nothing with the product path: it takes a dictionary of tensors under their checkpoint names and the raw
``config.json`` dictionary, and recomputes every position of one sequence from its token ids, the recurrences token by
token.  Used as the yard-stick of the CUDA kernels and engine; ``faults`` lets a test plant one mistake in a mechanism to
prove that a comparison would notice it.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


# ------------------------------------------------------------------------------------------------
# rotations
# ------------------------------------------------------------------------------------------------
def turn(x, positions, base, dims, pairs):
    """The first ``dims`` entries of ``x [n, ..., D]`` turn by position * base^(-2i / dims); ``pairs``: list of index
    pairs, the i-th of which turns with the i-th frequency."""
    out = x.clone()
    for i, (a, b) in enumerate(pairs):
        ang = (positions.to(F64) * float(base) ** (-2.0 * i / dims)).view(-1, *([1] * (x.dim() - 2)))
        u, v = x[..., a], x[..., b]
        out[..., a] = u * torch.cos(ang) - v * torch.sin(ang)
        out[..., b] = v * torch.cos(ang) + u * torch.sin(ang)
    return out


def turn_half(x, positions, base, dims):
    return turn(x, positions, base, dims, [(i, i + dims // 2) for i in range(dims // 2)])


def turn_neighbours(x, positions, base, dims):
    return turn(x, positions, base, dims, [(2 * i, 2 * i + 1) for i in range(dims // 2)])


# ------------------------------------------------------------------------------------------------
# hyper-connections
# ------------------------------------------------------------------------------------------------
def gather_streams(x, w_in):
    """``x [n, S, W]``: the sublayer's input before its norm."""
    return torch.einsum("nsw,s->nw", x, w_in)


def spread_streams(x, y, mix, w_out, faults=()):
    """New streams from all old ones (``mix [from, to]``) and the sublayer's output ``y [n, W]``."""
    if "mix_transposed" in faults:
        mix = mix.T
    return torch.einsum("nsw,st->ntw", x, mix) + w_out.view(1, -1, 1) * y.unsqueeze(1)


# ------------------------------------------------------------------------------------------------
# attention in chunks, with a learned sink
# ------------------------------------------------------------------------------------------------
def chunk_visible(n, size):
    """[n, n] boolean: query i sees key j <= i of its own chunk of ``size`` positions."""
    i = torch.arange(n)
    return (i.view(-1, 1) >= i.view(1, -1)) & (i.view(-1, 1) // size == i.view(1, -1) // size)


def sink_softmax(s, visible, sink):
    """``s [H, n, n]``, ``sink [H]`` (None: the usual softmax): exp(s) over the visible keys' sum plus exp(sink)."""
    s = s.masked_fill(~visible, -math.inf)
    top = s.amax(-1, keepdim=True)
    if sink is None:
        e = torch.exp(s - top)
        return e / e.sum(-1, keepdim=True)
    z = sink.view(-1, 1, 1).expand_as(top)
    top = torch.maximum(top, z)
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(z - top))


def chunk_attend(q, k, v, m, sink, eps, faults=()):
    """``q [n, H, dim]``, ``k [n, G, dim]``, ``v [n, G, vdim]`` as projected -> ``[n, H, vdim]``."""
    n, H, G = q.shape[0], q.shape[1], k.shape[1]
    pos = torch.arange(n)
    size = m["mask"]["size"] + ("chunk_plus_one" in faults) - ("chunk_minus_one" in faults)
    if "no_rotation" not in faults:
        f = turn_neighbours if "other_pairs" in faults else turn_half
        q, k = (f(t, pos, m["rot"]["base"], m["rot"]["dims"]) for t in (q, k))
    if "no_unit_norm" not in faults:
        q, k = rms(q, eps), rms(k, eps)
    head = torch.arange(H) % G if "heads_interleaved" in faults else torch.arange(H) // (H // G)
    s = torch.einsum("ihd,jhd->hij", q, k[:, head]) * m["scale"]
    p = sink_softmax(s, chunk_visible(n, size), None if "no_sink" in faults else sink)
    return torch.einsum("hij,jhd->ihd", p, v[:, head])


def chunk_attention(w, pre, m, h, eps, faults=()):
    n = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    o = chunk_attend((h @ w[pre + "q"].T).view(n, H, D), (h @ w[pre + "k"].T).view(n, G, D),
                     (h @ w[pre + "v"].T).view(n, G, V), m, w[pre + "sink"], eps, faults).reshape(n, H * V)
    if "no_gate" not in faults:
        o = o * torch.sigmoid(h @ w[pre + "g"].T)
    return o @ w[pre + "o"].T


# ------------------------------------------------------------------------------------------------
# gated linear attention
# ------------------------------------------------------------------------------------------------
def channel_decay(z, tau):
    """sigmoid(z)^(1 / tau), through its logarithm."""
    return torch.exp(torch.nn.functional.logsigmoid(z) / tau)


def linear_rule(q, k, v, alpha, state=None, faults=()):
    """``q, k, alpha [n, H, dim]``, ``v [n, H, vdim]`` -> outputs ``[n, H, vdim]`` and the last state ``[H, dim, vdim]``."""
    n, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=q.dtype) if state is None else state
    out = []
    for t in range(n):
        old = S
        if "decay_after_write" in faults:
            S = alpha[t].unsqueeze(-1) * (S + k[t].unsqueeze(-1) * v[t].unsqueeze(-2))
        else:
            S = alpha[t].unsqueeze(-1) * S + k[t].unsqueeze(-1) * v[t].unsqueeze(-2)
        out.append(torch.einsum("hdv,hd->hv", old if "read_before_write" in faults else S, q[t]))
    return torch.stack(out), S


def linear_attention(w, pre, m, h, eps, faults=()):
    n = h.shape[0]
    H, D, V = m["heads"], m["dim"], m["vdim"]
    q = (h @ w[pre + "q"].T).view(n, H, D) * D ** -0.5
    k, v = (h @ w[pre + "k"].T).view(n, H, D), (h @ w[pre + "v"].T).view(n, H, V)
    z = (h @ w[pre + "a1"].T) @ w[pre + "a2"].T + w[pre + "a2.b"]
    alpha = channel_decay(z.view(n, H, D), m["tau"])
    if "no_decay" in faults:
        alpha = torch.ones_like(alpha)
    if "one_decay_per_head" in faults:
        alpha = alpha.mean(-1, keepdim=True).expand_as(alpha)
    o, _ = linear_rule(q, k, v, alpha, faults=faults)
    o = (rms(o, eps) * w[pre + "norm"]).reshape(n, H * V)
    return (o * silu(h @ w[pre + "g"].T)) @ w[pre + "o"].T


def side_by_side(w, pre, m, h, eps, faults=()):
    return m["left_scale"] * chunk_attention(w, pre + "left.", m["left"], h, eps, faults) + \
        m["right_scale"] * linear_attention(w, pre + "right.", m["right"], h, eps, faults)


# ------------------------------------------------------------------------------------------------
# latent attention
# ------------------------------------------------------------------------------------------------
def latent_rows(w, pre, m, h, eps):
    """Latents and rotated shared key parts of every token: what a layer keeps, and what later ones may borrow."""
    kv = h @ w[pre + "dkv"].T
    R = m["kv_rank"]
    c = rms(kv[:, :R], eps) * w[pre + "dkv.norm"]
    kr = turn_neighbours(kv[:, R:], torch.arange(h.shape[0]), m["rot"]["base"], m["rot_dim"])
    return c, kr


def latent_attend(q, c, kr, w_uk, w_uv, m, faults=()):
    """``q [n, H, dim + rot_dim]`` unrotated -> ``[n, H, vdim]``."""
    n, H, D, V = q.shape[0], m["heads"], m["dim"], m["vdim"]
    f = turn_half if "other_latent_pairs" in faults else turn_neighbours
    qr = f(q[:, :, D:], torch.arange(n), m["rot"]["base"], m["rot_dim"])
    k, v = (c @ w_uk.T).view(n, H, D), (c @ w_uv.T).view(n, H, V)
    s = (torch.einsum("ihd,jhd->hij", q[:, :, :D], k) + torch.einsum("ihd,jd->hij", qr, kr)) * m["scale"]
    i = torch.arange(n)
    p = sink_softmax(s, i.view(-1, 1) >= i.view(1, -1), None)
    return torch.einsum("hij,jhd->ihd", p, v)


def latent_attention(w, pre, m, h, rows, eps, faults=()):
    n = h.shape[0]
    cq = rms(h @ w[pre + "dq"].T, eps) * w[pre + "dq.norm"]
    q = (cq @ w[pre + "uq"].T).view(n, m["heads"], m["dim"] + m["rot_dim"])
    o = latent_attend(q, *rows, w[pre + "uk"], w[pre + "uv"], m, faults).reshape(n, -1)
    if "no_latent_gate" not in faults:
        o = o * torch.sigmoid(h @ w[pre + "g"].T)
    return o @ w[pre + "o"].T


# ------------------------------------------------------------------------------------------------
# feed-forward
# ------------------------------------------------------------------------------------------------
def gated_unit(w, pre, h):
    return (silu(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


def route(z, r, faults=()):
    """Router logits ``z [n, E]`` -> weights and experts ``[n, top]``."""
    s = torch.softmax(z, -1)
    n, E = s.shape
    g = r.get("groups") or {"count": 1, "keep": 1}
    best = s.view(n, g["count"], -1).amax(-1)
    keep = torch.zeros(n, g["count"], dtype=torch.bool).scatter(1, best.topk(g["keep"], -1).indices, True)
    allowed = keep.repeat_interleave(E // g["count"], 1)
    if "no_groups" in faults:
        allowed = torch.ones_like(allowed)
    val, idx = s.masked_fill(~allowed, -1.0).topk(r["top"], -1)
    if "not_renormalized" not in faults:
        val = val / (val.sum(-1, keepdim=True) + 1e-20)
    return val * float(r.get("scale", 1.0)), idx


def experts(w, pre, p, h, faults=()):
    val, idx = route(h @ w[pre + "router"].T, p["router"], faults)
    out = torch.zeros_like(h)
    for e in range(p["router"]["experts"]):
        t, j = torch.nonzero(idx == e, as_tuple=True)
        if len(t):
            out[t] += val[t, j, None] * gated_unit(w, f"{pre}e{e}.", h[t])
    if p.get("shared"):
        gate = torch.sigmoid(h @ w[pre + "shared.sg"].T)
        out = out + (1.0 if "shared_ungated" in faults else gate) * gated_unit(w, pre + "shared.", h)
    return out


# ------------------------------------------------------------------------------------------------
# model
# ------------------------------------------------------------------------------------------------
def forward(weights, cfg, tokens, dtype=F64, faults=(), trace=None):
    """Logits ``[n, vocab]`` of one sequence; ``trace`` (a list) collects the sum of the streams after every layer."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    e = w["embed"][torch.as_tensor(list(tokens))] * cfg["embedding"]["scale"]
    x = e.unsqueeze(1).repeat(1, cfg["streams"], 1)
    rows = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]

        def sublayer(x, q, f):
            h = rms(gather_streams(x, w[f"{p}hc{q}.in"]), eps) * w[f"{p}norm{q}"]
            return spread_streams(x, f(h), w[f"{p}hc{q}.mix"], w[f"{p}hc{q}.out"], faults)

        def mixer(h):
            if layer["type"] == "parallel":
                return side_by_side(w, p + "mix.", m, h, eps, faults)
            src = m.get("kv_from")
            rows[i] = latent_rows(w, p + "mix.", m, h, eps) if src is None else rows[src]
            return latent_attention(w, p + "mix.", m, h, rows[i], eps, faults)

        x = sublayer(x, 1, mixer)
        f = layer.get("mlp")
        if f:
            x = sublayer(x, 2, lambda h: gated_unit(w, p + "mlp.", h) if f["kind"] == "dense"
                         else experts(w, p + "mlp.", f, h, faults))
        if trace is not None:
            trace.append(x.sum(1))
    return (rms(x.sum(1), eps) * w["final.norm"]) @ w["head"].T * cfg["logit_scale"]


def greedy(weights, cfg, tokens, n):
    """``n`` greedy continuation tokens, every step recomputed from the whole sequence."""
    seq = list(tokens)
    for _ in range(n):
        seq.append(int(forward(weights, cfg, seq)[-1].argmax()))
    return seq[len(tokens):]


# ------------------------------------------------------------------------------------------------
# random models
# ------------------------------------------------------------------------------------------------
def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, count, top, groups=None, scale=1.0, shared=None):
    return {"kind": "moe", "expert": {"ff": ff},
            "router": {"experts": count, "top": top, "scale": scale,
                       "groups": {"count": groups[0], "keep": groups[1]} if groups else {"count": 1, "keep": 1}},
            "shared": {"ff": shared} if shared else None}


def latent_layer(heads=4, dim=24, rot_dim=16, vdim=32, q_rank=40, kv_rank=64, base=10000.0, scale=None, kv_from=None,
                 mlp=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
         "rot": {"base": base, "dims": rot_dim}, "scale": scale if scale is not None else (dim + rot_dim) ** -0.5}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mlp": mlp, "mixer": m}


def parallel_layer(heads=4, kv_heads=2, dim=32, vdim=24, chunk=21, rot=16, base=5000.0, scale=None, lheads=3, ldim=16,
                   lvdim=24, tau=8.0, left_scale=0.7, right_scale=0.9, mlp=None):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": chunk},
            "rot": {"base": base, "dims": rot}, "scale": scale if scale is not None else dim ** -0.5}
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": left, "right": {"heads": lheads, "dim": ldim, "vdim": lvdim, "tau": tau},
                      "left_scale": left_scale, "right_scale": right_scale}}


def random_weights(cfg, seed=0, sharp=2.5, rank=6, spread=1.0):
    """Checkpoint tensors of ``cfg`` (bf16-representable fp32): projections keep unit variance, queries are scaled by
    ``sharp`` so that the attention is far from uniform; decays reach from a few tokens to hundreds.  ``spread`` below 1: a
    layer's experts have a part in common, so that a choice which a rounded input turns around changes little."""
    g = torch.Generator().manual_seed(seed)
    W, S = cfg["width"], cfg["streams"]

    def vec(n, gain=0.2, mean=1.0):
        return (mean + gain * torch.randn(n, generator=g)).bfloat16().float()

    def mat(n, k, gain=1.0):
        return (torch.randn(n, k, generator=g) * gain / math.sqrt(k)).bfloat16().float()

    w = {"embed": mat(cfg["vocab"], W, math.sqrt(W)), "final.norm": vec(W), "head": mat(cfg["vocab"], W, 2.0)}

    def hyper(p, q):
        w[f"{p}norm{q}"] = vec(W)
        w[f"{p}hc{q}.in"], w[f"{p}hc{q}.out"] = vec(S, 0.3, 1.0 / S), vec(S, 0.3)
        w[f"{p}hc{q}.mix"] = (0.8 * torch.eye(S) + 0.25 * torch.randn(S, S, generator=g)).bfloat16().float()

    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        hyper(p, 1)
        if layer["type"] == "parallel":
            a, b = m["left"], m["right"]
            pre = p + "mix.left."
            w[pre + "q"], w[pre + "k"] = mat(a["heads"] * a["dim"], W, sharp), mat(a["kv_heads"] * a["dim"], W)
            w[pre + "v"], w[pre + "g"] = mat(a["kv_heads"] * a["vdim"], W), mat(a["heads"] * a["vdim"], W)
            w[pre + "o"], w[pre + "sink"] = mat(W, a["heads"] * a["vdim"]), vec(a["heads"], 1.0, 1.5)
            pre = p + "mix.right."
            for c in "qk":
                w[pre + c] = mat(b["heads"] * b["dim"], W)
            for c in "vg":
                w[pre + c] = mat(b["heads"] * b["vdim"], W)
            w[pre + "o"], w[pre + "norm"] = mat(W, b["heads"] * b["vdim"]), vec(b["vdim"])
            w[pre + "a1"], w[pre + "a2"] = mat(rank, W), mat(b["heads"] * b["dim"], rank, 2.0)
            w[pre + "a2.b"] = vec(b["heads"] * b["dim"], 1.5, 1.0)
        else:
            pre, H = p + "mix.", m["heads"]
            w[pre + "dq"], w[pre + "dq.norm"] = mat(m["q_rank"], W), vec(m["q_rank"])
            w[pre + "uq"] = mat(H * (m["dim"] + m["rot_dim"]), m["q_rank"], sharp)
            if m.get("kv_from") is None:
                w[pre + "dkv"], w[pre + "dkv.norm"] = mat(m["kv_rank"] + m["rot_dim"], W), vec(m["kv_rank"])
            w[pre + "uk"], w[pre + "uv"] = mat(H * m["dim"], m["kv_rank"]), mat(H * m["vdim"], m["kv_rank"])
            w[pre + "g"], w[pre + "o"] = mat(H * m["vdim"], W), mat(W, H * m["vdim"])
        f = layer.get("mlp")
        if not f:
            continue
        hyper(p, 2)

        def unit(q, ff):
            w[q + "gate"], w[q + "up"], w[q + "down"] = mat(ff, W), mat(ff, W), mat(W, ff)

        if f["kind"] == "dense":
            unit(p + "mlp.", f["ff"])
        else:
            E = f["router"]["experts"]
            w[p + "mlp.router"] = mat(E, W, 2.0)
            unit(p + "common.", f["expert"]["ff"])
            for e in range(E):
                unit(f"{p}mlp.e{e}.", f["expert"]["ff"])
                for c in ("gate", "up", "down"):
                    own, common = w[f"{p}mlp.e{e}.{c}"], w[f"{p}common.{c}"]
                    w[f"{p}mlp.e{e}.{c}"] = (spread * own + math.sqrt(1.0 - spread ** 2) * common).bfloat16().float()
            for c in ("gate", "up", "down"):
                del w[f"{p}common.{c}"]
            if f.get("shared"):
                unit(p + "mlp.shared.", f["shared"]["ff"])
                w[p + "mlp.shared.sg"] = mat(1, W)
    return w
