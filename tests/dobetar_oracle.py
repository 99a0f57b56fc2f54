"""Plain, slow, float64 implementation of the Dobetar decoder, one function per mechanism.

It shares nothing with the product path: it takes a dictionary of tensors under their checkpoint names and the raw
``config.json`` dictionary, and recomputes every position of one sequence from its token ids.  Used as the yard-stick
of the CUDA kernels and engine; ``faults`` lets a test plant one mistake in a mechanism to prove that a comparison
would notice it.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def rms_norm(x, w, eps):
    """x / sqrt(mean(x^2) + eps) * w over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def bigram_rows(tokens, buckets, mul_prev, mul_cur):
    """Row of the bigram table of every token; the first token of a sequence takes the extra last row."""
    rows = []
    for i, t in enumerate(tokens):
        rows.append(buckets if i == 0 else (int(tokens[i - 1]) * mul_prev + int(t) * mul_cur) % buckets)
    return rows


def embed(w, cfg, tokens):
    e = cfg["embedding"]
    x = w["embed"][torch.as_tensor(list(tokens))] * e["scale"]
    b = e.get("bigram")
    if b:
        x = x + w["bigram"][torch.as_tensor(bigram_rows(tokens, b["buckets"], b["mul_prev"], b["mul_cur"]))]
    return x


def rotate_half_pairs(x, positions, base, dims):
    """Pairs (i, i + dims/2) of the first ``dims`` entries turn by position * base^(-2i/dims); the rest pass."""
    out = x.clone()
    half = dims // 2
    for i in range(half):
        a = positions.to(F64) * base ** (-2.0 * i / dims)
        a = a.view(-1, *([1] * (x.dim() - 2)))
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * torch.cos(a) - v * torch.sin(a)
        out[..., i + half] = v * torch.cos(a) + u * torch.sin(a)
    return out


def window_visible(n, size):
    """[n, n] boolean: query i sees key j when 0 <= i - j < size (all earlier keys without a size)."""
    d = torch.arange(n).view(-1, 1) - torch.arange(n).view(1, -1)
    return (d >= 0) & (d < size) if size else d >= 0


def latent_mix(q, kv, w_norm, w_uk, w_uv, m, eps, faults=()):
    """Attention of one sequence from its projections: ``q [n, H, dim + rot_dim]``, ``kv [n, kv_rank + rot_dim]``.
    Returns the heads' outputs ``[n, H, vdim]``."""
    n = q.shape[0]
    H, dim, rd, vd, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(n)
    c = rms_norm(kv[:, :R], w_norm, eps)
    q_rot, k_rot = q[:, :, dim:], kv[:, R:]
    rot = m.get("rot")
    if rot and rd:
        q_rot = rotate_half_pairs(q_rot, pos, float(rot["base"]), rot["dims"])
        k_rot = rotate_half_pairs(k_rot, pos, float(rot["base"]), rot["dims"])
    k = (c @ w_uk.T).view(n, H, dim)
    v = (c @ w_uv.T).view(n, H, vd)
    size = (m.get("mask") or {}).get("size")
    if size:
        size += ("window_plus_one" in faults) - ("window_minus_one" in faults)
    s = torch.einsum("ihd,jhd->hij", q[:, :, :dim], k) + torch.einsum("ihd,jd->hij", q_rot, k_rot)
    s = (s * m["scale"]).masked_fill(~window_visible(n, size), -math.inf)
    return torch.einsum("hij,jhd->ihd", torch.softmax(s, -1), v)


def latent_attention(w, pre, m, h, eps, faults=()):
    """Multi-head latent attention of one sequence ``h [n, width]`` (already normed); returns the mixer's output."""
    n = h.shape[0]
    q = (h @ w[pre + "q"].T).view(n, m["heads"], m["dim"] + m["rot_dim"])
    o = latent_mix(q, h @ w[pre + "dkv"].T, w[pre + "dkv.norm"], w[pre + "uk"], w[pre + "uv"], m, eps, faults)
    return o.reshape(n, -1) @ w[pre + "o"].T


def squared_relu_mlp(w, pre, h):
    return torch.relu(h @ w[pre + "up"].T) ** 2 @ w[pre + "down"].T


def expert(w, pre, x, limit):
    """Clamped gated unit: min(gate, limit) * sigmoid(1.702 gate) * (clamp(up) + 1)."""
    g = torch.clamp(x @ w[pre + "gate"].T, max=limit)
    u = torch.clamp(x @ w[pre + "up"].T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ w[pre + "down"].T


def route(w, pre, h, top):
    """Sigmoid scores; the ``top`` largest choose, and stay the weights as they are."""
    s = torch.sigmoid(h @ w[pre + "router"].T)
    val, idx = torch.topk(s, top, dim=-1)
    return val, idx


def moe_mlp(w, pre, p, h, faults=()):
    val, idx = route(w, pre, h, p["router"]["top"])
    if "renormalized" in faults:
        val = val / val.sum(-1, keepdim=True)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for s, e in zip(val[t], idx[t]):
            if "weight_on_output" in faults:
                out[t] += s * expert(w, f"{pre}e{int(e)}.", h[t:t + 1], p["expert"]["limit"])[0]
            else:
                out[t] += expert(w, f"{pre}e{int(e)}.", s * h[t:t + 1], p["expert"]["limit"])[0]
    return out


def softcap(z, cap):
    return cap * torch.tanh(z / cap) if cap else z


def forward(weights, cfg, tokens, dtype=F64, faults=(), trace=None):
    """Logits ``[n, vocab]`` of one sequence; ``trace`` (a list) collects the residual after every layer."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = embed(w, cfg, tokens)
    for i, layer in enumerate(cfg["layers"]):
        pre = f"l{i}."
        x = x + latent_attention(w, pre + "mix.", layer["mixer"], rms_norm(x, w[pre + "norm1"], eps), eps, faults)
        p = layer.get("mlp")
        if p:
            h = rms_norm(x, w[pre + "norm2"], eps)
            x = x + (squared_relu_mlp(w, pre + "mlp.", h) if p["kind"] == "dense"
                     else moe_mlp(w, pre + "mlp.", p, h, faults))
        if trace is not None:
            trace.append(x.clone())
    return softcap(rms_norm(x, w["final.norm"], eps) @ w["head"].T, cfg.get("logit_softcap"))


def greedy(weights, cfg, tokens, n):
    """``n`` greedy continuation tokens, every step recomputed from the whole sequence."""
    seq = list(tokens)
    for _ in range(n):
        seq.append(int(forward(weights, cfg, seq)[-1].argmax()))
    return seq[len(tokens):]


# ------------------------------------------------------------------------------------------------
# random models
# ------------------------------------------------------------------------------------------------
def latent_layer(heads=4, dim=32, rot_dim=16, vdim=24, kv_rank=64, window=11, base=10000.0, mlp=None, scale=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
                      "mask": {"size": window}, "rot": {"base": base, "dims": rot_dim},
                      "scale": scale if scale is not None else (dim + rot_dim) ** -0.5}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, limit=1.5):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def random_weights(cfg, seed=0, sharp=2.5):
    """Checkpoint tensors of ``cfg`` (bf16-representable fp32): projections keep unit variance, queries are scaled by
    ``sharp`` so that the attention is far from uniform."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]

    def mat(n, k, gain=1.0):
        return (torch.randn(n, k, generator=g) * gain / math.sqrt(k)).bfloat16().float()

    def norm(n):
        return (1.0 + 0.2 * torch.randn(n, generator=g)).bfloat16().float()

    w = {"embed": mat(cfg["vocab"], W, math.sqrt(W)), "final.norm": norm(W), "head": mat(cfg["vocab"], W, 2.0)}
    b = cfg["embedding"].get("bigram")
    if b:
        w["bigram"] = mat(b["buckets"] + 1, W, 2.0 * math.sqrt(W))
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        H, R = m["heads"], m["kv_rank"]
        w[p + "norm1"] = norm(W)
        w[p + "mix.q"] = mat(H * (m["dim"] + m["rot_dim"]), W, sharp)
        w[p + "mix.dkv"] = mat(R + m["rot_dim"], W)
        w[p + "mix.dkv.norm"] = norm(R)
        w[p + "mix.uk"] = mat(H * m["dim"], R)
        w[p + "mix.uv"] = mat(H * m["vdim"], R)
        w[p + "mix.o"] = mat(W, H * m["vdim"])
        f = layer.get("mlp")
        if not f:
            continue
        w[p + "norm2"] = norm(W)
        if f["kind"] == "dense":
            w[p + "mlp.up"], w[p + "mlp.down"] = mat(f["ff"], W), mat(W, f["ff"])
        else:
            w[p + "mlp.router"] = mat(f["router"]["experts"], W, 2.0)
            for e in range(f["router"]["experts"]):
                q = f"{p}mlp.e{e}."
                ff = f["expert"]["ff"]
                w[q + "gate"], w[q + "up"], w[q + "down"] = mat(ff, W, 2.0), mat(ff, W, 2.0), mat(W, ff)
    return w
