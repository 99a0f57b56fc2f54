"""Plain, slow, float64 implementation of the Gegorax decoder, one function per mechanism.

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


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# ------------------------------------------------------------------------------------------------
# attention over a window and pooled blocks
# ------------------------------------------------------------------------------------------------
def turn_neighbours(x, positions, base, dims, faults=()):
    """Entries 2i and 2i + 1 of the first ``dims`` of ``x [n, ..., D]`` turn by position * base^(-2i / dims)."""
    out = x.clone()
    for i in range(dims // 2):
        a, b = (i, i + dims // 2) if "other_pairs" in faults else (2 * i, 2 * i + 1)
        ang = (positions.to(F64) * float(base) ** (-2.0 * i / dims)).to(x.dtype).view(-1, *([1] * (x.dim() - 2)))
        u, v = x[..., a], x[..., b]
        out[..., a] = u * torch.cos(ang) - v * torch.sin(ang)
        out[..., b] = v * torch.cos(ang) + u * torch.sin(ang)
    return out


def visible(n, size, pool, faults=()):
    """Which of ``n`` tokens, and which of the blocks of ``pool`` tokens, every position sees: ``[n, n]``, ``[n, blocks]``."""
    if "window_plus_one" in faults:
        size += 1
    if "window_minus_one" in faults:
        size -= 1
    i, j = torch.arange(n).view(-1, 1), torch.arange(n).view(1, -1)
    tokens = (j <= i) & (i - j < size)
    if not pool or "no_blocks" in faults:
        return tokens, torch.zeros(n, 0, dtype=torch.bool)
    last = torch.arange(n // pool).view(1, -1) * pool + pool - 1
    early = {"block_early": 1, "block_late": -1}
    shift = sum(v for k, v in early.items() if k in faults)
    blocks = last <= i - size + shift
    if "partial_blocks" in faults:                 # a block counts as soon as its first token has left
        blocks = last - pool + 1 <= i - size
    return tokens, blocks


def pooled_attend(q, k, v, m, wq, wk, eps, faults=()):
    """``q [n, H, dim]``, ``k [n, G, dim]`` before norm and rotation, ``v [n, G, vdim]`` -> ``[n, H, vdim]``."""
    n, H, G = q.shape[0], q.shape[1], k.shape[1]
    mask = m.get("mask") or {}
    size, P = int(mask.get("size") or n), int(mask.get("pool") or 0)
    rot = m.get("rot") or {"base": 1.0, "dims": 0}
    turn = (lambda x: x) if "no_rotation" in faults else \
        (lambda x: turn_neighbours(x, torch.arange(n), rot["base"], rot["dims"], faults))
    if "norm_after_rotation" in faults:
        q, k = rms(turn(q), eps) * wq, rms(turn(k), eps) * wk
    else:
        if "no_norm" not in faults:
            q, k = rms(q, eps) * wq, rms(k, eps) * wk
        q, k = turn(q), turn(k)
    tokens, blocks = visible(n, size, P, faults)
    nb = blocks.shape[1]
    if nb:
        kb = k[:nb * P].view(nb, P, G, -1).mean(1)
        vb = v[:nb * P].view(nb, P, G, -1).mean(1)
        if "block_sums" in faults:
            kb = kb * P
        keys, vals, see = torch.cat([k, kb]), torch.cat([v, vb]), torch.cat([tokens, blocks], 1)
    else:
        keys, vals, see = k, v, tokens
    head = torch.arange(H) % G if "heads_interleaved" in faults else torch.arange(H) // (H // G)
    s = torch.einsum("ihd,jhd->hij", q, keys[:, head]) * m["scale"]
    p = torch.softmax(s.masked_fill(~see, float("-inf")), -1)
    return torch.einsum("hij,jhd->ihd", p, vals[:, head])


def pooled_attention(w, pre, m, h, eps, faults=()):
    n = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    o = pooled_attend((h @ w[pre + "q"].T).view(n, H, D), (h @ w[pre + "k"].T).view(n, G, D),
                      (h @ w[pre + "v"].T).view(n, G, V), m, w[pre + "q.norm"], w[pre + "k.norm"], eps, faults)
    return o.reshape(n, H * V) @ w[pre + "o"].T


# ------------------------------------------------------------------------------------------------
# state-space duality
# ------------------------------------------------------------------------------------------------
def short_conv(x, taps, bias):
    """``x [n, channels]``, ``taps [channels, T]`` (the last one the token's own), zeros before the first token."""
    n, T = x.shape[0], taps.shape[1]
    y = bias.expand_as(x).clone()
    for back in range(min(T, n)):
        y[back:] += x[:n - back] * taps[:, T - 1 - back]
    return y


def ssd_rule(x, B, C, dt, a_log, D, state=None, faults=()):
    """``x [n, H, vdim]``, ``B, C [n, G, N]``, ``dt [n, H]`` (positive) -> ``[n, H, vdim]``, last state ``[H, N, vdim]``."""
    n, H, V = x.shape
    G, N = B.shape[1], B.shape[2]
    head = torch.arange(H) % G if "groups_interleaved" in faults else torch.arange(H) // (H // G)
    S = torch.zeros(H, N, V, dtype=x.dtype) if state is None else state
    out = []
    for t in range(n):
        old = S
        S = torch.exp(-torch.exp(a_log) * dt[t]).view(H, 1, 1) * S
        step = torch.ones_like(dt[t]) if "unscaled_input" in faults else dt[t]
        S = S + step.view(H, 1, 1) * B[t, head].unsqueeze(-1) * x[t].unsqueeze(-2)
        y = torch.einsum("hnv,hn->hv", old if "read_before_write" in faults else S, C[t, head])
        out.append(y if "no_skip" in faults else y + D.view(H, 1) * x[t])
    return torch.stack(out), S


def gated_group_norm(y, z, weight, parts, eps, faults=()):
    if "gate_after_norm" in faults:
        return rms(y.unflatten(-1, (parts, -1)), eps).flatten(-2) * weight * silu(z)
    if "one_norm_group" in faults:
        parts = 1
    return rms((y * silu(z)).unflatten(-1, (parts, -1)), eps).flatten(-2) * weight


def ssd(w, pre, m, h, eps, faults=()):
    n = h.shape[0]
    H, V, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * V
    z, xbc, dt = (h @ w[pre + "in"].T).split([inner, inner + 2 * G * N, H], 1)
    xbc = short_conv(xbc, w[pre + "conv"], torch.zeros_like(w[pre + "conv.b"]) if "no_conv_bias" in faults else w[pre + "conv.b"])
    x, B, C = silu(xbc).split([inner, G * N, G * N], 1)
    dt = torch.nn.functional.softplus(dt + w[pre + "dt_bias"], threshold=1e9)
    y, _ = ssd_rule(x.view(n, H, V), B.view(n, G, N), C.view(n, G, N), dt, w[pre + "A_log"], w[pre + "D"], faults=faults)
    return gated_group_norm(y.flatten(1), z, w[pre + "norm"], m["norm_groups"], eps, faults) @ w[pre + "o"].T


def parallel(w, pre, m, h, eps, faults=()):
    a = pooled_attention(w, pre + "left.", m["left"], h, eps, faults)
    b = ssd(w, pre + "right.", m["right"], h, eps, faults)
    if "sides_unnormed" in faults:
        return 0.5 * (a * w[pre + "left.out"] + b * w[pre + "right.out"])
    return 0.5 * (rms(a, eps) * w[pre + "left.out"] + rms(b, eps) * w[pre + "right.out"])


# ------------------------------------------------------------------------------------------------
# generalized delta rule
# ------------------------------------------------------------------------------------------------
def channel_decay(z):
    return torch.exp(-math.exp(-0.5) * torch.sigmoid(z))


def general_delta_rule(r, k, v, w, a, state=None, faults=()):
    """``r, k, w, a [n, H, D]``, ``v [n, H, V]`` -> outputs ``[n, H, V]`` and the last state ``[H, D, V]``."""
    n, H, D = r.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=r.dtype) if state is None else state
    u = k if "no_unit_key" in faults else k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
    out = []
    for t in range(n):
        old = S
        kept = w[t].unsqueeze(-1) * S
        seen = torch.einsum("hd,hdv->hv", u[t], kept if "removal_after_decay" in faults else S)
        rate = a[t].mean(-1, keepdim=True).expand_as(a[t]) if "one_rate_per_head" in faults else a[t]
        S = kept - (rate * u[t]).unsqueeze(-1) * seen.unsqueeze(-2)
        if "no_removal" in faults:
            S = kept
        S = S + (u if "unit_write" in faults else k)[t].unsqueeze(-1) * v[t].unsqueeze(-2)
        out.append(torch.einsum("hdv,hd->hv", old if "read_before_write" in faults else S, r[t]))
    return torch.stack(out), S


def general_delta(w, pre, m, h, eps, faults=()):
    n, H, D = h.shape[0], m["heads"], m["dim"]
    r, k, v = ((h @ w[pre + c].T).view(n, H, D) for c in "rkv")
    low = h @ w[pre + "w1"].T
    if "no_tanh" not in faults:
        low = torch.tanh(low)
    decay = channel_decay(low @ w[pre + "w2"].T + w[pre + "w0"]).view(n, H, D)
    if "one_decay_per_head" in faults:
        decay = decay.mean(-1, keepdim=True).expand_as(decay)
    rate = torch.sigmoid(h @ w[pre + "a"].T + w[pre + "a.b"]).view(n, H, D)
    o, _ = general_delta_rule(r, k, v, decay, rate, faults=faults)
    o = rms(o, eps).reshape(n, H * D) * w[pre + "norm"]
    g = h @ w[pre + "g"].T
    return (o * (silu(g) if "silu_gate" in faults else torch.sigmoid(g))) @ w[pre + "o"].T


# ------------------------------------------------------------------------------------------------
# feed-forward
# ------------------------------------------------------------------------------------------------
def dense_unit(w, pre, h):
    return torch.relu(h @ w[pre + "up"].T) ** 2 @ w[pre + "down"].T


def clamped_unit(w, pre, h, limit, faults=()):
    g, u = h @ w[pre + "gate"].T, h @ w[pre + "up"].T
    if "no_clamp" not in faults:
        g, u = torch.clamp(g, max=limit), torch.clamp(u, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + (0.0 if "no_plus_one" in faults else 1.0))) @ w[pre + "down"].T


def route(z, top, faults=()):
    """Router logits (bias included) ``[n, E]`` -> weights and experts ``[n, top]``."""
    val, idx = z.topk(top, -1)
    if "softmax_over_all" in faults:
        return torch.softmax(z, -1).gather(-1, idx), idx
    return torch.softmax(val, -1), idx


def experts(w, pre, p, h, faults=()):
    z = h @ w[pre + "router"].T
    if "no_router_bias" not in faults:
        z = z + w[pre + "router.b"]
    val, idx = route(z, p["router"]["top"], faults)
    out = torch.zeros_like(h)
    for e in range(p["router"]["experts"]):
        t, j = torch.nonzero(idx == e, as_tuple=True)
        if len(t):
            out[t] += val[t, j, None] * clamped_unit(w, f"{pre}e{e}.", h[t], p["expert"]["limit"], faults)
    if p.get("shared") and "no_shared" not in faults:
        limit = p["expert" if "shared_limit" in faults else "shared"]["limit"]
        out = out + clamped_unit(w, pre + "shared.", h, limit, faults)
    return out


def feed_forward(w, pre, p, h, faults=()):
    return dense_unit(w, pre, h) if p["kind"] == "dense" else experts(w, pre, p, h, faults)


# ------------------------------------------------------------------------------------------------
# model
# ------------------------------------------------------------------------------------------------
def token_side(w, pre, x, e, eps):
    """What a layer's own embedding ``e [n, dim]`` of the token adds to the stream."""
    y = (gelu_tanh(x @ w[pre + "gate"].T) * e) @ w[pre + "proj"].T
    return rms(y, eps) * w[pre + "norm"]


def forward(weights, cfg, tokens, dtype=F64, faults=(), trace=None):
    """Logits ``[n, vocab]`` of one sequence; ``trace`` (a list) collects the stream after every layer."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    tokens = torch.as_tensor(list(tokens))
    x = w["embed"][tokens]
    side = (cfg.get("token_side") or {}).get("dim")
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer.get("mlp")
        h = rms(x, eps) * w[p + "norm1"]
        mix = parallel if layer["type"] == "parallel" else general_delta
        y = mix(w, p + "mix.", m, h, eps, faults)
        if f:
            hf = rms(x + y, eps) * w[p + "norm1"] if "sequential" in faults else h
            y = y + feed_forward(w, p + "mlp.", f, hf, faults)
        x = x + y
        if side and "no_side" not in faults:
            part = 0 if "side_of_layer_0" in faults else i
            x = x + token_side(w, p + "side.", x, w["side.embed"][tokens][:, part * side:(part + 1) * side], eps)
        if trace is not None:
            trace.append(x)
    return (rms(x, eps) * w["final.norm"]) @ w["head"].T


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


def moe(ff, count, top, limit=1.0, shared=None, shared_limit=1.75):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": count, "top": top},
            "shared": {"ff": shared, "limit": shared_limit} if shared else None}


def delta_layer(heads=3, dim=24, mlp=None):
    return {"type": "general_delta", "mixer": {"heads": heads, "dim": dim}, "mlp": mlp}


def parallel_layer(heads=4, kv_heads=2, dim=32, vdim=24, size=21, pool=5, rot=16, base=5000.0, scale=None, rheads=4,
                   rvdim=20, state=12, groups=2, conv=4, norm_groups=2, mlp=None):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size, "pool": pool},
            "rot": {"base": base, "dims": rot}, "scale": scale if scale is not None else dim ** -0.5}
    right = {"heads": rheads, "vdim": rvdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}
    return {"type": "parallel", "mixer": {"left": left, "right": right}, "mlp": mlp}


def random_weights(cfg, seed=0, sharp=2.0, rank=6, spread=1.0):
    """Checkpoint tensors of ``cfg`` (bf16-representable fp32): projections keep unit variance, query norms are scaled by
    ``sharp`` so that the attention is far from uniform.  ``spread`` below 1: a layer's experts have a part in common, so
    that a choice which a rounded input turns around changes little."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]

    def vec(n, gain=0.2, mean=1.0):
        return (mean + gain * torch.randn(n, generator=g)).bfloat16().float()

    def mat(n, k, gain=1.0):
        return (torch.randn(n, k, generator=g) * gain / math.sqrt(k)).bfloat16().float()

    w = {"embed": mat(cfg["vocab"], W, math.sqrt(W)), "final.norm": vec(W), "head": mat(cfg["vocab"], W, 2.0)}
    side = (cfg.get("token_side") or {}).get("dim")
    if side:
        w["side.embed"] = vec(cfg["vocab"] * side * len(cfg["layers"]), 1.0, 0.0).view(cfg["vocab"], -1)
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer.get("mlp")
        w[p + "norm1"] = vec(W)
        pre = p + "mix."
        if layer["type"] == "parallel":
            a, b = m["left"], m["right"]
            H, G, D, V = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            q = pre + "left."
            w[q + "q"], w[q + "k"], w[q + "v"] = mat(H * D, W), mat(G * D, W), mat(G * V, W)
            w[q + "q.norm"], w[q + "k.norm"], w[q + "o"] = vec(D, 0.2 * sharp, sharp), vec(D), mat(W, H * V)
            w[q + "out"] = vec(W)
            q, H, V, N, G = pre + "right.", b["heads"], b["vdim"], b["state"], b["groups"]
            inner, ch = H * V, H * V + 2 * G * N
            w[q + "in"] = mat(2 * inner + 2 * G * N + H, W)
            w[q + "conv"], w[q + "conv.b"] = vec(ch * b["conv"], 0.6, 0.2).view(ch, -1), vec(ch, 0.3, 0.0)
            w[q + "dt_bias"], w[q + "A_log"], w[q + "D"] = vec(H, 1.0, -1.5), vec(H, 1.0, 0.0), vec(H, 0.5)
            w[q + "norm"], w[q + "o"], w[q + "out"] = vec(inner), mat(W, inner), vec(W)
        else:
            n = m["heads"] * m["dim"]
            for c in "rkvga":
                w[pre + c] = mat(n, W)
            w[pre + "a.b"], w[pre + "w0"] = vec(n, 1.0, 0.0), vec(n, 2.0, -2.0)
            w[pre + "w1"], w[pre + "w2"] = mat(rank, W), mat(n, rank, 2.0)
            w[pre + "norm"], w[pre + "o"] = vec(n), mat(W, n)
        if f:
            q = p + "mlp."
            if f["kind"] == "dense":
                w[q + "up"], w[q + "down"] = mat(f["ff"], W), mat(W, f["ff"], 0.8)
            else:
                E, ff = f["router"]["experts"], f["expert"]["ff"]
                w[q + "router"], w[q + "router.b"] = mat(E, W, 1.5), vec(E, 0.7, 0.0)
                common = {"gate": mat(ff, W), "up": mat(ff, W), "down": mat(W, ff)}
                for e in range(E):
                    for c, base in common.items():
                        own = mat(*base.shape)
                        w[f"{q}e{e}.{c}"] = (spread * own + math.sqrt(1.0 - spread ** 2) * base).bfloat16().float()
                if f.get("shared"):
                    s = f["shared"]["ff"]
                    w[q + "shared.gate"], w[q + "shared.up"], w[q + "shared.down"] = mat(s, W), mat(s, W), mat(W, s)
        if side:
            w[p + "side.gate"], w[p + "side.proj"], w[p + "side.norm"] = mat(side, W), mat(W, side), vec(W, 0.2, 0.5)
    return w
