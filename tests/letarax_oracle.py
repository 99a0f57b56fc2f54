"""Plain, slow, float64 implementation of the Letarax decoder, one function per mechanism.

It shares nothing with the product path: it takes a dictionary of tensors under their checkpoint names and the raw
``config.json`` dictionary, and recomputes every position of one sequence from its token ids, the recurrences token by
token.  Used as the yard-stick of the CUDA kernels and engine; ``faults`` lets a test plant one mistake in a mechanism to
prove that a comparison would notice it.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64
UNIT_EPS = 1e-6


def rms_norm(x, w, eps):
    """Root-mean-square norm over the last dimension with the weight's distance from one."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * (1.0 + w)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


# ------------------------------------------------------------------------------------------------
# windowed attention with a sink
# ------------------------------------------------------------------------------------------------
def window_visible(n, size):
    """[n, n] boolean: query i sees key j when 0 <= i - j < size (all earlier keys without a size)."""
    d = torch.arange(n).view(-1, 1) - torch.arange(n).view(1, -1)
    return (d >= 0) & (d < size) if size else d >= 0


def sink_softmax(s, visible, sink=True):
    """exp(s) / (1 + sum exp(s)) over the visible keys; without ``sink`` the usual softmax."""
    s = s.masked_fill(~visible, -math.inf)
    top = s.amax(-1, keepdim=True).clamp_min(0.0) if sink else s.amax(-1, keepdim=True)
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + (torch.exp(-top) if sink else 0.0))


def mix_values(v, v_first, lam):
    return (1.0 - lam) * v + lam * v_first


def attend(q, k, v, scale, size, faults=()):
    """``q [n, H, dim]``, ``k [n, G, dim]``, ``v [n, G, vdim]`` -> ``[n, H, vdim]``; consecutive query heads share a
    key head."""
    n, H, G = q.shape[0], q.shape[1], k.shape[1]
    if size:
        size += ("window_plus_one" in faults) - ("window_minus_one" in faults)
    head = torch.arange(H) % G if "heads_interleaved" in faults else torch.arange(H) // (H // G)
    s = torch.einsum("ihd,jhd->hij", q, k[:, head]) * scale
    p = sink_softmax(s, window_visible(n, size), "no_sink" not in faults)
    return torch.einsum("hij,jhd->ihd", p, v[:, head])


def attention(w, pre, m, h, v_first, faults=()):
    """The mixer's output for ``h [n, width]`` and the layer's own values (before any mixing)."""
    n = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[pre + "q"].T + w[pre + "q.b"]).view(n, H, D)
    k = (h @ w[pre + "k"].T + w[pre + "k.b"]).view(n, G, D)
    v = own = (h @ w[pre + "v"].T + w[pre + "v.b"]).view(n, G, V)
    if v_first is not None and "no_value_mixing" not in faults:
        v = mix_values(v, v_first, w[pre + "vmix"])
    o = attend(q, k, v, m["scale"], (m.get("mask") or {}).get("size"), faults)
    return o.reshape(n, H * V) @ w[pre + "o"].T, own


# ------------------------------------------------------------------------------------------------
# gated delta rule
# ------------------------------------------------------------------------------------------------
def short_conv(x, taps):
    """``x [n, channels]``, ``taps [channels, K]``: y_t = sum_j taps[:, j] x_{t - (K - 1) + j}, zeros in front."""
    K = taps.shape[1]
    full = torch.cat([torch.zeros(K - 1, x.shape[1], dtype=x.dtype), x])
    return sum(full[j:j + x.shape[0]] * taps[:, j] for j in range(K))


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + UNIT_EPS)


def delta_gates(b, a, A_log, dt_bias):
    """Write strengths and per-token decays of every head."""
    return torch.sigmoid(b), torch.exp(-torch.exp(A_log) * torch.nn.functional.softplus(a + dt_bias, threshold=1e9))


def delta_rule(q, k, v, beta, g, state=None, faults=()):
    """``q, k [n, H, dim]``, ``v [n, H, vdim]``, ``beta, g [n, H]`` -> outputs ``[n, H, vdim]`` and the last state."""
    n, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=q.dtype) if state is None else state
    out = []
    for t in range(n):
        old = S
        S = g[t].view(H, 1, 1) * S
        u = beta[t].view(H, 1) * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t].unsqueeze(-1) * u.unsqueeze(-2)
        out.append(torch.einsum("hdv,hd->hv", old if "read_before_write" in faults else S, q[t]))
    return torch.stack(out), S


def gated_head_norm(o, gate, w, eps):
    return o / torch.sqrt((o * o).mean(-1, keepdim=True) + eps) * w * silu(gate)


def delta(w, pre, m, h, eps, faults=()):
    n = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    x = {c: silu(short_conv(h @ w[pre + c].T, w[f"{pre}{c}.conv"])) for c in "qkv"}
    head = torch.arange(H) // (H // G)
    q = unit(x["q"].view(n, G, D))[:, head] * D ** -0.5
    k = unit(x["k"].view(n, G, D))[:, head]
    beta, g = delta_gates(h @ w[pre + "b"].T, h @ w[pre + "a"].T, w[pre + "A_log"], w[pre + "dt_bias"])
    if "no_decay" in faults:
        g = torch.ones_like(g)
    o, _ = delta_rule(q, k, x["v"].view(n, H, V), beta, g, faults=faults)
    gate = (h @ w[pre + "g"].T).view(n, H, V)
    return gated_head_norm(o, gate, w[pre + "norm"], eps).reshape(n, H * V) @ w[pre + "o"].T


# ------------------------------------------------------------------------------------------------
# model
# ------------------------------------------------------------------------------------------------
def dense_mlp(w, pre, h):
    gate = h @ w[pre + "gate"].T + w[pre + "gate.b"]
    up = h @ w[pre + "up"].T + w[pre + "up.b"]
    return (gelu_tanh(gate) * up) @ w[pre + "down"].T + w[pre + "down.b"]


def forward(weights, cfg, tokens, dtype=F64, faults=(), trace=None):
    """Logits ``[n, vocab]`` of one sequence; ``trace`` (a list) collects the residual after every layer."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(list(tokens))]
    v_first = None
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = rms_norm(x, w[p + "norm1"], eps)
        if layer["type"] == "attention":
            mixing = bool(m.get("v_mix"))
            y, own = attention(w, p + "mix.", m, h, v_first if mixing else None, faults)
            if mixing and v_first is None:
                v_first = own
        else:
            y = delta(w, p + "mix.", m, h, eps, faults)
        x = x + rms_norm(y, w[p + "norm1b"], eps)
        if layer.get("mlp"):
            x = x + rms_norm(dense_mlp(w, p + "mlp.", rms_norm(x, w[p + "norm2"], eps)), w[p + "norm2b"], eps)
        if trace is not None:
            trace.append(x.clone())
    return rms_norm(x, w["final.norm"], eps) @ w["embed"].T


def greedy(weights, cfg, tokens, n):
    """``n`` greedy continuation tokens, every step recomputed from the whole sequence."""
    seq = list(tokens)
    for _ in range(n):
        seq.append(int(forward(weights, cfg, seq)[-1].argmax()))
    return seq[len(tokens):]


# ------------------------------------------------------------------------------------------------
# random models
# ------------------------------------------------------------------------------------------------
def attention_layer(heads=4, kv_heads=2, dim=32, vdim=24, window=11, scale=None, v_mix=True, ff=None):
    return {"type": "attention", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window},
                      "scale": scale if scale is not None else dim ** -0.5, "v_mix": v_mix}}


def delta_layer(heads=4, kv_heads=2, dim=16, vdim=24, conv=4, ff=None):
    return {"type": "delta", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def random_weights(cfg, seed=0, sharp=2.5):
    """Checkpoint tensors of ``cfg`` (bf16-representable fp32): projections keep unit variance, queries are scaled by
    ``sharp`` so that the attention is far from uniform; decays reach from a few tokens to hundreds."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]

    def vec(n, gain=1.0, mean=0.0):
        return (mean + gain * torch.randn(n, generator=g)).bfloat16().float()

    def mat(n, k, gain=1.0):
        return (torch.randn(n, k, generator=g) * gain / math.sqrt(k)).bfloat16().float()

    w = {"embed": mat(cfg["vocab"], W, math.sqrt(W)), "final.norm": vec(W, 0.2)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        w[p + "norm1"], w[p + "norm1b"] = vec(W, 0.2), vec(W, 0.2)
        mix = p + "mix."
        if layer["type"] == "attention":
            w[mix + "q"], w[mix + "k"], w[mix + "v"] = mat(H * D, W, sharp), mat(G * D, W), mat(G * V, W)
            for c, n in (("q", H * D), ("k", G * D), ("v", G * V)):
                w[f"{mix}{c}.b"] = vec(n, 0.5)
            if m.get("v_mix"):
                w[mix + "vmix"] = (0.2 + 0.6 * torch.rand((), generator=g)).bfloat16().float()
        else:
            w[mix + "q"], w[mix + "k"], w[mix + "v"] = mat(G * D, W), mat(G * D, W), mat(H * V, W)
            for c, n in (("q", G * D), ("k", G * D), ("v", H * V)):
                w[f"{mix}{c}.conv"] = mat(n, m["conv"], 1.5)
            w[mix + "b"], w[mix + "a"], w[mix + "g"] = mat(H, W), mat(H, W), mat(H * V, W)
            w[mix + "A_log"], w[mix + "dt_bias"] = vec(H, 0.7, -2.0), vec(H, 1.0, -1.0)
            w[mix + "norm"] = vec(V, 0.2, 1.0)
        w[mix + "o"] = mat(W, H * V)
        f = layer.get("mlp")
        if f:
            w[p + "norm2"], w[p + "norm2b"] = vec(W, 0.2), vec(W, 0.2)
            for c, n, k in (("gate", f["ff"], W), ("up", f["ff"], W), ("down", W, f["ff"])):
                w[f"{p}mlp.{c}"], w[f"{p}mlp.{c}.b"] = mat(n, k), vec(n, 0.3)
    return w
