"""Dodilix: a decoder with several residual streams (hyper-connections) whose layers are multi-head latent attention - with
a latent of its own or with the rows of an earlier layer - or chunked attention and gated linear attention side by side,
in any order, with silu-gated feed-forwards or group-routed experts beside a gated shared one.

``config.json`` describes the model layer by layer (``layers``: mixer and feed-forward of each), so every size and
constant is per layer here as well; the rank of the decays' projection is that of the checkpoint's tensor (kept in the
configuration as ``mixer.right.rank``).  The modules below only hold the weights, in the form the kernels read:

* latent mixer     ``in_proj`` latent and rotated key rows (none when the layer borrows them) and gate rows; ``q_down`` the
  queries' latent (kept dense, its product stays in 32-bit until it is normed); rotated rows of ``q_up`` and ``in_proj`` are
  reordered so that the pairs (2i, 2i + 1) of the design become (i, i + half), which changes no score
* parallel mixer   ``in_proj`` query, key, value and gate rows of the left side, then of the right; ``decay_down`` (kept
  dense) / ``decay_up`` / ``decay_bias``; ``o_proj`` both output projections next to one another, so that one product adds
  the sides (their scales belong to the sides' outputs)
* ``mlp.gate_up_proj``, expert and shared-expert rows  gate and up rows alternating in blocks of eight when the hidden size
  is a multiple of eight (a tensor-core tile then yields finished hidden units), else gate rows before up rows
* ``mlp.router``   router rows and, with a shared expert, its gate's row

The computation is the multistream engine's (``engine/multistream_engine.py``); ``DodilixForCausalLM.forward`` runs the same
step function for callers that drive the model through the transformers API.  The residual streams, norms, scores,
routers, the recurrence with its decays, and the logits are 32-bit in every mode.  CUDA only: a CPU call raises.
"""
from __future__ import annotations

import copy
from typing import Dict, Optional

import torch
from torch import nn
from transformers import PretrainedConfig, PreTrainedModel
from transformers.generation import GenerationMixin
from transformers.modeling_outputs import CausalLMOutputWithPast

from ..ops.linear_attn import LinearSpec
from ..ops.window_attn import AttnSpec
from .dobetar import StreamRMSNorm
from .letarax import interleave_gate_up

ARCHITECTURE = "Dodilix"
MIXERS = ("latent_attention", "parallel")
MAX_STREAMS = 16


class DodilixConfig(PretrainedConfig):
    model_type = "dodilix"
    attribute_map = {"vocab_size": "vocab", "hidden_size": "width"}

    def __init__(self, vocab=1024, width=256, layers=None, embedding=None, norm=None, streams=1, logit_scale=1.0,
                 architecture=ARCHITECTURE, **kwargs):
        self.vocab = int(vocab)
        self.width = int(width)
        self.layers = copy.deepcopy(list(layers or []))
        self.embedding = dict(embedding or {"scale": 1.0})
        self.norm = dict(norm or {"eps": 1e-6})
        self.streams = int(streams)
        self.logit_scale = float(logit_scale)
        self.architecture = architecture
        self.num_hidden_layers = len(self.layers)
        heads = [int(m.get("heads") or m["left"]["heads"]) for m in (layer["mixer"] for layer in self.layers)
                 if "heads" in m or "left" in m]
        self.num_attention_heads = max(heads) if heads else 1
        kwargs.setdefault("tie_word_embeddings", False)
        super().__init__(**kwargs)
        if not 1 <= self.streams <= MAX_STREAMS:
            raise ValueError(f"{self.streams} residual streams: 1 to {MAX_STREAMS} are supported")
        for i, layer in enumerate(self.layers):
            self._check(i, layer)

    def _check(self, i: int, layer: dict):
        m, mlp = layer["mixer"], layer.get("mlp")
        if layer.get("type") not in MIXERS:
            raise ValueError(f"layer {i}: mixer type {layer.get('type')!r} is not part of this architecture")
        if layer["type"] == "parallel":
            a = m["left"]
            if int(a["heads"]) % int(a["kv_heads"]):
                raise ValueError(f"layer {i}: {a['heads']} heads cannot share {a['kv_heads']} key / value heads evenly")
            if int(a["rot"]["dims"]) > int(a["dim"]):
                raise ValueError(f"layer {i}: {a['rot']['dims']} rotated dimensions in a head of {a['dim']}")
        else:
            if int((m.get("rot") or {}).get("dims", 0)) > int(m["rot_dim"]):
                raise ValueError(f"layer {i}: {m['rot']['dims']} rotated dimensions in a part of {m['rot_dim']}")
            src = m.get("kv_from")
            if src is not None:
                src = int(src)
                if not 0 <= src < i or self.layers[src]["type"] != "latent_attention" or \
                        self.layers[src]["mixer"].get("kv_from") is not None:
                    raise ValueError(f"layer {i}: layer {src} has no latents to lend")
                other = self.layers[src]["mixer"]
                if any(m.get(k) != other.get(k) for k in ("kv_rank", "rot_dim", "rot")):
                    raise ValueError(f"layer {i}: latents and rotation differ from those of layer {src}")
        if mlp is not None:
            if mlp.get("kind") not in ("dense", "moe"):
                raise ValueError(f"layer {i}: feed-forward kind {mlp.get('kind')!r} is not part of this architecture")
            if mlp["kind"] == "moe":
                r = mlp["router"]
                g = r.get("groups") or {"count": 1, "keep": 1}
                E, n, keep = int(r["experts"]), int(g["count"]), int(g["keep"])
                if E % n or not 1 <= keep <= n or int(r["top"]) > E // n * keep:
                    raise ValueError(f"layer {i}: cannot choose {r['top']} experts from {keep} of {n} groups of {E}")


class HyperConnection(nn.Module):
    """Weights with which a sublayer reads from and writes to the streams."""

    def __init__(self, streams: int):
        super().__init__()
        self.w_in = nn.Parameter(torch.full((streams,), 1.0 / streams))
        self.w_out = nn.Parameter(torch.ones(streams))
        self.mix = nn.Parameter(torch.eye(streams))

    def reset(self):
        nn.init.constant_(self.w_in, 1.0 / self.w_in.numel())
        nn.init.ones_(self.w_out)
        nn.init.eye_(self.mix)


class GatedLatentAttention(nn.Module):
    _ipex_keep_dense = ("q_down",)

    def __init__(self, config, mixer: dict, layer_idx: int):
        super().__init__()
        W, eps = config.width, config.norm["eps"]
        self.layer_idx = layer_idx
        self.heads, self.dim, self.rot_dim = int(mixer["heads"]), int(mixer["dim"]), int(mixer["rot_dim"])
        self.v_dim, self.kv_rank, self.q_rank = int(mixer["vdim"]), int(mixer["kv_rank"]), int(mixer["q_rank"])
        self.scale = float(mixer["scale"])
        rot = mixer.get("rot") or {}
        self.rot_base, self.rot_pairs = float(rot.get("base", 1.0)), int(rot.get("dims", 0)) // 2
        self.kv_from = None if mixer.get("kv_from") is None else int(mixer["kv_from"])
        self.kv_rows = self.kv_rank + self.rot_dim if self.kv_from is None else 0
        self.in_proj = nn.Linear(W, self.kv_rows + self.heads * self.v_dim, bias=False)
        self.kv_norm = StreamRMSNorm(self.kv_rank, eps) if self.kv_from is None else None
        self.q_down = nn.Linear(W, self.q_rank, bias=False)
        self.q_norm = StreamRMSNorm(self.q_rank, eps)
        self.q_up = nn.Linear(self.q_rank, self.heads * (self.dim + self.rot_dim), bias=False)
        self.k_up = nn.Parameter(torch.empty(self.heads * self.dim, self.kv_rank))
        self.v_up = nn.Parameter(torch.empty(self.heads * self.v_dim, self.kv_rank))
        self.o_proj = nn.Linear(self.heads * self.v_dim, W, bias=False)


class SideBySide(nn.Module):
    _ipex_keep_dense = ("decay_down",)

    def __init__(self, config, mixer: dict, layer_idx: int):
        super().__init__()
        W, eps, a, b = config.width, config.norm["eps"], mixer["left"], mixer["right"]
        self.layer_idx = layer_idx
        rot = a.get("rot") or {}
        self.rot_base = float(rot.get("base", 1.0))
        self.left = AttnSpec(heads=int(a["heads"]), kv_heads=int(a["kv_heads"]), dim=int(a["dim"]), vdim=int(a["vdim"]),
                             scale=float(a["scale"]), sink=True, chunk=int(a["mask"]["size"]),
                             rot_pairs=int(rot.get("dims", 0)) // 2, unit_eps=float(eps), gated=True,
                             gate_scale=float(mixer["left_scale"]))
        self.right = r = LinearSpec(heads=int(b["heads"]), dim=int(b["dim"]), vdim=int(b["vdim"]),
                                    rank=int(b.get("rank", 16)), tau=float(b["tau"]), out_scale=float(mixer["right_scale"]))
        self.in_proj = nn.Linear(W, self.left.rows + r.rows, bias=False)
        self.sink = nn.Parameter(torch.zeros(self.left.heads))
        self.decay_down = nn.Linear(W, r.rank, bias=False)
        self.decay_up = nn.Parameter(torch.zeros(r.heads * r.dim, r.rank))
        self.decay_bias = nn.Parameter(torch.zeros(r.heads * r.dim))
        self.head_norm = StreamRMSNorm(r.vdim, eps)
        self.o_proj = nn.Linear(self.left.heads * self.left.vdim + r.heads * r.vdim, W, bias=False)


class SiluGatedMLP(nn.Module):
    def __init__(self, config, mlp: dict):
        super().__init__()
        ff = int(mlp["ff"])
        self.interleaved = ff % 8 == 0
        self.gate_up_proj = nn.Linear(config.width, 2 * ff, bias=False)
        self.down_proj = nn.Linear(ff, config.width, bias=False)


class SiluExperts(nn.Module):
    """Rows of a bank of experts, or of a single one (``count`` None)."""

    def __init__(self, width: int, ff: int, count: Optional[int] = None):
        super().__init__()
        lead = () if count is None else (count,)
        self.gate_up_rows = nn.Parameter(torch.empty(*lead, 2 * ff, width))
        self.down_rows = nn.Parameter(torch.empty(*lead, width, ff))


class GroupRoutedMoE(nn.Module):
    def __init__(self, config, mlp: dict):
        super().__init__()
        r, shared = mlp["router"], mlp.get("shared")
        g = r.get("groups") or {"count": 1, "keep": 1}
        self.top_k, self.groups, self.keep = int(r["top"]), int(g["count"]), int(g["keep"])
        self.scale = float(r.get("scale", 1.0))
        E = int(r["experts"])
        self.router = nn.Linear(config.width, E + (shared is not None), bias=False)
        self.experts = SiluExperts(config.width, int(mlp["expert"]["ff"]), E)
        self.shared = SiluExperts(config.width, int(shared["ff"])) if shared is not None else None


class DodilixLayer(nn.Module):
    def __init__(self, config, layer: dict, layer_idx: int):
        super().__init__()
        eps, self.kind = config.norm["eps"], layer["type"]
        mixer_cls = SideBySide if self.kind == "parallel" else GatedLatentAttention
        self.norm1, self.hyper1 = StreamRMSNorm(config.width, eps), HyperConnection(config.streams)
        self.mixer = mixer_cls(config, layer["mixer"], layer_idx)
        mlp = layer.get("mlp")
        self.norm2 = StreamRMSNorm(config.width, eps) if mlp is not None else None
        self.hyper2 = HyperConnection(config.streams) if mlp is not None else None
        self.mlp = None if mlp is None else SiluGatedMLP(config, mlp) if mlp["kind"] == "dense" else \
            GroupRoutedMoE(config, mlp)


class DodilixModel(nn.Module):
    def __init__(self, config):
        super().__init__()
        self.embed_tokens = nn.Embedding(config.vocab, config.width)
        self.layers = nn.ModuleList(DodilixLayer(config, layer, i) for i, layer in enumerate(config.layers))
        self.norm = StreamRMSNorm(config.width, config.norm["eps"])


class DodilixForCausalLM(PreTrainedModel, GenerationMixin):
    config_class = DodilixConfig
    base_model_prefix = "model"
    _supports_sdpa = True
    _no_split_modules = ["DodilixLayer"]

    def __init__(self, config):
        super().__init__(config)
        self.model = DodilixModel(config)
        self.lm_head = nn.Linear(config.width, config.vocab, bias=False)
        # a recurrent state cannot be taken back to an earlier token
        self._ipex_rolls_back = all(layer["type"] != "parallel" for layer in config.layers)
        self.post_init()

    def get_input_embeddings(self):
        return self.model.embed_tokens

    def set_input_embeddings(self, value):
        self.model.embed_tokens = value

    def get_output_embeddings(self):
        return self.lm_head

    def set_output_embeddings(self, value):
        self.lm_head = value

    def _init_weights(self, module):
        if isinstance(module, HyperConnection):
            return module.reset()
        for p in module.parameters(recurse=False):
            if p.dim() >= 2:
                nn.init.normal_(p, 0.0, 0.02)

    @torch.no_grad()
    def forward(self, input_ids=None, attention_mask=None, position_ids=None, past_key_values=None,
                inputs_embeds=None, use_cache=None, labels=None, logits_to_keep=0, **kwargs):
        """Runs the multistream engine's step on ``input_ids [B, S]`` behind whatever ``past_key_values`` holds.  Positions
        follow from the cache and the left padding that ``attention_mask`` shows on the first call, so
        ``position_ids`` is not read."""
        from ..engine.multistream_engine import MultiStreamStack
        from ..engine.stream_engine import stack_for
        from ..ops.kv_cache import SlotCache
        if input_ids is None or inputs_embeds is not None:
            raise NotImplementedError("this architecture runs from token ids: pass input_ids")
        stack = stack_for(self, MultiStreamStack)
        cache = past_key_values if isinstance(past_key_values, SlotCache) else None
        if cache is None:
            if past_key_values is not None and past_key_values.get_seq_length() > 0:
                raise TypeError("a Dodilix model continues from a SlotCache only")
            cache = SlotCache(self.config)
        logits = stack.forward_padded(input_ids, attention_mask, cache, logits_to_keep)
        loss = None
        if labels is not None:
            loss = nn.functional.cross_entropy(logits[:, :-1].flatten(0, 1), labels[:, 1:].flatten())
        return CausalLMOutputWithPast(loss=loss, logits=logits,
                                      past_key_values=cache if use_cache is not False else None)


# ------------------------------------------------------------------------------------------------
# checkpoint names -> module names
# ------------------------------------------------------------------------------------------------
def split_pairs(rows: torch.Tensor, pairs: int) -> torch.Tensor:
    """Rows of a rotated part ``[..., rot_dim, width]``: of the first ``2 * pairs`` the even ones, then the odd ones."""
    turned, rest = rows[..., :2 * pairs, :], rows[..., 2 * pairs:, :]
    return torch.cat([turned[..., 0::2, :], turned[..., 1::2, :], rest], dim=-2)


def convert_checkpoint(state: Dict[str, torch.Tensor], config: DodilixConfig) -> Dict[str, torch.Tensor]:
    """Rename (and join) the tensors of a checkpoint; a missing or left-over tensor is an error."""
    src = dict(state)

    def take(name):
        if name not in src:
            raise KeyError(f"checkpoint has no tensor {name!r}")
        return src.pop(name)

    def join(prefix, names):
        return torch.cat([take(prefix + n) for n in names], dim=0)

    def unit(prefix):
        return interleave_gate_up(take(prefix + "gate"), take(prefix + "up"))

    out = {"model.embed_tokens.weight": take("embed"), "model.norm.weight": take("final.norm"),
           "lm_head.weight": take("head")}
    for i, layer in enumerate(config.layers):
        s, d, m, mlp = f"l{i}.", f"model.layers.{i}.", layer["mixer"], layer.get("mlp")
        mix, dst = s + "mix.", d + "mixer."
        for q in (1, 2) if mlp is not None else (1,):
            out[f"{d}norm{q}.weight"] = take(f"{s}norm{q}")
            for a, b in (("in", "w_in"), ("out", "w_out"), ("mix", "mix")):
                out[f"{d}hyper{q}.{b}"] = take(f"{s}hc{q}.{a}")
        if layer["type"] == "parallel":
            left, right = mix + "left.", mix + "right."
            out[dst + "in_proj.weight"] = torch.cat([join(left, "qkvg"), join(right, "qkvg")], dim=0)
            out[dst + "o_proj.weight"] = torch.cat([take(left + "o"), take(right + "o")], dim=1)
            out[dst + "sink"] = take(left + "sink")
            out[dst + "decay_down.weight"] = take(right + "a1")
            out[dst + "decay_up"], out[dst + "decay_bias"] = take(right + "a2"), take(right + "a2.b")
            out[dst + "head_norm.weight"] = take(right + "norm")
        else:
            H, D, rd, R = int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["kv_rank"])
            pairs = int((m.get("rot") or {}).get("dims", 0)) // 2
            rows = []
            if m.get("kv_from") is None:
                kv = take(mix + "dkv")
                rows = [kv[:R], split_pairs(kv[R:], pairs)]
                out[dst + "kv_norm.weight"] = take(mix + "dkv.norm")
            out[dst + "in_proj.weight"] = torch.cat([*rows, take(mix + "g")], dim=0)
            out[dst + "q_down.weight"], out[dst + "q_norm.weight"] = take(mix + "dq"), take(mix + "dq.norm")
            q = take(mix + "uq").unflatten(0, (H, D + rd))
            out[dst + "q_up.weight"] = torch.cat([q[:, :D], split_pairs(q[:, D:], pairs)], dim=1).flatten(0, 1)
            out[dst + "k_up"], out[dst + "v_up"] = take(mix + "uk"), take(mix + "uv")
            out[dst + "o_proj.weight"] = take(mix + "o")
        if mlp is None:
            continue
        f = s + "mlp."
        if mlp["kind"] == "dense":
            out[d + "mlp.gate_up_proj.weight"], out[d + "mlp.down_proj.weight"] = unit(f), take(f + "down")
            continue
        E, shared = int(mlp["router"]["experts"]), mlp.get("shared")
        out[d + "mlp.router.weight"] = join(f, ["router", "shared.sg"] if shared is not None else ["router"])
        out[d + "mlp.experts.gate_up_rows"] = torch.stack([unit(f"{f}e{e}.") for e in range(E)])
        out[d + "mlp.experts.down_rows"] = torch.stack([take(f"{f}e{e}.down") for e in range(E)])
        if shared is not None:
            out[d + "mlp.shared.gate_up_rows"] = unit(f + "shared.")
            out[d + "mlp.shared.down_rows"] = take(f + "shared.down")
    if src:
        raise KeyError(f"checkpoint tensors that the configuration does not name: {sorted(src)[:5]}")
    return out


def register():
    """Make the configuration and model class known to the Auto classes (idempotent)."""
    from transformers import AutoConfig, AutoModelForCausalLM
    AutoConfig.register(DodilixConfig.model_type, DodilixConfig, exist_ok=True)
    AutoModelForCausalLM.register(DodilixConfig, DodilixForCausalLM, exist_ok=True)


def build(config_dict: dict, state: Dict[str, torch.Tensor], dtype: Optional[torch.dtype]):
    """A model from a raw checkpoint (``config.json`` dictionary and tensors)."""
    config = DodilixConfig(**config_dict)
    config.architectures = [DodilixForCausalLM.__name__]
    for i, layer in enumerate(config.layers):
        name = f"l{i}.mix.right.a1"
        if layer["type"] == "parallel" and name in state:
            layer["mixer"]["right"]["rank"] = state[name].shape[0]
    dtype = dtype if isinstance(dtype, torch.dtype) else torch.bfloat16
    with torch.device("meta"):
        model = DodilixForCausalLM(config)
    tensors = {k: v.to(dtype) if v.is_floating_point() else v for k, v in convert_checkpoint(state, config).items()}
    model.load_state_dict(tensors, strict=True, assign=True)
    model.config.dtype = dtype
    return model.requires_grad_(False).eval()
