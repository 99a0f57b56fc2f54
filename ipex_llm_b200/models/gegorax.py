"""Gegorax: a decoder whose mixer and feed-forward read the same norm side by side and whose layers add an embedding of the
token of their own.  Mixers are a generalized delta rule, or windowed attention over tokens and pooled blocks beside a
state-space recurrence (each normed, then averaged), in any order; feed-forwards are squared-relu units or clamped experts
behind a soft-max router with a shared expert.

``config.json`` describes the model layer by layer (``layers``: mixer and feed-forward of each), so every size and
constant is per layer here as well; the rank of the decays' projection is that of the checkpoint's tensor (kept in the
configuration as ``mixer.rank``).  The modules below only hold the weights, in the form the kernels read:

* ``in_proj``   everything that reads the norm with 16-bit results.  delta: read, key, value, removal-rate and output-gate
  rows; parallel: query, key and value rows of the left side (rotated rows reordered so that the pairs (2i, 2i + 1) of the
  design become (i, i + half), which changes no score), then x, B, C and gate rows of the right; behind either the up rows of
  a dense feed-forward
* ``low_proj``  what has 32-bit results (kept dense): first half of the decays' projection, or the step sizes; then the
  router's rows
* ``out_proj``  delta: the mixer's output projection and, next to it, the down projection of a dense feed-forward, so that
  one product adds both; parallel: the down projection (none with experts), beside ``mixer.o_left`` and ``mixer.o_right``
* expert and shared-expert rows  gate and up rows alternating in blocks of eight when the hidden size is a multiple of eight
  (a tensor-core tile then yields finished hidden units), else gate rows before up rows

The computation is the parallel-block engine's (``engine/parallel_block_engine.py``); ``GegoraxForCausalLM.forward`` runs the
same step function for callers that drive the model through the transformers API.  The residual stream, norms, scores,
routers, the recurrences with their decays, rates and step sizes, and the logits are 32-bit in every mode.  CUDA only: a CPU
call raises.
"""
from __future__ import annotations

import copy
from typing import Dict, Optional

import torch
from torch import nn
from transformers import PretrainedConfig, PreTrainedModel
from transformers.generation import GenerationMixin
from transformers.modeling_outputs import CausalLMOutputWithPast

from ..ops.general_delta import GeneralDeltaSpec
from ..ops.ssd import SSDSpec
from ..ops.window_attn import AttnSpec
from .dobetar import StreamRMSNorm
from .dodilix import SiluExperts, split_pairs
from .letarax import interleave_gate_up

ARCHITECTURE = "Gegorax"
MIXERS = ("general_delta", "parallel")
UNIT_ALPHA = 1.702           # of the clamped unit's sigmoid
SIDE_SHARE = 0.5             # of each side of a parallel mixer


class GegoraxConfig(PretrainedConfig):
    model_type = "gegorax"
    attribute_map = {"vocab_size": "vocab", "hidden_size": "width"}

    def __init__(self, vocab=1024, width=256, layers=None, norm=None, token_side=None, architecture=ARCHITECTURE, **kwargs):
        self.vocab = int(vocab)
        self.width = int(width)
        self.layers = copy.deepcopy(list(layers or []))
        self.norm = dict(norm or {"eps": 1e-6})
        self.token_side = dict(token_side) if token_side else None
        self.architecture = architecture
        self.num_hidden_layers = len(self.layers)
        heads = [int(m.get("heads") or m["left"]["heads"]) for m in (layer["mixer"] for layer in self.layers)
                 if "heads" in m or "left" in m]
        self.num_attention_heads = max(heads) if heads else 1
        kwargs.setdefault("tie_word_embeddings", False)
        super().__init__(**kwargs)
        for i, layer in enumerate(self.layers):
            self._check(i, layer)

    @property
    def side_dim(self) -> int:
        return int((self.token_side or {}).get("dim") or 0)

    def _check(self, i: int, layer: dict):
        m, mlp = layer["mixer"], layer.get("mlp")
        if layer.get("type") not in MIXERS:
            raise ValueError(f"layer {i}: mixer type {layer.get('type')!r} is not part of this architecture")
        if layer["type"] == "parallel":
            a, b = m["left"], m["right"]
            if int(a["heads"]) % int(a["kv_heads"]):
                raise ValueError(f"layer {i}: {a['heads']} heads cannot share {a['kv_heads']} key / value heads evenly")
            if int((a.get("rot") or {}).get("dims", 0)) > int(a["dim"]):
                raise ValueError(f"layer {i}: {a['rot']['dims']} rotated dimensions in a head of {a['dim']}")
            mask = a.get("mask") or {}
            if mask.get("pool") and not mask.get("size"):
                raise ValueError(f"layer {i}: pooled blocks without a window")
            if int(b["heads"]) % int(b["groups"]):
                raise ValueError(f"layer {i}: {b['heads']} heads cannot share {b['groups']} groups evenly")
            if int(b["heads"]) * int(b["vdim"]) % int(b["norm_groups"]):
                raise ValueError(f"layer {i}: {b['heads']} x {b['vdim']} columns cannot be normed in {b['norm_groups']} parts")
        if mlp is not None:
            if mlp.get("kind") not in ("dense", "moe"):
                raise ValueError(f"layer {i}: feed-forward kind {mlp.get('kind')!r} is not part of this architecture")
            if mlp["kind"] == "moe" and not 1 <= int(mlp["router"]["top"]) <= int(mlp["router"]["experts"]):
                raise ValueError(f"layer {i}: cannot choose {mlp['router']['top']} of {mlp['router']['experts']} experts")


class GeneralDelta(nn.Module):
    """Weights of the recurrence between the layer's projections."""

    def __init__(self, config, mixer: dict):
        super().__init__()
        heads, dim = int(mixer["heads"]), int(mixer["dim"])
        self.spec = s = GeneralDeltaSpec(heads, dim, dim, int(mixer.get("rank", 16)))
        n = heads * dim
        self.rows, self.low_rows, self.out_columns = s.rows, s.rank, n
        self.decay_up = nn.Parameter(torch.zeros(n, s.rank))
        self.decay_bias, self.rate_bias = nn.Parameter(torch.zeros(n)), nn.Parameter(torch.zeros(n))
        self.head_norm = nn.Parameter(torch.ones(n))


class PooledAttentionBesideSSD(nn.Module):
    def __init__(self, config, mixer: dict):
        super().__init__()
        W, eps, a, b = config.width, config.norm["eps"], mixer["left"], mixer["right"]
        rot, mask = a.get("rot") or {}, a.get("mask") or {}
        self.rot_base = float(rot.get("base", 1.0))
        self.left = s = AttnSpec(heads=int(a["heads"]), kv_heads=int(a["kv_heads"]), dim=int(a["dim"]), vdim=int(a["vdim"]),
                                 scale=float(a["scale"]), window=int(mask.get("size") or 0), pool=int(mask.get("pool") or 0),
                                 rot_pairs=int(rot.get("dims", 0)) // 2, unit_eps=float(eps))
        self.right = r = SSDSpec(heads=int(b["heads"]), vdim=int(b["vdim"]), state=int(b["state"]), groups=int(b["groups"]),
                                 taps=int(b["conv"]), parts=int(b["norm_groups"]))
        self.rows, self.low_rows, self.out_columns = s.rows + r.rows, r.heads, 0
        self.q_norm, self.k_norm = StreamRMSNorm(s.dim, eps), StreamRMSNorm(s.dim, eps)
        self.o_left, self.left_out = nn.Linear(s.heads * s.vdim, W, bias=False), StreamRMSNorm(W, eps)
        self.conv, self.conv_bias = nn.Parameter(torch.zeros(r.channels, r.taps)), nn.Parameter(torch.zeros(r.channels))
        self.dt_bias, self.A_log = nn.Parameter(torch.zeros(r.heads)), nn.Parameter(torch.zeros(r.heads))
        self.skip = nn.Parameter(torch.ones(r.heads))
        self.inner_norm = StreamRMSNorm(r.inner, eps)
        self.o_right, self.right_out = nn.Linear(r.inner, W, bias=False), StreamRMSNorm(W, eps)


class ClampedMoE(nn.Module):
    def __init__(self, config, mlp: dict):
        super().__init__()
        r, shared = mlp["router"], mlp.get("shared")
        self.top_k, self.limit = int(r["top"]), float(mlp["expert"]["limit"])
        self.shared_limit = float(shared["limit"]) if shared is not None else 0.0
        self.router_bias = nn.Parameter(torch.zeros(int(r["experts"])))
        self.experts = SiluExperts(config.width, int(mlp["expert"]["ff"]), int(r["experts"]))
        self.shared = SiluExperts(config.width, int(shared["ff"])) if shared is not None else None


class TokenSide(nn.Module):
    """What a layer does with its part of the tokens' side embedding."""
    _ipex_keep_dense = ("gate", "proj")

    def __init__(self, config):
        super().__init__()
        self.gate = nn.Linear(config.width, config.side_dim, bias=False)
        self.proj = nn.Linear(config.side_dim, config.width, bias=False)
        self.norm = StreamRMSNorm(config.width, config.norm["eps"])


class GegoraxLayer(nn.Module):
    _ipex_keep_dense = ("low_proj",)

    def __init__(self, config, layer: dict):
        super().__init__()
        W, mlp, self.kind = config.width, layer.get("mlp"), layer["type"]
        self.norm1 = StreamRMSNorm(W, config.norm["eps"])
        self.mixer = m = (PooledAttentionBesideSSD if self.kind == "parallel" else GeneralDelta)(config, layer["mixer"])
        self.dense_ff = int(mlp["ff"]) if mlp is not None and mlp["kind"] == "dense" else 0
        self.moe = ClampedMoE(config, mlp) if mlp is not None and mlp["kind"] == "moe" else None
        self.in_proj = nn.Linear(W, m.rows + self.dense_ff, bias=False)
        routed = 0 if self.moe is None else self.moe.router_bias.numel()
        self.low_proj = nn.Linear(W, m.low_rows + routed, bias=False)
        joined = m.out_columns + self.dense_ff
        self.out_proj = nn.Linear(joined, W, bias=False) if joined else None
        self.side = TokenSide(config) if config.side_dim else None


class GegoraxModel(nn.Module):
    def __init__(self, config):
        super().__init__()
        self.embed_tokens = nn.Embedding(config.vocab, config.width)
        self.side_table = nn.Parameter(torch.empty(config.vocab, config.side_dim * len(config.layers))) if config.side_dim \
            else None
        self.layers = nn.ModuleList(GegoraxLayer(config, layer) for layer in config.layers)
        self.norm = StreamRMSNorm(config.width, config.norm["eps"])


class GegoraxForCausalLM(PreTrainedModel, GenerationMixin):
    config_class = GegoraxConfig
    base_model_prefix = "model"
    _supports_sdpa = True
    _no_split_modules = ["GegoraxLayer"]
    _ipex_rolls_back = False         # a recurrent state cannot be taken back to an earlier token

    def __init__(self, config):
        super().__init__(config)
        self.model = GegoraxModel(config)
        self.lm_head = nn.Linear(config.width, config.vocab, bias=False)
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
        for p in module.parameters(recurse=False):
            if p.dim() >= 2:
                nn.init.normal_(p, 0.0, 0.02)

    @torch.no_grad()
    def forward(self, input_ids=None, attention_mask=None, position_ids=None, past_key_values=None,
                inputs_embeds=None, use_cache=None, labels=None, logits_to_keep=0, **kwargs):
        """Runs the parallel-block engine's step on ``input_ids [B, S]`` behind whatever ``past_key_values`` holds.  Positions
        follow from the cache and the left padding that ``attention_mask`` shows on the first call, so
        ``position_ids`` is not read."""
        from ..engine.parallel_block_engine import ParallelBlockStack
        from ..engine.stream_engine import stack_for
        from ..ops.kv_cache import SlotCache
        if input_ids is None or inputs_embeds is not None:
            raise NotImplementedError("this architecture runs from token ids: pass input_ids")
        stack = stack_for(self, ParallelBlockStack)
        cache = past_key_values if isinstance(past_key_values, SlotCache) else None
        if cache is None:
            if past_key_values is not None and past_key_values.get_seq_length() > 0:
                raise TypeError("a Gegorax model continues from a SlotCache only")
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
def convert_checkpoint(state: Dict[str, torch.Tensor], config: GegoraxConfig) -> Dict[str, torch.Tensor]:
    """Rename (and join) the tensors of a checkpoint; a missing or left-over tensor is an error."""
    src = dict(state)

    def take(name):
        if name not in src:
            raise KeyError(f"checkpoint has no tensor {name!r}")
        return src.pop(name)

    def unit(prefix):
        return interleave_gate_up(take(prefix + "gate"), take(prefix + "up"))

    out = {"model.embed_tokens.weight": take("embed"), "model.norm.weight": take("final.norm"),
           "lm_head.weight": take("head")}
    if config.side_dim:
        out["model.side_table"] = take("side.embed")
    for i, layer in enumerate(config.layers):
        s, d, m, mlp = f"l{i}.", f"model.layers.{i}.", layer["mixer"], layer.get("mlp")
        mix, f, dst = s + "mix.", s + "mlp.", d + "mixer."
        out[d + "norm1.weight"] = take(s + "norm1")
        if layer["type"] == "parallel":
            a, b, left, right = m["left"], m["right"], mix + "left.", mix + "right."
            pairs = int((a.get("rot") or {}).get("dims", 0)) // 2

            def turned(name, heads):
                return split_pairs(take(left + name).unflatten(0, (heads, -1)), pairs).flatten(0, 1)

            inner, shared = int(b["heads"]) * int(b["vdim"]), 2 * int(b["groups"]) * int(b["state"])
            z, xbc, dt = take(right + "in").split([inner, inner + shared, int(b["heads"])])
            rows, low = [turned("q", int(a["heads"])), turned("k", int(a["kv_heads"])), take(left + "v"), xbc, z], [dt]
            for n in "qk":
                out[f"{dst}{n}_norm.weight"] = split_pairs(take(f"{left}{n}.norm").unsqueeze(-1), pairs).squeeze(-1)
            for side, name in ((left, "left"), (right, "right")):
                out[f"{dst}o_{name}.weight"], out[f"{dst}{name}_out.weight"] = take(side + "o"), take(side + "out")
            out[dst + "conv"], out[dst + "conv_bias"] = take(right + "conv"), take(right + "conv.b")
            out[dst + "dt_bias"], out[dst + "A_log"] = take(right + "dt_bias"), take(right + "A_log")
            out[dst + "skip"], out[dst + "inner_norm.weight"] = take(right + "D"), take(right + "norm")
            joined = []
        else:
            rows, low = [take(mix + c) for c in "rkvag"], [take(mix + "w1")]
            out[dst + "decay_up"], out[dst + "decay_bias"] = take(mix + "w2"), take(mix + "w0")
            out[dst + "rate_bias"], out[dst + "head_norm"] = take(mix + "a.b"), take(mix + "norm")
            joined = [take(mix + "o")]
        if mlp is not None and mlp["kind"] == "dense":
            rows.append(take(f + "up"))
            joined.append(take(f + "down"))
        elif mlp is not None:
            E, moe = int(mlp["router"]["experts"]), d + "moe."
            low.append(take(f + "router"))
            out[moe + "router_bias"] = take(f + "router.b")
            out[moe + "experts.gate_up_rows"] = torch.stack([unit(f"{f}e{e}.") for e in range(E)])
            out[moe + "experts.down_rows"] = torch.stack([take(f"{f}e{e}.down") for e in range(E)])
            if mlp.get("shared") is not None:
                out[moe + "shared.gate_up_rows"] = unit(f + "shared.")
                out[moe + "shared.down_rows"] = take(f + "shared.down")
        out[d + "in_proj.weight"], out[d + "low_proj.weight"] = torch.cat(rows), torch.cat(low)
        if joined:
            out[d + "out_proj.weight"] = torch.cat(joined, dim=1)
        if config.side_dim:
            for n in ("gate", "proj", "norm"):
                out[f"{d}side.{n}.weight"] = take(f"{s}side.{n}")
    if src:
        raise KeyError(f"checkpoint tensors that the configuration does not name: {sorted(src)[:5]}")
    return out


def register():
    """Make the configuration and model class known to the Auto classes (idempotent)."""
    from transformers import AutoConfig, AutoModelForCausalLM
    AutoConfig.register(GegoraxConfig.model_type, GegoraxConfig, exist_ok=True)
    AutoModelForCausalLM.register(GegoraxConfig, GegoraxForCausalLM, exist_ok=True)


def build(config_dict: dict, state: Dict[str, torch.Tensor], dtype: Optional[torch.dtype]):
    """A model from a raw checkpoint (``config.json`` dictionary and tensors)."""
    config = GegoraxConfig(**config_dict)
    config.architectures = [GegoraxForCausalLM.__name__]
    for i, layer in enumerate(config.layers):
        name = f"l{i}.mix.w1"
        if layer["type"] == "general_delta" and name in state:
            layer["mixer"]["rank"] = state[name].shape[0]
    dtype = dtype if isinstance(dtype, torch.dtype) else torch.bfloat16
    with torch.device("meta"):
        model = GegoraxForCausalLM(config)
    tensors = {k: v.to(dtype) if v.is_floating_point() else v for k, v in convert_checkpoint(state, config).items()}
    model.load_state_dict(tensors, strict=True, assign=True)
    model.config.dtype = dtype
    return model.requires_grad_(False).eval()
