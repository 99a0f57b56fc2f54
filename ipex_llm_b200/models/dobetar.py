"""Dobetar: a decoder with sliding-window multi-head latent attention, squared-ReLU and clamped mixture-of-experts
feed-forwards, a bigram embedding beside the token embedding and soft-capped logits.

``config.json`` describes the model layer by layer (``layers``: mixer and feed-forward of each), so every size and
constant is per layer here as well.  The modules below only hold the weights, in the form the kernels read:

* ``qkv_a_proj``  query rows of all heads, then the latent rows, then the shared rotated key rows - one product;
* ``k_up`` / ``v_up``  the per-head key and value up-projections, absorbed into queries and outputs while decoding;
* ``experts.gate_up_rows``  one ``[experts, 2 ff, width]`` bank with gate and up rows alternating in 16-row tiles when
  ``ff`` is a multiple of 16 (a tensor-core tile then yields finished hidden units), else gate rows before up rows.

The computation is the latent engine's (``engine/latent_engine.py``); ``DobetarForCausalLM.forward`` runs the same step
function for callers that drive the model through the transformers API (beam search, logits of whole prompts, ...).
The residual stream, norms, scores, routers and logits are 32-bit in every mode.  CUDA only: a CPU call raises.
"""
from __future__ import annotations

from typing import Dict, Optional

import torch
from torch import nn
from transformers import PretrainedConfig, PreTrainedModel
from transformers.generation import GenerationMixin
from transformers.modeling_outputs import CausalLMOutputWithPast

ARCHITECTURE = "Dobetar"


class DobetarConfig(PretrainedConfig):
    model_type = "dobetar"
    attribute_map = {"vocab_size": "vocab", "hidden_size": "width"}

    def __init__(self, vocab=1024, width=256, layers=None, embedding=None, norm=None, logit_softcap=None,
                 architecture=ARCHITECTURE, **kwargs):
        self.vocab = int(vocab)
        self.width = int(width)
        self.layers = list(layers or [])
        self.embedding = dict(embedding or {"scale": 1.0})
        self.norm = dict(norm or {"eps": 1e-6})
        self.logit_softcap = logit_softcap
        self.architecture = architecture
        self.num_hidden_layers = len(self.layers)
        heads = [int(m["mixer"]["heads"]) for m in self.layers if "heads" in m.get("mixer", {})]
        self.num_attention_heads = max(heads) if heads else 1
        kwargs.setdefault("tie_word_embeddings", False)
        super().__init__(**kwargs)
        for i, layer in enumerate(self.layers):
            if layer.get("type") != "latent_attention":
                raise ValueError(f"layer {i}: mixer type {layer.get('type')!r} is not part of this architecture")
            mlp = layer.get("mlp")
            if mlp is not None and mlp.get("kind") not in ("dense", "moe"):
                raise ValueError(f"layer {i}: feed-forward kind {mlp.get('kind')!r} is not part of this architecture")


class StreamRMSNorm(nn.Module):
    """Weight of an RMS norm over the 32-bit residual stream (or over a latent)."""

    def __init__(self, dim: int, eps: float):
        super().__init__()
        self.weight = nn.Parameter(torch.ones(dim))
        self.eps = float(eps)


class LatentAttention(nn.Module):
    def __init__(self, config, mixer: dict, layer_idx: int):
        super().__init__()
        self.layer_idx = layer_idx
        self.heads, self.dim = int(mixer["heads"]), int(mixer["dim"])
        self.rot_dim, self.v_dim = int(mixer.get("rot_dim", 0)), int(mixer["vdim"])
        self.kv_rank = int(mixer["kv_rank"])
        self.scale = float(mixer["scale"])
        mask = mixer.get("mask") or {}
        self.window = int(mask.get("size") or 0)                 # 0: every earlier key
        rot = mixer.get("rot") or {}
        self.rot_base, self.rot_pairs = float(rot.get("base", 1.0)), int(rot.get("dims", 0)) // 2
        if 2 * self.rot_pairs > self.rot_dim:
            raise ValueError(f"layer {layer_idx}: {2 * self.rot_pairs} rotated dimensions in a part of {self.rot_dim}")
        W = config.width
        self.q_rows = self.heads * (self.dim + self.rot_dim)
        self.qkv_a_proj = nn.Linear(W, self.q_rows + self.kv_rank + self.rot_dim, bias=False)
        self.kv_norm = StreamRMSNorm(self.kv_rank, config.norm["eps"])
        self.k_up = nn.Parameter(torch.empty(self.heads * self.dim, self.kv_rank))
        self.v_up = nn.Parameter(torch.empty(self.heads * self.v_dim, self.kv_rank))
        self.o_proj = nn.Linear(self.heads * self.v_dim, W, bias=False)


class SquaredReluMLP(nn.Module):
    def __init__(self, config, mlp: dict):
        super().__init__()
        self.up_proj = nn.Linear(config.width, int(mlp["ff"]), bias=False)
        self.down_proj = nn.Linear(int(mlp["ff"]), config.width, bias=False)


class DenseExperts(nn.Module):
    def __init__(self, experts: int, width: int, ff: int):
        super().__init__()
        self.num_experts, self.ff = experts, ff
        self.interleaved = ff % 16 == 0
        self.gate_up_rows = nn.Parameter(torch.empty(experts, 2 * ff, width))
        self.down_rows = nn.Parameter(torch.empty(experts, width, ff))


class ClampedMoE(nn.Module):
    """Sigmoid-routed experts, each of which reads its input scaled by the routing weight."""

    gate_alpha = 1.702           # slope of the gate's sigmoid, part of the design

    def __init__(self, config, mlp: dict):
        super().__init__()
        self.top_k = int(mlp["router"]["top"])
        self.limit = float(mlp["expert"]["limit"])
        E = int(mlp["router"]["experts"])
        self.router = nn.Linear(config.width, E, bias=False)
        self.experts = DenseExperts(E, config.width, int(mlp["expert"]["ff"]))


class DobetarLayer(nn.Module):
    def __init__(self, config, layer: dict, layer_idx: int):
        super().__init__()
        eps = config.norm["eps"]
        self.norm1 = StreamRMSNorm(config.width, eps)
        self.mixer = LatentAttention(config, layer["mixer"], layer_idx)
        mlp = layer.get("mlp")
        self.norm2 = StreamRMSNorm(config.width, eps) if mlp is not None else None
        self.mlp = None if mlp is None else \
            SquaredReluMLP(config, mlp) if mlp["kind"] == "dense" else ClampedMoE(config, mlp)


class DobetarModel(nn.Module):
    def __init__(self, config):
        super().__init__()
        self.embed_tokens = nn.Embedding(config.vocab, config.width)
        bigram = config.embedding.get("bigram")
        self.bigram = nn.Embedding(int(bigram["buckets"]) + 1, config.width) if bigram else None
        self.layers = nn.ModuleList(DobetarLayer(config, layer, i) for i, layer in enumerate(config.layers))
        self.norm = StreamRMSNorm(config.width, config.norm["eps"])


class DobetarForCausalLM(PreTrainedModel, GenerationMixin):
    config_class = DobetarConfig
    base_model_prefix = "model"
    _supports_sdpa = True
    _no_split_modules = ["DobetarLayer"]

    def __init__(self, config):
        super().__init__(config)
        self.model = DobetarModel(config)
        self.lm_head = nn.Linear(config.width, config.vocab, bias=False)
        self.post_init()

    def get_input_embeddings(self):
        return self.model.embed_tokens

    def set_input_embeddings(self, value):
        self.model.embed_tokens = value

    def get_output_embeddings(self):
        return self.lm_head

    def _init_weights(self, module):
        for p in module.parameters(recurse=False):
            if p.dim() >= 2:
                nn.init.normal_(p, 0.0, 0.02)

    @torch.no_grad()
    def forward(self, input_ids=None, attention_mask=None, position_ids=None, past_key_values=None,
                inputs_embeds=None, use_cache=None, labels=None, logits_to_keep=0, **kwargs):
        """Runs the latent engine's step on ``input_ids [B, S]`` behind whatever ``past_key_values`` holds.  Positions
        follow from the cache and the left padding that ``attention_mask`` shows on the first call, so
        ``position_ids`` is not read."""
        from ..engine.latent_engine import LatentStack
        from ..engine.stream_engine import stack_for
        from ..ops.kv_cache import LatentCache
        if input_ids is None or inputs_embeds is not None:
            raise NotImplementedError("this architecture embeds token pairs: pass input_ids")
        stack = stack_for(self, LatentStack)
        cache = past_key_values if isinstance(past_key_values, LatentCache) else None
        if cache is None:
            if past_key_values is not None and past_key_values.get_seq_length() > 0:
                raise TypeError("a Dobetar model continues from a LatentCache only")
            cache = LatentCache(self.config)
        logits = stack.forward_padded(input_ids, attention_mask, cache, logits_to_keep)
        loss = None
        if labels is not None:
            loss = nn.functional.cross_entropy(logits[:, :-1].flatten(0, 1), labels[:, 1:].flatten())
        return CausalLMOutputWithPast(loss=loss, logits=logits,
                                      past_key_values=cache if use_cache is not False else None)


# ------------------------------------------------------------------------------------------------
# checkpoint names -> module names
# ------------------------------------------------------------------------------------------------
def interleave_gate_up(gate: torch.Tensor, up: torch.Tensor) -> torch.Tensor:
    """``[ff, width]`` gate and up rows -> ``[2 ff, width]`` in the layout of ``DenseExperts.gate_up_rows``."""
    ff, w = gate.shape
    if ff % 16:
        return torch.cat([gate, up], dim=0)
    return torch.stack([gate.view(ff // 16, 16, w), up.view(ff // 16, 16, w)], dim=1).reshape(2 * ff, w)


def convert_checkpoint(state: Dict[str, torch.Tensor], config: DobetarConfig) -> Dict[str, torch.Tensor]:
    """Rename (and join) the tensors of a checkpoint; a missing or left-over tensor is an error."""
    src = dict(state)

    def take(name):
        if name not in src:
            raise KeyError(f"checkpoint has no tensor {name!r}")
        return src.pop(name)

    out = {"model.embed_tokens.weight": take("embed"), "model.norm.weight": take("final.norm"),
           "lm_head.weight": take("head")}
    if config.embedding.get("bigram"):
        out["model.bigram.weight"] = take("bigram")
    for i, layer in enumerate(config.layers):
        s, d = f"l{i}.", f"model.layers.{i}."
        out[d + "norm1.weight"] = take(s + "norm1")
        out[d + "mixer.qkv_a_proj.weight"] = torch.cat([take(s + "mix.q"), take(s + "mix.dkv")], dim=0)
        out[d + "mixer.kv_norm.weight"] = take(s + "mix.dkv.norm")
        out[d + "mixer.k_up"] = take(s + "mix.uk")
        out[d + "mixer.v_up"] = take(s + "mix.uv")
        out[d + "mixer.o_proj.weight"] = take(s + "mix.o")
        mlp = layer.get("mlp")
        if mlp is None:
            continue
        out[d + "norm2.weight"] = take(s + "norm2")
        if mlp["kind"] == "dense":
            out[d + "mlp.up_proj.weight"] = take(s + "mlp.up")
            out[d + "mlp.down_proj.weight"] = take(s + "mlp.down")
            continue
        E = int(mlp["router"]["experts"])
        out[d + "mlp.router.weight"] = take(s + "mlp.router")
        out[d + "mlp.experts.gate_up_rows"] = torch.stack(
            [interleave_gate_up(take(f"{s}mlp.e{e}.gate"), take(f"{s}mlp.e{e}.up")) for e in range(E)])
        out[d + "mlp.experts.down_rows"] = torch.stack([take(f"{s}mlp.e{e}.down") for e in range(E)])
    if src:
        raise KeyError(f"checkpoint tensors that the configuration does not name: {sorted(src)[:5]}")
    return out


def register():
    """Make the configuration and model class known to the Auto classes (idempotent)."""
    from transformers import AutoConfig, AutoModelForCausalLM
    AutoConfig.register(DobetarConfig.model_type, DobetarConfig, exist_ok=True)
    AutoModelForCausalLM.register(DobetarConfig, DobetarForCausalLM, exist_ok=True)


def build(config_dict: dict, state: Dict[str, torch.Tensor], dtype: Optional[torch.dtype]):
    """A model from a raw checkpoint (``config.json`` dictionary and tensors)."""
    config = DobetarConfig(**config_dict)
    config.architectures = [DobetarForCausalLM.__name__]
    dtype = dtype if isinstance(dtype, torch.dtype) else torch.bfloat16
    with torch.device("meta"):
        model = DobetarForCausalLM(config)
    tensors = {k: v.to(dtype) if v.is_floating_point() else v for k, v in convert_checkpoint(state, config).items()}
    model.load_state_dict(tensors, strict=True, assign=True)
    model.config.dtype = dtype
    return model.requires_grad_(False).eval()
