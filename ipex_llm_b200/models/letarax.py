"""Letarax: a decoder of windowed-attention layers (grouped heads, a sink in the soft-max, values mixed with those of an
earlier layer, no positions in the scores) and gated-delta-rule layers with short convolutions, in any order, with norms
before and after every sublayer, gelu-gated feed-forwards and the embedding table as output layer.

``config.json`` describes the model layer by layer (``layers``: mixer and feed-forward of each), so every size and
constant is per layer here as well.  The modules below only hold the weights, in the form the kernels read:

* ``mixer.in_proj``  attention: query, key and value rows with their biases; delta: query, key, value and output-gate rows
* ``mixer.gate_proj``  delta: rows of the write strengths, then of the decays (kept dense, their products stay in 32-bit)
* ``mixer.conv``  delta: convolution taps of the query, key and value channels
* ``mlp.gate_up_proj``  gate and up rows (and biases) alternating in blocks of eight when ``ff`` is a multiple of eight (a
  tensor-core tile then yields finished hidden units), else gate rows before up rows

The computation is the hybrid engine's (``engine/hybrid_engine.py``); ``LetaraxForCausalLM.forward`` runs the same step
function for callers that drive the model through the transformers API.  The residual stream, norms, scores, the
recurrence with its gates, and the logits are 32-bit in every mode.  CUDA only: a CPU call raises.
"""
from __future__ import annotations

from typing import Dict, Optional

import torch
from torch import nn
from transformers import PretrainedConfig, PreTrainedModel
from transformers.generation import GenerationMixin
from transformers.modeling_outputs import CausalLMOutputWithPast

from ..ops.delta import DeltaSpec
from ..ops.window_attn import AttnSpec
from .dobetar import StreamRMSNorm

ARCHITECTURE = "Letarax"
MIXERS = ("attention", "delta")


class LetaraxConfig(PretrainedConfig):
    model_type = "letarax"
    attribute_map = {"vocab_size": "vocab", "hidden_size": "width"}

    def __init__(self, vocab=1024, width=256, layers=None, norm=None, architecture=ARCHITECTURE, **kwargs):
        self.vocab = int(vocab)
        self.width = int(width)
        self.layers = list(layers or [])
        self.norm = dict(norm or {"eps": 1e-6})
        self.architecture = architecture
        self.num_hidden_layers = len(self.layers)
        heads = [int(m["mixer"]["heads"]) for m in self.layers if "heads" in m.get("mixer", {})]
        self.num_attention_heads = max(heads) if heads else 1
        kwargs.setdefault("tie_word_embeddings", True)
        super().__init__(**kwargs)
        shared = None
        for i, layer in enumerate(self.layers):
            if layer.get("type") not in MIXERS:
                raise ValueError(f"layer {i}: mixer type {layer.get('type')!r} is not part of this architecture")
            mlp, m = layer.get("mlp"), layer["mixer"]
            if mlp is not None and mlp.get("kind") != "dense":
                raise ValueError(f"layer {i}: feed-forward kind {mlp.get('kind')!r} is not part of this architecture")
            if int(m["heads"]) % int(m["kv_heads"]):
                raise ValueError(f"layer {i}: {m['heads']} heads cannot share {m['kv_heads']} key / value heads evenly")
            if layer["type"] == "attention" and m.get("v_mix"):
                size = (int(m["kv_heads"]), int(m["vdim"]))
                if shared not in (None, size):
                    raise ValueError(f"layer {i}: values of {size} cannot be mixed with earlier ones of {shared}")
                shared = size

    def value_mix_role(self, i: int) -> Optional[str]:
        """``first`` for the layer whose values the later ones mix in, ``mixed`` for those, else None."""
        mixing = [j for j, layer in enumerate(self.layers)
                  if layer["type"] == "attention" and layer["mixer"].get("v_mix")]
        return None if i not in mixing else "first" if i == mixing[0] else "mixed"


class WindowAttention(nn.Module):
    def __init__(self, config, mixer: dict, layer_idx: int):
        super().__init__()
        self.layer_idx = layer_idx
        mask = mixer.get("mask") or {}
        self.spec = AttnSpec(heads=int(mixer["heads"]), kv_heads=int(mixer["kv_heads"]), dim=int(mixer["dim"]),
                             vdim=int(mixer["vdim"]), scale=float(mixer["scale"]), window=int(mask.get("size") or 0),
                             sink=True)
        self.in_proj = nn.Linear(config.width, self.spec.rows, bias=True)
        self.o_proj = nn.Linear(self.spec.heads * self.spec.vdim, config.width, bias=False)
        self.mix_role = config.value_mix_role(layer_idx)
        self.value_share = nn.Parameter(torch.zeros(())) if self.mix_role else None


class GatedDelta(nn.Module):
    _ipex_keep_dense = ("gate_proj",)

    def __init__(self, config, mixer: dict, layer_idx: int):
        super().__init__()
        self.layer_idx = layer_idx
        self.spec = s = DeltaSpec(heads=int(mixer["heads"]), kv_heads=int(mixer["kv_heads"]), dim=int(mixer["dim"]),
                                  vdim=int(mixer["vdim"]), taps=int(mixer["conv"]))
        self.in_proj = nn.Linear(config.width, s.rows, bias=False)
        self.gate_proj = nn.Linear(config.width, 2 * s.heads, bias=False)
        self.conv = nn.Parameter(torch.zeros(s.channels, s.taps))
        self.A_log = nn.Parameter(torch.zeros(s.heads))
        self.dt_bias = nn.Parameter(torch.zeros(s.heads))
        self.norm = StreamRMSNorm(s.vdim, config.norm["eps"])
        self.o_proj = nn.Linear(s.heads * s.vdim, config.width, bias=False)


class GeluGatedMLP(nn.Module):
    def __init__(self, config, mlp: dict):
        super().__init__()
        ff = int(mlp["ff"])
        self.interleaved = ff % 8 == 0
        self.gate_up_proj = nn.Linear(config.width, 2 * ff, bias=True)
        self.down_proj = nn.Linear(ff, config.width, bias=True)


class LetaraxLayer(nn.Module):
    def __init__(self, config, layer: dict, layer_idx: int):
        super().__init__()
        eps, self.kind = config.norm["eps"], layer["type"]
        mixer_cls = WindowAttention if self.kind == "attention" else GatedDelta
        self.norm1, self.norm1b = StreamRMSNorm(config.width, eps), StreamRMSNorm(config.width, eps)
        self.mixer = mixer_cls(config, layer["mixer"], layer_idx)
        mlp = layer.get("mlp")
        self.norm2 = StreamRMSNorm(config.width, eps) if mlp is not None else None
        self.norm2b = StreamRMSNorm(config.width, eps) if mlp is not None else None
        self.mlp = GeluGatedMLP(config, mlp) if mlp is not None else None


class LetaraxModel(nn.Module):
    def __init__(self, config):
        super().__init__()
        self.embed_tokens = nn.Embedding(config.vocab, config.width)
        self.layers = nn.ModuleList(LetaraxLayer(config, layer, i) for i, layer in enumerate(config.layers))
        self.norm = StreamRMSNorm(config.width, config.norm["eps"])


class LetaraxForCausalLM(PreTrainedModel, GenerationMixin):
    config_class = LetaraxConfig
    base_model_prefix = "model"
    _supports_sdpa = True
    _no_split_modules = ["LetaraxLayer"]
    _tied_weights_keys = {"lm_head.weight": "model.embed_tokens.weight"}
    _ipex_rolls_back = False         # a recurrent state cannot be taken back to an earlier token

    def __init__(self, config):
        super().__init__(config)
        self.model = LetaraxModel(config)
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
        """Runs the hybrid engine's step on ``input_ids [B, S]`` behind whatever ``past_key_values`` holds.  Positions
        follow from the cache and the left padding that ``attention_mask`` shows on the first call, so
        ``position_ids`` is not read."""
        from ..engine.hybrid_engine import HybridStack
        from ..engine.stream_engine import stack_for
        from ..ops.kv_cache import SlotCache
        if input_ids is None or inputs_embeds is not None:
            raise NotImplementedError("this architecture runs from token ids: pass input_ids")
        stack = stack_for(self, HybridStack)
        cache = past_key_values if isinstance(past_key_values, SlotCache) else None
        if cache is None:
            if past_key_values is not None and past_key_values.get_seq_length() > 0:
                raise TypeError("a Letarax model continues from a SlotCache only")
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
def interleave_gate_up(gate: torch.Tensor, up: torch.Tensor) -> torch.Tensor:
    """Gate and up rows (or biases) in the order of ``GeluGatedMLP.gate_up_proj``."""
    ff = gate.shape[0]
    if ff % 8:
        return torch.cat([gate, up], dim=0)
    return torch.stack([gate.unflatten(0, (-1, 8)), up.unflatten(0, (-1, 8))], dim=1).flatten(0, 2)


def convert_checkpoint(state: Dict[str, torch.Tensor], config: LetaraxConfig) -> Dict[str, torch.Tensor]:
    """Rename (and join) the tensors of a checkpoint; a missing or left-over tensor is an error."""
    src = dict(state)

    def take(name):
        if name not in src:
            raise KeyError(f"checkpoint has no tensor {name!r}")
        return src.pop(name)

    def join(prefix, names, suffix=""):
        return torch.cat([take(f"{prefix}{n}{suffix}") for n in names], dim=0)

    embed = take("embed")
    out = {"model.embed_tokens.weight": embed, "lm_head.weight": embed, "model.norm.weight": take("final.norm")}
    for i, layer in enumerate(config.layers):
        s, d = f"l{i}.", f"model.layers.{i}."
        mix, dst = s + "mix.", d + "mixer."
        for n in ("norm1", "norm1b"):
            out[f"{d}{n}.weight"] = take(s + n)
        if layer["type"] == "attention":
            out[dst + "in_proj.weight"], out[dst + "in_proj.bias"] = join(mix, "qkv"), join(mix, "qkv", ".b")
            if config.value_mix_role(i):
                out[dst + "value_share"] = take(mix + "vmix").reshape(())
        else:
            out[dst + "in_proj.weight"] = join(mix, "qkvg")
            out[dst + "gate_proj.weight"] = join(mix, "ba")
            out[dst + "conv"] = join(mix, "qkv", ".conv")
            out[dst + "A_log"], out[dst + "dt_bias"] = take(mix + "A_log"), take(mix + "dt_bias")
            out[dst + "norm.weight"] = take(mix + "norm")
        out[dst + "o_proj.weight"] = take(mix + "o")
        if layer.get("mlp") is None:
            continue
        for n in ("norm2", "norm2b"):
            out[f"{d}{n}.weight"] = take(s + n)
        for suffix, part in ((".b", "bias"), ("", "weight")):
            out[f"{d}mlp.gate_up_proj.{part}"] = interleave_gate_up(take(f"{s}mlp.gate{suffix}"), take(f"{s}mlp.up{suffix}"))
            out[f"{d}mlp.down_proj.{part}"] = take(f"{s}mlp.down{suffix}")
    if src:
        raise KeyError(f"checkpoint tensors that the configuration does not name: {sorted(src)[:5]}")
    return out


def register():
    """Make the configuration and model class known to the Auto classes (idempotent)."""
    from transformers import AutoConfig, AutoModelForCausalLM
    AutoConfig.register(LetaraxConfig.model_type, LetaraxConfig, exist_ok=True)
    AutoModelForCausalLM.register(LetaraxConfig, LetaraxForCausalLM, exist_ok=True)


def build(config_dict: dict, state: Dict[str, torch.Tensor], dtype: Optional[torch.dtype]):
    """A model from a raw checkpoint (``config.json`` dictionary and tensors)."""
    config = LetaraxConfig(**config_dict)
    config.architectures = [LetaraxForCausalLM.__name__]
    dtype = dtype if isinstance(dtype, torch.dtype) else torch.bfloat16
    with torch.device("meta"):
        model = LetaraxForCausalLM(config)
    tensors = {k: v.to(dtype) if v.is_floating_point() else v for k, v in convert_checkpoint(state, config).items()}
    model.load_state_dict(tensors, strict=True, assign=True)
    model.tie_weights()
    model.config.dtype = dtype
    return model.requires_grad_(False).eval()
