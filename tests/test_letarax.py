"""Letarax on the CPU: configuration, checkpoint conversion, the cache's layers and slots, and the oracle the kernels are held
to (``tests/letarax_oracle.py``).  The kernels themselves: ``tests/test_gpu_hybrid.py``."""
import json
import os

import pytest
import torch

import letarax_oracle as O


def small_config(**kw):
    cfg = {"architecture": "Letarax", "vocab": 90, "width": 48, "norm": {"eps": 1e-5},
           "layers": [O.attention_layer(4, 2, 16, 12, window=5, ff=40),
                      O.delta_layer(4, 2, 12, 20, conv=3),
                      O.attention_layer(6, 2, 8, 12, window=9, ff=None),
                      O.attention_layer(3, 1, 16, 24, window=4, v_mix=False, ff=20),
                      O.delta_layer(3, 3, 16, 8, conv=4, ff=24)]}
    cfg.update(kw)
    return cfg


def write_checkpoint(path, cfg, w):
    from safetensors.torch import save_file
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.to(torch.bfloat16).contiguous() for k, v in w.items()}, os.path.join(path, "model.safetensors"))


def test_checkpoint_loads_through_the_auto_class(tmp_path):
    from ipex_llm.transformers import AutoModelForCausalLM
    from ipex_llm_b200.models.registry import family_for
    cfg = small_config()
    w = O.random_weights(cfg)
    write_checkpoint(str(tmp_path), cfg, w)
    model = AutoModelForCausalLM.from_pretrained(str(tmp_path), torch_dtype=torch.float32)
    assert type(model).__name__ == "LetaraxForCausalLM" and family_for(model).engine == "hybrid"
    assert model.config.vocab_size == 90 and model.config.hidden_size == 48 and model.config.num_hidden_layers == 5
    L = model.model.layers
    a = L[0].mixer
    assert (a.spec.heads, a.spec.kv_heads, a.spec.dim, a.spec.vdim, a.spec.window, a.spec.sink) == (4, 2, 16, 12, 5, True)
    assert [L[i].mixer.mix_role for i in (0, 2, 3)] == ["first", "mixed", None] and L[3].mixer.value_share is None
    assert torch.equal(a.in_proj.weight, torch.cat([w[f"l0.mix.{c}"] for c in "qkv"]))
    assert torch.equal(a.in_proj.bias, torch.cat([w[f"l0.mix.{c}.b"] for c in "qkv"]))
    assert torch.equal(L[2].mixer.value_share, w["l2.mix.vmix"])
    d = L[1].mixer
    assert (d.spec.taps, d.spec.channels, d.spec.rows) == (3, 2 * 2 * 12 + 80, 2 * 2 * 12 + 160)
    assert torch.equal(d.gate_proj.weight, torch.cat([w["l1.mix.b"], w["l1.mix.a"]]))
    assert torch.equal(d.conv, torch.cat([w[f"l1.mix.{c}.conv"] for c in "qkv"]))
    assert L[1].mlp is None and L[1].norm2 is None and L[4].mlp.interleaved
    assert torch.equal(model.lm_head.weight, w["embed"])
    bf = AutoModelForCausalLM.from_pretrained(str(tmp_path), load_in_low_bit="bf16", torch_dtype=torch.bfloat16)
    assert type(bf.model.layers[1].mixer.o_proj).__name__ == "BF16Linear"
    assert type(bf.model.layers[1].mixer.gate_proj) is torch.nn.Linear      # what steers the recurrence stays dense
    with pytest.raises(RuntimeError, match="CUDA"):
        model(torch.tensor([[1, 2, 3]]))


@pytest.mark.parametrize("ff,order", [(24, None), (20, "cat")])
def test_gate_and_up_rows_alternate_in_blocks_of_eight(ff, order):
    from ipex_llm_b200.models.letarax import interleave_gate_up
    g, u = torch.arange(float(ff)), torch.arange(100.0, 100.0 + ff)
    for r in (interleave_gate_up(g, u), interleave_gate_up(g.view(-1, 1), u.view(-1, 1)).flatten()):
        if order == "cat":
            assert torch.equal(r, torch.cat([g, u]))
        else:
            assert torch.equal(r[:8], g[:8]) and torch.equal(r[8:16], u[:8]) and torch.equal(r[40:], u[16:])


@pytest.mark.parametrize("fault", ["missing", "extra", "type", "kind", "heads", "shared values"])
def test_what_does_not_fit_is_an_error(fault):
    from ipex_llm_b200.models import letarax
    cfg = small_config()
    w = O.random_weights(cfg)
    if fault == "missing":
        del w["l4.mix.k.conv"]
    elif fault == "extra":
        w["l3.mix.vmix"] = torch.zeros(())
    elif fault == "type":
        cfg["layers"][0]["type"] = "something_else"
    elif fault == "kind":
        cfg["layers"][0]["mlp"]["kind"] = "sparse"
    elif fault == "heads":
        cfg["layers"][1]["mixer"]["heads"] = 5
    else:
        cfg["layers"][2]["mixer"]["vdim"] = 16
    with pytest.raises((KeyError, ValueError)):
        letarax.build(cfg, w, torch.float32)


def test_save_and_load_low_bit(tmp_path):
    """The package's own low-bit format: packed projections, dense gates, same config."""
    from ipex_llm.transformers import AutoModelForCausalLM
    cfg = small_config(width=64)
    cfg["layers"] = [O.delta_layer(4, 2, 16, 16), O.attention_layer(4, 2, 16, 16, window=7, ff=128)]
    src, dst = str(tmp_path / "src"), str(tmp_path / "dst")
    write_checkpoint(src, cfg, O.random_weights(cfg))
    model = AutoModelForCausalLM.from_pretrained(src, load_in_low_bit="sym_int4")
    assert type(model.model.layers[1].mixer.in_proj).__name__ == "LowBitLinear"
    model.save_low_bit(dst)
    again = AutoModelForCausalLM.load_low_bit(dst)
    a, b = model.state_dict(), again.state_dict()
    assert a.keys() == b.keys()
    for k in a:
        x, y = a[k], b[k]
        assert torch.equal(x.view(torch.uint8) if x.dtype == torch.uint8 else x.float(),
                           y.view(torch.uint8) if y.dtype == torch.uint8 else y.float()), k
    assert again.config.layers == cfg["layers"]


def test_save_pretrained_round_trip(tmp_path):
    from transformers import AutoModelForCausalLM
    from ipex_llm_b200.models import letarax
    cfg = small_config()
    model = letarax.build(cfg, O.random_weights(cfg), torch.float32)
    model.save_pretrained(str(tmp_path))
    again = AutoModelForCausalLM.from_pretrained(str(tmp_path), dtype=torch.float32)
    for k, v in model.state_dict().items():
        assert torch.equal(v, again.state_dict()[k]), k
    assert again.lm_head.weight.data_ptr() == again.model.embed_tokens.weight.data_ptr()


# ------------------------------------------------------------------------------------------------
# cache
# ------------------------------------------------------------------------------------------------
def mixed_cache(slots=2, capacity=8):
    from ipex_llm_b200.ops.kv_cache import DeltaStateShape, KeyValueShape, SlotCache
    shapes = [DeltaStateShape(3, 4, 5, 2, 39), KeyValueShape(2, 6, 3)]
    c = SlotCache()
    assert c.allocate(slots, capacity, shapes, torch.bfloat16, "cpu")
    return c, shapes


def test_cache_of_keys_values_and_states():
    c, shapes = mixed_cache()
    d, a = c.layers
    assert d._k.shape == (2, 3, 4, 5) and d._k.dtype == torch.float32 and d._v.shape == (2, 1, 2, 39)
    assert a._k.shape == (2, 2, 8, 6) and a._v.shape == (2, 2, 8, 3) and a._k.dtype == torch.bfloat16
    s, t = c.acquire(), c.acquire()
    d._k[t], a._v[t, 1, 7] = 3.0, 2.0
    assert c.allocate(3, 20, shapes, torch.bfloat16, "cpu")              # grows without losing what is there
    assert float(d._k[t].sum()) == 180.0 and float(a._v[t, 1, 7].sum()) == 6.0
    assert d._k.shape[0] == 3 and a._k.shape == (3, 2, 20, 6) and c.capacity == 20
    state = d._k
    c.allocate(3, 40, shapes, torch.bfloat16, "cpu")
    assert d._k is state                                                  # its size does not depend on the length
    c.release(s)
    assert c.acquire() == s and c.acquire() == 2
    assert [x is y for x, y in zip(c.step_state(), (d._k, d._v))] == [True, True]


def test_batch_surgery_moves_states_and_rows():
    c, _ = mixed_cache()
    d, a = c.layers
    c.advance_all(4)
    for b in range(2):
        d._k[b], d._v[b], a._k[b] = b + 1.0, b + 1.0, b + 1.0
    c.batch_repeat_interleave(2)
    assert [float(d._k[b, 0, 0, 0]) for b in range(4)] == [1, 1, 2, 2] and d._v.shape[0] == 4
    c.reorder_cache(torch.tensor([3, 0, 2, 1]))
    assert [float(d._v[b, 0, 0, 0]) for b in range(4)] == [2, 1, 2, 1] == [float(a._k[b, 0, 0, 0]) for b in range(4)]
    c.batch_select_indices(torch.tensor([1, 2]))
    assert [float(d._k[b, 0, 0, 0]) for b in range(2)] == [1, 2] and c.get_seq_length() == 4
    c.crop(4)
    with pytest.raises(NotImplementedError):
        c.crop(3)                                                         # a state does not go back
    c.release_all()
    assert c.get_seq_length() == 0 and c.acquire() == 0


def test_drafting_strategies_are_refused():
    from ipex_llm_b200.models import letarax
    from ipex_llm_b200.transformers.generation import ipex_generate
    cfg = small_config()
    model = letarax.build(cfg, O.random_weights(cfg), torch.float32)
    with pytest.raises(NotImplementedError, match="earlier token"):
        ipex_generate(model, torch.tensor([[1, 2]]), lookahead=2)


# ------------------------------------------------------------------------------------------------
# the oracle notices the mistakes it is there for
# ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("fault", ["window_plus_one", "window_minus_one", "no_sink", "no_value_mixing", "heads_interleaved",
                                   "read_before_write", "no_decay"])
def test_a_planted_mistake_shows(fault):
    cfg = small_config()
    w = O.random_weights(cfg)
    toks = torch.randint(0, 90, (14,), generator=torch.Generator().manual_seed(1)).tolist()
    good, bad = O.forward(w, cfg, toks), O.forward(w, cfg, toks, faults=(fault,))
    assert (good - bad).abs().max() > 0.05


def test_oracle_prefix_property():
    """Logits at a position depend on nothing behind it."""
    cfg = small_config()
    w = O.random_weights(cfg)
    toks = [3, 80, 17, 17, 44, 2, 9]
    full = O.forward(w, cfg, toks)
    for n in (1, 2, 5):
        assert torch.allclose(full[:n], O.forward(w, cfg, toks[:n]), atol=1e-10)


def test_oracle_recurrence_against_its_sum():
    """Without decay and with orthonormal keys, writing once stores v exactly and writing again replaces it."""
    H, D, V = 2, 6, 3
    e = torch.eye(D, dtype=torch.float64)
    k = e[[0, 1, 0, 5]].view(4, 1, D).expand(4, H, D)
    v = torch.randn(4, H, V, dtype=torch.float64)
    one = torch.ones(4, H, dtype=torch.float64)
    _, S = O.delta_rule(k, k, v, one, one)
    assert torch.allclose(S[:, 0], v[2]) and torch.allclose(S[:, 1], v[1]) and torch.allclose(S[:, 5], v[3])
    o, S2 = O.delta_rule(k[2:], k[2:], v[2:], one[2:], 0.5 * one[2:], state=S)
    assert torch.allclose(o, v[2:]) and torch.allclose(S2[:, 1], 0.25 * v[1])
    x = torch.randn(5, 4, dtype=torch.float64)
    taps = torch.randn(4, 3, dtype=torch.float64)
    assert torch.allclose(O.short_conv(x, taps)[2], (x[:3].T * taps).sum(1))
    assert torch.allclose(O.short_conv(x, taps)[0], x[0] * taps[:, 2])
    p = O.sink_softmax(torch.tensor([[-1.0, 2.0, 0.5]]), torch.tensor([[True, True, False]]))
    z = torch.exp(torch.tensor([-1.0, 2.0]))
    assert torch.allclose(p[0, :2], z / (1 + z.sum())) and float(p[0, 2]) == 0.0
