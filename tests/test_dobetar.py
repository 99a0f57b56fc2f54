"""Dobetar on the CPU: configuration, checkpoint conversion, the cache's slots, and the oracle the kernels are held to
(``tests/dobetar_oracle.py``).  The kernels themselves: ``tests/test_gpu_latent.py``."""
import json
import os

import pytest
import torch

import dobetar_oracle as O


def small_config(**kw):
    cfg = {"architecture": "Dobetar", "vocab": 90, "width": 48,
           "embedding": {"scale": 2.0, "bigram": {"buckets": 37, "mul_prev": 11, "mul_cur": 5}},
           "layers": [O.latent_layer(3, 16, 8, 12, 24, window=5, mlp=O.dense(40)),
                      O.latent_layer(2, 24, 4, 20, 32, window=9, base=500.0, mlp=O.moe(24, 5, 2)),
                      O.latent_layer(3, 16, 8, 12, 24, window=3, mlp=None)],
           "logit_softcap": 12.0, "norm": {"eps": 1e-5}}
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
    assert type(model).__name__ == "DobetarForCausalLM" and family_for(model).engine == "latent"
    assert model.config.vocab_size == 90 and model.config.hidden_size == 48 and model.config.num_hidden_layers == 3
    m0, m1 = model.model.layers[0].mixer, model.model.layers[1].mixer
    assert (m0.window, m1.window, m1.rot_base, m1.rot_pairs, m1.kv_rank) == (5, 9, 500.0, 2, 32)
    assert torch.equal(m0.qkv_a_proj.weight, torch.cat([w["l0.mix.q"], w["l0.mix.dkv"]]))
    ex = model.model.layers[1].mlp.experts
    assert not ex.interleaved                                       # 24 hidden units: no whole 16-row tiles
    assert torch.equal(ex.gate_up_rows[3], torch.cat([w["l1.mlp.e3.gate"], w["l1.mlp.e3.up"]]))
    assert model.model.layers[2].mlp is None and model.model.layers[2].norm2 is None
    bf = AutoModelForCausalLM.from_pretrained(str(tmp_path), load_in_low_bit="bf16", torch_dtype=torch.bfloat16)
    assert type(bf.model.layers[0].mixer.o_proj).__name__ == "BF16Linear"
    assert type(bf.model.layers[1].mlp.router) is torch.nn.Linear   # routers are not converted
    with pytest.raises(RuntimeError, match="CUDA"):
        model(torch.tensor([[1, 2, 3]]))


def test_gate_and_up_rows_alternate_in_tiles():
    from ipex_llm_b200.models.dobetar import interleave_gate_up
    g, u = torch.arange(32.0).view(32, 1), torch.arange(100.0, 132.0).view(32, 1)
    r = interleave_gate_up(g, u).flatten()
    assert torch.equal(r[:16], g[:16, 0]) and torch.equal(r[16:32], u[:16, 0])
    assert torch.equal(r[32:48], g[16:, 0]) and torch.equal(r[48:], u[16:, 0])


@pytest.mark.parametrize("fault", ["missing", "extra", "type", "kind", "rotation"])
def test_what_does_not_fit_is_an_error(fault):
    from ipex_llm_b200.models import dobetar
    cfg = small_config()
    w = O.random_weights(cfg)
    if fault == "missing":
        del w["l1.mlp.e4.down"]
    elif fault == "extra":
        w["l2.norm2"] = torch.ones(48)
    elif fault == "type":
        cfg["layers"][0]["type"] = "something_else"
    elif fault == "kind":
        cfg["layers"][0]["mlp"]["kind"] = "gated"
    else:
        cfg["layers"][0]["mixer"]["rot"]["dims"] = 10
    with pytest.raises((KeyError, ValueError)):
        dobetar.build(cfg, w, torch.float32)


def test_save_and_load_low_bit(tmp_path):
    """The package's own low-bit format: packed projections, dense experts and up-projections, same config."""
    from ipex_llm.transformers import AutoModelForCausalLM
    cfg = small_config(width=64)
    cfg["layers"] = [O.latent_layer(4, 16, 16, 16, 64, window=7, mlp=O.dense(128)),
                     O.latent_layer(4, 16, 16, 16, 64, window=7, mlp=O.moe(32, 4, 1))]
    src, dst = str(tmp_path / "src"), str(tmp_path / "dst")
    write_checkpoint(src, cfg, O.random_weights(cfg))
    model = AutoModelForCausalLM.from_pretrained(src, load_in_low_bit="sym_int4")
    assert type(model.model.layers[0].mixer.qkv_a_proj).__name__ == "LowBitLinear"
    model.save_low_bit(dst)
    again = AutoModelForCausalLM.load_low_bit(dst)
    a, b = model.state_dict(), again.state_dict()
    assert a.keys() == b.keys()
    for k in a:
        x, y = a[k], b[k]
        assert torch.equal(x.view(torch.uint8) if x.dtype == torch.uint8 else x.float(),
                           y.view(torch.uint8) if y.dtype == torch.uint8 else y.float()), k
    assert again.config.layers == cfg["layers"] and again.config.embedding == cfg["embedding"]


def test_rotary_table_matches_the_rotation():
    from ipex_llm_b200.ops.latent import rotary_table
    cos, sin = rotary_table(700, 300.0, 6, "cpu")
    x = torch.randn(700, 12, dtype=torch.float64)
    u, v = x[:, :6], x[:, 6:]
    mine = torch.cat([u * cos - v * sin, v * cos + u * sin], -1)
    assert torch.allclose(mine, O.rotate_half_pairs(x, torch.arange(700), 300.0, 12), atol=1e-6)


# ------------------------------------------------------------------------------------------------
# cache
# ------------------------------------------------------------------------------------------------
def test_cache_slots_are_given_back_and_reused():
    from ipex_llm_b200.ops.kv_cache import LatentCache
    c = LatentCache()
    assert c.allocate(2, 8, [24, 40], torch.float32, "cpu")
    assert not c.allocate(1, 8, [24, 40], torch.float32, "cpu")
    a, b = c.acquire(), c.acquire()
    assert (a, b) == (0, 1)
    with pytest.raises(RuntimeError):
        c.acquire()
    c.lengths[a] = 5
    c.layers[1]._k[a, 0, 4] = 7.0
    c.history[a, 4] = 3
    assert c.allocate(3, 20, [24, 40], torch.float32, "cpu")         # grows without losing what is there
    assert float(c.layers[1]._k[a, 0, 4, 0]) == 7.0 and int(c.history[a, 4]) == 3 and c.lengths == [5, 0, 0]
    assert c.layers[0]._k.shape == (3, 1, 20, 24) and c.layers[1]._k.shape == (3, 1, 20, 40)
    c.release(a)
    with pytest.raises(ValueError):
        c.release(a)
    assert c.acquire() == a and c.lengths[a] == 0 and c.acquire() == 2


def test_cache_batch_surgery_moves_the_history_too():
    from ipex_llm_b200.ops.kv_cache import LatentCache
    c = LatentCache()
    c.allocate(2, 6, [8], torch.float32, "cpu")
    c.set_first_rows([0, 2])
    c.advance_all(4)
    c.history[:, 3] = torch.tensor([10, 20], dtype=torch.int32)
    c.batch_repeat_interleave(2)
    assert c.history[:, 3].tolist() == [10, 10, 20, 20] and c.start.tolist() == [0, 0, 2, 2]
    c.reorder_cache(torch.tensor([3, 0, 2, 1]))
    assert c.history[:, 3].tolist() == [20, 10, 20, 10] and [c.first_row(i) for i in range(4)] == [2, 0, 2, 0]
    c.batch_select_indices(torch.tensor([1, 2]))
    assert c.history[:, 3].tolist() == [10, 20] and c.layers[0]._k.shape[0] == 2
    assert c.get_seq_length() == 4
    c.crop(3)
    assert c.get_seq_length() == 3 and c.lengths == [3, 3]


# ------------------------------------------------------------------------------------------------
# the oracle notices the mistakes it is there for
# ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("fault", ["window_plus_one", "window_minus_one", "renormalized", "weight_on_output"])
def test_a_planted_mistake_shows(fault):
    cfg = small_config()
    w = O.random_weights(cfg)
    toks = torch.randint(0, 90, (14,), generator=torch.Generator().manual_seed(1)).tolist()
    good, bad = O.forward(w, cfg, toks), O.forward(w, cfg, toks, faults=(fault,))
    assert (good - bad).abs().max() > 0.05


def test_oracle_prefix_property():
    """Logits at a position depend on nothing behind it, and the first token takes the extra bigram row."""
    cfg = small_config()
    w = O.random_weights(cfg)
    toks = [3, 80, 17, 17, 44, 2, 9]
    full = O.forward(w, cfg, toks)
    for n in (1, 2, 5):
        assert torch.allclose(full[:n], O.forward(w, cfg, toks[:n]), atol=1e-10)
    assert O.bigram_rows([3, 80, 17], 37, 11, 5) == [37, (3 * 11 + 80 * 5) % 37, (80 * 11 + 17 * 5) % 37]
