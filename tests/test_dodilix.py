"""Dodilix on the CPU: configuration, checkpoint conversion, the cache's layers, and the oracle the kernels are held to
(``tests/dodilix_oracle.py``).  The kernels themselves: ``tests/test_gpu_multistream.py``."""
import json
import os

import pytest
import torch

import dodilix_oracle as O


def small_config(**kw):
    cfg = {"architecture": "Dodilix", "vocab": 90, "width": 48, "norm": {"eps": 1e-5}, "streams": 3, "logit_scale": 0.75,
           "embedding": {"scale": 1.5},
           "layers": [O.latent_layer(3, 16, 8, 12, 20, 24, mlp=O.dense(40)),
                      O.parallel_layer(4, 2, 16, 12, 5, 8, lheads=2, ldim=12, lvdim=20, mlp=O.moe(24, 6, 3, (3, 2), 1.5, 16)),
                      O.latent_layer(2, 8, 8, 20, 28, 24, kv_from=0, mlp=O.moe(20, 4, 1)),
                      O.parallel_layer(3, 1, 16, 24, 7, 16, lheads=3, ldim=8, lvdim=8, tau=1.0, mlp=None)]}
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
    from ipex_llm_b200.engine import engine_class
    from ipex_llm_b200.models.registry import family_for
    cfg = small_config()
    w = O.random_weights(cfg)
    write_checkpoint(str(tmp_path), cfg, w)
    model = AutoModelForCausalLM.from_pretrained(str(tmp_path), torch_dtype=torch.float32)
    assert type(model).__name__ == "DodilixForCausalLM" and family_for(model).engine == "multistream"
    assert engine_class(model).__name__ == "MultiStreamEngine"
    assert model.config.vocab_size == 90 and model.config.hidden_size == 48 and model.config.num_hidden_layers == 4
    L = model.model.layers
    a, b = L[0].mixer, L[2].mixer
    assert (a.heads, a.dim, a.rot_dim, a.v_dim, a.q_rank, a.kv_rank, a.rot_pairs) == (3, 16, 8, 12, 20, 24, 4)
    dkv = w["l0.mix.dkv"]
    assert torch.equal(a.in_proj.weight, torch.cat([dkv[:24], dkv[24::2], dkv[25::2], w["l0.mix.g"]]))
    uq = w["l0.mix.uq"].view(3, 24, 20)
    assert torch.equal(a.q_up.weight.view(3, 24, 20), torch.cat([uq[:, :16], uq[:, 16::2], uq[:, 17::2]], 1))
    assert (b.kv_from, b.kv_norm, b.kv_rows) == (0, None, 0) and torch.equal(b.in_proj.weight, w["l2.mix.g"])
    p = L[1].mixer
    assert (p.left.chunk, p.left.rot_pairs, p.left.gate_scale, p.left.sink, p.left.gated) == (5, 4, 0.7, True, True)
    assert (p.right.rank, p.right.tau, p.right.out_scale, L[3].mixer.right.tau) == (6, 8.0, 0.9, 1.0)
    assert torch.equal(p.in_proj.weight, torch.cat([w[f"l1.mix.{s}.{c}"] for s in ("left", "right") for c in "qkvg"]))
    assert torch.equal(p.o_proj.weight, torch.cat([w["l1.mix.left.o"], w["l1.mix.right.o"]], 1))
    assert torch.equal(p.decay_up, w["l1.mix.right.a2"]) and torch.equal(p.decay_bias, w["l1.mix.right.a2.b"])
    assert torch.equal(L[1].hyper2.mix, w["l1.hc2.mix"]) and L[3].hyper2 is None and L[3].mlp is None
    f = L[1].mlp
    assert (f.top_k, f.groups, f.keep, f.scale) == (3, 3, 2, 1.5) and f.router.weight.shape == (7, 48)
    assert torch.equal(f.router.weight[6:], w["l1.mlp.shared.sg"])
    g, u = w["l1.mlp.e4.gate"], w["l1.mlp.e4.up"]
    assert torch.equal(f.experts.gate_up_rows[4, :24], torch.cat([g[:8], u[:8], g[8:16]]))
    assert L[2].mlp.shared is None and torch.equal(L[2].mlp.experts.gate_up_rows[1, :20], w["l2.mlp.e1.gate"])
    bf = AutoModelForCausalLM.from_pretrained(str(tmp_path), load_in_low_bit="bf16", torch_dtype=torch.bfloat16)
    m = bf.model.layers
    assert type(m[0].mixer.q_up).__name__ == "BF16Linear"
    for dense in (m[0].mixer.q_down, m[1].mixer.decay_down, m[1].mlp.router):    # 32-bit results, routers: not converted
        assert type(dense) is torch.nn.Linear
    with pytest.raises(RuntimeError, match="CUDA"):
        model(torch.tensor([[1, 2, 3]]))


@pytest.mark.parametrize("fault", ["missing", "extra", "type", "kind", "heads", "lender", "borrowed lender", "other rank",
                                   "rotation", "groups", "streams"])
def test_what_does_not_fit_is_an_error(fault):
    from ipex_llm_b200.models import dodilix
    cfg = small_config()
    w = O.random_weights(cfg)
    if fault == "missing":
        del w["l1.hc2.out"]
    elif fault == "extra":
        w["l3.norm2"] = torch.zeros(48)
    elif fault == "type":
        cfg["layers"][0]["type"] = "something_else"
    elif fault == "kind":
        cfg["layers"][0]["mlp"]["kind"] = "sparse"
    elif fault == "heads":
        cfg["layers"][1]["mixer"]["left"]["heads"] = 5
    elif fault == "lender":
        cfg["layers"][2]["mixer"]["kv_from"] = 1
    elif fault == "borrowed lender":
        cfg["layers"].append(O.latent_layer(2, 8, 8, 20, 28, 24, kv_from=2))
    elif fault == "other rank":
        cfg["layers"][2]["mixer"]["kv_rank"] = 16
    elif fault == "rotation":
        cfg["layers"][3]["mixer"]["left"]["rot"]["dims"] = 18
    elif fault == "groups":
        cfg["layers"][1]["mlp"]["router"]["top"] = 5
    else:
        cfg["streams"] = 17
    with pytest.raises((KeyError, ValueError)):
        dodilix.build(cfg, w, torch.float32)


@pytest.mark.parametrize("low_bit", [False, True])
def test_save_and_load(tmp_path, low_bit):
    """The package's own formats: packed (or plain) projections, dense experts, same configuration with the decays' rank."""
    from ipex_llm.transformers import AutoModelForCausalLM
    cfg = small_config(width=64)
    cfg["layers"] = [O.latent_layer(4, 16, 16, 16, 64, 64, mlp=O.dense(128)),
                     O.parallel_layer(4, 2, 16, 16, 7, 8, lheads=4, ldim=16, lvdim=16, mlp=O.moe(32, 4, 1, None, 1.0, 32))]
    src, dst = str(tmp_path / "src"), str(tmp_path / "dst")
    write_checkpoint(src, cfg, O.random_weights(cfg, rank=9))
    if low_bit:
        model = AutoModelForCausalLM.from_pretrained(src, load_in_low_bit="sym_int4")
        assert type(model.model.layers[1].mixer.in_proj).__name__ == "LowBitLinear"
        model.save_low_bit(dst)
        again = AutoModelForCausalLM.load_low_bit(dst)
    else:
        from transformers import AutoModelForCausalLM as Plain
        model = AutoModelForCausalLM.from_pretrained(src, torch_dtype=torch.float32)
        model.save_pretrained(dst)
        again = Plain.from_pretrained(dst, dtype=torch.float32)
    a, b = model.state_dict(), again.state_dict()
    assert a.keys() == b.keys()
    for k in a:
        x, y = a[k], b[k]
        assert torch.equal(x.view(torch.uint8) if x.dtype == torch.uint8 else x.float(),
                           y.view(torch.uint8) if y.dtype == torch.uint8 else y.float()), k
    assert again.config.layers == model.config.layers and again.config.streams == 3
    assert again.config.layers[1]["mixer"]["right"]["rank"] == 9 == again.model.layers[1].mixer.decay_up.shape[1]


def test_drafting_needs_a_model_without_states():
    from ipex_llm_b200.models import dodilix
    from ipex_llm_b200.transformers.generation import ipex_generate
    cfg = small_config()
    model = dodilix.build(cfg, O.random_weights(cfg), torch.float32)
    with pytest.raises(NotImplementedError, match="earlier token"):
        ipex_generate(model, torch.tensor([[1, 2]]), lookahead=2)
    cfg["layers"] = [cfg["layers"][0], cfg["layers"][2] | {"mixer": cfg["layers"][2]["mixer"]}]
    cfg["layers"][1]["mlp"] = None
    assert dodilix.build(cfg, O.random_weights(cfg), torch.float32)._ipex_rolls_back


# ------------------------------------------------------------------------------------------------
# rotation and cache
# ------------------------------------------------------------------------------------------------
def test_reordered_pairs_turn_like_neighbours():
    """Rows in the order of ``split_pairs`` turn as pairs (i, i + half): the same values in another order."""
    from ipex_llm_b200.models.dodilix import split_pairs
    x = torch.randn(9, 14, dtype=torch.float64)
    pos = torch.arange(9)
    order = split_pairs(torch.arange(14).view(14, 1), 5).flatten()
    assert order.tolist() == [0, 2, 4, 6, 8, 1, 3, 5, 7, 9, 10, 11, 12, 13]
    want = O.turn_neighbours(x, pos, 77.0, 10)[:, order]
    assert torch.allclose(O.turn_half(x[:, order], pos, 77.0, 10), want)


def test_states_without_convolutions_in_the_cache():
    from ipex_llm_b200.ops.kv_cache import DeltaStateShape, KeyValueShape, SlotCache
    shapes = [24, KeyValueShape(2, 6, 3), DeltaStateShape(3, 4, 5, 0, 0)]
    c = SlotCache()
    assert c.allocate(2, 8, shapes, torch.bfloat16, "cpu")
    lat, kv, st = c.layers
    assert lat._k.shape == (2, 1, 8, 24) and kv._v.shape == (2, 2, 8, 3) and st._k.shape == (2, 3, 4, 5)
    assert st._k.dtype == torch.float32 and st._v.numel() == 0
    c.advance_all(4)
    for b in range(2):
        st._k[b], lat._k[b] = b + 1.0, b + 1.0
    c.batch_repeat_interleave(2)
    c.reorder_cache(torch.tensor([3, 0, 2, 1]))
    assert [float(st._k[b, 0, 0, 0]) for b in range(4)] == [2, 1, 2, 1] == [float(lat._k[b, 0, 0, 0]) for b in range(4)]
    assert c.allocate(6, 20, shapes, torch.bfloat16, "cpu") and float(st._k[2, 1, 1, 1]) == 2.0
    with pytest.raises(NotImplementedError):
        c.crop(3)


# ------------------------------------------------------------------------------------------------
# the oracle notices the mistakes it is there for
# ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("fault", ["mix_transposed", "chunk_plus_one", "chunk_minus_one", "no_rotation", "other_pairs",
                                   "no_unit_norm", "heads_interleaved", "no_sink", "no_gate", "decay_after_write",
                                   "read_before_write", "no_decay", "one_decay_per_head", "other_latent_pairs",
                                   "no_latent_gate", "no_groups", "not_renormalized", "shared_ungated"])
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


def test_oracle_pieces_by_hand():
    e = torch.eye(4, dtype=torch.float64)
    k = e[[0, 1, 0]].view(3, 1, 4)
    v = torch.randn(3, 1, 2, dtype=torch.float64)
    half = torch.full((3, 1, 4), 0.5, dtype=torch.float64)
    o, S = O.linear_rule(k, k, v, half)
    assert torch.allclose(S[0, 0], v[2, 0] + 0.25 * v[0, 0]) and torch.allclose(S[0, 1], 0.5 * v[1, 0])
    assert torch.allclose(o[2], v[2] + 0.25 * v[0])
    vis = O.chunk_visible(7, 3)
    assert vis[2].tolist() == [True] * 3 + [False] * 4 and vis[3].tolist() == [False] * 3 + [True] + [False] * 3
    s = torch.tensor([[[-1.0, 2.0, 0.5]]], dtype=torch.float64)
    p = O.sink_softmax(s, torch.tensor([[True, True, False]]), torch.tensor([0.25], dtype=torch.float64))
    z = torch.exp(torch.tensor([-1.0, 2.0], dtype=torch.float64))
    assert torch.allclose(p[0, 0, :2], z / (torch.exp(torch.tensor(0.25)) + z.sum())) and float(p[0, 0, 2]) == 0.0
    r = {"experts": 4, "top": 2, "groups": {"count": 2, "keep": 1}, "scale": 3.0}
    val, idx = O.route(torch.tensor([[0.0, 2.0, 1.9, 1.8]], dtype=torch.float64), r)
    assert idx.tolist() == [[1, 0]] and torch.allclose(val.sum(), torch.tensor(3.0, dtype=torch.float64))
    assert torch.allclose(val[0, 0] / val[0, 1], torch.exp(torch.tensor(2.0, dtype=torch.float64)))
    x = torch.randn(2, 3, 5, dtype=torch.float64)
    y = torch.randn(2, 5, dtype=torch.float64)
    mix, out = torch.randn(3, 3, dtype=torch.float64), torch.randn(3, dtype=torch.float64)
    new = O.spread_streams(x, y, mix, out)
    assert torch.allclose(new[1, 2], sum(mix[s, 2] * x[1, s] for s in range(3)) + out[2] * y[1])
    assert torch.allclose(O.channel_decay(torch.tensor(-2.0), 4.0), torch.sigmoid(torch.tensor(-2.0)) ** 0.25)
