"""Gegorax on the CPU: configuration, checkpoint conversion, the cache's layers, and the oracle the kernels are held to
(``tests/gegorax_oracle.py``).  The kernels themselves: ``tests/test_gpu_parallel_block.py``."""
import json
import math
import os

import pytest
import torch

import gegorax_oracle as O


def small_config(**kw):
    cfg = {"architecture": "Gegorax", "vocab": 90, "width": 48, "norm": {"eps": 1e-5}, "token_side": {"dim": 6},
           "layers": [O.delta_layer(3, 16, mlp=O.dense(40)),
                      O.parallel_layer(4, 2, 16, 12, 5, 3, 8, rheads=6, rvdim=8, state=10, groups=2, conv=3, norm_groups=4,
                                       mlp=O.moe(24, 6, 3, 0.8, 16, 1.3)),
                      O.delta_layer(2, 20, mlp=O.moe(20, 4, 1, 1.0)),
                      O.parallel_layer(3, 1, 16, 24, 4, 2, 16, rheads=3, rvdim=12, state=8, groups=3, conv=4, norm_groups=1,
                                       mlp=O.dense(24)),
                      O.delta_layer(1, 24, mlp=None), O.parallel_layer(2, 2, 8, 8, 3, 4, 4, rheads=2, rvdim=8, state=6, groups=1,
                                                                       conv=2, norm_groups=2, mlp=None)]}
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
    w = O.random_weights(cfg, rank=7)
    write_checkpoint(str(tmp_path), cfg, w)
    model = AutoModelForCausalLM.from_pretrained(str(tmp_path), torch_dtype=torch.float32)
    assert type(model).__name__ == "GegoraxForCausalLM" and family_for(model).engine == "parallel_block"
    assert engine_class(model).__name__ == "ParallelBlockEngine"
    assert model.config.vocab_size == 90 and model.config.hidden_size == 48 and model.config.num_hidden_layers == 6
    L = model.model.layers
    a, b = L[0].mixer, L[1].mixer
    assert (a.spec.heads, a.spec.dim, a.spec.vdim, a.spec.rank) == (3, 16, 16, 7) and a.spec.decay == math.exp(-0.5)
    assert torch.equal(L[0].in_proj.weight, torch.cat([w[f"l0.mix.{c}"] for c in "rkvag"] + [w["l0.mlp.up"]]))
    assert torch.equal(L[0].out_proj.weight, torch.cat([w["l0.mix.o"], w["l0.mlp.down"]], 1))
    assert torch.equal(L[0].low_proj.weight, w["l0.mix.w1"]) and torch.equal(a.decay_up, w["l0.mix.w2"])
    assert torch.equal(a.decay_bias, w["l0.mix.w0"]) and torch.equal(a.rate_bias, w["l0.mix.a.b"])
    s, r = b.left, b.right
    assert (s.window, s.pool, s.rot_pairs, s.heads, s.kv_heads, s.sink, s.gated) == (5, 3, 4, 4, 2, False, False)
    assert (r.heads, r.vdim, r.state, r.groups, r.taps, r.parts, r.channels) == (6, 8, 10, 2, 3, 4, 88)
    q = w["l1.mix.left.q"].view(4, 16, 48)
    order = [0, 2, 4, 6, 1, 3, 5, 7, *range(8, 16)]
    assert torch.equal(L[1].in_proj.weight[:64].view(4, 16, 48), q[:, order])
    assert torch.equal(b.q_norm.weight, w["l1.mix.left.q.norm"][order])
    inn = w["l1.mix.right.in"]
    assert torch.equal(L[1].in_proj.weight[s.rows:], torch.cat([inn[48:136], inn[:48]]))
    assert torch.equal(L[1].low_proj.weight, torch.cat([inn[136:], w["l1.mlp.router"]])) and L[1].out_proj is None
    assert torch.equal(b.skip, w["l1.mix.right.D"]) and torch.equal(b.conv_bias, w["l1.mix.right.conv.b"])
    f = L[1].moe
    assert (f.top_k, f.limit, f.shared_limit) == (3, 0.8, 1.3) and torch.equal(f.router_bias, w["l1.mlp.router.b"])
    g, u = w["l1.mlp.e4.gate"], w["l1.mlp.e4.up"]
    assert torch.equal(f.experts.gate_up_rows[4, :24], torch.cat([g[:8], u[:8], g[8:16]]))
    assert L[2].moe.shared is None and torch.equal(L[2].moe.experts.gate_up_rows[1, :20], w["l2.mlp.e1.gate"])
    assert torch.equal(L[3].out_proj.weight, w["l3.mlp.down"]) and L[4].moe is None and L[5].out_proj is None
    assert torch.equal(model.model.side_table, w["side.embed"]) and torch.equal(L[3].side.proj.weight, w["l3.side.proj"])
    bf = AutoModelForCausalLM.from_pretrained(str(tmp_path), load_in_low_bit="bf16", torch_dtype=torch.bfloat16)
    m = bf.model.layers
    assert type(m[0].in_proj).__name__ == "BF16Linear"
    for dense in (m[0].low_proj, m[1].low_proj, m[2].side.gate):    # 32-bit results, token sides: not converted
        assert type(dense) is torch.nn.Linear
    with pytest.raises(RuntimeError, match="CUDA"):
        model(torch.tensor([[1, 2, 3]]))


def test_a_model_without_token_sides():
    from ipex_llm_b200.models import gegorax
    cfg = small_config(token_side=None)
    model = gegorax.build(cfg, O.random_weights(cfg), torch.float32)
    assert model.model.side_table is None and model.model.layers[0].side is None


@pytest.mark.parametrize("fault", ["missing", "extra", "type", "kind", "heads", "groups", "parts", "rotation", "pool", "top"])
def test_what_does_not_fit_is_an_error(fault):
    from ipex_llm_b200.models import gegorax
    cfg = small_config()
    w = O.random_weights(cfg)
    p = cfg["layers"][1]
    if fault == "missing":
        del w["l1.mix.right.D"]
    elif fault == "extra":
        w["l3.norm2"] = torch.zeros(48)
    elif fault == "type":
        cfg["layers"][0]["type"] = "something_else"
    elif fault == "kind":
        cfg["layers"][0]["mlp"]["kind"] = "sparse"
    elif fault == "heads":
        p["mixer"]["left"]["heads"] = 5
    elif fault == "groups":
        p["mixer"]["right"]["groups"] = 4
    elif fault == "parts":
        p["mixer"]["right"]["norm_groups"] = 5
    elif fault == "rotation":
        p["mixer"]["left"]["rot"]["dims"] = 18
    elif fault == "pool":
        p["mixer"]["left"]["mask"]["size"] = 0
    else:
        p["mlp"]["router"]["top"] = 7
    with pytest.raises((KeyError, ValueError)):
        gegorax.build(cfg, w, torch.float32)


@pytest.mark.parametrize("low_bit", [False, True])
def test_save_and_load(tmp_path, low_bit):
    """The package's own formats: packed (or plain) projections, dense experts, same configuration with the decays' rank."""
    from ipex_llm.transformers import AutoModelForCausalLM
    cfg = small_config(width=64)
    cfg["layers"] = [O.delta_layer(4, 16, mlp=O.dense(64)),
                     O.parallel_layer(4, 2, 16, 16, 7, 3, 8, rheads=4, rvdim=16, state=16, groups=2, mlp=O.moe(32, 4, 1, 1.0, 32))]
    src, dst = str(tmp_path / "src"), str(tmp_path / "dst")
    write_checkpoint(src, cfg, O.random_weights(cfg, rank=9))
    if low_bit:
        model = AutoModelForCausalLM.from_pretrained(src, load_in_low_bit="sym_int4")
        assert type(model.model.layers[1].in_proj).__name__ == "LowBitLinear"
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
    assert again.config.layers == model.config.layers and again.config.side_dim == 6
    assert again.config.layers[0]["mixer"]["rank"] == 9 == again.model.layers[0].mixer.decay_up.shape[1]


def test_drafting_needs_a_model_without_states():
    from ipex_llm_b200.models import gegorax
    from ipex_llm_b200.transformers.generation import ipex_generate
    cfg = small_config()
    model = gegorax.build(cfg, O.random_weights(cfg), torch.float32)
    with pytest.raises(NotImplementedError, match="earlier token"):
        ipex_generate(model, torch.tensor([[1, 2]]), lookahead=2)


def test_blocks_in_the_cache():
    """Rows of pooled blocks grow, move and are lent like the rows of tokens, a row per block."""
    from ipex_llm_b200.ops.kv_cache import DeltaStateShape, KeyValueShape, PooledShape, SlotCache
    shapes = [KeyValueShape(2, 6, 4), PooledShape(2, 6, 4, 5), DeltaStateShape(3, 4, 8, 3, 10)]
    c = SlotCache()
    assert c.allocate(2, 23, shapes, torch.bfloat16, "cpu")
    kv, pool, st = c.layers
    assert kv._k.shape == (2, 2, 23, 6) and pool._k.shape == (2, 2, 4, 6) and pool._v.shape == (2, 2, 4, 4)
    for b in range(2):
        pool._k[b], st._k[b] = b + 1.0, b + 1.0
    c.advance_all(21)
    assert pool._k.shape[2] == 4 and pool.get_seq_length() == 21
    c.reserve(10)
    assert c.layers[1]._k.shape[2] >= 6 and float(pool._k[1, 1, 3, 0]) == 2.0
    c.batch_repeat_interleave(2)
    c.reorder_cache(torch.tensor([3, 0, 2, 1]))
    assert [float(pool._k[b, 0, 0, 0]) for b in range(4)] == [2, 1, 2, 1] == [float(st._k[b, 0, 0, 0]) for b in range(4)]
    with pytest.raises(NotImplementedError):
        c.crop(3)


def test_packed_rows_of_blocks():
    from ipex_llm_b200.engine.stream_engine import Portions
    t = torch.tensor([20, 3, 90, 16], dtype=torch.int32)
    for lengths in (None, t.tolist()):
        p = Portions(torch.zeros(4, dtype=torch.int32), t, 90, True, t, t, 7, lengths)
        rows, n = p.pool_rows(5)
        assert rows.tolist() == [0, 8, 8, 32] and n == 40 and rows.dtype == torch.int32
        assert p.pool_rows(100)[1] == 8 and p.pool_rows(5)[0] is rows


# ------------------------------------------------------------------------------------------------
# the oracle notices the mistakes it is there for
# ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("fault", [
    "other_pairs", "window_plus_one", "window_minus_one", "no_blocks", "block_early", "block_late", "partial_blocks", "no_rotation",
    "norm_after_rotation", "no_norm", "block_sums", "heads_interleaved", "groups_interleaved", "unscaled_input", "read_before_write",
    "no_skip", "gate_after_norm", "one_norm_group", "no_conv_bias", "sides_unnormed", "no_unit_key", "removal_after_decay",
    "one_rate_per_head", "no_removal", "unit_write", "no_tanh", "one_decay_per_head", "silu_gate", "no_clamp", "no_plus_one",
    "softmax_over_all", "no_router_bias", "no_shared", "shared_limit", "sequential", "no_side", "side_of_layer_0"])
def test_a_planted_mistake_shows(fault):
    cfg = small_config()
    w = O.random_weights(cfg)
    toks = torch.randint(0, 90, (17,), generator=torch.Generator().manual_seed(1)).tolist()
    good, bad = O.forward(w, cfg, toks), O.forward(w, cfg, toks, faults=(fault,))
    assert (good - bad).abs().max() > 0.05


def test_oracle_prefix_property():
    """Logits at a position depend on nothing behind it."""
    cfg = small_config()
    w = O.random_weights(cfg)
    toks = [3, 80, 17, 17, 44, 2, 9, 60, 61, 5, 7, 7]
    full = O.forward(w, cfg, toks)
    for n in (1, 2, 5, 9):
        assert torch.allclose(full[:n], O.forward(w, cfg, toks[:n]), atol=1e-10)


def test_oracle_pieces_by_hand():
    tok, blk = O.visible(12, 4, 3)
    assert tok[6].tolist() == [False] * 3 + [True] * 4 + [False] * 5
    assert blk[5].tolist() == [False] * 4 and blk[6].tolist() == [True, False, False, False]     # 0..2 have left behind 6
    assert blk[8].tolist() == [True, False, False, False] and blk[9].tolist() == [True, True, False, False]
    # generalized delta: a unit key written twice is replaced by the rate, other keys only decay
    e = torch.eye(4, dtype=torch.float64)
    k = e[[0, 1, 0]].view(3, 1, 4) * math.sqrt(1 - 1e-6)
    v = torch.randn(3, 1, 2, dtype=torch.float64)
    half, rate = torch.full((3, 1, 4), 0.5, dtype=torch.float64), torch.full((3, 1, 4), 0.25, dtype=torch.float64)
    o, S = O.general_delta_rule(k, k, v, half, rate)
    c = math.sqrt(1 - 1e-6)
    first = c * v[0, 0]                                      # row 0 after the first token
    second = 0.5 * first                                     # ... after the second: decayed, key 1 does not touch it
    third = 0.5 * second - 0.25 * c * c * second + c * v[2, 0]
    assert torch.allclose(S[0, 0], third, atol=1e-8) and torch.allclose(S[0, 1], 0.5 * c * v[1, 0], atol=1e-8)
    assert torch.allclose(o[2, 0], c * third, atol=1e-8)
    # state space: two tokens
    x = torch.randn(2, 1, 3, dtype=torch.float64)
    B, C = torch.randn(2, 1, 2, dtype=torch.float64), torch.randn(2, 1, 2, dtype=torch.float64)
    dt = torch.tensor([[0.3], [0.7]], dtype=torch.float64)
    A, D = torch.tensor([0.2], dtype=torch.float64), torch.tensor([1.5], dtype=torch.float64)
    y, S = O.ssd_rule(x, B, C, dt, A, D)
    keep = math.exp(-math.exp(0.2) * 0.7)
    want = keep * 0.3 * (B[0, 0] @ C[1, 0]) * x[0, 0] + 0.7 * (B[1, 0] @ C[1, 0]) * x[1, 0] + 1.5 * x[1, 0]
    assert torch.allclose(y[1, 0], want)
    conv = O.short_conv(torch.tensor([[1.0], [2.0], [4.0]]), torch.tensor([[10.0, 1.0]]), torch.tensor([0.5]))
    assert conv.flatten().tolist() == [1.5, 12.5, 24.5]
    val, idx = O.route(torch.tensor([[0.0, 2.0, 1.9, -1.0]], dtype=torch.float64), 2)
    assert idx.tolist() == [[1, 2]] and torch.allclose(val.sum(), torch.tensor(1.0, dtype=torch.float64))
    assert torch.allclose(val[0, 0] / val[0, 1], torch.exp(torch.tensor(0.1, dtype=torch.float64)))
    w = {"gate": torch.tensor([[3.0]]), "up": torch.tensor([[-9.0]]), "down": torch.tensor([[1.0]])}
    got = float(O.clamped_unit(w, "", torch.tensor([[1.0]]), 0.5))
    assert abs(got - 0.5 / (1 + math.exp(-1.702 * 0.5)) * 0.5) < 1e-6
    assert torch.allclose(O.channel_decay(torch.tensor(0.0)), torch.tensor(math.exp(-0.5 * math.exp(-0.5))))
