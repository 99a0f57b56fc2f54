#!/usr/bin/env python
"""Headline benchmark: decode latency / throughput of low-bit Llama models on B200.

    python bench.py --gpus N --steps K --warmup W [--config 7b|70b-tp|7b-spec|mixtral-pp|qlora-dp|latent|hybrid|multistream|
                                                      parallel-block]
                    [--batch B]
                    [--model llama2-7b|llama3-70b] [--impl ours|reference|constructed]

``--config`` picks one of the benchmark set-ups (default: ``7b`` on one GPU, ``70b-tp`` on several):
``7b`` / ``70b-tp`` decode latency (below); ``7b-spec`` self-speculative decoding (fp16 target + int4 draft);
``mixtral-pp`` Mixtral-8x7B sym_int4 pipeline-parallel generation, batch 8, 1024 in / 128 out; ``qlora-dp`` QLoRA
fine-tuning of Llama-2-13B nf4, data parallel, sequence 512, micro-batch 4 per GPU; ``latent`` prompt and decode
throughput of the latent-attention decoder (Dobetar, bf16) at three sizes, beside a Llama-architecture model of equal
size (``value`` is the largest size's decode throughput at batch 1, ``config.sizes`` holds the rest); ``hybrid`` the same
for the decoder of attention and recurrent layers (Letarax); ``multistream`` for the decoder with several residual streams
(Dodilix), beside the two before it; ``parallel-block`` for the decoder whose mixer and feed-forward stand side by side
(Gegorax), beside the two before it.

One "step" is one decode step (one new token for every sequence of the batch) after a prompt pass of
``--prompt`` random tokens.  ``ms_per_step`` is therefore the reference harness's "2+ avg latency (ms/token)"
and ``value`` the whole-job decode throughput in tokens/s.

* N = 1, default model: Llama-2-7B architecture, random N(0, 0.02) weights, sym_int4 (group 64, fp16 scales),
  fp16 activations, fp8 e5m2 KV cache, batch 1, 1024 prompt tokens.
* N > 1: Llama-3-70B architecture in block-scaled fp8_e4m3 (128-blocks, fp32 scales), bf16 activations,
  tensor parallel over the N GPUs (one persistent kernel per token and rank: the row-parallel projections push
  their partial tiles into the peers' symmetric memory and reduce them in the same kernel, the lm_head is
  vocabulary-parallel; strong scaling: the same model and batch on more GPUs).
  ``--model llama3-70b`` runs the same model on one GPU.

Timing: W untimed steps, then K steps between CUDA events on the launching stream, barrier + synchronize on
both sides, max over ranks.  When K steps last less than a second, further blocks of K steps are timed the same way
until a second has passed; ``ms_per_step`` is the mean over all of them and ``steps_timed`` says how many ran
(``steps`` stays the K that was asked for).  Weights (3.6 GB and up) are far larger than the 126 MB L2, so every
step streams them from HBM again.  SM clocks and throttle reasons are sampled with nvidia-smi during the timed region.
The ``e2e`` figure drives the same decode through the public ``model.decode_step`` API with the step's input
token copied from pinned host memory and the sampled token read back to the host every step.
"""
from __future__ import annotations

import argparse
import json
import os
import statistics
import subprocess
import sys
import tempfile
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

MODELS = {
    "llama2-7b": dict(hidden_size=4096, intermediate_size=11008, num_hidden_layers=32, num_attention_heads=32,
                      num_key_value_heads=32, vocab_size=32000, rms_norm_eps=1e-5, rope_theta=10000.0,
                      max_position_embeddings=4096, low_bit="sym_int4", dtype="float16", prompt=1024, batch=1),
    "llama3-70b": dict(hidden_size=8192, intermediate_size=28672, num_hidden_layers=80, num_attention_heads=64,
                       num_key_value_heads=8, vocab_size=128256, rms_norm_eps=1e-5, rope_theta=500000.0,
                       max_position_embeddings=8192, low_bit="fp8_e4m3", dtype="bfloat16", prompt=2048, batch=1),
    "tiny": dict(hidden_size=256, intermediate_size=704, num_hidden_layers=2, num_attention_heads=4,
                 num_key_value_heads=4, vocab_size=32000, rms_norm_eps=1e-6, rope_theta=10000.0,
                 max_position_embeddings=2048, low_bit="sym_int4", dtype="float16", prompt=64, batch=1),
}


# Decode throughput of the cuBLAS + NCCL stand-in (baseline/constructed.py) measured on this hardware, tokens/s at
# batch 1, by (model, GPUs):
# the denominator of ``vs_baseline``.  Set-ups without a recorded number report null.
BASELINE_TOK_S = {("llama2-7b", 1): 171.0, ("llama3-70b", 2): 23.0, ("llama3-70b", 8): 22.1}
BASELINE_SAMPLES_S = {("llama2-13b", 1): 10.17}


def reference_arm(args):
    """The unmodified reference cannot be installed offline: its setup.py downloads the closed native libraries
    (libllama-api.so, bigdl-core-xe) from the network at build time, and it has no CUDA code path."""
    print(json.dumps({
        "impl": "reference",
        "unavailable": "pip install of the reference's python/llm fails offline (setup.py downloads its prebuilt "
                       "Intel-only native libraries at build time: URLError name resolution); no CUDA path exists"}))
    return 0


class ClockSampler:
    def __init__(self, gpu_index: int):
        self.path = tempfile.mktemp(suffix=".csv")
        self.proc = None
        self.gpu_index = gpu_index

    def start(self):
        q = ("index,clocks.sm,clocks.max.sm,power.draw,clocks_event_reasons.active,"
             "clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
             "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")
        try:
            self.proc = subprocess.Popen(["nvidia-smi", f"--query-gpu={q}", "--format=csv,noheader,nounits", "-lms",
                                          "100", "-i", str(self.gpu_index)], stdout=open(self.path, "w"),
                                         stderr=subprocess.DEVNULL)
        except Exception:  # noqa: BLE001
            self.proc = None

    def stop(self):
        out = {"sm_mhz": None, "sm_max_mhz": None, "reasons": [], "samples": 0}
        if self.proc is None:
            return out
        self.proc.terminate()
        try:
            self.proc.wait(timeout=5)
        except Exception:  # noqa: BLE001
            self.proc.kill()
        clocks, reasons, mx = [], set(), None
        try:
            with open(self.path) as f:
                for line in f:
                    p = [x.strip() for x in line.split(",")]
                    if len(p) < 9:
                        continue
                    try:
                        clocks.append(float(p[1]))
                        mx = float(p[2])
                    except ValueError:
                        continue
                    for name, v in zip(("hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"),
                                       p[5:9]):
                        if v.lower().startswith("active"):
                            reasons.add(name)
            os.unlink(self.path)
        except OSError:
            pass
        if clocks:
            out.update(sm_mhz=statistics.median(clocks), sm_max_mhz=mx, reasons=sorted(reasons), samples=len(clocks))
        return out


def other_config(args):
    """The set-ups that are not a decode-latency run: their own drivers measure them (CUDA events or the generate
    loop's per-token timers, max over ranks) and this wrapper prints the result in the common JSON shape."""
    world = int(os.environ.get("WORLD_SIZE", "1"))
    rank = int(os.environ.get("RANK", "0"))
    local_rank = int(os.environ.get("LOCAL_RANK", "0"))
    sampler = ClockSampler(local_rank)
    clocks_box = {}
    # the clocks are sampled during the measured region only (model building idles the GPU at its lowest clock)
    timed = ((lambda: sampler.start()), (lambda: clocks_box.update(c=sampler.stop()))) if rank == 0 else None
    if args.config == "mixtral-pp":
        from ipex_llm_b200.parallel import bench_pp
        argv = ["--model", args.model if args.model != "auto" else "mixtral-8x7b", "--batch", str(args.batch or 8),
                "--prompt", str(args.prompt or 1024), "--new-tokens", str(max(8, args.steps))]
        res = bench_pp.run(argv, timed=timed)
        extra = {"metric": "pipeline-parallel decode tokens/s (first_token_ms = prompt pass)", "scaling": "strong",
                 "dtype": "fp16", "parallelism": f"pp{world}"}
    elif args.config == "qlora-dp":
        from ipex_llm_b200.train import bench_qlora
        argv = ["--model", args.model if args.model != "auto" else "llama2-13b", "--steps", str(args.steps),
                "--warmup", str(args.warmup)]
        res = bench_qlora.run(argv, timed=timed)
        extra = {"metric": "QLoRA finetune samples/s", "scaling": "weak", "dtype": "bf16", "parallelism": f"dp{world}"}
    elif args.config == "latent":
        from ipex_llm_b200.utils import bench_latent
        res = bench_latent.run(["--iters", str(max(16, args.steps)), "--prompt", str(args.prompt or 2048)], timed=timed)
        extra = {"metric": "latent-attention decoder, decode tokens/s at batch 1", "scaling": "strong", "dtype": "bf16",
                 "parallelism": "single"}
    elif args.config == "hybrid":
        from ipex_llm_b200.utils import bench_hybrid
        res = bench_hybrid.run(["--iters", str(max(16, args.steps)), "--prompt", str(args.prompt or 2048)], timed=timed)
        extra = {"metric": "attention + recurrent decoder, decode tokens/s at batch 1", "scaling": "strong", "dtype": "bf16",
                 "parallelism": "single"}
    elif args.config == "multistream":
        from ipex_llm_b200.utils import bench_multistream
        res = bench_multistream.run(["--iters", str(max(16, args.steps)), "--prompt", str(args.prompt or 2048)], timed=timed)
        extra = {"metric": "multi-stream decoder, decode tokens/s at batch 1", "scaling": "strong", "dtype": "bf16",
                 "parallelism": "single"}
    elif args.config == "parallel-block":
        from ipex_llm_b200.utils import bench_parallel_block
        res = bench_parallel_block.run(["--iters", str(max(16, args.steps)), "--prompt", str(args.prompt or 2048)], timed=timed)
        extra = {"metric": "parallel-block decoder, decode tokens/s at batch 1", "scaling": "strong", "dtype": "bf16",
                 "parallelism": "single"}
    else:
        from ipex_llm_b200.utils import bench_speculative
        res = bench_speculative.run(["--new-tokens", str(max(32, args.steps))], timed=timed)
        extra = {"metric": "self-speculative decode tokens/s", "scaling": "strong", "dtype": "fp16",
                 "parallelism": "single"}
    clocks = clocks_box.get("c")
    if rank == 0 and res is not None:
        base = BASELINE_SAMPLES_S.get((res.get("model"), world)) if args.config == "qlora-dp" else None
        line = {"metric": extra["metric"], "value": res.get("value"), "unit": res.get("unit"), "n_gpus": world,
                "steps": args.steps, "warmup": args.warmup, "ms_per_step": res.get("ms_per_step"),
                "higher_is_better": True, "scaling": extra["scaling"],
                "vs_baseline": round(res["value"] / base, 3) if base and res.get("value") else None,
                "dtype": extra["dtype"], "impl": "ours",
                "data": "synthetic random token ids, random-init weights of the named architecture",
                "config": {"model": res.get("model"), "parallelism": extra["parallelism"],
                           **{k: v for k, v in res.items() if k not in ("metric", "value", "unit", "ms_per_step")}},
                "clocks": clocks}
        print(json.dumps(line))
    return 0


def _tp_reference_logits(model, cfg, ids, world, kv_fp8=False):
    """Plain fp32 PyTorch forward of a tensor-parallel Llama-architecture model over the weights it actually holds:
    every rank dequantizes its shards, the shards are gathered and reassembled (q / k / v and gate / up by rows,
    o_proj / down_proj by columns, lm_head by vocabulary rows).  Returns the logits of the second-to-last and of the
    last position of ``ids`` (the prompt pass' logits and the first decode step's).  ``kv_fp8``: the last position is
    a decode step that reads the e5m2 KV cache, so its attention sees K / V rounded to e5m2 (the prompt pass attends
    to the unrounded K / V it has just computed, here as in the engine)."""
    import math

    import torch
    import torch.distributed as dist

    def gather(t, dim):
        parts = [torch.empty_like(t) for _ in range(world)]
        dist.all_gather(parts, t.contiguous())
        return torch.cat(parts, dim=dim)

    def deq(mod):
        w = mod.weight
        return w.dequantize(torch.float32) if hasattr(w, "dequantize") else w.data.float()

    base = model.model
    H = cfg.hidden_size
    hd = getattr(cfg, "head_dim", None) or H // cfg.num_attention_heads
    Hq, Hkv = cfg.num_attention_heads, cfg.num_key_value_heads
    hq_l, hkv_l = Hq // world, Hkv // world
    S = ids.shape[1]
    x = base.embed_tokens.weight.data.float()[ids[0]]                       # [S, H]
    pos = torch.arange(S, device=x.device).unsqueeze(0)
    cos, sin = base.rotary_emb(x.unsqueeze(0), position_ids=pos)
    cos, sin = cos[0].float(), sin[0].float()

    def rms(v, w):
        return v * torch.rsqrt(v.pow(2).mean(-1, keepdim=True) + cfg.rms_norm_eps) * w.float()

    def rope(t):                                                            # [S, heads, hd], NeoX halves
        t1, t2 = t[..., : hd // 2], t[..., hd // 2:]
        return t * cos[:, None, :] + torch.cat([-t2, t1], dim=-1) * sin[:, None, :]

    for blk in base.layers:
        a = blk.self_attn
        wqkv = deq(a.qkv_proj)                                              # this rank: [q_s; k_s; v_s] rows
        wq = gather(wqkv[: hq_l * hd], 0)
        wk = gather(wqkv[hq_l * hd:(hq_l + hkv_l) * hd], 0)
        wv = gather(wqkv[(hq_l + hkv_l) * hd:], 0)
        wo = gather(deq(a.o_proj), 1)
        h = rms(x, blk.input_layernorm.weight.data)
        q = rope((h @ wq.t()).view(S, Hq, hd))
        k = rope((h @ wk.t()).view(S, Hkv, hd))
        v = (h @ wv.t()).view(S, Hkv, hd)
        k = k.repeat_interleave(Hq // Hkv, dim=1)
        v = v.repeat_interleave(Hq // Hkv, dim=1)
        sc = torch.einsum("qhd,khd->hqk", q, k) / math.sqrt(hd)
        sc = sc.masked_fill(~torch.ones(S, S, dtype=torch.bool, device=x.device).tril(), float("-inf"))
        att = torch.einsum("hqk,khd->qhd", torch.softmax(sc, dim=-1), v).reshape(S, Hq * hd)
        if kv_fp8:
            kq, vq = k.to(torch.float8_e5m2).float(), v.to(torch.float8_e5m2).float()
            sl = torch.einsum("hd,khd->hk", q[-1], kq) / math.sqrt(hd)
            att[-1] = torch.einsum("hk,khd->hd", torch.softmax(sl, dim=-1), vq).reshape(Hq * hd)
        x = x + att @ wo.t()
        del wq, wk, wv, wo, wqkv
        m = blk.mlp
        wg, wu, wd = gather(deq(m.gate_proj), 0), gather(deq(m.up_proj), 0), gather(deq(m.down_proj), 1)
        h = rms(x, blk.post_attention_layernorm.weight.data)
        x = x + (torch.nn.functional.silu(h @ wg.t()) * (h @ wu.t())) @ wd.t()
        del wg, wu, wd
    head = model.lm_head
    wl = deq(head)
    if getattr(head, "tp_gather", None) is not None and wl.shape[0] < cfg.vocab_size:
        wl = gather(wl, 0)
    out = rms(x[-2:], base.norm.weight.data) @ wl.t()
    return out[0:1], out[1:2]


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=128)
    ap.add_argument("--warmup", type=int, default=8)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference", "constructed"],
                    help="reference: the unmodified reference (unavailable offline); constructed: its semantics on "
                         "stock cuBLAS + NCCL (baseline/constructed.py)")
    ap.add_argument("--config", default="auto", choices=["auto", "7b", "70b-tp", "7b-spec", "mixtral-pp", "qlora-dp",
                                                           "latent", "hybrid", "multistream", "parallel-block"])
    ap.add_argument("--model", default="auto")
    ap.add_argument("--batch", type=int, default=None)
    ap.add_argument("--prompt", type=int, default=None)
    ap.add_argument("--low-bit", default=None)
    ap.add_argument("--no-e2e", action="store_true")
    ap.add_argument("--layers", type=int, default=None,
                    help="profiling only: truncate the model to this many layers (the JSON line then names it)")
    args = ap.parse_args()
    if args.impl == "reference":
        return reference_arm(args)
    if args.impl == "constructed":
        import runpy
        world = int(os.environ.get("WORLD_SIZE", "1"))
        model = args.model if args.model != "auto" else ("llama2-7b" if world == 1 else "llama3-70b")
        sys.argv = [os.path.join(ROOT, "baseline", "constructed.py"), "--model", model, "--steps", str(args.steps),
                    "--warmup", str(max(args.warmup, 3))] + (["--batch", str(args.batch)] if args.batch else []) + \
                   (["--layers", str(args.layers)] if args.layers else [])
        runpy.run_path(sys.argv[0], run_name="__main__")
        return 0
    args.warmup = max(args.warmup, 3)
    if args.config in ("mixtral-pp", "qlora-dp", "7b-spec", "latent", "hybrid", "multistream", "parallel-block"):
        return other_config(args)
    if args.config == "7b" and args.model == "auto":
        args.model = "llama2-7b"
    if args.config == "70b-tp" and args.model == "auto":
        args.model = "llama3-70b"

    import torch
    import torch.distributed as dist

    world = int(os.environ.get("WORLD_SIZE", "1"))
    rank = int(os.environ.get("RANK", "0"))
    local_rank = int(os.environ.get("LOCAL_RANK", "0"))
    if world > 1:
        os.environ.setdefault("MASTER_ADDR", "127.0.0.1")
        torch.cuda.set_device(local_rank)
        dist.init_process_group("nccl", device_id=torch.device("cuda", local_rank))
    else:
        torch.cuda.set_device(0)
    n_gpus = max(world, 1)
    if args.gpus != n_gpus and rank == 0:
        print(f"[bench] --gpus {args.gpus} but WORLD_SIZE={world}; running on {n_gpus}", file=sys.stderr)

    name = args.model
    if name == "auto":
        name = "llama2-7b" if n_gpus == 1 else "llama3-70b"
    spec = dict(MODELS[name])
    low_bit = args.low_bit or spec.pop("low_bit")
    spec.pop("low_bit", None)
    dtype = getattr(torch, spec.pop("dtype"))
    prompt = args.prompt or spec.pop("prompt")
    spec.pop("prompt", None)
    batch = args.batch or spec.pop("batch")
    spec.pop("batch", None)

    from transformers import LlamaConfig
    from ipex_llm.transformers import AutoModelForCausalLM
    from ipex_llm_b200.engine import get_engine

    if args.layers:
        spec["num_hidden_layers"] = args.layers
        name = f"{name}-{args.layers}layers-PROFILING-ONLY"
    cfg = LlamaConfig(tie_word_embeddings=False, **spec)
    tp_group = None
    if n_gpus > 1:
        from ipex_llm_b200.parallel.tp import TPGroup
        tp_group = TPGroup()
    t_load = time.time()
    model = AutoModelForCausalLM.from_config(cfg, load_in_low_bit=low_bit, device=f"cuda:{local_rank}",
                                             torch_dtype=dtype, seed=0, tp_group=tp_group)
    torch.cuda.synchronize()
    load_s = time.time() - t_load

    dev = torch.device("cuda", local_rank)
    g = torch.Generator(device="cpu").manual_seed(1234)
    ids_host = torch.randint(0, cfg.vocab_size, (batch, prompt), generator=g)
    # room for the warm-ups, the timed blocks (padded to a second, at most 4096 steps) and the end-to-end loop
    max_steps = max(args.steps, min(4096, 1536 // max(1, batch)))
    total_len = prompt + args.warmup * 2 + max_steps + args.steps + 48
    eng = get_engine(model, batch, total_len)
    kv_fp8 = eng.kv_fp8

    # ---- prompt pass (1st token), timed on the device ----
    ids = ids_host.to(dev)
    ev0, ev1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    first_cold_ms = first_ms = 0.0
    for attempt in range(2):       # the first pass pays one-time set-up (module load, workspaces); report the second
        torch.cuda.synchronize()
        ev0.record()
        logits = eng.prefill(ids)
        nxt = torch.argmax(logits, dim=-1)
        ev1.record()
        torch.cuda.synchronize()
        if attempt == 0:
            first_cold_ms = ev0.elapsed_time(ev1)
        first_ms = ev0.elapsed_time(ev1)
    eng.tokens[:batch] = nxt

    def barrier():
        if world > 1:
            dist.barrier()
        torch.cuda.synchronize()

    # ---- device-timed decode ----
    for _ in range(args.warmup):
        eng.decode_step(batch)
    barrier()
    sampler = ClockSampler(local_rank)
    if rank == 0:
        sampler.start()
    dev_ms, steps_timed = 0.0, 0
    while True:
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        for _ in range(args.steps):
            eng.decode_step(batch)
        e1.record()
        barrier()
        block_ms = e0.elapsed_time(e1)
        if world > 1:       # every rank must take the same decision: use the slowest rank's time
            tb = torch.tensor([block_ms], device=dev, dtype=torch.float64)
            dist.all_reduce(tb, op=dist.ReduceOp.MAX)
            block_ms = float(tb[0])
        dev_ms += block_ms
        steps_timed += args.steps
        if dev_ms >= 1000.0 or steps_timed + args.steps > max_steps:
            break

    # ---- end to end through the public per-step API: pinned host token in, sampled token out, every step ----
    e2e = None
    if not args.no_e2e:
        tok_host = torch.empty(batch, dtype=torch.int64).pin_memory()
        tok_host.copy_(eng.tokens[:batch].cpu())
        for _ in range(args.warmup):
            tok_host.copy_(model.decode_step(tok_host))
        barrier()
        t0 = time.perf_counter()
        for _ in range(args.steps):
            out_host = model.decode_step(tok_host)
            tok_host.copy_(out_host)
        torch.cuda.synchronize()
        e2e_s = time.perf_counter() - t0
        e2e = e2e_s
    clocks = sampler.stop() if rank == 0 else None

    # ---- the reference harness's own metric: per-token cost of model.generate (first token / mean of the rest) ----
    gen_stats = None
    if not args.no_e2e:
        n_new = min(32, max(4, args.steps))
        model.generate(ids, max_new_tokens=n_new, do_sample=False)       # warm-up (the harness does one too)
        model.generate(ids, max_new_tokens=n_new, do_sample=False)
        gen_stats = {"first_cost_ms": round(1e3 * float(model.first_token_time), 3),
                     "rest_cost_mean_ms": round(1e3 * float(model.rest_cost_mean), 4), "new_tokens": n_new}

    if world > 1:
        t = torch.tensor([e2e if e2e is not None else 0.0, first_ms], device=dev, dtype=torch.float64)
        dist.all_reduce(t, op=dist.ReduceOp.MAX)
        e2e_m, first_ms = t.tolist()
        e2e = e2e_m if e2e is not None else None

    # ---- tensor-parallel numerics: a two-layer model of the same shape, sharded over the ranks, against a plain
    # fp32 PyTorch forward over the SAME weights (every rank's dequantized shards gathered and reassembled): logits of
    # the prompt pass and of one decode step ----
    tp_check = None
    if world > 1 and not args.no_e2e:
        import copy
        launches = eng.kernel_launches_per_step
        del eng
        model._ipex_engine = None
        try:
            cfg2 = copy.deepcopy(cfg)
            cfg2.num_hidden_layers = 2
            ids2 = ids[:1, :96]
            small = AutoModelForCausalLM.from_config(cfg2, load_in_low_bit=low_bit, device=f"cuda:{local_rank}",
                                                     torch_dtype=dtype, seed=0, tp_group=tp_group)
            e2 = get_engine(small, 1, 256)
            lg0 = e2.prefill(ids2).float().clone()
            tok1 = torch.argmax(lg0, dim=-1)
            e2.tokens[:1] = tok1
            e2.decode_step(1)
            torch.cuda.synchronize()
            lg1 = e2.gather_logits(1).float().clone()
            ref0, ref1 = _tp_reference_logits(small, cfg2, torch.cat([ids2, tok1.view(1, 1)], dim=1), world,
                                              kv_fp8=e2.kv_fp8)
            if rank == 0:
                cos = torch.nn.functional.cosine_similarity
                tp_check = {"layers": 2, "prompt_tokens": int(ids2.shape[1]), "reference": "fp32 PyTorch forward over the "
                            "gathered dequantized shards (decode row: K / V through e5m2 like the cache)",
                            "prefill_logits_cos": round(float(cos(lg0, ref0, dim=-1).min()), 5),
                            "decode_logits_cos": round(float(cos(lg1, ref1, dim=-1).min()), 5),
                            "decode_max_abs_err": round(float((lg1 - ref1).abs().max()), 4),
                            "decode_logits_absmax": round(float(ref1.abs().max()), 4),
                            "same_argmax": bool(torch.equal(lg1.argmax(-1), ref1.argmax(-1)))}
        except Exception as e:  # noqa: BLE001  (the same code runs on every rank: a failure is reported, not fatal)
            tp_check = {"error": f"{type(e).__name__}: {e}"[:300]}
        dist.barrier()
    else:
        launches = eng.kernel_launches_per_step

    if rank == 0:
        ms_per_step = dev_ms / steps_timed
        value = batch * 1000.0 / ms_per_step
        base = BASELINE_TOK_S.get((name, n_gpus)) if batch == 1 else None
        line = {
            "metric": "decode tokens/s (2nd+ token latency in ms_per_step): Llama-2-7B int4 on 1 GPU, "
                      "Llama-3-70B fp8 tensor-parallel on N GPUs",
            "value": round(value, 3), "unit": "tokens/s", "n_gpus": n_gpus, "steps": args.steps,
            "warmup": args.warmup, "steps_timed": steps_timed, "ms_per_step": round(ms_per_step, 5),
            "higher_is_better": True, "scaling": "strong",
            "vs_baseline": round(value / base, 3) if base else None, "dtype": "fp16" if dtype == torch.float16 else "bf16",
            "data": "synthetic random token ids, random-init N(0,0.02) weights of the named architecture",
            "impl": "ours",
            "config": {"model": name, "low_bit": low_bit, "global_batch": batch, "seq_len": prompt,
                       "kv_cache": "fp8_e5m2" if kv_fp8 else str(dtype).replace("torch.", ""),
                       "parallelism": f"tp{n_gpus}" if n_gpus > 1 else "single",
                       "l2_policy": "inputs larger than L2: every step streams the full packed weights "
                                    f"({sum(p.numel() * p.element_size() for p in model.parameters()) / 1e9:.2f} GB)",
                       "decode_engine": "one persistent kernel per token (cuda-graph replay)"
                       if launches == 1 else "cuda-graph + programmatic dependent launch"},
            "first_token_ms": round(first_ms, 3),
            "first_token_cold_ms": round(first_cold_ms, 3),
            "model_build_s": round(load_s, 2),
            "gpu_launches": int(steps_timed * launches),
            "generate": gen_stats,
            "tp_check": tp_check,
            "clocks": clocks,
        }
        if e2e is not None:
            line["e2e"] = {"value": round(batch * args.steps / e2e, 3), "unit": "tokens/s",
                           "ms_per_step": round(1000.0 * e2e / args.steps, 5),
                           "h2d_bytes_per_step": 8 * batch, "d2h_bytes_per_step": 8 * batch,
                           "api": "model.decode_step(pinned_host_tokens) -> host tokens"}
        print(json.dumps(line))
    if world > 1:
        dist.destroy_process_group()
    return 0


if __name__ == "__main__":
    sys.exit(main())
