#!/usr/bin/env python
"""GPT-J-6B decode benchmark of the B200-native path (and its CPU reference arm).

    python bench.py [--gpus N] [--steps K] [--warmup W] [--impl mtj|reference]

One "step" is one decode step (one generated token per sequence) of the
GPT-J-6B architecture at a full sliding window (2047 cached tokens), batch 1,
greedy sampling, bf16 random-init N(0, 0.02) weights, after a prefill of a
1 x 2048 synthetic prompt.  Prints ONE JSON line.
"""
from __future__ import annotations

import argparse
import json
import os
import subprocess
import sys
import threading
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
PKG = os.path.join(ROOT, "mesh-transformer-jax_b200")
for _p in (ROOT, PKG):
    if _p not in sys.path:
        sys.path.insert(0, _p)

METRIC = "gptj6b_decode_tokens_per_s"
# dram__bytes_read.sum + dram__bytes_write.sum per launch from the ncu captures summarised under profiles/
# (GPT-J-6B layer shapes, batch 1, window 2047); the kernels read every weight byte exactly once.  The whole-step
# kernel was captured at 4 layers and its traffic scaled by the algorithmic bytes of the 28-layer step.
NCU_TRAFFIC = {"mega": 12.66e9, "in_proj": None, "ff_in_proj": None, "attention": 33.6e6, "out_proj": 171.4e6, "logits": 416.4e6}
UNIT = "tokens/s"

GPTJ_6B = {
    "layers": 28, "d_model": 4096, "n_heads": 16, "n_vocab": 50400,
    "norm": "layernorm", "pe": "rotary", "pe_rotary_dims": 64,
    "seq": 2048, "cores_per_replica": 1, "per_replica_batch": 1,
}


GPTJ_22B = dict(GPTJ_6B, layers=48, d_model=6144, n_heads=24)   # the ~22B scale-up (d_head 256, d_ff 24576)


def model_config(args):
    return GPTJ_22B if getattr(args, "model", "6b") == "22b" else GPTJ_6B


def workload_config(args, n_gpus):
    cfg = workload_config_6b(args, n_gpus)
    if getattr(args, "model", "6b") == "22b":
        cfg["workload"] = cfg["workload"].replace("GPT-J-6B (L28 d4096 h16 dh256 rot64 ff16384 V50400)",
                                                  "GPT-J-style 22B (L48 d6144 h24 dh256 rot64 ff24576 V50400)")
        cfg["l2"] = cfg["l2"].replace("11.7 GB", "44.1 GB")
        if getattr(args, "workload", "headline") == "serving":
            cfg["workload"] = cfg["workload"].replace("prompts of 1024", f"prompts of {serving_prompt(args)}")
    return cfg


def serving_prompt(args):
    return 1792 if getattr(args, "model", "6b") == "22b" else 1024


def workload_config_6b(args, n_gpus):
    if getattr(args, "workload", "headline") == "serving":
        return {
            "workload": "GPT-J-6B (L28 d4096 h16 dh256 rot64 ff16384 V50400) bf16 random-init; serving: prompts of "
                        "1024 uniform-random ids in [0, 50257) left-padded into seq 2048, then nucleus sampling "
                        "(top_p 0.9, temperature 1.0, seeded uniforms) one token per sequence per step",
            "batch": args.batch, "window": "prompt + generated tokens", "parallelism": f"mp{n_gpus}",
            "l2": "every step streams 11.7 GB of weights plus the KV cache (>> 126 MB L2), no flush needed",
        }
    return {
        "workload": "GPT-J-6B (L28 d4096 h16 dh256 rot64 ff16384 V50400) bf16 random-init; prefill 1x2048 "
                    "uniform-random ids, then greedy decode at a full 2047-token sliding window",
        "batch": args.batch, "window": GPTJ_6B["seq"] - 1, "parallelism": f"mp{n_gpus}",
        "l2": "every step streams 11.7 GB of weights (>> 126 MB L2), no flush needed",
    }


# ------------------------------------------------------------------ clocks ----
class ClockSampler:
    Q = ("clocks.sm,clocks.max.sm,power.draw,clocks_event_reasons.hw_slowdown,"
         "clocks_event_reasons.hw_thermal_slowdown,clocks_event_reasons.sw_thermal_slowdown,"
         "clocks_event_reasons.sw_power_cap")

    def __init__(self, index=0):
        self.samples, self.proc, self.index = [], None, index

    def start(self):
        try:
            self.proc = subprocess.Popen(
                ["nvidia-smi", f"--query-gpu={self.Q}", "--format=csv,noheader,nounits", "-lms", "100",
                 "-i", str(self.index)], stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
            threading.Thread(target=self._read, daemon=True).start()
        except OSError:
            self.proc = None

    def _read(self):
        for line in self.proc.stdout:
            self.samples.append((time.time(), line.strip()))

    def stop(self):
        if self.proc is not None:
            self.proc.terminate()
            try:
                self.proc.wait(timeout=5)
            except Exception:
                self.proc.kill()

    def summary(self, t0, t1):
        sm, mx, reasons = [], [], set()
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        for ts, line in self.samples:
            if ts < t0 or ts > t1 + 0.15:
                continue
            f = [x.strip() for x in line.split(",")]
            try:
                sm.append(float(f[0]))
                mx.append(float(f[1]))
            except (ValueError, IndexError):
                continue
            for n, v in zip(names, f[3:7]):
                if v.lower().startswith("active"):
                    reasons.add(n)
        if not sm:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": [], "samples": 0}
        sm.sort()
        return {"sm_mhz": sm[len(sm) // 2], "sm_max_mhz": max(mx), "reasons": sorted(reasons),
                "samples": len(sm)}


# --------------------------------------------------------------- reference ----
def run_reference(args):
    """The reference's algorithm on the host cores (CPU restatement: the
    reference's own JAX code cannot be imported without jax/haiku)."""
    rank = int(os.environ.get("RANK", "0"))
    if rank != 0:
        return
    from oracle import cpu_baseline
    steps, warmup = max(1, min(args.steps, 3)), max(1, min(args.warmup, 1))
    r = cpu_baseline.decode_tokens_per_s(GPTJ_6B, steps=steps, warmup=warmup, batch=args.batch)
    line = {
        "impl": "reference", "metric": METRIC, "value": r["value"], "unit": UNIT, "n_gpus": args.gpus,
        "steps": steps, "warmup": warmup, "ms_per_step": 1e3 * r["seconds"] / steps,
        "higher_is_better": True, "scaling": "strong", "vs_baseline": None, "dtype": "f32",
        "data": "synthetic", "config": workload_config(args, args.gpus),
        "cpu_baseline": {"value": r["value"], "unit": UNIT, "cores": r["cores"], "kind": "port",
                         "sample": r["sample"]},
        "e2e": {"value": r["value"], "unit": UNIT, "h2d_bytes_per_step": 0, "d2h_bytes_per_step": 0},
        "gpu_launches": 0,
    }
    print(json.dumps(line), flush=True)


# --------------------------------------------------------------------- mtj ----
def decode_bytes_per_step(cfg, batch, ctx, mp=1):
    """Algorithmic HBM bytes of one decode step, whole model (bf16)."""
    L, d, V = cfg["layers"], cfg["d_model"], cfg["n_vocab"]
    weights = 2 * (L * (12 * d * d + 5 * d + 2 * d) + d * V + V + 2 * d)
    kv = batch * ctx * L * 2 * d * 2 + batch * L * 2 * d * 2 + batch * d * 2
    return weights + kv


def forward_flops(cfg, batch, T):
    """Algorithmic flops of a full causal forward: GEMMs (12 d^2 per layer + d V per token) and the lower
    triangle of the attention (L 2 d T (T + 1) per sequence)."""
    L, d, V = cfg["layers"], cfg["d_model"], cfg["n_vocab"]
    return 2.0 * (L * 12 * d * d + d * V) * batch * T + L * 2.0 * d * T * (T + 1) * batch


def build_network(cfg, device, rank, world, seed=1234):
    """Random-init N(0, 0.02) bf16 weights.  Every rank draws the FULL leaf from a per-leaf seed and keeps its
    own slice (columns of q/v/k/ff-in and the projection, rows of o/ff-out and the embedding, exactly the
    split of layers.py:176,243,249-258,555), so the model is the same model at every N."""
    import torch
    from mesh_transformer._runtime import param_shapes
    from mesh_transformer.transformer_shard import CausalTransformer
    net = CausalTransformer(dict(cfg), device=device, init_weights=False)
    full_shapes = param_shapes(dict(cfg, cores_per_replica=1))
    gen = torch.Generator(device=device)
    params = {}
    index = 0
    for mod, leaves in full_shapes.items():
        out = {}
        for leaf, shape in leaves.items():
            index += 1
            if leaf == "scale":
                t = torch.ones(shape, dtype=torch.bfloat16, device=device)
            elif leaf in ("offset", "b"):
                t = torch.zeros(shape, dtype=torch.bfloat16, device=device)
            else:
                gen.manual_seed(seed * 1000003 + index)
                t = (torch.randn(shape, generator=gen, device=device, dtype=torch.float32) * 0.02).to(torch.bfloat16)
            if world > 1 and leaf not in ("scale", "offset"):
                row_split = mod.endswith("embedding_shard/~/linear") or mod.endswith("linear_3") or mod.endswith("linear_5")
                if leaf == "w":
                    t = t.chunk(world, dim=0 if row_split else 1)[rank]
                elif not row_split:                      # ff-in / projection bias: split like the columns
                    t = t.chunk(world, dim=0)[rank]
                # a bias added on every shard before the all-reduce (embedding, ff-out) counts once: rank 0 holds it
                elif rank != 0:
                    t = torch.zeros_like(t)
            out[leaf] = t.contiguous()[None]
        params[mod] = out
    net.state = {"params": params, "step": 0}
    return net


def _sha(a):
    import hashlib
    import numpy as np
    return hashlib.sha1(np.ascontiguousarray(a).tobytes()).hexdigest()[:16]


def run_mtj(args):
    import numpy as np
    import torch
    import torch.distributed as dist

    world = int(os.environ.get("WORLD_SIZE", "1"))
    rank = int(os.environ.get("RANK", "0"))
    local_rank = int(os.environ.get("LOCAL_RANK", "0"))
    if world != args.gpus:
        raise SystemExit(f"--gpus {args.gpus} but WORLD_SIZE={world}: launch with torch.distributed.run")
    torch.cuda.set_device(local_rank)
    device = torch.device("cuda", local_rank)
    if world > 1:
        dist.init_process_group("nccl", device_id=device)

    import __graft_entry__ as ge
    if rank == 0:
        ge.build()
    if world > 1:
        dist.barrier()
    from mesh_transformer._runtime import ShardRuntime

    def barrier():
        if world > 1:
            dist.barrier()
        torch.cuda.synchronize()

    def max_over_ranks(v):
        t = torch.tensor([float(v)], device=device)
        if world > 1:
            dist.all_reduce(t, op=dist.ReduceOp.MAX)
        return float(t.item())

    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)

    def timed(fn):
        """CUDA-event time (ms, max over ranks) of fn() bracketed by barrier + synchronize."""
        barrier()
        e0.record()
        fn()
        e1.record()
        barrier()
        return max_over_ranks(e0.elapsed_time(e1))

    def median(xs):
        xs = sorted(xs)
        return xs[len(xs) // 2]

    peaks = {}
    try:
        peaks = json.load(open(os.path.join(ROOT, "MEASURED_PEAKS.json")))
    except Exception:
        pass
    hbm_peak = float(peaks.get("hbm_gbs", 6650.0))
    tc_burst = float(peaks.get("bf16_tflops", 1590.0))
    tc_sustained = float(peaks.get("bf16_tflops_sustained", 1400.0))
    peak_kind = "measured" if "hbm_gbs" in peaks else "fallback"

    cfg = dict(model_config(args), cores_per_replica=world)
    if args.layers > 0:
        cfg["layers"] = args.layers
    seq, B, K, W = cfg["seq"], args.batch, args.steps, args.warmup
    net = build_network(cfg, device, rank, world)
    n_blocks = 5
    gen_cap = (n_blocks + 2) * K + W + 640
    rt = net._runtime(B, gen_cap)
    torch.cuda.empty_cache()

    rng = np.random.Generator(np.random.PCG64(0))
    serving = args.workload == "serving"
    prompt = serving_prompt(args) if serving else seq
    ctx = rng.integers(0, 50257 if serving else cfg["n_vocab"], size=(B, seq)).astype(np.uint32)
    ctx[:, :seq - prompt] = 0                      # left padding
    ctx_dev = torch.from_numpy(ctx.view(np.int32)).to(device)
    lens = [prompt] * B
    tiny = float(np.finfo(np.float32).tiny)

    def uniform_pool(batch, vocab):
        g = torch.Generator(device=device)
        g.manual_seed(1234)
        return [torch.rand((batch, vocab), generator=g, device=device).clamp_(tiny, 1.0 - 2.0 ** -24) for _ in range(4)]

    n_calls = [0]
    if serving:
        u_pool = uniform_pool(B, cfg["n_vocab"])
        top_p_dev = torch.full((B,), 0.9, device=device)
        temp_dev = torch.full((B,), 1.0, device=device)

    def decode(tok_in, tok_out, r=None):
        r = r or rt
        if serving:
            n_calls[0] += 1
            r.decode_step(tok_in, tok_out, None, greedy=False, top_p=top_p_dev, temp=temp_dev,
                          uniforms=u_pool[n_calls[0] % len(u_pool)])
        else:
            r.decode_step(tok_in, tok_out, None, greedy=True)

    # ---- prefill (reported beside the headline): median of 10 ----
    rt.prefill(ctx_dev, lens)
    prefill_ms = median([timed(lambda: rt.prefill(ctx_dev, lens)) for _ in range(10)])
    rt.profile_enable(True)                       # kernel-family times of one more prefill
    rt.prefill(ctx_dev, lens)
    prefill_prof = rt.profile_read()
    rt.profile_enable(False)

    sampler = ClockSampler(local_rank)
    if rank == 0:
        sampler.start()

    # ---- device-resident decode: the headline `value` ----
    tok_out = torch.empty((B,), dtype=torch.int32, device=device)
    first_ids = []
    for i in range(W):
        decode(None, tok_out)
        if i < 16:
            first_ids.append(tok_out.clone())
    torch.cuda.synchronize()
    t_warm = time.time()
    extra = 0
    while time.time() - t_warm < 0.3 and extra < 512:      # at least 0.3 s of steady stepping before the clock starts
        decode(None, tok_out)
        if len(first_ids) < 16:
            first_ids.append(tok_out.clone())
        extra += 1
        if extra % 8 == 0:
            torch.cuda.synchronize()
    launches0 = rt.launch_count()
    t_wall0 = time.time()
    block_ms = []
    for _ in range(n_blocks):                     # each block: exactly K steps, barrier + synchronize on both sides
        block_ms.append(timed(lambda: [decode(None, tok_out) for _ in range(K)]))
    t_wall1 = time.time()
    launches = (rt.launch_count() - launches0) // n_blocks
    ms_total = median(block_ms)

    # ---- per-family kernel time for the roofline (separate pass, events between launches) ----
    rt.profile_enable(True)
    for _ in range(min(K, 32)):
        decode(None, tok_out)
    prof = rt.profile_read()
    rt.profile_enable(False)
    # phase time stamps of the persistent decode kernel (when it is the path in use)
    phases = None
    if B <= max(1, rt.tuning["mega_max_batch"]) and os.environ.get("MTJ_NO_MEGA") != "1" \
            and os.environ.get("MTJ_NO_P2P") != "1":
        rt.mega_trace(True)
        for _ in range(3):
            decode(None, tok_out)
        torch.cuda.synchronize()
        tr = np.array(rt.mega_trace(False, read=True), dtype=np.float64)
        Lc = cfg["layers"]
        lay = tr[:6 * Lc].reshape(Lc, 6)
        dd = np.diff(lay, axis=1).mean(0) / 1e3
        phases = {"wait_x_us": dd[0], "ln_in_proj_us": dd[1], "attention_us": dd[2],
                  "out_proj_ff_columns_and_wait_us": dd[3], "out_proj_attn_columns_us": dd[4],
                  "layer_period_us": float(np.diff(lay[:, 0]).mean() / 1e3) if Lc > 1 else None,
                  "logits_us": (tr[6 * Lc + 2] - tr[6 * Lc + 1]) / 1e3,
                  "kernel_us": (tr[6 * Lc + 2] - tr[0]) / 1e3}
    rt.check_device_status()

    # ---- end to end through the public API: CausalTransformer.generate (host context in, host tokens out) ----
    opts = {"top_p": np.full(B, 0.9 if serving else 0.0), "temp": np.ones(B)}
    if serving:
        from mesh_transformer.sampling import nucleaus_sample
        net.config["sampler"] = nucleaus_sample
    net.generate(ctx, lens, 4, opts)                       # the step graph is captured, caches are warm
    e2e_runs = []
    gen_tokens = None
    for _ in range(3):
        barrier()
        _, gout = net.generate(ctx, lens, K, opts)
        tm = net.last_generate_timing
        e2e_runs.append((max_over_ranks(tm["decode_s"]), max_over_ranks(tm["prefill_s"])))
        gen_tokens = gout[0]
    e2e_decode_s, e2e_prefill_s = sorted(e2e_runs)[len(e2e_runs) // 2]
    if rank == 0:
        sampler.stop()
    greedy16 = [int(t[0].item()) for t in first_ids[:16]] if not serving else None

    # ---- second runtime: eval 8 x 2048 (config 4) and the serving workload at batch 32 (config 3) ----
    extra_blocks = {}
    barrier()
    net.close()
    if not serving and not args.headline_only:
        SB = 32
        rt2 = ShardRuntime(cfg, rank=rank, device=device, max_batch=SB, max_gen=5 * 32 + 64, max_rows=4096)
        rt2.load_params(net.state["params"])
        ids = np.random.Generator(np.random.PCG64(4)).integers(0, cfg["n_vocab"], size=(8, seq + 1)).astype(np.uint32)
        obs = torch.from_numpy(np.ascontiguousarray(ids[:, :-1]).view(np.int32)).to(device)
        tgt = torch.from_numpy(np.ascontiguousarray(ids[:, 1:]).view(np.int32)).to(device)
        ev_loss, ev_correct = rt2.eval_loss(obs, tgt, None)
        eval_ms = median([timed(lambda: rt2.eval_loss(obs, tgt, None)) for _ in range(10)])
        ev_loss, ev_correct = ev_loss.cpu().numpy(), ev_correct.cpu().numpy()
        eflops = forward_flops(cfg, 8, seq)
        extra_blocks["eval"] = {
            "tokens_per_s": 8 * seq / (eval_ms * 1e-3), "ms": eval_ms, "tokens": 8 * seq, "batch": 8, "seq": seq,
            "timing": "median of 10", "mean_loss": float(ev_loss.mean()),
            "tflops": eflops / (eval_ms * 1e-3) / 1e12,
            "frac_of_burst_peak": eflops / (eval_ms * 1e-3) / 1e12 / tc_burst / world,
            "note": "full-sequence causal forward of 8 x 2048 ids, vocab-sharded logits and cross-entropy; "
                    "random-init weights, so the loss sits near ln(n_vocab); fraction = algorithmic flops / time / "
                    "(bf16_tflops burst x n_gpus)"}
        parity_eval = {"eval_mean_loss": float(ev_loss.mean()), "eval_correct_count": int(ev_correct.sum()),
                       "eval_correct_sha": _sha(ev_correct),
                       "eval_loss_first8": [round(float(v), 4) for v in ev_loss[0, :8]]}
        # serving: prompts of 1024 ids in [0, 50257) left-padded into seq, nucleus sampling
        sp = 1024
        sctx = np.random.Generator(np.random.PCG64(5)).integers(0, 50257, size=(SB, seq)).astype(np.uint32)
        sctx[:, :seq - sp] = 0
        sctx_dev = torch.from_numpy(sctx.view(np.int32)).to(device)
        pool = uniform_pool(SB, cfg["n_vocab"])
        tp_dev, tt_dev = torch.full((SB,), 0.9, device=device), torch.full((SB,), 1.0, device=device)
        stok = torch.empty((SB,), dtype=torch.int32, device=device)
        cnt = [0]

        def sstep():
            cnt[0] += 1
            rt2.decode_step(None, stok, None, greedy=False, top_p=tp_dev, temp=tt_dev, uniforms=pool[cnt[0] % 4])

        rt2.prefill(sctx_dev, [sp] * SB)
        sprefill_ms = timed(lambda: rt2.prefill(sctx_dev, [sp] * SB))
        for _ in range(8):
            sstep()
        sl0 = rt2.launch_count()
        sblocks = [timed(lambda: [sstep() for _ in range(32)]) for _ in range(3)]
        s_launches = (rt2.launch_count() - sl0) // 3
        sms = median(sblocks) / 32
        sctx_avg = sp + 8 + 48
        sbytes = decode_bytes_per_step(cfg, SB, sctx_avg)
        rt2.check_device_status()
        extra_blocks["serving_b32"] = {
            "tokens_per_s": SB / (sms * 1e-3), "ms_per_step": sms, "batch": SB, "prompt": sp, "steps_per_block": 32,
            "block_ms": sblocks, "gpu_launches_per_block": s_launches,
            "prefill_tokens_per_s": SB * (sp - 1) / (sprefill_ms * 1e-3),
            "algorithmic_bytes_per_step": sbytes,
            "hbm_frac_of_peak": sbytes / (sms * 1e-3) / 1e9 / hbm_peak / world,
            "sampled_ids_sha": _sha(stok.cpu().numpy()),
            "note": "prompts of 1024 uniform-random ids in [0, 50257) left-padded into seq 2048, nucleus sampling "
                    "(top_p 0.9, temperature 1.0, seeded uniforms); fraction = whole-model bytes per step / time / "
                    "(measured HBM peak x n_gpus)"}
        barrier()
        rt2.close()
    else:
        parity_eval = {}
    net.state = None
    torch.cuda.empty_cache()

    # ---- third runtime (8 GPUs only): the ~22B scale-up, batch 32 at a 2048-token context (config 5) ----
    if world == 8 and not serving and not args.headline_only and args.model == "6b" and args.layers == 0:
        cfg22 = dict(GPTJ_22B, cores_per_replica=world)
        net22 = build_network(cfg22, device, rank, world, seed=4321)
        SB, sp = 32, 1792
        rt3 = ShardRuntime(cfg22, rank=rank, device=device, max_batch=SB, max_gen=3 * 16 + 32, max_rows=2048)
        rt3.load_params(net22.state["params"])
        net22.state = None
        torch.cuda.empty_cache()
        sctx = np.random.Generator(np.random.PCG64(6)).integers(0, 50257, size=(SB, seq)).astype(np.uint32)
        sctx[:, :seq - sp] = 0
        sctx_dev = torch.from_numpy(sctx.view(np.int32)).to(device)
        pool = uniform_pool(SB, cfg22["n_vocab"])
        tp_dev, tt_dev = torch.full((SB,), 0.9, device=device), torch.full((SB,), 1.0, device=device)
        stok = torch.empty((SB,), dtype=torch.int32, device=device)
        cnt = [0]

        def bstep():
            cnt[0] += 1
            rt3.decode_step(None, stok, None, greedy=False, top_p=tp_dev, temp=tt_dev, uniforms=pool[cnt[0] % 4])

        rt3.prefill(sctx_dev, [sp] * SB)
        bprefill_ms = timed(lambda: rt3.prefill(sctx_dev, [sp] * SB))
        for _ in range(8):
            bstep()
        bblocks = [timed(lambda: [bstep() for _ in range(16)]) for _ in range(3)]
        bms = median(bblocks) / 16
        bbytes = decode_bytes_per_step(cfg22, SB, sp + 8 + 24)
        rt3.check_device_status()
        extra_blocks["model_22b"] = {
            "tokens_per_s": SB / (bms * 1e-3), "ms_per_step": bms, "batch": SB, "prompt": sp, "block_ms": bblocks,
            "prefill_tokens_per_s": SB * (sp - 1) / (bprefill_ms * 1e-3), "algorithmic_bytes_per_step": bbytes,
            "hbm_frac_of_peak": bbytes / (bms * 1e-3) / 1e9 / hbm_peak / world,
            "workload": "GPT-J-style 22B (L48 d6144 h24 dh256 rot64 ff24576 V50400) bf16 random-init, mp8, "
                        "1792-token prompts, nucleus sampling top_p 0.9"}
        barrier()
        rt3.close()
    if world > 1:
        barrier()
        dist.destroy_process_group()
    if rank != 0:
        return

    d, dl, ffl = cfg["d_model"], cfg["d_model"] // world, 4 * cfg["d_model"] // world
    Vl, L = cfg["n_vocab"] // world, cfg["layers"]
    # keys a decode step attends to: the full window, or (serving) the prompt plus what has been generated so far
    ctx_avg = (seq - 1) if not serving else min(seq - 1, prompt + n_calls[0] // 2)
    # algorithmic bytes per launch of each decode kernel family on ONE rank (weights dominate)
    fam_bytes = {
        "in_proj": ((3 * dl + (0 if prof["ff_in_proj"][1] else ffl)) * d * 2 + 2 * d * 4
                    + B * (d * 4 + dl * 4 + 2 * dl * 2)),
        "ff_in_proj": ffl * d * 2 + ffl * 4 + 2 * d * 4 + B * (d * 4 + ffl * 4),
        "attention": B * ctx_avg * 2 * dl * 2 + B * 2 * dl * 4,
        "out_proj": d * (dl + ffl) * 2 + d * 4 + B * ((dl + ffl) * 4 + 2 * d * 4),
        "logits": Vl * d * 2 + Vl * 4 + 2 * d * 4 + B * (d * 4 + Vl * 4),
    }
    fam_kernel = {
        "in_proj": "in-projection (LN + Q/K/V rows, RoPE, KV-cache write)",
        "ff_in_proj": "in-projection (LN + FF-in rows, bias + GELU)",
        "attention": "decode attention over the paged KV cache",
        "out_proj": "out-projection ([attn | gelu(ff)] x [W_o ; W_ff_out] + bias + residual + LN stats)",
        "logits": "final LN + logits",
    }
    per_step = {"in_proj": L, "ff_in_proj": L, "attention": L, "out_proj": L, "logits": 1}
    fam = {}
    for k, (ms_sum, n) in prof.items():
        if not n:
            continue
        ms_l = ms_sum / n
        fam[k] = {"ms_per_launch": ms_l, "launches": n, "bytes_per_launch": fam_bytes[k],
                  "gbs": fam_bytes[k] / (ms_l * 1e-3) / 1e9, "ms_per_step": ms_l * per_step[k]}
    top = max(fam, key=lambda k: fam[k]["ms_per_step"]) if fam else None
    achieved = fam[top]["gbs"] if top else None
    pf = {k: v[0] for k, v in prefill_prof.items() if v[1]}
    gemm_flops = 2.0 * (L * 12 * d * d // world) * B * (prompt - 1)
    attn_flops = L * 2.0 * (d // world) * (prompt - 1) * prompt * B
    gemm_ms = pf.get("in_proj", 0.0) + pf.get("out_proj", 0.0)

    ms_step = ms_total / K
    value = B * K / (ms_total * 1e-3)
    step_bytes = decode_bytes_per_step(cfg, B, ctx_avg)
    rank_bytes = step_bytes / world               # weights, KV and their traffic shard evenly over the ranks
    if phases is not None:
        # one persistent kernel does the whole step: it is the dominant kernel
        top = "mega"
        fam_kernel["mega"] = ("decode_mega_kernel (whole decode step: embedding, L x [LN + in-proj, attention, "
                              "out-proj + residual], final LN + logits)")
        fam["mega"] = {"ms_per_launch": ms_step, "launches": K, "bytes_per_launch": rank_bytes,
                       "gbs": rank_bytes / (ms_step * 1e-3) / 1e9, "ms_per_step": ms_step}
        achieved = fam["mega"]["gbs"]
    frac = (achieved / hbm_peak) if achieved else None
    assert frac is None or frac <= 1.05, f"roofline fraction {frac} is not credible"
    prefill_flops = gemm_flops * world + attn_flops * world + 0.0
    line = {
        "metric": METRIC, "value": value, "unit": UNIT, "n_gpus": world, "steps": K,
        "warmup": W, "ms_per_step": ms_step, "higher_is_better": True, "scaling": "strong",
        "vs_baseline": None, "dtype": "bf16", "data": "synthetic", "config": workload_config(args, world),
        "timing": {"blocks": n_blocks, "block_ms": block_ms, "reported": "median block",
                   "extra_warmup_steps": extra, "note": f"each block is exactly {K} steps between barrier + "
                   "synchronize, CUDA events, max over ranks; the clock starts after the --warmup steps plus "
                   "0.3 s of steady stepping"},
        "e2e": {"value": B * K / e2e_decode_s, "unit": UNIT,
                "h2d_bytes_per_step": int(ctx.nbytes) / K, "d2h_bytes_per_step": 4 * B,
                "api": "CausalTransformer.generate(ctx, ctx_length, steps): host context in (pinned), host tokens "
                       "out; value = tokens / wall-clock of the decode part (median of 3 calls, max over ranks), "
                       "the prefill of the same call timed separately",
                "prefill_s": e2e_prefill_s, "decode_s": e2e_decode_s},
        "gpu_launches": launches,
        "clocks": sampler.summary(t_wall0, t_wall1),
        "roofline": {"bound": "hbm", "kernel": fam_kernel.get(top), "achieved": achieved, "peak": hbm_peak,
                     "unit": "GB/s", "frac": frac,
                     "traffic": NCU_TRAFFIC.get(top) if world == 1 and B == 1 and args.layers == 0 else None,
                     "peak_source": f"of {peak_kind}", "per": "GPU (this rank's share of the model's bytes)",
                     "algorithmic_bytes_per_launch": fam[top]["bytes_per_launch"] if top else None,
                     "ms_per_launch": fam[top]["ms_per_launch"] if top else None,
                     "note": ("whole-step persistent kernel; duration = CUDA-event time of the median block / steps "
                              "(includes the small token-selection kernel that follows it in the replayed graph)")
                     if top == "mega" else
                     ("kernel with the largest share of the decode step; time from CUDA events around each "
                      "launch in a separate pass (no graph replay, so launch gaps are included)")},
        "parity": dict({"greedy_first16": greedy16, "greedy_first16_sha": _sha(np.array(greedy16 or [], np.int64)),
                        "generate_first16": [int(v) for v in gen_tokens[0, :16, 0]],
                        "decode_loop_equals_generate": (greedy16 == [int(v) for v in gen_tokens[0, :16, 0]]
                                                        if greedy16 is not None and K >= 16 else None),
                        "note": "every N runs the same seeded model (full leaves drawn from one seed, sliced per "
                                "rank) on the same ids: these values agree across N up to summation order"},
                       **parity_eval),
        "mega_phases": phases,
        "kernel_families": fam,
        "step_hbm": {"algorithmic_bytes_per_step": step_bytes, "achieved_gbs": step_bytes / (ms_step * 1e-3) / 1e9,
                     "frac_of_peak": step_bytes / (ms_step * 1e-3) / 1e9 / hbm_peak / world},
        "prefill": {"tokens_per_s": B * (prompt - 1) / (prefill_ms * 1e-3), "ms": prefill_ms, "tokens": B * (prompt - 1),
                    "timing": "median of 10", "family_ms": pf,
                    "gemm_tflops_per_gpu": (gemm_flops / (gemm_ms * 1e-3) / 1e12) if gemm_ms else None,
                    "gemm_frac_of_burst_peak": (gemm_flops / (gemm_ms * 1e-3) / 1e12 / tc_burst) if gemm_ms else None,
                    "attention_tflops_per_gpu": (attn_flops / (pf["attention"] * 1e-3) / 1e12) if pf.get("attention") else None,
                    "whole_prefill_tflops": prefill_flops / (prefill_ms * 1e-3) / 1e12,
                    "whole_prefill_frac_of_burst_peak": prefill_flops / (prefill_ms * 1e-3) / 1e12 / tc_burst / world,
                    "peaks": {"bf16_tflops_burst": tc_burst, "bf16_tflops_sustained": tc_sustained,
                              "denominator": "burst (a prefill pass lasts milliseconds)"}},
    }
    line.update(extra_blocks)
    if args.layers > 0:
        line["profile_only"] = f"reduced depth: {args.layers} layers"
    if world == 1 and not args.no_cpu_baseline:
        from oracle import cpu_baseline
        r = cpu_baseline.decode_tokens_per_s(GPTJ_6B, steps=8, warmup=1, batch=1)      # about 13 s of host work
        line["cpu_baseline"] = {"value": r["value"], "unit": UNIT, "cores": r["cores"], "kind": "port",
                                "sample": r["sample"]}
    print(json.dumps(line), flush=True)


# ------------------------------------------------------- layer-stack models ----
def keselix_model(d):
    """A Keselix model with layers of a real model's proportions at width d: a state-space layer and a latent-attention
    layer in turn, the middle two run twice."""
    attn = {"type": "latent_attention",
            "mixer": {"heads": d // 128, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 512, "scale": 192 ** -0.5,
                      "mask": {"size": 1024}, "rot": {"base": 10000.0, "dims": 64}},
            "mlp": {"kind": "dense", "ff": d * 11 // 4}}
    ssm = {"type": "mamba1", "mixer": {"inner": 2 * d, "state": 16, "conv": 4, "dt_rank": d // 16}, "mlp": None}
    return {"architecture": "Keselix", "vocab": 32768, "width": d, "layers": [ssm, attn, ssm, attn],
            "loop": {"start": 1, "stop": 3, "times": 2}, "norm": {"eps": 1e-5}, "residual_mult": 0.5, "seq": 2048}


def bavutar_model(d):
    """A Bavutar model with layers of a real model's proportions at width d: delta-rule, attention, Mamba-2 and delta-rule
    layers, an attention layer that reads the first one's keys and values, and a Mamba-2 layer."""
    mlp = {"kind": "dense", "ff": 3 * d}
    attn = {"type": "attention", "mlp": mlp,
            "mixer": {"heads": d // 128, "kv_heads": d // 512, "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                      "q_temp": {"coef": 0.1, "every": 8192}}}
    delta = {"type": "channel_delta", "mlp": mlp,
             "mixer": {"heads": d // 128, "kv_heads": d // 128, "dim": 128, "vdim": 128, "conv": 4, "decay_rank": 128, "gate_rank": 128}}
    ssd = {"type": "mamba2", "mlp": mlp,
           "mixer": {"heads": d // 32, "vdim": 64, "state": 128, "groups": 8, "norm_groups": 8, "conv": 4}}
    late = dict(attn, mixer=dict(attn["mixer"], kv_from=1))
    return {"architecture": "Bavutar", "vocab": 32768, "width": d, "layers": [delta, attn, ssd, delta, late, ssd], "norm": {"eps": 1e-5},
            "postln_alpha": 2.0, "embedding": {"scale": 1.0}, "logit_softcap": 30.0, "seq": 2048}


def stack_work(cfg, runs, T):
    """(weight elements a decode step reads, flops of a T-token prompt without the logits, bytes of caches and states a
    sequence of T tokens moves in a decode step) over the layer runs."""
    from mesh_transformer.layer_stack import tensor_shapes
    import math
    shapes = tensor_shapes(cfg)
    weights = sum(math.prod(v) for i in runs for k, v in shapes.items()
                  if k.startswith(f"l{i}.") and len(v) > 1 and "conv" not in k and "A_log" not in k)
    if cfg.get("loop"):
        weights += cfg["loop"]["times"] * math.prod(shapes["loop.in"])
    extra, moved = 0, 0
    for i in runs:
        kind, m = cfg["layers"][i]["type"], cfg["layers"][i]["mixer"]
        if kind == "latent_attention":
            w = m["mask"]["size"]
            extra += 2 * sum(min(t + 1, w) for t in range(T)) * m["heads"] * (m["dim"] + m["rot_dim"] + m["vdim"])
            moved += min(T, w) * (m["kv_rank"] + m["rot_dim"]) * 2
        elif kind == "attention":
            extra += T * (T + 1) * m["heads"] * (m["dim"] + m["vdim"])
            moved += T * m["kv_heads"] * (m["dim"] + m["vdim"]) * 2
        elif kind == "mamba1":
            extra += 6 * T * m["inner"] * m["state"]
            moved += 2 * m["inner"] * 4 * (m["state"] + m["conv"] - 1)
        else:
            n = m["state"] if kind == "mamba2" else m["dim"]
            extra += (6 if kind == "mamba2" else 8) * T * m["heads"] * n * m["vdim"]
            moved += 2 * m["heads"] * n * m["vdim"] * 4
    return weights, 2 * weights * T + extra, moved


def run_stack(args):
    """A layer-stack model beside another at equal width and number of layer runs (Keselix beside GPT-J, Bavutar beside
    Keselix), one GPU, random weights: prefill of one 2048-token prompt, decode of 1, 8 and 32 sequences behind such
    prompts, kernel families."""
    import torch
    import __graft_entry__ as ge
    if args.gpus != 1:
        raise SystemExit("--workload stack runs on one GPU")
    ge.build()
    from mesh_transformer._runtime import ShardRuntime
    from mesh_transformer.transformer_shard import CausalTransformer
    torch.cuda.set_device(0)
    device = torch.device("cuda", 0)
    try:
        peaks = json.load(open(os.path.join(ROOT, "MEASURED_PEAKS.json")))
    except Exception:
        peaks = {}
    hbm, tc = float(peaks.get("hbm_gbs", 6650.0)), float(peaks.get("bf16_tflops", 1590.0))
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)

    def timed(fn):
        torch.cuda.synchronize()
        e0.record()
        fn()
        e1.record()
        torch.cuda.synchronize()
        return e0.elapsed_time(e1)

    def median(xs):
        return sorted(xs)[len(xs) // 2]

    sampler = ClockSampler(0)
    sampler.start()
    t_wall0 = time.time()
    T, K, W = 2048, args.steps, args.warmup
    sizes, launches = {}, 0
    names = {"keselix": ("keselix", "gptj"), "bavutar": ("bavutar", "keselix")}[args.stack_model]
    for d in [int(v) for v in args.stack_widths.split(",")]:
        models = {"keselix": lambda: (keselix_model(d), [0, 1, 2, 1, 2, 3]), "bavutar": lambda: (bavutar_model(d), list(range(6))),
                  "gptj": lambda: (dict(GPTJ_6B, layers=6, d_model=d, n_heads=d // 256, n_vocab=32768, early_cast=True), list(range(6)))}
        row = {}
        for name in names:
            cfg, runs = models[name]()
            net = CausalTransformer(dict(cfg), device=device, init_weights=False)
            net.state = net._init_state(seed=42)
            V = 32768
            if name != "gptj":
                weights, flops, cache = stack_work(cfg, runs, T - 1)
            else:
                weights = 12 * d * d * len(runs)
                flops = 2 * weights * (T - 1) + len(runs) * 2 * d * (T - 1) * T
                cache = len(runs) * (T - 1) * 2 * d * 2
            weights += V * d
            out = {"weights_read_per_step_mb": weights * 2 / 1e6}
            for B in (1, 8, 32):
                # every prompt twice, warm-up and K timed steps, the blocks, a profiled pass
                rt = ShardRuntime(net.config, device=device, max_batch=B, max_gen=W + 6 * K + 64, max_rows=4096)
                rt.load_params(net.state["params"])
                ctx = torch.randint(0, V, (B, T), dtype=torch.int32, device=device)
                rt.prefill(ctx, [T] * B)
                if B == 1:
                    rt.prefill(ctx, [T])
                    ms = median([timed(lambda: rt.prefill(ctx, [T])) for _ in range(7)])
                    rt.profile_enable(True)
                    rt.prefill(ctx, [T])
                    fam = {k: v[0] for k, v in rt.profile_read().items() if v[1]}
                    rt.profile_enable(False)
                    out["prefill_2048"] = {"ms": ms, "tokens_per_s": (T - 1) / ms * 1e3, "tflops": flops / ms / 1e9,
                                           "frac_of_bf16_peak": flops / ms / 1e9 / tc, "family_ms": fam}
                tok = torch.empty((B,), dtype=torch.int32, device=device)
                for _ in range(max(W, 3)):
                    rt.decode_step(None, tok)
                n0 = rt.launch_count()
                ms = median([timed(lambda: [rt.decode_step(None, tok) for _ in range(K)]) for _ in range(5)]) / K
                launches += (rt.launch_count() - n0) // 5
                rt.profile_enable(True)
                for _ in range(8):
                    rt.decode_step(None, tok)
                fam = {k: v[0] / 8 for k, v in rt.profile_read().items() if v[1]}
                rt.profile_enable(False)
                rt.check_device_status()
                nbytes = weights * 2 + B * cache
                out[f"decode_b{B}"] = {"ms_per_step": ms, "tokens_per_s": B / ms * 1e3, "gbs": nbytes / ms / 1e6,
                                       "frac_of_hbm_peak": nbytes / ms / 1e6 / hbm, "family_ms": fam,
                                       "launches_per_step": (rt.launch_count() - n0) / (5 * K + 8)}
                rt.close()
                del rt
            net.state = None
            torch.cuda.empty_cache()
            row[name] = out
        sizes[str(d)] = row
    sampler.stop()
    top = sizes[str(args.stack_widths.split(",")[-1])][names[0]]
    print(json.dumps({
        "metric": names[0] + "_decode_tokens_per_s", "value": top["decode_b1"]["tokens_per_s"], "unit": UNIT, "n_gpus": 1,
        "steps": K, "warmup": W, "ms_per_step": top["decode_b1"]["ms_per_step"], "higher_is_better": True, "scaling": "strong",
        "vs_baseline": None, "dtype": "bf16", "data": "synthetic", "gpu_launches": launches,
        "clocks": sampler.summary(t_wall0, time.time()),
        "peaks": {"hbm_gbs": hbm, "bf16_tflops": tc, "source": "measured" if peaks else "fallback"},
        "config": {"workload": f"layer-stack model ({names[0]}) beside {names[1]} at equal width and number of layer runs; "
                               "random weights; one 2048-token prompt, greedy decode",
                   "l2": "every step reads more weights than L2 holds", "parallelism": "mp1"},
        "sizes": sizes}), flush=True)


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=64)
    ap.add_argument("--warmup", type=int, default=8)
    ap.add_argument("--impl", default="mtj", choices=["mtj", "reference"])
    ap.add_argument("--batch", type=int, default=1)
    ap.add_argument("--model", default="6b", choices=["6b", "22b"],
                    help="6b: GPT-J-6B (the headline); 22b: the L48 d6144 h24 scale-up (fits 8 GPUs)")
    ap.add_argument("--workload", default="headline", choices=["headline", "serving", "stack"],
                    help="headline: full-window greedy decode; serving: 1024-token prompts + nucleus sampling; stack: a "
                         "layer-stack model (--stack-model) beside the closest other one at equal widths")
    ap.add_argument("--stack-widths", default="2048,4096", help="widths of --workload stack")
    ap.add_argument("--stack-model", default="keselix", choices=["keselix", "bavutar"],
                    help="model of --workload stack: keselix (beside GPT-J) or bavutar (beside keselix)")
    ap.add_argument("--no-cpu-baseline", action="store_true")
    ap.add_argument("--headline-only", action="store_true",
                    help="skip the eval 8 x 2048, serving batch-32 and (8 GPUs) 22B blocks of the JSON line")
    ap.add_argument("--layers", type=int, default=0,
                    help="profiling aid: run a reduced-depth model (same layer shapes) so that an ncu capture "
                         "stays small; the printed line is marked profile_only and is not a benchmark result")
    args = ap.parse_args()
    if args.impl == "reference":
        run_reference(args)
    elif args.workload == "stack":
        run_stack(args)
    else:
        run_mtj(args)


if __name__ == "__main__":
    main()
