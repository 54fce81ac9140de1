#!/usr/bin/env python3
"""Decode and prefill throughput of Falcon-H1 (1.5B layer sizes, random weights) on one B200.

    python bench.py [--gpus 1] [--steps K] [--warmup W] [--impl reference]

A step is one decode step of the whole batch (8 sequences by default, each continuing a
512-token prompt; the cache is sized for the 4096-token benchmark context).  The line
printed is one JSON object:
  value      decoded tokens per second, timed on the device (CUDA events around K replayed steps
             of the engine's captured decode step, sampling included)
  e2e        the same through the Python entry point LLM.generate(): host token ids in, host
             token ids out, every step copying its inputs from pinned memory and reading its
             result back
  prefill    one 2,048-token prompt: tokens per second, milliseconds, fraction of the bf16 peak
  roofline   bytes a decode step has to read (every weight once + the live cache) / its time,
             against the measured HBM bandwidth
  points     decode at batch 1, 16, 32 and 64, at batch 8 with 3,800-token prompts, and the workloads of the
             3B and 7B layer sizes (16 unequal prompts with 256 sampled tokens each; batch-64 decode from
             1,024-token prompts and one 8,192-token prompt)
The reference publishes no Falcon-H1 number (vs_baseline is null) and runs the model on the CPU only
(falcon_h1.c:78-83); --impl reference builds the unmodified reference and measures that CPU engine on the
same layer sizes at batch 1, the only batch it has (baseline/reference_arm.py).
"""
import argparse
import json
import os
import subprocess
import sys
import time

ROOT = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, ROOT)

# Falcon-H1-1.5B layer sizes (context 4096, tied embeddings, muP multipliers set)
CONFIG_1P5B = dict(
    architectures=["FalconH1ForCausalLM"], model_type="falcon_h1", vocab_size=65536, hidden_size=2048,
    num_hidden_layers=24, num_attention_heads=8, num_key_value_heads=2, head_dim=128, intermediate_size=4096,
    rope_theta=1e11, max_position_embeddings=4096, rms_norm_eps=1e-5, tie_word_embeddings=True,
    mamba_d_ssm=3072, mamba_n_heads=48, mamba_d_head=64, mamba_n_groups=1, mamba_d_state=256, mamba_d_conv=4,
    mamba_chunk_size=128, mamba_conv_bias=True, mamba_proj_bias=False, mamba_rms_norm=True,
    mamba_norm_before_gate=False, embedding_multiplier=5.66, lm_head_multiplier=0.039, key_multiplier=0.39,
    attention_in_multiplier=1.0, attention_out_multiplier=0.94, ssm_in_multiplier=1.25, ssm_out_multiplier=0.24,
    mlp_multipliers=[0.88, 0.3], ssm_multipliers=[0.35, 0.25, 0.7, 0.5, 0.35])
# the 3B and 7B layer sizes (their other options as above): --sizes 3B / 7B
CONFIG_3B = dict(CONFIG_1P5B, hidden_size=2560, num_hidden_layers=32, num_attention_heads=10, intermediate_size=8192,
                 mamba_d_ssm=4096, mamba_n_heads=32, mamba_d_head=128)
CONFIG_7B = dict(CONFIG_1P5B, hidden_size=3072, num_hidden_layers=44, num_attention_heads=12, intermediate_size=12288,
                 vocab_size=130048, max_position_embeddings=8192, tie_word_embeddings=False,
                 mamba_d_ssm=3072, mamba_n_heads=24, mamba_d_head=128)
CONFIGS = {"1.5B": CONFIG_1P5B, "3B": CONFIG_3B, "7B": CONFIG_7B}


def peaks():
    p = dict(hbm_gbs=6650.0, bf16_tflops=1590.0, source="fallback")
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.isfile(path):
        try:
            m = json.load(open(path))
            p = dict(hbm_gbs=float(m.get("hbm_gbs", p["hbm_gbs"])), bf16_tflops=float(m.get("bf16_tflops", p["bf16_tflops"])),
                     source="measured")
        except Exception:
            pass
    return p


def sizes(cfg):
    D, F, V, L = cfg["hidden_size"], cfg["intermediate_size"], cfg["vocab_size"], cfg["num_hidden_layers"]
    H, KV, hd = cfg["num_attention_heads"], cfg["num_key_value_heads"], cfg["head_dim"]
    Di, Hs, N, G, K = cfg["mamba_d_ssm"], cfg["mamba_n_heads"], cfg["mamba_d_state"], cfg["mamba_n_groups"], cfg["mamba_d_conv"]
    Cd = Di + 2 * G * N
    Pd = Di + Cd + Hs
    layer_w = D * (H * hd + 2 * KV * hd) + H * hd * D + D * Pd + Di * D + 2 * D * F + F * D
    return dict(D=D, F=F, V=V, L=L, H=H, KV=KV, hd=hd, Di=Di, Hs=Hs, N=N, G=G, K=K, Cd=Cd, Pd=Pd, layer_w=layer_w,
                P=Di // Hs)


def decode_bytes(cfg, batch, context):
    """Bytes one decode step has to read: every weight it uses once (bf16 matrices, head
    included), and the cache of the live sequences (bf16 keys and values up to `context`,
    the 32-bit conv window and SSM state)."""
    s = sizes(cfg)
    weights = (s["L"] * s["layer_w"] + s["V"] * s["D"]) * 2          # the head's matrix; a token's embedding row is 4 KB
    kv = 2 * s["L"] * s["KV"] * s["hd"] * 2 * context
    state = s["L"] * (s["Hs"] * s["P"] * s["N"] + (s["K"] - 1) * s["Cd"]) * 4
    return weights + batch * (kv + state)


def prefill_flops(cfg, T):
    s = sizes(cfg)
    gemm = 2 * T * s["L"] * s["layer_w"] + 2 * s["V"] * s["D"]          # head on one row
    attn = s["L"] * 2 * 2 * s["H"] * s["hd"] * T * (T + 1) / 2           # QK^T and PV, causal
    ssd = s["L"] * T * s["Hs"] * s["P"] * s["N"] * 6                       # state update + readout
    return gemm + attn + ssd


class Clocks:
    """Samples nvidia-smi while a timed region runs."""
    Q = ("clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,clocks_event_reasons.hw_thermal_slowdown,"
         "clocks_event_reasons.sw_thermal_slowdown,clocks_event_reasons.sw_power_cap")

    def __enter__(self):
        try:
            self.p = subprocess.Popen(["nvidia-smi", "-i", "0", f"--query-gpu={self.Q}", "--format=csv,noheader,nounits",
                                       "-lms", "100"], stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True)
        except OSError:
            self.p = None
        return self

    def __exit__(self, *a):
        self.result = dict(sm_mhz=None, sm_max_mhz=None, reasons=[])
        if self.p is None:
            return
        time.sleep(0.15)
        self.p.terminate()
        out, _ = self.p.communicate()
        sm, mx, reasons = [], [], set()
        for line in out.splitlines():
            f = [x.strip() for x in line.split(",")]
            if len(f) < 6 or not f[0].isdigit():
                continue
            sm.append(int(f[0]))
            mx.append(int(f[1]))
            for name, v in zip(("hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"), f[2:6]):
                if v.lower().startswith("active"):
                    reasons.add(name)
        if sm:
            sm.sort()
            self.result = dict(sm_mhz=sm[len(sm) // 2], sm_max_mhz=max(mx), reasons=sorted(reasons))


def time_decode(llm, tlc, batch, prompt_len, steps, warmup, seed):
    """Device time of `steps` decode steps of `batch` sequences through the engine's own decode step
    (EngineBackend.decode_step: reserve, upload, replay of the captured step, read-back, commit)."""
    import torch
    from tinyllama_c_b200 import ops
    from tinyllama_c_b200.engine import EngineBackend, StepEntry
    g = torch.Generator().manual_seed(seed)
    V = llm.model.vocab
    slots = [llm.cache.acquire() for _ in range(batch)]
    prompts = torch.randint(0, V, (batch, prompt_len), generator=g).tolist()
    # prompts in groups that bound activation memory
    group = max(1, 8192 // prompt_len)
    for i in range(0, batch, group):
        llm.step([StepEntry(s, p, ()) for s, p in zip(slots[i:i + group], prompts[i:i + group])])
    backend = EngineBackend(llm.model, llm.cache, tlc.GREEDY, llm._graphs, True)
    toks = torch.randint(0, V, (batch,), generator=g).tolist()

    def one():
        nonlocal toks
        toks = backend.decode_step([(s, [t]) for s, t in zip(slots, toks)])

    for _ in range(max(3, warmup)):
        one()
    torch.cuda.synchronize()
    l0 = ops.launch_count()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    with Clocks() as clk:
        e0.record()
        for _ in range(steps):
            one()
        e1.record()
        torch.cuda.synchronize()
    ms = e0.elapsed_time(e1) / steps
    launches = ops.launch_count() - l0
    ctx = prompt_len + max(3, warmup) + steps // 2
    for s in slots:
        llm.cache.release(s)
    ops.check_errors()
    return ms, launches, clk.result, ctx


def time_prefill(llm, T, seed, reps=3):
    import torch
    from tinyllama_c_b200 import ops
    from tinyllama_c_b200.engine import StepEntry
    g = torch.Generator().manual_seed(seed)
    best = None
    warm = 4                               # the first runs ramp the clocks and fill the tensor-map caches
    for r in range(reps + warm):
        toks = torch.randint(0, llm.model.vocab, (T,), generator=g).tolist()
        s = llm.cache.acquire()
        torch.cuda.synchronize()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        llm.step([StepEntry(s, toks, (T - 1,))])
        e1.record()
        torch.cuda.synchronize()
        llm.cache.release(s)
        if r >= warm:
            ms = e0.elapsed_time(e1)
            best = ms if best is None else min(best, ms)
    ops.check_errors()
    return best


def e2e_decode(llm, tlc, batch, prompt_len, steps, seed):
    import torch
    g = torch.Generator().manual_seed(seed)
    prompts = torch.randint(0, llm.config.vocab_size, (batch, prompt_len), generator=g).tolist()
    llm.generate(prompts, tlc.GREEDY, max_new_tokens=4, ignore_eos=True, max_batch=batch)      # warm-up, captures the graph
    llm.generate(prompts, tlc.GREEDY, max_new_tokens=steps + 1, ignore_eos=True, max_batch=batch)
    st = llm.last_stats
    return st["decode_tokens"] / st["decode_s"], st["h2d_bytes"] // max(1, st["decode_steps"]), \
        st["d2h_bytes"] // max(1, st["decode_steps"])


def time_generate(llm, tlc, n_prompts, lo, hi, new_tokens, temperature, seed):
    """Unequal prompts (lengths uniform in [lo, hi]) generated together through LLM.generate() with temperature
    sampling, every sequence to new_tokens: host token ids in and out, the second of two runs timed."""
    import torch
    g = torch.Generator().manual_seed(seed)
    lens = torch.randint(lo, hi + 1, (n_prompts,), generator=g).tolist()
    prompts = [torch.randint(0, llm.config.vocab_size, (n,), generator=g).tolist() for n in lens]
    sampling = tlc.SamplingParams(temperature=temperature, seed=seed)
    out = {}
    for run in range(2):
        torch.cuda.synchronize()
        t0 = time.perf_counter()
        llm.generate(prompts, sampling, max_new_tokens=new_tokens, ignore_eos=True, max_batch=n_prompts)
        torch.cuda.synchronize()
        out = dict(llm.last_stats, wall_s=time.perf_counter() - t0)
    return {"prompts": n_prompts, "prompt_tokens": sum(lens), "new_tokens": n_prompts * new_tokens,
            "temperature": temperature, "wall_s": round(out["wall_s"], 4),
            "prefill_tok_s": round(out["prefill_tokens"] / out["prefill_s"], 1),
            "decode_tok_s": round(out["decode_tokens"] / out["decode_s"], 1),
            "tok_s": round(n_prompts * new_tokens / out["wall_s"], 1)}


def main() -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=64)
    ap.add_argument("--warmup", type=int, default=8)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--layers", type=int, default=None, help="fewer layers than the model has (both numbers are reported)")
    ap.add_argument("--prompt-len", type=int, default=512)
    ap.add_argument("--no-points", action="store_true", help="skip the batch 1 / 64 points and the prefill")
    ap.add_argument("--sizes", default="1.5B", choices=sorted(CONFIGS), help="layer sizes of this Falcon-H1 model")
    ap.add_argument("--prefill-tokens", type=int, default=2048)
    ap.add_argument("--generate", type=int, default=0, metavar="N",
                    help="also generate 256 tokens for N prompts of 64..2048 tokens at temperature 0.7")
    ap.add_argument("--prefill-only", action="store_true", help="time the prompt of --prefill-tokens tokens only "
                    "(--steps repetitions when fewer than 8): what a profiler capture of the prompt kernels runs")
    ap.add_argument("--no-big", dest="big", action="store_false", help="skip the 3B and 7B workloads among the points")
    ap.add_argument("--no-pairs", action="store_true", help="run the linear layers on single blocks (128 x 256 tiles) instead "
                    "of pairs of blocks on 256 x 256 tiles: the comparison behind profiles/linear_tcgen05_prefill_2048.md")
    ap.add_argument("--design", default=None, choices=["turevik", "porarax", "sogazen", "kimutar", "kefetar", "fobatar"], help="instead of the benchmark line: prefill and decode "
                    "throughput of this design at layer sizes of a real model's order (random weights), beside the library's "
                    "closest other design (Falcon-H1 for turevik and sogazen, Turevik for porarax, Porarax for kimutar and fobatar, Kimutar for kefetar) at equal "
                    "width and layer count")
    ap.add_argument("--sizes-only", default=None, choices=["width 2048", "width 3072"], help="with --design: one of the two sizes")
    ap.add_argument("--ref-budget", type=float, default=600.0, help="seconds the reference arm may take (it runs fewer "
                    "layers, and says so, where all of them would take longer)")
    args = ap.parse_args()

    if args.impl == "reference":
        return reference_arm(args)
    if args.gpus != 1:
        print(f"bench.py measures one GPU; --gpus {args.gpus} is not supported by this single-GPU library")
        return 2

    if args.design:
        return design_compare(args)

    import torch
    import tinyllama_c_b200 as tlc
    if args.no_pairs:
        from tinyllama_c_b200 import ops
        ops.linear_pair_override(1)
    full_layers = CONFIGS[args.sizes]["num_hidden_layers"]
    if args.layers is None:
        args.layers = full_layers
    cfg = dict(CONFIGS[args.sizes], num_hidden_layers=args.layers)
    s = sizes(cfg)
    pk = peaks()
    ctx_len = cfg["max_position_embeddings"]
    model = tlc.random_model(cfg, seed=0, dtype="bfloat16")
    # room for 64 sequences of prompt + decoded tokens, for the long prompt and for the unequal batch
    per_seq = -(-(args.prompt_len + 2 * args.steps + 80) // 64) * 64
    room = max(64 * 1024, max(64, args.batch) * per_seq, args.prefill_tokens + 64, args.generate * (2048 + 256 + 64),
               8 * 3968)
    llm = tlc.LLM(model, max_tokens=room, max_seqs=max(64, args.batch, args.generate))

    if args.prefill_only:
        T = args.prefill_tokens
        pms = time_prefill(llm, T, seed=3, reps=args.steps if args.steps < 8 else 3)
        print(json.dumps({"prefill": {"value": round(T * 1000.0 / pms, 1), "tokens": T, "ms": round(pms, 3),
                                      "frac": round(prefill_flops(cfg, T) / (pms * 1e-3) / (pk["bf16_tflops"] * 1e12), 4)},
                          "layers": args.layers}))
        return 0

    ms, launches, clocks, ctx = time_decode(llm, tlc, args.batch, args.prompt_len, args.steps, args.warmup, seed=1)
    value = args.batch * 1000.0 / ms
    nbytes = decode_bytes(cfg, args.batch, ctx)
    achieved = nbytes / (ms * 1e-3) / 1e9
    e2e_v, h2d, d2h = e2e_decode(llm, tlc, args.batch, args.prompt_len, args.steps, seed=2)
    rec = {
        "metric": f"decode tok/s at batch {args.batch} (Falcon-H1-{args.sizes} sizes, {args.prompt_len}-token prompts, "
                  f"context {ctx_len})",
        "value": round(value, 1), "unit": "tok/s", "n_gpus": 1, "steps": args.steps, "warmup": max(3, args.warmup),
        "ms_per_step": round(ms, 4), "higher_is_better": True, "scaling": "weak", "vs_baseline": None,
        "dtype": "bf16", "data": "synthetic (random weights, uniform random token ids)",
        "config": {"model": f"Falcon-H1-{args.sizes} sizes", "global_batch": args.batch, "seq_len": ctx_len,
                   "prompt_len": args.prompt_len, "parallelism": "single GPU", "layers": args.layers,
                   "layers_full": full_layers, "hidden": cfg["hidden_size"],
                   "heads": f"{s['H']}q/{s['KV']}kv x{s['hd']}",
                   "intermediate": cfg["intermediate_size"], "vocab": cfg["vocab_size"],
                   "mamba": f"{s['Hs']} heads x{s['P']}, state {s['N']}, groups {s['G']}, conv {s['K']}",
                   "tied": cfg["tie_word_embeddings"],
                   "l2": f"inputs larger than L2 ({decode_bytes(cfg, 0, 0) / 1e9:.1f} GB of weights per step)"},
        "clocks": clocks, "gpu_launches": launches,
        "e2e": {"value": round(e2e_v, 1), "unit": "tok/s", "h2d_bytes_per_step": h2d, "d2h_bytes_per_step": d2h},
        "roofline": {"bound": "hbm", "achieved": round(achieved, 1), "peak": pk["hbm_gbs"], "unit": "GB/s",
                     "frac": round(achieved / pk["hbm_gbs"], 4), "peak_source": pk["source"]},
    }
    if not args.no_points:
        T = args.prefill_tokens
        pms = time_prefill(llm, T, seed=3)
        fl = prefill_flops(cfg, T)
        rec["prefill"] = {"value": round(T * 1000.0 / pms, 1), "tokens": T, "ms": round(pms, 3),
                          "frac": round(fl / (pms * 1e-3) / (pk["bf16_tflops"] * 1e12), 4)}
        pts = {}
        for b in (1, 16, 32, 64):
            m, _, _, c = time_decode(llm, tlc, b, args.prompt_len, max(16, args.steps // 2), 3, seed=4 + b)
            pts[f"decode_b{b}"] = round(b * 1000.0 / m, 1)
            pts[f"decode_b{b}_hbm_frac"] = round(decode_bytes(cfg, b, c) / (m * 1e-3) / 1e9 / pk["hbm_gbs"], 4)
        m, _, _, c = time_decode(llm, tlc, 8, 3800, max(16, args.steps // 2), 3, seed=31)
        pts["decode_b8_ctx3800"] = round(8 * 1000.0 / m, 1)
        pts["decode_b8_ctx3800_hbm_frac"] = round(decode_bytes(cfg, 8, c) / (m * 1e-3) / 1e9 / pk["hbm_gbs"], 4)
        rec["points"] = pts
    if args.generate:
        rec["generate"] = time_generate(llm, tlc, args.generate, 64, 2048, 256, 0.7, seed=9)
    if args.big and not args.no_points and args.sizes == "1.5B":
        del llm, model
        torch.cuda.empty_cache()
        rec["points"].update(big_workloads(tlc, pk))
    print(json.dumps(rec))
    return 0


# ---- another design beside Falcon-H1 ---------------------------------------------------------------------------------
def turevik_config(width, heads, kv_rank, ff, experts, top, expert_ff, shared_ff, gru, vocab):
    """Four layers with every kind of sublayer: latent attention with rows of its own and a dense feed-forward; latent
    attention over the first layer's rows and experts; minGRU and experts; latent attention and experts."""
    att = lambda **kw: dict(type="latent_attention", mixer=dict(heads=heads, dim=128, rot_dim=64, vdim=128, kv_rank=kv_rank,
                                                                scale=(128 + 64) ** -0.5, rot=dict(base=10000.0, dims=64), **kw))
    moe = dict(kind="moe", router=dict(experts=experts, top=top), expert=dict(ff=expert_ff), shared=dict(ff=shared_ff))
    return dict(architecture="Turevik", vocab=vocab, width=width, norm=dict(eps=1e-6), layers=[
        dict(att(), mlp=dict(kind="dense", ff=ff)), dict(att(kv_from=0), mlp=moe),
        dict(type="mingru", mixer=dict(width=gru), mlp=moe), dict(att(), mlp=moe)])


def turevik_work(cfg, batch, context, T):
    """(bytes a decode step of `batch` sequences at `context` must read, FLOPs of a prompt of T tokens)."""
    D, V = cfg["width"], cfg["vocab"]
    fixed, act_params, cache_bytes, att_flops = V * D, V * D, 0, 0.0
    expert_bytes = 0.0
    for layer in cfg["layers"]:
        m = layer["mixer"]
        if layer["type"] == "latent_attention":
            H, dn, r, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            n = H * (dn + r) * D + H * dn * R + H * dv * R + D * H * dv + (0 if "kv_from" in m else (R + r) * D)
            cache_bytes += batch * context * (R + r) * 2
            att_flops += 2.0 * H * (2 * R + r) * T * (T + 1) / 2
        else:
            n = 4 * m["width"] * D
        fixed += n
        act_params += n
        mlp = layer["mlp"]
        if mlp["kind"] == "dense":
            fixed += 3 * D * mlp["ff"]
            act_params += 3 * D * mlp["ff"]
        else:
            E, top, F = mlp["router"]["experts"], mlp["router"]["top"], mlp["expert"]["ff"]
            shared = 3 * D * mlp["shared"]["ff"] + D
            fixed += shared + E * D
            act_params += shared + E * D + top * 3 * D * F
            touched = E * (1.0 - (1.0 - 1.0 / E) ** (batch * top))          # expected distinct experts of a step
            expert_bytes += touched * 3 * D * F * 2
    return fixed * 2 + expert_bytes + cache_bytes, 2.0 * (act_params - V * D) * T + 2.0 * V * D + att_flops   # the head on one row


def porarax_config(width, heads, kv_heads, kv_rank, q_rank, window, experts, top, expert_ff, vocab):
    """Four layers with every kind of mixer, experts beside each: latent attention over a window with latents of its own;
    grouped-query attention (half of every head rotated); latent attention over the first layer's latents; the gated
    delta rule."""
    att = lambda **kw: dict(type="latent_attention", mixer=dict(heads=heads, dim=128, vdim=128, kv_rank=kv_rank, q_rank=q_rank,
                                                                scale=128 ** -0.5, mask=dict(size=window), **kw))
    moe = dict(kind="moe", router=dict(experts=experts, top=top), expert=dict(ff=expert_ff, limit=7.0))
    return dict(architecture="Porarax", vocab=vocab, width=width, norm=dict(eps=1e-6), layers=[
        dict(att(), mlp=moe),
        dict(type="attention", mixer=dict(heads=heads, kv_heads=kv_heads, dim=128, vdim=128, scale=128 ** -0.5,
                                          rot=dict(base=500000.0, dims=64)), mlp=moe),
        dict(att(kv_from=0), mlp=moe),
        dict(type="delta", mixer=dict(heads=heads, kv_heads=heads // 2, dim=128, vdim=128, conv=4), mlp=moe)])


def porarax_work(cfg, batch, context, T):
    """(bytes a decode step of `batch` sequences at `context` must read, FLOPs of a prompt of T tokens)."""
    D, V = cfg["width"], cfg["vocab"]
    fixed, cache_bytes, mix_flops, expert_bytes, expert_params = V * D, 0, 0.0, 0.0, 0
    for layer in cfg["layers"]:
        m = layer["mixer"]
        H, dk, dv = m["heads"], m["dim"], m["vdim"]
        if layer["type"] == "latent_attention":
            R, qr, W = m["kv_rank"], m["q_rank"], m["mask"]["size"]
            fixed += qr * D + H * dk * qr + H * dk * R + H * dv * R + D * H * dv + (0 if "kv_from" in m else R * D)
            cache_bytes += batch * min(context, W) * R * 2
            keys = sum(min(t + 1, W) for t in range(T)) if T > 1 else 1
            mix_flops += 2.0 * H * 2 * R * keys                       # scores and sums in the latent space
        elif layer["type"] == "attention":
            G = m["kv_heads"]
            fixed += (H * dk + G * dk + G * dv + H * dv) * D + D * H * dv
            cache_bytes += batch * context * G * (dk + dv) * 2
            mix_flops += 2.0 * H * (dk + dv) * T * (T + 1) / 2
        else:
            G = m["kv_heads"]
            fixed += (2 * G * dk + 2 * H * dv + 2 * H) * D + D * H * dv
            cache_bytes += batch * H * dk * dv * 4                    # the state, 32-bit
            mix_flops += 6.0 * H * dk * dv * T                        # the prediction M^T k, the write k w^T, the read-out M^T q
        mlp = layer["mlp"]
        E, top, F = mlp["router"]["experts"], mlp["router"]["top"], mlp["expert"]["ff"]
        fixed += E * D
        expert_params += top * 3 * D * F
        touched = E * (1.0 - (1.0 - 1.0 / E) ** (batch * top))              # expected distinct experts of a step
        expert_bytes += touched * 3 * D * F * 2
    return fixed * 2 + expert_bytes + cache_bytes, 2.0 * (fixed - V * D + expert_params) * T + 2.0 * V * D + mix_flops


def sogazen_config(width, heads, kv_heads, ssm_heads, ssm_vdim, state, wkv_heads, ff, experts, identity, top, expert_ff, vocab):
    """Four layers with every kind of sublayer: attention beside Mamba2 with a dense feed-forward; the same with experts;
    the wkv mixer with experts; attention beside Mamba2 with experts.  The attention and Mamba2 sizes are Falcon-H1's at
    that width."""
    par = dict(type="parallel", mixer=dict(
        left=dict(heads=heads, kv_heads=kv_heads, dim=128, vdim=128, scale=128 ** -0.5, softcap=30.0, rot=dict(base=1e6, dims=64)),
        right=dict(heads=ssm_heads, vdim=ssm_vdim, state=state, groups=1, norm_groups=2, conv=4)))
    moe = dict(kind="moe", router=dict(experts=experts, identity=identity, top=top), expert=dict(ff=expert_ff))
    return dict(architecture="Sogazen", vocab=vocab, width=width, norm=dict(eps=1e-6), logit_softcap=30.0, layers=[
        dict(par, mlp=dict(kind="dense", ff=ff, limit=7.0)), dict(par, mlp=moe),
        dict(type="wkv", mixer=dict(heads=wkv_heads, dim=64), mlp=moe), dict(par, mlp=moe)])


def sogazen_work(cfg, batch, context, T):
    """(bytes a decode step of `batch` sequences at `context` must read, FLOPs of a prompt of T tokens)."""
    D, V = cfg["width"], cfg["vocab"]
    fixed, cache_bytes, mix_flops, expert_bytes, expert_params = V * D, 0, 0.0, 0.0, 0.0
    for layer in cfg["layers"]:
        m = layer["mixer"]
        if layer["type"] == "parallel":
            a, s = m["left"], m["right"]
            H, G, dk, dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            fixed += (H * dk + G * dk) * D + D * H * dv                  # q, k (also the values), o
            cache_bytes += batch * context * G * (dk + dv) * 2
            mix_flops += 2.0 * H * (dk + dv) * T * (T + 1) / 2
            inner, N = s["heads"] * s["vdim"], s["state"]
            fixed += (2 * inner + 2 * s["groups"] * N + s["heads"]) * D + D * inner
            cache_bytes += batch * (s["heads"] * s["vdim"] * N + (s["conv"] - 1) * (inner + 2 * s["groups"] * N)) * 4
            mix_flops += 6.0 * s["heads"] * s["vdim"] * N * T             # the state's update and read-out
        else:
            HD, R = m["heads"] * m["dim"], max(8, D // 16)
            fixed += 4 * HD * D + R * D + HD * R + D * HD
            cache_bytes += batch * (m["heads"] * m["dim"] * m["dim"] + D) * 4
            mix_flops += 4.0 * m["heads"] * m["dim"] * m["dim"] * T       # the read-out S^T r and the update of S
        mlp = layer["mlp"]
        if mlp["kind"] == "dense":
            fixed += 3 * D * mlp["ff"]
            continue
        E, I, top, F = mlp["router"]["experts"], mlp["router"]["identity"], mlp["router"]["top"], mlp["expert"]["ff"]
        fixed += (E + I) * D
        expert_params += top * (E / (E + I)) * 2 * D * F                  # a choice is an expert with weights E times in E + I
        touched = E * (1.0 - (1.0 - 1.0 / (E + I)) ** (batch * top))      # expected distinct experts of a step
        expert_bytes += touched * 2 * D * F * 2
    return fixed * 2 + expert_bytes + cache_bytes, 2.0 * (fixed - V * D + expert_params) * T + 2.0 * V * D + mix_flops


def kimutar_config(width, heads, kv_heads, window, ff, experts, top, expert_ff, shared_ff, vocab):
    """Four layers with every kind of mixer and feed-forward: attention over a window that keeps four keys, with a sink,
    beside a dense feed-forward; the delta rule with a decay per channel beside experts; attention with two maps a head
    (half as many heads, so that the kernels see as many as in the first layer) beside experts; the delta rule again.  The
    last three layers are the repeated range, run once (as many layer runs as the design beside it has layers)."""
    moe = dict(kind="moe", router=dict(experts=experts, top=top, scale=2.0), expert=dict(ff=expert_ff), shared=dict(ff=shared_ff))
    delta = dict(type="channel_delta", mixer=dict(heads=heads, kv_heads=heads // 2, dim=128, vdim=128, conv=4, decay_rank=width // 16,
                                                  gate_rank=width // 16), mlp=moe)
    return dict(architecture="Kimutar", vocab=vocab, width=width, norm=dict(eps=1e-6), loop=dict(start=1, stop=4, times=1), layers=[
        dict(type="attention_2", mixer=dict(heads=heads, kv_heads=kv_heads, dim=128, vdim=128, scale=128 ** -0.5,
                                            rot=dict(base=500000.0, dims=128, scaling=dict(factor=8.0, low=1.0, high=4.0, original=8192)),
                                            mask=dict(size=window, keep_first=4)), mlp=dict(kind="dense", ff=ff)),
        delta,
        dict(type="attention", mixer=dict(heads=heads // 2, kv_heads=kv_heads // 2, dim=128, vdim=128, scale=128 ** -0.5, diff=0.3,
                                          rot=dict(base=500000.0, dims=64, scaling=dict(factor=2.0, original=8192, fast=32.0, slow=1.0))),
             mlp=moe),
        delta])


def kimutar_work(cfg, batch, context, T):
    """(bytes a decode step of `batch` sequences at `context` must read, FLOPs of a prompt of T tokens)."""
    D, V = cfg["width"], cfg["vocab"]
    fixed, cache_bytes, mix_flops, expert_bytes, expert_params = 2 * V * D, 0, 0.0, 0.0, 0        # the table and the head
    for layer in cfg["layers"]:
        m = layer["mixer"]
        H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        if layer["type"] == "attention_2":
            seen = m["mask"]["size"] + m["mask"]["keep_first"] if "mask" in m else 1 << 30
            fixed += (H * dk + G * dk + G * dv) * D + D * H * dv
            cache_bytes += batch * min(context, seen) * G * (dk + dv) * 2
            keys = sum(min(t + 1, seen) for t in range(T)) if T > 1 else 1
            mix_flops += 2.0 * H * (dk + dv) * keys
        elif layer["type"] == "attention":
            fixed += (2 * H * dk + 2 * G * dk + G * dv) * D + D * H * dv
            cache_bytes += batch * context * G * (2 * dk + dv) * 2            # two maps of keys, the values once
            mix_flops += 2.0 * 2 * H * (dk + dv) * T * (T + 1) / 2
        else:
            ra, rg = m["decay_rank"], m["gate_rank"]
            fixed += (2 * G * dk + H * dv + H + ra + rg) * D + H * dk * ra + H * dv * rg + D * H * dv
            cache_bytes += batch * H * dk * dv * 4                            # the state, 32-bit
            mix_flops += 6.0 * H * dk * dv * T
        mlp = layer["mlp"]
        if mlp["kind"] == "dense":
            fixed += 2 * D * mlp["ff"]
            continue
        E, top, F = mlp["router"]["experts"], mlp["router"]["top"], mlp["expert"]["ff"]
        fixed += (E + 1) * D + 3 * D * mlp["shared"]["ff"]
        expert_params += top * 3 * D * F
        touched = E * (1.0 - (1.0 - 1.0 / E) ** (batch * top))              # expected distinct experts of a step
        expert_bytes += touched * 3 * D * F * 2
    # (the table is read by rows, not as a whole)
    return (fixed - V * D) * 2 + expert_bytes + cache_bytes, 2.0 * (fixed - 2 * V * D + expert_params) * T + 2.0 * V * D + mix_flops


def kefetar_config(width, heads, kv_heads, ff, vocab):
    """Four layers with every kind of mixer, a dense feed-forward in each: retention; attention with convolved q, k and v, capped
    scores and an output gate, whose values lead the blended ones; retention; attention with blended values."""
    decay = [1.0 - 2.0 ** (-5.0 - 5.0 * h / heads) for h in range(heads)]
    ret = dict(type="retention", mixer=dict(heads=heads, dim=128, vdim=128, decay=decay, rot=dict(base=10000.0, dims=128)),
               mlp=dict(kind="dense", ff=ff))
    att = dict(type="attention", mixer=dict(heads=heads, kv_heads=kv_heads, dim=128, vdim=128, conv=4, scale=128 ** -0.5, softcap=50.0, v_mix=True,
                                            rot=dict(base=500000.0, dims=128, scaling=dict(factor=8.0))), mlp=dict(kind="dense", ff=ff))
    return dict(architecture="Kefetar", vocab=vocab, width=width, norm=dict(eps=1e-6), canon=dict(taps=4), layers=[ret, att, ret, att])


def kimutar_dense_config(width, heads, kv_heads, ff, vocab):
    """Kimutar's layers that are nearest to Kefetar's, at the same sizes and in the same order: the delta rule with a decay per
    channel, attention without a window, a dense feed-forward in each."""
    delta = dict(type="channel_delta", mixer=dict(heads=heads, kv_heads=heads, dim=128, vdim=128, conv=4, decay_rank=width // 16,
                                                  gate_rank=width // 16), mlp=dict(kind="dense", ff=ff))
    att = dict(type="attention_2", mixer=dict(heads=heads, kv_heads=kv_heads, dim=128, vdim=128, scale=128 ** -0.5,
                                              rot=dict(base=500000.0, dims=128, scaling=dict(factor=8.0, low=1.0, high=4.0, original=8192))),
               mlp=dict(kind="dense", ff=ff))
    return dict(architecture="Kimutar", vocab=vocab, width=width, norm=dict(eps=1e-6), layers=[delta, att, delta, att])


def kefetar_work(cfg, batch, context, T):
    """(bytes a decode step of `batch` sequences at `context` must read, FLOPs of a prompt of T tokens)."""
    D, V, taps = cfg["width"], cfg["vocab"], cfg["canon"]["taps"]
    fixed, cache_bytes, mix_flops = V * D, 0, 0.0                         # the head (the table is read by rows)
    for layer in cfg["layers"]:
        m = layer["mixer"]
        H, dk, dv = m["heads"], m["dim"], m["vdim"]
        if layer["type"] == "retention":
            fixed += (2 * H * dk + 2 * H * dv) * D + D * H * dv
            cache_bytes += batch * H * dk * dv * 4                        # the state, 32-bit
            mix_flops += 4.0 * H * dk * dv * T                            # the write k v^T and the read-out S^T q
        else:
            G = m["kv_heads"]
            fixed += (H * dk + G * dk + G * dv + H * dv) * D + D * H * dv
            cache_bytes += batch * context * G * (dk + dv) * 2 + batch * (m["conv"] - 1) * (H * dk + G * (dk + dv)) * 4
            mix_flops += 2.0 * H * (dk + dv) * T * (T + 1) / 2
        cache_bytes += batch * (taps - 1) * D * 4 * (2 if layer["mlp"] else 1)
        if layer["mlp"]:
            fixed += 2 * D * layer["mlp"]["ff"]
    return fixed * 2 + cache_bytes, 2.0 * (fixed - V * D) * T + 2.0 * V * D + mix_flops


def fobatar_config(width, heads, kv_heads, kv_rank, chunk, experts, top, expert_ff, vocab):
    """Four layers with both kinds of mixer, experts chosen by token id and a shared expert in each: attention over chunks with
    convolved and normed projections; latent attention with a rotated part; both again."""
    rot = lambda dims: dict(base=500000.0, dims=dims, scaling=dict(factor=8.0, original=4096, fast=32.0, slow=1.0))
    moe = dict(kind="moe", router=dict(experts=experts, top=top), expert=dict(ff=expert_ff, limit=7.0), shared=dict(ff=expert_ff, limit=7.0))
    att = dict(type="attention", mixer=dict(heads=heads, kv_heads=kv_heads, dim=128, vdim=128, conv=4, scale=128 ** -0.5, rot=rot(64),
                                            mask=dict(size=chunk)), mlp=moe)
    lat = dict(type="latent_attention", mixer=dict(heads=heads, dim=128, rot_dim=64, vdim=128, kv_rank=kv_rank, scale=192 ** -0.5,
                                                   rot=rot(64)), mlp=moe)
    return dict(architecture="Fobatar", vocab=vocab, width=width, embedding=dict(scale=4.0), norm=dict(eps=1e-6), residual_mult=0.5,
                layers=[att, lat, att, lat])


def porarax_attention_config(width, heads, kv_heads, kv_rank, chunk, experts, top, expert_ff, vocab):
    """Porarax's layers that are nearest to Fobatar's, at the same sizes and in the same order: attention, latent attention with a
    latent of its own (queries through a latent of a third of the width, a window wider than the prompt), experts in each."""
    moe = dict(kind="moe", router=dict(experts=experts, top=top), expert=dict(ff=expert_ff, limit=7.0))
    att = dict(type="attention", mixer=dict(heads=heads, kv_heads=kv_heads, dim=128, vdim=128, scale=128 ** -0.5,
                                            rot=dict(base=500000.0, dims=64)), mlp=moe)
    lat = dict(type="latent_attention", mixer=dict(heads=heads, dim=128, vdim=128, kv_rank=kv_rank, q_rank=width // 24 * 8,
                                                   scale=128 ** -0.5, mask=dict(size=1 << 20)), mlp=moe)
    return dict(architecture="Porarax", vocab=vocab, width=width, norm=dict(eps=1e-6), layers=[att, lat, att, lat])


def fobatar_work(cfg, batch, context, T):
    """(bytes a decode step of `batch` sequences at `context` must read, FLOPs of a prompt of T tokens)."""
    D, V = cfg["width"], cfg["vocab"]
    fixed, cache_bytes, mix_flops, expert_bytes, expert_params = V * D, 0, 0.0, 0.0, 0
    for layer in cfg["layers"]:
        m = layer["mixer"]
        H, dk, dv = m["heads"], m["dim"], m["vdim"]
        if layer["type"] == "attention":
            G, C = m["kv_heads"], m["mask"]["size"]
            fixed += (H * dk + G * dk + G * dv + H) * D + D * H * dv
            cache_bytes += batch * (context % C + 1) * G * (dk + dv) * 2 + batch * (m["conv"] - 1) * (H * dk + G * (dk + dv)) * 4
            mix_flops += 2.0 * H * (dk + dv) * sum(t % C + 1 for t in range(T))
        else:
            R, r = m["kv_rank"], m["rot_dim"]
            fixed += (H * (dk + r) + R + r + H) * D + H * (dk + dv) * R + D * H * dv
            cache_bytes += batch * context * (R + r) * 2
            mix_flops += 2.0 * H * (2 * R + r) * T * (T + 1) / 2           # scores and sums in the latent space
        mlp = layer["mlp"]
        E, top, F = mlp["router"]["experts"], mlp["router"]["top"], mlp["expert"]["ff"]
        fixed += 3 * D * mlp["shared"]["ff"]
        expert_params += top * 3 * D * F
        touched = E * (1.0 - (1.0 - top / E) ** batch)                      # expected distinct experts of a step
        expert_bytes += touched * 3 * D * F * 2
    return fixed * 2 + expert_bytes + cache_bytes, 2.0 * (fixed - V * D + expert_params) * T + 2.0 * V * D + mix_flops


def design_compare(args) -> int:
    """Another design beside the library's closest one at equal width and layer count (Turevik and Sogazen beside Falcon-H1,
    Porarax beside Turevik, Kimutar and Fobatar beside Porarax, Kefetar beside Kimutar): a prompt of --prefill-tokens tokens and decode steps at batch 8 and 64 from --prompt-len-token
    prompts, each as time and as a fraction of the measured peak for the bytes a step must read (decode) or the FLOPs a
    prompt needs (prefill)."""
    import torch
    import tinyllama_c_b200 as tlc
    pk = peaks()
    T, out = args.prefill_tokens, {}
    turevik = {"width 2048": turevik_config(2048, 16, 256, 4096, 32, 4, 1024, 1024, 4096, 65536),
               "width 3072": turevik_config(3072, 24, 256, 12288, 64, 6, 2048, 2048, 6144, 130048)}
    if args.design == "porarax":
        cases = {"width 2048": (porarax_config(2048, 16, 4, 256, 768, 1024, 32, 4, 1024, 65536), turevik["width 2048"]),
                 "width 3072": (porarax_config(3072, 24, 8, 256, 1024, 1024, 64, 6, 2048, 130048), turevik["width 3072"])}
        beside = "turevik"
    elif args.design == "kimutar":
        porarax = {"width 2048": porarax_config(2048, 16, 4, 256, 768, 1024, 32, 4, 1024, 65536),
                   "width 3072": porarax_config(3072, 24, 8, 256, 1024, 1024, 64, 6, 2048, 130048)}
        cases = {"width 2048": (kimutar_config(2048, 16, 4, 1024, 4096, 32, 4, 1024, 1024, 65536), porarax["width 2048"]),
                 "width 3072": (kimutar_config(3072, 24, 8, 1024, 12288, 64, 6, 2048, 2048, 130048), porarax["width 3072"])}
        beside = "porarax"
    elif args.design == "kefetar":
        sizes_of = {"width 2048": (2048, 16, 4, 4096, 65536), "width 3072": (3072, 24, 8, 12288, 130048)}
        cases = {k: (kefetar_config(*v), kimutar_dense_config(*v)) for k, v in sizes_of.items()}
        beside = "kimutar"
    elif args.design == "fobatar":
        sizes_of = {"width 2048": (2048, 16, 4, 256, 1024, 32, 4, 1024, 65536), "width 3072": (3072, 24, 8, 256, 1024, 64, 6, 2048, 130048)}
        cases = {k: (fobatar_config(*v), porarax_attention_config(*v)) for k, v in sizes_of.items()}
        beside = "porarax"
    elif args.design == "sogazen":
        cases = {"width 2048": (sogazen_config(2048, 8, 2, 48, 64, 256, 32, 4096, 32, 4, 4, 1024, 65536), dict(CONFIG_1P5B, num_hidden_layers=4)),
                 "width 3072": (sogazen_config(3072, 12, 2, 24, 128, 256, 48, 12288, 64, 8, 6, 2048, 130048), dict(CONFIG_7B, num_hidden_layers=4))}
        beside = "falcon_h1"
    else:
        cases = {"width 2048": (turevik["width 2048"], dict(CONFIG_1P5B, num_hidden_layers=4)),
                 "width 3072": (turevik["width 3072"], dict(CONFIG_7B, num_hidden_layers=4))}
        beside = "falcon_h1"
    work = {"turevik": turevik_work, "porarax": porarax_work, "sogazen": sogazen_work, "kimutar": kimutar_work,
            "kefetar": kefetar_work, "fobatar": fobatar_work}
    if args.sizes_only:
        cases = {k: v for k, v in cases.items() if k == args.sizes_only}
    for name, (tcfg, fcfg) in cases.items():
        for design, cfg in ((args.design, tcfg), (beside, fcfg)):
            model = tlc.random_model(cfg, seed=0, dtype="bfloat16")
            llm = tlc.LLM(model, max_tokens=64 * (args.prompt_len + 2 * args.steps + 128) + T, max_seqs=64)
            row = {}
            pms = time_prefill(llm, T, seed=3)
            ctx = args.prompt_len + args.steps // 2
            if design in work:
                flops = work[design](cfg, 1, 0, T)[1]
            else:
                flops = prefill_flops(cfg, T)
            row["prefill"] = {"tokens": T, "ms": round(pms, 3), "tok_s": round(T * 1000.0 / pms, 1),
                              "frac_of_measured_bf16": round(flops / (pms * 1e-3) / (pk["bf16_tflops"] * 1e12), 4)}
            for batch in (8, 64):
                ms, launches, clocks, ctx = time_decode(llm, tlc, batch, args.prompt_len, args.steps, args.warmup, seed=1)
                nbytes = work[design](cfg, batch, ctx, 1)[0] if design in work else decode_bytes(cfg, batch, ctx)
                row[f"decode_batch_{batch}"] = {"ms_per_step": round(ms, 4), "tok_s": round(batch * 1000.0 / ms, 1),
                                                "launches_per_step": launches // args.steps,
                                                "frac_of_measured_hbm": round(nbytes / (ms * 1e-3) / 1e9 / pk["hbm_gbs"], 4),
                                                "clocks": clocks}
            out.setdefault(name, {})[design] = row
            del llm, model
            torch.cuda.empty_cache()
    print(json.dumps({"design": args.design, "layers": 4, "dtype": "bf16", "data": "synthetic (random weights, uniform random token ids)",
                      "peaks": pk, "sizes": out}))
    return 0


def big_workloads(tlc, pk):
    """The workloads of the 3B and 7B layer sizes: 16 unequal prompts of 64..2,048 tokens with 256 tokens sampled
    for each at temperature 0.7 (3B); decode at batch 64 from 1,024-token prompts and one 8,192-token prompt (7B)."""
    import torch
    out = {}
    cfg = CONFIGS["3B"]
    llm = tlc.LLM(tlc.random_model(cfg, seed=0, dtype="bfloat16"), max_tokens=16 * (2048 + 256 + 64), max_seqs=16)
    g = time_generate(llm, tlc, 16, 64, 2048, 256, 0.7, seed=9)
    out["3b_generate_16_tok_s"] = g["tok_s"]
    out["3b_generate_16_wall_s"] = g["wall_s"]
    m, _, _, c = time_decode(llm, tlc, 16, 512, 16, 3, seed=41)
    out["3b_decode_b16"] = round(16 * 1000.0 / m, 1)
    out["3b_decode_b16_hbm_frac"] = round(decode_bytes(cfg, 16, c) / (m * 1e-3) / 1e9 / pk["hbm_gbs"], 4)
    del llm
    torch.cuda.empty_cache()
    cfg = CONFIGS["7B"]
    llm = tlc.LLM(tlc.random_model(cfg, seed=0, dtype="bfloat16"), max_tokens=64 * 1152, max_seqs=64)
    m, _, _, c = time_decode(llm, tlc, 64, 1024, 16, 3, seed=42)
    out["7b_decode_b64"] = round(64 * 1000.0 / m, 1)
    out["7b_decode_b64_hbm_frac"] = round(decode_bytes(cfg, 64, c) / (m * 1e-3) / 1e9 / pk["hbm_gbs"], 4)
    pms = time_prefill(llm, 8192, seed=43, reps=2)
    out["7b_prefill_8192_tok_s"] = round(8192 * 1000.0 / pms, 1)
    out["7b_prefill_8192_bf16_frac"] = round(prefill_flops(cfg, 8192) / (pms * 1e-3) / (pk["bf16_tflops"] * 1e12), 4)
    del llm
    torch.cuda.empty_cache()
    return out


def reference_arm(args) -> int:
    """The unmodified reference (its CPU engine, the only path it has for Falcon-H1) on the same layer sizes:
    decode at batch 1 after a prompt of --prompt-len tokens, and one prompt of --prefill-tokens tokens."""
    try:
        from baseline import reference_arm as ra
        cfg = dict(CONFIGS[args.sizes])
        steps, warmup = max(1, min(args.steps, 32)), max(3, min(args.warmup, 4))
        r = ra.measure(cfg, steps, warmup, args.prompt_len, args.prefill_tokens, budget_s=args.ref_budget,
                       layers=args.layers)
    except Exception as e:                                  # noqa: BLE001 -- any failure is reported, never raised
        msg = " ".join(str(e).split())[:300]
        print(json.dumps({"impl": "reference", "unavailable": f"the reference's CPU engine could not be built or run: {msg}"}))
        return 0
    s = sizes(cfg)
    tok_s = r["steps"] / r["decode_s"]
    rec = {
        "impl": "reference",
        "metric": f"decode tok/s at batch 1 (CodeClaper/tinyllama.c's CPU engine, {r['threads']} threads; Falcon-H1-"
                  f"{args.sizes} sizes, {args.prompt_len}-token prompt, context {cfg['max_position_embeddings']})",
        "value": round(tok_s, 3), "unit": "tok/s", "n_gpus": 0, "steps": r["steps"], "warmup": warmup,
        "ms_per_step": round(1000.0 * r["decode_s"] / r["steps"], 3), "higher_is_better": True, "scaling": "weak",
        "vs_baseline": None, "dtype": "bf16 weights, fp32 arithmetic (the reference's CPU path)",
        "data": "synthetic (random weights in a GGUF file, pseudo-random token ids)",
        "config": {"model": f"Falcon-H1-{args.sizes} sizes", "global_batch": 1, "seq_len": cfg["max_position_embeddings"],
                   "prompt_len": args.prompt_len, "parallelism": f"CPU, {r['threads']} threads", "layers": r["layers"],
                   "layers_full": r["layers_full"], "hidden": cfg["hidden_size"], "heads": f"{s['H']}q/{s['KV']}kv x{s['hd']}",
                   "intermediate": cfg["intermediate_size"], "vocab": cfg["vocab_size"],
                   "mamba": f"{s['Hs']} heads x{s['P']}, state {s['N']}, groups {s['G']}, conv {s['K']}",
                   "tied": cfg["tie_word_embeddings"], "gguf_gb": round(r["gguf_bytes"] / 1e9, 2)},
        "e2e": {"value": round(tok_s, 3), "unit": "tok/s", "h2d_bytes_per_step": 0, "d2h_bytes_per_step": 0,
                "note": "host token ids in and out is the reference's only interface; no device is involved"},
        "gpu_launches": 0,
    }
    if r["prefill_s"] > 0:
        rec["prefill"] = {"value": round(args.prefill_tokens / r["prefill_s"], 1), "tokens": args.prefill_tokens,
                          "ms": round(1000.0 * r["prefill_s"], 1)}
    print(json.dumps(rec))
    return 0


if __name__ == "__main__":
    sys.exit(main())
