"""bench.py --workload bezizen: prefill and decode throughput of the Bezizen layers (hyper-connected streams, learned positions, WKV time
mixing, window attention on convolved keys beside gated linear attention, experts chosen by softmax scores within groups;
leopard_b200/bezizen.py) at a few sizes that resemble a real model's layers, beside the framework's closest existing models on the same
step engine at the same width, window, expert sizes and vocabulary: the Zudalorn stack of benchmarks/seqlm_bench.py (retention as the like of
the matrix memories, experts) and the Komazen stack of benchmarks/komazen_bench.py (the same grouped-query attention and convolution
kernels, a post-norm kernel as the like of the hyper-connections).  Random weights, synthetic token ids, one GPU.

Per size: 4 layers [wkv, wkv, parallel, wkv], each with experts and a shared expert; four streams; wkv heads of 64, all others of 128;
  prefill   one request of `prompt` tokens per step through SeqLMEngine.step (cache and states written), tokens/s;
  decode    `batch` running requests with 512 tokens of history advanced by one token per step, tokens/s, for batch 1, 8 and 64;
  kernels   device time per native entry point of one prefill step and one decode step (CUDA events around every call) and the rate
            each reaches against its ceiling: the fp32 FMA peak for the attention kernel and the matrix memories (fp32 scores, states
            and sums), the measured copy bandwidth for the elementwise kernels, the states of a decode step and the weight-streaming
            decode products, the measured cuBLAS bf16 peak for the tcgen05 GEMM.  The like kernels of the other stacks stand beside them.
One JSON line in the shape bench.py prints for its other workloads; `value` is the prefill throughput of the middle size.
"""
from __future__ import annotations

import json

import torch

from benchmarks.komazen_bench import bench_komazen
from benchmarks.seqlm_bench import FP32_FMA_TFLOPS, HEAD, SIZES, TimedLib, _time, bench_size

STREAMS, WKV_HEAD, RANK, TAPS, POSITIONS = 4, 64, 64, 4, 8192
KINDS = ("wkv", "wkv", "parallel", "wkv")


def bezizen_config(s):
    H, G = s["heads"], max(s["heads"] // 4, 1)
    wkv = {"heads": H * HEAD // WKV_HEAD, "dim": WKV_HEAD}
    par = {"left": {"heads": H, "kv_heads": G, "dim": HEAD, "vdim": HEAD, "scale": HEAD ** -0.5, "conv": TAPS, "mask": {"size": s["window"]},
                    "q_temp": {"coef": 0.1, "every": 1024}},
           "right": {"heads": H, "dim": HEAD, "vdim": HEAD, "tau": 16.0}, "left_scale": 0.7, "right_scale": 0.7}
    moe = {"kind": "moe", "expert": {"ff": s["expert_ff"]}, "shared": {"ff": s["shared_ff"]},
           "router": {"experts": s["experts"], "top": s["top"], "scale": 2.0, "groups": {"count": 4, "keep": 2}}}
    return {"architecture": "Bezizen", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0},
            "streams": STREAMS, "max_positions": POSITIONS, "logit_scale": 1.0,
            "layers": [{"type": k, "mixer": wkv if k == "wkv" else par, "mlp": moe} for k in KINDS]}


def random_getter(cfg, dev, seed=1):
    g = torch.Generator(device=dev).manual_seed(seed)
    D, S = cfg["width"], cfg["streams"]
    shapes = {"embed": (cfg["vocab"], D), "pos": (cfg["max_positions"], D), "head": (cfg["vocab"], D), "final.norm": (D,)}
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer["mlp"]
        q = p + "mix."
        for n in "12":
            shapes.update({p + "norm" + n: (D,), f"{p}hc{n}.in": (S,), f"{p}hc{n}.out": (S,), f"{p}hc{n}.mix": (S, S)})
        if layer["type"] == "wkv":
            n = m["heads"] * m["dim"]
            shapes.update({q + "mu." + x: (D,) for x in "rkvgw"})
            shapes.update({q + x: (n, D) for x in "rkvg"})
            shapes.update({q + "w1": (RANK, D), q + "w2": (n, RANK), q + "w0": (n,), q + "u": (m["heads"], m["dim"]), q + "norm": (n,), q + "o": (D, n)})
        else:
            l, r = m["left"], m["right"]
            nq, nk, n, e = l["heads"] * l["dim"], l["kv_heads"] * l["dim"], r["heads"] * r["dim"], r["heads"] * r["vdim"]
            shapes.update({q + "left.q": (nq, D), q + "left.k": (nk, D), q + "left.q.conv": (nq, l["conv"]), q + "left.k.conv": (nk, l["conv"]),
                           q + "left.g": (nq, D), q + "left.o": (D, nq), q + "right.q": (n, D), q + "right.k": (n, D), q + "right.v": (e, D),
                           q + "right.g": (e, D), q + "right.o": (D, e), q + "right.norm": (r["vdim"],), q + "right.a1": (RANK, D),
                           q + "right.a2": (n, RANK), q + "right.a2.b": (n,)})
        shapes[p + "mlp.router"] = (f["router"]["experts"], D)
        for name, ff in [(f"e{e}", f["expert"]["ff"]) for e in range(f["router"]["experts"])] + [("shared", f["shared"]["ff"])]:
            shapes.update({f"{p}mlp.{name}.gate": (ff, D), f"{p}mlp.{name}.up": (ff, D), f"{p}mlp.{name}.down": (D, ff)})

    def get(name):
        shape = shapes[name]
        if name.endswith((".mix", ".u")) or len(shape) == 1:
            return (torch.rand(shape, device=dev, generator=g) * 0.5 + (0.0 if name.endswith(".mix") else 0.25)).to(torch.bfloat16)
        return (torch.randn(shape, device=dev, generator=g) * shape[1] ** -0.5).to(torch.bfloat16)
    return get


def bench_bezizen(name, s, dev, steps, warmup, peaks, prompt):
    from leopard_b200 import bezizen
    from leopard_b200.seqlm import SeqLMEngine, SeqLMWeights, StepEntry
    cfg_d = bezizen_config(s)
    cfg = bezizen.config_from_dict(cfg_d)
    eng = SeqLMEngine(cfg, SeqLMWeights(cfg, random_getter(cfg_d, dev), bezizen.tensor_name, dev), dtype="bfloat16",
                      max_tokens=64 * 600 + prompt, max_seqs=64)
    g = torch.Generator().manual_seed(0)
    toks = torch.randint(0, s["vocab"], (prompt,), generator=g).tolist()
    D, H, G, R, W = s["width"], s["heads"], max(s["heads"] // 4, 1), prompt, s["window"]
    hd, n_wkv = H * HEAD, KINDS.count("wkv")
    out = {"size": name, "width": D, "wkv_heads": hd // WKV_HEAD, "heads": H, "kv_heads": G, "window": W, "rank": RANK, "streams": STREAMS,
           **{k: s[k] for k in ("experts", "top", "expert_ff", "shared_ff")}, "prompt": prompt}

    def prefill():
        eng.step([StepEntry("p", toks, [prompt - 1])])
        eng.finish("p")
    ms = _time(prefill, steps, warmup)
    out["prefill_ms"], out["prefill_tokens_per_s"] = round(ms, 3), round(prompt / ms * 1e3, 1)
    plain = eng.L
    eng.L = TimedLib(plain)
    prefill()
    kp = eng.L.collect()
    out["prefill_gemm_shapes"] = [{"M": m, "N": n, "K": k, "ms": round(v[0], 4), "calls": v[1], "tflops": round(2.0 * m * n * k * v[1] / (v[0] * 1e-3) / 1e12, 1)}
                                  for (m, n, k), v in sorted(eng.L.gemm_shapes.items(), key=lambda kv: -kv[1][0])]
    eng.L = plain
    flops_gemm = sum(2.0 * x["M"] * x["N"] * x["K"] * x["calls"] for x in out["prefill_gemm_shapes"])
    attn_flops = H * sum(min(p + 1, W) for p in range(R)) * 4.0 * HEAD
    gla_flops = R * (n_wkv * hd * WKV_HEAD + hd * HEAD) * 4.0      # a multiply-add per state element for the update and one for the read-out
    n_sub = 2 * len(KINDS)
    # closing reads every copy and the result and writes every copy; opening writes the operand (fp32 ahead of the time mixing)
    hyper_bytes = R * D * (n_sub * (4.0 * STREAMS + 2.0) + n_wkv * 2.0 + n_sub * 4.0 * (1 + STREAMS) + 2.0)
    elem_bytes = {"lp_hyper_f32": hyper_bytes, "lp_token_shift_mix_f32": n_wkv * R * D * (4.0 + 5 * 2.0),
                  "lp_causal_conv_f32": R * (H + G) * HEAD * 8.0}

    def per_s(k, amount, unit):
        return round(amount / (k["ms"] * 1e-3) / unit, 2) if k and k["ms"] > 0 else None
    r = {}
    for key, flops in (("lp_gemm_bf16", flops_gemm), ("lp_window_attn_tiles", attn_flops), ("lp_gla", gla_flops)):
        r[key + "_tflops"] = per_s(kp.get(key), flops, 1e12)
    if r["lp_gemm_bf16_tflops"]:
        r["lp_gemm_bf16_of_bf16_peak"] = round(r["lp_gemm_bf16_tflops"] / peaks["bf16_burst"], 3)
    for k in ("lp_window_attn_tiles", "lp_gla"):
        if r[k + "_tflops"]:
            r[k + "_of_fp32_fma_peak"] = round(r[k + "_tflops"] / FP32_FMA_TFLOPS, 3)
    for k, nbytes in elem_bytes.items():
        v = per_s(kp.get(k), nbytes, 1e9)
        if v:
            r[k + "_gbs"], r[k + "_of_copy_peak"] = v, round(v / peaks["hbm_gbs"], 3)
    out["prefill_kernels"], out["prefill_rates"] = kp, r
    out["decode"] = {}
    for batch in (1, 8, 64):
        keys_ = [("d", i) for i in range(batch)]
        eng.step([StepEntry(k, toks[:512], []) for k in keys_])
        nxt = [int(t) for t in torch.randint(0, s["vocab"], (batch,), generator=g)]

        def decode():
            eng.step([StepEntry(k, [t], [0]) for k, t in zip(keys_, nxt)])
        ms = _time(decode, steps, warmup)
        d = {"ms_per_step": round(ms, 3), "tokens_per_s": round(batch / ms * 1e3, 1)}
        eng.L, eng.use_graphs = TimedLib(plain), False      # the breakdown needs the launches one by one
        decode()
        kd = eng.L.collect()
        eng.L, eng.use_graphs = plain, True
        d["kernels"] = kd
        # every weight matrix outside the experts is streamed once per step, the head included
        wbytes = 2.0 * (n_wkv * D * (5 * hd + 2 * RANK) + D * (2 * hd + G * HEAD + 4 * hd + RANK) + D * 2 * hd + len(KINDS) * 3 * D * s["shared_ff"]
                        + D * s["vocab"])
        if "lp_linear" in kd and batch <= 8:
            d["lp_linear_gbs"] = per_s(kd["lp_linear"], wbytes, 1e9)
            d["lp_linear_of_copy_peak"] = round(d["lp_linear_gbs"] / peaks["hbm_gbs"], 3)
        # states read and written once, and the second factor of every decay
        gla_bytes = batch * 8.0 * (n_wkv * hd * WKV_HEAD + hd * HEAD) + 2.0 * len(KINDS) * hd * RANK
        d["lp_gla_gbs"] = per_s(kd.get("lp_gla"), gla_bytes, 1e9)
        d["lp_gla_of_copy_peak"] = round(d["lp_gla_gbs"] / peaks["hbm_gbs"], 3)
        if "lp_window_attn" in kd:      # the cached rows are keys and values at once
            d["lp_window_attn_gbs"] = per_s(kd["lp_window_attn"], batch * 4.0 * G * HEAD * min(W, 513), 1e9)
        out["decode"][str(batch)] = d
        for k in keys_:
            eng.finish(k)
    del eng
    torch.cuda.empty_cache()
    return out


def run(args):
    import bench
    if args.impl == "reference":
        print(json.dumps({"impl": "reference", "unavailable": "the reference has no model of this kind; the comparison arms of this workload "
                                                              "are the framework's own Zudalorn and Komazen stacks"}), flush=True)
        return 0
    if not torch.cuda.is_available():
        raise SystemExit("bench.py needs a CUDA device: leopard_b200 has no CPU fallback")
    dev = torch.device("cuda", 0)
    torch.cuda.set_device(dev)
    peaks = bench.load_peaks()
    from leopard_b200 import _lib
    L = _lib.stream32_lib()
    n0 = L.lp_launch_count()
    only = [x for x in (getattr(args, "seqlm_sizes", None) or "").split(",") if x]
    prompt, sizes, zudalorn, komazen = 4096, [], [], []
    warmup = max(args.warmup, 3)
    keep = ("size", "prefill_ms", "prefill_tokens_per_s", "prefill_kernels", "prefill_rates", "decode")
    for name, s in SIZES.items():
        if only and name not in only:
            continue
        sizes.append(bench_bezizen(name, s, dev, args.steps, warmup, peaks, prompt))
        for rows, other in ((zudalorn, bench_size), (komazen, bench_komazen)):
            o = other(name, s, dev, args.steps, warmup, peaks, prompt)
            rows.append({k: o[k] for k in keep})
    mid = sizes[min(1, len(sizes) - 1)]
    line = {"metric": "bezizen_prefill_tokens_per_s", "value": mid["prefill_tokens_per_s"], "unit": "tokens/s", "n_gpus": 1,
            "steps": args.steps, "warmup": warmup, "ms_per_step": mid["prefill_ms"], "higher_is_better": True,
            "scaling": "weak", "vs_baseline": None, "dtype": "bf16", "data": "synthetic (random weights, random token ids)",
            "config": {"model": f"Bezizen 4-layer stack, {mid['size']}", "global_batch": 1, "seq_len": prompt,
                       "parallelism": "single GPU", "cache_policy": "weights + activations of a step exceed L2 at every size"},
            "gpu_launches": int(L.lp_launch_count() - n0), "peaks": peaks, "fp32_fma_peak_tflops": round(FP32_FMA_TFLOPS, 1),
            "sizes": sizes, "zudalorn_stack": zudalorn, "komazen_stack": komazen}
    print(json.dumps(line), flush=True)
    return 0
