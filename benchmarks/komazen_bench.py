"""bench.py --workload komazen: prefill and decode throughput of the Komazen layers (sliding-window latent attention with query latents, a
layer on another one's latents, an elementwise output gate; causal grouped-query attention with a temperature and a logarithmic
distance bias per head; gelu-gated units; norms after the sum; causal input convolutions; leopard_b200/komazen.py) at a few sizes that
resemble a real model's layers, beside the framework's closest existing models on the same step engine at the same width, head count and
vocabulary: the Zudalorn stack of benchmarks/seqlm_bench.py (the same latent attention kernels, dense units, experts) and the Kamosun
stack of benchmarks/kamosun_bench.py (the same grouped-query attention kernels, elementwise kernels around the stream).  Random weights,
synthetic token ids, one GPU.

Per size: 4 layers [latent + dense, latent on the first layer's latents + dense, attention + dense, attention + dense];
  prefill   one request of `prompt` tokens per step through SeqLMEngine.step (cache and carried inputs written), tokens/s;
  decode    `batch` running requests with 512 tokens of history advanced by one token per step, tokens/s, for batch 1, 8 and 64;
  kernels   device time per native entry point of one prefill step and one decode step (CUDA events around every call) and the rate
            each reaches against its ceiling: the fp32 FMA peak for the attention kernels and the per-head latent products (fp32
            scores and sums), the measured copy bandwidth for the elementwise kernels and the weight-streaming decode products, the
            measured cuBLAS bf16 peak for the tcgen05 GEMM.  The like kernels of the other stacks stand beside them.
One JSON line in the shape bench.py prints for its other workloads; `value` is the prefill throughput of the middle size.
"""
from __future__ import annotations

import json

import torch

from benchmarks.kamosun_bench import bench_kamosun
from benchmarks.seqlm_bench import FP32_FMA_TFLOPS, HEAD, SIZES, TimedLib, _time, bench_size

LAYERS, ROT, TAPS = 4, 64, 4


def _q_rank(s):
    return s["width"] // 2


def komazen_config(s):
    H, G = s["heads"], max(s["heads"] // 4, 1)
    lat = {"heads": H, "dim": HEAD, "rot_dim": ROT, "vdim": HEAD, "q_rank": _q_rank(s), "kv_rank": s["kv_rank"], "scale": (HEAD + ROT) ** -0.5,
           "rot": {"base": 5e4, "dims": ROT}, "mask": {"size": s["window"]}}
    att = {"heads": H, "kv_heads": G, "dim": HEAD, "vdim": HEAD, "scale": HEAD ** -0.5}
    dense = {"kind": "dense", "ff": s["ff"]}
    layers = [{"type": "latent_attention", "mixer": lat, "mlp": dense}, {"type": "latent_attention", "mixer": dict(lat, kv_from=0), "mlp": dense},
              {"type": "attention", "mixer": att, "mlp": dense}, {"type": "attention", "mixer": att, "mlp": dense}]
    return {"architecture": "Komazen", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0},
            "postln_alpha": 2.0, "canon": {"taps": TAPS}, "layers": layers}


def random_getter(cfg, dev, seed=1):
    g = torch.Generator(device=dev).manual_seed(seed)
    D = cfg["width"]
    shapes = {"embed": (cfg["vocab"], D), "head": (cfg["vocab"], D), "final.norm": (D,)}
    for i, layer in enumerate(cfg["layers"]):
        p, m, ff = f"l{i}.", layer["mixer"], layer["mlp"]["ff"]
        H, d, e = m["heads"], m["dim"], m["vdim"]
        shapes.update({p + "norm1": (D,), p + "norm2": (D,), p + "canon1": (D, cfg["canon"]["taps"]), p + "canon2": (D, cfg["canon"]["taps"]),
                       p + "mix.o": (D, H * e), p + "mlp.gate": (ff, D), p + "mlp.up": (ff, D), p + "mlp.down": (D, ff)})
        q = p + "mix."
        if layer["type"] == "latent_attention":
            r, c = m["q_rank"], m["kv_rank"]
            shapes.update({q + "dq": (r, D), q + "dq.norm": (r,), q + "uq": (H * (d + m["rot_dim"]), r), q + "uk": (H * d, c),
                           q + "uv": (H * e, c), q + "g": (H * e, D)})
            if m.get("kv_from") is None:
                shapes.update({q + "dkv": (c + m["rot_dim"], D), q + "dkv.norm": (c,)})
        else:
            G = m["kv_heads"]
            shapes.update({q + "q": (H * d, D), q + "k": (G * d, D), q + "v": (G * e, D), q + "q.norm": (d,), q + "k.norm": (d,),
                           q + "temp": (H,), q + "r1": (H,), q + "r2": (H,)})

    def get(name):
        shape = shapes[name]
        if len(shape) == 2:
            return (torch.randn(shape, device=dev, generator=g) * shape[1] ** -0.5).to(torch.bfloat16)
        return (torch.rand(shape, device=dev, generator=g) * 0.5 + 0.75).to(torch.bfloat16)
    return get


def bench_komazen(name, s, dev, steps, warmup, peaks, prompt):
    from leopard_b200 import komazen
    from leopard_b200.seqlm import SeqLMEngine, SeqLMWeights, StepEntry
    cfg_d = komazen_config(s)
    cfg = komazen.config_from_dict(cfg_d)
    eng = SeqLMEngine(cfg, SeqLMWeights(cfg, random_getter(cfg_d, dev), komazen.tensor_name, dev), dtype="bfloat16",
                      max_tokens=64 * 600 + prompt, max_seqs=64)
    g = torch.Generator().manual_seed(0)
    toks = torch.randint(0, s["vocab"], (prompt,), generator=g).tolist()
    D, H, G, R, W, C, Q, F = s["width"], s["heads"], max(s["heads"] // 4, 1), prompt, s["window"], s["kv_rank"], _q_rank(s), s["ff"]
    hd = H * HEAD
    out = {"size": name, "width": D, "heads": H, "kv_heads": G, "window": W, "q_rank": Q, "kv_rank": C, "ff": F, "taps": TAPS, "prompt": prompt}

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
    lat_keys = sum(min(p + 1, W) for p in range(R))
    lat_flops = 2 * H * lat_keys * (2.0 * (C + ROT) + 2.0 * C)
    head_flops = 2 * 2 * 2.0 * R * H * HEAD * C              # the per-head products around the latent attention of two layers
    attn_flops = 2 * H * (R * (R + 1) / 2) * 4.0 * HEAD
    n_sub = 2 * LAYERS
    elem_bytes = {"lp_post_norm_f32": n_sub * R * D * 12.0, "lp_causal_conv_f32": n_sub * R * D * 6.0,
                  "lp_glu_scaled_f32": LAYERS * R * F * (8.0 + 2.0)}

    def per_s(k, amount, unit):
        return round(amount / (k["ms"] * 1e-3) / unit, 2) if k and k["ms"] > 0 else None
    r = {}
    for key, flops in (("lp_gemm_bf16", flops_gemm), ("lp_window_attn_tiles", attn_flops), ("lp_latent_attend_tiles", lat_flops)):
        r[key + "_tflops"] = per_s(kp.get(key), flops, 1e12)
    heads_key = "lp_linear_heads" if "lp_linear_heads" in kp else "lp_linear"
    r["per_head_products_tflops"] = per_s(kp.get(heads_key), head_flops, 1e12)
    if r["lp_gemm_bf16_tflops"]:
        r["lp_gemm_bf16_of_bf16_peak"] = round(r["lp_gemm_bf16_tflops"] / peaks["bf16_burst"], 3)
    for k in ("lp_window_attn_tiles", "lp_latent_attend_tiles", "per_head_products"):
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
        if batch in (1, 8):
            eng.L, eng.use_graphs = TimedLib(plain), False      # the breakdown needs the launches one by one
            decode()
            kd = eng.L.collect()
            eng.L, eng.use_graphs = plain, True
            d["kernels"] = kd
            # every weight matrix is streamed once per step, the head included
            wbytes = 2.0 * (D * (2 * Q + C + ROT + 2 * hd) + 2 * Q * H * (HEAD + ROT) + 4 * hd * C + D * 2 * (hd + 2 * G * HEAD) + LAYERS * D * hd +
                            LAYERS * 3 * D * F + D * s["vocab"])
            if "lp_linear" in kd:
                d["lp_linear_gbs"] = per_s(kd["lp_linear"], wbytes, 1e9)
                d["lp_linear_of_copy_peak"] = round(d["lp_linear_gbs"] / peaks["hbm_gbs"], 3)
            if "lp_window_attn" in kd:      # keys and values every attention kernel walks
                d["lp_window_attn_gbs"] = per_s(kd["lp_window_attn"], batch * 2 * 4.0 * 2 * G * HEAD * 513, 1e9)
            if "lp_latent_attend" in kd:
                d["lp_latent_attend_gbs"] = per_s(kd["lp_latent_attend"], batch * 2 * 4.0 * (C + ROT) * min(W, 513), 1e9)
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
                                                              "are the framework's own Zudalorn and Kamosun stacks"}), flush=True)
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
    prompt, sizes, zudalorn, kamosun = 4096, [], [], []
    warmup = max(args.warmup, 3)
    keep = ("size", "prefill_ms", "prefill_tokens_per_s", "prefill_kernels", "prefill_rates", "decode")
    for name, s in SIZES.items():
        if only and name not in only:
            continue
        sizes.append(bench_komazen(name, s, dev, args.steps, warmup, peaks, prompt))
        for rows, other in ((zudalorn, bench_size), (kamosun, bench_kamosun)):
            o = other(name, s, dev, args.steps, warmup, peaks, prompt)
            rows.append({k: o[k] for k in keep})
    mid = sizes[min(1, len(sizes) - 1)]
    line = {"metric": "komazen_prefill_tokens_per_s", "value": mid["prefill_tokens_per_s"], "unit": "tokens/s", "n_gpus": 1,
            "steps": args.steps, "warmup": warmup, "ms_per_step": mid["prefill_ms"], "higher_is_better": True,
            "scaling": "weak", "vs_baseline": None, "dtype": "bf16", "data": "synthetic (random weights, random token ids)",
            "config": {"model": f"Komazen 4-layer stack, {mid['size']}", "global_batch": 1, "seq_len": prompt,
                       "parallelism": "single GPU", "cache_policy": "weights + activations of a step exceed L2 at every size"},
            "gpu_launches": int(L.lp_launch_count() - n0), "peaks": peaks, "fp32_fma_peak_tflops": round(FP32_FMA_TFLOPS, 1),
            "sizes": sizes, "zudalorn_stack": zudalorn, "kamosun_stack": kamosun}
    print(json.dumps(line), flush=True)
    return 0
