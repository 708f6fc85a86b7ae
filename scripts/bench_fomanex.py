"""Prefill and decode throughput of Fomanex next to Setirax and Vemepel, the framework's closest models (latent attention with sinks and gated
linear attention; latent attention with a rotated key part and routed experts), at equal layer sizes (`bench.py --arch fomanex`); `--arms`
also takes lududra, whose delta rule and experts it shares.

The models are random-init at shapes that resemble a real model's layers, keep bfloat16 weights and run through the same
`SequenceSession`.  Per arm: tokens / s end to end through the session (host control words, token ids and logits cross PCIe
every step) and device-only (the step's CUDA graph replayed with inputs resident), the HBM bytes a decoded token must move
(active weights + the caches and states it reads and writes) as a fraction of the measured copy bandwidth, and the prefill's
matmul FLOPs as a fraction of the measured dense bf16 throughput.
Timing: wall clock around synchronised replays, after warm-up.
"""
import json
import os
import sys

import numpy as np

HERE = os.path.dirname(os.path.abspath(__file__))
ROOT = os.path.dirname(HERE)
for d in (ROOT, HERE):
    if d not in sys.path:
        sys.path.insert(0, d)

from bench_lududra import SIZES as LUDUDRA_SIZES, lududra_arm, peaks, timed  # noqa: E402
from bench_setirax import SIZES as SETIRAX_SIZES, setirax_arm  # noqa: E402
from bench_vemepel import SIZES as VEMEPEL_SIZES, vemepel_arm  # noqa: E402

SIZES = {n: dict(width=s["width"], n_layers=s["n_layers"], heads=s["heads"], dim=s["dim"], experts=s["experts"], top=s["top"], ff=s["ff"], vocab=s["vocab"])
         for n, s in LUDUDRA_SIZES.items()}


def fomanex_arm(be, size, prefill_T, context, reps):
    from zgml_b200.host.fomanex import FomanexConfig, FomanexModel, synthetic_config, synthetic_tensors
    from zgml_b200.host.latent import expands
    from zgml_b200.host.session import SequenceSession
    cfgd = synthetic_config(**size)
    cfg = FomanexConfig.from_dict(cfgd)
    model = FomanexModel(be, cfg, synthetic_tensors(cfgd), "bfloat16")
    s = SequenceSession(be, model, n_slots=1, max_chunk=prefill_T, max_context=context + 1024)
    prompt = np.random.default_rng(0).integers(0, cfg.vocab, context).tolist()
    D = cfg.width
    active = state = 0           # weights / cache and state elements one decoded token touches
    attn_flops = walk_flops = 0  # f32 work of the prefill chunk that is not a matmul
    for i in cfg.runs:
        L, meta = cfg.layers[i], model.layer_meta[i]
        m, mlp = L["mixer"], L["mlp"]
        H, d = m["heads"], m["dim"]
        active += meta["n_in"] * D
        if L["type"] == "wkv":
            active += meta["C"] * (meta["rank"] + D)
            state += 2 * H * d * d
            walk_flops += 5 * H * d * d * prefill_T
        else:
            rd, dv, rank = m["rot_dim"], m["vdim"], m["kv_rank"]
            active += H * (d + dv) * rank + D * H * dv
            state += context * (rank + rd)
            per_key = d + rd + dv if expands(prefill_T, rank, rd, d, dv, model.wdt) else 2 * rank + rd
            attn_flops += 2 * H * per_key * prefill_T * prefill_T // 2
        active += 3 * D * meta["ff"] if mlp["kind"] == "dense" else meta["E"] * D + meta["top"] * 3 * D * meta["ff"]
    body = active
    active += cfg.vocab * D
    out = {"weights_gb": round(model.weight_bytes() / 1e9, 3), "active_params_per_token": active, "layers": [cfg.layers[i]["type"] for i in cfg.runs]}
    toks = prompt[:prefill_T]
    e2e = timed(lambda: (s.feed("p", toks, [prefill_T - 1]), s.release("p")), be.sync, reps)
    handle = s.program(prefill_T, "last")[1]
    dev = timed(lambda: be.lib.zg_cuda_execute_device(be.ctx, handle.ptr), be.sync, reps)
    out["prefill"] = {"tokens": prefill_T, "tok_s_e2e": round(prefill_T / e2e), "tok_s_device": round(prefill_T / dev), "ms_device": round(dev * 1e3, 3),
                      "matmul_tflops_device": round(2.0 * (body * prefill_T + cfg.vocab * D) / dev / 1e12, 1), "attention_gflop_f32": round(attn_flops / 1e9, 1),
                      "walk_gflop_f32": round(walk_flops / 1e9, 1), "kernels": be.program_stats(handle)["kernels"],
                      "tensor_core_linears": be.program_stats(handle)["tensor_core_linears"]}
    s.feed("d", prompt, [])
    tok = [1]
    e2e = timed(lambda: s.feed("d", tok, [0]), be.sync, 4 * reps)
    s.release("d")
    s.feed("d", prompt, [])
    handle = s.program(1, "last")[1]
    dev = timed(lambda: be.lib.zg_cuda_execute_device(be.ctx, handle.ptr), be.sync, 4 * reps)   # replays rewrite position `context`: same work every time
    bytes_tok = 2 * active + 4 * state
    out["decode"] = {"context": context, "tok_s_e2e": round(1 / e2e, 1), "tok_s_device": round(1 / dev, 1), "us_device": round(dev * 1e6, 1),
                     "bytes_per_token": bytes_tok, "hbm_gbs_device": round(bytes_tok / dev / 1e9, 1), "kernels": be.program_stats(handle)["kernels"]}
    out["dense_gemm_timeouts"] = be.program_stats(handle)["dense_gemm_timeouts"]
    s.close()
    model.close()
    return out


def run(args):
    from zgml_b200 import CudaBackend
    hbm, tf, how = peaks()
    be = CudaBackend(0)
    names = [n for n in (args.sizes.split(",") if args.sizes else SIZES)]
    res = {"bench": "fomanex_vs_setirax_vemepel", "peaks": {"hbm_gbs": hbm, "bf16_tflops": tf, "source": how}, "data": "synthetic random-init", "sizes": {}}
    chosen = (getattr(args, "arms", "") or "fomanex,setirax,vemepel").split(",")
    for n in names:
        entry = {"shape": SIZES[n]}
        for arm, fn, sizes in (("fomanex", fomanex_arm, SIZES), ("setirax", setirax_arm, SETIRAX_SIZES), ("vemepel", vemepel_arm, VEMEPEL_SIZES), ("lududra", lududra_arm, LUDUDRA_SIZES)):
            if arm not in chosen:
                continue
            try:
                e = fn(be, sizes[n], args.prefill_tokens, args.context, args.steps)
                e["decode"]["frac_of_hbm"] = round(e["decode"]["hbm_gbs_device"] / hbm, 3)
                e["prefill"]["frac_of_bf16"] = round(e["prefill"]["matmul_tflops_device"] / tf, 3)
                entry[arm] = e
            except Exception as ex:   # one arm failing must not hide the other
                entry[arm] = {"error": repr(ex)}
        res["sizes"][n] = entry
    res["gpu_launches"] = be.launch_count()
    be.close()
    print(json.dumps(res))
