"""Prefill and decode throughput of layer-planned models beside other models of equal width and depth (random weights).

    python bench.py --workload rokivik                     # both sizes, prompts and decoding, one JSON line each
    python bench.py --workload pesanex
    python benchmarks/bench_hybrid.py --design pesanex --kernels   # also per-kernel device times and roofline fractions

Sizes are those of real models' layers: width 2048 (beside Qwen3-1.7B) and width 4096 (beside Qwen3-8B), six layers of each.
Rokivik: Mamba-2, latent attention (windowed), Mamba-2, latent attention reading the first one's latents, Mamba-2, latent attention
over the whole context. Pesanex: softmax attention beside gated linear attention, retention, gated linear attention, and these three
again, every layer with a feed-forward; it stands beside Rokivik (the like recurrence) and Qwen3 (the like attention). Prompts are timed around the model's forward pass over staged inputs, decoding around the engine's own
step (captured graph), both with CUDA events after warm-up; the weights of a pass are several times the L2 (so is the cache
at the larger batches), nothing else is flushed. Each line carries SM clocks sampled during its timed region.
"""
from __future__ import annotations

import argparse
import copy
import json
import os
import re
import sys

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, ROOT)
sys.path.insert(0, os.path.join(ROOT, "benchmarks"))

import torch

SIZES = {
    "2048": dict(width=2048, ff=6144, heads=16, q_rank=768, kv_rank=512, mheads=64, groups=1, side=256, vocab=32768, like="qwen3-1.7B"),
    "4096": dict(width=4096, ff=12288, heads=32, q_rank=1536, kv_rank=512, mheads=128, groups=8, side=256, vocab=32768, like="qwen3-8B"),
}
MODELS = {"rokivik": ("rokivik", "qwen3"), "pesanex": ("pesanex", "rokivik", "qwen3")}
# Pesanex: heads of 128 (as many as fill the width); decay rank 16
KV_HEADS, GLA_DIM, HEAD = 8, 64, 128


WINDOW = 2048


def rokivik_config(s: dict, window: int = WINDOW) -> dict:
    def mamba():
        return {"type": "mamba2", "mixer": {"heads": s["mheads"], "vdim": 64, "state": 128, "groups": s["groups"], "conv": 4,
                                            "norm_groups": s["groups"]}, "mlp": {"kind": "dense", "ff": s["ff"]}}

    def latent(size, src=None):
        m = {"heads": s["heads"], "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": s["kv_rank"], "q_rank": s["q_rank"],
             "scale": 192 ** -0.5, "mask": {"size": size}, "rot": {"base": 10000.0, "dims": 64}}
        if src is not None:
            m["kv_from"] = src
        return {"type": "latent_attention", "mixer": m, "mlp": {"kind": "dense", "ff": s["ff"]}}

    return {"architecture": "Rokivik", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-6}, "token_side": {"dim": s["side"]},
            "layers": [mamba(), latent(window), mamba(), latent(window, 1), mamba(), latent(1 << 20)]}


def pesanex_config(s: dict) -> dict:
    h, mlp = s["heads"], {"kind": "dense", "ff": s["ff"]}
    gla = {"heads": h, "dim": GLA_DIM, "vdim": HEAD, "tau": 16.0}
    both = {"type": "parallel", "mixer": {"left": {"heads": h, "kv_heads": KV_HEADS, "dim": HEAD, "vdim": HEAD, "scale": HEAD ** 0.5 / 8,
                                                   "rot": {"base": 10000.0, "dims": 64}}, "right": gla}, "mlp": mlp}
    keep = {"type": "retention", "mixer": {"heads": h, "dim": HEAD, "vdim": HEAD, "decay": [1 - 2.0 ** -(5 + 7 * k / h) for k in range(h)],
                                           "rot": {"base": 10000.0, "dims": HEAD}}, "mlp": mlp}
    return {"architecture": "Pesanex", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-6}, "loop": {"start": 0, "stop": 0, "times": 1},
            "layers": [both, keep, {"type": "gla", "mixer": gla, "mlp": mlp}] * 2}


def peaks() -> dict:
    try:
        return json.load(open(os.path.join(ROOT, "MEASURED_PEAKS.json")))
    except Exception:  # noqa: BLE001
        return {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "fallback": True}


def build(kind: str, size: str, max_running: int, max_len: int, max_prefill: int):
    from miles_b200.engine import Engine
    from miles_b200.models import ModelConfig, ParamStore, build_model, get_config

    s = SIZES[size]
    if kind != "qwen3":
        cfg = ModelConfig.from_hf_config({"rokivik": rokivik_config, "pesanex": pesanex_config}[kind](s), name=f"{kind}-{size}")
    else:
        cfg = copy.copy(get_config(s["like"]))
        cfg.num_layers, cfg.vocab_size, cfg.tie_embeddings = 6, s["vocab"], False
    store = ParamStore(cfg, "cuda", torch.bfloat16)
    model = build_model(cfg, store)
    pages = max_running * ((max_len + 63) // 64 + 1) + 2
    return cfg, model, Engine(model, max_running=max_running, page_size=64, num_pages=pages, max_seq_len=max_len, max_prefill_tokens=max_prefill)


def prefill_pass(eng, model, cfg, lens: list):
    g = torch.Generator().manual_seed(0)
    parts, pages = [], []
    for i, n in enumerate(lens):
        pg = eng._alloc((n + 63) // 64)
        pages += pg
        parts.append((torch.randint(0, cfg.vocab_size, (n,), generator=g).tolist(), 0, list(pg), i))
    tokens, pos, cu, cu_t, meta = eng._stage_rows(parts)
    eng.pool.release(pages)
    return lambda: model.forward_hidden(tokens, pos, cu_t, meta=meta, kv_cache=eng.kv_cache, max_seqlen=max(lens))


def timed(fn, steps: int, warmup: int):
    from clocks import ClockSampler

    for _ in range(max(3, warmup)):
        fn()
    torch.cuda.synchronize()
    sampler = ClockSampler(torch.cuda.current_device())
    sampler.start()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    for _ in range(steps):
        fn()
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) / steps, sampler.stop()


def kernel_table(fn, steps: int = 5) -> dict:
    """Mean device microseconds and launches per pass of every kernel, by short name."""
    from torch.profiler import ProfilerActivity, profile

    fn()
    torch.cuda.synchronize()
    with profile(activities=[ProfilerActivity.CUDA]) as prof:
        for _ in range(steps):
            fn()
        torch.cuda.synchronize()
    out: dict = {}
    for ev in prof.events():
        if str(ev.device_type).endswith("CUDA"):
            name = re.sub(r"\(.*", "", re.sub(r"\((int|bool)\)", "", ev.name.replace("(anonymous namespace)::", "").replace("void ", "").replace("mb::", "")))[:70]
            t = out.setdefault(name, [0.0, 0])
            t[0] += ev.device_time_total if hasattr(ev, "device_time_total") else ev.cuda_time_total
            t[1] += 1
    return {k: (v[0] / v[1], v[1] / steps) for k, v in sorted(out.items(), key=lambda kv: -kv[1][0])}


def floors(cfg, kind: str, s: dict, T: int, ctx: int, prefill: bool) -> dict:
    """Per launch (bytes, flops) of the mixers' kernels, matched by kernel name; products are left out (they are the
    framework's GEMM and few-row kernels in both models)."""
    H, hd, P, N, G = s["width"], s["mheads"], 64, 128, s["groups"]
    inner, ch = hd * P, hd * P + 2 * G * N
    f = {}
    if kind == "rokivik":
        # (mean over the three attention layers: two windows and one whole context)
        R, W, h = 512, 576, s["heads"]
        seen = [min(i, WINDOW) for i in range(1, ctx + 1)]
        L = (2 * sum(seen) + sum(range(1, ctx + 1))) / 3 if prefill else (2 * seen[-1] + ctx) / 3
        if prefill:
            n = T // ctx
            c = 128
            chunks = n * ((ctx + c - 1) // c)
            st = chunks * hd * P * N * 4
            f["conv4_vec"] = (T * ch * 2 * 2, 0)
            f["chunk_state"] = (T * (inner + G * N) * 2 + st, 2 * T * hd * P * N)
            f["chunk_pass"] = (2 * st, 0)  # (fp32 in, two bf16 planes out)
            f["chunk_out"] = (T * (2 * inner + 2 * G * N) * 2 + st, 2 * T * hd * (P * N + (c + 1) / 2 * (N + P)))
            f["mamba_tail"] = (T * (3 * inner + 3 * s["ff"]) * 2, 0)
            f["latent_in"] = (T * (2 * (s["q_rank"] + W) + 3 * s["ff"]) * 2, 0)
            f["cached_prefill"] = (T * h * (192 + 128 + 256) * 2 + T * 64 * 2, 2 * n * L * h * (192 + 128))
            f["gather_rows"] = (2 * T * W * 2, 0)
            f["pad_q"] = (2 * T * h * 192 * 2, 0)
            f["side_finish"] = (T * H * (4 + 8 + 2), 0)
            f["side_gate"] = (T * s["side"] * (4 + 2 + 2), 0)
            f["cast_rows"] = (T * H * 6, 0)
            f["embed_norm"] = (T * H * (2 + 4 + 2), 0)
        else:
            f["step_kernel"] = (T * (hd * P * N * 8 + ch * 2 * 5 + inner * 2), 0)
            f["mamba_tail"] = (T * (3 * inner + 3 * s["ff"]) * 2, 0)
            f["latent_in"] = (T * (2 * (s["q_rank"] + W) + 3 * s["ff"]) * 2, 0)
            f["cached_decode"] = (T * L * W * 2 + T * h * (W * 2 + R * 4), 2 * T * L * h * (W + R))
            f["absorb_q"] = (h * 128 * R * 2 + T * h * (192 + W) * 2, 2 * T * h * 128 * R)
            f["latent_up"] = (h * 128 * R * 2 + T * h * (R * 4 + 128 * 2), 2 * T * h * 128 * R)
            f["absorb_mma"], f["up_mma"] = f["absorb_q"], f["latent_up"]
            f["side_fused"] = (2 * s["side"] * H * 2 + T * H * (4 + 4 + 4 + 2), 4 * T * s["side"] * H)
    elif kind == "pesanex":
        h, D, ff, c = s["heads"], HEAD, s["ff"], 128
        inner, attn = h * D, T * (2 * h + 2 * KV_HEADS) * D * 2  # (q, k, v in, q and the cache row out; or q, k, v in, result out)
        f["sandwich_kernel"] = (T * H * (14 + 4 * 2 / 12), 0)    # residual in and out, a result, the normed row; two results in 2 of 12
        f["gated_act"] = (T * ff * 2 * 3, 0)
        if prefill:
            n, L = T // ctx, sum(range(1, ctx + 1))
            chunks = n * ((ctx + c - 1) // c)
            for state, out, one_pass, N in (("lin_state", "lin_out", "chunk_pass_kernel<4, true>", GLA_DIM), ("chunk_state", "chunk_out", "chunk_pass_kernel<4, false>", D)):
                st, sums = chunks * inner * N * 4, T * h * N * 4 if N == GLA_DIM else 0
                f[state] = (T * h * (N + D) * 2 + sums + st, 2 * T * inner * N)
                f[out] = (T * h * (2 * N + 2 * D) * 2 + sums + st, 2 * T * h * (D * N + (c + 1) / 2 * (N + D)))
                f[one_pass] = (2 * st, 0)
            f["gate_kernel"] = (T * (h * GLA_DIM * 4 + 32), 0)
            f["lin_tail"] = (T * 3 * inner * 2, 0)
            f["head_rows"] = ((attn + T * 4 * inner * 2) / 2, 0)  # (mean of attention and of retention, whose q and k go in and out)
            f["gather_rows"] = (2 * T * 2 * KV_HEADS * D * 2, 0)
            f["cached_prefill"] = (attn, 4 * n * L * h * D)
            f["embed"] = (T * H * 8, 0)
        else:
            for lanes, N in ((16, GLA_DIM), (32, D)):  # gated, retention
                f[f"lin_step_kernel<__nv_bfloat16, {lanes}>"] = (T * (inner * N * 8 + h * (2 * N + 3 * D) * 2), 0)
            f["head_rows"] = (attn, 0)
            f["cached_decode"] = (T * ctx * 2 * KV_HEADS * D * 2 + T * inner * (2 + 4), 4 * T * ctx * inner)
            f["merge_kernel"] = (T * inner * (4 + 2), 0)
    else:
        hq, hk = cfg.num_q_heads, cfg.num_kv_heads
        if prefill:
            n, L = T // ctx, sum(range(1, ctx + 1))
            f["fa_fwd"] = (T * (2 * hq + 2 * hk) * 128 * 2, 4 * n * L * hq * 128)
            f["rmsnorm_fwd"] = (T * H * 2 * 2, 0)
            f["qk_norm_rope_fwd"] = (T * (hq + 2 * hk) * 128 * 2 * 2, 0)
            f["swiglu_fwd"] = (T * cfg.ffn_hidden_size * 2 * 3, 0)
        else:
            f["decode_mma"] = (T * ctx * 2 * hk * 128 * 2 + T * hq * 128 * 2 * 2, 4 * T * ctx * hq * 128)
            f["rmsnorm_fwd"] = (T * H * 2 * 2, 0)
            f["qk_norm_rope_fwd"] = (T * (hq + 2 * hk) * 128 * 2 * 2, 0)
            f["swiglu_fwd"] = (T * cfg.ffn_hidden_size * 2 * 3, 0)
    return f


def report_kernels(tag: dict, table: dict, fl: dict, pk: dict) -> None:
    total = sum(us * n for us, n in table.values())
    for name, (us, n) in table.items():
        row = dict(tag, kernel=name, us=round(us, 2), launches=round(n, 2), share=round(us * n / total, 4))
        for key, (nbytes, flops) in fl.items():
            if key in name:
                t_mem, t_mm = nbytes / (pk["hbm_gbs"] * 1e3), flops / (pk["bf16_tflops"] * 1e6)
                row.update(floor_us=round(max(t_mem, t_mm), 2), frac=round(max(t_mem, t_mm) / us, 3), bound="hbm" if t_mem >= t_mm else "tensor")
        if row["share"] >= 0.004:
            print(json.dumps(row), flush=True)


def run(design: str, sizes: list, steps: int, warmup: int, kernels: bool, prompts: list, batches: list, ctx: int) -> None:
    from miles_b200.engine import SamplingParams

    pk = peaks()
    for size in sizes:
        for kind in MODELS[design]:
            cfg, model, eng = build(kind, size, max(max(batches), 8192 // min(prompts) + 1), max(ctx + 1024, max(prompts)), max(16384, max(prompts)))
            name = cfg.name if kind != "qwen3" else f"{SIZES[size]['like']} layers x 6"
            base = {"model": name, "params_m": round(cfg.num_params() / 1e6), "layers": cfg.num_layers, "dtype": "bf16", "data": "random tokens and weights",
                    "l2": "weights larger than L2"}
            for n in prompts:
                lens = [n] * max(1, 8192 // n)
                fn = prefill_pass(eng, model, cfg, lens)
                ms, clocks = timed(fn, steps, warmup)
                print(json.dumps(dict(base, what="prefill", tokens=sum(lens), seq_len=n, ms=round(ms, 4), tokens_per_s=round(sum(lens) / ms * 1e3),
                                      clocks=clocks)), flush=True)
                if kernels:
                    report_kernels({"what": "prefill_kernel", "model": name, "seq_len": n}, kernel_table(fn),
                                   floors(cfg, kind, SIZES[size], sum(lens), n, True), pk)
            g = torch.Generator().manual_seed(1)
            for B in batches:
                for _ in range(B):
                    eng.add_request(torch.randint(0, cfg.vocab_size, (ctx,), generator=g).tolist(),
                                    SamplingParams(max_new_tokens=900, ignore_eos=True, sampling_seed=1))
                while eng.waiting or eng.prefilling:
                    eng.step()
                for _ in range(5):
                    eng.step()
                ms, clocks = timed(lambda: eng.step(), 10 * steps, warmup)
                print(json.dumps(dict(base, what="decode", batch=B, ctx=ctx, ms_per_step=round(ms, 4), tokens_per_s=round(B / ms * 1e3), clocks=clocks)), flush=True)
                if kernels:
                    report_kernels({"what": "decode_kernel", "model": name, "batch": B}, kernel_table(lambda: eng.step(), 20),
                                   floors(cfg, kind, SIZES[size], B, ctx, False), pk)
                eng.abort_request(abort_all=True)
                eng.pop_finished()
            model.check_status()
            del model, eng
            torch.cuda.empty_cache()


def main(argv=None, steps: int = 10, warmup: int = 3) -> None:
    ap = argparse.ArgumentParser()
    ap.add_argument("--design", choices=list(MODELS), default="rokivik")
    ap.add_argument("--sizes", default="2048,4096")
    ap.add_argument("--steps", type=int, default=steps)
    ap.add_argument("--warmup", type=int, default=warmup)
    ap.add_argument("--prompts", default="1024,8192", help="prompt lengths (batches of 8192 tokens)")
    ap.add_argument("--batches", default="1,8,64", help="decode batch sizes")
    ap.add_argument("--ctx", type=int, default=4096, help="cached tokens per sequence while decoding")
    ap.add_argument("--kernels", action="store_true", help="per-kernel device times next to their byte / operation floors")
    ns = ap.parse_args(argv)
    ints = lambda s: [int(v) for v in s.split(",")]
    run(ns.design, ns.sizes.split(","), ns.steps, ns.warmup, ns.kernels, ints(ns.prompts), ints(ns.batches), ns.ctx)


if __name__ == "__main__":
    main()
