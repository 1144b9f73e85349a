"""Serving throughput of the hybrid decoders (Famudra, Pozalorn) beside Llama at equal width and equal active feed-forward size.

    python bench.py --workload famudra             # the same measurement, one JSON line
    python bench.py --workload pozalorn
    python benchmarks/hybrid_bench.py --family pozalorn --sizes small,medium,large

Random weights, uniform random prompts, bf16, one GPU.  A hybrid decoder runs through its ``step`` (prompts eagerly, decode
steps as the captured graph); Llama through ``TPLlamaEngine`` with a group of one rank, the package's one-GPU serving path.
Both models have the same width, number of layers, vocabulary and context.  Llama's SwiGLU width is that of Pozalorn's gated
feed-forward, or 2/3 of the feed-forward width a Famudra token uses (three matrices against two).  Times are CUDA events;
weights and activations exceed L2.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import torch

sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))

VOCAB = 32768
SIZES = {      # width, layers, heads, head dim, q_rank, kv_rank, recurrence width, blocks, experts, top, ff, shared ff
    "small": dict(width=1024, layers=6, heads=16, dim=64, q_rank=384, kv_rank=256, rec=1024, blocks=8, experts=32, top=4,
                  ff=512, shared=1024),
    "medium": dict(width=2048, layers=4, heads=16, dim=128, q_rank=768, kv_rank=512, rec=2560, blocks=10, experts=64, top=6,
                   ff=1024, shared=2048),
    "large": dict(width=4096, layers=2, heads=32, dim=128, q_rank=1536, kv_rank=512, rec=4096, blocks=16, experts=64, top=6,
                  ff=1408, shared=2816),
}
POZALORN_SIZES = {      # width, layers, feed-forward, attention heads of `dim`, window, block; linear attention heads, dim, vdim
    "small": dict(width=1024, layers=6, ff=2816, heads=16, dim=64, window=1024, pool=16, lin_heads=8, lin_dim=64, lin_vdim=128),
    "medium": dict(width=2048, layers=6, ff=5504, heads=16, dim=128, window=1024, pool=16, lin_heads=16, lin_dim=64,
                   lin_vdim=128),
    "large": dict(width=4096, layers=3, ff=11008, heads=32, dim=128, window=1024, pool=16, lin_heads=32, lin_dim=64,
                  lin_vdim=128),
}
PROMPTS = ((1, 8192), (4, 2048))
DECODE = ((1, 2048), (32, 2048))


def famudra_config(s) -> dict:
    mlp = {"kind": "moe", "router": {"experts": s["experts"], "top": s["top"]}, "expert": {"ff": s["ff"]},
           "shared": {"ff": s["shared"]}}
    att = {"type": "latent_attention", "mlp": mlp,
           "mixer": dict(heads=s["heads"], dim=s["dim"], vdim=s["dim"], q_rank=s["q_rank"], kv_rank=s["kv_rank"],
                         scale=s["dim"] ** -0.5)}
    rec = {"type": "rglru", "mlp": mlp, "mixer": dict(width=s["rec"], blocks=s["blocks"], conv=4)}
    return {"architecture": "Famudra", "vocab": VOCAB, "width": s["width"], "norm": {"eps": 1e-6},
            "layers": [rec if i % 2 == 0 else att for i in range(s["layers"])]}


def pozalorn_config(s) -> dict:
    rot = {"base": 1e6, "dims": s["dim"], "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}
    att = dict(heads=s["heads"], kv_heads=max(1, s["heads"] // 4), dim=s["dim"], vdim=s["dim"], rot=rot, scale=s["dim"] ** -0.5)
    lin = dict(heads=s["lin_heads"], dim=s["lin_dim"], vdim=s["lin_vdim"])
    mixers = [("gla", dict(lin, tau=16.0)),
              ("attention", dict(att, mask={"size": s["window"], "pool": s["pool"]})),
              ("parallel", {"left": dict(att, mask={"size": s["window"]}), "left_scale": 0.5, "right_scale": 0.5,
                            "right": dict(lin, decay=[0.5 ** (2.0 ** -(8.0 * i / s["lin_heads"])) for i in range(s["lin_heads"])])})]
    return {"architecture": "Pozalorn", "vocab": VOCAB, "width": s["width"], "norm": {"eps": 1e-6},
            "layers": [{"type": mixers[i % 3][0], "mixer": mixers[i % 3][1], "mlp": {"kind": "dense", "ff": s["ff"]}}
                       for i in range(s["layers"])]}


def families():
    """name -> (sizes, configuration of a size, Llama's feed-forward width)."""
    return {"famudra": (SIZES, famudra_config, lambda s: (2 * (s["top"] * s["ff"] + s["shared"]) // 3 + 127) // 128 * 128),
            "pozalorn": (POZALORN_SIZES, pozalorn_config, lambda s: s["ff"])}


def timed(fn, iters: int, warmup: int) -> float:
    """Milliseconds per call."""
    for _ in range(warmup):
        fn()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    torch.cuda.synchronize()
    e0.record()
    for _ in range(iters):
        fn()
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) / iters


def measure_hybrid(family: str, s, steps: int, warmup: int) -> dict:
    from dart_pytorch_b200 import _native
    from dart_pytorch_b200.models import registry
    model = registry.architecture(family).build(families()[family][1](s), device="cuda", dtype=torch.bfloat16, init_std=0.02)
    model.eval()
    out = {"params": model.num_scalars(), "prefill": [], "decode": []}
    g = torch.Generator().manual_seed(0)
    for B, S in PROMPTS:
        t = torch.randint(0, VOCAB, (B, S), generator=g).cuda()
        cache = model.new_cache(S, B)
        rows = [b * S + S - 1 for b in range(B)]

        def prompt():
            cache.reset()
            model.step(cache, t, rows)
        ms = timed(prompt, max(3, steps // 8), warmup)
        out["prefill"].append({"batch": B, "tokens": S, "ms": ms, "tokens_per_s": B * S / ms * 1e3})
    for B, S in DECODE:
        t = torch.randint(0, VOCAB, (B, S), generator=g).cuda()
        cache = model.new_cache(S + 2 * (steps + warmup) + 8, B)
        model.step(cache, t, [])
        nxt = torch.randint(0, VOCAB, (B, 1), generator=g).cuda()
        ms = timed(lambda: model.step(cache, nxt), steps, warmup)
        out["decode"].append({"batch": B, "context": S, "ms": ms, "tokens_per_s": B / ms * 1e3,
                              "kernels_per_step": cache.graph[3]})
        del cache
    _native.raise_on_device_error()
    return out


def measure_llama(s, ffn: int, steps: int, warmup: int) -> dict:
    import torch.distributed as dist
    from dart_pytorch_b200.models.llama import LlamaConfig
    from dart_pytorch_b200.parallel.tp_llama import TPLlamaEngine
    if not dist.is_initialized():
        os.environ["NCCL_DEBUG"] = "NONE"          # standard output carries one JSON line
        os.environ.setdefault("MASTER_ADDR", "127.0.0.1")
        os.environ.setdefault("MASTER_PORT", "29577")
        dist.init_process_group("nccl", rank=0, world_size=1, device_id=torch.device("cuda", torch.cuda.current_device()))
    heads = s["width"] // s["dim"]
    out = {"ffn_dim": ffn, "prefill": [], "decode": []}
    g = torch.Generator().manual_seed(0)
    for kind, shapes in (("prefill", PROMPTS), ("decode", DECODE)):
        for B, S in shapes:
            ctx = S + (2 * (steps + warmup) + 8 if kind == "decode" else 0)
            cfg = LlamaConfig(vocab_size=VOCAB, max_ctx=ctx, embed_dim=s["width"], num_layers=s["layers"], num_heads=heads,
                              num_kv_heads=max(1, heads // 4), ffn_dim=ffn, tie_weights=False)
            eng = TPLlamaEngine(cfg, max_batch=B, max_ctx=ctx, max_rows=min(B * S, 8192))
            t = torch.randint(0, VOCAB, (B, S), generator=g).cuda()
            if kind == "prefill":
                def prompt():
                    eng.reset()
                    eng.prefill(t)
                ms = timed(prompt, max(3, steps // 8), warmup)
                out[kind].append({"batch": B, "tokens": S, "ms": ms, "tokens_per_s": B * S / ms * 1e3})
            else:
                eng.prefill(t)
                ms = timed(lambda: eng.decode_step(B), steps, warmup)
                out[kind].append({"batch": B, "context": S, "ms": ms, "tokens_per_s": B / ms * 1e3})
            del eng
            torch.cuda.empty_cache()
    return out


def measure(family: str, sizes, steps: int, warmup: int, llama: bool = True) -> dict:
    out = {}
    table, _, ffn = families()[family]
    for name in sizes:
        out[name] = {family: measure_hybrid(family, table[name], steps, warmup)}
        torch.cuda.empty_cache()
        if llama:
            out[name]["llama"] = measure_llama(table[name], ffn(table[name]), steps, warmup)
            torch.cuda.empty_cache()
    return out


def bench_line(args, sampler_cls) -> dict:
    """The line ``bench.py --workload <family>`` prints: decode throughput of the medium size at batch 32 as the value."""
    family, table = args.workload, families()[args.workload][0]
    sampler = sampler_cls(0)
    sampler.start()
    sizes = [s for s in args.sizes.split(",") if s]
    sampler.mark()
    r = measure(family, sizes, args.steps, args.warmup)
    clocks = sampler.stop()
    main = r.get("medium") or r[sizes[0]]
    dec = main[family]["decode"][-1]
    return {"metric": f"{family}_decode_tokens_per_s", "value": dec["tokens_per_s"], "unit": "tokens/s", "n_gpus": 1,
            "steps": args.steps, "warmup": args.warmup, "ms_per_step": dec["ms"], "higher_is_better": True,
            "vs_baseline": None, "dtype": "bf16", "data": "synthetic", "impl": "ours",
            "config": {"model": family, "sizes": {k: table[k] for k in sizes},
                       "cache_policy": "weights and activations exceed the 126 MB L2"},
            "gpu_launches": dec["kernels_per_step"] * args.steps, "clocks": clocks, "sizes": r}


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--family", default="famudra", choices=sorted(families()))
    ap.add_argument("--sizes", default="small,medium,large")
    ap.add_argument("--steps", type=int, default=64)
    ap.add_argument("--warmup", type=int, default=4)
    ap.add_argument("--no-llama", action="store_true")
    args = ap.parse_args()
    torch.cuda.set_device(0)
    print(json.dumps(measure(args.family, [s for s in args.sizes.split(",") if s], args.steps, args.warmup, not args.no_llama),
                     indent=1))


if __name__ == "__main__":
    main()
