"""Prefill and decode throughput of the layered decoders beside the framework's other models of equal layer sizes, on one GPU.

    python bench.py --family gunuvik [--model gunuvik-1.7b] [--steps K] [--warmup W]
    python bench.py --family ditilix [--model ditilix-1.7b|ditilix-moe]
    python bench.py --family niralix [--model niralix-1.7b|niralix-moe]
    python bench.py --family pidenex [--model pidenex-1.7b|pidenex-flat]

Random weights, random token ids, bf16.  All models go through their own engines: ``prefill`` on whole prompts and
decode ticks (CUDA graph) at a given context, reached with ``fast_forward``.  Comparison models: the plain Qwen3
backbone (one pass per token, no adapter) with the same width, heads and vocabulary and a feed-forward of 6144, for
Ditilix and Pidenex also Gunuvik of that size, for Niralix also Gunuvik and the routed Ditilix; ``*_per_layer`` divides by the
number of layer runs, because a recurrent layer has no feed-forward of its own and a layer of a loop runs several times.  Device time from CUDA
events around K calls after W warm-up calls; every call reads the weights (GBs), far more than the 126 MB L2.
"""
from __future__ import annotations

import gc
import json

PREFILL = ((64, 1024), (8, 8192), (1, 8192))           # prompts x tokens
DECODE = ((256, 1024), (256, 2304), (32, 2304), (1, 2304))     # rows x context


def _qwen3(dev):
    import torch
    from tah_b200 import TaHConfig, TaHForCausalLM
    from tah_b200.engine import TaHEngine
    from tah_b200.models import Qwen3Config, Qwen3ForCausalLM, gunuvik_preset
    gcfg = gunuvik_preset("gunuvik-1.7b")
    a = next(l.mixer for l in gcfg.layers if l.mixer.kind == "attention")
    ff = next(l.ff for l in gcfg.layers if l.ff).ff
    cfg = Qwen3Config(vocab_size=gcfg.vocab_size, hidden_size=gcfg.hidden_size, intermediate_size=ff,
                      num_hidden_layers=len(gcfg.layers), num_attention_heads=a.heads, num_key_value_heads=a.kv_heads,
                      head_dim=a.dim, tie_word_embeddings=False)
    with torch.device(dev):
        base = Qwen3ForCausalLM(cfg, dtype=torch.bfloat16)
    model = TaHForCausalLM(base, TaHConfig(max_iter=1, iter_decider="IterLabelDecider", adapter_kwargs=dict(r=0),
                                           train_loss="NextTokenPredLoss")).to(dev).eval()
    return lambda rows: TaHEngine(model, max_rows=rows), model, cfg


def _layered(name, dev):
    import torch
    from tah_b200.engine import HybridEngine
    from tah_b200.models import (DitilixForCausalLM, GunuvikForCausalLM, NiralixForCausalLM, PidenexForCausalLM, ditilix_preset,
                                 gunuvik_preset, niralix_preset, pidenex_preset)
    cls, preset = {"ditilix": (DitilixForCausalLM, ditilix_preset), "gunuvik": (GunuvikForCausalLM, gunuvik_preset),
                   "niralix": (NiralixForCausalLM, niralix_preset), "pidenex": (PidenexForCausalLM, pidenex_preset)}[name.split("-")[0]]
    model = cls(preset(name), dtype=torch.bfloat16, device=dev).init_random()
    return lambda rows: HybridEngine(model, max_rows=rows), model, model.config


def _prefill_ms(eng, ids, steps, warmup):
    import torch
    for _ in range(warmup):
        eng.prefill(ids, None, 1)
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    for _ in range(steps):
        eng.prefill(ids, None, 1)
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) / steps


def _tick_ms(eng, rows, ctx, vocab, steps, warmup, dev):
    """Device time of a decode tick of ``rows`` rows at context ``ctx``."""
    import torch
    ids = torch.randint(0, vocab, (rows, 16), device=dev)
    ev = [torch.cuda.Event(enable_timing=True) for _ in range(2)]

    def on_tick(t, s):
        if t == 2:
            eng.fast_forward(s, ctx)
        if t == 2 + warmup:
            ev[0].record()
        if t == 2 + warmup + steps:
            ev[1].record()
    res = eng.generate(ids, None, max_new_tokens=ctx + steps + warmup + 8, max_ticks=2 + warmup + steps, sync_every=1 << 30,
                       on_tick=on_tick)
    assert res.ticks == 2 + warmup + steps
    return ev[0].elapsed_time(ev[1]) / steps


def run(args):
    import torch
    from bench_clocks import ClockSampler
    dev = torch.device("cuda", 0)
    torch.cuda.set_device(dev)
    presets = {"gunuvik": ["gunuvik-1.7b"], "ditilix": ["ditilix-1.7b", "ditilix-moe"], "niralix": ["niralix-1.7b", "niralix-moe"],
               "pidenex": ["pidenex-1.7b", "pidenex-flat"]}
    beside = {"gunuvik": [], "ditilix": ["gunuvik-1.7b"], "niralix": ["gunuvik-1.7b", "ditilix-moe"], "pidenex": ["gunuvik-1.7b"]}
    names = [args.model] if args.model.startswith(args.family) else presets[args.family]
    builds = [(n, lambda d, n=n: _layered(n, d)) for n in names + beside[args.family]]
    builds.append(("qwen3 of the same sizes", _qwen3))
    steps, warmup = max(3, args.steps), max(3, args.warmup)
    sampler = ClockSampler(0)
    sampler.start()
    out = {"metric": "layered decoder prefill / decode, device-timed", "unit": "tokens/s", "n_gpus": 1, "steps": steps,
           "warmup": warmup, "dtype": "bf16", "data": "synthetic", "impl": "ours", "config": {"models": names},
           "models": {}}
    for label, build in builds:
        torch.manual_seed(0)
        make, model, cfg = build(dev)
        V, L = cfg.vocab_size, len(cfg.layer_runs()) if hasattr(cfg, "layer_runs") else cfg.num_hidden_layers
        rec = {"parameters": sum(p.numel() for p in model.parameters()), "prefill": {}, "decode": {}}
        for B, T in PREFILL:
            eng = make(B)
            ms = _prefill_ms(eng, torch.randint(0, V, (B, T), device=dev), max(3, steps // 8), 2)
            rec["prefill"][f"{B}x{T}"] = {"ms": round(ms, 3), "tokens_per_s": round(B * T / ms * 1e3, 1),
                                          "us_per_layer": round(ms * 1e3 / L, 1)}
            del eng
            gc.collect()
            torch.cuda.empty_cache()
        for B, ctx in DECODE:
            eng = make(B)
            ms = _tick_ms(eng, B, ctx, V, steps, warmup, dev)
            rec["decode"][f"{B}@{ctx}"] = {"ms": round(ms, 4), "tokens_per_s": round(B / ms * 1e3, 1),
                                           "us_per_layer": round(ms * 1e3 / L, 2), "kernels_per_tick": eng.kernel_launches_per_tick}
            del eng
            gc.collect()
            torch.cuda.empty_cache()
        out["models"][label] = rec
        del make, model
        gc.collect()
        torch.cuda.empty_cache()
    out["clocks"] = sampler.stop()
    print(json.dumps(out))
