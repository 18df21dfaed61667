"""Prefill and decode throughput of the hybrid decoder beside the Qwen3 backbone of equal layer sizes, on one GPU.

    python bench.py --family gunuvik [--model gunuvik-1.7b] [--steps K] [--warmup W]

Random weights, random token ids, bf16.  Both models go through their own engines: ``prefill`` on whole prompts and
decode ticks (CUDA graph) at a given context, reached with ``fast_forward``.  The comparison model is the plain Qwen3
backbone (one pass per token, no adapter) with the same width, heads, feed-forward and vocabulary; ``*_per_layer``
divides by the number of layers, because a recurrent layer has no feed-forward of its own.  Device time from CUDA
events around K calls after W warm-up calls; every call reads the weights (GBs), far more than the 126 MB L2.
"""
from __future__ import annotations

import gc
import json

PREFILL = ((64, 1024), (8, 8192), (1, 8192))           # prompts x tokens
DECODE = ((256, 1024), (256, 2304), (32, 2304), (1, 2304))     # rows x context


def _qwen3(gcfg, dev):
    import torch
    from tah_b200 import TaHConfig, TaHForCausalLM
    from tah_b200.engine import TaHEngine
    from tah_b200.models import Qwen3Config, Qwen3ForCausalLM
    a = next(l.mixer for l in gcfg.layers if l.mixer.kind == "attention")
    ff = next(l.ff for l in gcfg.layers if l.ff).ff
    cfg = Qwen3Config(vocab_size=gcfg.vocab_size, hidden_size=gcfg.hidden_size, intermediate_size=ff,
                      num_hidden_layers=len(gcfg.layers), num_attention_heads=a.heads, num_key_value_heads=a.kv_heads,
                      head_dim=a.dim, tie_word_embeddings=False)
    with torch.device(dev):
        base = Qwen3ForCausalLM(cfg, dtype=torch.bfloat16)
    model = TaHForCausalLM(base, TaHConfig(max_iter=1, iter_decider="IterLabelDecider", adapter_kwargs=dict(r=0),
                                           train_loss="NextTokenPredLoss")).to(dev).eval()
    return lambda rows: TaHEngine(model, max_rows=rows), model


def _gunuvik(gcfg, dev):
    import torch
    from tah_b200.engine import HybridEngine
    from tah_b200.models import GunuvikForCausalLM
    model = GunuvikForCausalLM(gcfg, dtype=torch.bfloat16, device=dev).init_random()
    return lambda rows: HybridEngine(model, max_rows=rows), model


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
    from tah_b200.models import gunuvik_preset
    dev = torch.device("cuda", 0)
    torch.cuda.set_device(dev)
    name = args.model if args.model.startswith("gunuvik") else "gunuvik-1.7b"
    gcfg = gunuvik_preset(name)
    V, L = gcfg.vocab_size, len(gcfg.layers)
    steps, warmup = max(3, args.steps), max(3, args.warmup)
    sampler = ClockSampler(0)
    sampler.start()
    out = {"metric": "hybrid decoder prefill / decode, device-timed", "unit": "tokens/s", "n_gpus": 1, "steps": steps,
           "warmup": warmup, "dtype": "bf16", "data": "synthetic", "impl": "ours", "config": {"model": name, "layers": L},
           "models": {}}
    for label, build in ((name, _gunuvik), ("qwen3 of the same sizes", _qwen3)):
        torch.manual_seed(0)
        make, model = build(gcfg, dev)
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
