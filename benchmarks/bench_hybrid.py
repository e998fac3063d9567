#!/usr/bin/env python
"""Prefill and decode throughput of hybrid decoders (random weights) beside other models at equal size, each through its own
serving engine on one GPU.

    python benchmarks/bench_hybrid.py                      # every size
    python benchmarks/bench_hybrid.py --models tonilix,vobotar,polosun,hybrid,llama
    python bench.py --hybrid [fozelix | polosun | vobotar | tonilix]    # the same, from the headline benchmark's command line

The models of a size have the same width, feed-forward, layer count, vocabulary and attention heads. ``hybrid`` has three
gated-delta layers (16 or 8 key heads, twice as many value heads, 128 x 128) to every chunked-attention layer; ``polosun``
cycles through retention (heads of 128 x 128), latent attention (64 + 64 rotated query columns a head, values of 128, a latent
of 512) and the gated recurrence (as many channels as the width, gate blocks of 256); ``vobotar`` through capped attention, attention
in a window of 1024 beside time mixing (heads of 64, as wide as the model) and beside state-space duality (heads of 64, twice as wide as
the model, a state of 128), with a side input of 128 columns per layer; ``tonilix`` has two layers of the delta rule with decays per channel
(heads of 128 x 128, as wide as the model) to every one of attention beside gated linear attention (heads of 64, as wide as the model), a
dense first feed-forward and then 6 of 32 experts, which together do the work of the dense one. bf16 weights and KV on all sides,
greedy. Prefill: ``seqs`` prompts of ``prompt`` tokens in one step; decode: a batch of
requests after that. Times are wall clock around engine steps with a device synchronise on both sides (inputs from the
host and the read of the chosen tokens included); ``gpu_ms`` is the captured decode step alone, from CUDA events. Every
step streams more weight bytes than L2 holds.
"""
from __future__ import annotations

import argparse
import gc
import json
import os
import sys
import time

sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))

SIZES = {
    "2048x8": dict(width=2048, ff=5632, layers=8, heads=16, kv=8, key_heads=8, vocab=32768),
    "4096x8": dict(width=4096, ff=14336, layers=8, heads=32, kv=8, key_heads=16, vocab=32768),
}


def build(kind, s, device, max_pos):
    import torch

    from tesseract_b200.models import HybridConfig, HybridModel, LlamaConfig, LlamaModel
    from tesseract_b200.models.hybrid import AttentionSpec, DeltaSpec, GLUSpec, LayerSpec
    if kind == "llama":
        cfg = LlamaConfig(vocab_size=s["vocab"], hidden_size=s["width"], num_hidden_layers=s["layers"], num_attention_heads=s["heads"],
                          num_key_value_heads=s["kv"], intermediate_size=s["ff"], max_position_embeddings=max_pos,
                          dtype=torch.bfloat16)
        return LlamaModel(cfg, device=device, init_std=0.02, seed=1)
    if kind == "polosun":
        from tesseract_b200.models import polosun
        from tesseract_b200.models.hybrid import LatentSpec, RetentionSpec, RGLRUSpec, Rotary
        h = s["heads"]
        layers = polosun.layer_cycle(
            s["layers"], LatentSpec(h, 64, 64, 128, 512, 128 ** -0.5, Rotary(64, 1e6)),
            RetentionSpec(h, 128, 128, tuple(1.0 - 2.0 ** (-5 - 7 * i / h) for i in range(h)), Rotary(128, 1e4)),
            RGLRUSpec(s["width"], s["width"] // 256, 4), s["ff"])
        return HybridModel(HybridConfig(s["vocab"], s["width"], layers, eps=1e-6, dtype=torch.bfloat16, form="parallel", residual_mult=0.5,
                                        depth_average=True, tied=False), device=device, init_std=0.02, seed=1)
    if kind == "vobotar":
        from tesseract_b200.models import vobotar
        W = s["width"]
        layers = vobotar.standard_layers(s["layers"], s["heads"], s["kv"], 128, 1024, W // 64, 64, 64, 2 * W // 64, 64, 128, s["ff"])
        return HybridModel(HybridConfig(s["vocab"], W, layers, eps=1e-6, dtype=torch.bfloat16, form="post", token_side=128), device=device,
                           init_std=0.02, seed=1)
    if kind == "tonilix":
        from tesseract_b200.models import tonilix
        from tesseract_b200.models.hybrid import Choice
        W = s["width"]
        layers = tonilix.standard_layers(s["layers"], s["heads"], s["kv"], 128, W // 128, 128, 128, W // 64, 64, s["ff"], s["ff"] // 4,
                                         Choice(32, 6, 4, 2, 1.0))
        return HybridModel(HybridConfig(s["vocab"], W, layers, eps=1e-6, dtype=torch.bfloat16, form="pre", tied=False, norm_parts=2,
                                        layer_scale=True, token_shift=True, sinusoid=True, embed_norm=True), device=device, init_std=0.02, seed=1)
    att = AttentionSpec(s["heads"], s["kv"], 128, 128, 128 ** -0.5, 4096)
    dlt = DeltaSpec(2 * s["key_heads"], s["key_heads"], 128, 128, 4)
    layers = [LayerSpec(att if i % 4 == 3 else dlt, GLUSpec(s["ff"], 7.0)) for i in range(s["layers"])]
    return HybridModel(HybridConfig(s["vocab"], s["width"], layers, dtype=torch.bfloat16), device=device, init_std=0.02, seed=1)


def measure(kind, s, seqs, prompt, decode_batches, steps, device):
    import random

    import torch

    from tesseract_b200 import _native
    from tesseract_b200.models import GenerateConfig
    from tesseract_b200.models.scheduler import EngineConfig
    from tesseract_b200.serving import make_engine
    rng = random.Random(0)
    top = max(decode_batches)
    new = steps + 96                                      # (requests start over several steps and must all still decode)
    per = {"prefill": prompt + 1, "decode": 1300 + new + 2}
    blocks = max(seqs * (per["prefill"] // 16 + 2), top * (per["decode"] // 16 + 2)) + 64
    model = build(kind, s, device, max(per.values()) + 16)
    extra = {"max_step_tokens": seqs * prompt + top} if kind != "llama" else {"max_prefill_tokens": seqs * prompt}
    eng = make_engine(model, EngineConfig(block_size=16, num_blocks=blocks, max_seq_len=max(per.values()), max_batch_size=top), **extra)
    prompts = [[rng.randrange(s["vocab"]) for _ in range(prompt)] for _ in range(seqs)]
    out = {"model": kind, "prefill": {"seqs": seqs, "prompt": prompt}, "decode": []}
    best = None
    for _ in range(5):                                    # two warm-up passes, then the best of three
        for p in prompts:
            eng.add_request(p, GenerateConfig(max_new_tokens=1))
        torch.cuda.synchronize(device)
        t0 = time.perf_counter()
        while eng.has_pending():
            eng.step()
        torch.cuda.synchronize(device)
        dt = time.perf_counter() - t0
        best = dt if best is None or _ < 2 else min(best, dt)
    out["prefill"].update(ms=round(best * 1e3, 3), tok_s=round(seqs * prompt / best))
    for B in decode_batches:
        eng.requests.clear()
        for i in range(B):
            eng.add_request([rng.randrange(s["vocab"]) for _ in range(1300)], GenerateConfig(max_new_tokens=new))
        while eng.waiting or len(eng.running) < B or any(r.generated < 4 for r in eng.running):
            eng.step()
        torch.cuda.synchronize(device)
        n0, t0 = _native.launch_count(), time.perf_counter()
        for _ in range(steps):
            eng.step()
        torch.cuda.synchronize(device)
        dt = (time.perf_counter() - t0) / steps
        assert len(eng.running) == B
        g = eng._graphs[eng._bucket(B)]["graph"]
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        for _ in range(8):                                # the recorded inputs once more: the same cells are rewritten
            g.replay()
        e1.record()
        torch.cuda.synchronize(device)
        out["decode"].append({"batch": B, "context": 1300, "ms": round(dt * 1e3, 3), "tok_s": round(B / dt),
                              "gpu_ms": round(e0.elapsed_time(e1) / 8, 3)})
        while eng.has_pending():
            eng.step()
    out["kernel_status"] = _native.read_status(torch.cuda.current_stream(device).cuda_stream)
    del eng, model
    gc.collect()
    torch.cuda.empty_cache()
    return out


def run(sizes=None, seqs=4, prompt=4096, decode_batches=(1, 32, 256), steps=24, device=None, models=("hybrid", "llama")):
    """{size: {model: ...}}"""
    import torch
    device = device or torch.device("cuda", 0)
    torch.cuda.set_device(device)
    res = {}
    for name in sizes or SIZES:
        res[name] = {k: measure(k, SIZES[name], seqs, prompt, decode_batches, steps, device) for k in models}
    return res


def main():
    ap = argparse.ArgumentParser(description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--sizes", default=",".join(SIZES))
    ap.add_argument("--seqs", type=int, default=4)
    ap.add_argument("--prompt", type=int, default=4096)
    ap.add_argument("--steps", type=int, default=24)
    ap.add_argument("--models", default="hybrid,llama", help="comma list of tonilix, vobotar, polosun, hybrid, llama")
    a = ap.parse_args()
    models = a.models.split(",")
    for name, r in run(a.sizes.split(","), a.seqs, a.prompt, steps=a.steps, models=models).items():
        for k in models:
            print(json.dumps({"size": name, **r[k]}), flush=True)


if __name__ == "__main__":
    main()
