"""Prefill and decode throughput of the dense-weight decoders at a few real layer sizes, each beside the model
closest to it at equal size (random weights, one GPU): Degedra beside the hybrid decoder
(`python bench.py --mode degedra`), Vekerax beside Degedra (`python bench.py --mode vekerax`).

    python -m mi50grad_b200.bench.degedra --model vekerax|degedra|hybrid --size 4k --phase decode|prefill --steps 2

runs one phase of one model a few times without timing anything (a small command for a profiler).
"""
from __future__ import annotations

import argparse
import json
import os

import torch

from ..config import (DegedraConfig, EngineConfig, LightningSpec, ParallelLayerSpec, QwenConfig, SSDSpec, StreamLayerSpec, VekeraxConfig,
                      WindowAttentionSpec)

# width, feed-forward, attention heads / kv heads / dim, recurrence heads (of 64, state 128, 8 groups), window, layers
SIZES = {
    "2k": (2048, 6144, 16, 4, 128, 32, 1024, 12),
    "4k": (4096, 12288, 32, 8, 128, 64, 1024, 8),
    "5k": (5120, 17408, 40, 8, 128, 80, 4096, 6),
}
VOCAB = 65536


def degedra_config(size: str) -> DegedraConfig:
    w, ff, h, kv, d, sh, win, n = SIZES[size]
    layer = ParallelLayerSpec(WindowAttentionSpec(h, kv, d, d, 1e6, d ** -0.5, win), SSDSpec(sh, 64, 128, 8, 4, 8), 0.7, 1.0, ff)
    return DegedraConfig(w, VOCAB, 1e-5, [layer] * n, 30.0)


def hybrid_config(size: str) -> QwenConfig:
    """The hybrid decoder with the same width, feed-forward, layer count and vocabulary: attention heads of 256
    (same total), DeltaNet value heads of 128 (same total as the recurrence's columns)."""
    w, ff, h, kv, d, sh, win, n = SIZES[size]
    return QwenConfig(hidden_size=w, intermediate_size=ff, num_hidden_layers=n, vocab_size=VOCAB, num_attention_heads=h * d // 256,
                      num_key_value_heads=max(1, kv * d // 256), head_dim=256, linear_num_value_heads=sh // 2,
                      linear_num_key_heads=sh // 4, linear_key_head_dim=128, linear_value_head_dim=128, full_attention_interval=2)


def vekerax_config(size: str) -> VekeraxConfig:
    """Same width, feed-forward, layer count and vocabulary; attention and lightning layers in turn, each mixer as
    wide as its counterpart in the Degedra layer (recurrent state of the same size in heads of 128), four streams."""
    w, ff, h, kv, d, sh, win, n = SIZES[size]
    att = StreamLayerSpec(WindowAttentionSpec(h, kv, d, 0, 0.0, d ** -0.5, win, vdim=d, head_norm=True, keep_first=4, softcap=30.0, sink=True), ff)
    rec = StreamLayerSpec(LightningSpec(sh // 2, 128, 128, tuple(1.0 - 2.0 ** (-1 - 8 * i / sh) for i in range(sh // 2))), ff)
    return VekeraxConfig(w, VOCAB, 1e-5, [att if i % 2 == 0 else rec for i in range(n)], 1.0, 1.0, 4)


MODELS = ("vekerax", "degedra", "hybrid", "hybrid-fp16attn")


def make(model: str, size: str, max_seq: int, batch: int):
    ecfg = EngineConfig(max_step_rows=64)
    if model == "vekerax":
        from ..engine.vekerax_engine import VekeraxEngine
        eng = VekeraxEngine(vekerax_config(size), max_seq_len=max_seq, max_batch=batch, engine_config=ecfg)
        eng.init_random(0)
    elif model == "degedra":
        from ..engine.mixer_engine import MixerEngine
        eng = MixerEngine(degedra_config(size), max_seq_len=max_seq, max_batch=batch, engine_config=ecfg)
        eng.init_random(0)
    else:
        from ..engine.engine import InferenceEngine
        eng = InferenceEngine(hybrid_config(size), max_seq_len=max_seq, max_batch=batch, engine_config=ecfg)
        eng.init_random(0, int4_attention=model != "hybrid-fp16attn")
    return eng


def _timed(fn, n):
    ev = [torch.cuda.Event(enable_timing=True) for _ in range(2)]
    torch.cuda.synchronize()
    ev[0].record()
    for _ in range(n):
        fn()
    ev[1].record()
    torch.cuda.synchronize()
    return ev[0].elapsed_time(ev[1]) / n


def gemm_flops_per_token(eng) -> float:
    """2 x the elements of every projection a prompt token goes through (the head runs on the last row only)."""
    n = 0
    for ly in eng.layers:
        for l in (ly.in_proj, ly.out_proj, ly.gate_up, ly.down):
            if l is not None:
                n += 2 * l.N * l.K
    return float(n)


def measure(model: str, size: str, steps: int, warmup: int, peaks: dict) -> dict:
    ctx, batch = 512, 8
    eng = make(model, size, 2048 + 64, batch)
    vocab = eng.config.vocab_size
    gen = torch.Generator().manual_seed(1)
    prompt = lambda n: torch.randint(0, vocab, (n,), generator=gen).tolist()
    out = {"weights_gb_per_token": round(eng.weight_bytes() / 1e9, 3)}

    def decode(seqs):
        for s in seqs:
            eng.reset(s)
            eng.prefill_tokens(prompt(ctx), s)
        eng.decode_tokens(max(3, warmup), seqs, collect=False)
        return _timed(lambda: eng.decode_tokens(steps, seqs, collect=False), 1) / steps
    t = decode([0])
    out["decode_bs1_tok_s"], out["decode_bs1_ms"] = round(1e3 / t, 1), round(t, 4)
    out["decode_bs1_hbm_gbs"] = round(eng.weight_bytes() / t / 1e6, 1)
    out["decode_bs1_of_measured_copy"] = round(eng.weight_bytes() / t / 1e6 / peaks["hbm_gbs"], 3)
    out["launches_per_step"] = eng.launches_per_step()
    t = decode(list(range(batch)))
    out[f"decode_bs{batch}_tok_s"], out[f"decode_bs{batch}_ms"] = round(batch * 1e3 / t, 1), round(t, 4)

    def prefill(n):
        p = prompt(n)

        def one():
            eng.reset(0)
            eng.prefill_tokens(p, 0)
        for _ in range(3):
            one()
        return _timed(one, max(3, steps // 16))
    for n in (512, 2048):
        t = prefill(n)
        out[f"pp{n}_tok_s"], out[f"pp{n}_ms"] = round(n * 1e3 / t, 1), round(t, 3)
        out[f"pp{n}_tflops"] = round(gemm_flops_per_token(eng) * n / t / 1e9, 1)
        out[f"pp{n}_of_measured_gemm"] = round(gemm_flops_per_token(eng) * n / t / 1e9 / peaks["bf16_tflops"], 3)
    # end to end through the generation API: token up, step, token down
    from ..generate.generate import TextGenerator
    r = TextGenerator(eng).benchmark_ids(prompt(ctx), steps)
    out["e2e_decode_tok_s"] = round(r["decode_tok_s"], 1)
    eng.cleanup()
    return out


def run(steps: int, warmup: int, sizes, sampler, models=("degedra", "hybrid", "hybrid-fp16attn")) -> dict:
    """models[0] is the one the headline value is of; the others stand beside it."""
    peaks = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "source": "fallback"}
    path = os.path.join(os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__)))), "MEASURED_PEAKS.json")
    if os.path.exists(path):
        peaks.update({k: v for k, v in json.load(open(path)).items() if k in peaks}, source="measured")
    res = {}
    sampler.start()
    for size in sizes:
        res[size] = {}
        for model in models:
            res[size][model] = measure(model, size, steps, warmup, peaks)
            torch.cuda.empty_cache()
    clocks = sampler.stop()
    first, main_model = sizes[-1], models[0]
    name = main_model.capitalize()
    dtype = "bf16 (hybrid: int4 weights, fp16 activations)" if "hybrid" in models else "bf16"
    return {
        "metric": f"decode tok/s (bs1), {name} {first} layers", "value": res[first][main_model]["decode_bs1_tok_s"], "unit": "tok/s",
        "n_gpus": 1, "steps": steps, "warmup": max(3, warmup), "ms_per_step": res[first][main_model]["decode_bs1_ms"],
        "higher_is_better": True, "scaling": "strong", "vs_baseline": None, "dtype": dtype,
        "data": "synthetic (random weights and token ids)", "impl": "ours", "clocks": clocks, "peaks": peaks,
        "config": {"model": name, "global_batch": 1, "seq_len": 512, "parallelism": "tp1", "vocab": VOCAB,
                   "sizes": {k: dict(zip(("width", "ff", "heads", "kv_heads", "dim", "ssd_heads", "window", "layers"), SIZES[k])) for k in sizes},
                   "l2": "inputs larger than L2 (weights of all layers per step)"},
        "results": res,
    }


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--model", default="degedra", choices=MODELS)
    ap.add_argument("--size", default="4k", choices=sorted(SIZES))
    ap.add_argument("--phase", default="decode", choices=["decode", "prefill"])
    ap.add_argument("--steps", type=int, default=2)
    ap.add_argument("--layers", type=int, default=0, help="fewer layers than the size has (0: all)")
    ap.add_argument("--ctx", type=int, default=512)
    a = ap.parse_args()
    if a.layers:
        SIZES[a.size] = SIZES[a.size][:-1] + (a.layers,)
    eng = make(a.model, a.size, max(2048, a.ctx) + 64, 1)
    ids = torch.randint(0, VOCAB, (a.ctx,), generator=torch.Generator().manual_seed(1)).tolist()
    eng.prefill_tokens(ids)
    for _ in range(a.steps):
        if a.phase == "decode":
            eng.decode_tokens(1, graph=False, collect=False)
        else:
            eng.reset(0)
            eng.prefill_tokens(ids)
    torch.cuda.synchronize()
    print("launches in the last step:", eng.launches_per_step())


if __name__ == "__main__":
    main()
