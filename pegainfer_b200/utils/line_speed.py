"""Throughput of a model line beside its closest neighbour at equal sizes, random weights: ``bench.py --line-speed LINE``.

* ``nemipel`` beside the Qwen3.5 line (linear-attention layers with recurrent state interleaved with paged attention).
* ``vekalorn`` beside the DeepSeek-V2 line (latent attention and mixture of experts in every layer): the same heads, latents
  and number of experts, and expert widths that give both the same expert weights (two matrices against three).
* ``zeripel`` beside the Kimi-K3 line (a recurrence with a decay per key channel, latent attention and sigmoid-routed experts
  with a shared one): the same layer order, heads, latents and expert weights; its full-attention layers stand in for both
  kinds of Zeripel attention, and its routed experts work behind two further projections of the stream's width.
* ``nonetar`` beside the Nemipel line (soft-capped attention and linear attention with one decay per head, f32 stream): the same
  layer order, heads, state sizes and feed-forward weights.  A Nonetar attention layer also has a recurrent block of the
  stream's width (three more square matrices and its gates), every layer four copies of the stream, its attention a window.

Device time (CUDA events) of whole steps of the executor: prefill steps of the given batches, and replays of the decode graph
at a batch and context.  Weights and state are larger than L2 at every size, so no flush is needed.
"""
from __future__ import annotations

import json
from dataclasses import dataclass, replace
from typing import Callable


@dataclass(frozen=True)
class Comparison:
    other: str
    names: tuple  # of the numbers that make a size
    sizes: tuple  # (name, numbers)
    prefill: tuple  # (sequences, tokens)
    decode: tuple  # (sequences, context)
    configs: Callable
    fixed: tuple = ()


def _nemipel_configs(width, ff, heads, kv_heads, lin_heads, periods=4, vocab=32768):
    from ..config import PRESETS, _nemipel

    a = _nemipel(width, vocab, ff, heads, kv_heads, 128, lin_heads, 128, 128, periods, lightning_ff=ff, max_position=16384)
    b = replace(PRESETS["qwen35-8b-shape"], vocab_size=vocab, hidden_size=width, num_layers=3 * periods, num_q_heads=heads, num_kv_heads=kv_heads, intermediate_size=ff,
                layer_types=("linear_attention", "full_attention", "linear_attention") * periods, gdn_num_k_heads=lin_heads // 2, gdn_num_v_heads=lin_heads, max_position=16384)
    return {"nemipel": a, "qwen35": b}


def _vekalorn_configs(width, heads, q_rank, window, experts, top, ff, periods, vocab=32768):
    from ..config import PRESETS, ExpertsSpec, _vekalorn

    a = _vekalorn(width, vocab, heads, q_rank, 512, 128, 64, 128, window, ExpertsSpec(experts, top, ff, 8, 4), periods, max_position=16384)
    b = replace(PRESETS["dsv2-lite"], vocab_size=vocab, hidden_size=width, num_layers=3 * periods, num_q_heads=heads, num_kv_heads=heads, q_lora_rank=q_rank, n_routed_experts=experts, n_shared_experts=0,
                num_experts_per_tok=top, moe_intermediate_size=ff * 2 // 3, first_k_dense_replace=0, n_group=8, topk_group=4, max_position=16384)
    return {"vekalorn": a, "deepseek_v2": b}


def _zeripel_configs(width, ff, heads, kv_heads, experts, top, expert_ff, shared_ff, periods, vocab=32768):
    from ..config import PRESETS, _zeripel, _zeripel_experts

    a = _zeripel(width, vocab, ff, heads, kv_heads, 128, 512, 128, 64, 128, heads, 128, 128, _zeripel_experts(experts, top, expert_ff, shared_ff, 2.5), periods, max_position=16384)
    b = replace(PRESETS["kimi-k3"], vocab_size=vocab, hidden_size=width, num_layers=4 * periods, layer_types=("full_attention", "full_attention", "linear_attention", "full_attention") * periods,
                num_q_heads=heads, num_kv_heads=heads, intermediate_size=ff, n_routed_experts=experts, num_experts_per_tok=top, n_shared_experts=shared_ff // expert_ff, moe_intermediate_size=expert_ff,
                latent_moe_dim=width, attn_res_block=4, expert_quant="bf16", max_position=16384)
    return {"zeripel": a, "kimi_k3": b}


def _nonetar_configs(width, ff, heads, kv_heads, window, ssd_heads, periods, vocab=32768):
    from ..config import MixerSpec, LayerSpec, _nemipel, _nonetar, _nonetar_parallel, _nonetar_ssd

    a = _nonetar(width, vocab, ff * 3 // 2, 4, _nonetar_parallel(heads, kv_heads, 128, 128, 128 ** -0.5, 50.0, window, width, width // 256, 4, (1.0, 0.5)), _nonetar_ssd(ssd_heads, 64, 128, 8, 8, 4), periods,
                 max_position=16384)
    b = _nemipel(width, vocab, ff, heads, kv_heads, 128, heads, 128, 128, periods, lightning_ff=ff, max_position=16384)
    attn, lin = MixerSpec("attention", heads, 128, 128, kv_heads=kv_heads, scale=128 ** -0.5, softcap=50.0), MixerSpec("lightning", ssd_heads // 2, 128, 128, decay=(0.98,) * (ssd_heads // 2))
    return {"nonetar": a, "nemipel": replace(b, layer_specs=tuple(LayerSpec(m, ff) for _ in range(periods) for m in (attn, attn, lin)))}


LINES = {
    "nemipel": Comparison("qwen35", ("width", "ff", "heads", "kv_heads", "recurrent_heads"), (("2048", (2048, 6144, 16, 8, 16)), ("4096", (4096, 12288, 32, 8, 32)), ("5120", (5120, 17408, 40, 8, 40))),
                          ((1, 4096), (8, 1024)), ((64, 1024), (8, 1024), (1, 1024)), _nemipel_configs, (("layers", 12), ("head_dim", 128))),
    "vekalorn": Comparison("deepseek_v2", ("width", "heads", "q_rank", "window", "experts", "top", "ff", "periods"),
                           (("2048", (2048, 16, 1536, 1024, 64, 6, 2112, 4)), ("4096", (4096, 32, 1536, 1024, 32, 4, 3072, 2)), ("7168", (7168, 64, 1536, 1024, 16, 4, 3072, 2))),
                           ((1, 4096), (8, 1024)), ((64, 1024), (16, 8192), (8, 1024), (1, 1024)), _vekalorn_configs,
                           (("kv_rank", 512), ("dim", 128), ("rot_dim", 64), ("vdim", 128), ("layers_per_period", "1 full + 2 windowed"))),
    "zeripel": Comparison("kimi_k3", ("width", "ff", "heads", "kv_heads", "experts", "top", "expert_ff", "shared_ff", "periods"),
                          (("2048", (2048, 8192, 16, 4, 64, 6, 1408, 2816, 3)), ("4096", (4096, 12288, 32, 8, 32, 4, 2048, 4096, 2)), ("7168", (7168, 18432, 64, 8, 16, 4, 2048, 2048, 2))),
                          ((1, 4096), (8, 1024)), ((64, 1024), (16, 8192), (8, 1024), (1, 1024)), _zeripel_configs,
                          (("kv_rank", 512), ("dim", 128), ("rot_dim", 64), ("layers_per_period", "latent, latent over the same cache, WKV, attention"))),
    "nonetar": Comparison("nemipel", ("width", "ff", "heads", "kv_heads", "window", "ssd_heads", "periods"),
                          (("2048", (2048, 6144, 16, 8, 1024, 64, 4)), ("4096", (4096, 12288, 32, 8, 2048, 128, 3)), ("5120", (5120, 16384, 40, 8, 4096, 160, 2))),
                          ((1, 4096), (8, 1024), (1, 16384)), ((64, 1024), (16, 8192), (8, 1024), (1, 1024)), _nonetar_configs,
                          (("dim", 128), ("streams", 4), ("layers_per_period", "2 attention (Nonetar: beside a recurrent block), 1 state-space / lightning"))),
}


def _timed(fn, n, warmup):
    import torch

    for _ in range(warmup):
        fn()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    torch.cuda.synchronize()
    e0.record()
    for _ in range(n):
        fn()
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) / n


def measure(cmp: Comparison, mcfg, steps: int, warmup: int, device="cuda:0") -> dict:
    import torch

    from ..config import EngineConfig
    from ..engine.build import build_engine
    from ..kv.request_kv import KvView
    from ..sched.executor import SeqStep, build_meta

    page, out = 16, {}
    longest = max(max(n for _, n in cmp.prefill), max(n for _, n in cmp.decode) + steps)
    blocks = max(n * ((length + page - 1) // page + 1) for n, length in cmp.prefill + cmp.decode) + 8
    eng = build_engine(EngineConfig(num_kv_blocks=blocks, max_decode_batch=64, max_model_len=longest + page, no_prefix_cache=True), mcfg, device=device, dtype=torch.bfloat16, start=False)
    ex = eng.executor
    try:
        out["weight_gb"] = round(torch.cuda.memory_allocated(device) / 1e9, 2)

        def sequences(n, length, new):
            per = (length + page - 1) // page
            return [SeqStep(rid=i, input_tokens=[(7 * j + i) % mcfg.vocab_size for j in range(new)], start_pos=length - new, view=KvView(list(range(1 + i * per, 1 + (i + 1) * per)), length, page)) for i in range(n)]

        for n, length in cmp.prefill:
            seqs = sequences(n, length, length)
            ids, meta = build_meta(seqs, page, device)
            ex.prepare_meta(seqs, meta)
            last = torch.tensor([meta.h_q_indptr[i + 1] - 1 for i in range(n)], dtype=torch.int32, device=device)
            ms = _timed(lambda: ex.model.logits(ex.model.forward_hidden(ids, meta, ex.kv), last), 8, warmup)
            out[f"prefill_{n}x{length}_tok_s"] = round(n * length / ms * 1e3)
            for s in seqs:
                ex.release_request(s.rid)
        for n, ctx in cmp.decode:
            seqs = sequences(n, ctx, 1)
            ex._graphs.run(seqs)
            b = next(x for x in ex._graphs.buckets if x >= n)
            ms = _timed(ex._graphs.graphs[(b, True)].replay, steps, warmup)
            out[f"decode_{n}x{ctx}_ms"], out[f"decode_{n}x{ctx}_tok_s"] = round(ms, 3), round(n / ms * 1e3)
            for s in seqs:
                ex.release_request(s.rid)
        from ..ops import cuda as K

        assert K.read_status(device) == 0, "device status word is set"
    finally:
        eng.shutdown()
        ex._graphs.release()
    return out


def run(name: str, steps: int = 64, warmup: int = 8, sampler=None) -> int:
    import gc

    import torch

    cmp = LINES[name]
    for size, numbers in cmp.sizes:
        line = {"metric": f"prefill and decode tok/s, {name} line beside the {cmp.other} line", "size": size, "config": dict(zip(cmp.names, numbers), **dict(cmp.fixed)), "dtype": "bf16",
                "data": "random-init weights, synthetic tokens", "steps": steps, "warmup": warmup}
        if sampler is not None:
            sampler.start()
        for fam, cfg in cmp.configs(*numbers).items():
            line[fam] = measure(cmp, cfg, steps, warmup)
            gc.collect()
            torch.cuda.empty_cache()
        if sampler is not None:
            line["clocks"] = sampler.stop()
        line[f"{name}_over_{cmp.other}"] = {k[:-6]: round(line[name][k] / line[cmp.other][k], 3) for k in line[name] if k.endswith("_tok_s")}
        print(json.dumps(line), flush=True)
    return 0
