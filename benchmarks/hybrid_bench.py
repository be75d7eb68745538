"""Prefill and decode throughput of a model with listed layers beside the closest model of this package at equal sizes (`bench.py --model
tuvutar`, `--model filasun`, `--model sapanex`, `--model gipozen`).

Tuvutar: the closest model is Kimi-K3's layer stack without experts and with a plain residual: latent attention between delta-rule layers and
dense gated MLPs in bf16 (its delta layers decay per key channel, its latent layers carry an output gate).  Both get the same width,
head counts and sizes, layer order, feed-forward in every layer, vocabulary, bf16 weights and caches, random weights, synthetic
prompts, and run through the same engine.

Filasun: the closest model is the dense Qwen3.5 stack (grouped-query attention and gated delta-net layers, bf16, one residual).  A parallel layer
(attention, decayed linear attention, a feed-forward of width ff) stands against an attention layer and a delta-net layer with a feed-forward of
ff / 2 each, a Mamba-2 layer with a feed-forward of ff / 2 against a delta-net layer: the same head counts, head sizes, state sizes per layer,
feed-forward weights, width and vocabulary; the attention window is the longest context, so that both read the same keys.

Sapanex: the closest model is the dense Qwen3.5 stack again, an attention layer after every three delta layers in both, the same head counts, head
sizes, state sizes, width and vocabulary; a feed-forward of two matrices of 3 ff / 2 stands against a gated one of three of ff.  Sapanex's attention
layers see a window of 1024 tokens and blocks of 16, Qwen3.5's the whole context.

Gipozen: the closest model is the Qwen3.5-MoE stack with attention in every layer: grouped-query attention with an output gate against two maps of half the
head size over the same values (equal projections and rows), dense and mixture layers in turn, the same experts, shared expert behind a gate, head
counts, width and vocabulary; a dense feed-forward of two matrices of 3 ff / 2 stands against a gated one of three of ff.  Gipozen's layers see a window
of 4096 tokens behind 16 kept ones, route over 4 identity experts more, and keep their own rows (`kv_from` is left out); Qwen3.5's see the whole context.

`prefill` is the device time of the scheduler's prompt steps (CUDA events around
LLM.step), `decode` the replay of one decode step on resident inputs (graph + lm_head + sampling)."""
from __future__ import annotations

import json


def sizes(name):
    return {"small": dict(width=2048, heads=16, groups=4, ff=6144, vocab=32768), "medium": dict(width=4096, heads=32, groups=2, ff=12288, vocab=65536),
            "large": dict(width=7168, heads=56, groups=1, ff=18432, vocab=65536)}[name]


def tuvutar_model(width, heads, groups, ff, vocab):
    from nanoengine_b200.models.config import ModelConfig, _delta_spec, _latent_spec
    layers = []
    for _ in range(groups):
        layers.append(_latent_spec(heads, 128, 64, 128, 512, ff, base=1e6))
        layers += [_delta_spec(heads, heads, 128, 128, 4, ff=ff) for _ in range(3)]
    return ModelConfig.from_dict({"architecture": "Tuvutar", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "layers": layers})


def kimi_model(width, heads, groups, ff, vocab):
    from nanoengine_b200.models.config import tiny_kimi_k3
    return tiny_kimi_k3(vocab_size=vocab, hidden_size=width, num_hidden_layers=4 * groups, num_attention_heads=heads, num_key_value_heads=heads,
                        q_lora_rank=None, kv_lora_rank=512, qk_nope_head_dim=128, qk_rope_head_dim=64, v_head_dim=128, intermediate_size=ff,
                        n_routed_experts=0, n_shared_experts=0, layer_types=["full_attention", "linear_attention", "linear_attention", "linear_attention"] * groups,
                        linear_num_key_heads=heads, linear_num_value_heads=heads, linear_key_head_dim=128, linear_value_head_dim=128, attn_res_block_size=0,
                        routed_expert_hidden_size=0, max_position_embeddings=16384)


def filasun_model(width, heads, groups, ff, vocab):
    from nanoengine_b200.models.config import ModelConfig, _mamba2_spec, _parallel_spec
    layers = []
    for _ in range(groups):
        layers += [_parallel_spec(heads, heads // 4, 128, 128, 16384, heads, 128, 128, ff=ff) for _ in range(2)]
        layers.append(_mamba2_spec(2 * heads, 64, 128, max(1, heads // 8), 4, max(1, heads // 8), ff=ff // 2))
    return ModelConfig.from_dict({"architecture": "Filasun", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "streams": 2, "logit_softcap": 30.0,
                                  "max_positions": 16384, "layers": layers})


def qwen_model(width, heads, groups, ff, vocab):
    from nanoengine_b200.models.config import tiny_qwen3_5
    kinds = (["full_attention", "linear_attention"] * 2 + ["linear_attention"]) * groups
    return tiny_qwen3_5(vocab_size=vocab, hidden_size=width, num_hidden_layers=len(kinds), layer_types=kinds, num_attention_heads=heads, num_key_value_heads=heads // 4,
                        head_dim=128, intermediate_size=ff // 2, linear_num_key_heads=heads, linear_num_value_heads=heads, linear_key_head_dim=128,
                        linear_value_head_dim=128, max_position_embeddings=16384)


def sapanex_model(width, heads, groups, ff, vocab):
    from nanoengine_b200.models.config import ModelConfig, _general_delta_spec, _pooled_attention_spec
    yarn = {"factor": 4.0, "original": 8192, "fast": 32.0, "slow": 1.0}
    layers = []
    for _ in range(groups):
        layers += [_general_delta_spec(heads, 128, 64, ff=3 * ff // 2) for _ in range(3)]
        layers.append(_pooled_attention_spec(heads, heads // 4, 128, 128, 1024, 16, 64, ff=3 * ff // 2, base=1e6, scaling=yarn))
    return ModelConfig.from_dict({"architecture": "Sapanex", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "embedding": {"scale": 8.0}, "postln_alpha": 2.0,
                                  "max_position_embeddings": 16384, "layers": layers})


def qwen_3to1_model(width, heads, groups, ff, vocab):
    from nanoengine_b200.models.config import tiny_qwen3_5
    kinds = (["linear_attention"] * 3 + ["full_attention"]) * groups
    return tiny_qwen3_5(vocab_size=vocab, hidden_size=width, num_hidden_layers=len(kinds), layer_types=kinds, num_attention_heads=heads, num_key_value_heads=heads // 4,
                        head_dim=128, intermediate_size=ff, linear_num_key_heads=heads, linear_num_value_heads=heads, linear_key_head_dim=128,
                        linear_value_head_dim=128, max_position_embeddings=16384)


def gipozen_model(width, heads, groups, ff, vocab):
    from nanoengine_b200.models.config import ModelConfig, _differential_spec
    layers = []
    for i in range(2 * groups):
        layers += [_differential_spec(heads, heads // 4, 64, 128, 4096, 16, 4, 0.4, ff=3 * ff // 2),
                   _differential_spec(heads, heads // 4, 64, 128, 4096, 16, 4, 0.4, experts=(64, 4, 8, ff // 8, ff // 4, 7.0))]
    return ModelConfig.from_dict({"architecture": "Gipozen", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "logit_scale": 1.0, "layers": layers})


def qwen_moe_model(width, heads, groups, ff, vocab):
    from nanoengine_b200.models.config import tiny_qwen3_5
    n = 4 * groups
    return tiny_qwen3_5(True, vocab_size=vocab, hidden_size=width, num_hidden_layers=n, layer_types=["full_attention"] * n, linear_num_value_heads=0,
                        linear_num_key_heads=0, num_attention_heads=heads, num_key_value_heads=heads // 4, head_dim=128, intermediate_size=ff, n_routed_experts=64,
                        num_experts_per_tok=8, moe_intermediate_size=ff // 8, shared_expert_intermediate_size=ff // 4, mlp_layer_types=["dense", "sparse"] * (n // 2),
                        max_position_embeddings=16384)


DESIGNS = {"gipozen": ("Gipozen", gipozen_model, "qwen3_5_moe_stack", qwen_moe_model),
           "sapanex": ("Sapanex", sapanex_model, "qwen3_5_stack", qwen_3to1_model),
           "tuvutar": ("Tuvutar", tuvutar_model, "kimi_k3_stack", kimi_model),
           "filasun": ("Filasun", filasun_model, "qwen3_5_stack", qwen_model)}


def measure(mc, seqs, prompt, steps, warmup, seed=0):
    import torch
    from nanoengine_b200 import Config, LLM, SamplingParams
    new = warmup + steps + 8
    pages = (prompt + new + 63) // 64 + 1
    llm = LLM(Config(model="bench", model_config=mc, dummy_weight=True, dtype="bfloat16", device="cuda", max_num_seqs=seqs, max_num_batched_tokens=8192,
                     max_model_len=prompt + new + 64, num_kvcache_blocks=seqs * pages + 8, enable_prefix_caching=False, cuda_graph_max_bs=seqs, seed=seed,
                     executor_backend="inproc", status_log_interval_s=0))
    g = torch.Generator().manual_seed(1)
    sp = SamplingParams(temperature=0.0, max_tokens=new, ignore_eos=True)
    for _ in range(seqs):
        llm.add_request(torch.randint(0, mc.vocab_size, (prompt,), generator=g).tolist(), sp)
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    sch, ms, toks, prev, n = llm.engine.scheduler, 0.0, 0, 0, 0
    while sch.num_waiting() > 0 or sch.num_prefilling(0) > 0:
        torch.cuda.synchronize()
        e0.record()
        llm.step()
        e1.record()
        e1.synchronize()
        done = sch.metrics_summary()["prompt_tokens"]
        if n >= 3:                                       # the first steps warm up
            ms += e0.elapsed_time(e1)
            toks += done - prev
        prev, n = done, n + 1
    for _ in range(max(3, warmup)):
        llm.step()
    runner = llm.engine.executor.runner
    same, launches, step = runner.graph_step_equals_eager(), runner.count_step_launches(), runner.make_resident_decode_step()
    for _ in range(3):
        step()
    torch.cuda.synchronize()
    e0.record()
    for _ in range(steps):
        step()
    e1.record()
    e1.synchronize()
    dev = e0.elapsed_time(e1) / steps
    llm.shutdown()
    del llm, runner, step
    import gc
    gc.collect()
    torch.cuda.empty_cache()
    return {"prefill_tok_s": round(toks / ms * 1e3, 1) if ms else None, "decode_tok_s": round(seqs / dev * 1e3, 1), "decode_ms": round(dev, 3),
            "launches_per_step": launches, "graph_equals_eager": same}


def main(args):
    import threading
    import torch
    import bench
    torch.cuda.set_device(0)
    title, own, closest_name, closest = DESIGNS[args.model]
    stop, samples = threading.Event(), []
    th = threading.Thread(target=bench._clock_sampler, args=(stop, samples), daemon=True)
    th.start()
    rows = []
    for name in args.sizes.split(","):
        s = sizes(name)
        for seqs, prompt in ((128, 2048), (16, 8192)):
            rows.append({"size": name, **s, "seqs": seqs, "prompt": prompt, args.model: measure(own(**s), seqs, prompt, args.steps, args.warmup),
                         closest_name: measure(closest(**s), seqs, prompt, args.steps, args.warmup) if not args.skip_closest else None})
    stop.set()
    th.join(timeout=2)
    first = rows[0][args.model]
    print(json.dumps({"metric": title + " decode out tok/s at the first size (prefill and the closest model in rows)", "value": first["decode_tok_s"],
                      "unit": "tokens/s", "n_gpus": 1, "steps": args.steps, "warmup": args.warmup, "ms_per_step": first["decode_ms"], "higher_is_better": True,
                      "vs_baseline": None, "dtype": "bf16", "data": "synthetic uniform-random token ids, random-init weights",
                      "config": {"model": args.model, "l2": "weights and states streamed every step exceed L2; no flush"}, "rows": rows,
                      "clocks": bench._summarise_clocks(samples), "impl": "ours"}))
    return 0
