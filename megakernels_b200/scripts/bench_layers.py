"""Prefill and decode throughput of a layer-list model beside the presets of its width that are
closest to it.

Run through ``bench.py --layer-list dumalix-1b``.  Random bf16 weights drawn on the device; the
weights of one pass exceed L2, so no flush is needed between iterations.  Device times are CUDA
events on the launching stream.
"""

from __future__ import annotations

import json
from dataclasses import replace

import torch

from megakernels_b200.demos.latency.scheduler import LatencyScheduleOptions, pick_num_attention_partitions
from megakernels_b200.dispatch import make_generator
from megakernels_b200.hybrid import HybridConfig, HybridForCausalLM
from megakernels_b200.llama import LlamaForCausalLM
from megakernels_b200.model_types import ExtraModelConfig
from megakernels_b200.registry import family_of_preset

# the llama preset whose decode step is measured beside it, the layer-list preset whose prefill is
CLOSEST = {"torirax-1b": ("llama-1b", None), "torirax-8b": ("llama-8b", None),
           "dumalix-1b": ("llama-1b", "torirax-1b"), "dumalix-8b": ("llama-8b", "torirax-8b")}
ATTENDED = 4096  # position of the first decoded token


def matrix_params(cfg: HybridConfig, head: bool = True) -> int:
    """Entries of the matrices a token meets (once per run of its layer)."""
    n = cfg.vocab_size * cfg.width if head else 0
    for i, enters in cfg.runs:
        m, mlp = cfg.layers[i].mixer, cfg.layers[i].mlp
        n += (m.in_rows + m.out_features) * cfg.width + 2 * cfg.width**2 * enters
        if m.kind == "latent_attention":
            n += m.heads * (m.dim + m.vdim) * m.rank
        if mlp is not None:
            n += (mlp.up_rows + mlp.ff) * cfg.width
    return n


def visible_keys(m, position: int) -> int:
    if m.kind == "attention":
        return position % m.chunk + 1
    return min(position + 1, m.window + m.keep_first)


def decode_bytes(cfg: HybridConfig, position: int) -> int:
    """Weights once, the visible keys and values, the recurrent matrices read and written."""
    n = 2 * matrix_params(cfg)
    for s in cfg.run_layers:
        m = s.mixer
        if m.kind == "delta_rule":
            n += 8 * m.heads * m.dim * m.dim + 4 * m.inner * m.rank
        else:
            n += 2 * visible_keys(m, position) * m.key_elems
    return n


def prefill_flops(cfg: HybridConfig, tokens: int, portion: int = 2048) -> float:
    """Matrix products of the layers plus the attention over the keys that are seen."""
    f = 2.0 * tokens * matrix_params(cfg, head=False)
    at = range(0, tokens, 64)
    for s in cfg.run_layers:
        m = s.mixer
        if m.kind == "delta_rule":
            f += tokens * m.heads * (10.0 * m.dim * m.dim)
            continue
        keys = sum(visible_keys(m, i) for i in at) / max(1, len(at))
        pair = {"diff_attention": 2 * (2 * m.dim + 2 * m.vdim), "attention": 2 * (m.dim + m.vdim),
                "latent_attention": 2 * (m.dim + getattr(m, "rot_dim", 0) + m.vdim)}[m.kind]
        f += tokens * keys * m.heads * pair
    return f


def timed(fn, reps: int, warmup: int = 3) -> float:
    """Milliseconds per call."""
    for _ in range(warmup):
        fn()
    torch.cuda.synchronize()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record()
    for _ in range(reps):
        fn()
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) / reps


def decode_ms(gen, position: int, steps: int, warmup: int):
    """(kernel ms, whole step ms with the step replayed as a graph)."""
    device = gen.model.device
    ids = torch.randint(0, gen.model.config.vocab_size, (warmup + steps, 1, 1), generator=torch.Generator().manual_seed(3)).to(device)
    globs = gen.schedule.globs
    for i in range(warmup):
        gen.run(ids[i], pos_id=position + i)
    torch.cuda.synchronize()
    events = []
    for i in range(steps):
        if hasattr(globs, "hidden_states"):
            globs.hidden_states[:] = gen.model.model.embed_tokens.embed_tokens.weight[ids[warmup + i]].reshape(globs.hidden_states.shape)
            gen.fill()
            globs.pos_id = position + warmup + i
        else:
            gen._place(ids[warmup + i], position + warmup + i)
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        gen.last_call = gen.interpreter.interpret(globs)
        b.record()
        events.append((a, b))
    gen.check()
    kernel = sum(a.elapsed_time(b) for a, b in events) / steps
    gen.enable_cuda_graph(warmup_pos=position)
    k = iter(range(10**9))
    step = timed(lambda: gen.run(ids[next(k) % len(ids)], pos_id=position + 5), steps, warmup)
    gen.check()
    return kernel, step


def hybrid_generator(cfg, max_len, portion=2048):
    extra = ExtraModelConfig(max_len_override=max_len, prefill_portion=portion)
    model = HybridForCausalLM.from_random(cfg, extra, draw_on="device")
    return make_generator(model)


def prefill_ms(gen, n: int, reps: int) -> float:
    toks = torch.randint(0, gen.model.config.vocab_size, (n,), generator=torch.Generator().manual_seed(1), device="cpu").to(gen.model.device)
    ms = timed(lambda: gen.feed(toks, 0, [n - 1]), reps)
    gen.check()
    return ms


def layer_parts(cfg: HybridConfig, tokens: int) -> dict:
    """Milliseconds of one layer of each kind at ``tokens`` tokens: stacks of eight, minus stacks of
    two (embedding, head of one row)."""
    stacks = {}
    for layer in cfg.layers:
        stacks.setdefault(layer.mixer.kind, replace(layer, mlp=None))
        if layer.mlp is not None:
            stacks.setdefault(layer.mixer.kind + "+mlp", layer)
    out = {}
    for name, layer in stacks.items():
        if getattr(layer.mixer, "kv_from", None) is not None:
            continue
        both = []
        for k in (2, 8):
            gen = hybrid_generator(replace(cfg, layers=(layer,) * k, loop=None, vocab_size=1024), tokens)
            both.append(prefill_ms(gen, tokens, 5))
            del gen
        out[name] = round((both[1] - both[0]) / 6, 4)
    return out


def prefill_table(gen, cfg, hbm: float, tflops: float) -> dict:
    out = {}
    for n in (64, 512, 2048, 8192):
        ms = prefill_ms(gen, n, 5)
        flops = prefill_flops(cfg, n)
        floor = max(flops / (tflops * 1e9), 2e-6 * matrix_params(cfg, False) / hbm)
        out[n] = {"ms": round(ms, 4), "tokens_per_s": round(n / ms * 1e3), "tflops": round(flops / ms * 1e-9, 1),
                  "of_roofline": round(floor / ms, 3)}
    return out


def decode_row(kernel: float, step: float, nbytes: int, hbm: float) -> dict:
    return {"kernel_ms": round(kernel, 4), "step_ms": round(step, 4), "bytes": nbytes, "gbs": round(nbytes / kernel * 1e-6),
            "of_roofline": round(nbytes / kernel * 1e-6 / hbm, 3)}


def run(args, sampler_cls, peaks: dict) -> None:
    hbm, tflops = peaks["hbm_gbs"], peaks["bf16_tflops_sustained"]
    torch.cuda.set_device(0)
    steps, warmup = min(args.steps, 128), max(3, args.warmup)
    cfg = family_of_preset(args.layer_list).presets[args.layer_list]()
    close, close_list = CLOSEST[args.layer_list]
    max_len = ATTENDED + steps + warmup + 16
    sampler = sampler_cls(0)
    sampler.start()
    with torch.inference_mode():
        gen = hybrid_generator(cfg, max(max_len, 8192))
        line = {"metric": "layer_list_decode_tokens_per_s", "unit": "tokens/s", "n_gpus": 1, "higher_is_better": True,
                "dtype": "bf16", "data": "synthetic (random weights)", "steps": steps, "warmup": warmup,
                "config": {"model": args.layer_list, "layers": cfg.num_hidden_layers, "layer_runs": len(cfg.runs), "width": cfg.width,
                           "position": ATTENDED, "l2": "weights of a pass exceed L2"}}
        line["prefill"] = prefill_table(gen, cfg, hbm, tflops)
        kernel, step = decode_ms(gen, ATTENDED, steps, warmup)
        line.update(value=1e3 / step, ms_per_step=step, decode=decode_row(kernel, step, decode_bytes(cfg, ATTENDED), hbm))
        del gen
        torch.cuda.empty_cache()
        line["prefill_ms_per_layer_2048"] = layer_parts(cfg, 2048)
        torch.cuda.empty_cache()

        lcfg = family_of_preset(close).presets[close]()
        extra = ExtraModelConfig(interleave_rope=True, max_len_override=max_len)
        model = LlamaForCausalLM.from_random(lcfg, extra, draw_on="device")
        n_part = pick_num_attention_partitions(ATTENDED, steps, model.device, model.num_kv_heads(), min_chunk_size=128)
        gen = make_generator(model, LatencyScheduleOptions(num_attention_partitions=n_part, coalesce_o_proj=True,
                                                           merge_in_last_partial=True))
        kernel, step = decode_ms(gen, ATTENDED, steps, warmup)
        H, I, D = lcfg.hidden_size, lcfg.intermediate_size, lcfg.head_dim
        Hq, Hk, L = lcfg.num_attention_heads, lcfg.num_key_value_heads, lcfg.num_hidden_layers
        nbytes = 2 * (L * ((Hq + 2 * Hk) * D * H + H * Hq * D + 3 * I * H) + lcfg.vocab_size * H) + 4 * ATTENDED * Hk * D * L
        line["closest"] = {"model": close, "layers": L, "decode": decode_row(kernel, step, nbytes, hbm),
                           "prefill_tokens_per_s": round(1e3 / step)}  # its prompts go through the decode kernel token by token
        if close_list:
            del gen, model
            torch.cuda.empty_cache()
            tcfg = family_of_preset(close_list).presets[close_list]()
            gen = hybrid_generator(tcfg, max(max_len, 8192))
            line["closest_layer_list"] = {"model": close_list, "layers": tcfg.num_hidden_layers,
                                          "prefill": prefill_table(gen, tcfg, hbm, tflops)}
            kernel, step = decode_ms(gen, ATTENDED, steps, warmup)
            line["closest_layer_list"]["decode"] = decode_row(kernel, step, decode_bytes(tcfg, ATTENDED), hbm)
            del gen
            torch.cuda.empty_cache()
            line["closest_layer_list"]["prefill_ms_per_layer_2048"] = layer_parts(tcfg, 2048)
    line["clocks"] = sampler.stop()
    print(json.dumps(line), flush=True)
