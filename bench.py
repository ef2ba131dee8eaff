"""Benchmark of the decode hot path: batch-1 Llama decode through the megakernel.

    python bench.py [--gpus N] [--steps K] [--warmup W] [--impl reference]
                    [--workload llama-3.1-8b|llama-3.2-1b|llama-3.1-70b] [--prefill P]

A step is one decoded token: embed the (teacher-forced, seeded) input token,
reset the barrier counters and residual accumulators, launch the megakernel
once, take the argmax.  At N=1 the workload is the Llama-3.1-8B-architecture
configuration (random-init bf16 weights, KV cache prefilled to 1024
positions).  At N>1 the SAME sequence is decoded tensor-parallel over the N
GPUs (column/row-split projections, KV heads split by rank, the all-reduce
after o-proj and down-proj inside the kernel over peer memory), so the curve
over N is a strong-scaling curve; ``--replicas`` runs N independent copies
instead (weak scaling, no data-path collective).

Rank 0 prints one JSON line.  ``value`` is tokens/s with all inputs resident in
HBM, timed with CUDA events around exactly K steps between barriers;
``e2e`` is the same metric with the token id coming from pinned host memory and
the produced token copied back to the host every step; ``roofline`` compares
the megakernel's average launch time against the measured HBM copy bandwidth;
``parity`` compares the logits of the first timed step (and, tensor parallel,
the ranks' residual streams with each other) with the CPU oracle, outside the
timed region; ``cpu_baseline`` times that oracle - the reference's torch decode
path restated - at full depth on the host cores for a few tokens.
``--impl reference`` times only that CPU path and prints the same kind of line.
"""

from __future__ import annotations

import argparse
import json
import os
import subprocess
import sys
import threading
import time
from pathlib import Path

ROOT = Path(__file__).resolve().parent
if str(ROOT) not in sys.path:
    sys.path.insert(0, str(ROOT))

import torch  # noqa: E402

METRIC = "batch1_decode_tokens_per_s"
UNIT = "tokens/s"
FALLBACK_HBM_GBS = 6650.0  # used when no measured copy bandwidth is on file (MEASURED_PEAKS.json)

# DRAM traffic of one megakernel launch relative to its algorithmic bytes, from an ncu capture
# of a 4-layer case (dram__bytes_read.sum + dram__bytes_write.sum over the algorithmic bytes);
# traffic grows in proportion to the layers streamed, so the full launch is scaled by the ratio.
NCU_TRAFFIC_RATIO = (2.8239e9 + 0.0368e9) / 2.8124e9

WORKLOADS = {
    # tp: shard the model over the ranks when N > 1 (False: replicas only)
    "llama-3.1-8b": dict(preset="llama_3_1_8b", prefill=1024, tp=True, parity_layers=0),
    "llama-3.2-1b": dict(preset="llama_3_2_1b", prefill=32, tp=False, parity_layers=0),
    # 139 GB of weights: the oracle check runs on the first layers only
    "llama-3.1-70b": dict(preset="llama_3_1_70b", prefill=2048, tp=True, parity_layers=4),
}


def parse_args():
    ap = argparse.ArgumentParser()
    ap.add_argument("--gpus", type=int, default=1)
    ap.add_argument("--steps", type=int, default=256)
    ap.add_argument("--warmup", type=int, default=16)
    ap.add_argument("--impl", default="ours", choices=["ours", "reference"])
    ap.add_argument("--workload", default="llama-3.1-8b", choices=sorted(WORKLOADS))
    ap.add_argument("--layers", type=int, default=0, help="override depth (profiling small cases)")
    ap.add_argument("--prefill", type=int, default=0)
    ap.add_argument("--sched", default="rr")
    ap.add_argument("--attn-partitions", type=int, default=0, help="0 = pick from the length")
    ap.add_argument("--no-coalesce-o-proj", action="store_true")
    ap.add_argument("--separate-reduction", action="store_true",
                    help="AttentionReduction instructions instead of the last partial of a KV head merging the rows")
    ap.add_argument("--cuda-graph", action="store_true",
                    help="replay one captured decode step per token instead of launching eagerly")
    ap.add_argument("--replicas", action="store_true",
                    help="N > 1: independent copies of the model instead of tensor parallelism")
    ap.add_argument("--tp-exchange", default="peer", choices=["peer", "nccl"],
                    help="tensor parallel: all-reduce inside the kernel over peer memory "
                         "(one launch per token) or NCCL between 2L+1 launches")
    ap.add_argument("--tp-chunks", type=int, default=0, help="chunks per in-kernel all-reduce (0 = H / 1024)")
    ap.add_argument("--batch", type=int, default=1,
                    help="independent sequences decoded per launch (2..8: the batched kernel; 9..64: its tcgen05 "
                         "build; each sequence gets a seeded random KV length in [256, 4096] unless --prefill is given)")
    ap.add_argument("--layer-list", default="", choices=["", "torirax-1b", "torirax-8b", "dumalix-1b", "dumalix-8b"],
                    help="instead of the llama workload: prefill and decode of a layer-list model, beside the presets "
                         "of its width that are closest to it (one GPU)")
    ap.add_argument("--no-cpu-baseline", action="store_true")
    ap.add_argument("--no-parity", action="store_true")
    ap.add_argument("--no-e2e", action="store_true")
    return ap.parse_args()


def model_config(args, layers: int = 0):
    from megakernels_b200.llama import LlamaConfig

    w = WORKLOADS[args.workload]
    depth = layers or args.layers
    overrides = {"num_hidden_layers": depth} if depth else {}
    cfg = getattr(LlamaConfig, w["preset"])(**overrides)
    prefill = args.prefill or w["prefill"]
    return cfg, prefill


def is_tensor_parallel(args, world: int) -> bool:
    return world > 1 and WORKLOADS[args.workload]["tp"] and not args.replicas


def sequence_lengths(args, prefill: int) -> list[int]:
    """KV length of every sequence: the workload's prefill, or (batched, no --prefill) seeded
    uniform lengths in [256, 4096]."""
    if args.batch > 1 and not args.prefill:
        return torch.randint(256, 4097, (args.batch,), generator=torch.Generator().manual_seed(4)).tolist()
    return [prefill] * args.batch


def workload_name(args, cfg, prefill: int, world: int) -> str:
    """The same string in both arms, so that their lines can be matched."""
    if args.batch > 1:
        lens = sequence_lengths(args, prefill)
        return (f"{args.workload} batched decode, {args.batch} independent sequences per launch, "
                f"{cfg.num_hidden_layers} layers, KV lengths {min(lens)}..{max(lens)} (mean {sum(lens) // len(lens)}), "
                "teacher-forced")
    name = f"{args.workload} batch-1 decode, {cfg.num_hidden_layers} layers, KV prefill {prefill}, teacher-forced"
    if is_tensor_parallel(args, world):
        how = "in-kernel all-reduce over peer memory" if args.tp_exchange == "peer" else "NCCL all-reduce"
        name += f", tensor parallel over {world} GPUs ({how} after o-proj and down-proj)"
    elif world > 1:
        name += f", {world} independent replicas"
    return name


def algorithmic_bytes_per_token(cfg, seq_len: int, tp: int = 1) -> dict:
    """Bytes one GPU must move per decoded token: every bf16 matrix of its shard once
    (layers split over ``tp`` ranks, LM head replicated), norms, KV read + append."""
    H, I, L, D = cfg.hidden_size, cfg.intermediate_size, cfg.num_hidden_layers, cfg.head_dim
    Hq, Hkv, V = cfg.num_attention_heads, cfg.num_key_value_heads, cfg.vocab_size
    per_layer = ((Hq + 2 * Hkv) * D * H + H * Hq * D + 3 * I * H) * 2 // tp
    weights = L * per_layer + V * H * 2
    norms = (2 * L + 1) * H * 2
    kv_row = 2 * Hkv * D * 2 * L // tp
    return dict(weights=weights, norms=norms, kv=kv_row * seq_len + kv_row)


def hbm_peak():
    path = ROOT / "MEASURED_PEAKS.json"
    if path.exists():
        try:
            return float(json.loads(path.read_text())["hbm_gbs"]), "measured"
        except Exception:
            pass
    return FALLBACK_HBM_GBS, "fallback"


class ClockSampler:
    """Samples SM clocks and throttle reasons with nvidia-smi while the timed region runs."""

    FIELDS = (
        "clocks.sm,clocks.max.sm,clocks_event_reasons.hw_slowdown,"
        "clocks_event_reasons.hw_thermal_slowdown,clocks_event_reasons.sw_thermal_slowdown,"
        "clocks_event_reasons.sw_power_cap"
    )

    def __init__(self, index: int):
        self.index = index
        self.rows: list[list[str]] = []
        self.proc = None
        self.thread = None

    def start(self):
        try:
            self.proc = subprocess.Popen(
                ["nvidia-smi", f"--query-gpu={self.FIELDS}", "--format=csv,noheader,nounits",
                 "-lms", "100", "-i", str(self.index)],
                stdout=subprocess.PIPE, stderr=subprocess.DEVNULL, text=True,
            )
        except OSError:
            return
        self.thread = threading.Thread(target=self._read, daemon=True)
        self.thread.start()

    def _read(self):
        for line in self.proc.stdout:
            parts = [p.strip() for p in line.split(",")]
            if len(parts) >= 6:
                self.rows.append(parts)

    def stop(self) -> dict:
        if self.proc is None:
            return {"sm_mhz": None, "sm_max_mhz": None, "reasons": [], "samples": 0}
        time.sleep(0.15)
        self.proc.terminate()
        try:
            self.proc.wait(timeout=2)
        except subprocess.TimeoutExpired:
            self.proc.kill()
        rows = self.rows
        mhz = sorted(float(r[0]) for r in rows if r[0].replace(".", "").isdigit())
        names = ["hw_slowdown", "hw_thermal_slowdown", "sw_thermal_slowdown", "sw_power_cap"]
        reasons = [n for i, n in enumerate(names) if any(r[2 + i].lower().startswith("active") for r in rows)]
        return {
            "sm_mhz": mhz[len(mhz) // 2] if mhz else None,
            "sm_max_mhz": float(rows[0][1]) if rows and rows[0][1].replace(".", "").isdigit() else None,
            "reasons": reasons,
            "samples": len(rows),
        }


# --------------------------------------------------------------------------- #
# CPU path (oracle port of the reference's torch decode step)
# --------------------------------------------------------------------------- #
def cpu_reference_model(cfg, max_len: int, source=None):
    """The oracle at full depth on the host.  ``source``: a model already on a GPU whose
    tensors are copied (same values as the kernel uses); else drawn here."""
    from megakernels_b200.llama import LlamaForCausalLM
    from megakernels_b200.model_types import ExtraModelConfig
    from oracle.llama_ref import TorchReferenceModel

    if source is not None:
        return TorchReferenceModel(source)
    extra = ExtraModelConfig(interleave_rope=True, max_len_override=max_len)
    if torch.cuda.is_available():
        # a seeded draw of 8e9 weights takes minutes on the host: draw on the GPU, copy down
        model = LlamaForCausalLM.from_random(cfg, extra, device="cuda:0", seed=0, draw_on="device")
        ref = TorchReferenceModel(model)
        del model
        torch.cuda.empty_cache()
        return ref
    return TorchReferenceModel(LlamaForCausalLM.from_random(cfg, extra, device="cpu", seed=0))


def time_cpu_path(ref, cfg, prefill: int, tokens: int, budget_s: float):
    """Time ``tokens`` decode steps of the oracle at KV length ``prefill`` (first one untimed)."""
    cores = os.cpu_count() or 1
    torch.set_num_threads(cores)
    ids = torch.randint(0, cfg.vocab_size, (tokens + 1,), generator=torch.Generator().manual_seed(3))
    per_token = []
    t_begin = time.perf_counter()
    for i in range(tokens + 1):
        t0 = time.perf_counter()
        ref.decode_token(int(ids[i]), prefill + i)
        if i > 0:  # the first token warms the thread pool and the page cache
            per_token.append(time.perf_counter() - t0)
        if time.perf_counter() - t_begin > budget_s and len(per_token) >= 2:
            break
    sec = sum(per_token) / len(per_token)
    return dict(
        value=1.0 / sec,
        unit=UNIT,
        cores=cores,
        kind="port",
        sample=(
            f"oracle/llama_ref.py (the reference's torch decode path restated) at full depth, "
            f"{cfg.num_hidden_layers} layers + LM head, {len(per_token)} tokens at KV length {prefill}"
        ),
    ), sec


def seeded_kv_prefix(ref, prefill: int):
    gen = torch.Generator().manual_seed(2)
    for c in (ref.k_cache, ref.v_cache):
        c[:, :, :prefill] = torch.randn(c[:, :, :prefill].shape, generator=gen).to(c.dtype)


def run_reference_arm(args):
    rank = int(os.environ.get("RANK", "0"))
    world = int(os.environ.get("WORLD_SIZE", "1"))
    if rank != 0:
        return
    cfg, prefill = model_config(args, WORLDS_CPU_DEPTH.get(args.workload, 0))
    full_cfg, _ = model_config(args)
    # every step is one decoded token of the workload; K + W tokens in total, bounded
    tokens = max(2, min(args.steps + args.warmup, 64))
    ref = cpu_reference_model(cfg, prefill + tokens + 2)
    seeded_kv_prefix(ref, prefill)
    base, sec = time_cpu_path(ref, cfg, prefill, tokens, budget_s=150.0)
    if cfg.num_hidden_layers != full_cfg.num_hidden_layers:
        # 70B does not fit the host: a reduced depth is timed and scaled, and labelled so
        scale = full_cfg.num_hidden_layers / cfg.num_hidden_layers
        sec *= scale
        base["value"] = 1.0 / sec
        base["sample"] += f"; layer time scaled by {scale:g} to {full_cfg.num_hidden_layers} layers (extrapolated)"
    line = {
        "impl": "reference",
        "metric": METRIC,
        "value": base["value"],
        "unit": UNIT,
        "n_gpus": args.gpus,
        "steps": args.steps,
        "warmup": args.warmup,
        "ms_per_step": sec * 1e3,
        "higher_is_better": True,
        "scaling": "strong" if is_tensor_parallel(args, world) else "weak",
        "vs_baseline": None,
        "dtype": "bf16",
        "data": "synthetic",
        "config": {"workload": workload_name(args, full_cfg, prefill, world),
                   "inputs": "larger than L2 (weights re-streamed from memory every step)"},
        "cpu_baseline": base,
        "e2e": {"value": base["value"], "unit": UNIT, "h2d_bytes_per_step": 0, "d2h_bytes_per_step": 0},
        "gpu_launches": 0,
    }
    print(json.dumps(line), flush=True)


# depth the CPU arm can hold in host memory (0 = full depth)
WORLDS_CPU_DEPTH = {"llama-3.1-70b": 8}


# --------------------------------------------------------------------------- #
# our arm
# --------------------------------------------------------------------------- #
def build_engine(args, device, tp_size=1, tp_rank=0, group=None, layers=0, steps=None):
    from megakernels_b200.demos.latency.scheduler import (
        LatencyScheduleOptions,
        pick_num_attention_partitions,
    )
    from megakernels_b200.dispatch import make_mk_interpreter, make_schedule_builder
    from megakernels_b200.generators import MK_Generator, TP_MK_Generator, TP_Peer_MK_Generator
    from megakernels_b200.llama import LlamaForCausalLM
    from megakernels_b200.model_types import ExtraModelConfig
    from megakernels_b200.scheduler import assign_to_sms, tensorize_instructions

    cfg, prefill = model_config(args, layers)
    steps = args.steps + args.warmup if steps is None else steps
    lens = sequence_lengths(args, prefill)
    total = max(lens) + steps + 8
    extra = ExtraModelConfig(
        interleave_rope=True, max_len_override=total, tp_size=tp_size, tp_rank=tp_rank, tp_group=group,
        max_batch_size=args.batch,
    )
    model = LlamaForCausalLM.from_random(cfg, extra, device=device, seed=0, draw_on="device")
    fill_kv_prefix(model, lens, cfg.num_key_value_heads, tp_size, tp_rank, device)
    n_part = args.attn_partitions or pick_num_attention_partitions(
        max(lens), steps, device, model.num_kv_heads(), min_chunk_size=128
    )
    if args.batch > 1:  # all sequences' partials of a layer should fit one wave of SMs
        n_part = args.attn_partitions or max(1, min(n_part, 148 // (args.batch * model.num_kv_heads())))
    peer = tp_size > 1 and args.tp_exchange == "peer"
    options = LatencyScheduleOptions(
        num_attention_partitions=n_part, coalesce_o_proj=not args.no_coalesce_o_proj,
        merge_in_last_partial=not args.separate_reduction,
        # chunks of 1024 elements: one pair per consumer thread, a multiple of the TP degree
        tp_all_reduce_chunks=(args.tp_chunks or max(tp_size, cfg.hidden_size // 1024)) if peer else 0,
        batch_size=args.batch,
    )
    schedule = make_schedule_builder("latency", options).build(model)
    schedule.globs.pos_id = prefill
    interp = make_mk_interpreter("latency")
    if peer:
        tensorize_instructions(schedule.globs, assign_to_sms(args.sched, schedule=schedule))
        generator = TP_Peer_MK_Generator(model, interp, schedule, group=group)
        launches_per_step = 1
    elif tp_size > 1:
        generator = TP_MK_Generator(model, interp, schedule, group=group, sched=args.sched)
        launches_per_step = len(generator.segments)
    else:
        tensorize_instructions(schedule.globs, assign_to_sms(args.sched, schedule=schedule))
        generator = MK_Generator(model, interp, schedule)
        launches_per_step = 1
    info = dict(attn_partitions=n_part, instructions=len(schedule.get_linear_instructions()),
                launches_per_step=launches_per_step)
    return cfg, prefill, model, schedule, generator, info


def fill_kv_prefix(model, lens, total_kv_heads, tp_size, tp_rank, device):
    """Seeded N(0,1) prefix of ``lens[b]`` positions for sequence b.  Every rank draws the full
    cache (same seed, same values) and keeps its own KV heads, so that the ranks together hold
    one sequence's cache."""
    gen = torch.Generator(device=device).manual_seed(2)
    per = total_kv_heads // tp_size
    for c in model.stacked_kv_cache:
        L, B, _, _, D = c.shape
        for layer in range(L):  # layer by layer: the full-width temporary stays small
            for b, n in enumerate(lens):
                full = torch.randn((n, total_kv_heads, D), generator=gen, device=device)
                c[layer, b, :n] = full[:, tp_rank * per : (tp_rank + 1) * per].to(c.dtype)


def check_parity(args, gen, schedule, model, cfg, prefill, token, pos, world, tp, rank, device):
    """Decode ``token`` at ``pos`` once more outside the timed region and compare the logits
    with the CPU oracle on the same weights and cache; returns (dict for the JSON line, oracle).

    Tensor parallel: rank 0 holds the oracle (the un-sharded model, rebuilt from the same seed)
    and all ranks compare their residual streams bit for bit.
    """
    import torch.distributed as dist

    from megakernels_b200.llama import LlamaForCausalLM
    from megakernels_b200.model_types import ExtraModelConfig
    from oracle.llama_ref import (
        COSINE_TOL, MARGIN_TOL, MAX_REL_TOL, TorchReferenceModel, depth_aware_tolerance, parity_metrics,
    )

    globs = schedule.globs
    torch.cuda.synchronize()
    # the cache as it is before the step (the step appends one row at `pos`)
    k_shard, v_shard = (c[:, :, : pos + 1].cpu() for c in model.stacked_kv_cache)
    out = gen.run(torch.tensor([[token]], device=device), pos_id=pos)
    gen.check()
    logits = globs.logits.cpu()
    result = {"checked": f"logits of the first timed step (token {token}, position {pos}) against the CPU oracle"}
    ref = None
    if tp:
        # the residual stream every rank ends up with: the tagged buffer of the in-kernel
        # exchange, or the accumulators the NCCL flavour sums between launches
        mine = globs.tp.hidden_tagged[:, 0].cpu() if globs.tp is not None else globs.residual_acc.cpu()
        streams = [None] * world
        dist.all_gather_object(streams, mine)
        caches = [None] * world
        dist.all_gather_object(caches, (k_shard, v_shard))
        result["ranks_bit_identical_residual"] = all(torch.equal(streams[0], s) for s in streams[1:])
    if rank == 0:
        if tp:
            extra = ExtraModelConfig(interleave_rope=True, max_len_override=pos + 2)
            full = LlamaForCausalLM.from_random(cfg, extra, device=device, seed=0, draw_on="device")
            ref = TorchReferenceModel(full)
            del full
            torch.cuda.empty_cache()
            k_full = torch.cat([c[0] for c in caches], dim=3)
            v_full = torch.cat([c[1] for c in caches], dim=3)
        else:
            ref = TorchReferenceModel(model, kv_len=pos + 2)
            k_full, v_full = k_shard, v_shard
        ref.k_cache[:, :, : pos + 1] = k_full
        ref.v_cache[:, :, : pos + 1] = v_full
        exact = ref.decode_token_exact(token, pos)  # float32 throughout: the oracle's own noise floor
        want = ref.decode_token(token, pos)
        m, floor, ours = parity_metrics(logits, want), parity_metrics(want, exact), parity_metrics(logits, exact)
        rel_tol, cos_tol, margin_tol = depth_aware_tolerance(want, exact)
        argmax_ok = m["argmax_equal"] or m["top2_margin"] <= MARGIN_TOL
        result.update(
            ok=bool(m["max_rel"] <= rel_tol and m["cosine"] >= cos_tol
                    and (m["argmax_equal"] or m["top2_margin"] <= margin_tol)
                    and result.get("ranks_bit_identical_residual", True)),
            meets_stated_tolerance=bool(m["max_rel"] <= MAX_REL_TOL and m["cosine"] >= COSINE_TOL and argmax_ok),
            max_rel=m["max_rel"], cosine=m["cosine"], argmax_equal=m["argmax_equal"],
            top2_margin=m["top2_margin"], fused_argmax_equals_torch=int(out) == int(logits.float().argmax()),
            oracle_vs_float32={"max_rel": floor["max_rel"], "cosine": floor["cosine"]},
            kernel_vs_float32={"max_rel": ours["max_rel"], "cosine": ours["cosine"]},
            tolerance=(f"stated: max_rel <= {MAX_REL_TOL}, cosine >= {COSINE_TOL}, argmax equal if margin > "
                       f"{MARGIN_TOL}; ok uses max_rel <= {rel_tol:.4g}, cosine >= {cos_tol:.6f}, margin > "
                       f"{margin_tol:.4g} = twice the bf16 oracle's own distance from the same step in float32 "
                       "(never below the stated values)"),
            layers=cfg.num_hidden_layers,
        )
    return result, ref


def check_parity_batched(gen, schedule, model, cfg, lens, tokens, step, device):
    """Batched launch: every sequence's logits against its own single-sequence oracle run."""
    from oracle.llama_ref import (
        COSINE_TOL, MARGIN_TOL, MAX_REL_TOL, TorchReferenceModel, depth_aware_tolerance, parity_metrics,
    )

    globs = schedule.globs
    torch.cuda.synchronize()
    pos = [n + step for n in lens]
    caches = {b: tuple(c[:, b : b + 1, : pos[b] + 2].cpu().clone() for c in model.stacked_kv_cache)
              for b in range(len(lens))}
    out = gen.run(tokens.view(-1, 1).to(device), pos_id=pos)
    gen.check()
    logits = globs.logits.cpu()
    ref = TorchReferenceModel(model, kv_len=8)
    worst = {"max_rel": 0.0, "cosine": 1.0}
    floor_worst = {"max_rel": 0.0, "cosine": 1.0}
    ok = literal = True
    # every sequence up to 8; beyond that a spread of 8 (each costs two full-depth oracle runs)
    checked = list(range(len(lens))) if len(lens) <= 8 else sorted({round(i * (len(lens) - 1) / 7) for i in range(8)})
    for b in checked:
        ref.k_cache, ref.v_cache = caches[b]
        exact = ref.decode_token_exact(int(tokens[b]), pos[b])
        want = ref.decode_token(int(tokens[b]), pos[b])
        m, floor = parity_metrics(logits[b], want), parity_metrics(want, exact)
        rel_tol, cos_tol, margin_tol = depth_aware_tolerance(want, exact)
        argmax_ok = m["argmax_equal"] or m["top2_margin"] <= MARGIN_TOL
        ok = (ok and m["max_rel"] <= rel_tol and m["cosine"] >= cos_tol
              and (m["argmax_equal"] or m["top2_margin"] <= margin_tol))
        literal = literal and m["max_rel"] <= MAX_REL_TOL and m["cosine"] >= COSINE_TOL and argmax_ok
        ok = ok and int(out[b]) == int(logits[b].float().argmax())
        worst = {"max_rel": max(worst["max_rel"], m["max_rel"]), "cosine": min(worst["cosine"], m["cosine"])}
        floor_worst = {"max_rel": max(floor_worst["max_rel"], floor["max_rel"]),
                       "cosine": min(floor_worst["cosine"], floor["cosine"])}
    return {
        "checked": f"logits of {len(checked)} of {len(lens)} sequences at the first timed step, each against its "
                   "own single-sequence run of the CPU oracle",
        "ok": bool(ok), "meets_stated_tolerance": bool(literal),
        "max_rel": worst["max_rel"], "cosine": worst["cosine"], "oracle_vs_float32": floor_worst,
        "tolerance": f"stated: max_rel <= {MAX_REL_TOL}, cosine >= {COSINE_TOL}; ok uses twice the bf16 oracle's own "
                     "distance from the same step in float32 (never below the stated values); worst sequence shown",
        "layers": cfg.num_hidden_layers,
    }, ref


def run_ours(args):
    rank = int(os.environ.get("RANK", "0"))
    world = int(os.environ.get("WORLD_SIZE", "1"))
    local_rank = int(os.environ.get("LOCAL_RANK", "0"))
    distributed = world > 1
    torch.cuda.set_device(local_rank)
    device = torch.device("cuda", local_rank)
    if distributed:
        import torch.distributed as dist

        os.environ.setdefault("NCCL_NVLS_ENABLE", "0")
        dist.init_process_group("nccl", device_id=device)

    def barrier():
        if distributed:
            dist.barrier()
        torch.cuda.synchronize()

    tp = is_tensor_parallel(args, world)
    if WORKLOADS[args.workload]["preset"] == "llama_3_1_70b" and world == 1 and not args.layers:
        raise SystemExit(f"{args.workload} does not fit one GPU at full depth: launch it on 2, 4 or 8 GPUs")
    K, W, B = args.steps, args.warmup, args.batch
    if B > 1 and (world > 1 or WORKLOADS[args.workload]["preset"] == "llama_3_1_70b"):
        raise SystemExit("--batch runs on one GPU (8B or 1B shape)")
    ids = torch.randint(0, 128256, (W + K, B), generator=torch.Generator().manual_seed(3))

    # ---- parity at reduced depth first, for workloads whose oracle does not fit the host ---- #
    parity = None
    parity_layers = WORKLOADS[args.workload]["parity_layers"] if not args.layers else 0
    if parity_layers and not args.no_parity:
        log(f"parity engine with {parity_layers} layers")
        cfg_s, prefill_s, model_s, sched_s, gen_s, _ = build_engine(
            args, device, tp_size=world if tp else 1, tp_rank=rank if tp else 0, layers=parity_layers, steps=8
        )
        parity, _ = check_parity(args, gen_s, sched_s, model_s, cfg_s, prefill_s, int(ids[0, 0]) % cfg_s.vocab_size,
                                 prefill_s, world, tp, rank, device)
        if hasattr(gen_s, "close"):
            gen_s.close()
        del model_s, sched_s, gen_s
        torch.cuda.empty_cache()

    log("building model and schedule")
    cfg, prefill, model, schedule, gen, info = build_engine(
        args, device, tp_size=world if tp else 1, tp_rank=rank if tp else 0
    )
    gen_holder = [gen]
    log(f"engine ready: {info}")
    ids = ids % cfg.vocab_size
    ids_dev = ids.to(device).view(W + K, B, 1)
    lens = sequence_lengths(args, prefill)

    def pos_at(step):  # position(s) of the token(s) decoded at `step`
        return prefill + step if B == 1 else [n + step for n in lens]

    # 2L+1 launches per token (NCCL exchange) are launch-bound without a graph
    use_graph = args.cuda_graph or (tp and args.tp_exchange == "nccl")

    # ---- warm-up ----------------------------------------------------------- #
    for i in range(min(W, 3)):
        gen.run(ids_dev[i], pos_id=pos_at(i))
    gen.check()
    log("eager warm-up done")
    if use_graph:
        gen.enable_cuda_graph(warmup_pos=prefill)
        log("graph captured")
    for i in range(W):
        gen.run(ids_dev[i], pos_id=pos_at(i))
    gen.check()

    # ---- parity of the first timed step, outside the timed region ---------- #
    ref = None
    if parity is None and not args.no_parity:
        if B > 1:
            parity, ref = check_parity_batched(gen, schedule, model, cfg, lens, ids[W], W, device)
        else:
            parity, ref = check_parity(args, gen, schedule, model, cfg, prefill, int(ids[W, 0]), prefill + W,
                                       world, tp, rank, device)
        log(f"parity: {parity}")

    # ---- device-resident timing: exactly K steps between barriers -------- #
    log("warm-up done, timing")
    sampler = ClockSampler(local_rank)
    start, end = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    launch_events = []
    interp = gen.interpreter
    globs = schedule.globs
    embed = model.model.embed_tokens.embed_tokens.weight
    barrier()
    log("barrier passed")
    sampler.start()
    torch.cuda.profiler.start()  # lets a profiler started with "profile from start off" see only the timed region
    start.record()
    if use_graph:
        for i in range(K):
            gen.run(ids_dev[W + i], pos_id=pos_at(W + i))
    else:
        for i in range(K):
            # the body of MK_Generator.run, with events around the kernel launch
            globs.hidden_states[:] = embed[ids_dev[W + i]].reshape(globs.hidden_states.shape)
            gen.fill()
            if B > 1:
                globs.pos_ids = pos_at(W + i)
            else:
                globs.pos_id = prefill + W + i
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            gen.last_call = interp.interpret(globs)
            e1.record()
            launch_events.append((e0, e1))
            if globs.tp is not None:
                globs.tp.epoch_device.add_(1)  # as TP_Peer_MK_Generator._step does
            gen._next_token()  # the kernel's own argmax word (torch.argmax if that is switched off)
    end.record()
    torch.cuda.profiler.stop()
    log("timed steps enqueued")
    barrier()
    log("timed steps finished")
    clocks = sampler.stop()
    gen.check()
    elapsed_ms = start.elapsed_time(end)
    if launch_events:
        kernel_ms = sum(a.elapsed_time(b) for a, b in launch_events) / K
        kernel_scope = "megakernel launch"
    else:
        # inside a graph the launches cannot be bracketed: the roofline covers the whole step
        kernel_ms = elapsed_ms / K
        kernel_scope = "whole decode step (graph replay" + (", incl. all-reduces)" if tp else ")")

    # ---- end to end: token id from pinned host memory, produced token back to host ---- #
    e2e = None
    if not args.no_e2e:
        host_in = torch.empty(B, dtype=torch.long).pin_memory()
        host_out = torch.empty(B, dtype=torch.long).pin_memory()
        dev_in = torch.empty(B, 1, dtype=torch.long, device=device)
        # re-decode the same positions: same work per step
        if not use_graph:
            # the public generator replays the whole step (embedding row, state reset, megakernel,
            # argmax) as one CUDA graph; the device-timed loop above stays eager so that each
            # megakernel launch can be bracketed by events
            gen.enable_cuda_graph(warmup_pos=prefill)
        for i in range(3):
            host_in.copy_(ids[W + i])
            dev_in.copy_(host_in.view(B, 1), non_blocking=True)
            host_out.copy_(gen.run(dev_in, pos_id=pos_at(W + i)).view(-1), non_blocking=True)
            torch.cuda.synchronize()
        barrier()
        t0 = time.perf_counter()
        step_s = []
        for i in range(K):
            host_in.copy_(ids[W + i])
            dev_in.copy_(host_in.view(B, 1), non_blocking=True)
            out = gen.run(dev_in, pos_id=pos_at(W + i))
            host_out.copy_(out.view(-1), non_blocking=True)
            torch.cuda.current_stream().synchronize()
            _ = int(host_out[0])
            step_s.append(time.perf_counter())
        torch.cuda.synchronize()
        e2e_s = time.perf_counter() - t0
        log("e2e per-step ms: " + " ".join(f"{(b - a) * 1e3:.2f}" for a, b in zip([t0] + step_s, step_s)))
        gen.check()
        e2e = e2e_s

    # ---- reduce over ranks ------------------------------------------------ #
    if distributed:
        t = torch.tensor([elapsed_ms, kernel_ms, e2e or 0.0], device=device, dtype=torch.float64)
        dist.all_reduce(t, op=dist.ReduceOp.MAX)
        elapsed_ms, kernel_ms, e2e_max = t.tolist()
        e2e = e2e_max if e2e is not None else None

    if rank == 0:
        peak, peak_kind = hbm_peak()
        mid = W + K // 2
        nbytes = algorithmic_bytes_per_token(cfg, lens[0] + mid, tp=world if tp else 1)
        # a batched launch streams the weights once and every sequence's own KV prefix
        nbytes["kv"] = sum(algorithmic_bytes_per_token(cfg, n + mid)["kv"] for n in lens) if B > 1 else nbytes["kv"]
        algo = sum(nbytes.values())
        achieved = algo / (kernel_ms * 1e-3) / 1e9
        replicas = B if B > 1 else (1 if tp else world)  # a tensor-parallel job decodes one sequence
        line = {
            "metric": METRIC if B == 1 else "batched_decode_tokens_per_s",
            "value": replicas * K / (elapsed_ms * 1e-3),
            "unit": UNIT,
            "n_gpus": world,
            "steps": K,
            "warmup": W,
            "ms_per_step": elapsed_ms / K,
            "higher_is_better": True,
            "scaling": "strong" if tp else "weak",
            "vs_baseline": None,
            "dtype": "bf16",
            "data": "synthetic",
            "config": {
                "workload": workload_name(args, cfg, prefill, world),
                "launch": "cuda graph replay" if use_graph else "eager",
                "e2e_launch": "cuda graph replay of the whole step",
                "inputs": "larger than L2 (weights re-streamed from HBM every step)",
                "sched": args.sched,
                **info,
            },
            "kernel_ms_per_launch": kernel_ms,
            "roofline_scope": kernel_scope,
            "roofline": {
                "bound": "hbm",
                "achieved": achieved,
                "peak": peak,
                "unit": "GB/s",
                "frac": achieved / peak,
                "peak_source": f"{peak_kind} copy bandwidth",
                "frac_of_nominal_8TBs": achieved / 8000.0,
                "weight_only_frac": (nbytes["weights"] / (kernel_ms * 1e-3) / 1e9) / peak,
                "kv_bytes_per_launch": nbytes["kv"],
                "algorithmic_bytes_per_launch": algo,  # per GPU and decoded token
                "traffic": algo * NCU_TRAFFIC_RATIO,
                "traffic_source": "ncu dram bytes of a 4-layer capture scaled to this launch",
            },
            "parity": parity,
            "clocks": clocks,
            "gpu_launches": world * K * info["launches_per_step"],
        }
        if e2e is not None:
            line["e2e"] = {
                "value": replicas * K / e2e,
                "unit": UNIT,
                "h2d_bytes_per_step": 8 * B,
                "d2h_bytes_per_step": 8 * B,
                "ms_per_step": e2e / K * 1e3,
            }
        if world == 1 and not args.no_cpu_baseline:
            if ref is None:
                ref = cpu_reference_model(cfg, prefill + 16, source=model)
            del model, schedule, gen
            gen_holder.clear()
            torch.cuda.empty_cache()
            if ref.k_cache.shape[2] < prefill + 12 or ref.k_cache.shape[1] != 1:
                ref.k_cache = torch.zeros(
                    (ref.k_cache.shape[0], 1, prefill + 12, *ref.k_cache.shape[3:]), dtype=ref.k_cache.dtype)
                ref.v_cache = torch.zeros_like(ref.k_cache)
                seeded_kv_prefix(ref, prefill)
            base, _ = time_cpu_path(ref, cfg, prefill, tokens=8, budget_s=25.0)
            line["cpu_baseline"] = base
        print(json.dumps(line), flush=True)
    if distributed:
        # Tear down in a fixed order: captured graphs hold NCCL kernels, and destroying the
        # communicator underneath them was seen to block at interpreter exit.
        dist.barrier()
        torch.cuda.synchronize()
        if gen_holder and getattr(gen_holder[0], "_graph", None) is not None:
            gen_holder[0]._graph = None
        sys.stdout.flush()
        sys.stderr.flush()
        os._exit(0)


def log(msg: str):
    """Progress lines on stderr when MKB_BENCH_VERBOSE is set (stdout carries only the JSON line)."""
    if os.environ.get("MKB_BENCH_VERBOSE"):
        print(f"[bench {time.strftime('%H:%M:%S')} rank {os.environ.get('RANK', '0')}] {msg}",
              file=sys.stderr, flush=True)


def main():
    args = parse_args()
    if args.layer_list:
        from megakernels_b200.scripts import bench_layers

        peaks = {"hbm_gbs": FALLBACK_HBM_GBS, "bf16_tflops_sustained": 1400.0}
        path = ROOT / "MEASURED_PEAKS.json"
        if path.exists():
            peaks.update({k: v for k, v in json.loads(path.read_text()).items() if k in peaks})
        bench_layers.run(args, ClockSampler, peaks)
    elif args.impl == "reference":
        run_reference_arm(args)
    else:
        run_ours(args)


if __name__ == "__main__":
    main()
