"""Torirax on the host: the plain restatement's mechanisms, configuration and checkpoint reading,
cache geometry, slots, schedules and the command-line programs."""

import json
import math
import subprocess
import sys
from dataclasses import replace
from pathlib import Path

import pytest
import torch

from megakernels_b200.demos.hybrid import instructions as I
from megakernels_b200.demos.hybrid.scheduler import HybridScheduleOptions, column_groups, row_ranges, state_columns
from megakernels_b200.dispatch import make_schedule_builder
from megakernels_b200.hybrid import DiffAttentionSpec, HybridConfig, HybridForCausalLM, LayerSpec, key_splits, tensor_shapes
from megakernels_b200.model_types import ExtraModelConfig
from megakernels_b200.registry import family_of_checkpoint, load_model
from megakernels_b200.scheduler import assign_to_sms, tensorize_instructions
from megakernels_b200.state import CacheRows, SlotPool, plan_cache_rows
from megakernels_b200.torirax import PRESETS, ToriraxForCausalLM
from oracle import torirax_ref as R
from tests.torirax_utils import EVEN, MODELS, ODD, make_weights, model_config, oracle_logits, rank_of, rel, tokens_for, write_checkpoint
from tests.torirax_utils import attention as attn_layer

ROOT = Path(__file__).resolve().parent.parent


def rnd(*shape, seed=0):
    return torch.randn(shape, generator=torch.Generator().manual_seed(seed), dtype=torch.float64)


# ---- the restatement's mechanisms against independent forms ------------------------------- #
def test_layer_norm_and_poly_norm():
    x, w = rnd(5, 12), rnd(12, seed=1)
    assert torch.allclose(R.layer_norm(x, w, 1e-3), torch.nn.functional.layer_norm(x, (12,), w, None, 1e-3))
    z, c = rnd(3, 9), torch.tensor([0.5, -1.0, 2.0, 0.25], dtype=torch.float64)
    rms = lambda v: v / (v.pow(2).mean(-1, keepdim=True) + 1e-3).sqrt()  # noqa: E731
    assert torch.allclose(R.poly_norm(z, c, 1e-3), 0.5 * rms(z) - rms(z * z) + 2 * rms(z * z * z) + 0.25)


def test_recurrence_equals_its_transition_matrices():
    """S_t = (diag(w) - (a u) u^T) S_{t-1} + k v^T, one head at a time as explicit matrices."""
    T, H, D = 7, 2, 5
    r, k, v, w, a = (rnd(T, H, D, seed=s) for s in range(5))
    w, a = torch.sigmoid(w), torch.sigmoid(a)
    got, last = R.delta_recurrence(r, k, v, w, a)
    for h in range(H):
        S = torch.zeros(D, D, dtype=torch.float64)
        for t in range(T):
            u = k[t, h] / math.sqrt(float(k[t, h] @ k[t, h]) + 1e-6)
            S = (torch.diag(w[t, h]) - torch.outer(a[t, h] * u, u)) @ S + torch.outer(k[t, h], v[t, h])
            assert torch.allclose(got[t, h], r[t, h] @ S)
        assert torch.allclose(last[h], S)
    # carried state: two halves equal the whole
    a1, s1 = R.delta_recurrence(*(x[:3] for x in (r, k, v, w, a)))
    a2, s2 = R.delta_recurrence(*(x[3:] for x in (r, k, v, w, a)), state=s1)
    assert torch.allclose(torch.cat([a1, a2]), got) and torch.allclose(s2, last)


def test_decay_stays_in_its_interval():
    d = R.channel_decay(rnd(6, 4) * 10, rnd(3, 4), rnd(8, 3) * 5, rnd(8))
    assert float(d.max()) <= 1.0 and float(d.min()) >= math.exp(-math.exp(-0.5)) - 1e-12


@pytest.mark.parametrize("size,keep", [(1, 0), (4, 0), (4, 2), (100, 3), (3, 50)])
def test_visibility_against_the_rule(size, keep):
    m = R.visibility(12, size, keep)
    for i in range(12):
        for j in range(12):
            assert bool(m[i, j]) == (j <= i and (i - j < size or j < keep)) == bool(R.visible(i, j, size, keep))


def test_lambda_and_maps():
    lam = R.diff_lambda(*(torch.tensor(v, dtype=torch.float64) for v in ([1.0, 2], [0.5, 0], [0.0, 1], [3.0, -1])), 0.2)
    assert float(lam) == pytest.approx(math.exp(0.5) - math.exp(-1) + 0.2)
    q, k, v = rnd(4, 3), rnd(4, 3, seed=1), rnd(4, 2, seed=2)
    got = R.attention_map(q, k, v, 0.7, R.visibility(4, 2, 1))
    s = [math.exp(0.7 * float(q[3] @ k[j])) for j in (0, 2, 3)]  # position 3 sees 2, 3 and the kept 0
    want = sum(x * v[j] for x, j in zip(s, (0, 2, 3))) / sum(s)
    assert torch.allclose(got[3], want)


def test_planted_mistakes_show_in_the_logits():
    """The test models are sensitive: a window or a kept prefix that is one position off, a
    missing subtraction or a lost state changes the logits by far more than any tolerance."""
    w = make_weights(ODD, qk_gain=3.0)
    toks = tokens_for(ODD, 60)
    want = oracle_logits(ODD, w, toks)
    for i in (1, 3):
        for key, d in (("size", 1), ("size", -1), ("keep_first", 1), ("keep_first", -1)):
            raw = json.loads(json.dumps(ODD))
            raw["layers"][i]["mixer"]["mask"][key] += d
            assert rel(oracle_logits(raw, w, toks), want) > 5e-3, (i, key, d)
    raw = json.loads(json.dumps(ODD))
    raw["layers"][1]["mixer"]["diff"] += 0.01
    assert rel(oracle_logits(raw, w, toks), want) > 1e-3
    assert rel(oracle_logits(ODD, w, toks[20:])[-1:], want[-1:]) > 5e-3  # what came before matters


# ---- configuration and checkpoint ----------------------------------------------------------- #
def test_checkpoint_reading_pads_stacks_and_folds(tmp_path):
    w = make_weights(ODD)
    path = write_checkpoint(tmp_path, ODD, w)
    assert family_of_checkpoint(path).name == "torirax"
    m = load_model(path, ExtraModelConfig(max_batch_size=2), device="cpu", dtype=torch.float32)
    assert isinstance(m, ToriraxForCausalLM) and m.setting == "hybrid" and m.config.eps == 3e-4
    spec = m.config.layers
    assert spec[0].mixer.rank == rank_of(0) and spec[0].mlp.ff == 100 and spec[2].mlp is None
    assert spec[3].mixer.kv_from == 1 and spec[1].mixer.kv_from is None
    p = m.layers[0]
    rows = torch.cat([w[f"l0.mix.{n}"] for n in ("r", "k", "v", "a", "g", "w1")]).float()
    assert p.in_w.shape == (5 * 72 + rank_of(0), 72) and torch.equal(p.in_w, rows)
    assert torch.equal(p.in_bias[3 * 72 : 4 * 72], w["l0.mix.a.b"].float()) and float(p.in_bias[: 3 * 72].abs().sum()) == 0
    p = m.layers[1]
    assert torch.equal(p.in_w, torch.cat([w[f"l1.mix.{n}"] for n in ("q", "g", "k", "v")]).float())
    assert p.up_w is None
    p = m.layers[3]
    assert torch.equal(p.in_w, torch.cat([w["l3.mix.q"], w["l3.mix.g"]]).float())
    assert p.down_w.shape == (72, 56) and float(p.down_w[:, 52:].abs().sum()) == 0
    lam = R.diff_lambda(*(w[f"l3.mix.{n}"].double() for n in ("lq1", "lk1", "lq2", "lk2")), 0.15)
    assert p.diff_lambda == pytest.approx(float(lam)) and p.act == tuple(w["l3.mlp.act"].float().tolist())
    # the reader's masks (29, 5) and the owner's (11, 3) share one cache
    assert m.state.rows[1] == CacheRows(keep=5, ring=315) and 3 not in m.state.keys
    assert m.state.matrices[2].shape == (2, 2, 41, 41) and m.state.matrices[2].dtype == torch.float32


def test_unknown_designs_and_kinds_are_refused(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Other"}))
    with pytest.raises(ValueError, match="no model family"):
        family_of_checkpoint(tmp_path)
    for change in ({"type": "mystery"}, {"mlp": {"kind": "routed", "ff": 8}}):
        raw = json.loads(json.dumps(ODD))
        raw["layers"][0].update(change)
        path = write_checkpoint(tmp_path / next(iter(change)), raw, make_weights(ODD))
        with pytest.raises(ValueError, match="unknown"):
            load_model(path, device="cpu")


def test_kv_from_must_name_an_earlier_layer_with_keys():
    m = DiffAttentionSpec(4, 2, 8, 8, 0.3, 5, 1, 0.2)
    cfg = lambda *ms: HybridConfig(16, 10, 20, 1e-5, 1.0, tuple(LayerSpec(x) for x in ms))  # noqa: E731
    cfg(m, replace(m, kv_from=0, window=9))
    for bad in ((replace(m, kv_from=0),), (m, replace(m, kv_from=1)), (m, replace(m, kv_from=0), replace(m, kv_from=1)),
                (m, replace(m, kv_from=0, kv_heads=1)), (replace(m, heads=3),)):
        with pytest.raises(ValueError):
            cfg(*bad)


def test_llama_checkpoints_still_resolve(tmp_path):
    from megakernels_b200.llama import LlamaConfig, LlamaForCausalLM
    from tests.test_host_surface import TINY
    from tests.test_host_surface import write_checkpoint as write_llama

    write_llama(tmp_path, LlamaConfig(**TINY))
    m = load_model(tmp_path, ExtraModelConfig(interleave_rope=True, max_len_override=32), device="cpu")
    assert isinstance(m, LlamaForCausalLM) and m.setting == "latency" and m.max_len() == 32
    with pytest.raises(ValueError, match="do not run in"):
        load_model(tmp_path, device="cpu", dtype=torch.float32)


# ---- cache geometry and slots ------------------------------------------------------------------ #
@pytest.mark.parametrize("window,keep,portion,max_len", [(5, 2, 4, 60), (1, 0, 2, 40), (7, 9, 3, 60), (90, 3, 8, 60), (4, 70, 4, 60)])
def test_no_visible_row_is_overwritten(window, keep, portion, max_len):
    """A portion is written before its first token attends: every key that any of its tokens sees
    must still be in its row, whatever the cut."""
    spec = DiffAttentionSpec(1, 1, 1, 1, 1.0, window, keep, 0.0)
    rows = plan_cache_rows([spec], max_len, portion)
    row_of = [rows.row(j) for j in range(max_len)]
    assert all(0 <= r < rows.total for r in row_of) and rows.total <= max_len + 1
    for start in range(max_len):
        end = min(start + portion, max_len)
        holder = {}
        for j in range(end):
            holder[row_of[j]] = j
        for i in range(start, end):
            for j in range(i + 1):
                if i - j < window or j < keep:
                    assert holder[row_of[j]] == j, (start, i, j)


def test_slot_pool():
    p = SlotPool(2)
    a, b = p.allocate(), p.allocate()
    assert {a, b} == {0, 1} and len(p) == 2
    with pytest.raises(RuntimeError):
        p.allocate()
    p.free(a)
    assert p.allocate() == a
    with pytest.raises(ValueError):
        p.free(5)


# ---- schedules ---------------------------------------------------------------------------------- #
def build(raw, dtype=torch.bfloat16, options=None, **extra):
    w = make_weights(raw)
    cfg_shapes = {n: tuple(t.shape) for n, t in w.items()}
    m = HybridForCausalLM.assemble(ToriraxForCausalLM.read_config(raw, lambda n: cfg_shapes[n]), ExtraModelConfig(**extra), "cpu", dtype, w.get)
    return make_schedule_builder("hybrid", options).build(m)


@pytest.mark.parametrize("name", sorted(MODELS))
@pytest.mark.parametrize("mode", ["rr", "zz", "wave", "dag"])
def test_schedule_covers_every_row_once_and_counts_its_arrivals(name, mode):
    sched = build(MODELS[name])
    g = sched.globs
    queues = assign_to_sms(mode, schedule=sched)
    flat = [i for q in queues for i in q]
    assert sorted(map(repr, flat)) == sorted(map(repr, sched.get_linear_instructions()))
    cfg = g.model.config
    by = {}
    for ins in flat:
        by.setdefault((type(ins), ins.layer_idx), []).append(ins)
    for i, spec in enumerate(cfg.layers):
        kinds = [I.NormProj, I.OutProj] + ([I.NormUp, I.Down] if spec.mlp else [])
        for cls in kinds:
            got = sorted((x.row_start, x.row_end) for x in by[cls, i])
            assert got[0][0] == 0 and got[-1][1] == I.matrix_shape(g, cls.opcode(), i)[0]
            assert all(a[1] == b[0] for a, b in zip(got, got[1:])) and all(a < b for a, b in got)
            assert int(g.arrivals[i, cls.opcode()]) == len(got)
        if spec.mixer.kind == "delta_rule":
            cells = [(x.head_idx, c) for x in by[I.DeltaStep, i] for c in range(x.col_start, x.col_end)]
            assert sorted(cells) == [(h, c) for h in range(spec.mixer.heads) for c in range(spec.mixer.dim)]
            assert int(g.arrivals[i, 2]) == len(by[I.DeltaStep, i])
        else:
            n = key_splits(spec.mixer, g.model.max_len(), 148)
            assert sorted((x.kv_head_idx, x.split_idx) for x in by[I.KeyAttention, i]) == \
                [(h, s) for h in range(spec.mixer.kv_heads) for s in range(n)]
            assert int(g.arrivals[i, 3]) == spec.mixer.kv_heads and n <= g.max_splits
    # a phase's instructions precede the next phase's in every queue
    order = lambda x: (len(cfg.layers) if isinstance(x, I.Head) else x.layer_idx, x.opcode())  # noqa: E731
    assert all([order(x) for x in q] == sorted(order(x) for x in q) for q in queues)
    tensorize_instructions(g, queues)
    assert g.instructions.shape[0] == 148 and g.instructions.dtype == torch.int32


def test_row_ranges_fit_the_partial_sums():
    for rows, k, size in ((128256, 2048, 2), (128256, 4096, 4), (7, 64, 2), (149, 8192, 2), (14336, 4096, 2)):
        r = row_ranges(rows, k, size, 148)
        assert r[0][0] == 0 and r[-1][1] == rows and all(a[1] == b[0] for a, b in zip(r, r[1:]))
        assert max(b - a for a, b in r) * column_groups(k, size) <= I.PARTIAL_SUMS
        assert max(b - a for a, b in r) <= I.MAX_ROWS
        assert len(r) <= 148 or len(r) % 148 == 0
    for heads, dim, want in ((1, 8, 16), (32, 64, 16), (64, 128, 64), (100, 256, 256), (6, 100, 16)):
        assert state_columns(heads, dim, 148) == want


def test_split_counts_and_options():
    sched = build(EVEN, options=HybridScheduleOptions(keys_per_split=8, state_columns=32))
    splits = [i for i in sched.get_linear_instructions() if isinstance(i, I.KeyAttention)]
    assert max(i.num_splits for i in splits) == 10 and sched.globs.max_splits == 10
    assert {i.col_end - i.col_start for i in sched.get_linear_instructions() if isinstance(i, I.DeltaStep)} == {32}
    assert key_splits(DiffAttentionSpec(8, 8, 64, 64, 1.0, 10**6, 0, 0.1), 10**6, 148) == 18


def test_presets_have_real_proportions():
    for name, make in PRESETS.items():
        cfg = make(2)
        assert tensor_shapes(cfg)["head"] == (128256, cfg.width)
        kinds = [s.mixer.kind for s in cfg.layers]
        assert kinds.count("delta_rule") == 4 and cfg.layers[5].mixer.kv_from == 2, name


# ---- programs ------------------------------------------------------------------------------------ #
def test_trace_run_refuses_a_dtype_no_kernel_has(tmp_path):
    from megakernels_b200.llama import LlamaConfig
    from tests.test_host_surface import TINY
    from tests.test_host_surface import write_checkpoint as write_llama

    write_llama(tmp_path, LlamaConfig(**TINY))
    r = subprocess.run([sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(tmp_path), "--dtype", "float32",
                        "--out", str(tmp_path)], input="", text=True, capture_output=True, timeout=120)
    assert r.returncode == 3 and "float32" in r.stderr


def test_generate_cli_knows_the_family():
    from megakernels_b200.registry import family_of_preset
    from megakernels_b200.scripts.generate import parse_cli

    cfg = parse_cli(["model=torirax-1b", "dtype=float32", "ntok=4"])
    assert cfg.dtype == "float32" and family_of_preset(cfg.model).name == "torirax"
    assert family_of_preset("llama-8b").name == "llama" and family_of_preset("nope") is None
    with pytest.raises(SystemExit):
        parse_cli(["setting=throughput"])


def test_oracle_runs_a_model_with_one_of_everything():
    raw = model_config([attn_layer(2, 1, 4, 4, size=3, keep_first=1)], width=16, vocab=11, max_positions=9)
    out = oracle_logits(raw, make_weights(raw), tokens_for(raw, 9))
    assert out.shape == (9, 11) and bool(torch.isfinite(out).all())
