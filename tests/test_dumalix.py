"""Dumalix on the CPU: the plain restatement's mechanisms against independent forms, the
configuration, rotation tables, cache geometry, schedules."""

import json
import math

import pytest
import torch

from megakernels_b200.demos.hybrid import instructions as I
from megakernels_b200.demos.hybrid.scheduler import head_row_ranges, row_ranges
from megakernels_b200.dispatch import make_schedule_builder
from megakernels_b200.dumalix import PRESETS, DumalixForCausalLM, read_layer
from megakernels_b200.hybrid import HybridConfig, HybridForCausalLM, LayerSpec, LoopSpec, PolyNormSpec, RopeSpec, YarnSpec, key_splits, tensor_shapes
from megakernels_b200.model_types import ExtraModelConfig
from megakernels_b200.registry import family_of_checkpoint, family_of_preset, load_model
from megakernels_b200.scheduler import assign_to_sms, tensorize_instructions
from megakernels_b200.state import CacheRows
from oracle import dumalix_ref as R
from tests.dumalix_utils import (
    EVEN, GROUPS, MODELS, ODD, RAGGED, WIDE, changed, chunked, config_of, latent, make_weights, model_config, oracle_logits, rel,
    tokens_for, write_checkpoint,
)


def rnd(*shape, seed=0):
    return torch.randn(shape, generator=torch.Generator().manual_seed(seed), dtype=torch.float64)


# ---- the restatement's mechanisms against independent forms ------------------------------- #
def test_norms():
    x, w = rnd(5, 12), rnd(12, seed=1)
    want = torch.nn.functional.rms_norm(x, (12,), w, 1e-3)
    assert torch.allclose(R.norm_plain(x, w, 1e-3), want)
    assert torch.allclose(R.norm_one_plus(x, w - 1, 1e-3), want)


@pytest.mark.parametrize("taps", [1, 2, 4, 9])
def test_convolution_is_causal_with_the_last_tap_on_the_current_token(taps):
    u, w = rnd(7, 3), rnd(3, taps, seed=1)
    want = torch.nn.functional.conv1d(u.T[None], w[:, None], padding=taps - 1, groups=3)[0, :, :7].T
    assert torch.allclose(R.causal_conv(u, w), want)


def test_gated_unit():
    g, u = torch.tensor([-3.0, 0.5, 9.0]), torch.tensor([5.0, -0.25, -5.0])
    sig = lambda x: 1 / (1 + math.exp(-x))  # noqa: E731
    want = [-3 * sig(-3 * 1.702) * 3, 0.5 * sig(0.851) * 0.75, 2 * sig(3.404) * -1]
    assert R.clamped_glu(g, u, 2.0).tolist() == pytest.approx(want)


def test_rotation_as_complex_numbers():
    x, f = rnd(6, 2, 9), [1.0, 0.3, 0.01]
    got = R.rotate(x, f, factor=1.25)
    z = torch.view_as_complex(x[..., :6].reshape(6, 2, 3, 2).contiguous())
    turn = 1.25 * torch.exp(1j * torch.arange(6, dtype=torch.float64)[:, None, None] * torch.tensor(f, dtype=torch.float64))
    assert torch.allclose(got[..., :6], torch.view_as_real(z * turn).reshape(6, 2, 6)) and torch.equal(got[..., 6:], x[..., 6:])
    assert torch.allclose(R.rotate(R.rotate(x, f), f, sign=-1), x)


def test_scaled_frequencies():
    y = {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}
    f, factor = R.yarn_frequencies(128, 10000.0, y)
    plain = R.plain_frequencies(128, 10000.0)
    assert factor == pytest.approx(0.1 * math.log(8) + 1)
    turns = [4096 * p / (2 * math.pi) for p in plain]
    for a, p, n in zip(f, plain, turns):  # fast pairs keep their frequency, slow ones lose the factor
        if n > 33 * 1.2:
            assert a == pytest.approx(p)
        elif n < 0.8:
            assert a == pytest.approx(p / 8)
        else:
            assert p / 8 - 1e-15 <= a <= p + 1e-15
    assert sorted(f, reverse=True) == f
    assert R.yarn_frequencies(6, 10.0, None) == (R.plain_frequencies(6, 10.0), 1.0)
    # everything on one side of the ramp: hi == lo
    f, _ = R.yarn_frequencies(4, 1e6, {"factor": 2.0, "original": 3, "fast": 9.0, "slow": 8.0})
    assert f == pytest.approx([1.0, 1e-3 / 2])


@pytest.mark.parametrize("spec", [RopeSpec(64, 10000.0, YarnSpec(8.0, 4096, 32.0, 1.0)), RopeSpec(6, 50.0), RopeSpec(2, 7.0, YarnSpec(3.0, 9, 2.0, 1.0)),
                                  RopeSpec(30, 300.0, YarnSpec(4.0, 64, 8.0, 0.5)), RopeSpec(4, 1e6, YarnSpec(2.0, 3, 9.0, 8.0))])
def test_rotation_tables_of_the_framework(spec):
    y = spec.scaling
    f, factor = R.yarn_frequencies(spec.dims, spec.base, y and dict(factor=y.factor, original=y.original, fast=y.fast, slow=y.slow))
    got, n = spec.table(3000), spec.dims // 2
    angle = torch.arange(3000, dtype=torch.float64)[:, None] * torch.tensor(f, dtype=torch.float64)
    assert got.shape == (3000, n, 2) and got.dtype == torch.float32
    assert torch.allclose(got[..., 0].double(), factor * angle.cos(), atol=2e-7, rtol=0)
    assert torch.allclose(got[..., 1].double(), factor * angle.sin(), atol=2e-7, rtol=0)


def test_chunks_count_from_the_sequence_start():
    m = R.chunk_visibility(12, 5)
    for i in range(12):
        assert [j for j in range(12) if m[i, j]] == list(range(i - i % 5, i + 1))


def test_a_sink_is_a_key_without_a_value():
    score, v = rnd(4, 4), rnd(4, 3, seed=1)
    got = R.softmax_with_sink(score, R.causal_visibility(4), torch.tensor(0.7, dtype=torch.float64)) @ v
    e = torch.exp(score[2, :3])
    assert torch.allclose(got[2], (e[:, None] * v[:3]).sum(0) / (e.sum() + math.exp(0.7)))
    huge = R.softmax_with_sink(score, R.causal_visibility(4), torch.tensor(2000.0, dtype=torch.float64))
    assert float(huge.abs().max()) == 0


def test_turned_values_depend_on_the_distance_only():
    """Rotating values by j and outputs by -i leaves rotations by j - i."""
    T, E, f = 6, 4, [0.9, 0.2]
    p, v = torch.softmax(rnd(T, T), -1), rnd(T, E, seed=1)
    got = R.rotate(p @ R.rotate(v, f), f, sign=-1)
    z, w = torch.view_as_complex(v.view(T, 2, 2)), torch.tensor(f, dtype=torch.float64)
    for i in range(T):
        want = sum(p[i, j] * z[j] * torch.exp(1j * (j - i) * w) for j in range(T))
        assert torch.allclose(got[i], torch.view_as_real(want).reshape(E))


def test_latent_attention_in_latent_space():
    """Absorbing the key expansion into the query and expanding the mixed latents gives the same."""
    raw = model_config([latent(3, 12, 6, 10, 20)])
    w = {k[len("l0.mix."):]: t.double() for k, t in make_weights(raw).items() if k.startswith("l0.mix.")}
    m, h, eps = raw["layers"][0]["mixer"], rnd(9, 72), 1e-5
    got = R.latent_attention_mixer(h, w.__getitem__, m, eps)
    q, down = (h @ w["q"].T).view(9, 3, 18), h @ w["dkv"].T
    c = R.norm_plain(down[:, :20], w["dkv.norm"], eps)
    f, factor = R.yarn_frequencies(6, m["rot"]["base"], m["rot"]["scaling"])
    kr, qr = R.rotate(down[:, 20:], f, factor), R.rotate(q[..., 12:], f, factor)
    heads = []
    for n in range(3):
        absorbed = q[:, n, :12] @ w["uk"].view(3, 12, 20)[n]
        p = R.softmax_with_sink((absorbed @ c.T + qr[:, n] @ kr.T) * m["scale"], R.causal_visibility(9))
        heads.append((p @ c) @ w["uv"].view(3, 10, 20)[n].T)
    assert torch.allclose(got, torch.cat(heads, -1) @ w["o"].T)


def test_runs_of_a_loop():
    want = [(0, False), (1, True), (2, False), (1, True), (2, False), (1, True), (2, False), (3, False), (4, False)]
    assert R.layer_runs(EVEN) == want == list(config_of(EVEN).runs)
    for raw in MODELS.values():
        assert R.layer_runs(raw) == list(config_of(raw).runs)
    spec = config_of(WIDE).layers[0]
    cfg = lambda loop: HybridConfig(8, 9, 10, 1e-5, 1.0, (spec, spec), loop=loop)  # noqa: E731
    for bad in (LoopSpec(0, 3, 2), LoopSpec(1, 1, 2), LoopSpec(-1, 1, 1), LoopSpec(0, 1, 0)):
        with pytest.raises(ValueError):
            cfg(bad)
    assert len(cfg(LoopSpec(1, 2, 4)).runs) == 5


def test_planted_mistakes_show_in_the_logits():
    """The test models are sensitive: each of these changes the logits by far more than any tolerance."""
    for raw in (ODD, EVEN, GROUPS):
        w = make_weights(raw, qk_gain=3.0)
        toks = tokens_for(raw, 80)
        want = oracle_logits(raw, w, toks)
        differs = lambda r=raw, ww=w: rel(oracle_logits(r, ww, toks), want)  # noqa: E731
        for i, layer in enumerate(raw["layers"]):
            m = layer["mixer"]
            if layer["type"] == "attention":
                if m["mask"]["size"] < 80:
                    assert min(differs(changed(raw, i, ("mixer", "mask", "size"), m["mask"]["size"] + d)) for d in (1, -1)) > 5e-3
                for name in ("temp", "sink"):
                    assert differs(ww={**w, f"l{i}.mix.{name}": w[f"l{i}.mix.{name}"] * 0}) > 5e-3, (i, name)
            if m["rot"]["dims"] > 2 or layer["type"] == "attention":  # (one pair turns by the position itself)
                assert differs(changed(raw, i, ("mixer", "rot", "base"), m["rot"]["base"] * 1.5)) > 3e-3, i
            if m["rot"]["scaling"]:
                assert differs(changed(raw, i, ("mixer", "rot", "scaling", "factor"), 2.0)) > 3e-3, i
            if layer["mlp"]:
                assert differs(changed(raw, i, ("mlp", "limit"), layer["mlp"]["limit"] * 1.2)) > 3e-3, i
            assert differs(ww={**w, f"l{i}.canon1": w[f"l{i}.canon1"].roll(1, dims=1)}) > 5e-3, i
        assert differs(changed(raw, None, ("loop", "times"), raw["loop"]["times"] + 1)) > 5e-3
        assert rel(oracle_logits(raw, w, toks[2:])[-1:], want[-1:]) > 5e-3  # what came before matters


# ---- configuration and checkpoint ----------------------------------------------------------- #
def test_checkpoint_reading_stacks_and_folds(tmp_path):
    w = make_weights(ODD)
    path = write_checkpoint(tmp_path, ODD, w)
    assert family_of_checkpoint(path).name == "dumalix"
    m = load_model(path, ExtraModelConfig(max_batch_size=2, max_len_override=90), device="cpu", dtype=torch.float32)
    assert isinstance(m, DumalixForCausalLM) and m.setting == "hybrid" and m.config.eps == 3e-4 and m.max_len() == 90
    assert {n: tuple(t.shape) for n, t in w.items()} == tensor_shapes(m.config) and m.positions is None
    specs = m.config.layers
    assert all(s.parallel and s.canon_taps == 3 for s in specs) and specs[2].mlp is None and specs[0].mixer.conv_taps == 3
    p = m.layers[0]
    assert torch.equal(p.in_w, torch.cat([w[f"l0.mix.{n}"] for n in "qkv"]).float()) and p.in_bias is None and p.ls1 is None
    assert torch.equal(p.norm1, 1 + w["l0.norm1"].float()) and torch.equal(m.final_norm, 1 + w["final.norm"].float())
    assert torch.equal(p.q_norm, w["l0.mix.q.norm"].float())
    assert torch.equal(p.conv_w, torch.cat([w[f"l0.mix.{n}.conv"] for n in "qkv"]).float().T)
    assert torch.allclose(p.canon_gain, (1 + w["l0.norm1"].float()) * (1 + w["l0.canon1"][:, -1].float()))
    assert torch.equal(p.up_w[0::2], w["l0.mlp.gate"].float()) and torch.equal(p.up_w[1::2], w["l0.mlp.up"].float())
    assert m.enter.shape == (72, 144)
    p = m.layers[1]
    assert torch.equal(p.in_w, torch.cat([w["l1.mix.q"], w["l1.mix.dkv"]]).float())
    assert p.absorb_w.shape == (3 * 20, 16) and torch.equal(p.absorb_w[20 + 7, :12], w["l1.mix.uk"][12:24, 7].float())
    assert torch.equal(p.expand_w[:, :20], torch.cat([w["l1.mix.uk"], w["l1.mix.uv"]]).float())
    # every pass has its own rows and inputs
    assert m.config.runs[2] == (0, True) and m.state.rows[2] == CacheRows(keep=0, ring=90)
    assert m.state.keys[0].shape == (2, 3, 90, 20) and m.state.keys[0].data_ptr() != m.state.keys[2].data_ptr()
    assert m.state.keys[1].shape == (2, 90, 40) and 1 not in m.state.values
    assert m.state.inputs[3].shape == (2, 2, 72) and m.state.projected[2].shape == (2, 2, 6 * 20 + 3 * 48) and 1 not in m.state.projected
    b = load_model(path, ExtraModelConfig(max_len_override=90, prefill_portion=4), device="cpu")
    assert read_layer(0, changed(ODD, 0, ("mixer", "conv"), 0)["layers"][0], 3, None).mixer.conv_taps == 0
    raw = changed(ODD, 0, ("x",), 0)["layers"][0]
    del raw["mixer"]["conv"]  # then the tensors say
    assert read_layer(0, raw, 3, lambda name: tuple(w[name].shape)).mixer.conv_taps == 3
    assert b.state.rows[0] == CacheRows(0, 11 + 4) and b.state.rows[1] == CacheRows(0, 90) and b.dtype == torch.bfloat16
    assert load_model(path, ExtraModelConfig(prefill_portion=4), device="cpu").max_len() == 32768  # the design sets no limit


def test_unknown_kinds_are_refused(tmp_path):
    for key, value in (("type", "mystery"), ("mlp", {"kind": "routed", "ff": 8, "limit": 1.0})):
        raw = changed(ODD, 0, (key,), value)
        path = write_checkpoint(tmp_path / key, raw, make_weights(ODD))
        with pytest.raises(ValueError, match="unknown"):
            load_model(path, device="cpu")
    with pytest.raises(ValueError, match="query heads"):
        config_of(changed(ODD, 0, ("mixer", "kv_heads"), 4))
    with pytest.raises(ValueError, match="beside"):
        HybridConfig(8, 9, 10, 1e-5, 1.0, (LayerSpec(config_of(ODD).layers[0].mixer, PolyNormSpec(8), parallel=True),))


def test_presets_and_command_line():
    from megakernels_b200.scripts.generate import parse_cli

    for name, make in PRESETS.items():
        cfg = make()
        assert family_of_preset(name).name == "dumalix" and cfg.vocab_size == 128256
        assert {s.mixer.kind for s in cfg.layers} == {"attention", "latent_attention"} and len(cfg.runs) in (16, 32)
        assert tensor_shapes(cfg)["loop.in"] == (cfg.width, 2 * cfg.width)
    assert parse_cli(["model=dumalix-1b", "dtype=float32"]).model == "dumalix-1b"


def test_random_weights_fill_every_tensor():
    m = HybridForCausalLM.from_random(config_of(RAGGED), ExtraModelConfig(max_len_override=20), device="cpu")
    assert abs(float(m.layers[0].norm1.mean()) - 1) < 0.1 and abs(float(m.final_norm.mean()) - 1) < 0.1
    assert all(bool(torch.isfinite(t.float()).all()) for p in m.layers for t in vars(p).values() if torch.is_tensor(t))


# ---- schedules ---------------------------------------------------------------------------------- #
def build(raw, dtype=torch.bfloat16, **extra):
    extra.setdefault("max_len_override", 200)
    m = HybridForCausalLM.assemble(config_of(raw), ExtraModelConfig(**extra), "cpu", dtype, make_weights(raw).get)
    return make_schedule_builder("hybrid").build(m)


def waits_for(cfg, ins):
    """(run, opcode counter) an instruction waits for, None at the start: the kernel's rule."""
    i, op = ins.layer_idx, ins.opcode()
    last = lambda k: None if k < 0 else (k, 4 if cfg.run_layers[k].parallel or cfg.run_layers[k].mlp is None else 6)  # noqa: E731
    if op == 7:
        return last(len(cfg.runs) - 1)
    latent_ = cfg.run_layers[i].mixer.kind == "latent_attention"
    if op == 8:
        return last(i - 1)
    if op in (1, 5):
        return (i, 8) if cfg.runs[i][1] else last(i - 1)
    return {9: (i, 1), 3: (i, 9 if latent_ else 1), 10: (i, 3), 6: (i, 5), 4: (i, 10 if latent_ else 3)}[op]


@pytest.mark.parametrize("name", sorted(MODELS))
@pytest.mark.parametrize("mode", ["rr", "zz", "wave", "dag"])
def test_schedule_covers_everything_once_and_runs_to_its_end(name, mode):
    sched = build(MODELS[name])
    g = sched.globs
    cfg = g.model.config
    queues = assign_to_sms(mode, schedule=sched)
    flat = [i for q in queues for i in q]
    assert sorted(map(repr, flat)) == sorted(map(repr, sched.get_linear_instructions()))
    by = {}
    for ins in flat:
        by.setdefault((type(ins), ins.layer_idx), []).append(ins)
    for i, (layer, enters) in enumerate(cfg.runs):
        spec = cfg.layers[layer]
        m = spec.mixer
        lat = m.kind == "latent_attention"
        kinds = [I.NormProj, I.OutProj] + [I.NormUp, I.Down] * (spec.mlp is not None) + [I.Enter] * enters + [I.Absorb, I.Expand] * lat
        for cls in kinds:
            got = sorted((x.row_start, x.row_end) for x in by.pop((cls, i)))
            assert got[0][0] == 0 and got[-1][1] == I.matrix_shape(g, cls.opcode(), i)[0]
            assert all(a[1] == b[0] for a, b in zip(got, got[1:])) and all(a < b for a, b in got)
            if cls is I.NormUp:
                assert all(a % 2 == 0 for a, _ in got)
            if cls in (I.Absorb, I.Expand):
                per = m.rank if cls is I.Absorb else m.vdim
                assert all(a // per == (b - 1) // per for a, b in got)
        n = key_splits(m, 200, 148)
        assert sorted((x.kv_head_idx, x.split_idx) for x in by.pop((I.KeyAttention, i))) == \
            [(h, s) for h in range(m.key_groups) for s in range(n)]
    assert set(by) == {(I.Head, 0)}
    # walk the queues with the kernel's waits: everything runs, and no counter passes its threshold early
    count, arrived, at = {}, {}, [0] * len(queues)
    heads_done = {}
    progress = True
    while progress:
        progress = False
        for q, queue in enumerate(queues):
            while at[q] < len(queue):
                ins = queue[at[q]]
                need = waits_for(cfg, ins)
                if need is not None and count.get(need, 0) < int(g.arrivals[need]):
                    break
                i, op = ins.layer_idx, ins.opcode()
                if op == 3:
                    k = (i, ins.kv_head_idx)
                    heads_done[k] = heads_done.get(k, 0) + 1
                    signal = heads_done[k] == ins.num_splits or cfg.run_layers[i].mixer.kind == "latent_attention"
                else:
                    signal = True
                mixer = cfg.run_layers[i].mixer.kind
                key = (i, (10 if mixer == "latent_attention" else 3) if op == 6 and cfg.run_layers[i].parallel else op)
                count[key] = count.get(key, 0) + signal
                at[q] += 1
                progress = True
    assert at == [len(q) for q in queues]
    assert all(n <= int(g.arrivals[k]) for k, n in count.items() if k[1] != 7)
    tensorize_instructions(g, queues)
    assert g.instructions.shape[0] == 148


def test_row_ranges_of_pairs_and_heads():
    for rows, k, unit in ((16384, 2048, 2), (10, 64, 2), (28672, 4096, 2)):
        r = row_ranges(rows, k, 2, 148, unit)
        assert r[0][0] == 0 and r[-1][1] == rows and all(a[1] == b[0] for a, b in zip(r, r[1:])) and all(a % unit == 0 for a, _ in r)
        assert max(b - a for a, b in r) <= I.MAX_ROWS
    r = head_row_ranges(16, 512, 128, 2, 148)
    assert len(r) == 144 and r[-1][1] == 8192 and all(a // 512 == (b - 1) // 512 for a, b in r)
    assert head_row_ranges(200, 3, 8, 2, 148) == [(3 * h, 3 * h + 3) for h in range(200)]


def test_oracle_runs_a_model_with_one_of_everything():
    raw = model_config([chunked(2, 1, 4, 4, size=3), latent(2, 4, 2, 4, 6, ff=5)], width=16, vocab=11, loop=(1, 2, 2))
    out, layers = [], []
    out = oracle_logits(raw, make_weights(raw), tokens_for(raw, 9), layers_out=layers)
    assert out.shape == (9, 11) and bool(torch.isfinite(out).all()) and len(layers) == 3
    assert json.loads(json.dumps(raw)) == raw
