"""Torirax on a GPU: every kernel path against the plain restatement, cuts of a sequence against
the whole, slots that are reused, windows' edges, long decoding, greedy generation."""

import json
import subprocess
import sys
from pathlib import Path

import pytest
import torch

from tests.torirax_utils import (
    BF16_TOL, EVEN, F32_TOL, MODELS, ODD, attention, delta, load, make_weights, model_config, oracle_logits, rel, run_cut,
    tokens_for, write_checkpoint,
)

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
DTYPES = [(torch.float32, F32_TOL), (torch.bfloat16, BF16_TOL)]


@pytest.fixture(scope="module")
def bench(tmp_path_factory):
    """name -> (raw, weights, checkpoint path, tokens, float64 logits), made once."""
    made = {}

    def get(name, raw=None, n=150, qk_gain=1.0):
        if name not in made:
            raw = raw or MODELS[name]
            w = make_weights(raw, qk_gain=qk_gain)
            path = write_checkpoint(tmp_path_factory.mktemp("m") / "ckpt", raw, w)
            toks = tokens_for(raw, n)
            made[name] = (raw, w, path, toks, oracle_logits(raw, w, toks))
        return made[name]

    return get


SINGLES = {
    "delta": [delta(3, 24)],
    "delta_wide_head": [delta(2, 130)],
    "delta_mlp": [delta(2, 64, ff=200)],
    "attention": [attention(6, 2, 16, 24, size=9, keep_first=2)],
    "attention_one_group": [attention(2, 2, 32, 64, size=20, keep_first=0, diff=0.0)],
    "attention_no_window": [attention(4, 1, 64, 64, size=1000, keep_first=3, scale=0.2)],
    "attention_mlp": [attention(4, 4, 10, 30, size=5, keep_first=7, ff=90)],
    "shared_keys": [attention(4, 2, 16, 32, size=6, keep_first=1), attention(4, 2, 16, 32, size=31, keep_first=4, kv_from=0)],
}


@pytest.mark.parametrize("dtype,tol", DTYPES)
@pytest.mark.parametrize("name", sorted(SINGLES))
def test_one_mechanism_alone(bench, name, dtype, tol):
    """A model of one layer (or one pair): prompt, and token by token."""
    raw, w, path, toks, want = bench(f"one/{name}", model_config(SINGLES[name]), n=40)
    gen = load(path, dtype)
    assert rel(run_cut(gen, toks, [40]), want) < tol
    assert rel(run_cut(gen, toks, []), want) < tol


@pytest.mark.parametrize("dtype,tol", DTYPES)
@pytest.mark.parametrize("name", sorted(MODELS))
def test_prompt_and_every_layer(bench, name, dtype, tol):
    raw, w, path, toks, want = bench(name)
    gen = load(path, dtype)
    got, ref = [], []
    logits = gen.feed(toks, 0, list(range(len(toks))), layers_out=got)
    gen.check()
    oracle_logits(raw, w, toks, layers_out=ref)
    for i, r in enumerate(ref):
        assert rel(got[0][i], r) < tol, f"layer {i}"
    assert rel(logits, want) < tol


@pytest.mark.parametrize("dtype,tol", DTYPES)
@pytest.mark.parametrize("name", sorted(MODELS))
def test_token_by_token_equals_the_prompt(bench, name, dtype, tol):
    raw, w, path, toks, want = bench(name)
    assert rel(run_cut(load(path, dtype), toks, []), want) < tol


@pytest.mark.parametrize("cuts", [[2] * 75, [3, 2, 5, 2, 7, 11, 2, 13, 1, 1, 17, 2], [1, 149], [149, 1], [64, 64, 22], [33] * 5])
@pytest.mark.parametrize("name", ["odd", "even", "ragged"])
def test_portions_of_several_sizes(bench, name, cuts):
    raw, w, path, toks, want = bench(name)
    assert rel(run_cut(load(path), toks, cuts), want) < F32_TOL


@pytest.mark.parametrize("portion", [2, 5, 16, 50])
@pytest.mark.parametrize("name", ["odd", "even"])
def test_small_rings_wrap(bench, name, portion):
    """Prompts longer than the portion limit are cut inside; with it the key/value rings shrink to
    window + portion rows and wrap many times."""
    raw, w, path, toks, want = bench(name)
    gen = load(path, portion=portion)
    rows = gen.model.state.rows
    assert min(r.ring for r in rows.values()) < 150
    assert rel(run_cut(gen, toks, [150]), want) < F32_TOL
    assert rel(run_cut(gen, toks, [portion, 1, portion, 1, 1, 2 * portion + 1], slot=1), want) < F32_TOL
    assert rel(run_cut(gen, toks, [100], slot=2), want) < F32_TOL


def test_peaked_attention_at_every_edge(bench):
    """Large scores: single keys dominate, so each position's logits depend on exactly which keys it
    sees - windows' edges, kept first positions and the first tokens included."""
    raw, w, path, toks, want = bench("peaked", ODD, n=120, qk_gain=3.0)
    for cuts in ([120], [], [7, 4, 11, 1, 1, 29, 28, 2, 2], [12, 12, 12, 12]):
        assert rel(run_cut(load(path, portion=40), toks, cuts), want) < 2 * F32_TOL, cuts


@pytest.mark.parametrize("distance", [-1, 0, 1])
@pytest.mark.parametrize("decoded", [False, True])
def test_one_outstanding_key_just_inside_and_outside(tmp_path, distance, decoded):
    """One token's key towers over all others; a query at window - 1, window and window + 1 from it
    sees it or does not, and the logits say which."""
    size, keep = 13, 3
    raw = model_config([attention(2, 1, 16, 24, size=size, keep_first=keep, scale=1.0)], vocab=40)
    w = make_weights(raw)
    needle = 7
    w["l0.mix.k.b"].zero_(), w["l0.mix.q.b"].zero_()
    w["embed"][needle] = 12 * w["embed"][needle]
    # keys and queries of the needle's direction stand out for every query token
    w["l0.mix.q.b"] += 0.5
    h = torch.nn.functional.layer_norm(w["embed"][needle].float() * 3, (raw["width"],))
    w["l0.mix.k"] = (w["l0.mix.k"].float() * 0.1 + 12.0 * h[None, :] / raw["width"]).to(torch.bfloat16)
    path = write_checkpoint(tmp_path / "c", raw, w)
    at = 20
    toks = [t if t != needle else 8 for t in tokens_for(raw, at + size + 2)]
    toks[at] = needle
    query = at + size - 1 + distance
    want = oracle_logits(raw, w, toks)
    without = list(toks)
    without[at] = 8
    depends = rel(oracle_logits(raw, w, without)[query : query + 1], want[query : query + 1]) > 1e-2
    assert depends == (distance <= 0), "the test's needle does not show"
    cut = [query, 1] if decoded else [query + 1]
    got = run_cut(load(path), toks[: query + 1], cut)
    assert rel(got, want[: query + 1]) < F32_TOL


@pytest.mark.parametrize("dtype,tol", DTYPES)
def test_far_kept_keys_and_long_decoding(bench, dtype, tol):
    """250 decoded tokens after a short prompt: kept positions hundreds of tokens back, rings that
    wrap under single tokens, recurrent state that is carried all the way."""
    raw, w, path, toks, want = bench("long", EVEN, n=300)
    gen = load(path, dtype, portion=32)
    assert rel(run_cut(gen, toks, [50]), want) < tol


@pytest.mark.parametrize("dtype,tol", DTYPES)
def test_requests_in_turn_and_slots_used_again(bench, dtype, tol):
    """Requests of unequal length, interleaved over all slots, then their slots again."""
    raw, w, path, toks, _ = bench("odd")
    gen = load(path, dtype, portion=24)
    pool = gen.model.slots
    for rnd in range(2):
        reqs = {i: tokens_for(raw, n, seed=10 * rnd + i) for i, n in enumerate((90, 7, 41))}
        slots = {i: pool.allocate() for i in reqs}
        out, at, turn = {i: [] for i in reqs}, dict.fromkeys(reqs, 0), 0
        while any(at[i] < len(t) for i, t in reqs.items()):
            for i, t in reqs.items():
                n = min((5, 1, 13, 2, 1)[(turn + i) % 5], len(t) - at[i])
                if n > 0:
                    out[i].append(gen.step(t[at[i] : at[i] + n], at[i], list(range(n)), slot=slots[i]))
                    at[i] += n
            turn += 1
        for i, t in reqs.items():
            assert rel(torch.cat(out[i]), oracle_logits(raw, w, t)) < tol, (rnd, i)
            pool.free(slots[i])


def test_logits_do_not_depend_on_slot_or_history(bench):
    """Bit-identical decode whatever ran before and wherever the sequence lives."""
    raw, w, path, toks, _ = bench("even")
    gen = load(path, torch.bfloat16)
    a = run_cut(gen, toks[:60], [40], slot=0)
    run_cut(gen, toks[30:], [100], slot=2)
    b = run_cut(gen, toks[:60], [40], slot=2)
    c = run_cut(load(path, torch.bfloat16), toks[:60], [40], slot=1)
    assert torch.equal(a, b) and torch.equal(a, c)


def test_wanted_places_and_limits(bench):
    raw, w, path, toks, want = bench("odd")
    gen = load(path, portion=20)
    got = gen.step(toks[:55], 0, [54, 0, 21, 20])
    assert rel(got, want[[54, 0, 21, 20]]) < F32_TOL
    assert gen.step(toks[55:57], 55, []).shape == (0, raw["vocab"])
    assert rel(gen.step(toks[57:58], 57, [0]), want[57:58]) < F32_TOL
    with pytest.raises(ValueError):
        gen.step([raw["vocab"]], 58, [])
    with pytest.raises(ValueError):
        gen.step([0] * 10, raw["max_positions"] - 5, [])


@pytest.mark.parametrize("graph", [False, True])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_greedy_generation(bench, dtype, graph):
    """Greedy tokens through the generator equal the argmax of the restatement on the same tokens
    (float32: the free-running sequence itself)."""
    raw, w, path, _, _ = bench("odd")
    prompt = tokens_for(raw, 23, seed=5)
    gen = load(path, dtype)
    n = 40
    out = torch.zeros(1, n, dtype=torch.long, device="cuda")
    out[:, 0] = gen.prefill(torch.tensor(prompt))
    if graph:
        gen.enable_cuda_graph(warmup_pos=len(prompt))
    gen.generate(out, len(prompt), n - 1)
    gen.check()
    got = out[0].tolist()
    logits = oracle_logits(raw, w, prompt + got[:-1])[len(prompt) - 1 :]
    top = logits.topk(2, dim=-1).values
    margin = (1e-3 if dtype == torch.float32 else 0.15) * float(logits.pow(2).mean().sqrt())
    sure = (top[:, 0] - top[:, 1]) > margin
    assert int(sure.sum()) > n // 2
    assert torch.equal(torch.tensor(got)[sure], logits.argmax(-1)[sure])


def test_generate_script_from_a_checkpoint(bench, capsys):
    from megakernels_b200.scripts.generate import main, parse_cli

    raw, w, path, _, _ = bench("even")
    prompt = tokens_for(raw, 9, seed=3)
    argv = [f"model={path}", "dtype=float32", "ntok=12", "once", "prompt_ids=" + ",".join(map(str, prompt))]
    out = main(parse_cli(argv)).cpu()
    assert "Tokens per second" in capsys.readouterr().out and out.shape == (1, 12)
    logits = oracle_logits(raw, w, prompt + out[0, :-1].tolist())[len(prompt) - 1 :]
    assert torch.equal(out[0], logits.argmax(-1))
    assert torch.equal(main(parse_cli(argv + ["sched=wave"])).cpu(), out)


@pytest.mark.parametrize("sched", ["zz", "wave", "dag"])
def test_other_assignments_give_the_same_bits(bench, sched):
    raw, w, path, toks, _ = bench("even")
    a = run_cut(load(path, torch.bfloat16), toks[:30], [20])
    b = run_cut(load(path, torch.bfloat16, sched=sched), toks[:30], [20])
    assert torch.equal(a, b)


def test_attention_splits_and_state_blocks_do_not_matter(bench):
    from megakernels_b200.demos.hybrid.scheduler import HybridScheduleOptions

    raw, w, path, toks, want = bench("even")
    for opts in (HybridScheduleOptions(keys_per_split=5), HybridScheduleOptions(keys_per_split=10**6, state_columns=32)):
        assert rel(run_cut(load(path, options=opts), toks, [100]), want) < F32_TOL


def test_a_wait_that_runs_out_is_reported_and_the_context_survives(bench):
    """A phase that expects one arrival more than the schedule has: the launch gives up after its
    time budget, the status names the wait, and the next launch works."""

    raw, w, path, toks, want = bench("odd")
    gen = load(path)
    gen.step(toks[:10], 0, [])
    globs = gen.schedule.globs
    call = gen.interpreter.bind(globs)
    call.g.wait_timeout_ms = 50
    globs.arrivals[2, 1] += 1
    with pytest.raises(RuntimeError, match="TIMEOUT"):
        gen.step(toks[10:11], 10, [0])
    globs.arrivals[2, 1] -= 1
    call.g.wait_timeout_ms = 0
    assert rel(run_cut(gen, toks[:40], [30]), want[:40]) < F32_TOL


def test_bad_schedules_are_refused_on_the_host(bench):
    raw, w, path, toks, _ = bench("odd")
    for word, value in ((0, 9), (1, 99), (3, 10**6), (2, -1)):
        gen = load(path)
        ins = gen.schedule.globs.instructions
        ins[0, 0, word] = value
        with pytest.raises(RuntimeError, match="INVALID_ARGUMENT"):
            gen.step(toks[:1], 0, [0])


@pytest.mark.parametrize("dtype,tol", [("float32", F32_TOL), ("bfloat16", BF16_TOL)])
def test_trace_run(bench, tmp_path, dtype, tol):
    raw, w, path, toks, want = bench("odd")
    steps, at = [], 0
    for k, n in enumerate((40, 1, 3, 1, 55)):
        steps.append({"step": k, "entries": [{"id": "q", "tokens": toks[at : at + n], "want": [0, n - 1] if k != 1 else []}],
                      "end": []})
        at += n
    steps[-1]["end"] = ["q"]
    for k in range(5):  # more requests than slots, one after another; one name twice
        steps.append({"step": 5 + k, "entries": [{"id": f"n{k % 4}", "tokens": toks[: 10 + k], "want": [9 + k]}], "end": [f"n{k % 4}"]})
    r = subprocess.run([sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(path), "--dtype", dtype, "--out",
                        str(tmp_path), "--max-tokens", "128"], input="".join(json.dumps(s) + "\n" for s in steps),
                       text=True, capture_output=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {k}" for k in range(10)]
    read = lambda k: torch.frombuffer(bytearray((tmp_path / f"{k}.f32").read_bytes()), dtype=torch.float32).view(-1, raw["vocab"])  # noqa: E731
    assert rel(read(0), want[[0, 39]]) < tol and not (tmp_path / "1.f32").exists()
    assert rel(read(2), want[[41, 43]]) < tol and rel(read(4), want[[45, 99]]) < tol
    for k in range(5):
        assert rel(read(5 + k), want[9 + k : 10 + k]) < tol
