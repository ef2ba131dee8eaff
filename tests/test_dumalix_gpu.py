"""Dumalix on a GPU: every kernel path against the plain restatement, cuts of a sequence against
the whole, slots that are reused, chunk edges, sinks, long decoding, greedy generation."""

import json
import subprocess
import sys
from pathlib import Path

import pytest
import torch

from tests.dumalix_utils import (
    BF16_TOL, EVEN, F32_TOL, GROUPS, MODELS, ODD, WIDE, changed, chunked, latent, load, make_weights, model_config, oracle_logits, rel,
    run_cut, tokens_for, write_checkpoint,
)

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
DTYPES = [(torch.float32, F32_TOL), (torch.bfloat16, BF16_TOL)]
MAX_LEN = 512


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


def start(path, dtype=torch.float32, max_len=MAX_LEN, **kw):
    return load(path, dtype, max_len=max_len, **kw)


SINGLES = {
    "chunked": [chunked(6, 2, 16, 24, size=9)],
    "chunked_odd_head": [chunked(2, 2, 15, 10, size=13, rot=6, conv=3)],
    "chunked_one_position": [chunked(3, 1, 8, 8, size=1)],
    "chunked_whole_sequence": [chunked(4, 4, 64, 64, size=1000, base=10000.0)],
    "chunked_wide": [chunked(2, 1, 200, 256, size=30, rot=100)],
    "chunked_one_tap": [chunked(2, 1, 16, 16, size=20, conv=1)],
    "chunked_plain_rotation": [chunked(2, 1, 32, 16, size=20, scaling=None)],
    "chunked_mlp": [chunked(4, 2, 32, 32, size=17, ff=90)],
    "latent": [latent(6, 16, 8, 24, 32)],
    "latent_odd": [latent(3, 7, 4, 5, 13)],
    "latent_wide": [latent(4, 128, 64, 128, 512, base=10000.0)],
    "latent_many_heads": [latent(20, 16, 16, 8, 24)],
    "latent_prime_heads": [latent(13, 8, 2, 8, 16, scaling=None)],
    "latent_mlp": [latent(2, 32, 16, 32, 64, ff=77, limit=0.3)],
}


@pytest.mark.parametrize("dtype,tol", DTYPES)
@pytest.mark.parametrize("name", sorted(SINGLES))
def test_one_mechanism_alone(bench, name, dtype, tol):
    """A model of one layer: prompt, and token by token."""
    raw, w, path, toks, want = bench(f"one/{name}", model_config(SINGLES[name]), n=40)
    gen = start(path, dtype)
    assert rel(run_cut(gen, toks, [40]), want) < tol
    assert rel(run_cut(gen, toks, []), want) < tol


@pytest.mark.parametrize("taps", [1, 2, 5])
@pytest.mark.parametrize("loop", [None, (0, 1, 4), (1, 2, 2), (0, 2, 2)])
def test_loops_and_input_convolutions(bench, taps, loop):
    raw = model_config([latent(2, 8, 4, 8, 12, ff=20), chunked(2, 1, 8, 8, size=6)], taps=taps, loop=loop)
    raw, w, path, toks, want = bench(f"loop/{taps}/{loop}", raw, n=30)
    gen = start(path)
    for cuts in ([30], [], [2, 1, 3, 2, 9]):
        assert rel(run_cut(gen, toks, cuts), want) < F32_TOL, cuts


@pytest.mark.parametrize("dtype,tol", DTYPES)
@pytest.mark.parametrize("name", sorted(MODELS))
def test_prompt_and_every_layer_run(bench, name, dtype, tol):
    raw, w, path, toks, want = bench(name)
    gen = start(path, dtype)
    got, ref = [], []
    logits = gen.feed(toks, 0, list(range(len(toks))), layers_out=got)
    gen.check()
    oracle_logits(raw, w, toks, layers_out=ref)
    assert got[0].shape[0] == len(ref)
    for i, r in enumerate(ref):
        assert rel(got[0][i], r) < tol, f"run {i}"
    assert rel(logits, want) < tol


@pytest.mark.parametrize("dtype,tol", DTYPES)
@pytest.mark.parametrize("name", sorted(MODELS))
def test_token_by_token_equals_the_prompt(bench, name, dtype, tol):
    raw, w, path, toks, want = bench(name)
    assert rel(run_cut(start(path, dtype), toks, []), want) < tol


@pytest.mark.parametrize("cuts", [[2] * 75, [3, 2, 5, 2, 7, 11, 2, 13, 1, 1, 17, 2], [1, 149], [149, 1], [64, 64, 22], [33] * 5])
@pytest.mark.parametrize("name", ["odd", "even", "ragged", "groups"])
def test_portions_of_several_sizes(bench, name, cuts):
    raw, w, path, toks, want = bench(name)
    assert rel(run_cut(start(path), toks, cuts), want) < F32_TOL


@pytest.mark.parametrize("name,cuts", [("even", [2] * 75), ("wide", [3, 2, 5, 128, 2, 7]), ("groups", [70, 1, 1, 60])])
def test_portions_in_bf16(bench, name, cuts):
    raw, w, path, toks, want = bench(name)
    assert rel(run_cut(start(path, torch.bfloat16), toks, cuts), want) < BF16_TOL


@pytest.mark.parametrize("dtype,tol", DTYPES)
@pytest.mark.parametrize("portion", [2, 5, 16, 50])
@pytest.mark.parametrize("name", ["odd", "even"])
def test_small_rings_wrap(bench, name, portion, dtype, tol):
    """Prompts longer than the portion limit are cut inside; with it the chunks' rings shrink to
    chunk + portion rows and wrap many times."""
    raw, w, path, toks, want = bench(name)
    gen = start(path, dtype, portion=portion)
    assert min(r.ring for r in gen.model.state.rows.values()) < 150
    assert rel(run_cut(gen, toks, [150]), want) < tol
    assert rel(run_cut(gen, toks, [portion, 1, portion, 1, 1, 2 * portion + 1], slot=1), want) < tol
    assert rel(run_cut(gen, toks, [100], slot=2), want) < tol


@pytest.mark.parametrize("name", ["odd", "even", "groups"])
def test_peaked_attention_at_every_edge(bench, name):
    """Large scores: single keys dominate, so each position's logits depend on exactly which keys it
    sees - chunk edges, far keys and the first tokens included."""
    raw, w, path, toks, want = bench(f"peaked/{name}", MODELS[name], n=130, qk_gain=4.0)
    gen = start(path, portion=40)
    for cuts in ([130], [], [7, 4, 11, 1, 1, 29, 28, 2, 2], [12, 12, 12, 12]):
        assert rel(run_cut(gen, toks, cuts), want) < 2 * F32_TOL, cuts


def needle_model(layer, needle, gain):
    """One layer whose keys stand out for one token and whose queries all look for it."""
    raw = model_config([layer], vocab=40)
    w = make_weights(raw)
    w["l0.canon1"].zero_()
    w["l0.norm1"].zero_()
    W = raw["width"]
    e = torch.randn(W, generator=torch.Generator().manual_seed(7))
    w["embed"][:, 0] = 4.0  # every token's query: channel 0
    w["embed"][needle] = e.to(torch.bfloat16)
    w["embed"][needle, 0] = 4.0
    h = w["embed"][needle].double()
    h = h / h.pow(2).mean().sqrt()
    h[0] = 0
    one = torch.randn(layer["mixer"]["dim"], generator=torch.Generator().manual_seed(8), dtype=torch.float64)
    return raw, w, (gain * h / W).to(torch.bfloat16), one


@pytest.mark.parametrize("dtype,tol", DTYPES)
@pytest.mark.parametrize("place", ["first", "last", "before"])
@pytest.mark.parametrize("decoded", [False, True])
def test_one_outstanding_key_just_inside_and_outside_a_chunk(tmp_path, place, decoded, dtype, tol):
    """One token's key towers over all others; the query is its chunk's last position.  The key is at
    the chunk's first position, at the query's own left, or just before the chunk: seen, seen, not."""
    size, needle = 16, 7
    layer = chunked(2, 1, 16, 24, size=size, rot=2, base=1e6, scaling=None, conv=1, scale=1.0)
    raw, w, h, one = needle_model(layer, needle, 6.0)
    w["l0.mix.q"].zero_(), w["l0.mix.k"].mul_(0.05)
    w["l0.mix.q"][:, 0] = one.repeat(2).to(torch.bfloat16)
    w["l0.mix.k"] += (one[:, None] * h[None, :].double()).to(torch.bfloat16)
    for n in "qk":
        w[f"l0.mix.{n}.norm"][:] = 1.5
        w[f"l0.mix.{n}.norm"][:2] = 0.0  # the rotated pair says nothing here
        w[f"l0.mix.{n}.conv"][:] = 1.0
    w["l0.mix.sink"][:], w["l0.mix.temp"][:] = 20.0, 1.0
    query = 4 * size - 1
    at = {"first": query - size + 1, "last": query - 1, "before": query - size}[place]
    toks = [t if t != needle else 8 for t in tokens_for(raw, query + 1)]
    without = list(toks)
    toks[at] = needle
    want = oracle_logits(raw, w, toks)
    shows = rel(oracle_logits(raw, w, without)[query:], want[query:]) > 5e-2
    assert shows == (place != "before"), "the test's needle does not show"
    path = write_checkpoint(tmp_path / "c", raw, w)
    got = run_cut(start(path, dtype), toks, [query, 1] if decoded else [query + 1])
    assert rel(got, want) < tol


@pytest.mark.parametrize("dtype,tol", DTYPES)
@pytest.mark.parametrize("decoded", [False, True])
@pytest.mark.parametrize("at", [0, 1, 63, 64, 200])
def test_one_outstanding_latent_far_back(tmp_path, at, decoded, dtype, tol):
    """A latent attention finds one key among hundreds, wherever it lies."""
    needle, n = 7, 301
    layer = latent(2, 16, 2, 24, 32, base=1e6, scaling=None, scale=1.0)
    raw, w, h, one = needle_model(layer, needle, 30.0)
    w["l0.mix.q"].zero_(), w["l0.mix.dkv"].mul_(0.3)
    w["l0.mix.q"][:16, 0] = one.to(torch.bfloat16)
    w["l0.mix.q"][18:34, 0] = one.to(torch.bfloat16)
    w["l0.mix.dkv"][5] = h
    w["l0.mix.uk"].mul_(0.05)
    w["l0.mix.uk"][:, 5] += one.repeat(2).to(torch.bfloat16)
    toks = [t if t != needle else 8 for t in tokens_for(raw, n)]
    without = list(toks)
    toks[at] = needle
    want = oracle_logits(raw, w, toks)
    assert rel(oracle_logits(raw, w, without)[-1:], want[-1:]) > 5e-2, "the test's needle does not show"
    path = write_checkpoint(tmp_path / "c", raw, w)
    got = run_cut(start(path, dtype), toks, [n - 1, 1] if decoded else [n])
    assert rel(got, want) < tol


@pytest.mark.parametrize("dtype,tol", DTYPES)
def test_sinks_and_temperatures_of_any_size(bench, dtype, tol):
    """A sink that swallows everything, one far below all scores, temperatures that are zero or negative."""
    raw = model_config([chunked(4, 2, 16, 16, size=20, ff=30)])
    w = make_weights(raw)
    w["l0.mix.sink"][:] = torch.tensor([200.0, -200.0, 0.0, 3.0])
    w["l0.mix.temp"][:] = torch.tensor([1.0, -4.0, 0.0, 2.5])
    toks = tokens_for(raw, 70)
    want = oracle_logits(raw, w, toks)
    import tempfile

    with tempfile.TemporaryDirectory() as d:
        gen = start(write_checkpoint(Path(d) / "c", raw, w), dtype)
    assert rel(run_cut(gen, toks, [70]), want) < tol
    assert rel(run_cut(gen, toks, [3]), want) < tol


@pytest.mark.parametrize("dtype,tol", DTYPES)
def test_far_keys_and_long_decoding(bench, dtype, tol):
    """Decoded tokens after a short prompt: latents hundreds of tokens back, chunks and rings that
    pass under single tokens, inputs of the convolutions carried all the way."""
    raw, w, path, toks, want = bench("long", EVEN, n=400, qk_gain=2.0)
    gen = start(path, dtype, portion=32)
    assert rel(run_cut(gen, toks, [50]), want) < 1.5 * tol


def test_many_tiles_of_queries_and_keys(bench):
    """Prompts of several hundred tokens: chunk edges inside and between tiles of the prefill attention."""
    raw = model_config([chunked(2, 1, 64, 64, size=150, ff=64), latent(2, 64, 32, 64, 64), chunked(2, 2, 32, 128, size=64)], width=128)
    raw, w, path, toks, want = bench("tiles", raw, n=700, qk_gain=2.0)
    gen = start(path, torch.bfloat16, max_len=800)
    for cuts in ([700], [300, 399, 1], [129, 1, 130, 64, 65, 311]):
        assert rel(run_cut(gen, toks, cuts), want) < BF16_TOL, cuts


@pytest.mark.parametrize("dtype,tol", DTYPES)
def test_requests_in_turn_and_slots_used_again(bench, dtype, tol):
    """Requests of unequal length, interleaved over all slots, then their slots again."""
    raw, w, path, toks, _ = bench("odd")
    gen = start(path, dtype, portion=24)
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


@pytest.mark.parametrize("name", ["even", "odd"])
def test_logits_do_not_depend_on_slot_or_history(bench, name):
    """Bit-identical decode whatever ran before and wherever the sequence lives."""
    raw, w, path, toks, _ = bench(name)
    gen = start(path, torch.bfloat16)
    a = run_cut(gen, toks[:60], [40], slot=0)
    run_cut(gen, toks[30:], [100], slot=2)
    b = run_cut(gen, toks[:60], [40], slot=2)
    c = run_cut(start(path, torch.bfloat16), toks[:60], [40], slot=1)
    assert torch.equal(a, b) and torch.equal(a, c)


def test_wanted_places_and_limits(bench):
    raw, w, path, toks, want = bench("odd")
    gen = start(path, portion=20, max_len=60)
    got = gen.step(toks[:55], 0, [54, 0, 21, 20])
    assert rel(got, want[[54, 0, 21, 20]]) < F32_TOL
    assert gen.step(toks[55:57], 55, []).shape == (0, raw["vocab"])
    assert rel(gen.step(toks[57:58], 57, [0]), want[57:58]) < F32_TOL
    with pytest.raises(ValueError):
        gen.step([raw["vocab"]], 58, [])
    with pytest.raises(ValueError):
        gen.step([0] * 3, 58, [])


@pytest.mark.parametrize("graph", [False, True])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", ["odd", "groups"])
def test_greedy_generation(bench, name, dtype, graph):
    """Greedy tokens through the generator equal the argmax of the restatement on the same tokens."""
    raw, w, path, _, _ = bench(name)
    prompt = tokens_for(raw, 23, seed=5)
    gen = start(path, dtype)
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
    argv = [f"model={path}", "dtype=float32", "ntok=12", "once", "max_len_override=300", "prompt_ids=" + ",".join(map(str, prompt))]
    out = main(parse_cli(argv)).cpu()
    assert "Tokens per second" in capsys.readouterr().out and out.shape == (1, 12)
    logits = oracle_logits(raw, w, prompt + out[0, :-1].tolist())[len(prompt) - 1 :]
    assert torch.equal(out[0], logits.argmax(-1))
    assert torch.equal(main(parse_cli(argv + ["sched=wave"])).cpu(), out)


@pytest.mark.parametrize("sched", ["zz", "wave", "dag"])
def test_other_assignments_give_the_same_bits(bench, sched):
    raw, w, path, toks, _ = bench("even")
    a = run_cut(start(path, torch.bfloat16), toks[:30], [20])
    b = run_cut(start(path, torch.bfloat16, sched=sched), toks[:30], [20])
    assert torch.equal(a, b)


@pytest.mark.parametrize("dtype,tol", DTYPES)
def test_attention_splits_do_not_matter(bench, dtype, tol):
    from megakernels_b200.demos.hybrid.scheduler import HybridScheduleOptions

    for name in ("even", "groups"):
        raw, w, path, toks, want = bench(name)
        for opts in (HybridScheduleOptions(keys_per_split=5), HybridScheduleOptions(keys_per_split=10**6)):
            assert rel(run_cut(start(path, dtype, options=opts), toks, [100]), want) < tol


def test_a_wait_that_runs_out_is_reported_and_the_context_survives(bench):
    """A phase that expects one arrival more than the schedule has: the launch gives up after its
    time budget, the status names the wait, and the next launch works."""
    raw, w, path, toks, want = bench("odd")
    gen = start(path)
    gen.step(toks[:10], 0, [])
    globs = gen.schedule.globs
    call = gen.interpreter.bind(globs)
    call.g.wait_timeout_ms = 50
    globs.arrivals[1, 9] += 1
    with pytest.raises(RuntimeError, match="TIMEOUT"):
        gen.step(toks[10:11], 10, [0])
    globs.arrivals[1, 9] -= 1
    call.g.wait_timeout_ms = 0
    assert rel(run_cut(gen, toks[:40], [30]), want[:40]) < F32_TOL


def test_bad_schedules_are_refused_on_the_host(bench):
    raw, w, path, toks, _ = bench("odd")

    def refused(op, word, value):
        gen = start(path)
        ins = gen.schedule.globs.instructions
        q, k = (int(x) for x in (ins[:, :, 0] == op).nonzero()[0])
        ins[q, k, word] = value
        with pytest.raises(RuntimeError, match="INVALID_ARGUMENT"):
            gen.step(toks[:1], 0, [0])

    refused(8, 1, 4)  # a run that starts no pass
    refused(8, 3, 10**6)
    refused(9, 3, 21)  # rows of two heads
    refused(10, 2, -1)
    refused(5, 2, 1)  # half a gated unit
    refused(3, 2, 77)
    refused(1, 0, 11)


@pytest.mark.parametrize("dtype,tol", [("float32", F32_TOL), ("bfloat16", BF16_TOL)])
def test_trace_run(bench, tmp_path, dtype, tol):
    raw, w, path, toks, want = bench("groups")
    steps, at = [], 0
    for k, n in enumerate((40, 1, 3, 1, 55)):
        steps.append({"step": k, "entries": [{"id": "q", "tokens": toks[at : at + n], "want": [0, n - 1] if k != 1 else []}], "end": []})
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
