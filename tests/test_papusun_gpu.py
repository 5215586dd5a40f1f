"""Papusun through the engine against the plain implementation, in float32 and in bfloat16: whole requests
(every layer's stream too), prompts continued token by token across page borders and every window's edge, a long
prompt and then decoding around the rings, batches of unequal requests against each alone with slots, pages and
states used again, the first tokens, long decoding, greedy generation through the entry point, and the trace replay
and the command line as a user runs them."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import brolm_b200 as bb
from tests.papusun_helpers import make_folder, oracle_inputs, random_prompts
from tests.plain import papusun_plain as plain

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
ROOT = os.path.normpath(os.path.join(os.path.dirname(os.path.abspath(__file__)), ".."))

# Largest error of a logit against the float64 oracle, relative to the largest logit of the compared rows.
TOL = {"float32": 2e-5, "bfloat16": 4e-2}
STORE = {"float32": torch.float32, "bfloat16": torch.bfloat16}
CASES = [(name, dtype) for name in "STU" for dtype in ("float32", "bfloat16")]


@pytest.fixture(scope="module")
def setups(tmp_path_factory):
    tmp = tmp_path_factory.mktemp("papusun")
    out = {}
    for name, dtype in CASES:
        folder = make_folder(tmp, name, STORE[dtype])
        config, weights = oracle_inputs(folder)
        if dtype == "bfloat16":
            errs = plain.rounding_errors(config, weights, random_prompts(config["vocab"], [9, 64, 150, 300], seed=21))
            ROUNDING[name] = (errs[int(0.9 * (len(errs) - 1))], errs[-1])
        if dtype == "float32":
            FLOAT[name] = max(TOL["float32"], 4 * own_float_error(config, weights))
        out[(name, dtype)] = (folder, config, weights, bb.load_model(folder, dtype=dtype, device=DEV))
    return out


def rel(got, ref):
    ref = ref.double()
    return float((got.double().cpu() - ref).abs().max()) / max(float(ref.abs().max()), 1e-3)


def own_float_error(config, weights):
    """The largest error the plain implementation itself makes in float32 on the requests of these tests: a result that is
    divided by its own root mean square and happens to be small leaves some positions with fewer digits than others."""
    worst = 0.0
    for seed, lens in ((13, [1, 140, 17, 66, 130]), (19, [420]), (14, [300])):
        for p in random_prompts(config["vocab"], lens, seed):
            ref = plain.forward(config, weights, p)
            plain.F64 = torch.float32
            try:
                own = plain.forward(config, weights, p).double()
            finally:
                plain.F64 = torch.float64
            worst = max(worst, float((own - ref).abs().max() / ref.abs().max()))
    return worst


FLOAT: dict = {}        # name -> the bar of a float32 row (filled by the fixture)
# name -> (nine rows in ten, all rows) of the error that rounding alone makes on the oracle (filled by the fixture)
ROUNDING: dict = {}


def check(got, ref, dtype, what, name):
    """float32: every row within the bar.  bfloat16: nine rows in ten within twice what rounding alone makes of nine rows
    in ten of that model, and none beyond twice what it makes of any row (these small random models have single
    positions where a result that is normed is itself small, so that its rounding is large; a wrong key or a lost
    state moves every row by far more)."""
    ref = ref.double()
    rows = (got.double().cpu() - ref).abs().reshape(-1, ref.shape[-1]).amax(dim=1) / max(float(ref.abs().max()), 1e-3)
    if dtype == "float32":
        assert float(rows.max()) <= FLOAT[name], f"{what}: relative error {float(rows.max()):.3e} exceeds {FLOAT[name]:.0e}"
        # (what is wrong for a reason other than rounding is wrong at more than a row in ten)
        assert float(rows.sort().values[int(0.9 * (len(rows) - 1))]) <= TOL[dtype], what
        return
    q90 = float(rows.sort().values[int(0.9 * (len(rows) - 1))])
    most, worst = ROUNDING[name]
    assert q90 <= 2 * most and float(rows.max()) <= 2 * worst, \
        f"{what}: relative error {q90:.3e} at nine rows in ten, {float(rows.max()):.3e} at worst"


@pytest.mark.parametrize("name,dtype", CASES)
def test_whole_requests_and_every_stream(setups, name, dtype):
    _, config, weights, model = setups[(name, dtype)]
    eng = bb.Engine(model, max_tokens=512)
    for p in random_prompts(config["vocab"], [1, 2, 9, 16, 17, 33, 64, 65, 150, 300], seed=11):
        streams = []
        ref = plain.forward(config, weights, p, streams)
        (s,) = eng.open(1)
        model.keep_streams = []
        got = eng.step([s], [p], want=[list(range(len(p)))])
        kept, model.keep_streams = model.keep_streams, None
        eng.close([s])
        check(got, ref, dtype, f"whole request of {len(p)}", name)
        assert len(kept) == len(streams) == len(config["layers"])
        for i, (a, b) in enumerate(zip(kept, streams)):
            check(a, b, dtype, f"stream after run {i} of a request of {len(p)}", name)


@pytest.mark.parametrize("name,dtype", CASES)
def test_prompt_then_token_by_token(setups, name, dtype):
    """Decoding crosses the pages' borders, the windows' edges and the scaling's original length, from the cache of the
    layer itself and from that of the layer it reads, and goes on from the state and the inputs that a prompt left, in
    every place among sixteen tokens."""
    _, config, weights, model = setups[(name, dtype)]
    (p,) = random_prompts(config["vocab"], [150], seed=12)
    ref = plain.forward(config, weights, p)
    eng = bb.Engine(model, max_tokens=256)
    for first in (1, 2, 3, 15, 16, 17, 63, 64, 70, 100):
        (s,) = eng.open(1)
        rows = [eng.step([s], [p[:first]], want=[list(range(first))]).clone()]
        for t in range(first, len(p)):
            rows.append(eng.step([s], [[p[t]]]).clone())
        eng.close([s])
        check(torch.cat(rows), ref, dtype, f"{first} tokens, then one by one", name)


@pytest.mark.parametrize("name,dtype", [("S", "float32"), ("T", "float32"), ("U", "float32"), ("U", "bfloat16")])
def test_long_prompt_then_decoding_far_back(setups, name, dtype):
    """A prompt of several pages, longer than every ring, then decoding: the newest keys of the prompt are read from the
    rings (a reader's window may be wider or narrower than the layer's it reads), and the state has hundreds of tokens
    behind it."""
    _, config, weights, model = setups[(name, dtype)]
    (p,) = random_prompts(config["vocab"], [420], seed=19)
    ref = plain.forward(config, weights, p)
    eng = bb.Engine(model, max_tokens=448)
    (s,) = eng.open(1)
    first = 385
    rows = [eng.step([s], [p[:first]], want=[list(range(first))]).clone()]
    for t in range(first, len(p)):
        rows.append(eng.step([s], [[p[t]]]).clone())
    eng.close([s])
    check(torch.cat(rows), ref, dtype, "385 tokens, then one by one", name)


@pytest.mark.parametrize("name,dtype", CASES)
def test_unequal_batches_against_each_alone(setups, name, dtype):
    _, config, weights, model = setups[(name, dtype)]
    reqs = random_prompts(config["vocab"], [1, 140, 17, 66, 130], seed=13)
    refs = [plain.forward(config, weights, p) for p in reqs]
    eng = bb.Engine(model, max_tokens=64 + 192 + 64 + 128 + 192, max_slots=5)
    alone = bb.Engine(model, max_tokens=192, max_slots=1)

    def run(engine, ids):
        """Half of each request as its prompt, the rest one by one; shorter requests leave earlier."""
        slots = dict(zip(ids, engine.open(len(ids))))
        done = {i: max(1, len(reqs[i]) // 2) for i in ids}
        first = engine.step([slots[i] for i in ids], [reqs[i][:done[i]] for i in ids],
                            want=[list(range(done[i])) for i in ids])
        got, at = {}, 0
        for i in ids:
            got[i] = [first[at:at + done[i]].clone()]
            at += done[i]
        live = [i for i in ids if done[i] < len(reqs[i])]
        for i in ids:
            if i not in live:
                engine.close([slots[i]])
        while live:
            out = engine.step([slots[i] for i in live], [[reqs[i][done[i]]] for i in live])
            for r, i in enumerate(live):
                got[i].append(out[r:r + 1].clone())
                done[i] += 1
            for i in live:
                if done[i] == len(reqs[i]):
                    engine.close([slots[i]])
            live = [i for i in live if done[i] < len(reqs[i])]
        return {i: torch.cat(v) for i, v in got.items()}

    for ids in ([0, 1, 2, 3, 4], [4, 2, 1], [3, 0, 4, 1, 2]):         # the same cache and states, batch after batch
        together = run(eng, ids)
        for i in ids:
            check(together[i], refs[i], dtype, f"request {i} in batch {ids}", name)
            single = run(alone, [i])[i]
            # what else is in the batch changes nothing beyond rounding
            assert rel(together[i], single.cpu()) <= (FLOAT[name] if dtype == "float32" else 2 * TOL[dtype])
    assert eng.cache.live_slots == 0 and all(g.pool.held_pages == 0 for g in eng.cache.kv_groups)


@pytest.mark.parametrize("name,dtype", [("S", "float32"), ("S", "bfloat16"), ("T", "float32"), ("U", "float32")])
def test_long_decoding_from_the_first_tokens(setups, name, dtype):
    _, config, weights, model = setups[(name, dtype)]
    (p,) = random_prompts(config["vocab"], [300], seed=14)
    ref = plain.forward(config, weights, p)
    eng = bb.Engine(model, max_tokens=320)
    (s,) = eng.open(1)
    rows = [eng.step([s], [p[:1]]).clone()]
    for t in range(1, len(p)):
        rows.append(eng.step([s], [[p[t]]]).clone())
    eng.close([s])
    got = torch.cat(rows)
    check(got[:4], ref[:4], dtype, "the first tokens", name)
    check(got, ref, dtype, "300 tokens one by one", name)


def test_a_used_slot_starts_from_zero_again(setups):
    """A sequence that takes the slot (and with it the state rows and pages) of one that ended sees nothing of it."""
    _, config, weights, model = setups[("S", "float32")]
    a, b = random_prompts(config["vocab"], [90, 40], seed=18)
    ref = plain.forward(config, weights, b)
    eng = bb.Engine(model, max_tokens=128, max_slots=1)
    (s,) = eng.open(1)
    eng.step([s], [a])
    eng.step([s], [[3]])
    eng.close([s])
    (s2,) = eng.open(1)
    assert s2 == s
    got = [eng.step([s2], [b[:20]], want=[list(range(20))]).clone()]
    got += [eng.step([s2], [[t]]).clone() for t in b[20:]]
    eng.close([s2])
    check(torch.cat(got), ref, "float32", "the slot's second tenant", "S")


@pytest.mark.parametrize("name,dtype", CASES)
def test_greedy_generation_through_the_entry_point(setups, name, dtype):
    _, config, weights, model = setups[(name, dtype)]
    eng = bb.Engine(model, max_tokens=512)
    prompts = random_prompts(config["vocab"], [5, 70, 1, 23], seed=16)
    opts = bb.GenerateOptions(max_new_tokens=12, sampling=bb.SamplingParams(temperature=0.0), stop_on_eos=False)
    outs = bb.generate(eng, prompts, eos_id=-1, opts=opts)
    for p, o in zip(prompts, outs):
        assert len(o) == 12
        ids = list(p)
        for tok in o:
            row = plain.forward(config, weights, ids)[-1]
            scale = float(row.abs().max())
            assert float(row.max() - row[tok]) <= TOL[dtype] * scale * 2, "not the oracle's best token (beyond rounding)"
            ids.append(tok)
    assert eng.cache.live_slots == 0


def run_trace(folder, dtype, out, max_tokens, steps):
    text = "".join(json.dumps(s) + "\n" for s in steps)
    proc = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype,
                           "--out", out, "--max-tokens", str(max_tokens)], input=text, capture_output=True, text=True,
                          timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [l for l in proc.stdout.splitlines() if l.startswith("done")] == [f"done {s['step']}" for s in steps]


@pytest.mark.parametrize("name,dtype", [("S", "float32"), ("S", "bfloat16")])
def test_trace_replay(setups, tmp_path, name, dtype):
    folder, config, weights, _ = setups[(name, dtype)]
    V = config["vocab"]
    reqs = random_prompts(V, [75, 9, 140], seed=17)
    refs = [plain.forward(config, weights, p) for p in reqs]
    pre = [60, 1, 100]
    steps = [{"step": 0, "entries": [{"id": f"r{i}", "tokens": reqs[i][:pre[i]], "want": [0, pre[i] - 1]}
                                     for i in range(3)], "end": []}]
    expect = {0: torch.cat([refs[i][[0, pre[i] - 1]] for i in range(3)])}
    done, live, n = list(pre), [0, 1, 2], 1
    while live:
        steps.append({"step": n, "entries": [{"id": f"r{i}", "tokens": [reqs[i][done[i]]],
                                              "want": [0] if done[i] % 3 else []} for i in live],
                      "end": [f"r{i}" for i in live if done[i] + 1 == len(reqs[i])]})
        rows = [refs[i][done[i]:done[i] + 1] for i in live if done[i] % 3]
        if rows:
            expect[n] = torch.cat(rows)
        for i in live:
            done[i] += 1
        live = [i for i in live if done[i] < len(reqs[i])]
        n += 1
    out = str(tmp_path / "replay")
    run_trace(folder, dtype, out, 128 + 64 + 192, steps)
    got = [torch.from_numpy(np.fromfile(os.path.join(out, f"{s}.f32"), dtype="<f4").reshape(-1, V).copy()) for s in expect]
    assert [g.shape for g in got] == [r.shape for r in expect.values()]
    check(torch.cat(got), torch.cat(list(expect.values())), dtype, "the replay's rows", name)
    assert sorted(os.listdir(out)) == sorted(f"{s}.f32" for s in expect)


def test_greedy_from_the_command_line(setups):
    folder, config, weights, _ = setups[("T", "float32")]
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "run_model"), "--model", folder, "--dtype", "float32",
                        "--ids", "5,17,3,9", "--ids", "20 7", "--max-new", "6"], capture_output=True, text=True,
                       timeout=600)
    assert r.returncode == 0, r.stderr
    lines = r.stdout.splitlines()
    got = [list(map(int, lines[i + 1].split())) for i, l in enumerate(lines) if l == "--- completion ---"]
    assert [len(g) for g in got] == [6, 6]
    for p, o in zip(([5, 17, 3, 9], [20, 7]), got):            # the family has no start token: the ids as given
        ids = list(p)
        for tok in o:
            row = plain.forward(config, weights, ids)[-1]
            assert float(row.max() - row[tok]) <= 1e-4 * float(row.abs().max())
            ids.append(tok)
