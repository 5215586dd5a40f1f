"""Papusun models drawn at random (layer order, every size, head counts, windows, which layer reads whose latents, taps,
rotations and their scaling, caps, scales) through the engine against the plain implementation: a prompt step of three
unequal requests, tokens one by one, and the same once more on the slots, pages and states that were given back.  In
float32 the bar of a request is the larger of 2e-5 and eight times the error the plain implementation itself makes when it
runs in float32.  In bfloat16 sizes that reach the tensor-core kernels are drawn more often; the bars are on the typical
row and on nine rows in ten: twice what rounding alone makes of them on the plain implementation."""
import os
import random

import pytest
import torch

import brolm_b200 as bb
from tests.plain import papusun_plain as plain
from tests.papusun_helpers import latent, left, model, oracle_inputs, parallel, random_prompts, right, rot, write_folder

pytestmark = pytest.mark.gpu


def draw_left(rng, tensor_sizes):
    kv = rng.choice([1, 2, 3])
    d = rng.choice([16, 32, 64, 80] if tensor_sizes else [4, 6, 8, 16, 20, 32, 64])
    dv = rng.choice([d, d, 16, 48, 112, 176] if tensor_sizes else [d, 3, 4, 12, 32, 80])
    scaling = rng.choice([None, (2.0, 1.0, 4.0, 16), (8.0, 1.0, 4.0, 64), (40.0, 2.0, 7.0, 128), (3.0, 1.5, 1.5, 32)])
    return left(kv * rng.choice([1, 2, 4]), kv, d, dv, rng.choice([0.1, 0.3, 1.0]), rng.choice([0.0, 5.0, 30.0]),
                rot(rng.choice([100.0, 10000.0]), 2 * rng.randint(1, d // 2), scaling))


def draw_right(rng):
    kv = rng.choice([1, 2, 3])
    return right(kv * rng.choice([1, 2, 3]), kv, rng.choice([4, 6, 16, 20, 64, 128, 140]), rng.choice([4, 7, 16, 24, 32, 64]),
                 rng.choice([1, 2, 3, 4, 4, 6]))


def draw_layers(rng, tensor_sizes):
    layers = []
    for i in range(rng.randint(1, 6)):
        ff = rng.choice([None, 20, 36, 64, 136])
        if rng.random() < 0.45:
            layers.append(parallel(draw_left(rng, tensor_sizes), draw_right(rng), rng.choice([1.0, 0.7, -1.3]),
                                   rng.choice([1.0, 0.4, 1.6]), ff=ff))
            continue
        own = [j for j, l in enumerate(layers) if l["type"] == "latent_attention" and "kv_from" not in l["mixer"]]
        heads = rng.choice([1, 2, 3, 4, 8, 16, 20])
        dn, dv = rng.choice([4, 6, 16, 32]), rng.choice([3, 8, 16, 40])
        size, scale = rng.choice([1, 2, 5, 31, 63, 64, 65, 100, 128, 150]), rng.choice([0.1, 0.3, 0.6])
        q_rank = rng.choice([5, 8, 24, 40])
        if own and rng.random() < 0.5:
            j = rng.choice(own)
            m = layers[j]["mixer"]
            layers.append(latent(heads, dn, m["rot_dim"], dv, q_rank, m["kv_rank"], scale, size, m["rot"]["base"], kv_from=j, ff=ff))
        else:
            layers.append(latent(heads, dn, rng.choice([2, 6, 8, 16, 32]), dv, q_rank, rng.choice([5, 16, 24, 48, 100]), scale,
                                 size, rng.choice([100.0, 10000.0]), ff=ff))
    return layers


def draw_config(seed, tensor_sizes=False):
    rng = random.Random(seed)
    return model(rng.choice([37, 64, 200, 577]), rng.choice([24, 40, 72, 136, 312]), rng.choice([1e-5, 1e-6]),
                 rng.choice([1, 5, 8, 24]), rng.choice([0.25, 1.0, 1.5, 8.0]), draw_layers(rng, tensor_sizes))


MORE = 14


def run_twice(folder, dtype, reqs, lens):
    eng = bb.Engine(bb.load_model(folder, dtype=dtype), max_tokens=1024, max_slots=3)
    rounds = []
    for _ in range(2):
        slots = eng.open(3)
        got = [[] for _ in reqs]
        first = eng.step(slots, [p[:n] for p, n in zip(reqs, lens)], want=[list(range(n)) for n in lens])
        at = 0
        for b, n in enumerate(lens):
            got[b].append(first[at:at + n].clone())
            at += n
        for j in range(MORE):
            out = eng.step(slots, [[p[n + j]] for p, n in zip(reqs, lens)])
            for b in range(3):
                got[b].append(out[b:b + 1].clone())
        eng.close(slots)
        rounds.append([torch.cat(g).cpu() for g in got])
    return rounds


@pytest.mark.parametrize("seed", range(16))
def test_a_drawn_model_prompt_decode_and_the_same_again(tmp_path, seed):
    folder = os.path.join(str(tmp_path), "drawn")
    write_folder(draw_config(seed), folder, seed, 0.15, torch.float32)
    config, weights = oracle_inputs(folder)
    rng = random.Random(seed + 1000)
    lens = [rng.choice([1, 2, 17, 58, 66, 121, 200]) for _ in range(3)]
    reqs = random_prompts(config["vocab"], [n + MORE for n in lens], seed)
    refs = [plain.forward(config, weights, p) for p in reqs]
    plain.F64 = torch.float32
    try:
        own = [float((plain.forward(config, weights, p).double() - r).abs().max() / r.abs().max()) for p, r in zip(reqs, refs)]
    finally:
        plain.F64 = torch.float64
    bars = [max(2e-5, 8 * e) for e in own]
    rounds = run_twice(folder, "float32", reqs, lens)
    for b, (r, bar) in enumerate(zip(refs, bars)):
        err = float((rounds[0][b].double() - r).abs().max() / r.abs().max())
        assert err <= bar, f"request {b} of {lens[b]} + {MORE} tokens: {err:.2e} against a bar of {bar:.1e}"
        assert torch.equal(rounds[0][b], rounds[1][b]), "the second tenants of the slots see something of the first"


@pytest.mark.parametrize("seed", range(100, 110))
def test_a_drawn_model_in_bfloat16(tmp_path, seed):
    folder = os.path.join(str(tmp_path), "drawn16")
    write_folder(draw_config(seed, tensor_sizes=True), folder, seed, 0.15, torch.bfloat16)
    config, weights = oracle_inputs(folder)
    rng = random.Random(seed + 1000)
    lens = [rng.choice([1, 2, 17, 58, 66, 121, 200]) for _ in range(3)]
    reqs = random_prompts(config["vocab"], [n + MORE for n in lens], seed)
    rounds = run_twice(folder, "bfloat16", reqs, lens)
    errs = []
    for b, p in enumerate(reqs):
        ref = plain.forward(config, weights, p)
        errs += ((rounds[0][b].double() - ref).abs().amax(dim=1) / ref.abs().max()).tolist()
        assert torch.equal(rounds[0][b], rounds[1][b]), "the second tenants of the slots see something of the first"
    errs.sort()
    own = plain.rounding_errors(config, weights, reqs)
    for share in (0.5, 0.9):
        at = int(share * (len(errs) - 1))
        assert errs[at] <= 2 * own[at], f"{errs[at]:.2e} at {share} of the rows, {own[at]:.2e} by rounding alone"
