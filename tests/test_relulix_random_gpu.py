"""Relulix models drawn at random (layer order, every size, head counts, windows, which layer reads whose keys and values,
decays, rotations, stretches, experts, limits) through the engine against the plain implementation: a prompt step of
three unequal requests, tokens one by one (past a window's edge when one lies near), and the same once more on the slots,
pages and states that were given back.  In float32 the bar of a request is the larger of 2e-5 and eight times the error
the plain implementation itself makes when it runs in float32.  In bfloat16 the drawn routers use all their experts (no
discrete choice) and sizes that reach the tensor-core kernels are drawn more often; the bars are on the typical row and on
nine rows in ten: twice what rounding alone makes of them on the plain implementation."""
import os
import random

import pytest
import torch

import brolm_b200 as bb
from tests.plain import relulix_plain as plain
from tests.relulix_helpers import attention, moe, oracle_inputs, random_prompts, retention, rot

pytestmark = pytest.mark.gpu


def draw_mlp(rng, discrete):
    if rng.random() < 0.25:
        return None
    experts = rng.choice([1, 2, 3, 4, 6, 9])
    return moe(rng.choice([8, 12, 20, 40, 72]), rng.choice([0.3, 1.0, 2.5]), experts,
               rng.randint(1, experts) if discrete else experts)


def draw_rot(rng, dim):
    scaling = rng.choice([None, (2.0, 16, 4.0, 1.0), (8.0, 64, 32.0, 1.0), (40.0, 128, 16.0, 2.0)])
    return rot(rng.choice([100.0, 10000.0]), 2 * rng.randint(1, dim // 2), scaling)


def draw_layers(rng, discrete, tensor_sizes):
    layers = []
    for i in range(rng.randint(1, 6)):
        mlp = draw_mlp(rng, discrete)
        if rng.random() < 0.35:
            heads, d = rng.choice([1, 2, 3, 6]), rng.choice([4, 6, 8, 20, 32, 64])
            r = draw_rot(rng, d)
            r.pop("scaling", None)
            layers.append(retention(heads, d, rng.choice([4, 7, 16, 32, 64]),
                                    [rng.choice([0.5, 0.9, 0.97, 0.999, 1.0]) for _ in range(heads)], r, mlp=mlp))
            continue
        own = [j for j, l in enumerate(layers) if l["type"] == "attention" and "kv_from" not in l["mixer"]]
        size = rng.choice([None, 1, 2, 5, 31, 63, 64, 65, 100, 128, 150])
        scale, cap = rng.choice([0.1, 0.3, 1.0]), rng.choice([0.0, 5.0, 30.0])
        if own and rng.random() < 0.5:
            j = rng.choice(own)
            m = layers[j]["mixer"]
            layers.append(attention(m["kv_heads"] * rng.choice([1, 2, 4]), m["kv_heads"], m["dim"], m["vdim"], scale, cap, size,
                                    m["rot"], kv_from=j, mlp=mlp))
            continue
        kv = rng.choice([1, 2, 3])
        d = rng.choice([16, 32, 64] if tensor_sizes else [4, 6, 8, 16, 20, 32, 64])
        dv = rng.choice([d, d, 16, 48, 80] if tensor_sizes else [d, 4, 8, 12, 32, 80])
        layers.append(attention(kv * rng.choice([1, 2, 4]), kv, d, dv, scale, cap, size, draw_rot(rng, d), mlp=mlp))
    return layers


def draw_config(seed, discrete=True, tensor_sizes=False):
    rng = random.Random(seed)
    return dict(architecture="Relulix", vocab=rng.choice([37, 64, 200, 577]), width=rng.choice([24, 40, 72, 136, 312]),
                norm=dict(eps=rng.choice([1e-5, 1e-6])), embedding=dict(scale=rng.choice([0.5, 1.0, 4.0, 12.0])),
                layers=draw_layers(rng, discrete, tensor_sizes))


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
    bb.write_random_model(bb.RelulixConfig.from_dict(draw_config(seed)), folder, seed=seed, weight_std=0.15, norm_std=0.3,
                          dtype=torch.float32)
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
    bb.write_random_model(bb.RelulixConfig.from_dict(draw_config(seed, discrete=False, tensor_sizes=True)), folder, seed=seed,
                          weight_std=0.15, norm_std=0.3, dtype=torch.bfloat16)
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
