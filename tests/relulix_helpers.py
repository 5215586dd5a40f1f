"""Shared by the Relulix tests: small configurations that differ from one another in every size and option, model
folders with random weights, and the oracle's view of them."""
from __future__ import annotations

import json
import os

import torch

import brolm_b200 as bb


def rot(base, dims, scaling=None):
    d = dict(base=base, dims=dims)
    if scaling:
        d["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return d


def attention(heads, kv_heads, dim, vdim, scale, softcap, size, rotation, kv_from=None, mlp=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, rot=rotation)
    if softcap:
        m["softcap"] = softcap
    if size:
        m["mask"] = dict(size=size)
    if kv_from is not None:
        m["kv_from"] = kv_from
    return dict(type="attention", mixer=m, mlp=mlp)


def retention(heads, dim, vdim, decay, rotation, mlp=None):
    return dict(type="retention", mixer=dict(heads=heads, dim=dim, vdim=vdim, decay=list(decay), rot=rotation), mlp=mlp)


def moe(ff, limit, experts, top):
    return dict(kind="moe", expert=dict(ff=ff, limit=limit), router=dict(experts=experts, top=top))


ROT_S = rot(100.0, 8, (2.0, 32, 8.0, 1.0))
ROT_U = rot(1000.0, 24, (8.0, 64, 16.0, 2.0))

# S: every routed layer uses all of its experts, so nothing hangs on a discrete choice and a rounded run can be held
# against the oracle.  Value heads smaller than key heads; a reader with more query heads and a wider window than the
# layer whose keys and values it reads, across a retention layer; no cap there; a layer without experts.
CFG_S = dict(
    architecture="Relulix", vocab=96, width=48, norm=dict(eps=1e-5), embedding=dict(scale=3.0),
    layers=[attention(4, 2, 16, 8, 0.3, 20.0, 37, ROT_S, mlp=moe(24, 1.5, 3, 3)),
            retention(3, 8, 16, (0.5, 0.9, 0.99), rot(50.0, 4), mlp=moe(16, 0.7, 2, 2)),
            attention(6, 2, 16, 8, 0.5, 0.0, 90, ROT_S, kv_from=0),
            attention(3, 3, 16, 16, 0.25, 5.0, 5, rot(10000.0, 16), mlp=moe(40, 3.0, 4, 4))])

# T: real routing (3 of 6, 1 of 4), head sizes that are no multiples of 8 or of 4, no window in one layer and two
# readers of it with windows of their own, one retention head with an odd value size, a window of one token, sizes that
# are no multiples of 16, one kv head.
CFG_T = dict(
    architecture="Relulix", vocab=50, width=40, norm=dict(eps=1e-6), embedding=dict(scale=0.5),
    layers=[retention(1, 6, 13, (0.97,), rot(10000.0, 6), mlp=moe(20, 1.0, 6, 3)),
            attention(3, 3, 12, 20, 0.3, 30.0, None, rot(500.0, 6), mlp=moe(36, 2.0, 4, 1)),
            attention(3, 3, 12, 20, 0.4, 8.0, 64, rot(500.0, 6), kv_from=1),
            attention(6, 3, 12, 20, 0.2, 30.0, 1, rot(500.0, 6), kv_from=1, mlp=moe(12, 0.5, 5, 2)),
            attention(6, 1, 8, 8, 0.35, 5.0, 70, rot(10000.0, 2, (4.0, 64, 32.0, 1.0)))])

# U: heads of one size that is a multiple of 16 (and one layer with larger value heads), windows of a whole number of
# pages, one more, and several pages; a reader whose window is narrower; positions far beyond the stretch's original
# length; a decay of exactly 1 and one of 0.999 over hundreds of tokens; every routed layer uses all of its experts.
CFG_U = dict(
    architecture="Relulix", vocab=64, width=32, norm=dict(eps=1e-5), embedding=dict(scale=5.5),
    layers=[attention(4, 4, 32, 32, 0.18, 25.0, 128, ROT_U, mlp=moe(16, 1.0, 4, 4)),
            attention(4, 4, 32, 32, 0.25, 50.0, 65, ROT_U, kv_from=0, mlp=moe(32, 2.5, 2, 2)),
            retention(2, 32, 64, (0.999, 1.0), rot(10000.0, 32), mlp=moe(16, 0.4, 2, 2)),
            attention(4, 1, 32, 48, 0.2, 10.0, 200, rot(1000.0, 32), mlp=moe(16, 1.2, 3, 3))])

CONFIGS = {"S": (CFG_S, 3, 0.15), "T": (CFG_T, 4, 0.2), "U": (CFG_U, 5, 0.2)}      # name -> (config, seed, weight std)


def make_folder(tmp_path, name: str, store=torch.float32) -> str:
    cfg, seed, std = CONFIGS[name]
    folder = os.path.join(str(tmp_path), f"relulix_{name}_{str(store).split('.')[-1]}")
    if not os.path.exists(os.path.join(folder, "model.safetensors")):
        bb.write_random_model(bb.RelulixConfig.from_dict(cfg), folder, seed=seed, weight_std=std, norm_std=0.3,
                              dtype=store)
    return folder


def oracle_inputs(folder: str):
    """(config dict, {name: tensor}) read without the framework's own reader."""
    from safetensors.torch import load_file
    with open(os.path.join(folder, "config.json")) as fh:
        config = json.load(fh)
    return config, load_file(os.path.join(folder, "model.safetensors"))


def random_prompts(vocab: int, lengths, seed: int):
    g = torch.Generator().manual_seed(seed)
    return [torch.randint(0, vocab, (n,), generator=g).tolist() for n in lengths]
