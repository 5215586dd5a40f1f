"""Shared by the Papusun tests: small configurations that differ from one another in every size and option, model
folders with random weights, and the oracle's view of them."""
from __future__ import annotations

import json
import os

import torch

import brolm_b200 as bb


def rot(base, dims, scaling=None):
    d = dict(base=base, dims=dims)
    if scaling:
        d["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return d


def left(heads, kv_heads, dim, vdim, scale, softcap, rotation):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, rot=rotation)
    if softcap:
        m["softcap"] = softcap
    return m


def right(heads, kv_heads, dim, vdim, conv):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv)


def parallel(a, r, left_scale, right_scale, ff=None):
    return dict(type="parallel", mixer=dict(left=a, right=r, left_scale=left_scale, right_scale=right_scale),
                mlp=dict(kind="dense", ff=ff) if ff else None)


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, size, base, kv_from=None, ff=None):
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, scale=scale,
             mask=dict(size=size), rot=dict(base=base, dims=rot_dim))
    if kv_from is not None:
        m["kv_from"] = kv_from
    return dict(type="latent_attention", mixer=m, mlp=dict(kind="dense", ff=ff) if ff else None)


def model(vocab, width, eps, side, logit_scale, layers):
    return dict(architecture="Papusun", vocab=vocab, width=width, norm=dict(eps=eps), token_side=dict(dim=side),
                logit_scale=logit_scale, layers=layers)


# S: a latent layer whose reader has more heads, other sizes and a wider window, across a parallel layer; more value heads
# than q/k heads in one recurrence; part of a head rotated; positions far beyond the scaling's original length.
CFG_S = model(96, 48, 1e-5, 12, 1.75, [
    latent(3, 12, 8, 10, 20, 24, 0.3, 37, 500.0, ff=40),
    parallel(left(4, 2, 16, 24, 0.4, 7.0, rot(100.0, 12, (3.0, 1.5, 5.0, 48))), right(6, 2, 16, 8, 3), 0.7, 1.3, ff=72),
    latent(5, 6, 8, 16, 32, 24, 0.45, 90, 500.0, kv_from=0),
    parallel(left(3, 3, 8, 8, 0.5, 0.0, rot(1000.0, 8)), right(2, 2, 24, 40, 5), -1.1, 0.6)])

# T: sizes that are no multiples of 8 or of 4, a convolution of one tap and one of two, a window of one token and two
# readers of it with windows of their own, no cap, one kv head, a layer without a feed-forward first.
CFG_T = model(51, 40, 1e-6, 5, 0.3, [
    parallel(left(6, 1, 10, 14, 0.35, 30.0, rot(10000.0, 6, (8.0, 1.0, 4.0, 64))), right(3, 1, 6, 13, 1), 1.0, 2.0),
    latent(2, 5, 6, 7, 18, 15, 0.5, 1, 10000.0, ff=28),
    latent(4, 9, 6, 12, 11, 15, 0.4, 64, 10000.0, kv_from=1, ff=20),
    parallel(left(2, 2, 12, 12, 0.3, 5.0, rot(50.0, 12, (2.0, 2.0, 2.0, 32))), right(4, 4, 5, 3, 2), 1.5, 0.5, ff=36),
    latent(1, 4, 6, 4, 9, 15, 0.6, 130, 10000.0, kv_from=1)])

# U: sizes the tensor-core kernels take (value heads of the key heads' size and of another), windows of a whole number of
# pages and one more, a reader whose window is narrower, q/k heads of the recurrence as long as a row of lanes and longer.
CFG_U = model(64, 64, 1e-5, 16, 2.0, [
    parallel(left(4, 4, 32, 32, 0.18, 25.0, rot(1000.0, 32, (5.0, 1.0, 4.0, 128))), right(2, 1, 128, 32, 4), 0.8, 0.9, ff=64),
    latent(4, 16, 16, 32, 32, 48, 0.2, 128, 10000.0, ff=128),
    parallel(left(4, 1, 32, 48, 0.2, 10.0, rot(10000.0, 16)), right(2, 2, 136, 16, 4), 1.25, 1.0, ff=64),
    latent(8, 32, 16, 16, 64, 48, 0.15, 65, 10000.0, kv_from=1, ff=64),
    latent(4, 16, 32, 16, 24, 32, 0.2, 200, 300.0)])

CONFIGS = {"S": (CFG_S, 3, 0.15), "T": (CFG_T, 4, 0.2), "U": (CFG_U, 5, 0.15)}      # name -> (config, seed, weight std)


def shape_up(name: str, t: torch.Tensor) -> torch.Tensor:
    """Random vectors lie around 0, where the design's own would hide: gains around 1, the newest tap of a convolution
    around 1, decays from nearly 1 (a state that lasts) to a half."""
    leaf = name.rsplit(".", 1)[-1]
    if leaf.startswith("norm") or name.endswith(".norm"):
        return t + 1.0
    if leaf == "conv":
        t = t.clone()
        t[:, -1] += 1.0
        return t
    if leaf == "A_log":
        return torch.linspace(-5.0, 0.0, t.numel(), dtype=torch.float32).to(t.dtype) + t
    return t


def write_folder(config: dict, folder: str, seed: int, std: float, store) -> str:
    from safetensors.torch import load_file, save_file
    bb.write_random_model(bb.PapusunConfig.from_dict(config), folder, seed=seed, weight_std=std, norm_std=0.3, dtype=store)
    path = os.path.join(folder, "model.safetensors")
    save_file({k: shape_up(k, v.float()).to(v.dtype).contiguous() for k, v in load_file(path).items()}, path + ".new")
    os.replace(path + ".new", path)
    return folder


def make_folder(tmp_path, name: str, store=torch.float32) -> str:
    cfg, seed, std = CONFIGS[name]
    folder = os.path.join(str(tmp_path), f"papusun_{name}_{str(store).split('.')[-1]}")
    if not os.path.exists(os.path.join(folder, "model.safetensors")):
        write_folder(cfg, folder, seed, std, store)
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
