"""Papusun without a GPU: configuration, layout, tensor names, what the cache keeps (also for layers that read another
layer's latents), the tables the parts build on the host, and the oracle's own consistency."""
import copy
import json
import os

import pytest
import torch

import brolm_b200 as bb
from brolm_b200 import kernels
from brolm_b200.cache import Cache, KVSpec, StateSpec
from brolm_b200.config import ConfigError
from brolm_b200.parts import RotaryEmbedding, part_class
from tests.papusun_helpers import CFG_S, CFG_T, CFG_U, make_folder, oracle_inputs, random_prompts, rot
from tests.plain import papusun_plain as plain

F64 = torch.float64


def test_config_is_chosen_by_its_architecture_key(tmp_path):
    path = os.path.join(str(tmp_path), "config.json")
    with open(path, "w") as fh:
        json.dump(CFG_S, fh)
    cfg = bb.load_config(path)
    assert isinstance(cfg, bb.PapusunConfig) and cfg.width == 48 and len(cfg.layers) == 4
    assert bb.PapusunConfig.from_dict(cfg.to_dict()) == cfg
    assert cfg.logit_scale == 1.75 and cfg.eps == 1e-5 and cfg.side_dim == 12


@pytest.mark.parametrize("edit,what", [
    (lambda c: c["layers"][0].update(type="other"), "type"),
    (lambda c: c["layers"][1]["mixer"].pop("left"), "left"),
    (lambda c: c["layers"][1]["mixer"].pop("right_scale"), "right_scale"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][1]["mixer"]["left"].pop("scale"), "scale"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=18), "dims"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"]["scaling"].pop("high"), "high"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"]["scaling"].update(low=9.0), "low"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(kv_heads=4), "kv_heads"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(conv=0), "conv"),
    (lambda c: c["layers"][0]["mixer"].pop("q_rank"), "q_rank"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=10), "dims"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=1), "kv_from"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=2), "kv_from"),
    (lambda c: c["layers"][2]["mixer"].update(kv_rank=16), "kv_rank"),
    (lambda c: c["layers"][2]["mixer"].update(rot=dict(base=50.0, dims=8)), "rot"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "kind"),
    (lambda c: c["layers"][0]["mlp"].pop("ff"), "ff"),
    (lambda c: c["norm"].pop("eps"), "eps"),
    (lambda c: c.pop("token_side"), "dim"),
    (lambda c: c.pop("logit_scale"), "logit_scale"),
])
def test_bad_configurations_are_named(edit, what):
    c = copy.deepcopy(CFG_S)
    edit(c)
    with pytest.raises(ConfigError) as e:
        bb.PapusunConfig.from_dict(c)
    assert what in str(e.value)


def test_layout_names_and_caches():
    m = bb.Model(bb.PapusunConfig.from_dict(CFG_S), dtype="float32", device="cpu")
    names = m.expected_tensors()
    for n in ("embed", "side.embed", "head", "final.norm", "l0.norm1", "l0.norm2", "l0.mix.dq", "l0.mix.dq.norm", "l0.mix.uq",
              "l0.mix.dkv", "l0.mix.dkv.norm", "l0.mix.uk", "l0.mix.uv", "l0.mix.g", "l0.mix.o", "l0.mlp.gate", "l0.side.gate",
              "l1.mix.left.q.b", "l1.mix.left.v", "l1.mix.right.q.conv", "l1.mix.right.A_log", "l1.mix.right.dt_bias",
              "l1.mix.right.b", "l1.mix.right.a", "l1.mix.right.norm", "l2.mix.uk", "l3.side.norm", "l3.side.proj"):
        assert n in names, n
    for n in ("l2.mix.dkv", "l2.mix.dkv.norm", "l2.norm2", "l2.mlp.gate", "l3.norm2", "l1.mix.left.o.b", "l1.mix.right.q.b",
              "l0.mix.q", "l0.mix.sink"):
        assert n not in names, n
    assert names["side.embed"].shape == (96, 48) and not names["head"].optional
    assert names["l0.mix.g"].shape == (3, 48) and names["l0.mix.dkv"].shape == (32, 48) and names["l0.mix.uq"].shape == (60, 20)
    assert names["l1.mix.right.v.conv"].shape == (48, 3) and names["l1.mix.right.norm"].shape == (8,)
    assert m.layout.head.scale == 1.75
    specs = m.cache_specs()
    state = kernels.decay_state_size(6, 16, 8) + 3 * (2 * 2 * 16 + 6 * 8)
    # layer 2 reads layer 0's latents through a wider window, which is what layer 0's cache then keeps
    assert specs[0] == KVSpec(1, 32, 90, values=False) and specs[2] is None
    assert specs[1] == (KVSpec(2, 16, None, v_dim=24), StateSpec((state,), torch.float32))
    t = bb.Model(bb.PapusunConfig.from_dict(CFG_T), dtype="float32", device="cpu").cache_specs()
    assert t[1] == KVSpec(1, 32, 130, values=False) and t[2] is None and t[4] is None
    assert t[0][1] == StateSpec((3 * 13 * 8,), torch.float32)            # one tap: nothing is kept beside the state
    u = bb.Model(bb.PapusunConfig.from_dict(CFG_U), dtype="float32", device="cpu").cache_specs()
    assert u[1] == KVSpec(1, 64, 128, values=False) and u[3] is None     # the reader's window is the narrower one


def test_the_shared_ring_holds_what_the_wider_window_sees():
    m = bb.Model(bb.PapusunConfig.from_dict(CFG_S), dtype="float32", device="cpu")
    cache = Cache(m.cache_specs(), 640, torch.float32, "cpu")
    assert cache.entries[2] is None and cache.entries[0].group.ring == 128
    s = cache.alloc_slot()
    cache.reserve({s: 300})
    rows = cache.write_rows(cache.entries[0].group_id, [s], [0], [300])
    assert (rows >= 0).sum() == 128 and (rows[300 - 90:] >= 0).all()


def test_parts_refuse_what_they_cannot_do():
    lat, delta, side = (part_class("mixer", "latent_attention"), part_class("mixer", "gated_delta_rule"),
                        part_class("feedforward", "token_side"))
    base = dict(hidden=8, heads=2, dim=4, rot_dim=4, vdim=4, kv_rank=8, scale=1.0, eps=1e-5)
    for kw in (dict(gate="row"), dict(lends_kv=True, borrows_kv=True)):
        with pytest.raises(ValueError):
            lat(**base, **kw)
    for kw in (dict(heads=3, kv_heads=2), dict(taps=0), dict(dim=600)):
        with pytest.raises(ValueError):
            delta(**{**dict(hidden=8, heads=2, kv_heads=2, dim=8, v_dim=8, taps=2, eps=1e-5), **kw})
    for kw in (dict(first=10), dict(activation="tanh")):
        with pytest.raises(ValueError):
            side(**{**dict(hidden=8, dim=4, vocab=9, table_cols=12, first=4), **kw})
    bands = dict(factor=2.0, low=1.0, high=4.0, original=64)
    for kw in (dict(bands={**bands, "low": 0.0}), dict(bands=dict(factor=2.0)),
               dict(bands=bands, stretch=dict(factor=2.0, original=64, fast=8.0, slow=1.0))):
        with pytest.raises(ValueError):
            RotaryEmbedding(16, 100.0, **kw)


@pytest.mark.parametrize("r", [rot(100.0, 12, (3.0, 1.5, 5.0, 48)), rot(10000.0, 16, (8.0, 1.0, 4.0, 256)),
                               rot(50.0, 12, (2.0, 2.0, 2.0, 32)), rot(500.0, 6), rot(10000.0, 2, (4.0, 1.0, 4.0, 4))])
def test_rotation_table_against_the_oracle(r):
    part = RotaryEmbedding(head_dim=16, theta=r["base"], rotary_dim=r["dims"], bands=r.get("scaling"), pairing="interleaved")
    part.prepare(700, torch.device("cpu"))
    x = torch.zeros(700, 1, 16, dtype=F64)
    x[:, 0, 0:r["dims"]:2] = 1.0                               # u = 1, v = 0: the rotated pair is (cos, sin)
    y = plain.rotate(x, r)
    assert torch.allclose(part.table[..., 0].double(), y[:, 0, 0:r["dims"]:2], atol=1e-6)
    assert torch.allclose(part.table[..., 1].double(), y[:, 0, 1:r["dims"]:2], atol=1e-6)


def test_oracle_frequencies_in_their_three_bands():
    f = plain.frequencies(rot(10000.0, 32, (8.0, 1.0, 4.0, 512)))
    bare = plain.frequencies(rot(10000.0, 32))
    turns = [2 * torch.pi / x for x in bare]
    kinds = [0 if t < 128 else 2 if t > 512 else 1 for t in turns]
    assert set(kinds) == {0, 1, 2}
    for a, b, k in zip(f, bare, kinds):
        assert (k == 0 and a == b) or (k == 2 and abs(a - b / 8) < 1e-15) or (k == 1 and b / 8 < a < b)


def test_oracle_is_causal(tmp_path):
    for name in ("S", "T"):
        config, weights = oracle_inputs(make_folder(tmp_path, name))
        (p,) = random_prompts(config["vocab"], [110], seed=5)
        full = plain.forward(config, weights, p)
        assert torch.allclose(plain.forward(config, weights, p[:67]), full[:67], atol=1e-9)
        assert full.shape == (110, config["vocab"]) and bool(torch.isfinite(full).all())


def test_every_mechanism_moves_the_result(tmp_path):
    """A model without one of its mechanisms differs from itself by far more than rounding."""
    config, weights = oracle_inputs(make_folder(tmp_path, "S"))
    (p,) = random_prompts(config["vocab"], [130], seed=6)
    ref = plain.forward(config, weights, p)

    def moved(edit, tensors=None):
        c = copy.deepcopy(config)
        edit(c)
        return float((plain.forward(c, tensors or weights, p) - ref).abs().max() / ref.abs().max())
    mix = lambda c, i: c["layers"][i]["mixer"]
    assert moved(lambda c: mix(c, 0)["mask"].update(size=36)) > 1e-3
    assert moved(lambda c: mix(c, 2)["mask"].update(size=91)) > 1e-4
    assert moved(lambda c: mix(c, 1)["left"].update(softcap=0.0)) > 1e-4
    assert moved(lambda c: mix(c, 1)["left"]["rot"].pop("scaling")) > 1e-3
    assert moved(lambda c: mix(c, 1).update(right_scale=1.2)) > 1e-3
    assert moved(lambda c: c.update(logit_scale=1.7)) > 1e-3
    zero = lambda *names: {k: (torch.zeros_like(v) if k in names else v) for k, v in weights.items()}
    for names in (("l0.mix.g",), ("l1.mix.left.k.b",), ("l1.mix.right.b",), ("l1.mix.right.dt_bias",), ("l2.side.norm",),
                  ("side.embed",), ("l3.mix.right.q.conv",)):
        assert moved(lambda c: None, zero(*names)) > 1e-4, names


def test_oracle_delta_rule_against_its_own_definition():
    """With beta = 1 and no decay a key that comes back returns the value last written for it; in two pieces as in one."""
    g = torch.Generator().manual_seed(1)
    T, H, d, dv = 24, 2, 6, 5
    k = plain.unit_length(torch.randn(T, H, d, generator=g, dtype=F64))
    v = torch.randn(T, H, dv, generator=g, dtype=F64)
    k[20] = k[3]
    one = torch.ones(T, H, dtype=F64)
    o, _ = plain.delta_states(k, k, v, one, one)
    assert torch.allclose(o, v, atol=1e-5)                     # (unit vectors up to the 1e-6 under their root)
    decay, beta = torch.rand(T, H, generator=g, dtype=F64), torch.rand(T, H, generator=g, dtype=F64)
    q = torch.randn(T, H, d, generator=g, dtype=F64)
    full, S = plain.delta_states(q, k, v, decay, beta)
    a, Sa = plain.delta_states(q[:9], k[:9], v[:9], decay[:9], beta[:9])
    b, Sb = plain.delta_states(q[9:], k[9:], v[9:], decay[9:], beta[9:], Sa)
    assert torch.allclose(torch.cat([a, b]), full, atol=1e-12) and torch.allclose(Sb, S, atol=1e-12)


def test_oracle_window_edge_shows():
    g = torch.Generator().manual_seed(2)
    T, H, d, W = 30, 2, 8, 10
    k, v = torch.randn(T, 1, d, generator=g, dtype=F64), torch.randn(T, 1, 4, generator=g, dtype=F64)
    q = torch.zeros(T, H, d, dtype=F64)
    q[-1] = 4.0 * k[T - W, 0]                                  # the oldest key the last query sees
    inside = plain.softmax_attention(q, k, v, 1.0, window=W)[-1]
    assert torch.allclose(inside[0], v[T - W, 0], atol=0.05)
    assert float((plain.softmax_attention(q, k, v, 1.0, window=W - 1)[-1] - inside).abs().max()) > 0.1
