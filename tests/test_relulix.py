"""Relulix without a GPU: configuration, layout, tensor names, what the cache keeps (also for layers that read another
layer's keys and values), the tables the parts build on the host, and the oracle's own consistency."""
import copy
import json
import os

import pytest
import torch

import brolm_b200 as bb
from brolm_b200.cache import Cache, CacheError, KVSpec, StateSpec, shared_spec
from brolm_b200.config import ConfigError
from brolm_b200.parts import RotaryEmbedding, part_class
from tests.relulix_helpers import CFG_S, CFG_T, CFG_U, make_folder, oracle_inputs, random_prompts, rot
from tests.plain import relulix_plain as plain

F64 = torch.float64


def test_config_is_chosen_by_its_architecture_key(tmp_path):
    path = os.path.join(str(tmp_path), "config.json")
    with open(path, "w") as fh:
        json.dump(CFG_S, fh)
    cfg = bb.load_config(path)
    assert isinstance(cfg, bb.RelulixConfig) and cfg.width == 48 and len(cfg.layers) == 4
    assert bb.RelulixConfig.from_dict(cfg.to_dict()) == cfg
    assert cfg.embedding_scale == 3.0 and cfg.eps == 1e-5


@pytest.mark.parametrize("edit,what", [
    (lambda c: c["layers"][0].update(type="other"), "type"),
    (lambda c: c["layers"][1]["mixer"].update(decay=[0.5, 0.9]), "decay"),
    (lambda c: c["layers"][1]["mixer"].update(decay=[0.5, 0.9, 1.5]), "decay"),
    (lambda c: c["layers"][1]["mixer"].pop("rot"), "rot"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=10), "dims"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"].pop("vdim"), "vdim"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][3]["mixer"]["rot"].update(dims=7), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("fast"), "fast"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=1), "kv_from"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=3), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=2), "kv_from"),
    (lambda c: c["layers"][2]["mixer"].update(vdim=16), "vdim"),
    (lambda c: c["layers"][2]["mixer"].update(rot=dict(base=50.0, dims=8)), "rot"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=4), "top"),
    (lambda c: c["layers"][0]["mlp"]["expert"].pop("limit"), "limit"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "kind"),
    (lambda c: c["norm"].pop("eps"), "eps"),
    (lambda c: c.pop("embedding"), "scale"),
])
def test_bad_configurations_are_named(edit, what):
    c = copy.deepcopy(CFG_S)
    edit(c)
    with pytest.raises(ConfigError) as e:
        bb.RelulixConfig.from_dict(c)
    assert what in str(e.value)


def test_layout_names_and_caches():
    m = bb.Model(bb.RelulixConfig.from_dict(CFG_S), dtype="float32", device="cpu")
    names = m.expected_tensors()
    for n in ("embed", "head", "final.norm", "l0.norm1", "l0.mix.q", "l0.mix.q.b", "l0.mix.k.b", "l0.mix.v.b", "l0.mix.o",
              "l0.mlp.router", "l0.mlp.router.b", "l0.mlp.e2.gate", "l1.mix.q", "l1.mix.g", "l1.mix.o", "l1.mlp.e1.down",
              "l2.mix.q", "l2.mix.q.b", "l2.mix.o", "l3.mix.v.b"):
        assert n in names, n
    for n in ("l0.mix.o.b", "l1.mix.q.b", "l1.mix.norm", "l2.mix.k", "l2.mix.k.b", "l2.mix.v", "l2.mix.v.b", "l2.mlp.router",
              "l0.norm2", "l0.mix.sink"):
        assert n not in names, n
    assert names["l0.norm1"].shape == () and names["final.norm"].shape == () and not names["head"].optional
    assert names["l0.mix.v"].shape == (16, 48) and names["l2.mix.q"].shape == (96, 48) and names["l2.mix.o"].shape == (48, 48)
    assert names["l1.mix.g"].shape == (48, 48) and names["l0.mlp.router.b"].shape == (3,)
    specs = m.cache_specs()
    # layer 2 reads layer 0's keys and values through a wider window, which is what layer 0's cache then keeps
    assert specs == [KVSpec(2, 16, 90, v_dim=8), StateSpec((3 * 16 * 8,), torch.float32), None, KVSpec(3, 16, 5)]
    t = bb.Model(bb.RelulixConfig.from_dict(CFG_T), dtype="float32", device="cpu").cache_specs()
    assert t[1] == KVSpec(3, 12, None, v_dim=20) and t[2] is None and t[3] is None
    u = bb.Model(bb.RelulixConfig.from_dict(CFG_U), dtype="float32", device="cpu").cache_specs()
    assert u[0] == KVSpec(4, 32, 128) and u[1] is None                   # the reader's window is the narrower one


def test_a_random_gain_lies_around_one(tmp_path):
    folder = make_folder(tmp_path, "S")
    _, weights = oracle_inputs(folder)
    gains = [v for k, v in weights.items() if k.endswith("norm1") or k == "final.norm"]
    assert len(gains) == 5 and all(g.shape == () and 0.0 < float(g) < 2.5 and float(g) != 1.0 for g in gains)


@pytest.mark.parametrize("own,readers,want", [
    (KVSpec(2, 16, 64), [], KVSpec(2, 16, 64)),
    (KVSpec(2, 16, 64), [KVSpec(2, 16, 64)], KVSpec(2, 16, 64)),
    (KVSpec(2, 16, 64), [KVSpec(2, 16, 10), KVSpec(2, 16, 200)], KVSpec(2, 16, 200)),
    (KVSpec(2, 16, 64), [KVSpec(2, 16, None)], KVSpec(2, 16, None)),
    (KVSpec(2, 16, None), [KVSpec(2, 16, 10)], KVSpec(2, 16, None)),
    (KVSpec(2, 16, None, chunk=32), [KVSpec(2, 16, 100)], KVSpec(2, 16, 100)),
    (KVSpec(2, 16, 64, keep_first=3), [KVSpec(2, 16, 40, keep_first=5)], KVSpec(2, 16, 64, keep_first=5)),
])
def test_what_a_shared_entry_keeps(own, readers, want):
    assert shared_spec(own, readers) == want


def test_a_reader_of_other_sizes_is_an_error():
    for other in (KVSpec(3, 16, 64), KVSpec(2, 8, 64), KVSpec(2, 16, 64, v_dim=8), StateSpec((4,))):
        with pytest.raises(CacheError):
            shared_spec(KVSpec(2, 16, 64), [other])


def test_the_shared_ring_holds_what_the_wider_window_sees():
    m = bb.Model(bb.RelulixConfig.from_dict(CFG_S), dtype="float32", device="cpu")
    cache = Cache(m.cache_specs(), 640, torch.float32, "cpu")
    assert cache.entries[2] is None and cache.entries[0].group.ring == 128 and cache.entries[3].group.ring == 64
    s = cache.alloc_slot()
    cache.reserve({s: 300})
    rows = cache.write_rows(cache.entries[0].group_id, [s], [0], [300])
    assert (rows >= 0).sum() == 128 and (rows[300 - 90:] >= 0).all()


@pytest.mark.parametrize("build", [
    lambda c: c(hidden=8, n_q=2, n_kv=1, head_dim=8, scale=1.0, bias="q"),
    lambda c: c(hidden=8, n_q=2, n_kv=1, head_dim=8, scale=1.0, sink="one"),
    lambda c: c(hidden=8, n_q=2, n_kv=1, head_dim=8, scale=1.0, borrows_kv=True, lends_kv=True),
    lambda c: c(hidden=8, n_q=2, n_kv=1, head_dim=8, scale=1.0, borrows_kv=True, taps=3),
])
def test_attention_options_that_do_not_go_together(build):
    with pytest.raises(ValueError):
        build(part_class("mixer", "attention"))


def test_other_parts_refuse_what_they_cannot_do():
    decay, experts = part_class("mixer", "decay_attention"), part_class("feedforward", "routed_experts")
    for kw in (dict(norm="head", gate=False), dict(norm=True, gate="silu"), dict(norm="rows"), dict(gate="tanh"),
               dict(position=RotaryEmbedding(16, 100.0, pairing="interleaved"))):
        with pytest.raises(ValueError):
            decay(hidden=8, heads=1, dim=8, v_dim=8, decay=[0.5], eps=1e-5, **kw)
    with pytest.raises(ValueError):
        experts(hidden=8, inter=8, experts=2, top=1, activation="clamped_gate", gated=True, scale_input=False)


@pytest.mark.parametrize("r", [rot(100.0, 8, (2.0, 32, 8.0, 1.0)), rot(30000.0, 12, (6.0, 512, 24.0, 1.5)),
                               rot(10000.0, 2, (4.0, 64, 32.0, 1.0)), rot(500.0, 6)])
def test_rotation_table_against_the_oracle(r):
    part = RotaryEmbedding(head_dim=16, theta=r["base"], rotary_dim=r["dims"], stretch=r.get("scaling"))
    part.prepare(700, torch.device("cpu"))
    half = r["dims"] // 2
    x = torch.zeros(700, 1, 16, dtype=F64)
    x[:, 0, :half] = 1.0                                       # u = 1, v = 0: the rotated pair is (cos, sin)
    y = plain.rotate(x, r)
    assert torch.allclose(part.table[..., 0].double(), y[:, 0, :half], atol=1e-6)
    assert torch.allclose(part.table[..., 1].double(), y[:, 0, half:2 * half], atol=1e-6)


def test_oracle_is_causal_and_its_parts_add_up(tmp_path):
    for name in ("S", "T"):
        config, weights = oracle_inputs(make_folder(tmp_path, name))
        (p,) = random_prompts(config["vocab"], [110], seed=5)
        full = plain.forward(config, weights, p)
        assert torch.allclose(plain.forward(config, weights, p[:67]), full[:67], atol=1e-9)
        assert full.shape == (110, config["vocab"]) and bool(torch.isfinite(full).all())


def test_oracle_window_edge_sink_and_cap_show():
    """A key that carries the weight, at the window's last place and one further back; the sink's share; the cap."""
    g = torch.Generator().manual_seed(2)
    T, H, d, W = 30, 2, 8, 10
    k = torch.randn(T, 1, d, generator=g, dtype=F64)
    v = torch.randn(T, 1, 4, generator=g, dtype=F64)
    q = torch.zeros(T, H, d, dtype=F64)
    q[-1] = 4.0 * k[T - W, 0]                                  # the oldest key the last query sees
    inside = plain.windowed_attention(q, k, v, 1.0, 0.0, W)[-1]
    assert torch.allclose(inside[0], v[T - W, 0], atol=0.05)
    outside = plain.windowed_attention(q, k, v, 1.0, 0.0, W - 1)[-1]
    assert float((outside - inside).abs().max()) > 0.1
    low = torch.zeros(T, H, d, dtype=F64)                      # all scores 0: n keys share n / (n + 1) of the weight
    none = plain.windowed_attention(low, k, v, 1.0, 0.0, W)
    assert torch.allclose(none[0, 0], v[0, 0] / 2.0) and torch.allclose(none[-1, 0], v[T - W:, 0].sum(dim=0) / (W + 1))
    capped = plain.windowed_attention(q, k, v, 1.0, 2.0, W)[-1]
    assert float((capped - inside).abs().max()) > 0.1


def test_oracle_retention_against_its_quadratic_form():
    g = torch.Generator().manual_seed(1)
    T, H, d, dv = 40, 3, 6, 5
    q, k = torch.randn(T, H, d, generator=g, dtype=F64), torch.randn(T, H, d, generator=g, dtype=F64)
    v = torch.randn(T, H, dv, generator=g, dtype=F64)
    decay = torch.tensor([0.5, 0.97, 1.0], dtype=F64)
    o, S = plain.decayed_state(q, k, v, decay)
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    for h in range(H):
        w = (q[:, h] @ k[:, h].T) * torch.where(j <= i, decay[h] ** (i - j).clamp(min=0).double(), torch.zeros(()).double())
        assert torch.allclose(w @ v[:, h], o[:, h], atol=1e-10)
    a, Sa = plain.decayed_state(q[:25], k[:25], v[:25], decay)
    b, Sb = plain.decayed_state(q[25:], k[25:], v[25:], decay, Sa)
    assert torch.allclose(torch.cat([a, b]), o, atol=1e-12) and torch.allclose(Sb, S, atol=1e-12)
    # rotation makes the product of two rows depend on their distance alone
    r = rot(100.0, 4)
    qa, ka = plain.rotate(q[:1], r, first=30), plain.rotate(k[:1], r, first=13)
    qb, kb = plain.rotate(q[:1], r, first=17), plain.rotate(k[:1], r, first=0)
    assert torch.allclose((qa * ka).sum(-1), (qb * kb).sum(-1), atol=1e-10)


def test_oracle_choice_of_experts_and_clamps():
    z = torch.tensor([0.5, 2.0, -1.0, 2.0, 1.0], dtype=F64)
    got = plain.choose(z, 3)
    assert [e for e, _ in got] == [1, 3, 4]                    # ties: the lower index
    assert torch.allclose(torch.stack([w for _, w in got]), torch.softmax(torch.tensor([2.0, 2.0, 1.0], dtype=F64), 0))
    t = {"gate": torch.tensor([[3.0], [-3.0]], dtype=F64), "up": torch.tensor([[5.0], [-5.0]], dtype=F64),
         "down": torch.eye(2, dtype=F64)}
    y = plain.clamped_expert(torch.ones(1, 1, dtype=F64), t, "", 2.0)[0]
    sig = lambda a: 1.0 / (1.0 + torch.exp(torch.tensor(-a, dtype=F64)))
    assert torch.allclose(y[0], 2.0 * sig(1.702 * 2.0) * 3.0) and torch.allclose(y[1], -3.0 * sig(1.702 * -3.0) * -1.0)
