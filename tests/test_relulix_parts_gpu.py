"""The mechanisms Relulix added or combined, each alone against the plain implementation, with inputs made so that a
fault shows: a key that carries the weight just inside and just outside a window (packed and from the pages of a ring,
also a ring wider than the window), the sink of score 0 at the first tokens, queries alone through the row kernel,
rotation and scale ahead of the decayed recurrence, the norm per head with a silu gate, the biased router whose weights
are the softmax over the chosen, the clamped gate of the experts, the norm with one number for a gain."""
import math

import pytest
import torch

from brolm_b200 import kernels
from brolm_b200.parts import RotaryEmbedding, part_class
from tests.plain import relulix_plain as plain
from tests.relulix_helpers import rot

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F64 = torch.float64


def close(got, ref, dtype, what=""):
    tol = 2e-5 if dtype == torch.float32 else 2.5e-2
    scale = max(float(ref.abs().max()), 1e-3)
    err = float((got.double().cpu() - ref.double()).abs().max()) / scale
    assert err <= tol, f"{what}: relative error {err:.3e} exceeds {tol:.0e}"


def table_of(r, n):
    part = RotaryEmbedding(head_dim=r["dims"], theta=r["base"], rotary_dim=r["dims"], stretch=r.get("scaling"))
    part.prepare(n, torch.device(DEV))
    return part.table


# --- windows and the sink ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,hd,vd,window,cap", [(4, 2, 16, 16, 1, 0.0), (3, 3, 12, 20, 37, 20.0), (4, 1, 32, 32, 64, 30.0),
                                                  (2, 2, 64, 64, 65, 50.0), (4, 2, 32, 48, 127, 8.0), (2, 1, 16, 16, 200, 0.0)])
def test_a_key_at_the_windows_edge_of_a_prompt(dtype, H, G, hd, vd, window, cap):
    """The last queries each look for one key: the window's last place and the place beyond it, around page borders."""
    g = torch.Generator().manual_seed(window + hd)
    T = window + 150
    k = torch.randn(T, G, hd, generator=g)
    k = k / k.norm(dim=-1, keepdim=True)
    v = torch.randn(T, G, vd, generator=g)
    q = 0.1 * torch.randn(T, H, hd, generator=g)
    back = [window - 1, window, max(0, window - 2), window + 1, 0, 64]
    places = [T - 1 - 9 * i for i in range(6)] + [window - 1 + (window == 1), min(window, T - 1)]
    for i, p in enumerate(places):
        n = min(back[i % 6], p)
        for h in range(H):
            q[p, h] = 9.0 * k[p - n, h // (H // G)]
    q, k, v = q.to(dtype), k.to(dtype), v.to(dtype)
    ref = plain.windowed_attention(q.double(), k.double(), v.double(), 1.0, cap, window)
    for other in (window + 1, max(1, window - 1)):             # a window that is one token off is seen
        off = plain.windowed_attention(q.double(), k.double(), v.double(), 1.0, cap, other)
        assert other == window or float((off - ref).abs().max()) > 0.1
    cu = torch.tensor([0, T], dtype=torch.int32, device=DEV)
    kvl = torch.tensor([T], dtype=torch.int32, device=DEV)
    sink = torch.zeros(H, dtype=torch.float32, device=DEV)
    common = dict(n_kv=G, group=H // G, head_dim=hd, scale=1.0, cap=cap, window=window, batch=1, max_q_len=T, sink=sink)
    qd, kd, vd_ = (x.reshape(T, -1).to(DEV) for x in (q, k, v))
    out = torch.empty(T, H * vd, dtype=dtype, device=DEV)
    kernels.attention_simt(qd, out, cu, kvl, k=kd, v=vd_, v_dim=vd, **common)
    close(out.view(T, H, vd), ref, dtype, "exact kernel")
    if dtype == torch.bfloat16 and kernels.attention_headmix_ok(hd, vd, H // G, False):
        out.zero_()
        kernels.attention_headmix_prefill(qd, out, cu, kd, vd_, v_dim=vd, **common)
        close(out.view(T, H, vd), ref, dtype, "tensor cores, rows of two sizes")
        if hd == vd:
            out.zero_()
            kernels.attention_prefill_mma(qd, out, cu, kd, vd_, **common)
            close(out.view(T, H, vd), ref, dtype, "tensor cores, rows of one size")


@pytest.mark.parametrize("dtype,vd", [(torch.float32, 48), (torch.float32, 16), (torch.bfloat16, 48), (torch.bfloat16, 16)])
@pytest.mark.parametrize("window,ring", [(64, 64), (37, 64), (65, 128), (136, 192), (37, 192), (100, 1 << 30)])
def test_a_key_at_the_windows_edge_of_a_ring(dtype, vd, window, ring):
    """Decoding: one query per sequence over scattered pages (NaN in places never written); the ring may be wider than
    the window, as it is for a layer that reads the cache of one with a wider window."""
    g = torch.Generator().manual_seed(window)
    H, G, hd, page = 4, 2, 16, 64
    lengths = [1, window, window + 1, 64, 65, 130, 300, 301, 41]
    backs = [0, window - 1, window - 1, 63, window, window - 1, window - 1, window, 3]
    places = [p if ring == 1 << 30 else p % ring for p in range(max(lengths))]
    B = len(lengths)
    ks, vs, qs = [], [], []
    for n, back in zip(lengths, backs):
        k = torch.randn(n, G, hd, generator=g)
        k = k / k.norm(dim=-1, keepdim=True)
        ks.append(k.to(dtype))
        vs.append(torch.randn(n, G, vd, generator=g).to(dtype))
        tgt = max(0, n - 1 - back)
        qs.append(torch.stack([9.0 * k[tgt, h // (H // G)] for h in range(H)]).to(dtype))
    pages_per = [(min(n, ring) + page - 1) // page for n in lengths]
    n_pages = sum(pages_per) + 3
    order = iter(torch.randperm(n_pages, generator=g).tolist())
    pt = torch.zeros(B, max(pages_per), dtype=torch.int32)
    kp = torch.full((n_pages, G, page, hd), float("nan")).to(dtype)
    vp = torch.full((n_pages, G, page, vd), float("nan")).to(dtype)
    for b, n in enumerate(lengths):
        for j in range(pages_per[b]):
            pt[b, j] = next(order)
        for p in range(n):
            at = places[p]
            kp[int(pt[b, at // page]), :, at % page] = ks[b][p]
            vp[int(pt[b, at // page]), :, at % page] = vs[b][p]
    refs = [plain.windowed_attention(qs[b].double()[None], ks[b].double(), vs[b].double(), 1.0, 15.0, window, first=n - 1)[0]
            for b, n in enumerate(lengths)]
    cu, kvl = torch.arange(B + 1, dtype=torch.int32, device=DEV), torch.tensor(lengths, dtype=torch.int32, device=DEV)
    q = torch.stack(qs).reshape(B, -1).to(DEV)
    common = dict(ring=ring, page_size=page, n_kv=G, group=H // G, head_dim=hd, scale=1.0, cap=15.0, window=window, batch=B,
                  sink=torch.zeros(H, dtype=torch.float32, device=DEV))
    out = torch.empty(B, H * vd, dtype=dtype, device=DEV)

    def compare(what):
        assert bool(torch.isfinite(out.float()).all()), f"{what}: a place of the cache that was never written was read"
        for b, n in enumerate(lengths):
            close(out[b].view(H, vd), refs[b], dtype, f"{what}, sequence of {n}")
        out.zero_()
    kernels.attention_simt(q, out, cu, kvl, k_pages=kp.to(DEV), v_pages=vp.to(DEV), page_table=pt.to(DEV), v_dim=vd, max_q_len=1,
                           **common)
    compare("exact kernel")
    if dtype == torch.bfloat16:
        for splits in (1, 2, 3):
            kernels.attention_headmix_decode(q, out, cu, kvl, kp.to(DEV), vp.to(DEV), pt.to(DEV), ring_from=0, v_dim=vd,
                                             n_splits=splits, **common)
            compare(f"rows of two sizes, {splits} splits")
            if hd == vd:
                kernels.attention_decode_mma(q, out, cu, kvl, kp.to(DEV), vp.to(DEV), pt.to(DEV), n_splits=splits, **common)
                compare(f"rows of one size, {splits} splits")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_sink_at_the_first_tokens(dtype):
    """All scores 0: the n visible keys share n / (n + 1) of the weight.  Scores far below 0: next to nothing is left."""
    T, H, hd, W = 9, 2, 16, 4
    g = torch.Generator().manual_seed(1)
    v = torch.randn(T, H, hd, generator=g).to(dtype)
    k = torch.ones(T, H, hd, dtype=dtype)
    q = torch.zeros(T, H, hd, dtype=dtype)
    q[:, 1] = -2.0                                              # head 1: every score is -32
    cu, kvl = torch.tensor([0, T], dtype=torch.int32, device=DEV), torch.tensor([T], dtype=torch.int32, device=DEV)
    out = torch.empty(T, H * hd, dtype=dtype, device=DEV)
    args = dict(n_kv=H, group=1, head_dim=hd, scale=1.0, cap=0.0, window=W, batch=1, max_q_len=T,
                sink=torch.zeros(H, dtype=torch.float32, device=DEV))
    runs = [lambda: kernels.attention_simt(q.reshape(T, -1).to(DEV), out, cu, kvl, k=k.reshape(T, -1).to(DEV),
                                           v=v.reshape(T, -1).to(DEV), **args)]
    if dtype == torch.bfloat16:
        runs.append(lambda: kernels.attention_prefill_mma(q.reshape(T, -1).to(DEV), out, cu, k.reshape(T, -1).to(DEV),
                                                          v.reshape(T, -1).to(DEV), **args))
    for run in runs:
        run()
        got = out.view(T, H, hd).double().cpu()
        for t in range(T):
            n = min(t + 1, W)
            close(got[t, 0], v[t + 1 - n:t + 1, 0].double().sum(dim=0) / (n + 1), dtype, f"token {t}")
        assert float(got[:, 1].abs().max()) < 1e-10


# --- queries alone --------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("n_q,hd,r", [(4, 16, rot(100.0, 8, (2.0, 32, 8.0, 1.0))), (3, 12, rot(500.0, 6)), (2, 64, rot(1000.0, 64))])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_queries_alone_through_the_row_kernel(n_q, hd, r, dtype):
    g = torch.Generator().manual_seed(hd)
    T = 21
    proj, bias = torch.randn(T, n_q * hd, generator=g) * 2, torch.randn(n_q * hd, generator=g)
    pos = torch.arange(T, dtype=torch.int32, device=DEV)
    pos[7] = -1                                                 # a padding row is left untouched
    out = torch.full((T, n_q * hd), 7.0, dtype=dtype, device=DEV)
    kernels.qkv_finish(proj.to(DEV), bias.to(DEV), n_q, 0, hd, 8, pos, out, cos_sin=table_of(r, T), rotary_dim=r["dims"])
    ref = plain.rotate((proj + bias).double().view(T, n_q, hd), r)
    ref[7] = 7.0
    close(out.view(T, n_q, hd), ref, dtype)


# --- retention -------------------------------------------------------------------------------------------------------
def scan(q, k, v, decay, cuts, state, slot, r=None, k_scale=1.0, pad=0):
    """One sequence through rotate_heads / decay_scan in pieces of the given lengths, as the mixer does it: pieces of
    several tokens are rotated ahead of the scan, single tokens inside it.  q, k, v (T, H, .)."""
    T, H, d = q.shape
    dv = v.shape[-1]
    row = torch.cat([q.reshape(T, -1), k.reshape(T, -1), v.reshape(T, -1), torch.zeros(T, pad)], dim=1).to(DEV)
    dm1 = torch.tensor([x - 1.0 for x in decay], dtype=F64).float().to(DEV)
    table = table_of(r, T) if r else None
    outs, at = [], 0
    for n in cuts:
        out = torch.empty(n, H * dv, dtype=torch.float32, device=DEV)
        piece, opts = row[at:at + n].clone(), dict(cos_sin=table, k_scale=k_scale)
        if n > 1:
            kernels.rotate_heads(piece, 0, H * d, H, d, torch.arange(at, at + n, dtype=torch.int32, device=DEV), table, k_scale)
            opts = {}
        kernels.decay_scan(piece, 0, H * d, 2 * H * d, H, d, dv, "none", dm1, torch.tensor([0, n], dtype=torch.int32, device=DEV),
                           torch.tensor([at + n], dtype=torch.int32, device=DEV), torch.tensor([slot], dtype=torch.int32, device=DEV),
                           state, out, 1, n, **opts)
        outs.append(out)
        at += n
    return torch.cat(outs).view(T, H, dv)


@pytest.mark.parametrize("H,d,dv,r,pad", [(3, 8, 16, rot(50.0, 4), 0), (1, 6, 13, rot(10000.0, 6), 1), (2, 32, 64, rot(10000.0, 32), 0),
                                          (2, 128, 128, rot(10000.0, 128), 0), (5, 20, 7, rot(300.0, 10, (4.0, 32, 8.0, 1.0)), 3),
                                          (1, 256, 40, rot(1000.0, 64), 0), (2, 64, 48, None, 0), (3, 32, 32, rot(10.0, 2), 0)])
def test_retention_in_pieces(H, d, dv, r, pad):
    g = torch.Generator().manual_seed(d + dv)
    T = 140
    q, k = torch.randn(T, H, d, generator=g), torch.randn(T, H, d, generator=g)
    v = torch.randn(T, H, dv, generator=g)
    decay = [0.5, 0.999, 1.0, 0.9, 0.97][:H]
    turn = (lambda x: plain.rotate(x.double(), r)) if r else (lambda x: x.double())
    ref, S = plain.decayed_state(turn(q), turn(k) / math.sqrt(d), v.double(), torch.tensor(decay, dtype=F64))
    size = kernels.decay_state_size(H, d, dv)
    for cuts in ([T], [1] * T, [64, 1, 1, 20, 2, 52], [139, 1], [2] * 70):
        state = torch.zeros(3, size + 8, dtype=torch.float32, device=DEV)
        state[0] = float("nan")                                # another sequence's row is never touched
        got = scan(q, k, v, decay, cuts, state, 1, r, d ** -0.5, pad)
        close(got, ref, torch.float32, f"cuts {cuts[:4]}")
        close(state[1, :size].view(H, dv, -1)[:, :, :d].transpose(1, 2), S, torch.float32, "the state after the last token")
        assert bool(torch.isnan(state[0]).all()) and float(state[2].abs().max()) == 0.0


def test_retention_step_of_unequal_sequences_and_a_padding_row():
    g = torch.Generator().manual_seed(10)
    H, d, dv, r = 2, 16, 20, rot(100.0, 12)
    lens = [5, 1, 33]
    size = kernels.decay_state_size(H, d, dv)
    state = torch.zeros(5, size, dtype=torch.float32, device=DEV)
    state[4] = 7.0                                              # the padding rows' spare row
    slots, decay = [2, 0, 3], [0.95, 0.8]
    q, k = [torch.randn(n + 1, H, d, generator=g) for n in lens], [torch.randn(n + 1, H, d, generator=g) for n in lens]
    v = [torch.randn(n + 1, H, dv, generator=g) for n in lens]
    for b, n in enumerate(lens):
        scan(q[b][:n], k[b][:n], v[b][:n], decay, [n], state, slots[b], r, d ** -0.5)
    last = torch.cat([torch.cat([x[b][-1].reshape(1, -1) for x in (q, k, v)], dim=1) for b in range(3)] +
                     [torch.full((1, 2 * H * d + H * dv), float("nan"))]).to(DEV)
    out = torch.full((4, H * dv), 3.0, dtype=torch.float32, device=DEV)
    kernels.decay_scan(last, 0, H * d, 2 * H * d, H, d, dv, "none", torch.tensor([-0.05, -0.2], device=DEV),
                       torch.arange(5, dtype=torch.int32, device=DEV),
                       torch.tensor([n + 1 for n in lens] + [0], dtype=torch.int32, device=DEV),
                       torch.tensor(slots + [4], dtype=torch.int32, device=DEV), state, out, 4, 1, cos_sin=table_of(r, 64),
                       k_scale=d ** -0.5)
    for b in range(3):
        ref, _ = plain.decayed_state(plain.rotate(q[b].double(), r), plain.rotate(k[b].double(), r) / math.sqrt(d), v[b].double(),
                                     torch.tensor(decay, dtype=F64))
        close(out[b].view(H, dv), ref[-1], torch.float32, f"sequence of {lens[b]}")
    assert float((out[3] - 3.0).abs().max()) == 0.0 and float((state[4] - 7.0).abs().max()) == 0.0
    assert float(state[1].abs().max()) == 0.0


def test_rotate_heads_leaves_everything_else_alone():
    g = torch.Generator().manual_seed(4)
    T, H, d, r = 9, 3, 8, rot(100.0, 4)
    rows = torch.randn(T, 3 + 2 * H * d + 5, generator=g)
    pos = torch.tensor([0, 5, 6, -1, 3, 700, 2, 1, 90], dtype=torch.int32)
    got = rows.clone().to(DEV)
    kernels.rotate_heads(got, 3, 3 + H * d, H, d, pos.to(DEV), table_of(r, 701), 0.3)
    ref = rows.double()
    for t in range(T):
        if int(pos[t]) >= 0:
            qk = rows[t, 3:3 + 2 * H * d].double().view(1, 2 * H, d)
            turned = plain.rotate(qk, r, first=int(pos[t]))
            turned[:, H:] *= 0.3
            ref[t, 3:3 + 2 * H * d] = turned.reshape(-1)
    close(got, ref, torch.float32)
    assert torch.equal(got[:, :3].cpu(), rows[:, :3]) and torch.equal(got[:, 3 + 2 * H * d:].cpu(), rows[:, 3 + 2 * H * d:])


@pytest.mark.parametrize("heads,hd", [(3, 16), (2, 7), (16, 128), (1, 512), (2, 600), (5, 4)])
@pytest.mark.parametrize("gate", ["silu", "sigmoid"])
def test_norm_per_head_with_a_gate(heads, hd, gate):
    g = torch.Generator().manual_seed(heads * hd)
    T, cols = 19, heads * hd
    y = torch.randn(T, cols, generator=g) * 3
    y[:, :hd] *= 1e-3                                          # a head whose mean square is near eps
    wide = torch.randn(T, cols + 24, generator=g) * 2
    gain = torch.randn(cols, generator=g)
    z = wide[:, 24:].double()
    act = plain.silu(z) if gate == "silu" else torch.sigmoid(z)
    for w in (None, gain):
        ref = plain.unit_rms(y.double().view(T, heads, hd), 1e-5).reshape(T, cols) * act * (w.double() if w is not None else 1.0)
        for od in (torch.float32, torch.bfloat16):
            out = torch.empty(T, cols, dtype=od, device=DEV)
            kernels.head_norm_gate(y.to(DEV), wide.to(DEV)[:, 24:], w.to(DEV) if w is not None else None, 1e-5, heads, gate, out)
            close(out, ref, od)


# --- experts ---------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("E,top,tokens,spread", [(8, 4, 50, 1.0), (6, 1, 9, 1.0), (4, 4, 300, 1.0), (64, 6, 300, 1.0),
                                                 (40, 5, 33, 60.0), (1, 1, 5, 1.0), (33, 33, 70, 20.0)])
def test_router_with_a_bias_and_the_softmax_over_the_chosen(E, top, tokens, spread):
    """With a wide spread a softmax over all experts would lose the order of the small ones; here the scores decide."""
    g = torch.Generator().manual_seed(E * 7 + top)
    W = 48
    x = torch.randn(tokens, W, generator=g)
    router = torch.randn(E, W, generator=g) * 0.3 * spread
    bias = torch.randn(E, generator=g) * 2.0
    ids = torch.empty(tokens, top, dtype=torch.int32, device=DEV)
    wts = torch.empty(tokens, top, dtype=torch.float32, device=DEV)
    raw = x.double() @ router.double().T
    for use_product in (False, True):
        if use_product:
            kernels.route_pick(raw.float().to(DEV), top, ids, wts, "softmax_chosen", bias=bias.to(DEV))
        else:
            kernels.route_topk(x.to(DEV), router.to(DEV), top, ids, wts, "softmax_chosen", bias=bias.to(DEV))
        changed = 0
        for t in range(tokens):
            z = raw[t] + bias.double()
            want = plain.choose(z, top)
            got = ids[t].tolist()
            assert got == [e for e, _ in want] or \
                float((z[got] - torch.stack([z[e] for e, _ in want])).abs().max()) < 1e-4 * spread, (t, got, want)
            if got == [e for e, _ in want]:
                assert torch.allclose(wts[t].double().cpu(), torch.stack([w for _, w in want]), atol=2e-4 if spread > 1 else 1e-5)
            changed += [e for e, _ in plain.choose(raw[t], top)] != [e for e, _ in want]
        assert E == 1 or changed > 0                            # the bias matters in this test
        assert torch.allclose(wts.sum(dim=1).cpu(), torch.ones(tokens), atol=1e-5)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("W,ff,E,top,limit,tokens", [(48, 24, 3, 3, 0.5, 7), (64, 40, 6, 2, 2.0, 300), (40, 12, 5, 5, 1.0, 70),
                                                     (128, 64, 4, 4, 0.3, 600)])
def test_experts_with_a_clamped_gate(dtype, W, ff, E, top, limit, tokens):
    g = torch.Generator().manual_seed(ff)
    part = part_class("feedforward", "routed_experts")(hidden=W, inter=ff, experts=E, top=top, activation="clamped_gate", limit=limit,
                                                       scale_input=False, gated=True, router="softmax_chosen", router_bias=True)
    t = {}
    for name, spec in part.param_specs().items():
        t[name] = (torch.randn(spec.shape, generator=g) * (0.3 if spec.role == "matrix" else 1.0)).to(dtype)
    part.bind({n: x.to(DEV) for n, x in t.items()})
    x = torch.randn(tokens, W, generator=g).to(dtype)
    flat = {n.replace("router_bias", "router.b"): v.double() for n, v in t.items()}
    pre = x.double() @ flat["e0.up"].T
    assert float((pre.abs() > limit).double().mean()) > 0.1 and float((x.double() @ flat["e0.gate"].T > limit).double().mean()) > 0.05
    mlp = dict(expert=dict(limit=limit), router=dict(top=top))
    ref = plain.routed(x.double(), flat, "", mlp)
    got = part.forward(x.to(DEV), None)
    if top == E or dtype == torch.float32:
        close(got, ref, dtype)
    else:                                                       # a close call may fall the other way in bfloat16
        err = (got.double().cpu() - ref).abs().amax(dim=1) / ref.abs().max()
        assert float(err.sort().values[int(0.95 * tokens)]) <= 2.5e-2


def test_norm_with_one_number():
    part = part_class("norm", "rmsnorm")(size=72, eps=1e-3, scalar=True)
    assert part.param_specs()["weight"].shape == ()
    g = torch.Generator().manual_seed(0)
    x = torch.randn(11, 72, generator=g) * 0.1
    for dtype in (torch.float32, torch.bfloat16):
        gain = torch.tensor(1.75, dtype=dtype)
        part.bind({"weight": gain.to(DEV)})
        ref = plain.scalar_norm(x.double(), 1.75, 1e-3)
        close(part.apply(x.to(DEV), torch.float32), ref, torch.float32)
        rows = torch.tensor([3, 0], dtype=torch.int32, device=DEV)
        close(part.apply(x.to(DEV), torch.float32, rows), ref[[3, 0]], torch.float32)
