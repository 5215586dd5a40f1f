"""The mechanisms Papusun added or combined, each alone against the plain implementation, with inputs made so that a fault
shows: layer norm alone and behind a residual sum, the delta rule in one piece, token by token and in uneven pieces, the
rows of latent attention in their three parts, a gate per head on a product per head, a table's part behind an activation,
scaled logits, a key that stands out at a window's edge of a latent row and far back under a cap."""
import math

import pytest
import torch

from brolm_b200 import kernels
from brolm_b200.parts import LayerNorm, RMSNorm, RotaryEmbedding, add_then_norm
from tests.papusun_helpers import rot
from tests.plain import papusun_plain as plain

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F64 = torch.float64


def close(got, ref, dtype=torch.float32, what="", tol=None):
    tol = tol or (2e-5 if dtype == torch.float32 else 2.5e-2)
    assert bool(torch.isfinite(got.float()).all()), f"{what}: not finite"
    err = float((got.double().cpu() - ref.double()).abs().max()) / max(float(ref.abs().max()), 1e-3)
    assert err <= tol, f"{what}: relative error {err:.3e} exceeds {tol:.0e}"


def i32(*x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


# --- layer norm ----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("W", [7, 40, 256, 1024, 1028, 2048, 3072, 4096, 8192, 8200])
@pytest.mark.parametrize("wd", [torch.float32, torch.bfloat16])
def test_layer_norm_alone_and_behind_the_sum(W, wd):
    g = torch.Generator().manual_seed(W)
    T, parts = 5, 3
    h = torch.randn(T, W, generator=g) + 3.0                   # a mean well off zero
    h[1] = 1e-2 * torch.randn(W, generator=g) + 100.0          # a spread not far above the eps, a mean far from zero
    h[2] = 0.25                                                # no spread at all
    y = torch.randn(parts, T, W, generator=g)
    y[:, 1:3] *= 1e-4
    w, wp = torch.randn(W, generator=g).to(wd), torch.randn(W, generator=g).to(wd)
    eps = 1e-5
    norm, post = LayerNorm(W, eps), RMSNorm(W, 1e-3, offset=0.5)
    norm.bind({"weight": w.to(DEV)})
    post.bind({"weight": wp.to(DEV)})
    ref = lambda x: plain.layer_norm(x.double(), w.double(), eps)
    out = norm.apply(h.to(DEV), torch.float32)
    close(out[[0, 3, 4]], ref(h)[[0, 3, 4]], what="alone")
    close(out[1], ref(h)[1], what="far from zero", tol=2e-3)   # (a float has three digits left for such a row's spread)
    assert float(out[2].abs().max()) <= 1e-2
    close(norm.apply(h.to(DEV), torch.bfloat16, rows=i32(4, 0)), ref(h)[[4, 0]], torch.bfloat16, "picked rows")
    total = y.double().sum(dim=0)
    for with_post in (False, True):
        for p in (1, parts):
            s = y[0].double() if p == 1 else total
            if with_post:
                s = s / torch.sqrt((s * s).mean(-1, keepdim=True) + 1e-3) * (0.5 + wp.double())
            hd = h.to(DEV)
            yd = (y[0] if p == 1 else y).to(DEV).contiguous()
            out = add_then_norm(hd, yd, post if with_post else None, norm, torch.float32)
            close(hd, h.double() + s, what="the stream")
            close(out[[0, 3, 4]], ref(h.double() + s)[[0, 3, 4]], what=f"{p} parts, post {with_post}")


# --- the gated delta rule ------------------------------------------------------------------------------------------
def delta_inputs(G, d, H, dv, K, T, seed):
    g = torch.Generator().manual_seed(seed)
    C = 2 * G * d + H * dv
    cols = (C + 2 * H + 3) // 4 * 4
    proj = torch.randn(T, cols, generator=g)
    taps = 0.5 * torch.randn(K, C, generator=g)
    taps[-1] += 1.0
    a_log = torch.linspace(-6.0, 0.5, H) if H > 1 else torch.tensor([-3.0])
    return proj, taps, a_log, 0.5 * torch.randn(H, generator=g)


def delta_reference(proj, taps, a_log, dt_bias, G, d, H, dv):
    x, T = proj.double(), proj.shape[0]
    C = 2 * G * d + H * dv
    u = plain.silu(plain.short_conv(x[:, :C], taps.double().T))
    q = plain.unit_length(u[:, :G * d].view(T, G, d)) * d ** -0.5
    k = plain.unit_length(u[:, G * d:2 * G * d].view(T, G, d))
    own = [h // (H // G) for h in range(H)]
    beta = torch.sigmoid(x[:, C:C + H])
    dt = torch.nn.functional.softplus(x[:, C + H:C + 2 * H] + dt_bias.double(), threshold=100.0)
    decay = torch.exp(-torch.exp(a_log.double()) * dt)
    return plain.delta_states(q[:, own], k[:, own], u[:, 2 * G * d:].view(T, H, dv), decay, beta)[0].reshape(T, H * dv)


SIZES = [(1, 6, 1, 7, 1), (2, 16, 4, 8, 3), (1, 20, 3, 5, 6), (2, 64, 2, 40, 4), (1, 128, 2, 128, 4), (2, 128, 6, 48, 2),
         (1, 136, 2, 16, 4), (1, 256, 1, 33, 4), (1, 260, 2, 20, 3), (1, 512, 1, 24, 4)]


class DeltaCase:
    """A sequence's slot among others whose rows are full of NaN."""

    def __init__(self, G, d, H, dv, K, T, seed):
        self.sizes, self.K = (G, d, H, dv), K
        self.proj, self.taps, self.a_log, self.dt_bias = delta_inputs(G, d, H, dv, K, T, seed)
        self.ref = delta_reference(self.proj, self.taps, self.a_log, self.dt_bias, G, d, H, dv)
        self.tail = kernels.decay_state_size(H, d, dv)
        n = self.tail + (K if K > 1 else 0) * (2 * G * d + H * dv)
        self.state = torch.full((4, (n + 3) // 4 * 4), float("nan"), device=DEV)
        self.consts = tuple(t.to(DEV) for t in (self.a_log, self.dt_bias))
        self.taps_dev = self.taps.to(DEV)

    def run(self, pieces, slot=2):
        """The sequence in pieces; a piece of one token goes through the single-token kernel."""
        G, d, H, dv = self.sizes
        self.state[slot].zero_()
        outs, at = [], 0
        for n in pieces:
            x = self.proj[at:at + n].to(DEV)
            out = torch.full((n, H * dv), float("nan"), device=DEV)
            seq = (i32(0, n), i32(at + n), i32(slot), self.state, self.tail)
            if n == 1:
                kernels.delta_step(x, self.taps_dev, G, d, H, dv, *self.consts, *seq, out, 1)
            else:
                kernels.delta_prompt(x, self.taps_dev, G, d, H, dv, *self.consts, torch.zeros(n, dtype=torch.int32, device=DEV),
                                     torch.arange(at, at + n, dtype=torch.int32, device=DEV), *seq, out, 1, n)
            outs.append(out)
            at += n
        return torch.cat(outs)


@pytest.mark.parametrize("G,d,H,dv,K", SIZES)
def test_delta_rule_in_one_piece_and_in_many(G, d, H, dv, K):
    T = 75
    case = DeltaCase(G, d, H, dv, K, T, seed=d + dv)
    for pieces in ([T], [1] * T, [16, 16, 43], [2] * 37 + [1], [3, 1, 17, 2, 33, 1, 1, 15, 2], [48, 1, 1, 1, 16, 8]):
        close(case.run(pieces), case.ref, what=f"pieces {pieces[:9]}", tol=5e-6 * math.sqrt(d))
    assert bool(torch.isnan(case.state[[0, 1, 3]]).all()), "a neighbour's row was written"


def test_delta_rule_remembers_for_thousands_of_tokens():
    """A decay so close to one that a float holds few digits of its distance to it: the first token's value is read back
    after three thousand tokens whose keys are other directions."""
    G = H = 1
    d, dv, K, T = 32, 16, 1, 3000
    case = DeltaCase(G, d, H, dv, K, T, seed=9)
    g = torch.Generator().manual_seed(10)
    proj = case.proj
    case.taps.fill_(1.0)
    case.taps_dev = case.taps.to(DEV)
    axes = torch.full((T, d), -30.0)                           # silu(-30) is next to nothing: unit vectors along one axis
    pick = 1 + torch.randint(0, d - 1, (T,), generator=g)
    pick[0] = 0
    axes[torch.arange(T), pick] = 5.0
    proj[:, d:2 * d] = axes                                    # keys: the first token alone has axis 0
    proj[:, :d] = -30.0
    proj[:, 0] = 5.0                                           # queries: axis 0 throughout
    proj[:, 2 * d + dv] = 4.0
    case.a_log.fill_(-7.0)
    case.consts = tuple(t.to(DEV) for t in (case.a_log, case.dt_bias))
    case.ref = delta_reference(proj, case.taps, case.a_log, case.dt_bias, G, d, H, dv)
    assert 1e-3 < float(case.ref[-1].abs().max()) < 0.5 * float(case.ref[0].abs().max())
    for pieces in ([T], [2000] + [1] * 200 + [800]):
        got = case.run(pieces).double().cpu()
        rows = (got - case.ref).abs().amax(dim=1) / case.ref.abs().amax(dim=1)
        assert float(rows.max()) <= 2e-5, f"{float(rows.max()):.2e}"


@pytest.mark.parametrize("G,d,H,dv,K", [(2, 16, 4, 8, 3), (1, 128, 2, 64, 4), (1, 20, 2, 6, 5)])
def test_delta_rule_of_a_batch_with_padding(G, d, H, dv, K):
    """Unequal sequences packed into one step on shuffled slots, then single tokens in a step with padding rows."""
    lens, slots = [33, 1, 16, 70, 2], [3, 0, 5, 1, 4]
    cases = [DeltaCase(G, d, H, dv, K, n + 3, seed=20 + n) for n in lens]
    base = cases[0]
    state = torch.full((7, base.state.shape[1]), float("nan"), device=DEV)
    state[slots] = 0.0
    x = torch.cat([c.proj[:n] for c, n in zip(cases, lens)]).to(DEV)
    T = sum(lens)
    out = torch.full((T, H * dv), float("nan"), device=DEV)
    cu = [0]
    for n in lens:
        cu.append(cu[-1] + n)
    seq = torch.cat([torch.full((n,), b, dtype=torch.int32) for b, n in enumerate(lens)]).to(DEV)
    pos = torch.cat([torch.arange(n, dtype=torch.int32) for n in lens]).to(DEV)
    # every sequence's own constants would differ: they share the first one's
    refs = [delta_reference(c.proj, base.taps, base.a_log, base.dt_bias, G, d, H, dv) for c in cases]
    kernels.delta_prompt(x, base.taps_dev, G, d, H, dv, *base.consts, seq, pos, i32(*cu), i32(*lens), i32(*slots), state, base.tail,
                         out, len(lens), max(lens))
    for b, n in enumerate(lens):
        close(out[cu[b]:cu[b + 1]], refs[b][:n], what=f"sequence of {n} in a batch", tol=5e-5)
    for j in range(3):
        rows = torch.cat([c.proj[n + j:n + j + 1] for c, n in zip(cases, lens)] + [torch.full((2, x.shape[1]), float("nan"))]).to(DEV)
        one = torch.full((7, H * dv), float("nan"), device=DEV)
        before = state[[2, 6]].clone()
        kernels.delta_step(rows, base.taps_dev, G, d, H, dv, *base.consts, torch.arange(8, dtype=torch.int32, device=DEV),
                           i32(*[n + j + 1 for n in lens], 0, 0), i32(*slots, 6, 6), state, base.tail, one, 7)
        for b, n in enumerate(lens):
            close(one[b], refs[b][n + j], what=f"token {j} after {n}", tol=5e-5)
        assert torch.equal(before.isnan(), state[[2, 6]].isnan()) and bool(one[5:].isnan().all())


# --- latent attention ----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,dn,dr,R,Q", [(3, 5, 6, 15, 11), (4, 16, 8, 24, 40), (1, 4, 2, 8, 3)])
def test_latent_rows_in_their_three_parts(dtype, H, dn, dr, R, Q):
    g = torch.Generator().manual_seed(R)
    T, D, page = 9, (R + dr + 15) // 16 * 16, 64
    r = rot(50.0, dr)
    part = RotaryEmbedding(dr, r["base"], dr, pairing="interleaved")
    part.prepare(200, torch.device(DEV))
    proj = torch.randn(T, Q + R + dr + 3, generator=g).to(dtype)
    queries = torch.randn(T, H * (dn + dr), generator=g).to(dtype)
    gain, gq = torch.randn(R, generator=g).to(dtype), torch.randn(Q, generator=g).to(dtype)
    first = 60
    positions = torch.arange(first, first + T, dtype=torch.int32, device=DEV)
    pages = torch.full((2, 1, page, D), float("nan"), dtype=dtype, device=DEV)
    cache_rows = torch.arange(page + 3, page + 3 + T, dtype=torch.int32, device=DEV)
    cache_rows[2] = -1
    lat, cq = (torch.full((T, n), float("nan"), dtype=dtype, device=DEV) for n in (D, Q))
    qlat = torch.full((T, H * D), float("nan"), dtype=dtype, device=DEV)
    args = (proj.to(DEV), Q, positions, part.table, dr, gain.to(DEV), 1e-5, H, dn, dr, R)
    kernels.latent_rows(*args, lat, None, pages=pages, cache_rows=cache_rows, pairing="interleaved", cq=cq, cq_gain=gq.to(DEV))
    x = proj.double()
    c = plain.unit_rms(x[:, Q:Q + R], 1e-5) * gain.double()
    kr = plain.rotate(x[:, None, Q + R:Q + R + dr], r, first)[:, 0]
    close(lat[:, :R + dr], torch.cat([c, kr], dim=1), dtype, "the latent row")
    assert not bool(lat[:, R + dr:].any())
    close(cq, plain.unit_rms(x[:, :Q], 1e-5) * gq.double(), dtype, "the queries' latent")
    kept = pages[1, 0, 3:3 + T]
    assert torch.equal(kept[[0, 1, 3, 8]], lat[[0, 1, 3, 8]]) and bool(kept[2].isnan().all()) and bool(pages[0].isnan().all())
    kernels.latent_rows(*args, None, qlat, pairing="interleaved", queries=queries.to(DEV), width=D)
    qr = plain.rotate(queries.double().view(T, H, dn + dr)[..., dn:], r, first)
    got = qlat.view(T, H, D)
    close(got[..., R:R + dr], qr, dtype, "the rotated query parts")
    assert bool(got[..., :R].isnan().all()) and not bool(got[..., R + dr:].any())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,H,N,K", [(1, 3, 7, 16), (8, 4, 40, 24), (70, 5, 16, 32), (33, 2, 9, 13)])
def test_a_gate_per_head_on_a_product_per_head(dtype, T, H, N, K):
    g = torch.Generator().manual_seed(T)
    a, w = torch.randn(T, H * K, generator=g).to(dtype), torch.randn(H, N, K, generator=g).to(dtype)
    for gate_dtype in (dtype, torch.float32):
        wide = (3.0 * torch.randn(T, H + 5, generator=g)).to(gate_dtype)
        out = torch.empty(T, H * N, dtype=dtype, device=DEV)
        kernels.heads_linear(a.to(DEV), K, w.to(DEV), out, N, gate=wide.to(DEV)[:, 2:2 + H])
        ref = torch.einsum("thk,hnk->thn", a.double().view(T, H, K), w.double()) * torch.sigmoid(wide[:, 2:2 + H].double())[..., None]
        close(out, ref.reshape(T, H * N), dtype)


@pytest.mark.parametrize("dtype,row", [(torch.float32, 48), (torch.bfloat16, 48), (torch.bfloat16, 112)])
@pytest.mark.parametrize("window", [1, 37, 64, 65])
def test_a_latent_row_at_the_windows_edge(dtype, row, window):
    """Key and value are one row: the last queries look for the window's last place, the one beyond it and near ones."""
    g = torch.Generator().manual_seed(window)
    T, H = window + 90, 4
    c = torch.randn(T, row, generator=g)
    c = c / c.norm(dim=-1, keepdim=True)
    q = 0.1 * torch.randn(T, H, row, generator=g)
    for i, back in enumerate((window - 1, window, max(0, window - 2), window + 1, 0)):
        q[T - 1 - 7 * i] = 12.0 * c[T - 1 - 7 * i - back]
    c, q = c.to(dtype), q.to(dtype)
    ref = plain.softmax_attention(q.double(), c.double()[:, None], c.double()[:, None], 1.0, window=window)
    off = plain.softmax_attention(q.double(), c.double()[:, None], c.double()[:, None], 1.0, window=window + 1)
    assert float((off - ref).abs().max()) > 0.1
    cd, qd = c.to(DEV), q.reshape(T, -1).to(DEV)
    common = dict(n_kv=1, group=H, head_dim=row, scale=1.0, cap=0.0, window=window, batch=1)
    out = torch.empty(T, H * row, dtype=dtype, device=DEV)
    kernels.attention_simt(qd, out, i32(0, T), i32(T), k=cd, v=cd, max_q_len=T, **common)
    close(out.view(T, H, row), ref, dtype, "exact kernel, prompt")
    if dtype == torch.bfloat16:
        out.zero_()
        kernels.attention_prefill_mma(qd, out, i32(0, T), cd, cd, max_q_len=T, **common)
        close(out.view(T, H, row), ref, dtype, "tensor cores, prompt")
    # decoding from a ring on pages handed out in any order, NaN where nothing was written
    ring = (window + 63) // 64 * 64
    held = min(T, ring)
    n_pages = (held + 63) // 64
    order = torch.randperm(n_pages + 2, generator=g)[:n_pages]
    pages = torch.full((n_pages + 2, 1, 64, row), float("nan")).to(dtype)
    for p in range(T):
        at = p % ring
        pages[int(order[at // 64]), 0, at % 64] = c[p]
    pt, pd = order.to(torch.int32)[None].to(DEV), pages.to(DEV)
    one = torch.empty(1, H * row, dtype=dtype, device=DEV)
    paged = dict(k_pages=pd, v_pages=pd, page_table=pt, ring=ring, page_size=64)
    kernels.attention_simt(qd[-1:], one, i32(0, 1), i32(T), max_q_len=1, **common, **paged)
    close(one.view(H, row), ref[-1], dtype, "exact kernel, ring")
    if dtype == torch.bfloat16:
        for splits in (1, 2):
            one.zero_()
            kernels.attention_decode_mma(qd[-1:], one, i32(0, 1), i32(T), pd, pd, pt, ring=ring, page_size=64, n_splits=splits, **common)
            close(one.view(H, row), ref[-1], dtype, "tensor cores, ring")


# --- capped attention: a far key among hundreds --------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,d,dv,cap", [(8, 2, 112, 176, 18.0), (4, 2, 32, 32, 15.0), (2, 2, 12, 20, 10.0), (4, 1, 64, 48, 0.0)])
def test_a_far_key_under_a_cap(dtype, H, G, d, dv, cap):
    g = torch.Generator().manual_seed(d)
    T = 700
    k = torch.randn(T, G, d, generator=g)
    k = k / k.norm(dim=-1, keepdim=True)
    v = torch.randn(T, G, dv, generator=g)
    q = 0.1 * torch.randn(T, H, d, generator=g)
    for p, j in ((699, 0), (698, 63), (690, 64), (650, 1), (640, 127), (512, 300)):
        for h in range(H):
            q[p, h] = 14.0 * k[j, h // (H // G)]
    q, k, v = q.to(dtype), k.to(dtype), v.to(dtype)
    ref = plain.softmax_attention(q.double(), k.double(), v.double(), 1.0, cap)
    common = dict(n_kv=G, group=H // G, head_dim=d, scale=1.0, cap=cap, window=0, batch=1)
    qd, kd, vd = (x.reshape(T, -1).to(DEV) for x in (q, k, v))
    out = torch.empty(T, H * dv, dtype=dtype, device=DEV)
    kernels.attention_simt(qd, out, i32(0, T), i32(T), k=kd, v=vd, v_dim=dv, max_q_len=T, **common)
    close(out.view(T, H, dv), ref, dtype, "exact kernel")
    if dtype == torch.bfloat16 and kernels.attention_headmix_ok(d, dv, H // G, False):
        out.zero_()
        kernels.attention_headmix_prefill(qd, out, i32(0, T), kd, vd, v_dim=dv, max_q_len=T, **common)
        close(out.view(T, H, dv), ref, dtype, "tensor cores")


# --- the rest ------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_a_tables_part_behind_an_activation(dtype):
    g = torch.Generator().manual_seed(3)
    for T, n, first, cols, parts in ((1, 1, 0, 1, 1), (7, 5, 10, 20, 3), (300, 12, 24, 36, 1)):
        z = torch.randn(parts, T, n, generator=g)
        table = torch.randn(11, cols, generator=g).to(dtype)
        ids = torch.randint(0, 11, (T,), generator=g)
        out = torch.empty(T, n, dtype=dtype, device=DEV)
        kernels.table_gate((z[0] if parts == 1 else z).contiguous().to(DEV), ids.to(torch.int32).to(DEV), table.to(DEV), first, "gelu_tanh", out)
        close(out, plain.gelu_tanh(z.double().sum(dim=0)) * table.double()[ids][:, first:first + n], dtype)


def test_scaled_logits():
    g = torch.Generator().manual_seed(4)
    for T in (1, 9, 40, 128):
        x, w = torch.randn(T, 64, generator=g).bfloat16(), torch.randn(200, 64, generator=g).bfloat16()
        out = torch.empty(T, 200, device=DEV)
        ref = x.double() @ w.double().T * 0.375
        kernels.gemm_stream(x.to(DEV), w.to(DEV), out, "softcap", scale=0.375)
        close(out, ref)
        kernels.gemm_stream(x.to(DEV), w.to(DEV), out, "softcap", cap=2.0, scale=0.375)
        close(out, 2.0 * torch.tanh(ref / 2.0))
    y = torch.randn(5, 33, generator=g)
    out = torch.empty(5, 33, device=DEV)
    kernels.softcap(y.to(DEV), out, 0.0, 3.5)
    close(out, 3.5 * y.double())


@pytest.mark.parametrize("shape", [(3, 37), (300, 1024)])
def test_the_weighted_sum_of_two_mixers(shape):
    g = torch.Generator().manual_seed(5)
    a, b = torch.randn(*shape, generator=g), torch.randn(2, *shape, generator=g)
    out = torch.empty(shape, device=DEV)
    kernels.scaled_sum(a.to(DEV), -1.25, b.to(DEV), 0.5, out)
    close(out, -1.25 * a.double() + 0.5 * b.double().sum(dim=0))
