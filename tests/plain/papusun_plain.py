"""Papusun restated plainly: whole sequences, float64, one function per mechanism.

Nothing here is shared with the package: the functions take the tensors of a checkpoint by name (a dict of float64
tensors) and the configuration as the dict config.json holds.  Notation: T tokens, W width, x the residual stream
(T, W), n the normed input of a sublayer.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def kept(x):
    """Every result that a run in a 16-bit element type rounds before the next product passes through here; a test that
    asks how large an error rounding alone makes puts a rounding in its place (``rounded_forward``)."""
    return x


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# --- norms ---------------------------------------------------------------------------------------------------------
def layer_norm(x, gain, eps):
    """Mean taken off, divided by the standard deviation, a gain, no bias: the norm of the layers and of the output."""
    c = x - x.mean(dim=-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(dim=-1, keepdim=True) + eps) * gain


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def unit_length(x):
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


# --- rotation ------------------------------------------------------------------------------------------------------
def frequencies(rot: dict):
    """Angle per position of every pair.  With ``scaling``: turns shorter than original / high keep their frequency,
    turns longer than original / low have it divided by the factor, those between get a blend of both."""
    dims, base = int(rot["dims"]), float(rot["base"])
    plain = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return plain
    factor, low, high, original = (float(sc[k]) for k in ("factor", "low", "high", "original"))
    out = []
    for f in plain:
        turn = 2.0 * math.pi / f
        if turn < original / high:
            out.append(f)
        elif turn > original / low:
            out.append(f / factor)
        else:
            s = (original / turn - low) / (high - low)
            out.append((1.0 - s) * f / factor + s * f)
    return out


def rotate(x, rot: dict, first: int = 0):
    """x (T, heads, d) at positions first, first + 1, ...: entries 2i and 2i + 1 of a head form a pair."""
    f = frequencies(rot)
    n = 2 * len(f)
    a = (torch.arange(x.shape[0], dtype=F64)[:, None] + first) * torch.tensor(f, dtype=F64)[None, :]
    c, s = torch.cos(a).to(x.dtype)[:, None, :], torch.sin(a).to(x.dtype)[:, None, :]
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    out = x.clone()
    out[..., 0:n:2] = u * c - v * s
    out[..., 1:n:2] = v * c + u * s
    return out


# --- softmax attention ---------------------------------------------------------------------------------------------
def softmax_attention(q, k, v, scale, cap=0.0, window=None, first=0):
    """q (Tq, H, d) at positions first, first + 1, ...; k (Tk, G, d), v (Tk, G, dv) at positions 0, 1, ...: the query
    at i weighs the keys j <= i (with a window: i - window < j) by the softmax of their scores.  (Tq, H, dv)."""
    Tq, H, _ = q.shape
    Tk, G, _ = k.shape
    back = (torch.arange(Tq)[:, None] + first) - torch.arange(Tk)[None, :]
    seen = back >= 0
    if window:
        seen = seen & (back < window)
    heads = []
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        if cap:
            s = cap * torch.tanh(s / cap)
        s = torch.where(seen, s, torch.full_like(s, float("-inf")))
        heads.append(torch.softmax(s, dim=-1) @ v[:, g])
    return torch.stack(heads, dim=1)


def capped_attention(n, t, p, m):
    """Attention with biases on q, k and v, rotated queries and keys and capped scores."""
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = n.shape[0]
    q = rotate((n @ t[p + "q"].T + t[p + "q.b"]).view(T, H, d), m["rot"])
    k = rotate((n @ t[p + "k"].T + t[p + "k.b"]).view(T, G, d), m["rot"])
    v = (n @ t[p + "v"].T + t[p + "v.b"]).view(T, G, dv)
    o = softmax_attention(kept(q), kept(k), kept(v), m["scale"], m.get("softcap") or 0.0)
    return kept(o.reshape(T, H * dv)) @ t[p + "o"].T


# --- latent attention ----------------------------------------------------------------------------------------------
def latent_attention(n, t, p, m, eps, lent):
    """``lent``: layer index -> (latents, rotated shared key part) of the latent layers so far that have their own; the
    layer adds its pair under ``lent["here"]`` unless it reads another layer's."""
    H, dn, dr, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    T = n.shape[0]
    cq = kept(unit_rms(n @ t[p + "dq"].T, eps) * t[p + "dq.norm"])
    q = (cq @ t[p + "uq"].T).view(T, H, dn + dr)
    if m.get("kv_from") is None:
        row = n @ t[p + "dkv"].T
        c = kept(unit_rms(row[:, :R], eps) * t[p + "dkv.norm"])
        shared = kept(rotate(row[:, None, R:], m["rot"]))
        lent["here"] = (c, shared)
    else:
        c, shared = lent[m["kv_from"]]
    q = torch.cat([q[..., :dn], rotate(q[..., dn:], m["rot"])], dim=-1)
    k = torch.cat([(c @ t[p + "uk"].T).view(T, H, dn), shared.expand(T, H, dr)], dim=-1)
    v = (c @ t[p + "uv"].T).view(T, H, dv)
    o = softmax_attention(kept(q), kept(k), kept(v), m["scale"], 0.0, (m.get("mask") or {}).get("size"))
    o = kept(o) * torch.sigmoid(n @ t[p + "g"].T)[:, :, None]
    return kept(o.reshape(T, H * dv)) @ t[p + "o"].T


# --- gated delta rule ----------------------------------------------------------------------------------------------
def short_conv(u, taps):
    """u (T, C), taps (C, K): every channel's newest K inputs (zeros before the start) weighed by its taps."""
    T, K = u.shape[0], taps.shape[1]
    padded = torch.cat([torch.zeros(K - 1, u.shape[1], dtype=u.dtype), u])
    return sum(padded[j:j + T] * taps[:, j] for j in range(K))


def delta_states(q, k, v, decay, beta, S=None):
    """q, k (T, H, d), v (T, H, dv), decay, beta (T, H): the state is decayed, then the value it holds for k is moved
    by the share beta towards v, then it is read with q.  Returns (o (T, H, dv), the last S (H, d, dv))."""
    T, H, d = q.shape
    if S is None:
        S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype)
    rows = []
    for i in range(T):
        S = S * decay[i, :, None, None]
        u = beta[i, :, None] * (v[i] - torch.einsum("hdv,hd->hv", S, k[i]))
        S = S + k[i, :, :, None] * u[:, None, :]
        rows.append(torch.einsum("hdv,hd->hv", S, q[i]))
    return torch.stack(rows), S


def delta_rule(n, t, p, m, eps):
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = n.shape[0]
    q = unit_length(silu(short_conv(n @ t[p + "q"].T, t[p + "q.conv"])).view(T, G, d)) * d ** -0.5
    k = unit_length(silu(short_conv(n @ t[p + "k"].T, t[p + "k.conv"])).view(T, G, d))
    v = silu(short_conv(n @ t[p + "v"].T, t[p + "v.conv"])).view(T, H, dv)
    beta = torch.sigmoid(n @ t[p + "b"].T)
    dt = torch.nn.functional.softplus(n @ t[p + "a"].T + t[p + "dt_bias"], threshold=100.0)
    decay = torch.exp(-torch.exp(t[p + "A_log"]) * dt)
    own = [h // (H // G) for h in range(H)]                       # which q / k head a value head works with
    o, _ = delta_states(q[:, own], k[:, own], v, decay, beta)
    o = unit_rms(o, eps) * t[p + "norm"]
    return kept(o.reshape(T, H * dv) * silu(n @ t[p + "g"].T)) @ t[p + "o"].T


# --- feed-forward, per-token side input ----------------------------------------------------------------------------
def dense(n, t, p):
    return kept(silu(kept(n @ t[p + "gate"].T)) * kept(n @ t[p + "up"].T)) @ t[p + "down"].T


def side_input(x, e, t, p, eps):
    """x (T, W) the stream, e (T, D) this layer's part of the tokens' own rows: what is added to the stream."""
    g = kept(gelu_tanh(kept(x) @ t[p + "gate"].T) * e)
    return unit_rms(g @ t[p + "proj"].T, eps) * t[p + "norm"]


# --- the model -----------------------------------------------------------------------------------------------------
def forward(config: dict, tensors: dict, tokens, streams=None):
    """Logits (T, vocab) of one sequence; ``streams`` (a list) receives the residual stream after every layer."""
    t = {k: (v.to(F64) if v.is_floating_point() else v) for k, v in tensors.items()}
    eps = float(config["norm"]["eps"])
    ids = torch.tensor(tokens)
    D = config["token_side"]["dim"]
    x = t["embed"][ids]
    lent = {}
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        n = kept(layer_norm(x, t[p + "norm1"], eps))
        if layer["type"] == "latent_attention":
            y = latent_attention(n, t, p + "mix.", m, eps, lent)
            if "here" in lent:
                lent[i] = lent.pop("here")
        else:
            y = m["left_scale"] * capped_attention(n, t, p + "mix.left.", m["left"]) \
                + m["right_scale"] * delta_rule(n, t, p + "mix.right.", m["right"], eps)
        x = x + y
        if layer.get("mlp") is not None:
            x = x + dense(kept(layer_norm(x, t[p + "norm2"], eps)), t, p + "mlp.")
        x = x + side_input(x, t["side.embed"][ids][:, i * D:(i + 1) * D], t, p + "side.", eps)
        if streams is not None:
            streams.append(x.clone())
    return (kept(layer_norm(x, t["final.norm"], eps)) @ t["head"].T) * float(config["logit_scale"])


def rounded_forward(config: dict, tensors: dict, tokens):
    """``forward`` with every kept result rounded to bfloat16."""
    global kept
    exact = kept
    kept = lambda x: x.to(torch.bfloat16).to(x.dtype)
    try:
        return forward(config, tensors, tokens)
    finally:
        kept = exact


def rounding_errors(config: dict, tensors: dict, requests):
    """What rounding alone does to the rows of these requests: every row's largest error relative to its request's
    largest logit, smallest first."""
    out = []
    for p in requests:
        ref = forward(config, tensors, p)
        out += ((rounded_forward(config, tensors, p) - ref).abs().amax(dim=1) / ref.abs().max()).tolist()
    return sorted(out)
