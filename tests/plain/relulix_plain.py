"""Relulix restated plainly: whole sequences, float64, one function per mechanism.

Nothing here is shared with the package: the functions take the tensors of a checkpoint by name (a dict of float64
tensors) and the configuration as the dict config.json holds.  Notation: T tokens, W width, x the residual stream
(T, W), n the input of a layer's two sublayers (the normed stream).
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def kept(x):
    """Every result that a run in a 16-bit element type rounds before the next product passes through here; a test that
    asks how large an error rounding alone makes puts a rounding in its place (``rounded_forward``)."""
    return x


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def scalar_norm(x, gain, eps):
    """The norm of a layer and of the output: one number multiplies every coordinate of the unit row."""
    return kept(unit_rms(x, eps) * gain)


# --- rotation ------------------------------------------------------------------------------------------------------
def frequencies(rot: dict):
    """(angle per position of every pair, the factor both cos and sin are multiplied by)."""
    dims, base = int(rot["dims"]), float(rot["base"])
    plain = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return plain, 1.0
    factor, original = float(sc["factor"]), float(sc["original"])

    def pair_with(turns):            # the pair that goes round `turns` times over the original length
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    first = max(math.floor(pair_with(float(sc["fast"]))), 0)
    last = min(math.ceil(pair_with(float(sc["slow"]))), dims - 1)
    out = []
    for i, f in enumerate(plain):
        share = min(max((i - first) / max(last - first, 0.001), 0.0), 1.0)
        out.append(f / factor * share + f * (1.0 - share))
    return out, 0.1 * math.log(factor) + 1.0


def rotate(x, rot: dict, first: int = 0):
    """x (T, heads, d) at positions first, first + 1, ...: entries i and i + dims/2 of a head form a pair."""
    f, mag = frequencies(rot)
    half = len(f)
    a = (torch.arange(x.shape[0], dtype=F64)[:, None] + first) * torch.tensor(f, dtype=F64)[None, :]
    c, s = (torch.cos(a) * mag).to(x.dtype)[:, None, :], (torch.sin(a) * mag).to(x.dtype)[:, None, :]
    u, v = x[..., :half], x[..., half:2 * half]
    out = x.clone()
    out[..., :half] = u * c - v * s
    out[..., half:2 * half] = v * c + u * s
    return out


# --- attention -----------------------------------------------------------------------------------------------------
def windowed_attention(q, k, v, scale, cap, window, null_sink=True, first=0):
    """q (Tq, H, d) at positions first, first + 1, ...; k (Tk, G, d), v (Tk, G, dv) at positions 0, 1, ...  A query at
    i weighs the keys i - window < j <= i by exp(score) over (1 +) the sum of the exponentials.  (Tq, H, dv)."""
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
        m = s.max(dim=-1, keepdim=True).values
        if null_sink:
            m = m.clamp(min=0.0)
        e = torch.exp(s - m)
        below = e.sum(dim=-1, keepdim=True)
        if null_sink:
            below = below + torch.exp(-m)          # a score of 0 that has no value
        heads.append((e / below) @ v[:, g])
    return torch.stack(heads, dim=1)


def attention(n, t, p, m, lent):
    """``lent``: layer index -> (rotated keys, values) of the attention layers so far that have their own; the layer
    adds its pair under ``lent["here"]`` unless it reads another layer's."""
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = n.shape[0]
    q = rotate((n @ t[p + "q"].T + t[p + "q.b"]).view(T, H, d), m["rot"])
    if m.get("kv_from") is not None:
        k, v = lent[m["kv_from"]]
    else:
        k = rotate((n @ t[p + "k"].T + t[p + "k.b"]).view(T, G, d), m["rot"])
        v = (n @ t[p + "v"].T + t[p + "v.b"]).view(T, G, dv)
        lent["here"] = (k, v)
    o = windowed_attention(kept(q), kept(k), kept(v), m["scale"], m.get("softcap") or 0.0, (m.get("mask") or {}).get("size"))
    return kept(o.reshape(T, H * dv)) @ t[p + "o"].T


# --- retention -----------------------------------------------------------------------------------------------------
def decayed_state(q, k, v, decay, S=None):
    """q, k (T, H, d), v (T, H, dv), decay (H,): S <- decay S + k v^T, o = S^T q, token by token.
    Returns (o (T, H, dv), the last S (H, d, dv))."""
    T, H, d = q.shape
    if S is None:
        S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype)
    rows = []
    for i in range(T):
        S = S * decay[:, None, None] + k[i, :, :, None] * v[i, :, None, :]
        rows.append((S * q[i, :, :, None]).sum(dim=1))
    return torch.stack(rows), S


def retention(n, t, p, m, eps):
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    T = n.shape[0]
    q = rotate((n @ t[p + "q"].T).view(T, H, d), m["rot"])
    k = rotate((n @ t[p + "k"].T).view(T, H, d), m["rot"]) / math.sqrt(d)
    v = (n @ t[p + "v"].T).view(T, H, dv)
    o, _ = decayed_state(q, k, v, torch.tensor(m["decay"], dtype=F64).to(q.dtype))
    o = unit_rms(o, eps).reshape(T, H * dv)                    # every head by its own root mean square
    return kept(o * silu(n @ t[p + "g"].T)) @ t[p + "o"].T


# --- routed experts ------------------------------------------------------------------------------------------------
def clamped_expert(n, t, p, limit):
    g = torch.clamp(kept(n @ t[p + "gate"].T), max=limit)
    u = torch.clamp(kept(n @ t[p + "up"].T), min=-limit, max=limit)
    return kept(g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ t[p + "down"].T


def choose(z, top: int):
    """z (E,) logits of one token -> [(expert, weight)]: the ``top`` largest (ties: the lower index), weighted by the
    softmax over those alone."""
    best = sorted(range(z.numel()), key=lambda e: (-float(z[e]), e))[:top]
    w = torch.softmax(z[best], dim=0)
    return list(zip(best, w))


def routed(n, t, p, mlp):
    r = mlp["router"]
    z = n @ t[p + "router"].T + t[p + "router.b"]
    out = torch.zeros_like(n)
    for i in range(n.shape[0]):
        for e, w in choose(z[i], r["top"]):
            out[i] += w * clamped_expert(n[i:i + 1], t, f"{p}e{e}.", float(mlp["expert"]["limit"]))[0]
    return out


# --- the model -----------------------------------------------------------------------------------------------------
def forward(config: dict, tensors: dict, tokens, streams=None):
    """Logits (T, vocab) of one sequence; ``streams`` (a list) receives the residual stream after every layer."""
    t = {k: (v.to(F64) if v.is_floating_point() else v) for k, v in tensors.items()}
    eps = float(config["norm"]["eps"])
    x = t["embed"][torch.tensor(tokens)] * float(config["embedding"]["scale"])
    lent = {}
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        n = scalar_norm(x, t[p + "norm1"], eps)
        if layer["type"] == "attention":
            y = attention(n, t, p + "mix.", layer["mixer"], lent)
            if "here" in lent:
                lent[i] = lent.pop("here")
        else:
            y = retention(n, t, p + "mix.", layer["mixer"], eps)
        if layer.get("mlp") is not None:
            y = y + routed(n, t, p + "mlp.", layer["mlp"])
        x = x + y
        if streams is not None:
            streams.append(x.clone())
    return scalar_norm(x, t["final.norm"], eps) @ t["head"].T


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
