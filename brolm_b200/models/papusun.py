"""Papusun as a layout of parts.

Pre-norm layers (layer norms with a gain) that end with an input of their own per token: h += n(proj(gelu(gate(h)) * e)),
e being the layer's part of the token's row in a table shared by all layers.  Two kinds of mixer: attention (biases on q,
k and v, a rotation of neighbouring pairs with frequencies scaled by wavelength, capped scores) side by side with a gated
delta rule, or windowed latent attention (queries through a latent of their own, a gate per head; a layer may read an
earlier layer's latents instead of having its own); a dense gated feed-forward; an output matrix of its own and scaled
logits.  Every size and constant comes from config.json.

Tensor names: ``embed``, ``side.embed``, ``final.norm``, ``head`` and, for layer i, ``l<i>.norm1``, ``l<i>.norm2``,
``l<i>.mix.left.{q,q.b,k,k.b,v,v.b,o}`` and
``l<i>.mix.right.{q,q.conv,k,k.conv,v,v.conv,b,a,A_log,dt_bias,norm,g,o}`` (parallel) or
``l<i>.mix.{dq,dq.norm,uq,dkv,dkv.norm,uk,uv,g,o}`` (latent attention; without dkv and dkv.norm where another layer's
latents are read), ``l<i>.mlp.{gate,up,down}``, ``l<i>.side.{gate,proj,norm}``.
"""
from __future__ import annotations

from ..config import PapusunConfig, register_architecture
from ..parts import BlockSpec, EmbeddingSpec, HeadSpec, LayerCall, ModelLayout, PartSpec


def _rotation(dim: int, rot: dict) -> PartSpec:
    return PartSpec("position", "rope", dict(head_dim=dim, theta=float(rot["base"]), rotary_dim=rot["dims"],
                                             pairing="interleaved", bands=rot.get("scaling")))


def _parallel(W: int, m: dict, eps: float, p: str) -> PartSpec:
    a, r = m["left"], m["right"]
    names = {"o": p + "left.o"}
    for n in ("q", "k", "v"):
        names[n], names[n + "_bias"] = f"{p}left.{n}", f"{p}left.{n}.b"
    left = PartSpec("mixer", "attention",
                    dict(hidden=W, n_q=a["heads"], n_kv=a["kv_heads"], head_dim=a["dim"], v_dim=a["vdim"],
                         scale=float(a["scale"]), softcap=float(a.get("softcap") or 0.0), bias="qkv",
                         position=_rotation(a["dim"], a["rot"])), names)
    names = {n: f"{p}right.{n}" for n in ("q", "k", "v", "b", "a", "A_log", "dt_bias", "norm", "g", "o")}
    names.update({n + "_conv": f"{p}right.{n}.conv" for n in ("q", "k", "v")})
    right = PartSpec("mixer", "gated_delta_rule",
                     dict(hidden=W, heads=r["heads"], kv_heads=r["kv_heads"], dim=r["dim"], v_dim=r["vdim"],
                          taps=r["conv"], eps=eps), names)
    return PartSpec("mixer", "side_by_side", dict(left=left, right=right, left_scale=float(m["left_scale"]),
                                                  right_scale=float(m["right_scale"])))


def _latent(W: int, m: dict, eps: float, p: str, lends: bool) -> PartSpec:
    borrows = m.get("kv_from") is not None
    names = {n: p + n for n in ("dq", "uq", "uk", "uv", "g", "o")} | {"dq_norm": p + "dq.norm"}
    if not borrows:
        names |= {"dkv": p + "dkv", "dkv_norm": p + "dkv.norm"}
    return PartSpec("mixer", "latent_attention",
                    dict(hidden=W, heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], vdim=m["vdim"],
                         kv_rank=m["kv_rank"], q_rank=m["q_rank"], scale=float(m["scale"]), eps=eps,
                         window=m["mask"]["size"] if m.get("mask") is not None else None, sink=False, gate="head",
                         position=_rotation(m["rot_dim"], m["rot"]), lends_kv=lends, borrows_kv=borrows), names)


def papusun_layout(cfg: PapusunConfig) -> ModelLayout:
    W, eps, D, n = cfg.width, cfg.eps, cfg.side_dim, len(cfg.layers)

    def norm(name: str) -> PartSpec:
        return PartSpec("norm", "layernorm", dict(size=W, eps=eps), {"weight": name})

    read = {layer["mixer"].get("kv_from") for layer in cfg.layers}       # whose latents a later layer reads
    blocks, schedule = [], []
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer["mixer"]
        if layer["type"] == "parallel":
            mixer = _parallel(W, m, eps, p + "mix.")
        else:
            mixer = _latent(W, m, eps, p + "mix.", lends=i in read)
        ff = None
        if layer.get("mlp") is not None:
            ff = PartSpec("feedforward", "gated", dict(hidden=W, inter=layer["mlp"]["ff"], activation="silu"),
                          {mat: f"{p}mlp.{mat}" for mat in ("gate", "up", "down")})
        side = PartSpec("feedforward", "token_side",
                        dict(hidden=W, dim=D, vocab=cfg.vocab, table_cols=n * D, first=i * D, activation="gelu_tanh"),
                        {"gate": p + "side.gate", "proj": p + "side.proj", "table": "side.embed"})
        blocks.append(BlockSpec(
            kind="sandwich_side", mixer=mixer, pre_mixer_norm=norm(p + "norm1"), feedforward=ff,
            pre_ffn_norm=norm(p + "norm2") if ff is not None else None,
            more={"side": side, "entry": PartSpec("norm", "cast", dict(size=W)),
                  "post_side_norm": PartSpec("norm", "rmsnorm", dict(size=W, eps=eps), {"weight": p + "side.norm"})}))
        schedule.append(LayerCall(i, cache_of=m.get("kv_from")))
    return ModelLayout(
        embedding=EmbeddingSpec("embed", cfg.vocab, W),
        blocks=blocks,
        schedule=schedule,
        final_norm=norm("final.norm"),
        head=HeadSpec("head", scale=float(cfg.logit_scale)))


register_architecture(PapusunConfig, papusun_layout)
