"""Relulix as a layout of parts.

Layers in the parallel arrangement with one norm (x += mixer(n(x)) + ff(n(x))), the norm's gain a single number; two
kinds of mixer: attention (biases on q, k and v, a stretched rotation of part of a head, capped scores, a sliding
window, a sink with score 0; a layer may read an earlier layer's keys and values instead of having its own) and
retention (rotated q and k, a fixed decay per head, every head's result normed by itself, a silu gate); routed experts
with a biased router (softmax over the chosen scores) and a clamped gate; the embedding scaled; an output matrix of
its own.  Every size and constant comes from config.json.

Tensor names: ``embed``, ``final.norm``, ``head`` and, for layer i, ``l<i>.norm1``, ``l<i>.mix.{q,q.b,k,k.b,v,v.b,o}``
(attention; without k, k.b, v, v.b where another layer's are read), ``l<i>.mix.{q,k,v,g,o}`` (retention),
``l<i>.mlp.{router,router.b,e<j>.{gate,up,down}}``.
"""
from __future__ import annotations

from ..config import RelulixConfig, register_architecture
from ..parts import BlockSpec, EmbeddingSpec, HeadSpec, LayerCall, ModelLayout, PartSpec


def _rotation(dim: int, rot: dict) -> PartSpec:
    return PartSpec("position", "rope", dict(head_dim=dim, theta=float(rot["base"]), rotary_dim=rot["dims"],
                                             stretch=rot.get("scaling")))


def _attention(W: int, m: dict, p: str, lends: bool) -> PartSpec:
    borrows = m.get("kv_from") is not None
    names = {"o": p + "o"}
    for n in ("q",) if borrows else ("q", "k", "v"):
        names[n], names[n + "_bias"] = p + n, p + n + ".b"
    return PartSpec("mixer", "attention",
                    dict(hidden=W, n_q=m["heads"], n_kv=m["kv_heads"], head_dim=m["dim"], v_dim=m["vdim"],
                         scale=float(m["scale"]), softcap=float(m.get("softcap") or 0.0),
                         window=m["mask"]["size"] if m.get("mask") is not None else None,
                         position=_rotation(m["dim"], m["rot"]), bias="qkv", sink="zero", lends_kv=lends,
                         borrows_kv=borrows), names)


def _retention(W: int, m: dict, eps: float, p: str) -> PartSpec:
    return PartSpec("mixer", "decay_attention",
                    dict(hidden=W, heads=m["heads"], dim=m["dim"], v_dim=m["vdim"], decay=tuple(m["decay"]), eps=eps,
                         activation="none", norm="head", gate="silu", position=_rotation(m["dim"], m["rot"]),
                         k_scale=m["dim"] ** -0.5),
                    {n: p + n for n in ("q", "k", "v", "g", "o")})


def _experts(W: int, mlp: dict, p: str) -> PartSpec:
    n = mlp["router"]["experts"]
    names = {"router": p + "router", "router_bias": p + "router.b"}
    for e in range(n):
        for mat in ("gate", "up", "down"):
            names[f"e{e}.{mat}"] = f"{p}e{e}.{mat}"
    return PartSpec("feedforward", "routed_experts",
                    dict(hidden=W, inter=mlp["expert"]["ff"], experts=n, top=mlp["router"]["top"],
                         activation="clamped_gate", limit=float(mlp["expert"]["limit"]), scale_input=False, gated=True,
                         router="softmax_chosen", router_bias=True), names)


def relulix_layout(cfg: RelulixConfig) -> ModelLayout:
    W, eps = cfg.width, cfg.eps

    def norm(name: str) -> PartSpec:
        return PartSpec("norm", "rmsnorm", dict(size=W, eps=eps, scalar=True), {"weight": name})

    read = {layer["mixer"].get("kv_from") for layer in cfg.layers}       # whose keys and values a later layer reads
    blocks, schedule = [], []
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer["mixer"]
        if layer["type"] == "attention":
            mixer = _attention(W, m, p + "mix.", lends=i in read)
        else:
            mixer = _retention(W, m, eps, p + "mix.")
        mlp = layer.get("mlp")
        blocks.append(BlockSpec(kind="parallel_one_norm", mixer=mixer, pre_mixer_norm=norm(p + "norm1"),
                                feedforward=_experts(W, mlp, p + "mlp.") if mlp is not None else None))
        schedule.append(LayerCall(i, cache_of=m.get("kv_from")))
    return ModelLayout(
        embedding=EmbeddingSpec("embed", cfg.vocab, W, scale=cfg.embedding_scale),
        blocks=blocks,
        schedule=schedule,
        final_norm=norm("final.norm"),
        head=HeadSpec("head"))


register_architecture(RelulixConfig, relulix_layout)
