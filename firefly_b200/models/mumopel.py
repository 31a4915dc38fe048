"""Mumopel as data: a ``ModelSpec`` made of registered parts.

The residual is several streams that every part reads and writes (``hyper_connections``), with a layer norm in front of
each part.  The mixer is grouped-query softmax attention within chunks of positions (``gqa_attention``): one norm over all
query heads together and one over all key heads, interleaved rotary positions on a head's first elements, and a learned
sink a head in the softmax's denominator.  The feed-forward is a SwiGLU (``gated_mlp``), routed experts of the clamped form
whose weights are the softmax over the chosen logits, with a shared expert (``grouped_experts``), or nothing.  A range of
layers may run several times with the same weights; every pass has a cache of its own (the schedule names a layer once per
run).  The output is a layer norm of the streams' sum and the embedding table as the head, its logits capped by a tanh.
Tensor names: ``embed``, ``l<i>.norm1``, ``l<i>.norm2`` (+ ``.b``), ``l<i>.hc1.*``, ``l<i>.hc2.*``, ``l<i>.mix.*``,
``l<i>.mlp.*``, ``final.norm`` (+ ``.b``).
"""
from __future__ import annotations

from ..config.base import LayerSpec, ModelSpec, PartSpec, ScheduleEntry
from ..config.mumopel import MumopelConfig
from .registry import register_architecture

# The design has no longest position (angles are formed from the position); the engine's block tables and its cache
# sizing still want a bound on a request's length.
MAX_POSITIONS = 1 << 20


def _norm(cfg: MumopelConfig, prefix: str) -> PartSpec:
    return PartSpec("layer_norm", dict(size=cfg.width, eps=cfg.norm_eps, weight_leaf="", bias_leaf=".b"), prefix=prefix)


def _attention(cfg: MumopelConfig, mx, p: str):
    """(mixer, position encoding or None)."""
    mask, rot, dim = mx.get("mask"), mx.get("rot"), int(mx["dim"])
    mixer = PartSpec("gqa_attention", dict(
        hidden_size=cfg.width, num_heads=int(mx["heads"]), num_kv_heads=int(mx["kv_heads"]), head_dim=dim,
        value_dim=int(mx["vdim"]), scale=float(mx["scale"]), chunk=int(mask["size"]) if mask else None, qk_norm=True,
        qk_norm_over="all", qk_norm_eps=cfg.norm_eps, q_norm_leaf="q.norm", k_norm_leaf="k.norm", sink_leaf="sink",
        q_leaf="q", k_leaf="k", v_leaf="v", o_leaf="o"), prefix=p)
    position = None
    if rot and int(rot["dims"]) > 0:
        position = PartSpec("rotary", dict(head_dim=dim, rotary_dim=int(rot["dims"]), theta=float(rot["base"]), max_positions=0,
                                           pairing="interleaved"))
    return mixer, position


def _feed_forward(cfg: MumopelConfig, ml, p: str):
    if ml is None:
        return None
    if ml["kind"] == "dense":
        return PartSpec("gated_mlp", dict(hidden_size=cfg.width, intermediate_size=int(ml["ff"]), activation="silu"), prefix=p)
    shared = ml.get("shared")
    return PartSpec("grouped_experts", dict(
        hidden_size=cfg.width, experts=int(ml["router"]["experts"]), top=int(ml["router"]["top"]), ff=int(ml["expert"]["ff"]),
        limit=float(ml["expert"]["limit"]), score="chosen_softmax", renormalize=False, router_bias="router.b",
        shared_ff=int(shared["ff"]) if shared else 0, shared_limit=float(shared["limit"]) if shared else 0.0), prefix=p)


def mumopel_spec(cfg: MumopelConfig) -> ModelSpec:
    layers = []
    for i, L in enumerate(cfg.layers):
        p = f"l{i}"
        mixer, position = _attention(cfg, L["mixer"], f"{p}.mix")
        ff = _feed_forward(cfg, L.get("mlp"), f"{p}.mlp")
        halves = (1, 2) if ff is not None else (1,)
        # a layer without a feed-forward needs no second half's vectors; a file may hold them all the same
        unused = () if ff is not None else ((f"{p}.norm2", cfg.width), (f"{p}.norm2.b", cfg.width), (f"{p}.hc2.in", cfg.streams),
                                            (f"{p}.hc2.out", cfg.streams), (f"{p}.hc2.mix", (cfg.streams, cfg.streams)))
        layers.append(LayerSpec("hyper_connections", mixer, ff, tuple(_norm(cfg, f"{p}.norm{q}") for q in halves), position,
                                params=dict(streams=cfg.streams, connections=tuple(f"{p}.hc{q}" for q in halves),
                                            unused_vectors=unused)))
    order = list(range(len(layers)))
    if cfg.loop:
        a, b = cfg.loop["start"], cfg.loop["stop"]
        order = order[:a] + order[a:b] * cfg.loop["times"] + order[b:]
    return ModelSpec(
        vocab_size=cfg.vocab, hidden_size=cfg.width, max_positions=MAX_POSITIONS,
        embedding=PartSpec("token_embedding", dict(vocab_size=cfg.vocab, hidden_size=cfg.width, tensor="embed")),
        layers=tuple(layers), schedule=tuple(ScheduleEntry(i) for i in order),
        final_norm=PartSpec("stream_sum", dict(streams=cfg.streams, norm=_norm(cfg, "final.norm"))),
        head=PartSpec("lm_head", dict(vocab_size=cfg.vocab, hidden_size=cfg.width, tensor="head", tied_to="embed",
                                      softcap=cfg.logit_softcap or 0.0)),
    )


register_architecture("Mumopel", MumopelConfig, mumopel_spec)
