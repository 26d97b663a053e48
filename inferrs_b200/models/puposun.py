"""The Puposun decoder, written down as a :class:`ModelSpec`.

This file holds no arithmetic.  It says which parts the design is made of, with which tensor names and which
config.json values:

* a layer has one norm; the mixer and the feed-forward read its output side by side and both join the stream
  (arrangement ``parallel``);
* both mixers are grouped-query attention whose values are the projected keys (before rotation; no projection of their
  own).  "attention": biases on q, k and the output, the two halves of the rotated numbers turn together, scores squashed
  by a cap, every earlier key visible, a sink of score 0 in the softmax.  "attention_2": no biases, neighbouring numbers
  turn together, a sliding window beside the sequence's first tokens, one sigmoid gate per head;
* the feed-forward is routed experts chosen by sigmoid scores with a correction, inside the best groups, and weighed by
  their share of the chosen scores;
* a run of layers may be passed several times with the same weights; the embedding output joins the stream at the start
  of every pass but the first;
* embedding rows are scaled, logits squashed by a cap;
* tensors: ``embed``, ``l<i>.norm1``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``, ``head``.
"""
from __future__ import annotations

from ..config.base import register_architecture
from ..config.puposun import PuposunConfig, PuposunLayer
from ..parts.spec import (AttentionSpec, LayerSpec, ModelSpec, NormSpec, PositionSpec, RoutedExpertsSpec, SubLayerSpec,
                          default_schedule, looped_schedule)

ARCHITECTURE = "Puposun"
SINK_SCORE = 0.0         # the softmax of "attention" has one added to its denominator


def _position(cfg: PuposunConfig, layer: PuposunLayer, kind: str) -> PositionSpec:
    rot = layer.get("rot")
    if not rot:
        return PositionSpec(kind="none", max_positions=cfg.max_positions)
    return PositionSpec(kind=kind, rot_dim=int(rot["dims"]), theta=float(rot["base"]), max_positions=cfg.max_positions)


def _mixer(cfg: PuposunConfig, layer: PuposunLayer, p: str) -> AttentionSpec:
    sizes = dict(width=cfg.width, n_heads=layer.get("heads"), n_kv_heads=layer.get("kv_heads"), head_dim=layer.get("dim"),
                 value_is_key=True, scale=float(layer.get("scale")), q_proj=f"{p}.q", k_proj=f"{p}.k", o_proj=f"{p}.o")
    if layer.type == "attention":
        cap = layer.get("softcap")
        return AttentionSpec(**sizes, position=_position(cfg, layer, "rotary_scaled"), q_bias=f"{p}.q.b", k_bias=f"{p}.k.b",
                             o_bias=f"{p}.o.b", score_cap=None if cap is None else float(cap), sink_score=SINK_SCORE)
    mask = layer.get("mask")
    return AttentionSpec(**sizes, position=_position(cfg, layer, "rotary_scaled_interleaved"), head_gate=f"{p}.g",
                         window=int(mask["size"]) if mask else None,
                         keep_first=int(mask.get("keep_first", 0)) if mask else 0)


def _feed_forward(cfg: PuposunConfig, layer: PuposunLayer, p: str) -> RoutedExpertsSpec:
    router = layer.mlp_get("router")
    groups = router.get("groups") or {"count": 0, "keep": 0}
    return RoutedExpertsSpec(
        width=cfg.width, inner=layer.mlp_get("expert")["ff"], top=router["top"], router=f"{p}.router", router_bias=None,
        experts=tuple((f"{p}.e{e}.gate", f"{p}.e{e}.up", f"{p}.e{e}.down") for e in range(router["experts"])),
        scoring="sigmoid_share", route_scale=float(router["scale"]), correction=f"{p}.correction",
        groups=groups["count"], groups_keep=groups["keep"])


def build_spec(cfg: PuposunConfig) -> ModelSpec:
    layers = []
    for i, layer in enumerate(cfg.layers):
        subs = [SubLayerSpec(part=_mixer(cfg, layer, f"l{i}.mix"), category="mixer",
                             norm=NormSpec(size=cfg.width, eps=cfg.norm_eps, weight=f"l{i}.norm1"))]
        if layer.mlp is not None:
            subs.append(SubLayerSpec(part=_feed_forward(cfg, layer, f"l{i}.mlp"), category="feed_forward"))
        layers.append(LayerSpec(sublayers=tuple(subs), arrangement="parallel"))
    schedule = default_schedule(len(layers)) if cfg.loop is None \
        else looped_schedule(len(layers), *cfg.loop, add_embedding=True)
    return ModelSpec(
        vocab_size=cfg.vocab,
        width=cfg.width,
        embedding="embed",
        layers=tuple(layers),
        schedule=schedule,
        final_norm=NormSpec(size=cfg.width, eps=cfg.norm_eps, weight="final.norm"),
        lm_head="head",
        lm_head_optional=False,
        max_positions=cfg.max_positions,
        embedding_scale=cfg.embedding_scale,
        logit_softcap=cfg.logit_softcap,
        eos_token_ids=cfg.eos_token_ids,
        architecture=ARCHITECTURE,
    )


register_architecture(ARCHITECTURE, PuposunConfig, build_spec, model_type="puposun", replace=True)
