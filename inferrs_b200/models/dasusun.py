"""The Dasusun decoder, written down as a :class:`ModelSpec`.

This file holds no arithmetic.  It says which parts the design is made of, with which tensor names and which
config.json values:

* every sub-layer has a norm before it and one on its output, RMS norms whose weights are stored around zero, and a
  vector that scales what it adds to the stream; what a mixer reads is first replaced by itself plus a short causal
  convolution over time (``canon.taps`` taps per channel);
* what a layer hands on is a learned weighted sum of the embedding and all layers' results so far;
* the mixer is attention over cached latents (queries through a latent of their own, keys and values made per head from
  one latent per token, one rotated key part shared by all heads, with frequencies that may be stretched for long
  contexts), inside a sliding window or over every earlier token;
* the feed-forward is down(gelu_tanh(up)); the embedding table is the head;
* tensors: ``embed``, ``l<i>.norm1|norm1b|ls1|canon1|dwa``, ``l<i>.mix.*``, and with a feed-forward
  ``l<i>.norm2|norm2b|ls2``, ``l<i>.mlp.up|down``, ``final.norm``.
"""
from __future__ import annotations

from ..config.base import register_architecture
from ..config.dasusun import DasusunConfig
from ..parts.spec import (DenseSpec, DepthAverageSpec, InputConvSpec, LatentAttentionSpec, LayerSpec, ModelSpec, NormSpec,
                          PositionSpec, SubLayerSpec, default_schedule)

ARCHITECTURE = "Dasusun"


def _norm(cfg: DasusunConfig, name: str) -> NormSpec:
    return NormSpec(size=cfg.width, eps=cfg.norm_eps, weight=name, weight_offset=1.0)


def _mixer(cfg: DasusunConfig, i: int) -> LatentAttentionSpec:
    layer, p = cfg.layers[i], f"l{i}.mix"
    rot, mask = layer.get("rot"), layer.get("mask")
    scaling = rot.get("scaling")
    position = PositionSpec(kind="rotary_scaled", rot_dim=int(rot["dims"]), theta=float(rot["base"]),
                            max_positions=cfg.max_positions,
                            scaling=None if not scaling else tuple(float(scaling[k])
                                                                   for k in ("factor", "original", "fast", "slow")))
    return LatentAttentionSpec(
        width=cfg.width, n_heads=layer.get("heads"), key_dim=layer.get("dim"), value_dim=layer.get("vdim"),
        q_rank=layer.get("q_rank"), kv_rank=layer.get("kv_rank"), scale=float(layer.get("scale")), eps=cfg.norm_eps,
        dq_proj=f"{p}.dq", dq_norm=f"{p}.dq.norm", uq_proj=f"{p}.uq", dkv_proj=f"{p}.dkv", dkv_norm=f"{p}.dkv.norm",
        uk_proj=f"{p}.uk", uv_proj=f"{p}.uv", o_proj=f"{p}.o", window=int(mask["size"]) if mask else None,
        rot_dim=layer.get("rot_dim"), position=position)


def build_spec(cfg: DasusunConfig) -> ModelSpec:
    layers = []
    for i, layer in enumerate(cfg.layers):
        subs = [SubLayerSpec(part=_mixer(cfg, i), category="mixer", norm=_norm(cfg, f"l{i}.norm1"),
                             post_norm=_norm(cfg, f"l{i}.norm1b"), layer_scale=f"l{i}.ls1",
                             input_conv=InputConvSpec(width=cfg.width, taps=cfg.canon_taps, weight=f"l{i}.canon1"))]
        if layer.ff is not None:
            subs.append(SubLayerSpec(part=DenseSpec(width=cfg.width, inner=layer.ff, up_proj=f"l{i}.mlp.up",
                                                    down_proj=f"l{i}.mlp.down", activation="gelu_tanh"),
                                     category="feed_forward", norm=_norm(cfg, f"l{i}.norm2"),
                                     post_norm=_norm(cfg, f"l{i}.norm2b"), layer_scale=f"l{i}.ls2"))
        layers.append(LayerSpec(sublayers=tuple(subs), arrangement="sandwich",
                                depth_average=DepthAverageSpec(weight=f"l{i}.dwa", results=i + 2),
                                unused=tuple((f"l{i}.{n}", (cfg.width,)) for n in layer.idle)))
    return ModelSpec(
        vocab_size=cfg.vocab,
        width=cfg.width,
        embedding="embed",
        layers=tuple(layers),
        schedule=default_schedule(len(layers)),
        final_norm=_norm(cfg, "final.norm"),
        lm_head="embed",
        lm_head_optional=False,
        max_positions=cfg.max_positions,
        eos_token_ids=cfg.eos_token_ids,
        architecture=ARCHITECTURE,
    )


register_architecture(ARCHITECTURE, DasusunConfig, build_spec, model_type="dasusun", replace=True)
