"""A model assembled from a :class:`ModelSpec`: embedding, scheduled layers, last norm, head.

Nothing here is specific to an architecture.  The reference's counterpart is
``Qwen3Model::forward`` (inferrs-models/src/models/qwen3.rs:398-407): embed,
run the layers, norm, and logits for the rows that are wanted (the reference
wants only the last, inferrs-models/src/models/attention_utils.rs:382-395).
"""
from __future__ import annotations

import inspect
from typing import Dict, List, Optional

import torch

from .. import kernels
from ..cache.storage import KVNeed, StateNeed
from ..parts.basic import Linear, NoNorm, SandwichUpdate, SumUpdate
from ..parts.blocks import BuiltSubLayer, depth_planes
from ..parts.registry import part_class
from ..parts.spec import ModelSpec, TensorDecl
from ..runtime import Runtime


class ModelError(ValueError):
    pass


def declared_tensors(spec: ModelSpec) -> List[TensorDecl]:
    """Every tensor the model's parts expect, in a fixed order, each name once."""
    decls: List[TensorDecl] = [TensorDecl(spec.embedding, (spec.vocab_size, spec.width))]
    for layer in spec.layers:
        for sub in layer.sublayers:
            _check_category(sub.category)
            if sub.norm is not None:
                decls += part_class("norm", sub.norm).declare(sub.norm)
            if sub.part is not None:
                decls += part_class(sub.category, sub.part).declare(sub.part)
            for after in (sub.post_norm, getattr(sub, "sum_norm", None)):
                if after is not None:
                    decls += part_class("norm", after).declare(after)
        decls += _arrangement_tensors(layer)
    if spec.position_table is not None:
        decls.append(TensorDecl(spec.position_table, (spec.max_positions, spec.width)))
    if spec.embedding_norm is not None:
        decls += part_class("norm", spec.embedding_norm).declare(spec.embedding_norm)
    decls += part_class("norm", spec.final_norm).declare(spec.final_norm)
    decls.append(TensorDecl(spec.lm_head, (spec.vocab_size, spec.width), optional=spec.lm_head_optional))
    seen, out = {}, []
    for d in decls:
        if d.name in seen:
            if seen[d.name].shape != d.shape:
                raise ModelError(f"tensor '{d.name}' is declared with shapes {seen[d.name].shape} and {d.shape}")
            continue
        seen[d.name] = d
        out.append(d)
    return out


def _arrangement_tensors(layer) -> List[TensorDecl]:
    """Tensors that belong to the way a layer's sub-layers hang on the residual (an arrangement with ``declare``)."""
    cls = part_class("arrangement", _Arrangement(layer.arrangement))
    return list(cls.declare(layer)) if hasattr(cls, "declare") else []


def _check_category(category: str):
    if category not in ("mixer", "feed_forward"):
        raise ModelError(f"a sub-layer is a 'mixer' or a 'feed_forward', got category '{category}'")


def _mixers(spec: ModelSpec, layer: int):
    """The mixer descriptions of a layer with their classes.  Every mixer of a layer gets the schedule entry's one
    cache id, so at most one of them may keep a cache or a state."""
    out = [(m, part_class("mixer", m)) for m in spec.layers[layer].parts_of("mixer")]
    keepers = [m for m, cls in out if cls.cache_need(m) is not None or cls.state_need(m) is not None]
    if len(keepers) > 1:
        raise ModelError(f"layer {layer} has {len(keepers)} mixers that keep a cache or a state; a schedule entry "
                         f"names one cache, so a layer can have one such mixer")
    return out


def check_schedule(spec: ModelSpec):
    """The schedule names existing layers; every cache has exactly one writer, which runs before its readers."""
    if not spec.schedule:
        raise ModelError("the schedule is empty")
    writers: Dict[int, int] = {}
    averages = depth_planes(spec) > 0
    for i, e in enumerate(spec.schedule):
        if not 0 <= e.layer < len(spec.layers):
            raise ModelError(f"schedule entry {i} names layer {e.layer}; the model has {len(spec.layers)}")
        if e.add_embedding:
            first = spec.layers[e.layer].sublayers[0].norm if spec.layers[e.layer].sublayers else None
            if spec.streams is not None or spec.position_table is not None or spec.embedding_norm is not None or averages \
                    or spec.layers[e.layer].arrangement not in ("sequential", "parallel") \
                    or getattr(first, "kind", None) != "rms" or getattr(first, "groups", 1) != 1:
                raise ModelError(f"schedule entry {i} adds the embedding before layer {e.layer}: that layer starts with a "
                                 f"plain RMS norm, in a sequential or a parallel block, on a residual of one stream that "
                                 f"starts from the plain embedding")
        average = spec.layers[e.layer].depth_average
        if averages and (average is None or average.results != i + 2):
            raise ModelError(f"schedule entry {i} runs layer {e.layer}: with averages over depth every layer averages the "
                             f"{i + 2} results that stand then")
        for mixer, cls in _mixers(spec, e.layer):
            if cls.cache_need(mixer) is None and cls.state_need(mixer) is None:
                continue
            writes = cls.writes_cache(mixer) if hasattr(cls, "writes_cache") else True
            if writes:
                if e.cache in writers:
                    raise ModelError(f"cache {e.cache} is written by schedule entries {writers[e.cache]} and {i}")
                writers[e.cache] = i
            elif e.cache not in writers:
                raise ModelError(f"schedule entry {i} reads cache {e.cache} before any entry has written it")


def cache_needs(spec: ModelSpec):
    """(paged needs, fixed-size state needs) per cache id, asked of the mixers in the schedule."""
    check_schedule(spec)
    kv: Dict[int, KVNeed] = {}
    states: Dict[int, StateNeed] = {}
    for e in spec.schedule:
        for mixer, cls in _mixers(spec, e.layer):
            need = cls.cache_need(mixer)
            if need is not None:
                if e.cache in kv and kv[e.cache] != need:
                    raise ModelError(f"cache {e.cache} is used with different needs: {kv[e.cache]} and {need}")
                kv[e.cache] = need
            st = cls.state_need(mixer)
            if st is not None:
                if e.cache in states and states[e.cache] != st:
                    raise ModelError(f"state {e.cache} is used with different needs")
                states[e.cache] = st
    return kv, states


def side_state_needs(spec: ModelSpec):
    """Per-request states beside the mixers' own, keyed by (cache id, owning description): what the short
    convolutions in front of sub-layers and behind projections keep of earlier steps.  Asked of every mixer class and
    arrangement class that has a static ``side_states`` (mixer: of its description; arrangement: of the layer's),
    which answers a list of (owner, StateNeed)."""
    out = {}
    for e in spec.schedule:
        layer = spec.layers[e.layer]
        asked = [(cls, m) for m, cls in _mixers(spec, e.layer)]
        asked.append((part_class("arrangement", _Arrangement(layer.arrangement)), layer))
        for cls, d in asked:
            for owner, need in (cls.side_states(d) if hasattr(cls, "side_states") else ()):
                key = (e.cache, owner)
                if key in out and out[key] != need:
                    raise ModelError(f"the state of {owner!r} under cache {e.cache} is used with different needs")
                out[key] = need
    return out


def _layer_tensor_names(layer) -> List[str]:
    names = []
    for sub in layer.sublayers:
        for kind, d in (("norm", sub.norm), (sub.category, sub.part), ("norm", sub.post_norm),
                        ("norm", getattr(sub, "sum_norm", None))):
            if d is not None:
                names += [t.name for t in part_class(kind, d).declare(d)]
    names += [t.name for t in _arrangement_tensors(layer)]
    return names


class Model:
    def __init__(self, spec: ModelSpec, weights: Dict[str, torch.Tensor], rt: Runtime, consume: bool = False):
        """``consume``: a layer's tensors are taken out of ``weights`` as soon as its parts are built (unless a later
        layer names them too), so that tensors which a part has fused into a new one are given back layer by layer
        instead of standing twice in memory until the whole model is built."""
        check_schedule(spec)
        self.spec = spec
        self.rt = rt
        self.embedding = weights[spec.embedding]
        self.position_table = weights[spec.position_table] if spec.position_table is not None else None
        if spec.streams is not None and spec.streams < 1:
            raise ModelError(f"a residual has at least one stream, got {spec.streams}")
        self.blocks = []
        last_use = {}
        if consume:
            for i, layer in enumerate(spec.layers):
                for name in _layer_tensor_names(layer):
                    last_use[name] = i
        for i, layer in enumerate(spec.layers):
            built = []
            for sub in layer.sublayers:
                _check_category(sub.category)
                # "no norm" is a part too: it is where the sub-layer before is added to the residual stream
                norm = part_class("norm", sub.norm)(sub.norm, weights, rt) if sub.norm is not None \
                    else NoNorm(None, weights, rt)
                post = part_class("norm", sub.post_norm)(sub.post_norm, weights, rt) \
                    if sub.post_norm is not None else None
                sum_norm = part_class("norm", sub.sum_norm)(sub.sum_norm, weights, rt) \
                    if getattr(sub, "sum_norm", None) is not None else None
                # a sub-layer without a part (an arrangement may allow it) is its norms alone
                part = part_class(sub.category, sub.part)(sub.part, weights, rt) if sub.part is not None else None
                built.append(BuiltSubLayer(sub.category, part, norm, post, sum_norm))
            arrangement = part_class("arrangement", _Arrangement(layer.arrangement))
            if getattr(arrangement, "needs_weights", False):
                self.blocks.append(arrangement(layer, built, weights, rt))
            else:
                self.blocks.append(arrangement(layer, built))
            if consume:
                for name in _layer_tensor_names(layer):
                    if last_use[name] == i and name not in (spec.embedding, spec.lm_head):
                        weights.pop(name, None)
        self.depth_planes = depth_planes(spec)
        if self.depth_planes:
            if spec.streams is not None or spec.position_table is not None or spec.embedding_norm is not None:
                raise ModelError("averages over depth start from the plain embedding on a residual of one stream")
        self.embedding_again = any(e.add_embedding for e in spec.schedule)
        self._takes_after = ["after" in inspect.signature(b.forward).parameters for b in self.blocks]
        self.embedding_norm = None
        if spec.embedding_norm is not None:
            if spec.streams is not None or getattr(spec.embedding_norm, "groups", 1) != 1:
                raise ModelError("a norm on the embedding is a plain RMS norm on a residual of one stream")
            self.embedding_norm = (weights[spec.embedding_norm.weight].to(torch.float32).contiguous(),
                                   float(spec.embedding_norm.eps))
        self.final_norm = part_class("norm", spec.final_norm)(spec.final_norm, weights, rt)
        head = weights.get(spec.lm_head)
        if head is None:
            if not spec.lm_head_optional:
                raise ModelError(f"tensor '{spec.lm_head}' is missing and the model does not tie its head")
            head = self.embedding  # the table stands in (qwen3.rs:366-373)
        self.tied = head is self.embedding
        self.head = Linear(head, rt)

    def forward(self, ctx) -> torch.Tensor:
        """Run the step's rows through all scheduled layers; float32 logits [wanted rows, vocab]."""
        n = ctx.token_ids.shape[0]
        scale = 1.0 if self.spec.embedding_scale is None else self.spec.embedding_scale
        pending = None
        if self.depth_planes:
            # the embedding is the first of the results that later layers look back on; the first norm reads it there
            planes = torch.empty((self.depth_planes, n, self.spec.width), dtype=torch.float32, device=self.rt.device)
            ctx.extra["depth_planes"] = planes
            residual = torch.empty((n, self.spec.width), dtype=torch.float32, device=self.rt.device)
            kernels.embedding_gather(self.embedding, ctx.token_ids, planes[0], self.rt.dtype, scale)
            pending = SandwichUpdate(None, source=planes[0])
        elif self.spec.streams is None and self.position_table is None:
            residual = torch.empty((n, self.spec.width), dtype=torch.float32, device=self.rt.device)
            again = torch.empty_like(residual) if self.embedding_again else None     # for the passes that add it again
            kernels.embedding_gather(self.embedding, ctx.token_ids, residual, self.rt.dtype, scale,
                                     **({} if again is None else {"copy": again}))
        else:
            # a residual of several streams [rows, streams, width], each the embedding (plus the position's vector)
            residual = torch.empty((n, self.spec.streams or 1, self.spec.width), dtype=torch.float32,
                                   device=self.rt.device)
            kernels.embedding_streams(self.embedding, ctx.token_ids, self.position_table, ctx.positions, residual,
                                      self.rt.dtype, scale)
            if self.spec.streams is None:
                residual = residual.view(n, self.spec.width)
        if self.embedding_norm is not None:
            kernels.scaled_add_norm(residual, None, 1.0, self.embedding_norm[0], self.embedding_norm[1], None,
                                    self.rt.dtype)
        schedule = self.spec.schedule
        for k, entry in enumerate(schedule):
            block = self.blocks[entry.layer]
            if entry.add_embedding:
                u = SumUpdate.of(pending)
                if u is None:
                    raise ModelError(f"schedule entry {k}: the embedding joins the stream beside a plain pending output")
                pending = SumUpdate(u.delta, u.bias, plus=again)
            # a block that wants to know what runs after it (to fold the norm between into the products around it)
            # is told; the last block's output goes to the last norm, which reads a choice of rows
            if k + 1 < len(schedule) and self._takes_after[entry.layer] and not schedule[k + 1].add_embedding:
                after = getattr(self.blocks[schedule[k + 1].layer], "entry", None)
                pending = block.forward(ctx, entry.cache, residual, pending, after=after() if after else None)
            else:
                pending = block.forward(ctx, entry.cache, residual, pending)
        if ctx.logit_rows.shape[0] == 0:
            return torch.empty((0, self.spec.vocab_size), dtype=torch.float32, device=self.rt.device)
        h = self.final_norm.add_norm(residual, pending, rows=ctx.logit_rows)
        logits = self.head(h, out_dtype=torch.float32)
        if self.spec.logit_scale is not None or self.spec.logit_softcap is not None:
            kernels.logit_scale_softcap(logits, 1.0 if self.spec.logit_scale is None else self.spec.logit_scale,
                                        self.spec.logit_softcap, self.rt.dtype)
        return logits


class _Arrangement:
    """The arrangement's name as a description with a ``kind``."""

    def __init__(self, kind: str):
        self.kind = kind
