"""How a layer's sub-layers and their norms are arranged around the residual stream."""
from __future__ import annotations

from typing import List, Optional

import torch

from .. import kernels
from ..cache.storage import StateNeed
from .basic import GatedUpdate, Linear, SandwichUpdate, StreamUpdate, SumUpdate, fuse_rows
from .registry import register_arrangement
from .spec import TensorDecl


class BuiltSubLayer:
    """A sub-layer whose parts are built: ``part`` with its ``category`` ("mixer" or "feed_forward"),
    the ``norm`` before it and the ``post_norm`` after it (either may be None)."""

    def __init__(self, category: str, part, norm=None, post_norm=None, sum_norm=None):
        self.category, self.part, self.norm, self.post_norm = category, part, norm, post_norm
        self.sum_norm = sum_norm     # the norm of the stream itself after this sub-layer (norm_after_sum blocks)

    def run(self, ctx, cache_id: int, h, sink=None):
        kw = {} if sink is None else {"sink": sink}
        y = self.part.forward(ctx, cache_id, h, **kw) if self.category == "mixer" else self.part.forward(ctx, h, **kw)
        return self.post_norm.norm(y) if self.post_norm is not None else y

    def run_part(self, ctx, cache_id: int, h):
        """The part alone, without the norm on its output."""
        return self.part.forward(ctx, cache_id, h) if self.category == "mixer" else self.part.forward(ctx, h)

    def takes_scaled_rows(self, n_rows: int) -> bool:
        """Whether this sub-layer can be handed scaled rows in place of its norm's output: the norm must be able to
        give a sink to the product before it, and the part must say that it reads scaled rows."""
        f = getattr(self.part, "takes_scaled_rows", None)
        plain_norm = hasattr(self.norm, "sink") and getattr(getattr(self.norm, "spec", None), "groups", 1) == 1
        return f is not None and plain_norm and bool(f(n_rows))

    def feeds_sink(self, n_rows: int) -> bool:
        f = getattr(self.part, "feeds_sink", None)
        return f is not None and self.post_norm is None and bool(f(n_rows))


class SequentialBlock:
    """For every sub-layer in turn: x += post_norm(part(norm(x))).  With two sub-layers, a mixer and a
    feed-forward with a norm each, this is the reference's decoder layer
    (inferrs-models/src/models/qwen3.rs:285-300).

    The residual stream ``x`` is float32 and is updated in place.  An addition is not done where
    the sub-layer ends but inside the norm kernel that follows it, so the block hands its last
    sub-layer's output on as ``pending`` and takes the previous block's in.
    """

    def __init__(self, spec, sublayers: List[BuiltSubLayer]):
        if not sublayers:
            raise ValueError("a layer needs at least one sub-layer")
        if any(s.norm is None for s in sublayers):
            # the output of the sub-layer before is added inside the norm kernel: "no norm" is a part too
            raise ValueError("every sub-layer of a sequential block needs a norm part (NoNorm where there is none)")
        self.spec = spec
        self.sublayers = list(sublayers)

    def parts(self):
        """Every part of the block (the runner asks each whether it is ``graph_safe``)."""
        for s in self.sublayers:
            yield s.part
            if s.norm is not None:
                yield s.norm
            if s.post_norm is not None:
                yield s.post_norm

    def entry(self) -> BuiltSubLayer:
        """The sub-layer that takes what the block before hands on."""
        return self.sublayers[0]

    def forward(self, ctx, cache_id: int, residual: torch.Tensor, pending, after: Optional[BuiltSubLayer] = None):
        """``after``: the sub-layer that runs after this block (the next block's entry), if the caller knows it.  Where
        a sub-layer's last product and the next sub-layer's first both fold norms at this step's number of rows,
        the addition to the residual stream and the norm between them run inside the two products: the producer gets
        the norm's sink and hands on scaled rows, which the norm passes through."""
        n_rows = residual.shape[0]
        for i, s in enumerate(self.sublayers):
            h = s.norm.add_norm(residual, pending)
            nxt = self.sublayers[i + 1] if i + 1 < len(self.sublayers) else after
            fold = nxt is not None and s.feeds_sink(n_rows) and nxt.takes_scaled_rows(n_rows)
            pending = s.run(ctx, cache_id, h, sink=nxt.norm.sink(residual) if fold else None)
        return pending


register_arrangement("sequential", SequentialBlock)


class InputConv:
    """What a sub-layer reads is replaced by itself plus its causal convolution over time, per channel (see
    :class:`~inferrs_b200.parts.spec.InputConvSpec`).  The sums are float32; the last taps - 1 inputs of every
    request are kept in its slot of the state that the description owns under the layer's cache id."""

    def __init__(self, spec, weights):
        if spec.taps < 1:
            raise ValueError(f"a convolution has at least one tap, got {spec.taps}")
        self.spec = spec
        self.weight = weights[spec.weight].to(torch.float32).t().contiguous()      # tap-major, as the kernel reads it

    @staticmethod
    def declare(spec) -> List[TensorDecl]:
        return [TensorDecl(spec.weight, (spec.width, spec.taps), init="uniform:0:0.3")]

    @staticmethod
    def state_need(spec) -> Optional[StateNeed]:
        return StateNeed(shape=((spec.taps - 1) * spec.width,)) if spec.taps > 1 else None

    def single_rows(self, ctx, cache_id: int):
        """What a norm kernel needs to apply this convolution itself in a step in which every request brings one row."""
        s = self.spec
        return (self.weight, ctx.storage.side_state(cache_id, s) if s.taps > 1 else None, 0, ctx.slots, ctx.row_request)

    def __call__(self, ctx, cache_id: int, h: torch.Tensor) -> torch.Tensor:
        s = self.spec
        state = ctx.storage.side_state(cache_id, s) if s.taps > 1 else None
        out = torch.empty_like(h)
        single = ctx.max_q_len == 1          # every request brings one row: the kernel moves the kept rows on itself
        kernels.causal_conv_rows(h, 0, self.weight, state, 0, ctx.q_start, ctx.slots, ctx.row_request, out, True,
                                 shift_single=single)
        if state is not None and not single:
            kernels.conv_state_shift(h, 0, s.width, s.taps, state, 0, ctx.q_start, ctx.slots, ctx.n_requests)
        return out


class HyperConnectionBlock:
    """A block on a residual that is several streams wide, x_1 .. x_S [rows, S, width] in float32.  Every sub-layer has
    a :class:`~inferrs_b200.parts.spec.StreamConnectionSpec`: it reads u = sum_s read[s] x_s through its norm, and
    its output y comes back as x_t <- sum_s mix[s, t] x_s + gain[t] y, all streams at once from the old ones.  A
    sub-layer with an ``input_conv`` reads norm(u) plus its short convolution over time.

    As in :class:`SequentialBlock` the output is not brought in where the sub-layer ends: the norm kernel that
    follows does the update, the read and the norm in one pass over the streams, so the block hands its last
    sub-layer's output on as a pending :class:`~inferrs_b200.parts.basic.StreamUpdate`.
    """

    needs_weights = True     # the model hands the arrangement the weights too: the connections' tensors

    @staticmethod
    def declare(spec) -> List[TensorDecl]:
        out = []
        for s in spec.sublayers:
            c = s.connection
            if c is None:
                raise ValueError("every sub-layer of a hyper-connection block needs a connection")
            out += [TensorDecl(c.read, (c.streams,), init=f"uniform:{1.0 / c.streams}:0.1"),
                    TensorDecl(c.gain, (c.streams,), init="uniform:1:0.2"),
                    TensorDecl(c.mix, (c.streams, c.streams), init="identity:0.1")]
            if s.input_conv is not None:
                out += InputConv.declare(s.input_conv)
        return out

    @staticmethod
    def side_states(spec):
        """The inputs that the sub-layers' convolutions keep, each under its own description."""
        needs = [(s.input_conv, InputConv.state_need(s.input_conv)) for s in spec.sublayers if s.input_conv is not None]
        return [(owner, need) for owner, need in needs if need is not None]

    def __init__(self, spec, sublayers: List[BuiltSubLayer], weights=None, rt=None):
        if not sublayers:
            raise ValueError("a layer needs at least one sub-layer")
        if weights is None:
            raise ValueError("a hyper-connection block needs the weights of its connections")
        self.spec = spec
        self.sublayers = list(sublayers)
        self.connections = []
        for s, built in zip(spec.sublayers, sublayers):
            c = s.connection
            if c is None or not hasattr(built.norm, "add_norm") or built.post_norm is not None:
                raise ValueError("a sub-layer of a hyper-connection block has a connection, a norm before it and none "
                                 "after it")
            self.connections.append(tuple(weights[name].to(torch.float32).contiguous() for name in (c.read, c.gain, c.mix)))
        self.streams = spec.sublayers[0].connection.streams
        if any(s.connection.streams != self.streams for s in spec.sublayers):
            raise ValueError("the sub-layers of a block hang on the same number of streams")
        self.convs = [InputConv(s.input_conv, weights) if s.input_conv is not None else None for s in spec.sublayers]

    def parts(self):
        for s in self.sublayers:
            if s.part is not None:
                yield s.part
            yield s.norm

    def forward(self, ctx, cache_id: int, residual: torch.Tensor, pending):
        if residual.dim() != 3 or residual.shape[1] != self.streams:
            raise ValueError(f"a hyper-connection block of {self.streams} streams got a residual of shape "
                             f"{tuple(residual.shape)}")
        for s, (read, gain, mix), conv in zip(self.sublayers, self.connections, self.convs):
            if s.part is None:       # a sub-layer without a part: its tensors are read and nothing runs
                continue
            h = s.norm.add_norm(residual, pending, read=read)
            if conv is not None:
                h = conv(ctx, cache_id, h)
            pending = StreamUpdate(s.run(ctx, cache_id, h), mix, gain)
        return pending


register_arrangement("hyper_connections", HyperConnectionBlock)


class StreamCopy:
    """What a block that norms after the sum hands on in place of a pending output: nothing is left to add, and
    ``rows`` holds the stream as it stands, in the activation dtype, for whoever reads the stream itself next."""

    def __init__(self, rows: torch.Tensor):
        self.rows = rows


class NormAfterSumBlock:
    """For every sub-layer in turn: x <- norm(scale * x + part(x)), with ``scale`` the layer's ``residual_scale``
    and ``norm`` the sub-layer's ``sum_norm``.  The parts read the stream itself, and the stream itself is
    normalised: float32, in place, by one kernel that also writes the copy in the activation dtype that the next
    part reads.  A sub-layer without a part contributes nothing to its sum.

    The block hands on a :class:`StreamCopy` (the next block of this kind reads it instead of casting the stream
    again); a pending output from a block of another kind is added first.
    """

    def __init__(self, spec, sublayers: List[BuiltSubLayer]):
        if not sublayers:
            raise ValueError("a layer needs at least one sub-layer")
        for s in sublayers:
            if s.sum_norm is None or s.post_norm is not None or not isinstance(s.norm, _no_norm()):
                raise ValueError("a sub-layer of a block that norms after the sum has a sum_norm and no other norm")
            if getattr(s.sum_norm.spec, "groups", 1) != 1:
                raise ValueError("the norm after the sum is a plain RMS norm (no groups)")
        self.spec = spec
        self.sublayers = list(sublayers)
        self.scale = float(spec.residual_scale)
        # norm weights as float32, once
        self.weights = [s.sum_norm.weight.to(torch.float32).contiguous() for s in sublayers]

    def parts(self):
        for s in self.sublayers:
            if s.part is not None:
                yield s.part
            yield s.sum_norm

    def forward(self, ctx, cache_id: int, residual: torch.Tensor, pending):
        if residual.dim() != 2:
            raise ValueError("a block that norms after the sum runs on the plain residual [rows, width]")
        rt_dtype = self.sublayers[0].sum_norm.rt.dtype
        if isinstance(pending, StreamCopy):
            h = pending.rows
        else:
            h = self.sublayers[0].norm.add_norm(residual, pending)      # adds what is pending; the stream as act rows
        for s, w in zip(self.sublayers, self.weights):
            y = s.run(ctx, cache_id, h) if s.part is not None else None
            h = torch.empty(residual.shape, dtype=rt_dtype, device=residual.device)
            kernels.scaled_add_norm(residual, y, self.scale, w, s.sum_norm.spec.eps, h, rt_dtype)
        return StreamCopy(h)


def _no_norm():
    from .basic import NoNorm
    return NoNorm


register_arrangement("norm_after_sum", NormAfterSumBlock)


class GatedResidualBlock:
    """For every sub-layer in turn: h = norm(x), x += sigmoid(W h + b) * part(h), with W and b from the sub-layer's
    :class:`~inferrs_b200.parts.spec.ResidualGateSpec`.  The gate reads the same normalised rows as the part.  A
    sub-layer without a part adds nothing: its norm's and gate's tensors are read and not used.

    As in :class:`SequentialBlock` nothing is added where the sub-layer ends: the block hands its last sub-layer's
    output on with the gate's pre-activations as a pending :class:`~inferrs_b200.parts.basic.GatedUpdate`, and the norm
    kernel that follows does sigmoid, product, addition to the float32 stream and norm in one pass.
    """

    needs_weights = True     # the model hands the arrangement the weights too: the gates' tensors

    @staticmethod
    def declare(spec) -> List[TensorDecl]:
        out = []
        for s in spec.sublayers:
            c = s.connection
            if c is None or not hasattr(c, "weight") or not hasattr(c, "bias"):
                raise ValueError("every sub-layer of a gated-residual block needs a residual gate")
            width = _width_of(s)
            out += [TensorDecl(c.weight, (width, width)), TensorDecl(c.bias, (width,), init="uniform:0:0.5")]
        return out

    def __init__(self, spec, sublayers: List[BuiltSubLayer], weights=None, rt=None):
        if not sublayers:
            raise ValueError("a layer needs at least one sub-layer")
        if weights is None or rt is None:
            raise ValueError("a gated-residual block needs the weights of its gates")
        self.spec = spec
        self.sublayers = list(sublayers)
        self.gates = []
        for s, built in zip(spec.sublayers, sublayers):
            if s.connection is None or built.post_norm is not None or not hasattr(built.norm, "add_norm"):
                raise ValueError("a sub-layer of a gated-residual block has a gate, a norm before it and none after it")
            self.gates.append((Linear(weights[s.connection.weight], rt),
                               weights[s.connection.bias].to(torch.float32).contiguous()))

    def parts(self):
        for s in self.sublayers:
            if s.part is not None:
                yield s.part
            yield s.norm

    def forward(self, ctx, cache_id: int, residual: torch.Tensor, pending):
        if residual.dim() != 2:
            raise ValueError("a gated-residual block runs on the plain residual [rows, width]")
        for s, (gate, bias) in zip(self.sublayers, self.gates):
            if s.part is None:
                continue
            h = s.norm.add_norm(residual, pending)
            y = s.run(ctx, cache_id, h)
            pending = GatedUpdate(y, gate(h), bias)
        return pending


def _width_of(sub) -> int:
    """The stream's width as a sub-layer's descriptions give it."""
    for d in (sub.norm, sub.part):
        for name in ("size", "width"):
            if d is not None and hasattr(d, name):
                return int(getattr(d, name))
    raise ValueError("a sub-layer of a gated-residual block needs a norm or a part that says how wide the stream is")


register_arrangement("gated_residual", GatedResidualBlock)


class SandwichBlock:
    """For every sub-layer in turn: h = norm(x), h += conv(h) (where it has an ``input_conv``), x += layer_scale *
    post_norm(part(h)); with a ``depth_average`` the block hands on the weighted sum of the embedding and all layers'
    results so far instead of its own result.  A sub-layer without a norm on its output adds it as it is.

    As in :class:`SequentialBlock` nothing is added where a sub-layer ends: its raw output is handed on as a pending
    :class:`~inferrs_b200.parts.basic.SandwichUpdate`, and the kernel of the norm that follows does the output's norm and
    scale, the addition to the float32 stream, the average over depth and the norm in one pass (in steps of single rows
    the next sub-layer's convolution too).  The results of earlier layers stand in the step's planes
    (:func:`depth_planes`), float32.
    """

    needs_weights = True     # the model hands the arrangement the weights too: scales, averages and convolutions

    @staticmethod
    def declare(spec) -> List[TensorDecl]:
        out = []
        for s in spec.sublayers:
            if s.layer_scale is not None:
                out.append(TensorDecl(s.layer_scale, (_width_of(s),), init="uniform:1:0.3"))
            if s.input_conv is not None:
                out += InputConv.declare(s.input_conv)
        if spec.depth_average is not None:
            n = spec.depth_average.results
            out.append(TensorDecl(spec.depth_average.weight, (n,), init=f"uniform:{1.0 / n}:{0.5 / n}"))
        return out + [TensorDecl(name, shape) for name, shape in spec.unused]

    @staticmethod
    def side_states(spec):
        """The inputs that the sub-layers' convolutions keep, each under its own description."""
        needs = [(s.input_conv, InputConv.state_need(s.input_conv)) for s in spec.sublayers if s.input_conv is not None]
        return [(owner, need) for owner, need in needs if need is not None]

    def __init__(self, spec, sublayers: List[BuiltSubLayer], weights=None, rt=None):
        if not sublayers:
            raise ValueError("a layer needs at least one sub-layer")
        if weights is None:
            raise ValueError("a sandwich block needs the weights of its scales")
        self.spec = spec
        self.sublayers = list(sublayers)
        self.posts, self.convs = [], []
        for s, built in zip(spec.sublayers, sublayers):
            if built.norm is None or not hasattr(built.norm, "add_norm") or built.sum_norm is not None:
                raise ValueError("a sub-layer of a sandwich block has a norm before it")
            # the norm's weight and the scale behind it are one vector, in float32
            post, eps = None, 0.0
            if built.post_norm is not None:
                if getattr(built.post_norm.spec, "kind", None) != "rms" or getattr(built.post_norm.spec, "groups", 1) != 1:
                    raise ValueError("the norm on a sub-layer's output is a plain RMS norm")
                post, eps = built.post_norm.weight.to(torch.float32), float(built.post_norm.spec.eps)
                if s.layer_scale is not None:
                    post = post * weights[s.layer_scale].to(torch.float32)
                post = post.contiguous()
            elif s.layer_scale is not None:
                raise ValueError("a sub-layer's scale stands behind a norm on its output")
            self.posts.append((post, eps))
            self.convs.append(InputConv(s.input_conv, weights) if s.input_conv is not None else None)
        self.average = None
        if spec.depth_average is not None:
            self.average = weights[spec.depth_average.weight].to(torch.float32).contiguous()
            if spec.depth_average.results < 2:
                raise ValueError("an average over depth has the embedding and this layer's result at least")

    def parts(self):
        for s in self.sublayers:
            yield s.part
            yield s.norm
            if s.post_norm is not None:
                yield s.post_norm

    def forward(self, ctx, cache_id: int, residual: torch.Tensor, pending):
        if residual.dim() != 2:
            raise ValueError("a sandwich block runs on the plain residual [rows, width]")
        for s, (post, eps), conv in zip(self.sublayers, self.posts, self.convs):
            if conv is not None and ctx.max_q_len == 1:
                h = s.norm.add_norm(residual, pending, conv=conv.single_rows(ctx, cache_id))
            else:
                h = s.norm.add_norm(residual, pending)
                if conv is not None:
                    h = conv(ctx, cache_id, h)
            pending = SandwichUpdate(s.run_part(ctx, cache_id, h), post, eps)
        if self.average is not None:
            planes, n = ctx.extra["depth_planes"], self.spec.depth_average.results - 1
            pending.average = (planes[:n], self.average)
            pending.result = planes[n] if n < planes.shape[0] else None      # the last result is read by nobody else
        return pending


def depth_planes(spec) -> int:
    """How many results of earlier layers (the embedding among them) a model's averages over depth look back on."""
    return max([layer.depth_average.results - 1 for layer in spec.layers if layer.depth_average is not None], default=0)


register_arrangement("sandwich", SandwichBlock)


class ParallelBlock:
    """h = norm(x), x += the sum of part(h) over all sub-layers: there is one norm, the first sub-layer's, and every
    sub-layer reads its output.

    Where all parts let their products be joined (``joins_products``), the block has two: one makes every part's
    projections of h side by side, each part turns its columns into its columns of one wide row (``middle``), and the
    second product takes that row to the sum of the parts' outputs, because [A | B] [a; b] = A a + B b; the addition of
    the sub-layers is part of its float32 accumulation.  A part that routes rows (``router_beside_norm``) has its choice made
    by the norm's kernel where that is better.  Parts that do not join run one after the other, and their outputs are
    added.

    As in :class:`SequentialBlock` nothing is added to the stream where the block ends: its output is handed on (with the
    joined products' bias as a :class:`~inferrs_b200.parts.basic.SumUpdate`)."""

    PAD_ROWS = 64        # the joined projection's rows are filled up to a multiple of this

    def __init__(self, spec, sublayers: List[BuiltSubLayer]):
        if not sublayers:
            raise ValueError("a layer needs at least one sub-layer")
        if isinstance(sublayers[0].norm, _no_norm()) or not hasattr(sublayers[0].norm, "add_norm") \
                or any(not isinstance(s.norm, _no_norm()) for s in sublayers[1:]) \
                or any(s.post_norm is not None or s.sum_norm is not None or s.part is None for s in sublayers):
            raise ValueError("the sub-layers of a parallel block have one norm, before the first of them")
        self.spec = spec
        self.sublayers = list(sublayers)
        self.norm = sublayers[0].norm
        self.routed = [s.part for s in sublayers if hasattr(s.part, "router_beside_norm")]
        self.joined = all(getattr(s.part, "joins_products", lambda: False)() for s in sublayers)
        if self.joined:
            self._join(self.norm.rt)

    def _join(self, rt):
        ins, outs, biases = zip(*[s.part.hand_over_products() for s in self.sublayers])
        self.in_cols = _columns([w.shape[0] for w in ins])
        self.mid_cols = _columns([w.shape[1] for w in outs])
        n_in = self.in_cols[-1][1]
        pad = -n_in % self.PAD_ROWS
        fill = [torch.zeros((pad, ins[0].shape[1]), dtype=ins[0].dtype, device=ins[0].device)] if pad else []
        self.in_product = Linear(fuse_rows(list(ins) + fill), rt)
        if len({w.dtype for w in outs}) > 1:
            outs = [w.to(torch.float32) for w in outs]
        self.out_product = Linear(torch.cat(list(outs), dim=1).contiguous(), rt)
        biases = [b.to(torch.float32) for b in biases if b is not None]
        self.bias = sum(biases[1:], biases[0]).contiguous() if biases else None

    def parts(self):
        yield self.norm
        for s in self.sublayers:
            yield s.part

    def forward(self, ctx, cache_id: int, residual: torch.Tensor, pending):
        if residual.dim() != 2:
            raise ValueError("a parallel block runs on the plain residual [rows, width]")
        n = residual.shape[0]
        router = self.routed[0].router_beside_norm(n) if len(self.routed) == 1 and self.joined \
            and getattr(self.norm, "routes_rows", False) and SumUpdate.of(pending) is not None else None
        shares = None
        if router is not None:
            h, shares = self.norm.add_norm(residual, pending, router=router)
        else:
            h = self.norm.add_norm(residual, pending)
        if not self.joined:
            total = None
            for s in self.sublayers:
                y = s.run_part(ctx, cache_id, h)
                if total is None:
                    total = y
                else:
                    before, total = total, torch.empty_like(y)
                    kernels.scaled_sum(before, 1.0, y, 1.0, total)
            return total
        proj = self.in_product(h)
        mid = torch.empty((n, self.mid_cols[-1][1]), dtype=proj.dtype, device=proj.device)
        for s, (c0, c1), (m0, m1) in zip(self.sublayers, self.in_cols, self.mid_cols):
            s.part.middle(ctx, cache_id, h, proj[:, c0:c1], mid[:, m0:m1], shares=shares if s.part in self.routed else None)
        y = self.out_product(mid)
        return y if self.bias is None else SumUpdate(y, self.bias)


def _columns(sizes):
    """(first, one past the last) of consecutive runs of these sizes."""
    out, at = [], 0
    for n in sizes:
        out.append((at, at + n))
        at += n
    return out


register_arrangement("parallel", ParallelBlock)
