"""Arrangements of norms, mixer and feed-forward inside a layer."""

from __future__ import annotations

import torch

from pagedserve_b200.cache.manager import StateNeed
from pagedserve_b200.parts.base import Block, register_part
from pagedserve_b200.parts.parallel import padded, state_share
from pagedserve_b200.weights.loader import ParamSpec


@register_part("block", "pre_norm")
class PreNormBlock(Block):
    """h += mixer(norm(h)); h += feed_forward(norm(h))
    (reference: src/model/paged_decoder.py:181-189, 210-228).  The residual stream ``h``
    is float32 and is updated in place; the adds happen in the epilogues of the
    mixer's and the feed-forward's last matrix products.  A layer whose feed-forward is the ``none`` part has
    the first sublayer only, and no second norm."""

    graph_safe = True

    @property
    def required_norms(self):
        if getattr(self.feed_forward, "is_empty", False):
            return ("pre_mixer",)
        return ("pre_mixer", "pre_feed_forward")

    @staticmethod
    def _normed(norm, consumer, hidden):
        # a consumer whose first operation is a matrix product may take the norm unevaluated
        if getattr(consumer, "accepts_deferred_norm", False) and hasattr(norm, "defer"):
            return norm.defer(hidden)
        return norm.forward(hidden)

    def forward(self, hidden, ctx, layer):
        self.mixer.forward(self._normed(self.norms["pre_mixer"], self.mixer, hidden), hidden, ctx, layer)
        if getattr(self.feed_forward, "is_empty", False):
            return
        self.feed_forward.forward(self._normed(self.norms["pre_feed_forward"], self.feed_forward, hidden),
                                  hidden, ctx)


@register_part("block", "parallel_pre_norm")
class ParallelPreNormBlock(Block):
    """x <- x + s1 * mixer(norm1(x)) + s2 * feed_forward(norm2(x)), both of the same x: two RMS norms (``pre_mixer``,
    ``pre_feed_forward``) with gains of their own, ``s1`` and ``s2`` a factor per coordinate (``scales``: the tensors'
    names; absent: 1).  A layer whose feed-forward is the ``none`` part has the mixer only, and no second norm.

    One kernel norms the row for both; after it x may change, so both results are added into x where they are made, times
    their factors, by the epilogues of the mixer's and the feed-forward's last products (``Part.set_result_factor``).  The
    residual rows, norms and sums are float32.

    params: scales = dict(mixer, feed_forward) or None, init_std."""

    graph_safe = True

    def __init__(self, params, prefix, env, mixer, feed_forward, norms):
        super().__init__(params, prefix, env, mixer, feed_forward, norms)
        self.alone = getattr(feed_forward, "is_empty", False)
        for norm in norms.values():
            if norm.params.get("has_mean", True) or norm.params.get("has_bias", True):
                raise ValueError("parallel_pre_norm: the norms are RMS norms without a bias")
        if not self.alone and norms["pre_mixer"].params["eps"] != norms["pre_feed_forward"].params["eps"]:
            raise ValueError("parallel_pre_norm: both norms have one eps")

    @property
    def required_norms(self):
        return ("pre_mixer",) if self.alone else ("pre_mixer", "pre_feed_forward")

    def _scaled(self):
        scales = self.params.get("scales") or {}
        return [(scales[role], part) for role, part in (("mixer", self.mixer), ("feed_forward", self.feed_forward))
                if role in scales and not (role == "feed_forward" and self.alone)]

    def param_specs(self):
        width = self.norms["pre_mixer"].params["width"]
        return [(ParamSpec(self._n(name), (width,), "vector"), ("ones_plus_normal", self.params.get("init_std", 0.1)))
                for name, _ in self._scaled()]

    def bind(self, tensors):
        for name, part in self._scaled():
            part.set_result_factor(tensors[self._n(name)].contiguous())

    def forward(self, hidden, ctx, layer):
        ops = self.env.ops
        norm = self.norms["pre_mixer"]
        if self.alone:
            deferred = getattr(self.mixer, "accepts_deferred_norm", False)
            self.mixer.forward(norm.defer(hidden) if deferred else norm.forward(hidden), hidden, ctx, layer)
            return
        second = self.norms["pre_feed_forward"]
        h1 = ops.empty(hidden.shape, self.env.dtype, hidden.device)
        h2 = ops.empty(hidden.shape, self.env.dtype, hidden.device)
        ops.rms_norm_pair(hidden, norm.weight, second.weight, float(norm.params["eps"]), h1, h2)
        self.mixer.forward(h1, hidden, ctx, layer)
        self.feed_forward.forward(h2, hidden, ctx)


class StreamCarrier:
    """What runs through the layers of a model with several residual streams: the streams ``[S, T, W]``, the
    row ``u`` that the open sublayer reads, the row ``y`` it adds its result into, and the (mix, out) weights of
    a sublayer that has run but whose update of the streams is still to be done."""

    def __init__(self, streams, u, y):
        self.streams = streams
        self.u = u
        self.y = y
        self.pending = None


@register_part("block", "hyper_pre_norm")
class HyperPreNormBlock(Block):
    """A pre-norm layer over S residual streams x_1 .. x_S instead of one (all equal to the embedded rows at the
    start, summed at the end).  For each sublayer f (the mixer, then the feed-forward if the layer has one) with
    its own weights in[S], out[S], mix[S, S]:

        u = sum_s in[s] x_s;   y = f(norm(u));   x_t <- sum_s mix[s, t] x_s + out[t] y   (all t from the old x)

    Everything is float32.  The update of one sublayer and the read of the next are one pass over the streams
    (``ops.hyper_step``): a sublayer leaves its update pending and whatever comes next (the feed-forward, the
    next layer, the end of the model) does it together with its own read.  The sublayer adds its result into a
    zeroed row, exactly as it would into the residual row of a plain layer, so every mixer and feed-forward
    works here unchanged.

    params: streams, names (a dict: mixer -> prefix of its three tensors, feed_forward -> likewise), init_std;
    tensors are ``<prefix>.in``, ``<prefix>.out``, ``<prefix>.mix``."""

    graph_safe = True

    def _sublayers(self):
        names = self.params["names"]
        if getattr(self.feed_forward, "is_empty", False):
            return [names["mixer"]]
        return [names["mixer"], names["feed_forward"]]

    @property
    def required_norms(self):
        if getattr(self.feed_forward, "is_empty", False):
            return ("pre_mixer",)
        return ("pre_mixer", "pre_feed_forward")

    def param_specs(self):
        S = self.params["streams"]
        if not (isinstance(S, int) and 0 < S <= 8):
            raise ValueError("hyper_pre_norm: between 1 and 8 streams")
        std = self.params.get("init_std", 0.1)
        specs = []
        for name in self._sublayers():
            specs += [(ParamSpec(self._n(name + ".in"), (S,), "vector"), ("ones_plus_normal", std)),
                      (ParamSpec(self._n(name + ".out"), (S,), "vector"), ("ones_plus_normal", std)),
                      (ParamSpec(self._n(name + ".mix"), (S, S), "vector"), ("eye_plus_normal", std))]
        return specs

    def bind(self, tensors):
        self.weights = [tuple(tensors[self._n(f"{name}.{which}")].contiguous() for which in ("in", "out", "mix"))
                        for name in self._sublayers()]

    def begin(self, hidden, ctx):
        ops, S = self.env.ops, self.params["streams"]
        streams = ops.empty((S,) + tuple(hidden.shape), torch.float32, hidden.device)
        u = ops.empty(hidden.shape, torch.float32, hidden.device)
        y = ops.empty(hidden.shape, torch.float32, hidden.device)
        ops.hyper_begin(hidden, self.weights[0][0], streams, u, y)
        return StreamCarrier(streams, u, y)

    def _open(self, carrier, w_in):
        """Make ``carrier.u`` the input of the sublayer whose read weights are ``w_in`` (None: the plain sum)."""
        if carrier.pending is None:
            return                                 # ``begin`` of this very block has done it
        w_out, mix = carrier.pending
        self.env.ops.hyper_step(carrier.streams, carrier.y, mix, w_out, w_in, carrier.u)
        carrier.pending = None

    @staticmethod
    def _normed(norm, consumer, rows):
        if getattr(consumer, "accepts_deferred_norm", False) and hasattr(norm, "defer"):
            return norm.defer(rows)
        return norm.forward(rows)

    def forward(self, hidden, ctx, layer):
        carrier = hidden
        w_in, w_out, mix = self.weights[0]
        self._open(carrier, w_in)
        self.mixer.forward(self._normed(self.norms["pre_mixer"], self.mixer, carrier.u), carrier.y, ctx, layer)
        carrier.pending = (w_out, mix)
        if len(self.weights) > 1:
            w_in, w_out, mix = self.weights[1]
            self._open(carrier, w_in)
            self.feed_forward.forward(self._normed(self.norms["pre_feed_forward"], self.feed_forward, carrier.u),
                                      carrier.y, ctx)
            carrier.pending = (w_out, mix)

    def end(self, carrier, ctx):
        self._open(carrier, None)
        return carrier.u


class ResidualCarrier:
    """What runs through the layers of a model that norms its sublayers' results: the float32 rows ``x``, the same
    rows in the compute type (``x_cast``: what the sublayers' products read; ``x`` itself in a float32 engine), the
    zeroed float32 rows ``y`` a sublayer adds its result into, and, where the layers end with an average over
    depth, ``history`` [entries, T, W]: the embedded rows and every layer's result so far."""

    def __init__(self, x, x_cast, y, history):
        self.x = x
        self.x_cast = x_cast
        self.y = y
        self.history = history


@register_part("block", "post_norm")
class PostNormBlock(Block):
    """x <- x + norm(mixer(x)); x <- x + norm(feed_forward(x)): the sublayers read the rows themselves and the norm
    (``post_mixer``, ``post_feed_forward``: :class:`GroupRMSNorm`) is applied to what they return.  The residual rows
    and the sums are float32.  A layer whose feed-forward is the ``none`` part has the first half only.

    ``depth`` = dict(index, name, entries): the layer ends with an average over depth.  With X_0 the embedded rows and
    X_(i+1) this layer's result (``index`` = i), what goes on to the next layer (and, behind the last, to the
    model's norm) is sum_(j <= i+1) w[j] X_j with w the tensor ``name`` of i + 2 numbers; ``entries`` is the number
    of layer runs of the model plus one (the rows the history holds).

    A sublayer adds its result into a zeroed row exactly as it would into the residual row of a pre-norm layer, so
    every mixer and feed-forward works here unchanged; one kernel then norms that row, adds it, clears it, stores and
    averages over depth where the layer ends, and leaves the new rows in the compute type for the next product."""

    graph_safe = True

    @property
    def required_norms(self):
        if getattr(self.feed_forward, "is_empty", False):
            return ("post_mixer",)
        return ("post_mixer", "post_feed_forward")

    def param_specs(self):
        depth = self.params.get("depth")
        if not depth:
            return []
        if not (0 <= depth["index"] < depth["entries"] - 1):
            raise ValueError("post_norm: a layer's index lies below the number of history entries")
        return [(ParamSpec(self._n(depth["name"]), (depth["index"] + 2,), "vector"),
                 ("share_plus_normal", depth.get("init_std", 0.2)))]

    def bind(self, tensors):
        depth = self.params.get("depth")
        self.depth_weight = tensors[self._n(depth["name"])].contiguous() if depth else None

    def begin(self, hidden, ctx):
        ops, depth = self.env.ops, self.params.get("depth")
        history = ops.empty((depth["entries"],) + tuple(hidden.shape), torch.float32, hidden.device) if depth else None
        x_cast = hidden if self.env.dtype == torch.float32 else ops.empty(hidden.shape, self.env.dtype, hidden.device)
        y = ops.empty(hidden.shape, torch.float32, hidden.device)
        ops.depth_begin(hidden, history[0] if depth else None, None if x_cast is hidden else x_cast, y)
        return ResidualCarrier(hidden, x_cast, y, history)

    def _close(self, carrier, norm, ends_layer):
        depth = self.params.get("depth") if ends_layer else None
        x_cast = None if carrier.x_cast is carrier.x else carrier.x_cast
        if depth:
            norm.add_into(carrier.y, carrier.x, x_cast, carrier.history, depth["index"] + 2, self.depth_weight)
        else:
            norm.add_into(carrier.y, carrier.x, x_cast)

    def forward(self, hidden, ctx, layer):
        carrier = hidden
        alone = getattr(self.feed_forward, "is_empty", False)
        self.mixer.forward(carrier.x_cast, carrier.y, ctx, layer)
        self._close(carrier, self.norms["post_mixer"], alone)
        if not alone:
            self.feed_forward.forward(carrier.x_cast, carrier.y, ctx)
            self._close(carrier, self.norms["post_feed_forward"], True)

    def end(self, carrier, ctx):
        return carrier.x


class SandwichCarrier:
    """What runs through the layers of a model that norms what its sublayers read and what they return: the float32 rows
    ``x``, the float32 rows ``y`` a sublayer adds its result into, ``inverse`` [T] (room for one over the root mean
    square of every row of ``x``, which a layer's first norm needs), and what the last sublayer has left to do:
    ``pending`` = (gain of its norm or None, factor on its result, eps)."""

    def __init__(self, x, y, inverse, pending):
        self.x = x
        self.y = y
        self.inverse = inverse
        self.pending = pending


@register_part("block", "sandwich_norm")
class SandwichNormBlock(Block):
    """x <- x + s1 * post(mixer(c(pre(x)))); x <- x + s2 * post(feed_forward(pre(x))): norms before and after each
    sublayer (four RMS norms without a mean; gains of one number or of the row's width), ``s1`` and ``s2`` a factor per
    coordinate (``scales``: the tensors' names), and, with ``conv`` = dict(taps, name), c(h)_t = h_t + sum over d < taps of
    w[:, taps - 1 - d] h_(t-d), channel by channel, rows before position 0 taken as zero; w [W, taps].  A layer whose
    feed-forward is the ``none`` part has the first sublayer only.  The residual rows, norms, sums and the convolution are
    float32; a sublayer reads rows of the compute type.

    A request keeps, in every layer, the last taps - 1 rows that the convolution read (float32, divided by their root
    mean square, without the gain, which is folded into the taps) in front of the mixer's own state.

    A sublayer adds its result into a zeroed row exactly as it would into the residual row of a pre-norm layer, so every
    mixer and feed-forward works here unchanged.  One kernel (``ops.sandwich_close``) then norms that row, adds it, clears
    it, and prepares what comes next.  Behind the mixer that is the feed-forward's normed rows.  Behind a layer it is left
    pending for the next one: in a step of single tokens the same kernel goes on with that layer's convolution, else it
    forms the root mean square that the convolution's kernel applies when it reads the rows.

    params: scales = dict(mixer, feed_forward), conv (None), init_std."""

    graph_safe = True
    takes_output_scale = True

    @property
    def required_norms(self):
        if getattr(self.feed_forward, "is_empty", False):
            return ("pre_mixer", "post_mixer")
        return ("pre_mixer", "post_mixer", "pre_feed_forward", "post_feed_forward")

    def __init__(self, params, prefix, env, mixer, feed_forward, norms):
        super().__init__(params, prefix, env, mixer, feed_forward, norms)
        conv = self.params.get("conv")
        if conv is not None and not (isinstance(conv["taps"], int) and 1 <= conv["taps"] <= 16):
            raise ValueError("sandwich_norm: a convolution has 1 to 16 taps")
        for norm in norms.values():
            if norm.params.get("has_mean", True) or norm.params.get("has_bias", True):
                raise ValueError("sandwich_norm: the norms are RMS norms without a bias")
        self.width = norms["pre_mixer"].params["width"]
        self.taps = conv["taps"] if conv is not None else 1
        self.kept = (self.taps - 1) * self.width

    def state_need(self):
        own, need = self.kept, self.mixer.state_need()
        if need is None:
            return StateNeed((own,), "float32") if own else None
        if not own:
            return need
        if need.dtype != "float32" or len(need.shape) != 1:
            raise ValueError("sandwich_norm: a mixer's state is rows of float32 numbers")
        return StateNeed((padded(own) + need.shape[0],), "float32")

    def param_specs(self):
        p, std = self.params, self.params.get("init_std", 0.1)
        names = [p["scales"]["mixer"]]
        if not getattr(self.feed_forward, "is_empty", False):
            names.append(p["scales"]["feed_forward"])
        specs = [(ParamSpec(self._n(name), (self.width,), "vector"), ("ones_plus_normal", std)) for name in names]
        if p.get("conv"):
            specs.append((ParamSpec(self._n(p["conv"]["name"]), (self.width, self.taps), "vector"),
                          ("normal", 0.5 * self.taps ** -0.5)))
        return specs

    def bind(self, tensors):
        # (the blocks are bound before their norms: the products with the norms' gains are formed when first needed)
        p = self.params
        self._tensors = {role: tensors[self._n(name)] for role, name in p["scales"].items()
                         if self._n(name) in tensors}
        self._taps = tensors[self._n(p["conv"]["name"])] if p.get("conv") else None
        self._gains = None

    def _folded(self):
        """(gain behind the mixer, gain behind the feed-forward, taps of the rows divided by their root mean square)."""
        if self._gains is None:
            norms, scales = self.norms, self._tensors
            after_mixer = (norms["post_mixer"].weight * scales["mixer"]).contiguous()
            after_ff = None
            if "post_feed_forward" in norms:
                after_ff = (norms["post_feed_forward"].weight * scales["feed_forward"]).contiguous()
            taps = torch.zeros((self.width, self.taps), dtype=torch.float32, device=after_mixer.device)
            if self._taps is not None:
                taps += self._taps
            taps[:, -1] += 1.0                                        # h itself
            self._gains = (after_mixer, after_ff, (taps * norms["pre_mixer"].weight[:, None]).contiguous())
        return self._gains

    def begin(self, hidden, ctx):
        ops = self.env.ops
        y = ops.empty(hidden.shape, torch.float32, hidden.device)
        inverse = ops.empty((hidden.shape[0],), torch.float32, hidden.device)
        return SandwichCarrier(hidden, y, inverse, (None, 1.0, self.norms["pre_mixer"].params["eps"]))

    def forward(self, hidden, ctx, layer):
        carrier, ops = hidden, self.env.ops
        after_mixer, after_ff, taps = self._folded()
        own = layer
        kept = None
        if layer.state is not None:
            if self.kept:
                kept = layer.state[:, :self.kept]
                at = padded(self.kept)
                own = state_share(layer, at, layer.state.shape[1] - at) if layer.state.shape[1] > at else layer
        x = carrier.x
        h = ops.empty(x.shape, self.env.dtype, x.device)
        gain, factor, eps = carrier.pending
        if getattr(ctx, "single_tokens", False) and ops.close_conv_ok(carrier.y, taps, self.taps, kept):
            ops.sandwich_close_conv(carrier.y, x, gain, factor, eps, taps, self.taps, kept, ctx, h)
        else:
            ops.sandwich_close(carrier.y, x, gain, factor, eps, row_scale=carrier.inverse)
            ops.short_conv(x, taps, self.taps, self.width, kept, ctx, h, row_scale=carrier.inverse)
        self.mixer.forward(h, carrier.y, ctx, own)
        alone = getattr(self.feed_forward, "is_empty", False)
        eps = self.norms["post_mixer"].params["eps"]
        if alone:
            carrier.pending = (after_mixer, self.mixer.output_scale, eps)
            return
        h = ops.empty(x.shape, self.env.dtype, x.device)
        ops.sandwich_close(carrier.y, x, after_mixer, self.mixer.output_scale, eps,
                           next_gain=self.norms["pre_feed_forward"].weight, out=h)
        self.feed_forward.forward(h, carrier.y, ctx)
        carrier.pending = (after_ff, 1.0, eps)

    def end(self, carrier, ctx):
        self.env.ops.sandwich_close(carrier.y, carrier.x, *carrier.pending)
        return carrier.x
