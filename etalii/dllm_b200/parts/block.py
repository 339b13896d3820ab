"""Arrangements of a layer's parts. A block class declares the parts it takes as `PARTS` (name -> role), is built
with them as keyword arguments, exposes them as `parts` (name -> part) and its one mixer as `mixer`, and runs them
in `forward(x, batch, cache, rt, write_cache)` on the float32 residual stream x.

"pre_norm": x += mixer(norm(x)); x += feed_forward(norm(x)) (reference: src/etalii_dllm/transformer.py:493-558).
"output_norm": x += norm(mixer(x)); x += norm(feed_forward(x)): the sublayers read the stream itself and the norm sits
on what they return.
"filtered_pre_norm": x += mixer(filter(norm(x))); x += feed_forward(norm(x)); x += token_input(x): a filter over time
sits between the first norm and the mixer; the feed-forward and the token input are optional.
"sandwich_norm": x += norm(mixer(norm(x))); x += norm(feed_forward(norm(x))), the feed-forward optional; optionally the
stream then becomes a weighted sum of all layers' results so far.
"shared_norm": x += mixer(h) + feed_forward(h) with one h = norm(x), the feed-forward optional."""
from __future__ import annotations

import torch

from ..kernels import ops
from .norm import RMSNorm, StreamOperand, leave_normed, taken_normed
from .registry import register_part
from .spec import ParamSpec


def normed(norm, consumer, x, rt):
    """The norm's output for `consumer`: a consumer that says so gets the norm still pending and may apply it
    inside its own kernel."""
    if getattr(consumer, "accepts_pending_norm", False) and hasattr(norm, "lazy"):
        return norm.lazy(x, rt)
    return norm.forward(x, rt)


class PreNormBlock:
    PARTS = {"mixer": "mixer", "feed_forward": "feed_forward", "mixer_norm": "norm", "feed_forward_norm": "norm"}

    def __init__(self, mixer, feed_forward, mixer_norm, feed_forward_norm) -> None:
        self.mixer, self.feed_forward = mixer, feed_forward
        self.mixer_norm, self.feed_forward_norm = mixer_norm, feed_forward_norm
        self.parts = {"mixer": mixer, "feed_forward": feed_forward, "mixer_norm": mixer_norm,
                      "feed_forward_norm": feed_forward_norm}
        # each norm feeds exactly one part here, so its weight may move into that part's first product
        for norm, consumer in ((mixer_norm, mixer), (feed_forward_norm, feed_forward)):
            if hasattr(norm, "give_weight_to"):
                norm.give_weight_to(consumer)

    def forward(self, x, batch, cache, rt, write_cache: bool = True) -> None:
        self.mixer.forward(normed(self.mixer_norm, self.mixer, x, rt), x, batch, cache, rt, write_cache)
        self.feed_forward.forward(normed(self.feed_forward_norm, self.feed_forward, x, rt), x, batch, rt)


class PreNormMixerBlock:
    """A layer without a feed-forward: x += mixer(norm(x))."""

    PARTS = {"mixer": "mixer", "mixer_norm": "norm"}

    def __init__(self, mixer, mixer_norm) -> None:
        self.mixer, self.mixer_norm = mixer, mixer_norm
        self.parts = {"mixer": mixer, "mixer_norm": mixer_norm}
        if hasattr(mixer_norm, "give_weight_to"):
            mixer_norm.give_weight_to(mixer)

    def forward(self, x, batch, cache, rt, write_cache: bool = True) -> None:
        self.mixer.forward(normed(self.mixer_norm, self.mixer, x, rt), x, batch, cache, rt, write_cache)


def stream_input(consumer, x, rt):
    """The stream as `consumer`'s input: a consumer that says so (`accepts_stream`) gets it still in float32 with
    the rounding pending, anyone else the rounded activations. Where the kernel that last wrote the stream also left
    its rounding (`leave_rounded`) and no kernel has run since, that copy is the rounding."""
    ready = None
    kept = getattr(rt, "stream_rounded", None)
    if kept is not None and kept[0] == x.data_ptr() and kept[1] == tuple(x.shape) and kept[2] == ops.launches:
        ready = kept[3]
    operand = StreamOperand(x, rt, ready)
    return operand if getattr(consumer, "accepts_stream", False) else operand.tensor()


def add_normed_output(norm, x, out, rt) -> None:
    """x += norm(out); in bfloat16 the same kernel leaves the new rows rounded for whoever reads the stream next."""
    copy = rt.ws.buffer("stream_operand", tuple(x.shape), rt.dtype) if rt.dtype == torch.bfloat16 else None
    norm.add_normed(x, out, rt, copy)
    rt.stream_rounded = (x.data_ptr(), tuple(x.shape), ops.launches, copy) if copy is not None else None


class OutputNormBlock:
    """x += mixer_norm(mixer(x)); x += feed_forward_norm(feed_forward(x)). Each sublayer writes its float32 output to
    a work buffer (`epilogue=ops.EPI_STORE_F32`) and the norm adds the normed rows into the stream in one kernel
    (`add_normed`), which also leaves the stream's rounding for the next sublayer's products."""

    PARTS = {"mixer": "mixer", "feed_forward": "feed_forward", "mixer_norm": "norm", "feed_forward_norm": "norm"}

    def __init__(self, mixer, feed_forward, mixer_norm, feed_forward_norm) -> None:
        self.mixer, self.feed_forward = mixer, feed_forward
        self.mixer_norm, self.feed_forward_norm = mixer_norm, feed_forward_norm
        self.parts = {"mixer": mixer, "feed_forward": feed_forward, "mixer_norm": mixer_norm,
                      "feed_forward_norm": feed_forward_norm}

    def forward(self, x, batch, cache, rt, write_cache: bool = True) -> None:
        out = rt.ws.buffer("sublayer_out", tuple(x.shape), torch.float32)
        self.mixer.forward(stream_input(self.mixer, x, rt), out, batch, cache, rt, write_cache,
                           epilogue=ops.EPI_STORE_F32)
        add_normed_output(self.mixer_norm, x, out, rt)
        self.feed_forward.forward(stream_input(self.feed_forward, x, rt), out, batch, rt, epilogue=ops.EPI_STORE_F32)
        add_normed_output(self.feed_forward_norm, x, out, rt)


class OutputNormMixerBlock:
    """A layer without a feed-forward: x += mixer_norm(mixer(x))."""

    PARTS = {"mixer": "mixer", "mixer_norm": "norm"}

    def __init__(self, mixer, mixer_norm) -> None:
        self.mixer, self.mixer_norm = mixer, mixer_norm
        self.parts = {"mixer": mixer, "mixer_norm": mixer_norm}

    def forward(self, x, batch, cache, rt, write_cache: bool = True) -> None:
        out = rt.ws.buffer("sublayer_out", tuple(x.shape), torch.float32)
        self.mixer.forward(stream_input(self.mixer, x, rt), out, batch, cache, rt, write_cache,
                           epilogue=ops.EPI_STORE_F32)
        add_normed_output(self.mixer_norm, x, out, rt)


class FilteredPreNormBlock:
    """x += mixer(filter(mixer_norm(x))); then, where the layer has them, x += feed_forward(feed_forward_norm(x)) and
    x += token_input(x). The filter (a short convolution over time) keeps a history of its own beside what the mixer
    keeps: the block answers for the layer's cache need and hands each part its view."""

    PARTS = {"mixer": "mixer", "mixer_norm": "norm", "mixer_filter": "filter"}
    OPTIONAL_PARTS = {"feed_forward": "feed_forward", "feed_forward_norm": "norm", "token_input": "token_input"}

    def __init__(self, mixer, mixer_norm, mixer_filter, feed_forward=None, feed_forward_norm=None,
                 token_input=None) -> None:
        if (feed_forward is None) != (feed_forward_norm is None):
            raise ValueError("a feed-forward and its norm come together")
        self.mixer, self.mixer_norm, self.mixer_filter = mixer, mixer_norm, mixer_filter
        self.feed_forward, self.feed_forward_norm, self.token_input = feed_forward, feed_forward_norm, token_input
        self.parts = {name: part for name, part in (
            ("mixer", mixer), ("mixer_norm", mixer_norm), ("mixer_filter", mixer_filter),
            ("feed_forward", feed_forward), ("feed_forward_norm", feed_forward_norm), ("token_input", token_input))
            if part is not None}
        if feed_forward is not None and hasattr(feed_forward_norm, "give_weight_to"):
            feed_forward_norm.give_weight_to(feed_forward)
        self._filter_keeps = mixer_filter.cache_need() is not None
        self._mixer_keeps = hasattr(mixer, "cache_need") and mixer.cache_need() is not None

    def cache_need(self):
        from ..cache.paged import CacheNeed

        needs = []
        if self._mixer_keeps:
            needs.append(self.mixer.cache_need())
        if self._filter_keeps:
            needs.append(self.mixer_filter.cache_need())
        if not needs:
            return None
        return CacheNeed("several", parts=tuple(needs))

    def forward(self, x, batch, cache, rt, write_cache: bool = True) -> None:
        views = list(cache) if cache is not None else []
        mixer_view = views.pop(0) if self._mixer_keeps else None
        history = views.pop(0) if self._filter_keeps else None
        h = self.mixer_filter.forward(self.mixer_norm, x, batch, history, rt)
        self.mixer.forward(h, x, batch, mixer_view, rt, write_cache)
        if self.feed_forward is not None:
            self.feed_forward.forward(normed(self.feed_forward_norm, self.feed_forward, x, rt), x, batch, rt)
        if self.token_input is not None:
            self.token_input.forward(x, batch, rt)


class DepthAverage:
    """What leaves layer `index` of `layers`: the sum over j = 0 .. index + 1 of weight[j] X_j, with X_0 the embedding's
    output and X_(i + 1) the result of layer i before this sum. The X_j of a step live in a work buffer [layers, tokens,
    hidden] float32 (the last layer's result is read by nobody)."""

    def __init__(self, index: int, layers: int) -> None:
        self.index, self.layers = int(index), int(layers)
        self.weight = None

    @staticmethod
    def parameters(index, layers) -> dict[str, ParamSpec]:
        return {"weight": ParamSpec((int(index) + 2,), "last_one")}

    def bind(self, tensors, rt) -> None:
        self.weight = rt.to_device(tensors["weight"], torch.float32)

    def results(self, x: torch.Tensor, rt) -> torch.Tensor:
        return rt.ws.buffer("layer_results", (self.layers, *x.shape), torch.float32)


class SandwichNormBlock:
    """x += mixer_output_norm(mixer(mixer_norm(x))); then, where the layer has one, x += feed_forward_output_norm(
    feed_forward(feed_forward_norm(x))); then, with a `depth_average`, the stream becomes the weighted sum of all layers'
    results so far. (A multiplier of the sublayers is the output norms' `factor`.) Each sublayer writes its float32
    output to a work buffer and ONE kernel does everything from there to the next product's operand: the output's norm,
    the residual sum, the sum over the layers, and the norm in front of whoever reads the stream next (the model tells a
    block whose norm that is: `leads_to`)."""

    PARTS = {"mixer": "mixer", "mixer_norm": "norm", "mixer_output_norm": "norm"}
    OPTIONAL_PARTS = {"feed_forward": "feed_forward", "feed_forward_norm": "norm", "feed_forward_output_norm": "norm",
                      "depth_average": "stream_mix"}
    LIBRARIES = ("stream_update",)

    def __init__(self, mixer, mixer_norm, mixer_output_norm, feed_forward=None, feed_forward_norm=None,
                 feed_forward_output_norm=None, depth_average=None) -> None:
        together = (feed_forward, feed_forward_norm, feed_forward_output_norm)
        if any(part is None for part in together) != all(part is None for part in together):
            raise ValueError("a feed-forward and its two norms come together")
        self.mixer, self.mixer_norm, self.mixer_output_norm = mixer, mixer_norm, mixer_output_norm
        self.feed_forward, self.feed_forward_norm = feed_forward, feed_forward_norm
        self.feed_forward_output_norm, self.depth_average = feed_forward_output_norm, depth_average
        self.parts = {name: part for name, part in (
            ("mixer", mixer), ("mixer_norm", mixer_norm), ("mixer_output_norm", mixer_output_norm),
            ("feed_forward", feed_forward), ("feed_forward_norm", feed_forward_norm),
            ("feed_forward_output_norm", feed_forward_output_norm), ("depth_average", depth_average))
            if part is not None}
        self._next = None  # (norm, last): the norm of whoever reads the stream behind this block
        self._told = False

    def leads_to(self, norm, last: bool = False) -> None:
        """`norm`: what the next reader of the stream norms it by (None: not known); `last`: that reader wants single
        rows of a prompt, so the whole stream is normed for it in steps of single tokens only. A block that runs
        several times with different readers behind it norms for none."""
        if self._told and (self._next is None or self._next[0] is not norm):
            self._next = None
        else:
            self._next = (norm, bool(last)) if getattr(norm, "weight", None) is not None and \
                isinstance(norm, RMSNorm) else None
        self._told = True

    def _update(self, x, out, output_norm, following, rt, average=None, keep_first=None, mix_first: bool = False) -> None:
        """The kernel behind a sublayer: see `ops.stream_update`."""
        normed_out = None
        if following is not None:
            normed_out = rt.ws.buffer("stream_normed", tuple(x.shape), rt.dtype)
        results = average.results(x, rt) if average is not None else None
        ops.stream_update(x, out, output_norm.weight, output_norm.eps,
                          first_result=keep_first, results=results,
                          index=average.index if average is not None else 0,
                          coefficients=average.weight if average is not None else None,
                          first_from_stream=mix_first,
                          next_weight=following.weight if following is not None else None,
                          next_eps=following.eps if following is not None else 0.0, normed=normed_out)
        if following is not None:
            leave_normed(following, x, rt, normed_out)

    def forward(self, x, batch, cache, rt, write_cache: bool = True) -> None:
        out = rt.ws.buffer("sublayer_out", tuple(x.shape), torch.float32)
        following = None
        if self._next is not None and (batch.is_decode or not self._next[1]):
            following = self._next[0]
        average = self.depth_average
        # the first layer's input is the embedding's output: its first kernel keeps it for the sums over the layers
        keep = average.results(x, rt)[0] if average is not None and average.index == 0 else None
        h = taken_normed(self.mixer_norm, x, rt)
        if h is None:
            h = self.mixer_norm.forward(x, rt)
        self.mixer.forward(h, out, batch, cache, rt, write_cache, epilogue=ops.EPI_STORE_F32)
        if self.feed_forward is None:
            self._update(x, out, self.mixer_output_norm, following, rt, average, keep, keep is not None)
            return
        self._update(x, out, self.mixer_output_norm, self.feed_forward_norm, rt, None, keep)
        h = taken_normed(self.feed_forward_norm, x, rt)
        self.feed_forward.forward(h, out, batch, rt, epilogue=ops.EPI_STORE_F32)
        self._update(x, out, self.feed_forward_output_norm, following, rt, average)


class SharedNormBlock:
    """x += mixer(h) + feed_forward(h) with h = mixer_norm(x), an RMS norm; the feed-forward is optional. One kernel makes h
    in every form its readers take: plain rows, rows with a 1 behind them for parts whose biases are a column of their
    matrix (`wants_ones`). Both readers have their input before either adds to the stream. Output biases of the parts that
    give them away (`take_output_bias`) are one row vector of the layer, which the same kernel adds to the stream."""

    PARTS = {"mixer": "mixer", "mixer_norm": "norm"}
    OPTIONAL_PARTS = {"feed_forward": "feed_forward"}

    def __init__(self, mixer, mixer_norm, feed_forward=None) -> None:
        self.mixer, self.mixer_norm, self.feed_forward = mixer, mixer_norm, feed_forward
        self.parts = {name: part for name, part in (("mixer", mixer), ("mixer_norm", mixer_norm),
                                                    ("feed_forward", feed_forward)) if part is not None}
        readers = [part for part in (mixer, feed_forward) if part is not None]
        self._with_ones = any(getattr(part, "wants_ones", False) for part in readers)
        self._plain = not all(getattr(part, "wants_ones", False) for part in readers)
        biases = [part.take_output_bias() for part in readers if hasattr(part, "take_output_bias")]
        biases = [bias for bias in biases if bias is not None]
        self.output_bias = sum(biases[1:], biases[0]).contiguous() if biases else None

    def forward(self, x, batch, cache, rt, write_cache: bool = True) -> None:
        rows, hidden = x.shape
        plain = rt.ws.buffer("normed", (rows, hidden), rt.dtype) if self._plain else None
        ones = rt.ws.buffer("normed_ones", (rows, ops.ones_width(hidden)), rt.dtype) if self._with_ones else None
        ops.norm_operands(x, self.mixer_norm.weight, self.mixer_norm.eps, plain, ones, self.output_bias)
        operand = lambda part: ones if getattr(part, "wants_ones", False) else plain  # noqa: E731
        self.mixer.forward(operand(self.mixer), x, batch, cache, rt, write_cache)
        if self.feed_forward is not None:
            self.feed_forward.forward(operand(self.feed_forward), x, batch, rt)


register_part("block", "shared_norm", SharedNormBlock)
register_part("stream_mix", "depth_average", DepthAverage)
register_part("block", "sandwich_norm", SandwichNormBlock)
register_part("block", "pre_norm", PreNormBlock)
register_part("block", "filtered_pre_norm", FilteredPreNormBlock)
register_part("block", "output_norm", OutputNormBlock)
register_part("block", "output_norm_mixer", OutputNormMixerBlock)
register_part("block", "pre_norm_mixer", PreNormMixerBlock)
