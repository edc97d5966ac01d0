"""A layer at run time, and how its parts are wired.

A block arrangement is a function ``run(ctx, layer, cache, residual32)`` registered under a name;
it finds the layer's parts by the names it expects (``layer.norm1`` ...) and says which names
those are in ``requires``, so that a layer that lacks one is refused when the model is built.
Mixers and feed-forwards add their output to the 32-bit residual stream: in place (they return
nothing), or into another tensor that they return (a kernel that fuses the whole part cannot
always write where it reads); an arrangement hands the stream on with ``stream_after`` and
returns the tensor that holds it at the end (or nothing, if that is the one it was given).
``pre_norm``: ``x += mixer(norm1(x)); x += ff(norm2(x))`` (src/minigpt_infer/model.py:112-115).
``pre_norm_mixer_only``: ``x += mixer(norm1(x))``, for a layer without a feed-forward.
``sandwich_norm``: a norm on both sides of each sublayer, ``x += norm1b(mixer(norm1(x)))``, then, if the layer has a
feed-forward, ``x += norm2b(ff(norm2(x)))``, then, if it has one, the layer's token input (``side_input``), which
reads the stream and the step's tokens and adds into the stream.  The norm behind a sublayer reads its output (what the
sublayer returns, or, of one that can only add, a zeroed 32-bit buffer that it added into) and adds into the stream in
one kernel; where the feed-forward takes plain rows, that kernel also applies the norm in front of it.
``post_norm``: norms behind the sublayers only, ``x += r * norm1(mixer(x))``, then, if the layer has a feed-forward,
``x += r * norm2(ff(x))``, with ``r`` the layer's setting ``residual_scale``.  The sublayers read the stream itself, in the
compute dtype; the norm behind a sublayer writes that copy of the new stream on its way, for the next sublayer or layer.
"""

from __future__ import annotations

from typing import Any, Callable

from .base import register_arrangement


class Layer:
    """The built parts of one layer, by their names in the layer, and the arrangement's function."""

    def __init__(self, parts: dict[str, Any], roles: dict[str, str], run: Callable[..., None],
                 prefix: str = "", settings: dict[str, Any] | None = None) -> None:
        self._parts = dict(parts)
        self.settings = dict(settings or {})      # numbers of the arrangement itself
        self.roles = dict(roles)
        self.run = run
        self.prefix = prefix
        missing = [n for n in getattr(run, "requires", ()) if n not in self._parts]
        if missing:
            raise ValueError(f"layer {prefix!r}: its arrangement needs parts named {missing}; "
                             f"it has {sorted(self._parts)}")

    def __getattr__(self, name: str):
        try:
            return self.__dict__["_parts"][name]
        except KeyError:
            raise AttributeError(f"layer {self.__dict__.get('prefix', '')!r} has no part {name!r}") from None

    def parts(self) -> list:
        return list(self._parts.values())

    def get(self, name: str):
        """The part of that name, or None if the layer has none."""
        return self._parts.get(name)

    def cache_spec(self):
        """What the layer keeps per request: its mixer's wish.  One cache per layer: of several
        mixers at most one may keep something."""
        specs = [spec for name, part in self._parts.items() if self.roles[name] == "mixer"
                 for spec in [part.cache_spec()] if spec is not None]
        if len(specs) > 1:
            raise ValueError(f"layer {self.prefix!r}: more than one of its mixers keeps a cache")
        return specs[0] if specs else None


def _normed(ctx, norm, consumer, residual32):
    """The norm's result, as a deferred norm if its consumer can fuse it."""
    run = norm.defer if getattr(consumer, "accepts_deferred_norm", False) else norm.forward
    return run(ctx, residual32)


def stream_after(returned, residual32):
    """The tensor that holds the residual stream after a part ran: what the part returned, or, if
    it returned nothing, the tensor it was given (it added in place)."""
    return residual32 if returned is None else returned


def pre_norm(ctx, layer: Layer, cache, residual32):
    x = residual32
    x = stream_after(layer.mixer.forward(ctx, cache, _normed(ctx, layer.norm1, layer.mixer, x), x), x)
    return stream_after(layer.feed_forward.forward(ctx, _normed(ctx, layer.norm2, layer.feed_forward, x), x), x)


pre_norm.requires = ("norm1", "mixer", "norm2", "feed_forward")
register_arrangement("pre_norm")(pre_norm)


def pre_norm_mixer_only(ctx, layer: Layer, cache, residual32):
    x = residual32
    return stream_after(layer.mixer.forward(ctx, cache, _normed(ctx, layer.norm1, layer.mixer, x), x), x)


pre_norm_mixer_only.requires = ("norm1", "mixer")
register_arrangement("pre_norm_mixer_only")(pre_norm_mixer_only)


def sandwich_norm(ctx, layer: Layer, cache, residual32):
    x = residual32
    rows, width = x.shape

    def add(part, norm, run, then=None):
        chained = {} if then is None else {"then": then}
        if part.returns_output:
            return norm.add_normed(ctx, run(None), x, **chained)
        # one zeroed buffer serves every sublayer of the pass: the norm behind a sublayer leaves it as zeros again
        zeros = ctx.ops.zeros32(rows, width, ctx)
        y = stream_after(run(zeros), zeros)
        return norm.add_normed(ctx, y, x, clear=y is zeros, **chained)
    mixer, ff = layer.mixer, layer.get("feed_forward")
    then = None
    if ff is not None and not ff.accepts_deferred_norm and layer.norm1b.chains and layer.norm2.chains:
        then = layer.norm2
    u = add(mixer, layer.norm1b, lambda into: mixer.forward(ctx, cache, _normed(ctx, layer.norm1, mixer, x), into), then)
    if ff is not None:
        if then is None:
            u = _normed(ctx, layer.norm2, ff, x)
        add(ff, layer.norm2b, lambda into: ff.forward(ctx, u, into))
    side = layer.get("side_input")
    if side is not None:
        side.forward(ctx, x)
    return None


sandwich_norm.requires = ("norm1", "mixer", "norm1b")
register_arrangement("sandwich_norm")(sandwich_norm)


def _stream_rows(ctx, x):
    """The stream in the compute dtype: the copy that the norm behind the last sublayer wrote, if it is of ``x``."""
    kept = ctx.shared.get("stream rows")
    return kept[1] if kept is not None and kept[0] is x else ctx.ops.cast(x, ctx.act_dtype)


def post_norm(ctx, layer: Layer, cache, residual32):
    x = residual32
    r = layer.settings.get("residual_scale", 1.0)
    rows = _stream_rows(ctx, x)

    def add(part, norm, run):
        if part.returns_output:
            return norm.add_normed(ctx, run(None), x, scale=r, rows_dtype=ctx.act_dtype)
        zeros = ctx.ops.zeros32(*x.shape, ctx)
        y = stream_after(run(zeros), zeros)
        return norm.add_normed(ctx, y, x, clear=y is zeros, scale=r, rows_dtype=ctx.act_dtype)
    mixer, ff = layer.mixer, layer.get("feed_forward")
    rows = add(mixer, layer.norm1, lambda into: mixer.forward(ctx, cache, rows, into))
    if ff is not None:
        rows = add(ff, layer.norm2, lambda into: ff.forward(ctx, rows, into))
    ctx.shared["stream rows"] = (x, rows)
    return None


post_norm.requires = ("norm1", "mixer")
post_norm.keeps_stream_rows = True     # leaves ctx.shared["stream rows"] valid for the layer that follows
register_arrangement("post_norm")(post_norm)
