"""The arrangement of a layer's parts around the residual stream.

Parity: src/llmserve/model/llama.py:131-135 — ``x += mixer(norm(x)); x += ff(norm(x))``.
The residual stream is a 32-bit tensor that the norms update in place: each part returns its
contribution, and the next norm adds it before normalising (one pass over the row instead of
three).  In bfloat16 the last product of a part adds into the stream itself (see ``ops.ResidualSink``): a
small step's product also hands the stream on already normalised for the next norm, so a decode step has
no norm launches of its own; a large step's product leaves a norm kernel that only reads the stream.
"""

from __future__ import annotations

import torch

from .. import ops
from .base import Block, CompositeSpec, FeedForward, Mixer, Norm, StateSpec, TensorSpec, register_part


def _takes_factored(part) -> bool:
    """Whether a part reads its input in factored form (``ops.NormedInput``): by default every part that takes a sink for its
    last product does; one whose first kernel wants the normed rows themselves says ``takes_factored = False`` and gets them
    from the norm's own kernel."""
    return bool(getattr(part, "takes_factored", getattr(part, "accepts_sink", False)))


class PreNormBlock(Block):
    roles = {"mixer_norm": "norm", "mixer": "mixer", "ff_norm": "norm", "feed_forward": "feed_forward"}

    def __init__(self, mixer_norm: Norm, mixer: Mixer, ff_norm: Norm, feed_forward: FeedForward, residual_scale: float = 1.0):
        self.mixer_norm = mixer_norm
        self.mixer = mixer
        self.ff_norm = ff_norm
        self.feed_forward = feed_forward
        self.residual_scale = float(residual_scale)  # x += residual_scale * part(norm(x))
        # whether the part behind each norm takes the stream in factored form (ops.NormedInput); where it does not, the
        # product in front of the norm is not asked for that form (it would only be multiplied out again)
        mixer_norm.feeds_factored = _takes_factored(mixer)
        ff_norm.feeds_factored = _takes_factored(feed_forward)

    @property
    def graph_safe(self) -> bool:
        return all(p.graph_safe for p in (self.mixer_norm, self.mixer, self.ff_norm, self.feed_forward))

    def forward(self, resid, pending, ctx, cache, next_norm=None):
        x = self._normed(self.mixer_norm, resid, pending, self.mixer)
        sink = self._sink(self.mixer, self.ff_norm, resid, ctx)
        pending = self.mixer.forward(x, ctx, cache, sink=sink) if sink else self.mixer.forward(x, ctx, cache)
        x = self._normed(self.ff_norm, resid, self._scaled(pending), self.feed_forward)
        sink = self._sink(self.feed_forward, next_norm, resid, ctx)
        return self._scaled(self.feed_forward.forward(x, ctx, sink=sink) if sink else self.feed_forward.forward(x, ctx))

    def _scaled(self, pending):
        """A part's contribution as the stream is to take it: times this block's ``residual_scale``."""
        if self.residual_scale != 1.0 and isinstance(pending, torch.Tensor):
            return ops.Scaled(pending, self.residual_scale)
        return pending

    @staticmethod
    def _normed(norm, resid, pending, consumer):
        """``pending`` is a contribution still to be added (a tensor, or one with its factor), or the stream already
        summed and normalised for ``norm`` by the part before (a fused decode kernel did both).  A consumer
        that does not say it takes the factored form gets a plain tensor."""
        if isinstance(pending, ops.NormedInput):
            if pending.norm is not norm:
                raise RuntimeError("a part handed the residual stream on normalised for another norm")
            return pending if _takes_factored(consumer) else pending.materialize()
        if isinstance(pending, ops.BranchSum) and hasattr(norm, "add_branches"):
            x = norm.add_branches(resid, pending)  # the branches' meeting, the sum into the stream and the norm as one kernel
            if x is not None:
                return x
        delta, alpha = ops.split_pending(pending)
        if alpha != 1.0:
            return norm.add_forward(resid, delta, alpha=alpha)
        return norm.add_forward(resid, delta)

    def _sink(self, part, norm, resid, ctx):
        """A sink for the part's last product, if the part takes one and another norm follows (the last part of the
        last layer keeps its contribution: only the rows whose logits are wanted are summed).  Where that norm is an
        RMS norm its weight goes along, so that a small step's product can hand the stream on normalised."""
        if norm is None or not getattr(part, "accepts_sink", False):
            return None
        if not ops.ResidualSink.usable(ctx.num_tokens, getattr(norm, "out_dtype", None)):
            return None
        fused = getattr(norm, "fused_params", None)
        weight, eps = fused() if fused is not None else (None, 0.0)
        if self.residual_scale != 1.0:
            weight = None  # the product that also normalises adds its result unscaled
        if not getattr(norm, "feeds_factored", True):
            weight = None  # whoever reads that norm wants a plain tensor: the product only adds, the norm runs as a kernel
        return ops.ResidualSink(resid, weight, eps, norm, alpha=self.residual_scale)


class MixerOnlyBlock(PreNormBlock):
    """A layer without a feed-forward: ``x += residual_scale * mixer(norm(x))``."""

    roles = {"mixer_norm": "norm", "mixer": "mixer"}

    def __init__(self, mixer_norm: Norm, mixer: Mixer, residual_scale: float = 1.0):
        self.mixer_norm = mixer_norm
        self.mixer = mixer
        self.residual_scale = float(residual_scale)
        mixer_norm.feeds_factored = _takes_factored(mixer)

    @property
    def graph_safe(self) -> bool:
        return all(p.graph_safe for p in (self.mixer_norm, self.mixer))

    def forward(self, resid, pending, ctx, cache, next_norm=None):
        x = self._normed(self.mixer_norm, resid, pending, self.mixer)
        sink = self._sink(self.mixer, next_norm, resid, ctx)
        return self._scaled(self.mixer.forward(x, ctx, cache, sink=sink) if sink else self.mixer.forward(x, ctx, cache))


class ParallelBlock(PreNormBlock):
    """Mixer and feed-forward side by side, each behind a norm of its own of the same rows, with an optional token shift on what
    the mixer reads:

        h = norm1(x),  h_t <- h_t + shift * (h_(t-1) - h_t)          (``token_shift``: a tensor ``shift [hidden]`` of this block)
        x <- x + mixer(h) + feed_forward(norm2(x))

    ``h_(t-1)`` is the unshifted h of the token in front in the same request (zeros in front of the first); the last one of every
    step is kept in a 32-bit state slot beside what the mixer keeps.  Both norms, the shift and the slot are one kernel.  Where
    both parts end in a plain product (``joins_output``) the block stacks the two matrices side by side and runs one product
    that adds both contributions into the stream."""

    accepts_sink = True  # the joined product's end may add into the stream

    def __init__(self, mixer_norm: Norm, mixer: Mixer, ff_norm: Norm | None, feed_forward: FeedForward | None, hidden_size: int,
                 token_shift: bool = False, shift_name: str = "shift"):
        self.mixer_norm, self.mixer, self.ff_norm, self.feed_forward = mixer_norm, mixer, ff_norm, feed_forward
        self.hidden_size, self.token_shift, self.shift_name = int(hidden_size), bool(token_shift), shift_name
        self.residual_scale = 1.0
        # two norms read the rows, and a shifted row is no multiple of one row: nobody in front can hand the stream on normalised
        mixer_norm.feeds_factored = False
        self.shift: torch.Tensor | None = None
        self.w_join: torch.Tensor | None = None  # [hidden, mixer's inner size + feed-forward's]

    def owned_parts(self):
        return [p for p in (self.mixer_norm, self.mixer, self.ff_norm, self.feed_forward) if p is not None]

    @property
    def graph_safe(self) -> bool:
        return all(p.graph_safe for p in self.owned_parts())

    def tensors(self):
        return {self.shift_name: TensorSpec((self.hidden_size,), init="half_plus_normal")} if self.token_shift else {}

    def bind(self, tensors, dtype, device) -> None:
        """Called after the parts' own ``bind``."""
        if self.token_shift:
            self.shift = tensors[self.shift_name].to(device=device, dtype=torch.float32).contiguous()
        ends = [p for p in (self.mixer, self.feed_forward) if p is not None]
        if all(p.joins_output for p in ends):
            self.w_join = torch.cat([p.release_output_matrix() for p in ends], dim=1).contiguous()

    def cache_spec(self):
        spec = self.mixer.cache_spec()
        if not self.token_shift:
            return spec
        parts = spec.parts if isinstance(spec, CompositeSpec) else (spec,)
        return CompositeSpec((*parts, StateSpec((self.hidden_size,), torch.float32)))

    def _views(self, cache):
        """``(the mixer's view, the state slots of the shift or None)``."""
        if not self.token_shift:
            return cache, None
        *mine, state = cache.parts
        return (type(cache)(mine) if isinstance(self.mixer.cache_spec(), CompositeSpec) else mine[0]), state

    def forward(self, resid, pending, ctx, cache, next_norm=None):
        delta, alpha = ops.split_pending(pending)
        if delta is not None:
            ops.stream_inject(resid, delta, alpha)
        view, state = self._views(cache)
        h, g = self.mixer_norm.pair_forward(resid, self.ff_norm, ctx, self.shift, None if state is None else state.states,
                                            None if state is None else state.slots)
        if self.w_join is None:
            y = self.mixer.forward(h, ctx, view)
            if self.feed_forward is None:
                return y
            delta, alpha = ops.split_pending(y)
            z = self.feed_forward.forward(g, ctx)
            ops.stream_inject(resid, delta, alpha)
            return z
        width = self.mixer.output_width
        rows = torch.empty((h.shape[0], self.w_join.shape[1]), dtype=h.dtype, device=h.device)
        self.mixer.forward(h, ctx, view, into=rows[:, :width])
        if self.feed_forward is not None:
            self.feed_forward.forward(g, ctx, into=rows[:, width:])
        sink = self._sink(self, next_norm, resid, ctx)
        if sink is not None:
            handed_on = sink.linear(rows, self.w_join)
            if handed_on is not None:
                return handed_on
        return ops.linear(rows, self.w_join, out_dtype=torch.float32)


class ParallelMixerOnlyBlock(ParallelBlock):
    """The same without a feed-forward: ``x <- x + mixer(h)``."""

    roles = {"mixer_norm": "norm", "mixer": "mixer"}

    def __init__(self, mixer_norm: Norm, mixer: Mixer, hidden_size: int, token_shift: bool = False, shift_name: str = "shift"):
        super().__init__(mixer_norm, mixer, None, None, hidden_size, token_shift, shift_name)


class PostNormBlock(Block):
    """A layer whose parts read the stream itself and whose norms stand behind them:

        x <- x + norm1(mixer(x))        x <- x + norm2(feed_forward(x))

    A part's product leaves its result in 32-bit; one kernel adds a bias that the part left for it (``Part.leaves_bias``), norms,
    sums into the stream and writes the stream's new rows in the compute type for the part behind (``ops.StreamCopy``).  In 32-bit
    the parts read the stream's own rows."""

    roles = {"mixer": "mixer", "mixer_norm": "norm", "feed_forward": "feed_forward", "ff_norm": "norm"}
    reads_stream = True

    def __init__(self, mixer: Mixer, mixer_norm: Norm, feed_forward: FeedForward | None = None, ff_norm: Norm | None = None):
        self.mixer, self.mixer_norm, self.feed_forward, self.ff_norm = mixer, mixer_norm, feed_forward, ff_norm

    def owned_parts(self):
        return [p for p in (self.mixer, self.mixer_norm, self.feed_forward, self.ff_norm) if p is not None]

    @property
    def graph_safe(self) -> bool:
        return all(p.graph_safe for p in self.owned_parts())

    def first_norm(self):
        return None  # the stream meets a part first

    def forward(self, resid, pending, ctx, cache, next_norm=None):
        x = self._read(resid, pending)
        x = self._take_up(resid, self.mixer.forward(x, ctx, cache), self.mixer_norm)
        if self.feed_forward is not None:
            more = {"leave_bias": True} if self.feed_forward.leaves_bias else {}
            x = self._take_up(resid, self.feed_forward.forward(x, ctx, **more), self.ff_norm)
        return ops.StreamCopy(x)

    def _read(self, resid, pending):
        """The stream's rows in the compute type, with everything added."""
        if isinstance(pending, ops.StreamCopy):
            return pending.rows
        delta, alpha = ops.split_pending(pending)
        if delta is not None:
            ops.stream_inject(resid, delta, alpha)
        return resid if self.mixer_norm.out_dtype == torch.float32 else resid.to(self.mixer_norm.out_dtype)

    @staticmethod
    def _take_up(resid, result, norm):
        bias = None
        if isinstance(result, ops.Biased):
            result, bias = result.tensor, result.bias
        result, alpha = ops.split_pending(result)
        if alpha != 1.0:
            result = result * alpha
        copy_dtype = norm.out_dtype if norm.out_dtype != torch.float32 else None
        copy = norm.after_forward(resid, result, bias=bias, copy_dtype=copy_dtype)
        return resid if copy is None else copy


class PostNormMixerOnlyBlock(PostNormBlock):
    """The same without a feed-forward: ``x <- x + norm1(mixer(x))``."""

    roles = {"mixer": "mixer", "mixer_norm": "norm"}

    def __init__(self, mixer: Mixer, mixer_norm: Norm):
        super().__init__(mixer, mixer_norm)


class HyperConnectionBlock(Block):
    """A pre-norm layer over a residual stream kept in S copies ``x_1 .. x_S`` (hyper-connections).  For each of its parts
    q (1: the mixer, 2: the feed-forward) it owns ``hc<q>.in [S]``, ``hc<q>.out [S]`` and ``hc<q>.mix [S, S]``:

        u = sum_s in[s] x_s        y = part(norm(u))        x_t <- sum_s mix[s, t] x_s + out[t] * y     (all t at once)

    ``resid`` is ``[S, N, hidden]`` (``ModelPlan.streams``).  What a part returns travels as an ``ops.StreamUpdate``; the
    copies take it up in the same kernel that reads them in and norms for the next part (``Norm.add_streams``), so a
    part costs one pass over the copies.  ``feed_forward`` may be absent (None): the layer then has no second part."""

    roles = {"mixer_norm": "norm", "mixer": "mixer", "ff_norm": "norm", "feed_forward": "feed_forward"}

    def __init__(self, mixer_norm: Norm, mixer: Mixer, ff_norm: Norm | None = None, feed_forward: FeedForward | None = None,
                 streams: int = 1, names: tuple[str, str] = ("hc1", "hc2")):
        if not 1 <= int(streams) <= 8:
            raise ValueError(f"a residual stream is kept in one to eight copies, got {streams}")
        self.mixer_norm, self.mixer, self.ff_norm, self.feed_forward = mixer_norm, mixer, ff_norm, feed_forward
        self.streams, self.names = int(streams), tuple(names)
        self.hc: list[tuple[torch.Tensor, torch.Tensor, torch.Tensor]] = []  # per part: (in, mix, out), 32-bit

    def owned_parts(self):
        return [p for p in (self.mixer_norm, self.mixer, self.ff_norm, self.feed_forward) if p is not None]

    @property
    def graph_safe(self) -> bool:
        return all(p.graph_safe for p in self.owned_parts())

    def _parts(self) -> int:
        return 1 if self.feed_forward is None else 2

    def tensors(self):
        S, specs = self.streams, {}
        for name in self.names[: self._parts()]:
            specs[f"{name}.in"] = TensorSpec((S,), init="ones_plus_normal")
            specs[f"{name}.out"] = TensorSpec((S,), init="ones_plus_normal")
            specs[f"{name}.mix"] = TensorSpec((S, S), init="eye_plus_normal")
        return specs

    def bind(self, tensors, dtype, device) -> None:
        f32 = lambda t: t.to(device=device, dtype=torch.float32).contiguous()  # noqa: E731
        self.hc = [(f32(tensors[f"{n}.in"]), f32(tensors[f"{n}.mix"]), f32(tensors[f"{n}.out"])) for n in self.names[: self._parts()]]

    def forward(self, resid, pending, ctx, cache, next_norm=None):
        if resid.dim() != 3 or resid.shape[0] != self.streams:
            raise RuntimeError(f"this block reads a residual stream in {self.streams} copies, got a tensor of shape {tuple(resid.shape)}")
        if pending is not None and not isinstance(pending, ops.StreamUpdate):
            raise RuntimeError("a stream kept in copies takes up what a part returned together with that part's mixing weights")
        read_in, mix, take = self.hc[0]
        x = self.mixer_norm.add_streams(resid, pending, read_in)
        pending = ops.StreamUpdate(self.mixer.forward(x, ctx, cache), mix, take)
        if self.feed_forward is None:
            return pending
        read_in, mix, take = self.hc[1]
        x = self.ff_norm.add_streams(resid, pending, read_in)
        return ops.StreamUpdate(self.feed_forward.forward(x, ctx), mix, take)


class HyperConnectionMixerOnlyBlock(HyperConnectionBlock):
    """The same without a feed-forward: one part a layer."""

    roles = {"mixer_norm": "norm", "mixer": "mixer"}

    def __init__(self, mixer_norm: Norm, mixer: Mixer, streams: int = 1, names: tuple[str, str] = ("hc1", "hc2")):
        super().__init__(mixer_norm, mixer, None, None, streams=streams, names=names)


register_part("block", "hyper_connection", HyperConnectionBlock)
register_part("block", "hyper_connection_mixer_only", HyperConnectionMixerOnlyBlock)
register_part("block", "parallel", ParallelBlock)
register_part("block", "parallel_mixer_only", ParallelMixerOnlyBlock)
register_part("block", "post_norm", PostNormBlock)
register_part("block", "post_norm_mixer_only", PostNormMixerOnlyBlock)
register_part("block", "pre_norm", PreNormBlock)
register_part("block", "pre_norm_mixer_only", MixerOnlyBlock)
