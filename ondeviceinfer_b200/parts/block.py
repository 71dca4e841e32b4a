"""Arrangement of norms, mixer and feed-forward in a layer."""

from __future__ import annotations

import torch

from ..cache import StateNeed
from ..config.specs import GatedPostNormBlockSpec, ParallelBlockSpec, PreNormBlockSpec, ReinjectSpec, SandwichBlockSpec, ScaledParallelBlockSpec, StreamMixBlockSpec
from ..kernels.ops import STREAM_MIX_MAX_STREAMS, STREAM_MIX_MAX_WIDTH
from ..weights.tensors import TensorDecl
from .base import Part, build_part, register_part


class PreNormBlock(Part):
    """h += mixer(norm(h)); h += feed_forward(norm(h))  (ondeviceinfer/model.py:49-63); the second half is
    left out for a spec without a feed-forward."""

    finishes_residual_adds = True     # its norms take over a residual add that a product left pending

    def __init__(self, spec: PreNormBlockSpec) -> None:
        super().__init__(spec)
        self.mixer_norm = build_part(spec.mixer_norm)
        self.mixer = build_part(spec.mixer)
        # a layer without a feed-forward has neither the part nor its norm
        self.ffn_norm = build_part(spec.ffn_norm) if spec.ffn is not None else None
        self.ffn = build_part(spec.ffn) if spec.ffn is not None else None

    def _children(self):
        return tuple(part for part in (self.mixer_norm, self.mixer, self.ffn_norm, self.ffn) if part is not None)

    def tensor_decls(self):
        return [d for part in self._children() for d in part.tensor_decls()]

    def load(self, fetch, runtime) -> None:
        self.runtime = runtime
        for part in self._children():
            part.load(fetch, runtime)

    def cache_needs(self):
        return tuple(self.mixer.cache_needs())

    @property
    def graph_safe(self) -> bool:
        return all(getattr(part, "graph_safe", False) for part in self._children())

    @staticmethod
    def _normed(norm, consumer, hidden, ctx):
        """norm(hidden); left to the consumer's first product when the product that wrote ``hidden``
        has left the rows' sums of squares in ``ctx.residual_sumsq`` and both sides know how."""
        known = getattr(ctx, "residual_sumsq", None)
        ctx.residual_sumsq = None
        pending = getattr(ctx, "pending_residual_add", None)
        if pending is not None:
            # a product of the part before is still to be added to the stream: in this norm's pass if it is
            # this stream and the norm knows how, else now
            if len(pending) == 2 and pending[0] is hidden and getattr(norm, "adds", False):
                ctx.pending_residual_add = None
                return norm(hidden, add=pending[1])
            from .linear import flush_residual_add
            flush_residual_add(ctx)
        if known is not None and known[0] is hidden and getattr(norm, "lazy", None) is not None and getattr(consumer, "takes_lazy_norm", False):
            return norm.lazy(hidden, known[1])
        return norm(hidden)

    def forward(self, hidden, ctx, view) -> None:
        # This block finishes residual adds that its parts' last products leave pending (in the norm that follows,
        # here or in the next block; the model flushes the last one): it says so, and only then is an add deferred.
        ctx.defers_residual_add = True
        self.mixer.forward(self._normed(self.mixer_norm, self.mixer, hidden, ctx), ctx, view, hidden)
        if self.ffn is not None:
            self.ffn.forward(self._normed(self.ffn_norm, self.ffn, hidden, ctx), ctx, hidden)


class SandwichBlock(Part):
    """h += post_norm(mixer(norm(h))); h += post_norm(feed_forward(norm(h))): a norm on both sides of each sublayer.

    A sublayer's output is taken in fp32, normed in fp32 and added to the fp32 stream in one kernel
    (``ops.rmsnorm_add``), or, when the next sublayer's norm follows at once, together with that norm
    (``ops.rmsnorm_add_norm``): the block leaves the add pending on the step's context (``(hidden, output, weight,
    eps)``), the next norm of this or the following block of this kind finishes it, and the model flushes what is
    left.  A part that says ``returns_output`` (its ``forward`` returns the output when given no residual) is
    asked for that; any other part adds into a zeroed fp32 buffer, as the part interface says, so every
    registered mixer and feed-forward fits."""

    finishes_residual_adds = True     # its norms take over an add that the block before left pending

    def __init__(self, spec: SandwichBlockSpec) -> None:
        super().__init__(spec)
        self.mixer_norm = build_part(spec.mixer_norm)
        self.mixer = build_part(spec.mixer)
        self.mixer_post_norm = build_part(spec.mixer_post_norm)
        has = spec.ffn is not None
        self.ffn_norm = build_part(spec.ffn_norm) if has else None
        self.ffn = build_part(spec.ffn) if has else None
        self.ffn_post_norm = build_part(spec.ffn_post_norm) if has else None
        for norm in (self.mixer_post_norm, self.ffn_post_norm):
            if norm is not None and not hasattr(norm.spec, "eps"):
                raise TypeError("the norm after a sublayer must be an RMS norm (a weight and eps)")

    def _children(self):
        return tuple(part for part in (self.mixer_norm, self.mixer, self.mixer_post_norm, self.ffn_norm, self.ffn,
                                       self.ffn_post_norm) if part is not None)

    def tensor_decls(self):
        return [d for part in self._children() for d in part.tensor_decls()]

    def load(self, fetch, runtime) -> None:
        self.runtime = runtime
        for part in self._children():
            part.load(fetch, runtime)

    def cache_needs(self):
        return tuple(self.mixer.cache_needs())

    @property
    def graph_safe(self) -> bool:
        return all(getattr(part, "graph_safe", False) for part in self._children())

    @staticmethod
    def _branch(part, hidden, call):
        """The fp32 output of a sublayer: ``call(residual)`` runs it."""
        if getattr(part, "returns_output", False):
            return call(None)
        branch = torch.zeros_like(hidden)
        call(branch)
        return branch

    @staticmethod
    def _normed(norm, hidden, ctx):
        """norm(hidden) for the next sublayer; a sublayer output that is still to be normed and added to this
        stream is finished in the same kernel when the norm allows it, else beforehand."""
        from ..kernels import ops
        from .linear import flush_residual_add
        pending = getattr(ctx, "pending_residual_add", None)
        if (pending is not None and len(pending) == 4 and pending[0] is hidden
                and getattr(norm.spec, "scale_in_fp32", False) and hasattr(norm, "weight")):
            out = torch.empty(hidden.shape, dtype=norm.runtime.dtype, device=hidden.device)
            if ops.rmsnorm_add_norm(hidden, pending[1], pending[2], pending[3], norm.weight, norm.spec.eps, out):
                ctx.pending_residual_add = None
                return out
        flush_residual_add(ctx)
        return norm(hidden)

    def forward(self, hidden, ctx, view) -> None:
        ctx.defers_residual_add = False        # the parts' own products add (or return) at once
        normed = self._normed(self.mixer_norm, hidden, ctx)
        out = self._branch(self.mixer, hidden, lambda r: self.mixer.forward(normed, ctx, view, r))
        ctx.pending_residual_add = (hidden, out, self.mixer_post_norm.weight, self.mixer_post_norm.spec.eps)
        if self.ffn is not None:
            normed = self._normed(self.ffn_norm, hidden, ctx)
            out = self._branch(self.ffn, hidden, lambda r: self.ffn.forward(normed, ctx, r))
            ctx.pending_residual_add = (hidden, out, self.ffn_post_norm.weight, self.ffn_post_norm.spec.eps)
        ctx.residual_sumsq = None


class GatedPostNormBlock(Part):
    """x <- x + norm1(mixer(x) * sigmoid(R1 x + r1)); x <- x + norm2(feed_forward(x) * sigmoid(R2 x + r2)).

    The sublayers and the gates' products read the stream's rows in the compute dtype; ``ops.gated_norm_add`` takes a
    sublayer's fp32 output (a part that says ``returns_output`` returns it; any other adds into a zeroed buffer) and the
    gate's fp32 logits, gates, norms and adds to the stream in fp32, and writes the new rows in the compute dtype for
    whoever reads them next: the feed-forward, or the next block of this kind (``ctx.stream_copy``)."""

    renews_stream_copy = True

    def __init__(self, spec: GatedPostNormBlockSpec) -> None:
        super().__init__(spec)
        has = spec.ffn is not None
        if has != (spec.ffn_norm is not None) or (not has and spec.ffn_gate_name is not None):
            raise ValueError("a feed-forward comes with its norm (and perhaps its gate), or none of them")
        self.mixer = build_part(spec.mixer)
        self.mixer_norm = build_part(spec.mixer_norm)
        self.ffn = build_part(spec.ffn) if has else None
        self.ffn_norm = build_part(spec.ffn_norm) if has else None
        for norm in (self.mixer_norm, self.ffn_norm):
            if norm is not None and not (getattr(norm.spec, "scale_in_fp32", False) and hasattr(norm.spec, "eps")):
                raise TypeError("the norm after a sublayer is an RMS norm that scales in fp32")

    def _children(self):
        return tuple(part for part in (self.mixer, self.mixer_norm, self.ffn, self.ffn_norm) if part is not None)

    def tensor_decls(self):
        s = self.spec
        decls = [d for part in self._children() for d in part.tensor_decls()]
        for weight, bias in ((s.mixer_gate_name, s.mixer_gate_bias_name), (s.ffn_gate_name, s.ffn_gate_bias_name)):
            if weight is not None:
                decls.append(TensorDecl(weight, (s.hidden_size, s.hidden_size)))
                if bias is not None:
                    decls.append(TensorDecl(bias, (s.hidden_size,)))
        return decls

    def load(self, fetch, runtime) -> None:
        self.runtime = runtime
        for part in self._children():
            part.load(fetch, runtime)
        s = self.spec
        gate = lambda weight, bias: (None if weight is None else fetch.matrix(weight),
                                     None if weight is None or bias is None else fetch.vector(bias))
        self.mixer_gate = gate(s.mixer_gate_name, s.mixer_gate_bias_name)
        self.ffn_gate = gate(s.ffn_gate_name, s.ffn_gate_bias_name)

    def cache_needs(self):
        return tuple(self.mixer.cache_needs())

    @property
    def graph_safe(self) -> bool:
        return all(getattr(part, "graph_safe", False) for part in self._children())

    def _rows(self, hidden, ctx):
        """The stream's rows in the compute dtype."""
        from ..kernels import ops
        if self.runtime.dtype == torch.float32:
            return hidden
        known = ctx.stream_copy
        if known is not None and known[0] is hidden and known[1].dtype == self.runtime.dtype:
            return known[1]
        rows = torch.empty(hidden.shape, dtype=self.runtime.dtype, device=hidden.device)
        ops.cast_rows(hidden, rows)
        return rows

    def _half(self, hidden, ctx, part, norm, gate, call):
        from ..kernels import ops
        from .linear import linear
        x = self._rows(hidden, ctx)
        weight, bias = gate
        logits = None if weight is None else linear(x, weight, bias=bias, out_dtype=torch.float32)
        out = SandwichBlock._branch(part, hidden, lambda residual: call(x, residual))
        ctx.residual_sumsq = None
        rows = None
        if self.runtime.dtype != torch.float32:
            rows = torch.empty(hidden.shape, dtype=self.runtime.dtype, device=hidden.device)
        ops.gated_norm_add(hidden, out, logits, norm.weight, norm.spec.eps, rows)
        ctx.stream_copy = None if rows is None else (hidden, rows)

    def forward(self, hidden, ctx, view) -> None:
        ctx.defers_residual_add = False        # the parts' own products add (or return) at once
        self._half(hidden, ctx, self.mixer, self.mixer_norm, self.mixer_gate,
                   lambda x, residual: self.mixer.forward(x, ctx, view, residual))
        if self.ffn is not None:
            self._half(hidden, ctx, self.ffn, self.ffn_norm, self.ffn_gate,
                       lambda x, residual: self.ffn.forward(x, ctx, residual))


class ParallelBlock(Part):
    """h = norm(x); x += m (mixer(h + conv(h)) + feed_forward(h)): one norm whose output both sublayers read, a
    short causal convolution over time in front of the mixer, one scaled add.

    ``ops.canon_norm`` makes h and h + conv(h) in one pass over the stream (the norm's weight is one number);
    the rows of h before a sequence's first token of the step come from the sequence's state, the fp32 h of its
    last taps - 1 positions (a :class:`~ondeviceinfer_b200.cache.StateNeed` of the block, zero when a sequence
    starts), which the same launch moves on for a sequence that brings one token and ``ops.canon_state`` for the
    others.  The mixer's fp32 output (a part that says ``returns_output``
    returns it; any other adds into a zeroed buffer) takes the feed-forward's as its residual add, and
    ``ops.scaled_add`` adds the sum to the stream."""

    def __init__(self, spec: ParallelBlockSpec) -> None:
        super().__init__(spec)
        self.norm = build_part(spec.norm)
        self.mixer = build_part(spec.mixer)
        self.ffn = build_part(spec.ffn) if spec.ffn is not None else None
        if not (getattr(spec.norm, "scalar_weight", False) and getattr(spec.norm, "scale_in_fp32", False)):
            raise TypeError("this block's norm has one number as its weight and scales in fp32")
        if spec.conv_taps < 1 or (spec.conv_name is None and spec.conv_taps != 1):
            raise ValueError("conv_taps is at least 1, and 1 without a convolution")
        if spec.conv_taps > 64:
            raise ValueError(f"the convolution kernels take up to 64 taps, got {spec.conv_taps}")
        self.taps = spec.conv_taps if spec.conv_name is not None else 1

    def _children(self):
        return tuple(part for part in (self.norm, self.mixer, self.ffn) if part is not None)

    def tensor_decls(self):
        decls = [d for part in self._children() for d in part.tensor_decls()]
        if self.spec.conv_name is not None:
            decls.append(TensorDecl(self.spec.conv_name, (self.spec.hidden_size, self.spec.conv_taps)))
        return decls

    def load(self, fetch, runtime) -> None:
        self.runtime = runtime
        for part in self._children():
            part.load(fetch, runtime)
        if self.spec.conv_name is not None:
            self.taps_w = fetch.vector(self.spec.conv_name)
        else:       # no convolution: one tap of zero, h + 0 h
            self.taps_w = torch.zeros((self.spec.hidden_size, 1), dtype=torch.float32, device=runtime.device)

    def _state_need(self):
        return StateNeed((self.taps - 1, self.spec.hidden_size), torch.float32, "conv before the mixer")

    def cache_needs(self):
        needs = tuple(self.mixer.cache_needs())
        return needs + ((self._state_need(),) if self.taps > 1 else ())

    @property
    def graph_safe(self) -> bool:
        return all(getattr(part, "graph_safe", False) for part in self._children())

    def forward(self, hidden, ctx, view) -> None:
        ctx.defers_residual_add = False        # the parts' own products add (or return) at once
        ctx.residual_sumsq = None
        state = view.states[-1] if self.taps > 1 else None      # the block's need is the last one it names
        n = hidden.shape[0]
        h = torch.empty((n, self.spec.hidden_size), dtype=self.runtime.dtype, device=hidden.device)
        hc = torch.empty_like(h)
        eps = self.norm.spec.eps
        from ..kernels import ops
        ops.canon_norm(hidden, self.norm.scalar, eps, self.taps_w, state, ctx.tok_seq, ctx.cu_q, ctx.slots, h, hc)
        if ctx.max_q_len > 1:       # the state of a sequence that brings one token moved on in the launch above
            ops.canon_state(hidden, self.norm.scalar, eps, self.taps_w, state, ctx.tok_seq, ctx.cu_q, ctx.slots)
        if getattr(self.mixer, "returns_output", False):
            branch = self.mixer.forward(hc, ctx, view, None)
        else:
            branch = torch.zeros_like(hidden)
            self.mixer.forward(hc, ctx, view, branch)
        if self.ffn is not None:
            self.ffn.forward(h, ctx, branch)
        ctx.residual_sumsq = None
        ops.scaled_add(hidden, branch, self.spec.residual_mult)


class ScaledParallelBlock(Part):
    """x <- x + s1 * mixer(norm1(x)) + s2 * feed_forward(norm2(x)), then an optional part that adds to the new stream.

    Both norms read the same rows, so ``ops.dual_norm`` makes them in one pass from one sum of squares (the norms
    must be RMS norms of one eps that scale in fp32).  Each sublayer's fp32 output (a part that says
    ``returns_output`` returns it; any other adds into a zeroed buffer) is multiplied lane by lane by its stored
    vector and added in ``ops.scaled_add2``, which also leaves the new rows in the compute dtype for the part after
    (``after.wants_copy``).  Norms, scales and sums are fp32 in both compute dtypes."""

    def __init__(self, spec: ScaledParallelBlockSpec) -> None:
        super().__init__(spec)
        self.mixer_norm = build_part(spec.mixer_norm)
        self.mixer = build_part(spec.mixer)
        has = spec.ffn is not None
        if has != (spec.ffn_norm is not None) or has != (spec.ffn_scale_name is not None):
            raise ValueError("a feed-forward comes with its norm and its scale, or none of the three")
        self.ffn_norm = build_part(spec.ffn_norm) if has else None
        self.ffn = build_part(spec.ffn) if has else None
        self.after = build_part(spec.after) if spec.after is not None else None
        for norm in (spec.mixer_norm, spec.ffn_norm):
            if norm is not None and not (getattr(norm, "scale_in_fp32", False) and not getattr(norm, "scalar_weight", False)):
                raise TypeError("this block's norms are RMS norms with a weight per lane that scale in fp32")
        self.one_pass = has and spec.mixer_norm.eps == spec.ffn_norm.eps

    def _children(self):
        return tuple(part for part in (self.mixer_norm, self.mixer, self.ffn_norm, self.ffn, self.after) if part is not None)

    def tensor_decls(self):
        s = self.spec
        decls = [d for part in self._children() for d in part.tensor_decls()]
        decls.append(TensorDecl(s.mixer_scale_name, (s.hidden_size,), "one_plus_normal"))
        if self.ffn is not None:
            decls.append(TensorDecl(s.ffn_scale_name, (s.hidden_size,), "one_plus_normal"))
        return decls

    def load(self, fetch, runtime) -> None:
        self.runtime = runtime
        for part in self._children():
            part.load(fetch, runtime)
        self.mixer_scale = fetch.vector(self.spec.mixer_scale_name)
        self.ffn_scale = fetch.vector(self.spec.ffn_scale_name) if self.ffn is not None else None

    def cache_needs(self):
        return tuple(self.mixer.cache_needs())

    @property
    def graph_safe(self) -> bool:
        return all(getattr(part, "graph_safe", False) for part in self._children())

    def forward(self, hidden, ctx, view) -> None:
        from ..kernels import ops
        ctx.defers_residual_add = False        # the parts' own products add (or return) at once
        ctx.residual_sumsq = None
        if self.one_pass:
            h1 = torch.empty(hidden.shape, dtype=self.runtime.dtype, device=hidden.device)
            h2 = torch.empty_like(h1)
            ops.dual_norm(hidden, self.mixer_norm.weight, self.ffn_norm.weight, self.mixer_norm.spec.eps, h1, h2)
        else:
            h1 = self.mixer_norm(hidden)
            h2 = self.ffn_norm(hidden) if self.ffn is not None else None
        if getattr(self.mixer, "returns_output", False):
            mixed = self.mixer.forward(h1, ctx, view, None)
        else:
            mixed = torch.zeros_like(hidden)
            self.mixer.forward(h1, ctx, view, mixed)
        fed = None
        if self.ffn is not None:
            if getattr(self.ffn, "returns_output", False):
                fed = self.ffn.forward(h2, ctx, None)
            else:
                fed = torch.zeros_like(hidden)
                self.ffn.forward(h2, ctx, fed)
        ctx.residual_sumsq = None
        copy = None
        if self.after is not None and getattr(self.after, "wants_copy", False):
            copy = torch.empty(hidden.shape, dtype=self.runtime.dtype, device=hidden.device)
        ops.scaled_add2(hidden, mixed, self.mixer_scale, fed, self.ffn_scale, copy)
        if self.after is not None:
            if copy is not None:
                self.after.forward(hidden, ctx, copy)
            else:
                self.after.forward(hidden, ctx)


class StreamMixBlock(Part):
    """Parallel residual streams (hyper-connections): u = sum_s in[s] x_s; y = sublayer(norm(u)); then, all at once,
    x_t <- sum_s mix[s, t] x_s + m out[t] y; the mixer first, then the feed-forward.

    ``hidden`` is [tokens, streams * hidden].  A sublayer's fp32 output is left pending (:class:`~.linear.StreamUpdate`) and
    the next norm, of this or the following block of this kind, mixes the streams, sums its input and norms it in one
    pass (``ops.stream_mix``); the model finishes the last one.  A part that says ``returns_output`` returns its output;
    any other adds into a zeroed buffer."""

    finishes_residual_adds = True     # its norms take over an update that the block before left pending

    def __init__(self, spec: StreamMixBlockSpec) -> None:
        super().__init__(spec)
        has = spec.ffn is not None
        if has != (spec.ffn_norm is not None) or (not has and spec.ffn_names is not None):
            raise ValueError("a feed-forward comes with its norm (and perhaps its stream coefficients), or none of them")
        if spec.streams < 1 or spec.streams > STREAM_MIX_MAX_STREAMS or spec.hidden_size > STREAM_MIX_MAX_WIDTH:
            raise ValueError(f"the stream kernel takes 1 to {STREAM_MIX_MAX_STREAMS} streams of up to {STREAM_MIX_MAX_WIDTH} lanes")
        if spec.streams > 1 and (spec.mixer_names is None or (has and spec.ffn_names is None)):
            raise ValueError("several streams need their coefficients' tensors")
        self.mixer_norm = build_part(spec.mixer_norm)
        self.mixer = build_part(spec.mixer)
        self.ffn_norm = build_part(spec.ffn_norm) if has else None
        self.ffn = build_part(spec.ffn) if has else None
        for norm in (self.mixer_norm, self.ffn_norm):
            if norm is not None and not (hasattr(norm.spec, "bias_name") and norm.spec.streams == 1):
                raise TypeError("this block's norms are layer norms of one stream's width")

    def _children(self):
        return tuple(part for part in (self.mixer_norm, self.mixer, self.ffn_norm, self.ffn) if part is not None)

    def tensor_decls(self):
        s = self.spec
        decls = [d for part in self._children() for d in part.tensor_decls()]
        for named in (s.mixer_names, s.ffn_names):
            if named is not None:
                decls += [TensorDecl(named[0], (s.streams,), "one_plus_normal"), TensorDecl(named[1], (s.streams,), "one_plus_normal"),
                          TensorDecl(named[2], (s.streams, s.streams))]
        return decls

    def load(self, fetch, runtime) -> None:
        self.runtime = runtime
        for part in self._children():
            part.load(fetch, runtime)
        coefficients = lambda named: (None, None, None) if named is None else tuple(fetch.vector(name) for name in named)
        self.mixer_coef, self.ffn_coef = coefficients(self.spec.mixer_names), coefficients(self.spec.ffn_names)

    def cache_needs(self):
        return tuple(self.mixer.cache_needs())

    @property
    def graph_safe(self) -> bool:
        return all(getattr(part, "graph_safe", False) for part in self._children())

    def _half(self, hidden, ctx, part, norm, coefficients, call):
        from ..kernels import ops
        from .linear import StreamUpdate, flush_residual_add
        s = self.spec
        in_coef, out_coef, mix = coefficients
        n = hidden.shape[0]
        x = torch.empty((n, s.hidden_size), dtype=self.runtime.dtype, device=hidden.device)
        read = dict(in_coef=in_coef, weight=norm.weight, bias=norm.bias, eps=norm.spec.eps, out=x)
        pending = ctx.pending_residual_add
        if isinstance(pending, StreamUpdate) and pending.hidden is hidden:
            ctx.pending_residual_add = None
            pending.finish(**read)
        else:
            flush_residual_add(ctx)
            ops.stream_mix(hidden, streams=s.streams, **read)
        if getattr(part, "returns_output", False):
            y = call(x, None)
        else:
            y = torch.zeros((n, s.hidden_size), dtype=torch.float32, device=hidden.device)
            call(x, y)
        ctx.residual_sumsq = None
        ctx.pending_residual_add = StreamUpdate(hidden, y, s.streams, mix, out_coef, s.residual_mult)

    def forward(self, hidden, ctx, view) -> None:
        ctx.defers_residual_add = False        # the parts' own products add (or return) at once
        self._half(hidden, ctx, self.mixer, self.mixer_norm, self.mixer_coef,
                   lambda x, residual: self.mixer.forward(x, ctx, view, residual))
        if self.ffn is not None:
            self._half(hidden, ctx, self.ffn, self.ffn_norm, self.ffn_coef,
                       lambda x, residual: self.ffn.forward(x, ctx, residual))


class Reinject(Part):
    """h <- W [h ; e] + steps[index], e the embedding's output (``ctx.embedded``): what opens a pass of a looped
    stack.  It keeps no cache and returns the new stream (the model goes on with what a layer returns)."""

    graph_safe = True
    reads_embedding = True      # the model keeps the embedding's output on the step's context for it

    def tensor_decls(self):
        s = self.spec
        return [TensorDecl(s.weight_name, (s.hidden_size, 2 * s.hidden_size)),
                TensorDecl(s.steps_name, (s.num_steps, s.hidden_size))]

    def load(self, fetch, runtime) -> None:
        self.runtime = runtime
        self.weight = fetch.matrix(self.spec.weight_name)
        self.step = fetch.vector(self.spec.steps_name)[self.spec.index].contiguous()

    def cache_needs(self):
        return ()

    def forward(self, hidden, ctx, view):
        from ..kernels import ops
        from .linear import linear
        both = torch.empty((hidden.shape[0], 2 * self.spec.hidden_size), dtype=self.runtime.dtype, device=hidden.device)
        ops.concat_cast(hidden, ctx.embedded, both)
        ctx.residual_sumsq = None
        return linear(both, self.weight, bias=self.step, out_dtype=torch.float32)


register_part(PreNormBlockSpec, PreNormBlock)
register_part(SandwichBlockSpec, SandwichBlock)
register_part(GatedPostNormBlockSpec, GatedPostNormBlock)
register_part(ParallelBlockSpec, ParallelBlock)
register_part(ScaledParallelBlockSpec, ScaledParallelBlock)
register_part(StreamMixBlockSpec, StreamMixBlock)
register_part(ReinjectSpec, Reinject)
