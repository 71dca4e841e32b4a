"""Two mixers on the same input, side by side: the result is left_scale * left + right_scale * right.

Each of the two is any registered mixer and keeps what it would keep alone: the part names the needs of the left one
and then those of the right one, and hands each a view of the layer's cache with its own share (at most one of the
two may keep keys and values; fixed-size states are told apart by their order).  Both outputs are taken in fp32 (a
part that says ``returns_output`` returns it, any other adds into a zeroed buffer) and summed by ``ops.weighted_sum``.

When both say ``joins``, they share their products: one product makes the input rows of both, each writes its heads,
times its scale, to columns of its own of one buffer, and one product with the two output matrices side by side sums
them (the scales join the heads in fp32 before their one rounding).
"""

from __future__ import annotations

import torch

from ..cache import CacheView, KVNeed, StateNeed
from ..config.specs import SideBySideMixersSpec
from ..kernels import ops
from .base import Part, build_part, register_part
from .linear import linear


class SideBySideMixers(Part):
    returns_output = True   # forward(..., residual=None) returns the fp32 output instead of adding it

    def __init__(self, spec: SideBySideMixersSpec) -> None:
        super().__init__(spec)
        self.left = build_part(spec.left)
        self.right = build_part(spec.right)
        needs = [tuple(self.left.cache_needs()), tuple(self.right.cache_needs())]
        if sum(any(isinstance(n, KVNeed) for n in side) for side in needs) > 1:
            raise ValueError("only one of two mixers side by side may keep keys and values")
        self.n_left_states = sum(isinstance(n, StateNeed) for n in needs[0])

    def tensor_decls(self):
        return list(self.left.tensor_decls()) + list(self.right.tensor_decls())

    def load(self, fetch, runtime) -> None:
        self.runtime = runtime
        self.left.load(fetch, runtime)
        self.right.load(fetch, runtime)
        self.joined = bool(getattr(self.left, "joins", False) and getattr(self.right, "joins", False))
        if self.joined:
            parts = (self.left, self.right)
            self.in_cols = (0, self.left.w_in.shape[0])
            self.w_in = torch.cat([part.w_in for part in parts], 0)
            self.b_in = None
            if any(part.b_in is not None for part in parts):
                self.b_in = torch.cat([part.b_in if part.b_in is not None
                                       else torch.zeros(part.w_in.shape[0], dtype=torch.float32, device=runtime.device)
                                       for part in parts])
            # the right one's columns start on a multiple of 8; columns in between are zero on both sides of the product
            lanes = [part.w_o.shape[1] for part in parts]
            self.out_cols = (0, -(-lanes[0] // 8) * 8)
            self.out_width = self.out_cols[1] + -(-lanes[1] // 8) * 8
            self.w_o = torch.zeros((self.left.w_o.shape[0], self.out_width), dtype=runtime.dtype, device=runtime.device)
            for part, col, n in zip(parts, self.out_cols, lanes):
                self.w_o[:, col:col + n] = part.w_o
                part.w_in = part.b_in = part.w_o = None          # held once, here
            self.out_gaps = self.out_width != sum(lanes)

    def cache_needs(self):
        return tuple(self.left.cache_needs()) + tuple(self.right.cache_needs())

    @property
    def graph_safe(self) -> bool:
        return getattr(self.left, "graph_safe", False) and getattr(self.right, "graph_safe", False)

    @staticmethod
    def _share(view, states):
        return CacheView(kv_group=view.kv_group, keys=view.keys, values=view.values, writes_kv=view.writes_kv,
                         state=states[0] if states else None, states=tuple(states))

    @staticmethod
    def _output(part, x, ctx, view):
        if getattr(part, "returns_output", False):
            return part.forward(x, ctx, view, None)
        out = torch.zeros((x.shape[0], part.spec.hidden_size), dtype=torch.float32, device=x.device)
        part.forward(x, ctx, view, out)
        return out

    def forward(self, x, ctx, view, residual):
        """Adds the weighted sum to ``residual`` (fp32); with ``residual`` None returns it as a new fp32 tensor."""
        s = self.spec
        if self.joined:
            proj = linear(x, self.w_in, bias=self.b_in)
            heads = (torch.zeros if self.out_gaps else torch.empty)((x.shape[0], self.out_width), dtype=x.dtype, device=x.device)
            shares = (view.states[:self.n_left_states], view.states[self.n_left_states:])
            for part, states, col, out_col, scale in zip((self.left, self.right), shares, self.in_cols, self.out_cols,
                                                         (s.left_scale, s.right_scale)):
                part.heads_into(proj, col, ctx, self._share(view, states), heads, out_col, scale)
            if residual is None:
                return linear(heads, self.w_o, out_dtype=torch.float32)
            linear(heads, self.w_o, residual=residual, track=ctx)
            return None
        left = self._output(self.left, x, ctx, self._share(view, view.states[:self.n_left_states]))
        right = self._output(self.right, x, ctx, self._share(view, view.states[self.n_left_states:]))
        ctx.residual_sumsq = None
        ops.weighted_sum(left, left, right, s.left_scale, s.right_scale)
        if residual is None:
            return left
        ops.residual_add(residual, left)
        return None


register_part(SideBySideMixersSpec, SideBySideMixers)
