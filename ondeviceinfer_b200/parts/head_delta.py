"""The gated delta rule with one decay per head: a recurrent mixer whose cache is a matrix state per head and the last
inputs of its short convolutions.

Steps of ``forward``: one product for q, k, v (before their convolutions) and the output gate's logits; one, fp32 out,
for the decay's and the step size's inner terms (what enters the recurrence besides q, k and v stays in 32 bits); then
``ops.head_delta`` (``csrc/delta_head.cu``: convolutions with SiLU and their state, unit vectors, decays, the recurrence
over each sequence's tokens in order, four at a time, the per-head norm of the read-outs times silu of the gate); then
the output projection.

The state [heads, qk_dim, v_dim] and the convolution inputs [taps - 1, channels] are fp32 rows of the cache's state
groups, zero when a sequence starts, advanced over all tokens a sequence brings in a step.
"""

from __future__ import annotations

import torch

from ..cache import StateNeed
from ..config.specs import HeadDeltaSpec
from ..kernels import ops
from ..weights.tensors import TensorDecl
from .base import Part, register_part
from .linear import linear


class HeadDelta(Part):
    graph_safe = True   # no host work that depends on the step's values
    returns_output = True   # forward(..., residual=None) returns the fp32 output instead of adding it

    def __init__(self, spec: HeadDeltaSpec) -> None:
        super().__init__(spec)
        for key in ("num_heads", "num_kv_heads", "qk_dim", "v_dim", "conv_taps"):
            if getattr(spec, key) <= 0:
                raise ValueError(f"{key} must be positive, got {getattr(spec, key)}")
        if spec.num_heads % spec.num_kv_heads != 0:
            raise ValueError("heads must be divisible by kv_heads")
        if spec.conv_taps > ops.HEAD_DELTA_MAX_TAPS or spec.qk_dim > ops.HEAD_DELTA_MAX_DIM:
            raise ValueError(f"the delta rule kernels take up to {ops.HEAD_DELTA_MAX_TAPS} taps and key sizes up to "
                             f"{ops.HEAD_DELTA_MAX_DIM}")
        self.qk_channels = spec.num_kv_heads * spec.qk_dim
        self.v_channels = spec.num_heads * spec.v_dim
        self.channels = 2 * self.qk_channels + self.v_channels

    def tensor_decls(self):
        s = self.spec
        H, qk, v = s.hidden_size, self.qk_channels, self.v_channels
        return [TensorDecl(s.name("q"), (qk, H)), TensorDecl(s.name("q_conv"), (qk, s.conv_taps)),
                TensorDecl(s.name("k"), (qk, H)), TensorDecl(s.name("k_conv"), (qk, s.conv_taps)),
                TensorDecl(s.name("v"), (v, H)), TensorDecl(s.name("v_conv"), (v, s.conv_taps)),
                TensorDecl(s.name("b"), (s.num_heads, H)), TensorDecl(s.name("A_log"), (s.num_heads,)),
                TensorDecl(s.name("norm"), (s.v_dim,), "one_plus_normal"), TensorDecl(s.name("a"), (s.num_heads, H)),
                TensorDecl(s.name("dt_bias"), (s.num_heads,)), TensorDecl(s.name("g"), (v, H)),
                TensorDecl(s.name("o"), (H, v))]

    def load(self, fetch, runtime) -> None:
        s = self.spec
        self.runtime = runtime
        self.w_in = torch.cat([fetch.matrix(s.name(r)) for r in ("q", "k", "v", "g")], 0)
        self.w_ab = torch.cat([fetch.matrix(s.name(r)) for r in ("a", "b")], 0)
        self.taps = torch.cat([fetch.vector(s.name(r)) for r in ("q_conv", "k_conv", "v_conv")], 0).t().contiguous()
        self.a_log = fetch.vector(s.name("A_log"))
        self.dt_bias = fetch.vector(s.name("dt_bias"))
        self.out_norm = fetch.vector(s.name("norm"))
        self.w_o = fetch.matrix(s.name("o"))

    def cache_needs(self):
        s = self.spec
        needs = [StateNeed((s.num_heads, s.qk_dim, s.v_dim), torch.float32, "delta state")]
        if s.conv_taps > 1:
            needs.append(StateNeed((s.conv_taps - 1, self.channels), torch.float32, "convolution inputs"))
        return tuple(needs)

    def forward(self, x, ctx, view, residual):
        """Adds the mixer's output to ``residual`` (fp32); with ``residual`` None returns it as a new fp32 tensor."""
        s = self.spec
        proj = linear(x, self.w_in)
        ab = linear(x, self.w_ab, out_dtype=torch.float32)
        out = torch.empty((x.shape[0], self.v_channels), dtype=proj.dtype, device=proj.device)
        ops.head_delta(proj, ab, self.taps, self.a_log, self.dt_bias, self.out_norm,
                       view.states[1] if s.conv_taps > 1 else None, view.states[0], out, ctx.cu_q, ctx.tok_seq, ctx.slots,
                       n_seqs=ctx.n_seqs, max_q_len=ctx.max_q_len, heads=s.num_heads, kv_heads=s.num_kv_heads, d=s.qk_dim,
                       dv=s.v_dim, eps=s.norm_eps, unit_eps=s.unit_eps)
        if residual is None:
            return linear(out, self.w_o, out_dtype=torch.float32)
        linear(out, self.w_o, residual=residual, track=ctx)
        return None


register_part(HeadDeltaSpec, HeadDelta)
