"""Retention: linear attention with a fixed decay per head, a recurrent mixer whose cache is a matrix state per head.

Steps of ``forward``: one product for q, k, v and the output gate's logits; then ``ops.retention`` (``csrc/retention.cu``:
rotation, the recurrence over each sequence's tokens, the norm of every head's read-out, silu of the gate); then the
output projection.  bfloat16 prompts take chunks of 64 tokens side by side on the tensor cores, with fp32 operands split
into two bfloat16 numbers; single tokens, short portions and float32 go through the recurrence in order.

The state [heads, qk_dim, v_dim] is fp32 rows of the cache's state group, zero when a sequence starts, advanced over all
tokens that a sequence brings in a step.  Everything between the two products is fp32.
"""

from __future__ import annotations

import torch

from ..cache import StateNeed
from ..config.specs import RetentionSpec
from ..kernels import ops
from ..weights.tensors import TensorDecl
from .base import Part, build_part, register_part
from .linear import linear


class Retention(Part):
    graph_safe = True   # no host work that depends on the step's values
    returns_output = True   # forward(..., residual=None) returns the fp32 output instead of adding it
    joins = True            # may share its products with a mixer beside it

    def __init__(self, spec: RetentionSpec) -> None:
        super().__init__(spec)
        for key in ("num_heads", "qk_dim", "v_dim"):
            if getattr(spec, key) <= 0:
                raise ValueError(f"{key} must be positive, got {getattr(spec, key)}")
        if len(spec.decay) != spec.num_heads:
            raise ValueError(f"{len(spec.decay)} decays for {spec.num_heads} heads")
        if spec.qk_dim > ops.RETENTION_MAX_DIM:
            raise ValueError(f"the retention kernels take key sizes up to {ops.RETENTION_MAX_DIM}")
        self.position = build_part(spec.position)

    def tensor_decls(self):
        s = self.spec
        qk, v = s.num_heads * s.qk_dim, s.num_heads * s.v_dim
        return [TensorDecl(s.name("q"), (qk, s.hidden_size)), TensorDecl(s.name("k"), (qk, s.hidden_size)),
                TensorDecl(s.name("v"), (v, s.hidden_size)), TensorDecl(s.name("g"), (v, s.hidden_size)),
                TensorDecl(s.name("o"), (s.hidden_size, v))] + self.position.tensor_decls()

    def load(self, fetch, runtime) -> None:
        s = self.spec
        self.runtime = runtime
        rows = [fetch.matrix(s.name(role)) for role in ("q", "k", "v", "g")]
        pad = -sum(len(r) for r in rows) % 8
        if pad:
            rows.append(torch.zeros((pad, s.hidden_size), dtype=rows[0].dtype, device=rows[0].device))
        self.w_in, self.b_in = torch.cat(rows, 0), None
        self.w_o = fetch.matrix(s.name("o"))
        self.decay = torch.tensor(s.decay, dtype=torch.float64).to(torch.float32).to(runtime.device)
        self.position.load(fetch, runtime)

    def cache_needs(self):
        s = self.spec
        return (StateNeed((s.num_heads, s.qk_dim, s.v_dim), torch.float32, "retention state"),)

    def forward(self, x, ctx, view, residual):
        """Adds the mixer's output to ``residual`` (fp32); with ``residual`` None returns it as a new fp32 tensor."""
        s = self.spec
        heads = torch.empty((x.shape[0], s.num_heads * s.v_dim), dtype=x.dtype, device=x.device)
        self.heads_into(linear(x, self.w_in), 0, ctx, view, heads, 0, 1.0)
        if residual is None:
            return linear(heads, self.w_o, out_dtype=torch.float32)
        linear(heads, self.w_o, residual=residual, track=ctx)
        return None

    def heads_into(self, proj, col, ctx, view, out, out_col, scale) -> None:
        s = self.spec
        tables = self.position.rotary_tables(ctx)
        cos, sin = tables if tables is not None else (None, None)
        ops.retention(proj, cos, sin, self.decay, view.states[0], out, ctx.cu_q, ctx.tok_seq, ctx.slots, n_seqs=ctx.n_seqs,
                      max_q_len=ctx.max_q_len, heads=s.num_heads, d=s.qk_dim, dv=s.v_dim, rot=self.position.rot_dim,
                      interleaved=bool(getattr(self.position, "interleaved", False)), eps=s.norm_eps, out_scale=scale, col=col,
                      out_col=out_col)


register_part(RetentionSpec, Retention)
