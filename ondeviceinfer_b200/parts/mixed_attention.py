"""Grouped-query attention inside chunks whose heads mix their scores before the softmax.

Mixing is folded into the queries.  The mixed score of head h is sum_g T[h, g] q_g . k_kv(g); with the query heads
grouped by their key head j this is sum_j (sum_(g in group j) T[h, g] q_g) . k_j: one query of kv_heads * head_dim lanes
per head against a position's whole key row.  So the kernels need no pass over a tile of all heads' scores; a head's
scores are one long dot product, accumulated key head by key head, and the values stay grouped.  Steps of ``forward``:

1. one product for the concatenated q, k, v projections;
2. head preparation (``csrc/mixed.cu``): the RMS norms over a token's whole q and k rows, the rotation of half-split
   pairs, the mixed queries, k and v to the token's row of the paged cache;
3. attention over the cache pages of the query's own chunk: bfloat16 on the tensor cores (``csrc/attention_mixed_mma.cu``,
   a form for prompts and portions and a split-key form for single tokens; prompts with heads of 64 or 128 lanes in
   ``csrc/attention_tcgen05.cu``), float32 and rows that those refuse on the CUDA cores (``csrc/attention_simt.cu``);
4. the output projection.

A chunk of c positions is seen by its own positions only, so a sequence's pages older than c positions are never read
again: the cache keeps a ring of pages as for a window of c.  Norms, rotation, mixing, scores and softmax are fp32 in
both compute dtypes.  Heads are stored in rows of a multiple of 16 lanes (zeros behind the head's own).
"""

from __future__ import annotations

import torch

from ..cache import PAGE_SIZE, KVNeed
from ..config.specs import MixedAttentionSpec
from ..kernels import ops
from ..weights.tensors import TensorDecl
from .attention import TCGEN05_MIN_Q_LEN
from .base import Part, build_part, register_part
from .linear import linear


class MixedAttention(Part):
    graph_safe = True   # no host work that depends on the step's values: may be captured in a CUDA graph
    returns_output = True   # forward(..., residual=None) returns the fp32 output instead of adding it

    def __init__(self, spec: MixedAttentionSpec) -> None:
        super().__init__(spec)
        if spec.num_heads <= 0 or spec.num_kv_heads <= 0 or spec.num_heads % spec.num_kv_heads != 0:
            raise ValueError("query heads must be a positive multiple of the key/value heads")
        for key in ("head_dim", "value_dim"):
            if not 1 <= getattr(spec, key) <= 512:
                raise ValueError(f"{key}={getattr(spec, key)}: the attention kernels take heads of up to 512 lanes")
        if spec.chunk is not None and spec.chunk <= 0:
            raise ValueError("chunk must be positive")
        if spec.has("q_norm") != spec.has("k_norm") or spec.has("q_norm") != (spec.row_norm_eps is not None):
            raise ValueError("the row norms' weights come in a pair and go with row_norm_eps")
        self.position = build_part(spec.position)
        if getattr(self.position, "interleaved", False):
            raise ValueError("this attention's head preparation rotates half-split pairs only")
        # stored heads are padded with zero lanes to the width the kernels read at a time
        self.lanes, self.v_lanes = (-(-d // 16) * 16 for d in (spec.head_dim, spec.value_dim))

    # ------------------------------------------------------------------ tensors

    def tensor_decls(self):
        s = self.spec
        q, k, v = s.num_heads * s.head_dim, s.num_kv_heads * s.head_dim, s.num_kv_heads * s.value_dim
        decls = [TensorDecl(s.name("q"), (q, s.hidden_size)), TensorDecl(s.name("k"), (k, s.hidden_size)),
                 TensorDecl(s.name("v"), (v, s.hidden_size)),
                 TensorDecl(s.name("o"), (s.hidden_size, s.num_heads * s.value_dim))]
        if s.has("q_norm"):
            decls += [TensorDecl(s.name("q_norm"), (q,), "one_plus_normal"), TensorDecl(s.name("k_norm"), (k,), "one_plus_normal")]
        if s.has("talk"):
            decls.append(TensorDecl(s.name("talk"), (s.num_heads, s.num_heads)))
        return decls + self.position.tensor_decls()

    def load(self, fetch, runtime) -> None:
        s = self.spec
        self.runtime = runtime
        self.w_qkv = torch.cat([fetch.matrix(s.name(r)) for r in ("q", "k", "v")], 0)
        w_o = fetch.matrix(s.name("o"))
        if self.v_lanes != s.value_dim:      # the columns of the heads' padding lanes are zero
            padded = torch.zeros((s.hidden_size, s.num_heads, self.v_lanes), dtype=w_o.dtype, device=w_o.device)
            padded[:, :, :s.value_dim] = w_o.view(s.hidden_size, s.num_heads, s.value_dim)
            w_o = padded.view(s.hidden_size, s.num_heads * self.v_lanes)
        self.w_o = w_o
        self.q_norm, self.k_norm = (fetch.vector(s.name(r)) if s.has(r) else None for r in ("q_norm", "k_norm"))
        self.talk = fetch.vector(s.name("talk")) if s.has("talk") else None      # fp32 [heads, heads]
        self.position.load(fetch, runtime)

    def cache_needs(self):
        s = self.spec
        return (KVNeed(s.num_kv_heads, self.lanes, s.chunk, value_dim=self.v_lanes),)

    # ------------------------------------------------------------------ step

    def forward(self, x, ctx, view, residual):
        """Adds the mixer's output to ``residual`` (fp32); with ``residual`` None returns it as a new fp32 tensor."""
        s = self.spec
        n = x.shape[0]
        group = view.kv_group
        page_start, page_ids = ctx.page_table(group.index)
        tables = self.position.rotary_tables(ctx)
        cos, sin = tables if tables is not None else (None, None)
        width = self.lanes * (s.num_kv_heads if self.talk is not None else 1)
        q = torch.empty((n, s.num_heads * width), dtype=x.dtype, device=x.device)
        ops.mixed_prep(linear(x, self.w_qkv), q, view.keys, view.values, self.q_norm, self.k_norm, self.talk, cos, sin,
                       ctx.tok_seq, ctx.tok_pos, page_start, page_ids, nq=s.num_heads, nkv=s.num_kv_heads, d=s.head_dim,
                       dv=s.value_dim, lanes=self.lanes, v_lanes=self.v_lanes, rot_dim=self.position.rot_dim,
                       page_size=PAGE_SIZE, ring_pages=group.ring_pages, write_kv=view.writes_kv,
                       eps=s.row_norm_eps if s.row_norm_eps is not None else 0.0)
        o = self.attend(q, ctx, view, page_start, page_ids)
        if residual is None:
            return linear(o, self.w_o, out_dtype=torch.float32)
        linear(o, self.w_o, residual=residual, track=ctx)
        return None

    def attend(self, q, ctx, view, page_start, page_ids):
        """The attention output [tokens, heads * v_lanes]."""
        s = self.spec
        mixed = self.talk is not None
        o = torch.empty((ctx.n_tokens, s.num_heads * self.v_lanes), dtype=q.dtype, device=q.device)
        where = (q, view.keys, view.values, o, ctx.cu_q, ctx.past, page_start, page_ids)
        common = dict(n_seqs=ctx.n_seqs, nq=s.num_heads, nkv=s.num_kv_heads, d=self.lanes, page_size=PAGE_SIZE,
                      ring_pages=view.kv_group.ring_pages, chunk=s.chunk or 0, scale=s.scale, mixed=mixed)
        keys = ctx.max_kv_len if s.chunk is None else min(ctx.max_kv_len, s.chunk)
        tensor_cores = ops.attention_mixed_supported(q.dtype, self.lanes, self.v_lanes, s.num_kv_heads, mixed)
        splits, partial = 1, None
        if ctx.max_q_len == 1:
            # single tokens: cut the visible keys so that enough blocks run side by side (a chunk may straddle a tile more)
            if tensor_cores:
                rows, tiles = (s.num_heads + 15) // 16, (keys + 63) // 64 + (1 if s.chunk is not None else 0)
            else:
                rows, tiles = s.num_kv_heads * ((s.num_heads // s.num_kv_heads + 15) // 16), (keys + 255) // 256
            splits = max(1, min(32, 296 // max(ctx.n_seqs * rows, 1), tiles))
            if splits > 1:
                partial = torch.empty((ctx.n_tokens * s.num_heads * splits * (self.v_lanes + 2),), dtype=torch.float32,
                                      device=q.device)
        if (tensor_cores and ctx.max_q_len > TCGEN05_MIN_Q_LEN and self.lanes == self.v_lanes
                and (ops.attention_tcgen05_mixed_rows(self.lanes, s.num_kv_heads) > 0 if mixed
                     else self.lanes in ops.TCGEN05_ATTENTION_HEAD_DIMS)):
            # bf16 prompts with heads of 64 or 128 lanes: scores and outputs in tensor memory
            ops.attention_tcgen05(*where, max_q_len=ctx.max_q_len, **common)
        elif tensor_cores:
            ops.attention_mixed(*where, max_q_len=ctx.max_q_len, dv=self.v_lanes, splits=splits, partial=partial, **common)
        else:
            ops.attention_simt(*where, max_q_len=ctx.max_q_len, window=0, dv=self.v_lanes, splits=splits, partial=partial, **common)
        return o


register_part(MixedAttentionSpec, MixedAttention)
