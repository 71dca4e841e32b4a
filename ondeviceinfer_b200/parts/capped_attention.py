"""Grouped-query attention with rotated, unit-normed queries and keys, squashed scores and a window.

Steps of ``forward``: one matrix product for the concatenated q, k, v projections (v heads have a width of their
own); head preparation (``csrc/capped.cu``): rotation of neighbouring-lane pairs, then every q and k head divided
by its root mean square, q to the query buffer, k and v to the token's row of the paged cache (a ring of pages
per sequence when the layer has a window); attention over the cache pages with the scores squashed by
c tanh(score / c) and keys outside the window left out (bfloat16 with heads in steps of 16:
``csrc/attention_capped_mma.cu`` on the tensor cores, a form for prompts and portions and a split-key form for
single tokens; prompts with key and value heads of 64 or 128 lanes: ``csrc/attention_tcgen05.cu``, the kernel of
the plain attention, which takes the window, the ring and the cap as arguments; float32 and other head sizes: the
CUDA-core kernel ``csrc/attention_simt.cu``); the output projection.  Rotation, unit norm, scores and
softmax are fp32 in both compute dtypes.  Optional: queries that grow slowly with the position (in the head preparation), a
learned bias of the scores by distance (a stored table of buckets, laid out at load as one number per distance), and a
sigmoid gate per head or per lane that the input product makes along with q, k and v and the attention kernels apply
on their way out.  Every constant (scale, cap, window, eps, rotated lanes, frequency
scaling) is a field of the spec; a field that is None switches its mechanism off.
"""

from __future__ import annotations

import math

import torch

from ..cache import PAGE_SIZE, KVNeed
from ..config.specs import CappedAttentionSpec
from ..kernels import ops
from ..weights.tensors import TensorDecl
from .base import Part, build_part, register_part
from .attention import TCGEN05_MIN_Q_LEN
from .linear import linear


def distance_bucket(n: int, rows: int, reach: float) -> int:
    """The row of a table of ``rows`` distance biases that a distance of n positions reads: n itself below rows / 2, then
    buckets that grow logarithmically up to ``reach``, beyond which everything is in the last one.  Host arithmetic in
    double."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(reach / half) * (rows - half)))


def distance_entries(rows: int, reach: float) -> list:
    """The buckets of the distances 0, 1, .. up to the first that reads the last row."""
    entries = []
    while not entries or entries[-1] != rows - 1:
        entries.append(distance_bucket(len(entries), rows, reach))
    return entries


class CappedAttention(Part):
    graph_safe = True   # no host work that depends on the step's values: may be captured in a CUDA graph
    returns_output = True   # forward(..., residual=None) returns the fp32 output instead of adding it
    joins = True            # may share its products with a mixer beside it

    def __init__(self, spec: CappedAttentionSpec) -> None:
        super().__init__(spec)
        if spec.num_heads <= 0 or spec.num_kv_heads <= 0 or spec.num_heads % spec.num_kv_heads != 0:
            raise ValueError("query heads must be a positive multiple of the key/value heads")
        if not 1 <= spec.head_dim <= 512:
            raise ValueError(f"head_dim={spec.head_dim}: the attention kernels take heads of up to 512 lanes")
        # the attention kernel reads heads four lanes at a time: stored q and k heads are padded with zero lanes
        self.lanes = -(-spec.head_dim // 4) * 4
        if spec.value_dim <= 0:
            raise ValueError("value_dim must be positive")
        if spec.values_are_keys and spec.value_dim != spec.head_dim:
            raise ValueError("values that are the keys have the keys' width")
        if spec.window is not None and spec.window <= 0:
            raise ValueError("window must be positive")
        if spec.softcap is not None and spec.softcap <= 0:
            raise ValueError("softcap must be positive")
        if spec.keep_first < 0 or (spec.keep_first > 0 and spec.window is None):
            raise ValueError("keep_first is a number of first positions kept beside a window")
        if spec.has("q_norm") != spec.has("k_norm") or (spec.has("q_norm") and spec.unit_norm_eps is None):
            raise ValueError("weights of the per-head norm come in a pair and go with unit_norm_eps")
        if spec.q_temperature is not None and spec.q_temperature[1] <= 0:
            raise ValueError("q_temperature: (coef, every) with a positive number of positions")
        if (spec.bias_rows > 0) != spec.has("rel") or (spec.bias_rows > 0 and (spec.bias_rows < 2 or spec.bias_reach <= spec.bias_rows // 2)):
            raise ValueError("a distance bias has a table of at least 2 rows and reaches beyond half as many positions")
        if spec.gate not in (None, "head", "lane") or (spec.gate is not None) != spec.has("g"):
            raise ValueError("gate is 'head' or 'lane' and has a tensor")
        self.position = build_part(spec.position)
        if self.position.rot_dim > 0 and not getattr(self.position, "interleaved", False):
            raise ValueError("this attention's head preparation rotates neighbouring-lane pairs only")

    # ------------------------------------------------------------------ tensors

    def tensor_decls(self):
        s = self.spec
        q, k, v = s.num_heads * s.head_dim, s.num_kv_heads * s.head_dim, s.num_kv_heads * s.value_dim
        decls = [TensorDecl(s.name("q"), (q, s.hidden_size)), TensorDecl(s.name("k"), (k, s.hidden_size))]
        if not s.values_are_keys:
            decls.append(TensorDecl(s.name("v"), (v, s.hidden_size)))
        decls.append(TensorDecl(s.name("o"), (s.hidden_size, s.num_heads * s.value_dim)))
        decls += [TensorDecl(s.name(role), (size,)) for role, size in (("q_bias", q), ("k_bias", k), ("v_bias", v)) if s.has(role)]
        decls += [TensorDecl(s.name(role), (s.head_dim,), "one_plus_normal") for role in ("q_norm", "k_norm") if s.has(role)]
        if s.gate is not None:
            decls.append(TensorDecl(s.name("g"), (self._gate_rows(), s.hidden_size)))
        if s.bias_rows > 0:
            decls.append(TensorDecl(s.name("rel"), (s.bias_rows, s.num_heads)))
        return decls + self.position.tensor_decls()

    def _gate_rows(self) -> int:
        return self.spec.num_heads * (self.spec.value_dim if self.spec.gate == "lane" else 1)

    def load(self, fetch, runtime) -> None:
        s = self.spec
        self.runtime = runtime
        # q, k, v and gate rows concatenated: one product yields [tokens, nq d + nkv d + nkv dv + gate] (no v rows when
        # the values are the keys); zero rows behind them make their number a multiple of 8
        roles = ["q", "k"] + ([] if s.values_are_keys else ["v"]) + (["g"] if s.gate is not None else [])
        rows = [fetch.matrix(s.name(role)) for role in roles]
        sizes = [len(r) for r in rows]
        self.gate_col = sum(sizes[:-1]) if s.gate is not None else None
        pad = -sum(sizes) % 8
        if pad:
            rows.append(torch.zeros((pad, s.hidden_size), dtype=rows[0].dtype, device=rows[0].device))
        self.w_in = torch.cat(rows, 0)
        self.w_o = fetch.matrix(s.name("o"))
        # biases (fp32) concatenated like their weights; rows without one add zero
        self.b_in = None
        if any(s.has(role + "_bias") for role in roles):
            zeros = lambda size: torch.zeros(size, dtype=torch.float32, device=runtime.device)
            self.b_in = torch.cat([fetch.vector(s.name(role + "_bias")) if s.has(role + "_bias") else zeros(size)
                                   for role, size in zip(roles, sizes)] + [zeros(pad)])
        self.rel = None
        if s.bias_rows > 0:       # one number per head and distance
            table = fetch.vector(s.name("rel"))
            index = torch.tensor(distance_entries(s.bias_rows, s.bias_reach), device=table.device)
            self.rel = table[index].t().contiguous()
        self.q_norm_w = fetch.vector(s.name("q_norm")) if s.has("q_norm") else None
        self.k_norm_w = fetch.vector(s.name("k_norm")) if s.has("k_norm") else None
        self.position.load(fetch, runtime)

    def cache_needs(self):
        s = self.spec
        return (KVNeed(s.num_kv_heads, self.lanes, s.window, value_dim=s.value_dim, keep_first=s.keep_first),)

    # ------------------------------------------------------------------ step

    def forward(self, x, ctx, view, residual):
        """Adds the mixer's output to ``residual`` (fp32); with ``residual`` None returns it as a new fp32 tensor."""
        s = self.spec
        o = torch.empty((x.shape[0], s.num_heads * s.value_dim), dtype=x.dtype, device=x.device)
        self.heads_into(linear(x, self.w_in, bias=self.b_in), 0, ctx, view, o, 0, 1.0)
        if residual is None:
            return linear(o, self.w_o, out_dtype=torch.float32)
        linear(o, self.w_o, residual=residual, track=ctx)
        return None

    def heads_into(self, proj, col, ctx, view, out, out_col, scale) -> None:
        """Everything between the two products: ``proj`` holds the input product from column ``col`` on, ``out`` receives
        the heads, times ``scale``, from column ``out_col`` on."""
        s = self.spec
        group = view.kv_group
        page_start, page_ids = ctx.page_table(group.index)
        tables = self.position.rotary_tables(ctx)
        cos, sin = tables if tables is not None else (None, None)
        q = torch.empty((proj.shape[0], s.num_heads * self.lanes), dtype=proj.dtype, device=proj.device)
        ops.rot_unit_prep(proj, q, view.keys, view.values, cos, sin, ctx.tok_seq,
                          ctx.tok_pos, page_start, page_ids, nq=s.num_heads, nkv=s.num_kv_heads, d=s.head_dim,
                          dv=s.value_dim, rot_dim=self.position.rot_dim, page_size=PAGE_SIZE, ring_pages=group.ring_pages,
                          write_kv=view.writes_kv, unit_eps=s.unit_norm_eps, d_store=self.lanes,
                          v_from_k=s.values_are_keys, q_weight=self.q_norm_w, k_weight=self.k_norm_w,
                          q_temperature=s.q_temperature, col=col)
        gate = None if s.gate is None else (proj, col + self.gate_col, s.gate == "head")
        self.attend(q, ctx, view, page_start, page_ids, out, dict(rel=self.rel, gate=gate, out_scale=scale, out_col=out_col))

    def attend(self, q, ctx, view, page_start, page_ids, o, way) -> None:
        """The attention's heads into ``o``; ``way``: the bias by distance, the gate, the factor and the columns (keyword
        arguments of the attention kernels)."""
        s = self.spec
        tensor_cores = ops.attention_capped_supported(q.dtype, self.lanes, s.value_dim)
        common = dict(n_seqs=ctx.n_seqs, nq=s.num_heads, nkv=s.num_kv_heads, d=self.lanes, dv=s.value_dim, page_size=PAGE_SIZE,
                      ring_pages=view.kv_group.ring_pages, window=s.window or 0, scale=s.scale, softcap=s.softcap or 0.0,
                      sink=s.sink, keep=s.keep_first, **way)
        if (tensor_cores and ctx.max_q_len > TCGEN05_MIN_Q_LEN and self.lanes == s.value_dim
                and ops.attention_tcgen05_takes(self.lanes, bias_entries=0 if self.rel is None else self.rel.shape[1],
                                                out_ld=o.shape[1], out_col=way["out_col"], gate=way["gate"])):
            # bf16 prompts with heads of 64 or 128 lanes: scores and outputs in tensor memory (tcgen05)
            ops.attention_tcgen05(q, view.keys, view.values, o, ctx.cu_q, ctx.past, page_start, page_ids, n_seqs=ctx.n_seqs,
                                  max_q_len=ctx.max_q_len, nq=s.num_heads, nkv=s.num_kv_heads, d=self.lanes, page_size=PAGE_SIZE,
                                  scale=s.scale, window=s.window or 0, ring_pages=view.kv_group.ring_pages,
                                  softcap=s.softcap or 0.0, sink=s.sink, keep=s.keep_first, **way)
            return
        if tensor_cores and ctx.max_q_len > 1 and way["out_col"] % 2 == 0 and o.shape[1] % 2 == 0:
            # other bf16 prompts and portions: the mma.sync form
            ops.attention_capped(q, view.keys, view.values, o, ctx.cu_q, ctx.past, page_start, page_ids,
                                 max_q_len=ctx.max_q_len, **common)
            return
        splits, partial = 1, None
        if ctx.max_q_len == 1:
            # single tokens: cut the visible keys so that enough blocks run side by side
            block_rows = s.num_kv_heads * ((s.num_heads // s.num_kv_heads + 15) // 16)
            keys = ctx.max_kv_len if s.window is None else min(ctx.max_kv_len, s.window + s.keep_first)
            if tensor_cores:
                tiles = (keys + 63) // 64 + (1 if s.window is not None else 0)      # a window may straddle one tile more
                tiles += 1 if s.keep_first > 0 else 0                               # and so may the kept first keys
                splits = max(1, min(32, 296 // max(ctx.n_seqs * block_rows, 1), tiles))
            else:
                splits = max(1, min(32, 296 // max(ctx.n_seqs * block_rows, 1), (keys + 255) // 256))
            if splits > 1:
                partial = torch.empty((ctx.n_tokens * s.num_heads * splits * (s.value_dim + 2),), dtype=torch.float32,
                                      device=q.device)
        if tensor_cores and ctx.max_q_len == 1:
            ops.attention_capped_decode(q, view.keys, view.values, o, ctx.cu_q, ctx.past, page_start, page_ids,
                                        splits=splits, partial=partial, **common)
            return
        ops.attention_simt(q, view.keys, view.values, o, ctx.cu_q, ctx.past, page_start, page_ids,
                           max_q_len=ctx.max_q_len, splits=splits, partial=partial, **common)


register_part(CappedAttentionSpec, CappedAttention)
