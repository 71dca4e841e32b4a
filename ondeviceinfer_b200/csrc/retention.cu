// Retention: linear attention with a fixed decay per head, for ragged batches of token runs; what lies between the mixer's
// input product and its output product.
//
// Per sequence and head, with q and k rotated, k scaled, and the state S [d, dv] (fp32, zero at the start):
//     S <- g S + k v^T;   o = S^T q
// then o / sqrt(mean(o^2) + eps) * silu(gate), times a constant, rounded once to T.  Everything between the two products
// is fp32: the tensor-core forms split their fp32 operands into two bf16 numbers each (a high and a low part) and add the
// products that matter (high x high, high x low, low x high), which keeps about 16 bits of every factor; values come from
// the projection in bf16 and need no split.
//
// Two forms:
//  * single tokens, short portions and float32: `step` (one token per sequence: a block per sequence and head streams the
//    state through registers once, and finishes the head) and `walk` (a block per sequence, head and block of columns keeps
//    its part of the state in shared memory and takes the tokens in order; `finish` norms and gates);
//  * bf16 prompts: chunks of 64 tokens side by side.  With g_n = g^n and i, j counted inside a chunk of L tokens,
//        U_c = sum_j g_(L-1-j) k_j v_j^T                                   (`chunk_sums`, all chunks at once)
//        S_c = g_L S_(c-1) + U_(c-1)                                       (`chunk_scan`, elementwise over the chunks)
//        o_i = g_(i+1) S_c^T q_i + sum_(j<=i) g_(i-j) (q_i . k_j) v_j      (`chunk_outputs`, all chunks at once)
//    (only products of decays, never a quotient).
#include "common.cuh"

#define RT_CHUNK 64

struct RetentionArgs {
  const void* proj;       // [n_tokens, ld] in T, from this mixer's first column on: q (H d), k (H d), v (H dv), gate (H dv)
  const float* cos_t;     // null: no rotation; [n_tokens, rot / 2]
  const float* sin_t;
  const float* decay;     // [heads]
  float* state;           // [slots, heads, d, dv]
  float* chunks;          // chunk form: [n_tokens / 64 + n_seqs, heads, d, dv] scratch
  float* o;               // walk form: [n_tokens, heads dv] scratch
  void* out;              // [n_tokens, out_ld] in T, from this mixer's first column on
  const int* cu_q;
  const int* tok_seq;
  const int* slots;
  int n_tokens, n_seqs, max_q_len, ld, heads, d, dv, rot, interleaved, out_ld, norm;
  float eps, k_scale, out_scale;
};

// Lane i of a head's row after the rotation.
template <typename T>
__device__ __forceinline__ float rt_lane(const RetentionArgs& a, const T* row, int i, int t) {
  const float x = to_f<T>(row[i]);
  if (i >= a.rot) return x;
  const int half = a.rot >> 1;
  int pair, other;
  bool first;
  if (a.interleaved) { pair = i >> 1; first = !(i & 1); other = i ^ 1; }
  else { first = i < half; pair = first ? i : i - half; other = first ? i + half : i - half; }
  const float cs = a.cos_t[(size_t)t * half + pair], sn = a.sin_t[(size_t)t * half + pair], y = to_f<T>(row[other]);
  return first ? fmaf(-y, sn, x * cs) : fmaf(y, sn, x * cs);
}

// Eight neighbouring lanes (bf16, aligned rows; a rotation in halves whose halves are multiples of 8 lanes, or none).
__device__ __forceinline__ void rt_unpack8(const uint4 raw, float* v) {
  const __nv_bfloat162* h = (const __nv_bfloat162*)&raw;
#pragma unroll
  for (int e = 0; e < 4; ++e) { const float2 f = __bfloat1622float2(h[e]); v[2 * e] = f.x; v[2 * e + 1] = f.y; }
}
__device__ __forceinline__ void rt_lanes8(const RetentionArgs& a, const bf16* row, int i, int t, float* v) {
  rt_unpack8(*(const uint4*)(row + i), v);
  if (i >= a.rot) return;
  const int half = a.rot >> 1;
  const bool first = i < half;
  const int pair = first ? i : i - half;
  float y[8], cs[8], sn[8];
  rt_unpack8(*(const uint4*)(row + (first ? i + half : i - half)), y);
  const float4* cp = (const float4*)(a.cos_t + (size_t)t * half + pair);
  const float4* sp = (const float4*)(a.sin_t + (size_t)t * half + pair);
  const float4 c0 = cp[0], c1 = cp[1], s0 = sp[0], s1 = sp[1];
  cs[0] = c0.x; cs[1] = c0.y; cs[2] = c0.z; cs[3] = c0.w; cs[4] = c1.x; cs[5] = c1.y; cs[6] = c1.z; cs[7] = c1.w;
  sn[0] = s0.x; sn[1] = s0.y; sn[2] = s0.z; sn[3] = s0.w; sn[4] = s1.x; sn[5] = s1.y; sn[6] = s1.z; sn[7] = s1.w;
#pragma unroll
  for (int e = 0; e < 8; ++e) v[e] = first ? fmaf(-y[e], sn[e], v[e] * cs[e]) : fmaf(y[e], sn[e], v[e] * cs[e]);
}

// g^n by squaring (n < 2^16; 0^0 = 1).
__device__ __forceinline__ float rt_power(float g, int n) {
  float r = 1.f;
  for (; n > 0; n >>= 1) { if (n & 1) r *= g; g *= g; }
  return r;
}

__device__ __forceinline__ float rt_silu(float z) { return z / (1.f + expf(-z)); }

// ------------------------------------------------------------------------------ one token per sequence

// V columns a thread per access; threads tid / (dv / V) take the rows in turn.
template <typename T, int V>
__global__ void __launch_bounds__(256)
rt_step_kernel(RetentionArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float rt_smem[];
  __shared__ float scratch[33];
  const int h = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x, d = a.d, dv = a.dv;
  const int t = a.cu_q[seq], slot = a.slots[seq];
  float* qs = rt_smem;                   // [d]
  float* ks = qs + d;                    // [d]
  float* part = ks + d + ((4 - (2 * d & 3)) & 3);      // [row groups][columns], aligned
  const T* base = (const T*)a.proj + (size_t)t * a.ld;
  for (int i = tid; i < 2 * d; i += blockDim.x) {
    const bool is_k = i >= d;
    const T* row = base + (size_t)((is_k ? a.heads : 0) + h) * d;
    const float x = rt_lane<T>(a, row, is_k ? i - d : i, t);
    if (is_k) ks[i - d] = x * a.k_scale; else qs[i] = x;
  }
  const T* v_row = base + (size_t)2 * a.heads * d + (size_t)h * dv;
  const T* gate = v_row + (size_t)a.heads * dv;
  float* S = a.state + ((size_t)slot * a.heads + h) * d * dv;
  const float g = a.decay[h];
  __syncthreads();
  // columns in passes of at most `cols` accesses, so that every thread has one
  const int nc = (dv + V - 1) / V, cols = min(nc, (int)blockDim.x), groups = blockDim.x / cols;
  float ss = 0.f;
  for (int c0 = 0; c0 < nc; c0 += cols) {
    const int c = c0 + tid % cols, grp = tid / cols;
    const bool live = c < nc && grp < groups;
    float o[V] = {}, v[V];
    if (live) {
#pragma unroll
      for (int e = 0; e < V; ++e) v[e] = to_f<T>(v_row[c * V + e]);
#pragma unroll 8
      for (int r = grp; r < d; r += groups) {
        float* p = S + (size_t)r * dv + c * V;
        float x[V];
        if (V == 4) { const float4 f = *(const float4*)p; x[0] = f.x; x[1 % V] = f.y; x[2 % V] = f.z; x[3 % V] = f.w; }
        else x[0] = p[0];
        const float k = ks[r], q = qs[r];
#pragma unroll
        for (int e = 0; e < V; ++e) { x[e] = fmaf(g, x[e], k * v[e]); o[e] = fmaf(q, x[e], o[e]); }
        if (V == 4) *(float4*)p = make_float4(x[0], x[1 % V], x[2 % V], x[3 % V]);
        else p[0] = x[0];
      }
#pragma unroll
      for (int e = 0; e < V; ++e) part[((size_t)grp * nc + c) * V + e] = o[e];
    }
  }
  __syncthreads();
  for (int i = tid; i < dv; i += blockDim.x) {
    float x = part[i];
    for (int r = 1; r < groups; ++r) x += part[(size_t)r * nc * V + i];
    part[i] = x;
    ss = fmaf(x, x, ss);
  }
  float inv = a.out_scale;
  if (a.norm) inv *= 1.0f / sqrtf(block_sum(ss, scratch) / (float)dv + a.eps);
  T* out = (T*)a.out + (size_t)t * a.out_ld + (size_t)h * dv;
  for (int i = tid; i < dv; i += blockDim.x) out[i] = from_f<T>(part[i] * inv * rt_silu(to_f<T>(gate[i])));
}

// ------------------------------------------------------------------------------ tokens in order

#define RT_WALK_TOKENS 16

// A thread keeps rows tid / CB, tid / CB + groups, .. of one of the block's CB columns.
template <typename T>
__global__ void __launch_bounds__(256)
rt_walk_kernel(RetentionArgs a, int CB) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float rt_smem[];
  const int h = blockIdx.y, seq = blockIdx.z, tid = threadIdx.x, d = a.d, dv = a.dv, c0 = blockIdx.x * CB;
  const int q_begin = a.cu_q[seq], q_len = a.cu_q[seq + 1] - q_begin, slot = a.slots[seq];
  if (q_len <= 0) return;
  const int groups = 256 / CB, col = tid % CB, grp = tid / CB;
  float* S = rt_smem;                                     // [d][CB]
  float* qs = S + (size_t)d * CB;                         // [tokens][d]
  float* ks = qs + RT_WALK_TOKENS * d;
  float* vs = ks + RT_WALK_TOKENS * d;                    // [tokens][CB]
  float* part = vs + RT_WALK_TOKENS * CB;                 // [tokens][256]
  float* S_g = a.state + ((size_t)slot * a.heads + h) * d * dv;
  const bool live = c0 + col < dv;
  for (int r = grp; r < d; r += groups) S[r * CB + col] = live ? S_g[(size_t)r * dv + c0 + col] : 0.f;
  const float g = a.decay[h];
  for (int base = 0; base < q_len; base += RT_WALK_TOKENS) {
    const int nt = min(RT_WALK_TOKENS, q_len - base);
    __syncthreads();
    for (int i = tid; i < nt * 2 * d; i += 256) {
      const int tt = i / (2 * d), e = i % (2 * d), t = q_begin + base + tt;
      const bool is_k = e >= d;
      const T* row = (const T*)a.proj + (size_t)t * a.ld + (size_t)((is_k ? a.heads : 0) + h) * d;
      const float x = rt_lane<T>(a, row, is_k ? e - d : e, t);
      if (is_k) ks[tt * d + e - d] = x * a.k_scale; else qs[tt * d + e] = x;
    }
    for (int i = tid; i < nt * CB; i += 256) {
      const int tt = i / CB, c = c0 + i % CB;
      vs[i] = c < dv ? to_f<T>(((const T*)a.proj)[(size_t)(q_begin + base + tt) * a.ld + (size_t)2 * a.heads * d + (size_t)h * dv + c]) : 0.f;
    }
    __syncthreads();
    for (int tt = 0; tt < nt; ++tt) {
      const float v = vs[tt * CB + col];
      float o = 0.f;
#pragma unroll 4
      for (int r = grp; r < d; r += groups) {
        const float x = fmaf(g, S[r * CB + col], ks[tt * d + r] * v);
        S[r * CB + col] = x;
        o = fmaf(qs[tt * d + r], x, o);
      }
      part[tt * 256 + tid] = o;
    }
    __syncthreads();
    for (int i = tid; i < nt * CB; i += 256) {
      const int tt = i / CB, c = i % CB;
      float x = 0.f;
      for (int r = 0; r < groups; ++r) x += part[tt * 256 + r * CB + c];
      if (c0 + c < dv) a.o[(size_t)(q_begin + base + tt) * a.heads * dv + (size_t)h * dv + c0 + c] = x;
    }
  }
  if (live)
    for (int r = grp; r < d; r += groups) S_g[(size_t)r * dv + c0 + col] = S[r * CB + col];
}

// One warp per (token, head): norm, gate, constant.
template <typename T>
__global__ void __launch_bounds__(128)
rt_finish_kernel(RetentionArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31, dv = a.dv;
  const long item = (long)blockIdx.x * 4 + (threadIdx.x >> 5);
  if (item >= (long)a.n_tokens * a.heads) return;
  const size_t t = item / a.heads;
  const int h = (int)(item % a.heads);
  const float* o = a.o + item * dv;
  const T* gate = (const T*)a.proj + t * a.ld + (size_t)2 * a.heads * a.d + (size_t)(a.heads + h) * dv;
  T* out = (T*)a.out + t * a.out_ld + (size_t)h * dv;
  float ss = 0.f;
  for (int i = lane; i < dv; i += 32) ss = fmaf(o[i], o[i], ss);
  ss = warp_sum(ss);
  const float inv = a.norm ? a.out_scale / sqrtf(ss / (float)dv + a.eps) : a.out_scale;
  for (int i = lane; i < dv; i += 32) out[i] = from_f<T>(o[i] * inv * rt_silu(to_f<T>(gate[i])));
}

// ------------------------------------------------------------------------------ chunks of 64 tokens on the tensor cores

__device__ __forceinline__ uint32_t rt_addr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void rt_ldm(uint32_t addr, uint32_t* r) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void rt_ldm_trans(uint32_t addr, uint32_t* r) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void rt_mma(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// x = high + low, two bf16 numbers
__device__ __forceinline__ void rt_split2(float x, float y, uint32_t& high, uint32_t& low) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const float2 f = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(x - f.x, y - f.y);
  high = *(const uint32_t*)&h;
  low = *(const uint32_t*)&l;
}

// Which tokens chunk `c` of sequence `seq` has, and where its state lies in the scratch: sequences take the places from
// cu_q / 64 + their number on, which no two share.
__device__ __forceinline__ bool rt_chunk(const RetentionArgs& a, int seq, int c, int& t0, int& n, size_t& place) {
  const int q_begin = a.cu_q[seq], q_len = a.cu_q[seq + 1] - q_begin;
  if (c * RT_CHUNK >= q_len) return false;
  t0 = q_begin + c * RT_CHUNK;
  n = min(RT_CHUNK, q_len - c * RT_CHUNK);
  place = (size_t)(q_begin / RT_CHUNK + seq + c);
  return true;
}

// One head's q or k rows of a chunk, rotated and times `scale` (and g^(n-1-row) with `weights`), split, into
// [64][W] rows of high and low parts; lanes from d on and rows from n on are zero.
__device__ __forceinline__ void rt_stage_rows(const RetentionArgs& a, bf16* high, bf16* low, int W, const bf16* src, int t0, int n,
                                              float scale, const float* weights, int vec, int tid, int threads) {
  const int d16 = (a.d + 15) & ~15;
  const int pieces = d16 / 8;
  for (int i = tid; i < RT_CHUNK * pieces; i += threads) {
    const int r = i / pieces, e0 = 8 * (i % pieces);
    float v[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] = 0.f;
    if (r < n) {
      const bf16* row = src + (size_t)(t0 + r) * a.ld;
      if (vec) { if (e0 < a.d) rt_lanes8(a, row, e0, t0 + r, v); }
      else {
#pragma unroll
        for (int e = 0; e < 8; ++e) if (e0 + e < a.d) v[e] = rt_lane<bf16>(a, row, e0 + e, t0 + r);
      }
      const float w = weights != nullptr ? scale * weights[n - 1 - r] : scale;
#pragma unroll
      for (int e = 0; e < 8; ++e) v[e] *= w;
    }
    uint4 hi, lo;
    rt_split2(v[0], v[1], hi.x, lo.x); rt_split2(v[2], v[3], hi.y, lo.y);
    rt_split2(v[4], v[5], hi.z, lo.z); rt_split2(v[6], v[7], hi.w, lo.w);
    *(uint4*)(high + r * W + e0) = hi;
    *(uint4*)(low + r * W + e0) = lo;
  }
}

// `cols` columns (a multiple of 16) of the head's values from column c0 on into [64][W] rows; the rest is zero.
__device__ __forceinline__ void rt_stage_values(const RetentionArgs& a, bf16* dst, int W, int c0, int cols, const bf16* src, int t0,
                                                int n, int vec, int tid, int threads) {
  const int pieces = cols / 8;
  for (int i = tid; i < RT_CHUNK * pieces; i += threads) {
    const int r = i / pieces, e0 = 8 * (i % pieces);
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (r < n) {
      const bf16* row = src + (size_t)(t0 + r) * a.ld;
      if (vec) { if (c0 + e0 < a.dv) v = *(const uint4*)(row + c0 + e0); }
      else {
        bf16* p = (bf16*)&v;
#pragma unroll
        for (int e = 0; e < 8; ++e) if (c0 + e0 + e < a.dv) p[e] = row[c0 + e0 + e];
      }
    }
    *(uint4*)(dst + r * W + e0) = v;
  }
}

#define RT_CB 64            // columns of the values per block of chunk_sums and per turn of chunk_outputs

// U of a chunk, RT_CB columns of it: rows are key lanes, 16 a warp at a time.
__global__ void __launch_bounds__(256)
rt_chunk_sums_kernel(RetentionArgs a, int vec) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) uint8_t rt_bytes[];
  __shared__ float pw[RT_CHUNK + 1];
  const int seq = blockIdx.z, col_blocks = (a.dv + RT_CB - 1) / RT_CB;
  const int h = blockIdx.y / col_blocks, c0 = blockIdx.y % col_blocks * RT_CB;
  int t0, n;
  size_t place;
  if (!rt_chunk(a, seq, blockIdx.x, t0, n, place)) return;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, d16 = (a.d + 15) & ~15, WK = d16 + 8, WV = RT_CB + 8;
  bf16* kh = (bf16*)rt_bytes;
  bf16* kl = kh + RT_CHUNK * WK;
  bf16* vs = kl + RT_CHUNK * WK;
  if (tid <= RT_CHUNK) pw[tid] = rt_power(a.decay[h], tid);
  __syncthreads();
  const bf16* base = (const bf16*)a.proj;
  rt_stage_rows(a, kh, kl, WK, base + (size_t)(a.heads + h) * a.d, t0, n, a.k_scale, pw, vec, tid, 256);
  rt_stage_values(a, vs, WV, c0, RT_CB, base + (size_t)2 * a.heads * a.d + (size_t)h * a.dv, t0, n, vec, tid, 256);
  __syncthreads();
  float* U = a.chunks + (place * a.heads + h) * a.d * a.dv;
  const int m = lane >> 3, r = lane & 7;
  for (int row0 = warp * 16; row0 < d16; row0 += 8 * 16) {
    float acc[RT_CB / 8][4] = {};
#pragma unroll
    for (int kk = 0; kk < RT_CHUNK / 16; ++kk) {
      // A = k^T: matrices (lanes row0 .. + 7, tokens kk*16 .. + 7), (lanes + 8, same tokens), (lanes, tokens + 8), (both + 8)
      uint32_t ah[4], al[4];
      const int at = (kk * 16 + (m >> 1) * 8 + r) * WK + row0 + (m & 1) * 8;
      rt_ldm_trans(rt_addr(kh + at), ah);
      rt_ldm_trans(rt_addr(kl + at), al);
#pragma unroll
      for (int np = 0; np < RT_CB / 16; ++np) {
        uint32_t b[4];
        rt_ldm_trans(rt_addr(vs + (kk * 16 + (m & 1) * 8 + r) * WV + np * 16 + (m >> 1) * 8), b);
        rt_mma(acc[2 * np], ah, b[0], b[1]);
        rt_mma(acc[2 * np], al, b[0], b[1]);
        rt_mma(acc[2 * np + 1], ah, b[2], b[3]);
        rt_mma(acc[2 * np + 1], al, b[2], b[3]);
      }
    }
    const int lo = row0 + (lane >> 2), c = c0 + (lane & 3) * 2;
    const bool pair = (a.dv & 1) == 0;
#pragma unroll
    for (int i = 0; i < RT_CB / 8; ++i) {
      const int cc = c + 8 * i;
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int row = lo + 8 * half;
        if (row >= a.d || cc >= a.dv) continue;
        float* dst = U + (size_t)row * a.dv + cc;
        if (pair) *(float2*)dst = make_float2(acc[i][2 * half], acc[i][2 * half + 1]);
        else { dst[0] = acc[i][2 * half]; if (cc + 1 < a.dv) dst[1] = acc[i][2 * half + 1]; }
      }
    }
  }
}

// The state in front of every chunk in place of its sum, and the sequence's new state.
template <int V>
__global__ void __launch_bounds__(128)
rt_chunk_scan_kernel(RetentionArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int seq = blockIdx.z, h = blockIdx.y, size = a.d * a.dv;
  const int i = V * (blockIdx.x * blockDim.x + threadIdx.x);
  if (i >= size) return;
  const int q_begin = a.cu_q[seq], q_len = a.cu_q[seq + 1] - q_begin;
  if (q_len <= 0) return;
  const int n_chunks = (q_len + RT_CHUNK - 1) / RT_CHUNK;
  const size_t step = (size_t)a.heads * size;
  float* p = a.chunks + ((size_t)(q_begin / RT_CHUNK + seq) * a.heads + h) * size + i;
  float* st = a.state + ((size_t)a.slots[seq] * a.heads + h) * size + i;
  const float g = a.decay[h], gc = rt_power(g, RT_CHUNK), gl = rt_power(g, q_len - (n_chunks - 1) * RT_CHUNK);
  float S[V];
  auto load = [&](const float* src, float* v) {
    if (V == 4) { const float4 f = *(const float4*)src; v[0] = f.x; v[1 % V] = f.y; v[2 % V] = f.z; v[3 % V] = f.w; }
    else v[0] = src[0];
  };
  auto store = [&](float* dst, const float* v) {
    if (V == 4) *(float4*)dst = make_float4(v[0], v[1 % V], v[2 % V], v[3 % V]);
    else dst[0] = v[0];
  };
  load(st, S);
  int c = 0;
  for (; c + 8 < n_chunks; c += 8) {            // eight loads in flight
    float u[8][V];
#pragma unroll
    for (int j = 0; j < 8; ++j) load(p + (size_t)(c + j) * step, u[j]);
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      store(p + (size_t)(c + j) * step, S);
#pragma unroll
      for (int e = 0; e < V; ++e) S[e] = fmaf(gc, S[e], u[j][e]);
    }
  }
  for (; c < n_chunks; ++c) {
    float u[V];
    load(p + (size_t)c * step, u);
    store(p + (size_t)c * step, S);
    const float w = c + 1 < n_chunks ? gc : gl;
#pragma unroll
    for (int e = 0; e < V; ++e) S[e] = fmaf(w, S[e], u[e]);
  }
  store(st, S);
}

// The read-outs of a chunk's tokens for one head: 8 warps, warp w takes token rows 16 (w % 4) .. + 15 and half w / 4 of the
// keys (scores) and of the columns of a turn (read-outs).
__global__ void __launch_bounds__(256)
rt_chunk_outputs_kernel(RetentionArgs a, int vec) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) uint8_t rt_bytes[];
  __shared__ float pw[RT_CHUNK + 1], sums[2][RT_CHUNK];
  const int seq = blockIdx.z, h = blockIdx.y;
  int t0, n;
  size_t place;
  if (!rt_chunk(a, seq, blockIdx.x, t0, n, place)) return;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, d = a.d, dv = a.dv, d16 = (d + 15) & ~15, WQ = d16 + 8;
  constexpr int WV = RT_CB + 8, WP = RT_CHUNK + 8;
  const int turns = (dv + RT_CB - 1) / RT_CB, WO = turns * RT_CB + 4;
  bf16* qh = (bf16*)rt_bytes;                      // q, high and low [64][WQ]
  bf16* ql = qh + RT_CHUNK * WQ;
  bf16* ph = ql + RT_CHUNK * WQ;                   // decayed scores [64][WP]
  bf16* pl = ph + RT_CHUNK * WP;
  bf16* vs = pl + RT_CHUNK * WP;                   // a turn's values [64][WV]
  bf16* un = vs + RT_CHUNK * WV;                   // k [64][WQ] twice, then a turn's state [d16][WV] twice
  const int un_elems = max(2 * RT_CHUNK * WQ, 2 * d16 * WV);
  float* o = (float*)(un + un_elems);              // [64][WO]
  if (tid <= RT_CHUNK) pw[tid] = rt_power(a.decay[h], tid);
  const bf16* base = (const bf16*)a.proj;
  bf16 *kh = un, *kl = un + RT_CHUNK * WQ;
  rt_stage_rows(a, qh, ql, WQ, base + (size_t)h * d, t0, n, 1.f, nullptr, vec, tid, 256);
  rt_stage_rows(a, kh, kl, WQ, base + (size_t)(a.heads + h) * d, t0, n, a.k_scale, nullptr, vec, tid, 256);
  __syncthreads();
  const int m = lane >> 3, r = lane & 7, row0 = (warp & 3) * 16, part = warp >> 2;
  const int lo = row0 + (lane >> 2), hi = lo + 8, cq = (lane & 3) * 2;
  // scores of this warp's 16 tokens with 32 keys, times g^(i - j), into ph and pl; keys behind every token's own are skipped
  {
    float acc[4][4] = {};
    if (part * 32 <= row0 + 15) {
      for (int ks = 0; ks < d16 / 16; ++ks) {
        uint32_t ah[4], al[4];
        const int at = (row0 + (m & 1) * 8 + r) * WQ + ks * 16 + (m >> 1) * 8;
        rt_ldm(rt_addr(qh + at), ah);
        rt_ldm(rt_addr(ql + at), al);
#pragma unroll
        for (int np = 0; np < 2; ++np) {
          uint32_t bh[4], bl[4];
          const int bt = (part * 32 + np * 16 + (m >> 1) * 8 + r) * WQ + ks * 16 + (m & 1) * 8;
          rt_ldm(rt_addr(kh + bt), bh);
          rt_ldm(rt_addr(kl + bt), bl);
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            rt_mma(acc[2 * np + e], ah, bh[2 * e], bh[2 * e + 1]);
            rt_mma(acc[2 * np + e], ah, bl[2 * e], bl[2 * e + 1]);
            rt_mma(acc[2 * np + e], al, bh[2 * e], bh[2 * e + 1]);
          }
        }
      }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int j = part * 32 + i * 8 + cq;
      uint32_t h2, l2;
      rt_split2(j <= lo ? acc[i][0] * pw[lo - j] : 0.f, j + 1 <= lo ? acc[i][1] * pw[lo - j - 1] : 0.f, h2, l2);
      *(uint32_t*)(ph + lo * WP + j) = h2;
      *(uint32_t*)(pl + lo * WP + j) = l2;
      rt_split2(j <= hi ? acc[i][2] * pw[hi - j] : 0.f, j + 1 <= hi ? acc[i][3] * pw[hi - j - 1] : 0.f, h2, l2);
      *(uint32_t*)(ph + hi * WP + j) = h2;
      *(uint32_t*)(pl + hi * WP + j) = l2;
    }
  }
  const float* S = a.chunks + (place * a.heads + h) * d * dv;
  const bf16* v_src = base + (size_t)2 * a.heads * d + (size_t)h * dv;
  bf16 *sh = un, *sl = un + d16 * WV;
  float ss_lo = 0.f, ss_hi = 0.f;
  for (int turn = 0; turn < turns; ++turn) {
    const int c0 = turn * RT_CB;
    __syncthreads();                               // the scores are written; the turn before has left vs and the state
    rt_stage_values(a, vs, WV, c0, RT_CB, v_src, t0, n, vec, tid, 256);
    for (int i = tid; i < d16 * (RT_CB / 4); i += 256) {
      const int row = i / (RT_CB / 4), c = c0 + 4 * (i % (RT_CB / 4));
      float4 f = make_float4(0.f, 0.f, 0.f, 0.f);
      if (row < d) {
        const float* src = S + (size_t)row * dv + c;
        if ((dv & 3) == 0) { if (c < dv) f = *(const float4*)src; }
        else {
          if (c < dv) f.x = src[0];
          if (c + 1 < dv) f.y = src[1];
          if (c + 2 < dv) f.z = src[2];
          if (c + 3 < dv) f.w = src[3];
        }
      }
      uint2 h2, l2;
      rt_split2(f.x, f.y, h2.x, l2.x); rt_split2(f.z, f.w, h2.y, l2.y);
      *(uint2*)(sh + row * WV + c - c0) = h2;
      *(uint2*)(sl + row * WV + c - c0) = l2;
    }
    __syncthreads();
    float acc[4][4] = {};
    for (int ks = 0; ks < d16 / 16; ++ks) {        // S^T q
      uint32_t ah[4], al[4];
      const int at = (row0 + (m & 1) * 8 + r) * WQ + ks * 16 + (m >> 1) * 8;
      rt_ldm(rt_addr(qh + at), ah);
      rt_ldm(rt_addr(ql + at), al);
#pragma unroll
      for (int np = 0; np < 2; ++np) {
        uint32_t bh[4], bl[4];
        const int bt = (ks * 16 + (m & 1) * 8 + r) * WV + part * 32 + np * 16 + (m >> 1) * 8;
        rt_ldm_trans(rt_addr(sh + bt), bh);
        rt_ldm_trans(rt_addr(sl + bt), bl);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          rt_mma(acc[2 * np + e], ah, bh[2 * e], bh[2 * e + 1]);
          rt_mma(acc[2 * np + e], ah, bl[2 * e], bl[2 * e + 1]);
          rt_mma(acc[2 * np + e], al, bh[2 * e], bh[2 * e + 1]);
        }
      }
    }
    const float g_lo = pw[lo + 1], g_hi = pw[hi + 1];
#pragma unroll
    for (int i = 0; i < 4; ++i) { acc[i][0] *= g_lo; acc[i][1] *= g_lo; acc[i][2] *= g_hi; acc[i][3] *= g_hi; }
    for (int kk = 0; kk <= (warp & 3); ++kk) {     // the chunk's own keys, 16 at a time up to the tokens' own
      uint32_t ah[4], al[4];
      const int at = (row0 + (m & 1) * 8 + r) * WP + kk * 16 + (m >> 1) * 8;
      rt_ldm(rt_addr(ph + at), ah);
      rt_ldm(rt_addr(pl + at), al);
#pragma unroll
      for (int np = 0; np < 2; ++np) {
        uint32_t b[4];
        rt_ldm_trans(rt_addr(vs + (kk * 16 + (m & 1) * 8 + r) * WV + part * 32 + np * 16 + (m >> 1) * 8), b);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          rt_mma(acc[2 * np + e], ah, b[2 * e], b[2 * e + 1]);
          rt_mma(acc[2 * np + e], al, b[2 * e], b[2 * e + 1]);
        }
      }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {                  // columns from dv on are zero
      const int c = c0 + part * 32 + i * 8 + cq;
      *(float2*)(o + lo * WO + c) = make_float2(acc[i][0], acc[i][1]);
      *(float2*)(o + hi * WO + c) = make_float2(acc[i][2], acc[i][3]);
      ss_lo = fmaf(acc[i][0], acc[i][0], fmaf(acc[i][1], acc[i][1], ss_lo));
      ss_hi = fmaf(acc[i][2], acc[i][2], fmaf(acc[i][3], acc[i][3], ss_hi));
    }
  }
#pragma unroll
  for (int x = 1; x < 4; x <<= 1) {
    ss_lo += __shfl_xor_sync(0xffffffffu, ss_lo, x);
    ss_hi += __shfl_xor_sync(0xffffffffu, ss_hi, x);
  }
  if ((lane & 3) == 0) { sums[part][lo] = ss_lo; sums[part][hi] = ss_hi; }
  __syncthreads();
  const bf16* gate = v_src + (size_t)a.heads * dv;
  bf16* out = (bf16*)a.out + (size_t)h * dv;
  auto factor = [&](int row) {
    return a.norm ? a.out_scale / sqrtf((sums[0][row] + sums[1][row]) / (float)dv + a.eps) : a.out_scale;
  };
  if (vec) {
    const int pieces = dv / 8;
    for (int i = tid; i < n * pieces; i += 256) {
      const int row = i / pieces, c = 8 * (i % pieces);
      const float inv = factor(row);
      float z[8];
      rt_unpack8(*(const uint4*)(gate + (size_t)(t0 + row) * a.ld + c), z);
      const float* x = o + row * WO + c;
      const float4 x0 = *(const float4*)x, x1 = *(const float4*)(x + 4);
      uint4 p;
      __nv_bfloat162* p2 = (__nv_bfloat162*)&p;
      p2[0] = __floats2bfloat162_rn(x0.x * inv * rt_silu(z[0]), x0.y * inv * rt_silu(z[1]));
      p2[1] = __floats2bfloat162_rn(x0.z * inv * rt_silu(z[2]), x0.w * inv * rt_silu(z[3]));
      p2[2] = __floats2bfloat162_rn(x1.x * inv * rt_silu(z[4]), x1.y * inv * rt_silu(z[5]));
      p2[3] = __floats2bfloat162_rn(x1.z * inv * rt_silu(z[6]), x1.w * inv * rt_silu(z[7]));
      *(uint4*)(out + (size_t)(t0 + row) * a.out_ld + c) = p;
    }
  } else {
    for (int i = tid; i < n * dv; i += 256) {
      const int row = i / dv, c = i % dv;
      out[(size_t)(t0 + row) * a.out_ld + c] =
          __float2bfloat16_rn(o[row * WO + c] * factor(row) * rt_silu(__bfloat162float(gate[(size_t)(t0 + row) * a.ld + c])));
    }
  }
}

static size_t rt_sums_smem(int d) {
  const int d16 = (d + 15) & ~15;
  return sizeof(bf16) * (size_t)RT_CHUNK * (2 * (d16 + 8) + RT_CB + 8);
}
static size_t rt_outputs_smem(int d, int dv) {
  const int d16 = (d + 15) & ~15, WQ = d16 + 8, turns = (dv + RT_CB - 1) / RT_CB;
  const size_t un = 2 * (size_t)RT_CHUNK * WQ > 2 * (size_t)d16 * (RT_CB + 8) ? 2 * (size_t)RT_CHUNK * WQ : 2 * (size_t)d16 * (RT_CB + 8);
  return sizeof(bf16) * ((size_t)RT_CHUNK * (2 * WQ + 2 * (RT_CHUNK + 8) + RT_CB + 8) + un) + sizeof(float) * (size_t)RT_CHUNK * (turns * RT_CB + 4);
}
#define RT_SMEM_LIMIT (220 * 1024)

// Columns of the walk form's blocks: a power of two that divides 256, as many as shared memory holds, no more than dv needs.
static int rt_walk_columns(int d, int dv) {
  for (int cb = 128; cb >= 4; cb >>= 1) {
    const size_t smem = sizeof(float) * ((size_t)d * cb + (size_t)RT_WALK_TOKENS * (2 * d + cb + 256));
    if (smem <= 200 * 1024 && (cb <= 4 || cb / 2 < dv)) return cb;
  }
  return 0;
}

// Whether prompts of these heads can take the chunk form (bf16).
extern "C" int odi_retention_takes_chunks(int d, int dv) { return rt_outputs_smem(d, dv) <= RT_SMEM_LIMIT && d <= 1024; }

template <typename K>
static int rt_configure(K kernel, size_t smem) {
  if (smem <= 40 * 1024) return 0;
  return (int)cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
}

template <typename T>
static int launch_in_order(const RetentionArgs& a, cudaStream_t stream) {
  if (a.max_q_len == 1) {
    const bool vec = a.dv % 4 == 0 && ((uintptr_t)a.state & 15) == 0;
    const int V = vec ? 4 : 1, nc = (a.dv + V - 1) / V, cols = nc < 256 ? nc : 256, groups = 256 / cols;
    const size_t smem = sizeof(float) * (2 * (size_t)a.d + 4 + (size_t)groups * nc * V);
    if (smem > 200 * 1024) return ODI_ERR_UNSUPPORTED;
    auto kernel = vec ? rt_step_kernel<T, 4> : rt_step_kernel<T, 1>;
    const int rc = rt_configure(kernel, smem);
    return rc != 0 ? rc : launch_pdl(kernel, dim3(a.heads, a.n_seqs), dim3(256), smem, stream, a);
  }
  const int cb = rt_walk_columns(a.d, a.dv);
  if (cb == 0) return ODI_ERR_UNSUPPORTED;
  const size_t smem = sizeof(float) * ((size_t)a.d * cb + (size_t)RT_WALK_TOKENS * (2 * a.d + cb + 256));
  int rc = rt_configure(rt_walk_kernel<T>, smem);
  if (rc == 0) rc = launch_pdl(rt_walk_kernel<T>, dim3((a.dv + cb - 1) / cb, a.heads, a.n_seqs), dim3(256), smem, stream, a, cb);
  if (rc == 0) rc = launch_pdl(rt_finish_kernel<T>, dim3((unsigned)(((long)a.n_tokens * a.heads + 3) / 4)), dim3(128), 0, stream, a);
  return rc;
}

static int launch_chunks(const RetentionArgs& a, cudaStream_t stream) {
  const int half = a.rot / 2, n_chunks = (a.max_q_len + RT_CHUNK - 1) / RT_CHUNK, col_blocks = (a.dv + RT_CB - 1) / RT_CB;
  const int vec = a.d % 8 == 0 && a.dv % 8 == 0 && a.ld % 8 == 0 && a.out_ld % 8 == 0 &&
                  (a.cos_t == nullptr || (!a.interleaved && half % 8 == 0)) &&
                  (((uintptr_t)a.proj | (uintptr_t)a.out | (uintptr_t)a.cos_t | (uintptr_t)a.sin_t) & 15) == 0;
  const size_t s1 = rt_sums_smem(a.d), s3 = rt_outputs_smem(a.d, a.dv);
  int rc = rt_configure(rt_chunk_sums_kernel, s1);
  if (rc == 0) rc = rt_configure(rt_chunk_outputs_kernel, s3);
  if (rc == 0) rc = launch_pdl(rt_chunk_sums_kernel, dim3(n_chunks, a.heads * col_blocks, a.n_seqs), dim3(256), s1, stream, a, vec);
  const int size = a.d * a.dv;
  const bool wide = size % 4 == 0 && (((uintptr_t)a.chunks | (uintptr_t)a.state) & 15) == 0;
  const int items = wide ? size / 4 : size;
  if (rc == 0)
    rc = launch_pdl(wide ? rt_chunk_scan_kernel<4> : rt_chunk_scan_kernel<1>, dim3((items + 127) / 128, a.heads, a.n_seqs), dim3(128), 0,
                    stream, a);
  if (rc == 0) rc = launch_pdl(rt_chunk_outputs_kernel, dim3(n_chunks, a.heads, a.n_seqs), dim3(256), s3, stream, a, vec);
  return rc;
}

// form 0: tokens in order; 1: chunks side by side (bf16; `chunks` holds their states).
extern "C" int odi_retention(const RetentionArgs* args, int form, int dtype, cudaStream_t stream) {
  RetentionArgs a = *args;
  if (a.n_tokens <= 0 || a.n_seqs <= 0) return 0;
  if (a.heads <= 0 || a.d <= 0 || a.dv <= 0 || a.rot < 0 || a.rot > a.d || (a.rot & 1)) return ODI_ERR_ARGUMENT;
  if (a.cos_t == nullptr) a.rot = 0;
  if (a.heads > 65535 || a.n_seqs > 65535 || (long)a.heads * ((a.dv + RT_CB - 1) / RT_CB) > 65535) return ODI_ERR_UNSUPPORTED;
  if (form == 1) {
    if (dtype != 1 || a.chunks == nullptr || !odi_retention_takes_chunks(a.d, a.dv)) return ODI_ERR_UNSUPPORTED;
    odi_rc = launch_chunks(a, stream);
  } else {
    if (a.max_q_len > 1 && a.o == nullptr) return ODI_ERR_ARGUMENT;
    odi_rc = dtype == 0 ? launch_in_order<float>(a, stream) : launch_in_order<bf16>(a, stream);
  }
  return launch_status();
}
