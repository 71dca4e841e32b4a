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
#define RT_CB 64            // columns of the values per turn

struct RetentionArgs {
  const void* proj;       // [n_tokens, ld] in T, from this mixer's first column on: q (H d), k (H d), v (H dv), gate (H dv)
  const float* cos_t;     // null: no rotation; [n_tokens, rot / 2]
  const float* sin_t;
  const float* decay;     // [heads]
  float* state;           // [slots, heads, d, dv]
  float* chunks;          // chunk form: [n_tokens / 64 + n_seqs, heads, d, dv rounded up to 8] scratch
  void* qk;               // chunk form: [n_tokens, heads, 4, d rounded up to 16] bf16 scratch
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

// Eight neighbouring bf16 numbers.
__device__ __forceinline__ void rt_unpack8(const uint4 raw, float* v) {
  const __nv_bfloat162* h = (const __nv_bfloat162*)&raw;
#pragma unroll
  for (int e = 0; e < 4; ++e) { const float2 f = __bfloat1622float2(h[e]); v[2 * e] = f.x; v[2 * e + 1] = f.y; }
}
// g^n by squaring (n < 2^16; 0^0 = 1).
__device__ __forceinline__ float rt_power(float g, int n) {
  float r = 1.f;
  for (; n > 0; n >>= 1) { if (n & 1) r *= g; g *= g; }
  return r;
}

__device__ __forceinline__ float rt_silu(float z) { return z / (1.f + expf(-z)); }

// ------------------------------------------------------------------------------ one token per sequence

#define RT_STEP_ROWS 8      // rows of the state that a thread has in flight

// V columns a thread per access; the threads of a column take its rows in turn.  What the block needs from memory (rows of
// the state, values, gates, q and k) is requested before anything waits.
template <typename T, int V, int THREADS>
__global__ void __launch_bounds__(THREADS)
rt_step_kernel(RetentionArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float rt_smem[];
  __shared__ float scratch[33];
  const int h = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x, d = a.d, dv = a.dv;
  const int t = a.cu_q[seq], slot = a.slots[seq];
  float* qs = rt_smem;                   // [d]
  float* ks = qs + d;                    // [d]
  float* part = ks + d;                  // [row groups][columns]
  const T* base = (const T*)a.proj + (size_t)t * a.ld;
  const T* v_row = base + (size_t)2 * a.heads * d + (size_t)h * dv;
  const T* gate = v_row + (size_t)a.heads * dv;
  float* S = a.state + ((size_t)slot * a.heads + h) * d * dv;
  // columns in passes of at most one access a thread
  const int nc = (dv + V - 1) / V, cols = min(nc, THREADS), groups = THREADS / cols, grp = tid / cols;
  const float g = a.decay[h];
  const float z0 = tid < dv ? to_f<T>(gate[tid]) : 0.f;
  auto load = [&](float (&x)[RT_STEP_ROWS][V], int c, int r0) {
#pragma unroll
    for (int j = 0; j < RT_STEP_ROWS; ++j) {
      const int r = r0 + j * groups;
      if (r < d) {
        const float* p = S + (size_t)r * dv + c * V;
        if (V == 4) { const float4 f = *(const float4*)p; x[j][0] = f.x; x[j][1 % V] = f.y; x[j][2 % V] = f.z; x[j][3 % V] = f.w; }
        else x[j][0] = p[0];
      }
    }
  };
  for (int c0 = 0; c0 < nc; c0 += cols) {
    const int c = c0 + tid % cols;
    const bool live = c < nc && grp < groups;
    float x[RT_STEP_ROWS][V], o[V] = {}, v[V];
    if (live) {
      load(x, c, grp);
#pragma unroll
      for (int e = 0; e < V; ++e) v[e] = to_f<T>(v_row[c * V + e]);
    }
    if (c0 == 0) {
      for (int i = tid; i < 2 * d; i += THREADS) {
        const bool is_k = i >= d;
        const T* row = base + (size_t)((is_k ? a.heads : 0) + h) * d;
        const float y = rt_lane<T>(a, row, is_k ? i - d : i, t);
        if (is_k) ks[i - d] = y * a.k_scale; else qs[i] = y;
      }
      __syncthreads();
    }
    if (live) {
      for (int r0 = grp; r0 < d; r0 += RT_STEP_ROWS * groups) {
        if (r0 != grp) load(x, c, r0);
#pragma unroll
        for (int j = 0; j < RT_STEP_ROWS; ++j) {
          const int r = r0 + j * groups;
          if (r < d) {
            float* p = S + (size_t)r * dv + c * V;
            const float k = ks[r], q = qs[r];
#pragma unroll
            for (int e = 0; e < V; ++e) { x[j][e] = fmaf(g, x[j][e], k * v[e]); o[e] = fmaf(q, x[j][e], o[e]); }
            if (V == 4) *(float4*)p = make_float4(x[j][0], x[j][1 % V], x[j][2 % V], x[j][3 % V]);
            else p[0] = x[j][0];
          }
        }
      }
#pragma unroll
      for (int e = 0; e < V; ++e) part[((size_t)grp * nc + c) * V + e] = o[e];
    }
  }
  __syncthreads();
  float ss = 0.f, first = 0.f;           // a thread's first column stays in a register
  for (int i = tid; i < dv; i += THREADS) {
    float x = part[i];
    for (int r = 1; r < groups; ++r) x += part[(size_t)r * nc * V + i];
    if (i == tid) first = x; else part[i] = x;
    ss = fmaf(x, x, ss);
  }
  float inv = a.out_scale;
  if (a.norm) inv *= 1.0f / sqrtf(block_sum(ss, scratch) / (float)dv + a.eps);
  T* out = (T*)a.out + (size_t)t * a.out_ld + (size_t)h * dv;
  for (int i = tid; i < dv; i += THREADS)
    out[i] = from_f<T>((i == tid ? first : part[i]) * inv * rt_silu(i == tid ? z0 : to_f<T>(gate[i])));
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

// 16 bytes of split numbers: the high and the low parts of eight.
__device__ __forceinline__ void rt_split8(const float* v, uint4& hi, uint4& lo) {
  rt_split2(v[0], v[1], hi.x, lo.x); rt_split2(v[2], v[3], hi.y, lo.y);
  rt_split2(v[4], v[5], hi.z, lo.z); rt_split2(v[6], v[7], hi.w, lo.w);
}
__device__ __forceinline__ void rt_cp16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(rt_addr(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void rt_cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void rt_cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// The head's values of a chunk into [64][W] rows; rows from n on and columns from dv to `cols` (a multiple of 16) are zero.
// With `vec` by asynchronous copies (the caller commits and waits).  TURNS > 0: `cols` is TURNS * RT_CB.
template <int TURNS>
__device__ __forceinline__ void rt_stage_values(const RetentionArgs& a, bf16* dst, int W, int cols, const bf16* src, int t0, int n,
                                                int vec, int tid) {
  const int pieces = TURNS > 0 ? TURNS * (RT_CB / 8) : cols / 8;
  for (int i = tid; i < RT_CHUNK * pieces; i += 256) {
    const int r = i / pieces, c = 8 * (i % pieces);
    const bf16* row = src + (size_t)(t0 + r) * a.ld + c;
    bf16* to = dst + r * W + c;
    if (vec && r < n && c < a.dv) { rt_cp16(to, row); continue; }
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (!vec && r < n) {
      bf16* p = (bf16*)&v;
#pragma unroll
      for (int e = 0; e < 8; ++e) if (c + e < a.dv) p[e] = row[e];
    }
    *(uint4*)to = v;
  }
}

// A chunk of one head: q and k rotated, k scaled, both split, into `qk` for rt_chunk_outputs; and the sum of its k v^T, each
// token weighed by g^(tokens behind it), into `chunks`.  A block's 8 warps take 16 key lanes each at a time.
__global__ void __launch_bounds__(256, 2)
rt_chunk_sums_kernel(RetentionArgs a, int vec) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) uint8_t rt_bytes[];
  __shared__ float pw[RT_CHUNK + 1];
  const int seq = blockIdx.z, h = blockIdx.y;
  int t0, n;
  size_t place;
  if (!rt_chunk(a, seq, blockIdx.x, t0, n, place)) return;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, d = a.d, d16 = (d + 15) & ~15, WK = d16 + 8;
  const int dvp = (a.dv + 7) & ~7, turns = (a.dv + RT_CB - 1) / RT_CB, WV = turns * RT_CB + 8;
  bf16* kh = (bf16*)rt_bytes;                      // weighted k, high and low [64][WK]
  bf16* kl = kh + RT_CHUNK * WK;
  bf16* vs = kl + RT_CHUNK * WK;                   // [64][WV]
  const bf16* base = (const bf16*)a.proj;
  rt_stage_values<0>(a, vs, WV, turns * RT_CB, base + (size_t)2 * a.heads * d + (size_t)h * a.dv, t0, n, vec, tid);
  rt_cp_commit();
  if (tid <= RT_CHUNK) pw[tid] = rt_power(a.decay[h], tid);
  __syncthreads();
  const bf16* q_src = base + (size_t)h * d;
  const bf16* k_src = base + (size_t)(a.heads + h) * d;
  bf16* split = (bf16*)a.qk + ((size_t)t0 * a.heads + h) * 4 * d16;      // a token's rows: q high, q low, k high, k low
  auto put = [&](int r, int c, const float* q, const float* k) {  // eight lanes of token r (k scaled)
    uint4 hi, lo;
    bf16* dst = split + (size_t)r * a.heads * 4 * d16 + c;
    rt_split8(q, hi, lo);
    *(uint4*)dst = hi; *(uint4*)(dst + d16) = lo;
    rt_split8(k, hi, lo);
    *(uint4*)(dst + 2 * d16) = hi; *(uint4*)(dst + 3 * d16) = lo;
    float w[8];
    const float g = pw[n - 1 - r];
#pragma unroll
    for (int e = 0; e < 8; ++e) w[e] = k[e] * g;
    rt_split8(w, hi, lo);
    *(uint4*)(kh + r * WK + c) = hi; *(uint4*)(kl + r * WK + c) = lo;
  };
  if (vec) {
    // an item: eight lanes of the first half and their partners in the second, or eight lanes that do not turn
    const int half = a.rot >> 1, pairs = half / 8, items = pairs + (d16 - a.rot) / 8;
    for (int i = tid; i < n * items; i += 256) {
      const int r = i / items, x = i % items;
      const bf16* q_row = q_src + (size_t)(t0 + r) * a.ld;
      const bf16* k_row = k_src + (size_t)(t0 + r) * a.ld;
      if (x < pairs) {
        const int c = 8 * x;
        const uint4 qa = *(const uint4*)(q_row + c), qb = *(const uint4*)(q_row + c + half);
        const uint4 ka = *(const uint4*)(k_row + c), kb = *(const uint4*)(k_row + c + half);
        const float4* cp = (const float4*)(a.cos_t + (size_t)(t0 + r) * half + c);
        const float4* sp = (const float4*)(a.sin_t + (size_t)(t0 + r) * half + c);
        float cs[8], sn[8], u[8], v[8], q1[8], q2[8], k1[8], k2[8];
        *(float4*)cs = cp[0]; *(float4*)(cs + 4) = cp[1];
        *(float4*)sn = sp[0]; *(float4*)(sn + 4) = sp[1];
        rt_unpack8(qa, u); rt_unpack8(qb, v);
#pragma unroll
        for (int e = 0; e < 8; ++e) { q1[e] = fmaf(-v[e], sn[e], u[e] * cs[e]); q2[e] = fmaf(u[e], sn[e], v[e] * cs[e]); }
        rt_unpack8(ka, u); rt_unpack8(kb, v);
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          k1[e] = fmaf(-v[e], sn[e], u[e] * cs[e]) * a.k_scale;
          k2[e] = fmaf(u[e], sn[e], v[e] * cs[e]) * a.k_scale;
        }
        put(r, c, q1, k1);
        put(r, c + half, q2, k2);
      } else {
        const int c = a.rot + 8 * (x - pairs);
        float q[8] = {}, k[8] = {};
        if (c < d) {
          rt_unpack8(*(const uint4*)(q_row + c), q);
          rt_unpack8(*(const uint4*)(k_row + c), k);
        }
#pragma unroll
        for (int e = 0; e < 8; ++e) k[e] *= a.k_scale;
        put(r, c, q, k);
      }
    }
  } else {
    const int pieces = d16 / 8;
    for (int i = tid; i < n * pieces; i += 256) {
      const int r = i / pieces, c = 8 * (i % pieces);
      float q[8], k[8];
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        q[e] = c + e < d ? rt_lane<bf16>(a, q_src + (size_t)(t0 + r) * a.ld, c + e, t0 + r) : 0.f;
        k[e] = c + e < d ? rt_lane<bf16>(a, k_src + (size_t)(t0 + r) * a.ld, c + e, t0 + r) * a.k_scale : 0.f;
      }
      put(r, c, q, k);
    }
  }
  for (int i = tid; i < (RT_CHUNK - n) * (WK / 8); i += 256) {    // rows behind the chunk's tokens
    const int r = n + i / (WK / 8), c = 8 * (i % (WK / 8));
    *(uint4*)(kh + r * WK + c) = make_uint4(0u, 0u, 0u, 0u);
    *(uint4*)(kl + r * WK + c) = make_uint4(0u, 0u, 0u, 0u);
  }
  rt_cp_wait<0>();
  __syncthreads();
  float* U = a.chunks + (place * a.heads + h) * d * dvp;
  const int m = lane >> 3, r = lane & 7;
  for (int row0 = warp * 16; row0 < d16; row0 += 8 * 16) {
    // A = k^T: matrices (lanes row0 .. + 7, tokens kk*16 .. + 7), (lanes + 8, same tokens), (lanes, tokens + 8), (both + 8)
    uint32_t ah[RT_CHUNK / 16][4], al[RT_CHUNK / 16][4];
#pragma unroll
    for (int kk = 0; kk < RT_CHUNK / 16; ++kk) {
      const int at = (kk * 16 + (m >> 1) * 8 + r) * WK + row0 + (m & 1) * 8;
      rt_ldm_trans(rt_addr(kh + at), ah[kk]);
      rt_ldm_trans(rt_addr(kl + at), al[kk]);
    }
    for (int c0 = 0; c0 < a.dv; c0 += RT_CB) {
      float acc[RT_CB / 8][4] = {};
#pragma unroll
      for (int kk = 0; kk < RT_CHUNK / 16; ++kk) {
#pragma unroll
        for (int np = 0; np < RT_CB / 16; ++np) {
          uint32_t b[4];
          rt_ldm_trans(rt_addr(vs + (kk * 16 + (m & 1) * 8 + r) * WV + c0 + np * 16 + (m >> 1) * 8), b);
          rt_mma(acc[2 * np], ah[kk], b[0], b[1]);
          rt_mma(acc[2 * np], al[kk], b[0], b[1]);
          rt_mma(acc[2 * np + 1], ah[kk], b[2], b[3]);
          rt_mma(acc[2 * np + 1], al[kk], b[2], b[3]);
        }
      }
      const int lo = row0 + (lane >> 2), c = c0 + (lane & 3) * 2;
#pragma unroll
      for (int i = 0; i < RT_CB / 8; ++i)
        if (c + 8 * i < dvp) {
          if (lo < d) *(float2*)(U + (size_t)lo * dvp + c + 8 * i) = make_float2(acc[i][0], acc[i][1]);
          if (lo + 8 < d) *(float2*)(U + (size_t)(lo + 8) * dvp + c + 8 * i) = make_float2(acc[i][2], acc[i][3]);
        }
    }
  }
}

// The state in front of every chunk in place of its sum, and the sequence's new state.  A thread takes eight neighbouring
// columns of a row; what it leaves in their 32 bytes are the eight high parts and then the eight low parts of the state.
__global__ void __launch_bounds__(128)
rt_chunk_scan_kernel(RetentionArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int seq = blockIdx.z, h = blockIdx.y, dvp = (a.dv + 7) & ~7;
  const int i = 8 * (blockIdx.x * blockDim.x + threadIdx.x);
  if (i >= a.d * dvp) return;
  const int q_begin = a.cu_q[seq], q_len = a.cu_q[seq + 1] - q_begin;
  if (q_len <= 0) return;
  const int n_chunks = (q_len + RT_CHUNK - 1) / RT_CHUNK, row = i / dvp, c0 = i % dvp;
  const size_t step = (size_t)a.heads * a.d * dvp;
  float* p = a.chunks + ((size_t)(q_begin / RT_CHUNK + seq) * a.heads + h) * a.d * dvp + i;
  float* st = a.state + (((size_t)a.slots[seq] * a.heads + h) * a.d + row) * a.dv + c0;
  const float g = a.decay[h], gc = rt_power(g, RT_CHUNK), gl = rt_power(g, q_len - (n_chunks - 1) * RT_CHUNK);
  const bool whole = (a.dv & 3) == 0 && c0 + 8 <= a.dv && ((uintptr_t)a.state & 15) == 0;
  float S[8];
  if (whole) { *(float4*)S = *(const float4*)st; *(float4*)(S + 4) = *(const float4*)(st + 4); }
  else {
#pragma unroll
    for (int e = 0; e < 8; ++e) S[e] = c0 + e < a.dv ? st[e] : 0.f;
  }
  auto turn = [&](float* at, const float* u, float w) {
    uint4 hi, lo;
    rt_split8(S, hi, lo);
    *(uint4*)at = hi; *(uint4*)(at + 4) = lo;
#pragma unroll
    for (int e = 0; e < 8; ++e) S[e] = fmaf(w, S[e], u[e]);
  };
  int c = 0;
  for (; c + 4 < n_chunks; c += 4) {            // four chunks' loads in flight
    float u[4][8];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      *(float4*)u[j] = *(const float4*)(p + (size_t)(c + j) * step);
      *(float4*)(u[j] + 4) = *(const float4*)(p + (size_t)(c + j) * step + 4);
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) turn(p + (size_t)(c + j) * step, u[j], gc);
  }
  for (; c < n_chunks; ++c) {
    float u[8];
    *(float4*)u = *(const float4*)(p + (size_t)c * step);
    *(float4*)(u + 4) = *(const float4*)(p + (size_t)c * step + 4);
    turn(p + (size_t)c * step, u, c + 1 < n_chunks ? gc : gl);
  }
  if (whole) { *(float4*)st = *(const float4*)S; *(float4*)(st + 4) = *(const float4*)(S + 4); }
  else {
#pragma unroll
    for (int e = 0; e < 8; ++e) if (c0 + e < a.dv) st[e] = S[e];
  }
}

// The read-outs of a chunk's tokens for one head: 8 warps, warp w takes token rows 16 (w % 4) .. + 15 and half w / 4 of the
// keys (scores) and of the columns of a turn (read-outs).  TURNS turns of 64 columns stay in registers until the norm.
template <int TURNS>
__global__ void __launch_bounds__(256, TURNS <= 2 ? 2 : 1)
rt_chunk_outputs_kernel(RetentionArgs a, int vec) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) uint8_t rt_bytes[];
  __shared__ float pw[RT_CHUNK + 1], sums[2][RT_CHUNK];
  const int seq = blockIdx.z, h = blockIdx.y;
  int t0, n;
  size_t place;
  if (!rt_chunk(a, seq, blockIdx.x, t0, n, place)) return;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, d = a.d, dv = a.dv, d16 = (d + 15) & ~15, WQ = 2 * d16 + 8;
  constexpr int WP = RT_CHUNK + 8, WS = RT_CB + 8, WV = TURNS * RT_CB + 8;
  const int dvp = (dv + 7) & ~7;
  bf16* qh = (bf16*)rt_bytes;                      // q, high and then low parts in a row [64][WQ]
  bf16* ql = qh + d16;
  bf16* ph = qh + RT_CHUNK * WQ;                   // decayed scores [64][WP]
  bf16* pl = ph + RT_CHUNK * WP;
  bf16* vs = pl + RT_CHUNK * WP;                   // values [64][WV]
  bf16* un = vs + RT_CHUNK * WV;                   // k [64][WQ] like q, then a turn's state [d16][WS] twice
  bf16 *kh = un, *kl = un + d16;
  const bf16* base = (const bf16*)a.proj;
  const bf16* v_src = base + (size_t)2 * a.heads * d + (size_t)h * dv;
  {
    const bf16* split = (bf16*)a.qk + ((size_t)t0 * a.heads + h) * 4 * d16;
    const int half = d16 / 4;                      // 16-byte pieces of q (and of k) in a token's row
    for (int r = warp; r < RT_CHUNK; r += 8)
      for (int x = lane; x < 2 * half; x += 32) {
        bf16* dst = (x < half ? qh + 8 * x : kh + 8 * (x - half)) + r * WQ;
        if (r < n) rt_cp16(dst, split + (size_t)r * a.heads * 4 * d16 + 8 * x);
        else *(uint4*)dst = make_uint4(0u, 0u, 0u, 0u);
      }
    rt_cp_commit();
  }
  rt_stage_values<TURNS>(a, vs, WV, TURNS * RT_CB, v_src, t0, n, vec, tid);
  rt_cp_commit();
  if (tid <= RT_CHUNK) pw[tid] = rt_power(a.decay[h], tid);
  rt_cp_wait<1>();
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
  const bf16* S = (const bf16*)(a.chunks + (place * a.heads + h) * d * dvp);     // per eight columns: high parts, low parts
  bf16 *sh = un, *sl = un + d16 * WS;
  float out_acc[TURNS][4][4];
  float ss_lo = 0.f, ss_hi = 0.f;
#pragma unroll
  for (int turn = 0; turn < TURNS; ++turn) {
    const int c0 = turn * RT_CB;
    __syncthreads();                               // the scores are written; k, or the turn before, is done with `un`
    for (int i = tid; i < d16 * (RT_CB / 4); i += 256) {
      const int row = i / (RT_CB / 4), x = i % (RT_CB / 4), c = 8 * (x >> 1);
      bf16* dst = ((x & 1) ? sl : sh) + row * WS + c;
      if (row < d && c0 + c < dvp) rt_cp16(dst, S + 2 * ((size_t)row * dvp + c0 + c) + 8 * (x & 1));
      else *(uint4*)dst = make_uint4(0u, 0u, 0u, 0u);
    }
    rt_cp_commit();
    rt_cp_wait<0>();
    __syncthreads();
    float (&acc)[4][4] = out_acc[turn];
#pragma unroll
    for (int i = 0; i < 4; ++i) { acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f; }
#pragma unroll 2
    for (int ks = 0; ks < d16 / 16; ++ks) {        // S^T q
      uint32_t ah[4], al[4];
      const int at = (row0 + (m & 1) * 8 + r) * WQ + ks * 16 + (m >> 1) * 8;
      rt_ldm(rt_addr(qh + at), ah);
      rt_ldm(rt_addr(ql + at), al);
#pragma unroll
      for (int np = 0; np < 2; ++np) {
        uint32_t bh[4], bl[4];
        const int bt = (ks * 16 + (m & 1) * 8 + r) * WS + part * 32 + np * 16 + (m >> 1) * 8;
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
        rt_ldm_trans(rt_addr(vs + (kk * 16 + (m & 1) * 8 + r) * WV + c0 + part * 32 + np * 16 + (m >> 1) * 8), b);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          rt_mma(acc[2 * np + e], ah, b[2 * e], b[2 * e + 1]);
          rt_mma(acc[2 * np + e], al, b[2 * e], b[2 * e + 1]);
        }
      }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {                  // columns from dv on are zero
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
  // two columns a lane: four lanes write 16 neighbouring bytes
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int row = e ? hi : lo;
    if (row >= n) continue;
    const float inv = a.norm ? a.out_scale / sqrtf((sums[0][row] + sums[1][row]) / (float)dv + a.eps) : a.out_scale;
    const bf16* gate = v_src + (size_t)a.heads * dv + (size_t)(t0 + row) * a.ld;
    bf16* out = (bf16*)a.out + (size_t)(t0 + row) * a.out_ld + (size_t)h * dv;
#pragma unroll
    for (int turn = 0; turn < TURNS; ++turn)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int c = turn * RT_CB + part * 32 + i * 8 + cq;
        const float x = out_acc[turn][i][2 * e] * inv, y = out_acc[turn][i][2 * e + 1] * inv;
        if (vec) {
          if (c < dv) {
            const float2 z = __bfloat1622float2(*(const __nv_bfloat162*)(gate + c));
            *(__nv_bfloat162*)(out + c) = __floats2bfloat162_rn(x * rt_silu(z.x), y * rt_silu(z.y));
          }
        } else {
          if (c < dv) out[c] = __float2bfloat16_rn(x * rt_silu(__bfloat162float(gate[c])));
          if (c + 1 < dv) out[c + 1] = __float2bfloat16_rn(y * rt_silu(__bfloat162float(gate[c + 1])));
        }
      }
  }
}

// Turns that chunk_outputs is compiled for.
static int rt_turns(int dv) {
  const int t = (dv + RT_CB - 1) / RT_CB;
  return t <= 1 ? 1 : (t <= 2 ? 2 : (t <= 4 ? 4 : 8));
}
static size_t rt_sums_smem(int d, int dv) {
  const int d16 = (d + 15) & ~15;
  return sizeof(bf16) * (size_t)RT_CHUNK * (2 * (d16 + 8) + (dv + RT_CB - 1) / RT_CB * RT_CB + 8);
}
static size_t rt_outputs_smem(int d, int dv) {
  const int d16 = (d + 15) & ~15, WQ = 2 * d16 + 8;
  const size_t k = (size_t)RT_CHUNK * WQ, state = 2 * (size_t)d16 * (RT_CB + 8);
  return sizeof(bf16) * ((size_t)RT_CHUNK * (WQ + 2 * (RT_CHUNK + 8) + rt_turns(dv) * RT_CB + 8) + (k > state ? k : state));
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
extern "C" int odi_retention_takes_chunks(int d, int dv) {
  return dv <= 8 * RT_CB && rt_outputs_smem(d, dv) <= RT_SMEM_LIMIT && rt_sums_smem(d, dv) <= RT_SMEM_LIMIT;
}

template <typename K>
static int rt_configure(K kernel, size_t smem) {
  if (smem <= 40 * 1024) return 0;
  return (int)cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
}

template <typename T>
static int launch_in_order(const RetentionArgs& a, cudaStream_t stream) {
  if (a.max_q_len == 1) {
    const bool vec = a.dv % 4 == 0 && ((uintptr_t)a.state & 15) == 0, big = vec && (long)a.d * a.dv > 8192;
    const int V = vec ? 4 : 1, threads = big ? 512 : 256, nc = (a.dv + V - 1) / V, cols = nc < threads ? nc : threads,
              groups = threads / cols;
    const size_t smem = sizeof(float) * (2 * (size_t)a.d + (size_t)groups * nc * V);
    if (smem > 200 * 1024) return ODI_ERR_UNSUPPORTED;
    auto kernel = big ? rt_step_kernel<T, 4, 512> : vec ? rt_step_kernel<T, 4, 256> : rt_step_kernel<T, 1, 256>;
    const int rc = rt_configure(kernel, smem);
    return rc != 0 ? rc : launch_pdl(kernel, dim3(a.heads, a.n_seqs), dim3(threads), smem, stream, a);
  }
  const int cb = rt_walk_columns(a.d, a.dv);
  if (cb == 0) return ODI_ERR_UNSUPPORTED;
  const size_t smem = sizeof(float) * ((size_t)a.d * cb + (size_t)RT_WALK_TOKENS * (2 * a.d + cb + 256));
  int rc = rt_configure(rt_walk_kernel<T>, smem);
  if (rc == 0) rc = launch_pdl(rt_walk_kernel<T>, dim3((a.dv + cb - 1) / cb, a.heads, a.n_seqs), dim3(256), smem, stream, a, cb);
  if (rc == 0) rc = launch_pdl(rt_finish_kernel<T>, dim3((unsigned)(((long)a.n_tokens * a.heads + 3) / 4)), dim3(128), 0, stream, a);
  return rc;
}

template <int TURNS>
static int launch_outputs(const RetentionArgs& a, int n_chunks, int vec, cudaStream_t stream) {
  const size_t smem = rt_outputs_smem(a.d, a.dv);
  const int rc = rt_configure(rt_chunk_outputs_kernel<TURNS>, smem);
  return rc != 0 ? rc : launch_pdl(rt_chunk_outputs_kernel<TURNS>, dim3(n_chunks, a.heads, a.n_seqs), dim3(256), smem, stream, a, vec);
}

static int launch_chunks(const RetentionArgs& a, cudaStream_t stream) {
  const int half = a.rot / 2, n_chunks = (a.max_q_len + RT_CHUNK - 1) / RT_CHUNK;
  const int vec = a.d % 8 == 0 && a.dv % 8 == 0 && a.ld % 8 == 0 && a.out_ld % 8 == 0 &&
                  (a.cos_t == nullptr || (!a.interleaved && half % 8 == 0)) &&
                  (((uintptr_t)a.proj | (uintptr_t)a.out | (uintptr_t)a.cos_t | (uintptr_t)a.sin_t) & 15) == 0;
  const size_t s1 = rt_sums_smem(a.d, a.dv);
  int rc = rt_configure(rt_chunk_sums_kernel, s1);
  if (rc == 0) rc = launch_pdl(rt_chunk_sums_kernel, dim3(n_chunks, a.heads, a.n_seqs), dim3(256), s1, stream, a, vec);
  const int items = a.d * ((a.dv + 7) / 8);
  if (rc == 0) rc = launch_pdl(rt_chunk_scan_kernel, dim3((items + 127) / 128, a.heads, a.n_seqs), dim3(128), 0, stream, a);
  if (rc != 0) return rc;
  switch (rt_turns(a.dv)) {
    case 1: return launch_outputs<1>(a, n_chunks, vec, stream);
    case 2: return launch_outputs<2>(a, n_chunks, vec, stream);
    case 4: return launch_outputs<4>(a, n_chunks, vec, stream);
    default: return launch_outputs<8>(a, n_chunks, vec, stream);
  }
}

// form 0: tokens in order; 1: chunks side by side (bf16; `chunks` holds their states).
extern "C" int odi_retention(const RetentionArgs* args, int form, int dtype, cudaStream_t stream) {
  RetentionArgs a = *args;
  if (a.n_tokens <= 0 || a.n_seqs <= 0) return 0;
  if (a.heads <= 0 || a.d <= 0 || a.dv <= 0 || a.rot < 0 || a.rot > a.d || (a.rot & 1)) return ODI_ERR_ARGUMENT;
  if (a.cos_t == nullptr) a.rot = 0;
  if (a.heads > 65535 || a.n_seqs > 65535) return ODI_ERR_UNSUPPORTED;
  if (form == 1) {
    if (dtype != 1 || a.chunks == nullptr || a.qk == nullptr || !odi_retention_takes_chunks(a.d, a.dv)) return ODI_ERR_UNSUPPORTED;
    odi_rc = launch_chunks(a, stream);
  } else {
    if (a.max_q_len > 1 && a.o == nullptr) return ODI_ERR_ARGUMENT;
    odi_rc = dtype == 0 ? launch_in_order<float>(a, stream) : launch_in_order<bf16>(a, stream);
  }
  return launch_status();
}
