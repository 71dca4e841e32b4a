// The gated delta rule with one decay per head, for ragged batches of token runs: what lies between the mixer's input
// products and its output product.
//
// Per sequence and head the state S [d, dv] (fp32, zero at the start) goes through, for each token in order,
//     S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q
// with g = exp(-exp(A_log) softplus(a + dt_bias)) and beta = sigmoid(b), one number each per head.  q, k and v come from
// a short causal convolution per channel followed by SiLU; q and k are unit vectors per key head, q times d^-1/2; head h
// reads key head h / (heads / kv_heads).  Everything behind the projections is fp32 in both compute dtypes.
//
// Four tokens at a time.  Let S be the state before tokens 0..3, G_i = g_0 .. g_i and D_ij = g_(j+1) .. g_i.  Then
//     u_i = beta_i (v_i - G_i S^T k_i - sum_(j<i) D_ij (k_j . k_i) u_j)
//     o_i = G_i S^T q_i + sum_(j<=i) D_ij (k_j . q_i) u_j
//     S  <- G_3 S + sum_j D_3j k_j u_j^T
// (products of decays only: nothing is divided), so one walk over the state gives the eight products S^T k_i and S^T q_i
// whose sums over the lanes of a column run side by side, and a second walk updates it: a quarter of the chain of
// shuffles that token by token would take, and fewer operations per token.  The tokens that are left (and single-token
// steps) go one by one.
//
// Kernels:
//  prep       per token: convolution with SiLU of all channels, unit vectors, decays and step sizes; the convolution's
//             state of a sequence that brings one token moves on in the same launch;
//  conv_state the convolution's state of the other sequences: the last taps - 1 inputs;
//  groups     the numbers of every group of four tokens: products of decays and of the group's vectors;
//  rule       the recurrence: a block per (sequence, head, block of COLS value columns); a column of S lies in the
//             registers of RS neighbouring lanes, R rows each (two rows in a register pair: packed fp32
//             operations), two columns a thread; 16 tokens of q, k, v and the groups' numbers are staged in shared
//             memory, the next 16 by asynchronous copies meanwhile;
//  out_norm   per (token, head): o / rms(o) (eps inside the root) * weight * silu(gate), rounded once to T.
#include "common.cuh"

#define HD_MAX_TAPS 16
#define HD_CPT 2            // value columns per thread
#define HD_COEFS 32         // numbers of a group of four tokens: see hd_groups_kernel

struct HeadDeltaArgs {
  const void* proj;       // [n_tokens, ld] in T: q (kv_heads d), k (kv_heads d), v (heads dv), gate (heads dv)
  const float* ab;        // [n_tokens, 2 heads]: a, then b
  const float* taps;      // [taps_n, C], C = 2 kv_heads d + heads dv; the last row weighs the current token
  const float* a_log;     // [heads]
  const float* dt_bias;   // [heads]
  const float* norm_w;    // [dv]
  float* conv_state;      // [slots, taps_n - 1, C]; null when taps_n == 1
  float* state;           // [slots, heads, d, dv]
  float* qk;              // [n_tokens, kv_heads, 2, d] scratch: unit q (scaled), unit k
  float* gb;              // [n_tokens, heads, 2] scratch: decay, step size
  float* coefs;           // [ceil(n_tokens / 4), heads, HD_COEFS] scratch: the groups' numbers
  float* o;               // [n_tokens, heads dv] scratch: v, then the read-outs in its place
  void* out;              // [n_tokens, heads dv] in T
  const int* cu_q;
  const int* tok_seq;
  const int* slots;
  int n_tokens, n_seqs, max_q_len, ld, heads, kv_heads, d, dv, taps_n;
  float eps, unit_eps;
};

__device__ __forceinline__ float hd_softplus(float x) { return x > 20.f ? x : log1pf(expf(x)); }

template <typename T>
__device__ __forceinline__ float hd_input(const HeadDeltaArgs& a, int C, int q_begin, int slot, int idx, int c) {
  // input `idx` of the sequence's run in this step; negative indices reach into the convolution state
  if (idx >= 0) return to_f<T>(((const T*)a.proj)[(size_t)(q_begin + idx) * a.ld + c]);
  return a.conv_state[((size_t)slot * (a.taps_n - 1) + (a.taps_n - 1 + idx)) * C + c];
}

// V neighbouring channels at once: floats, and inputs in T (V = 4: 16- resp. 8-byte accesses).
template <int V> __device__ __forceinline__ void hd_loadf(const float* p, float* v) {
  if (V == 4) { const float4 x = *(const float4*)p; v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w; }
  else v[0] = p[0];
}
template <int V> __device__ __forceinline__ void hd_storef(float* p, const float* v) {
  if (V == 4) *(float4*)p = make_float4(v[0], v[1], v[2], v[3]);
  else p[0] = v[0];
}
template <typename T, int V> __device__ __forceinline__ void hd_loadt(const T* p, float* v) {
  if (V == 1) { v[0] = to_f<T>(p[0]); return; }
  if (sizeof(T) == 4) { hd_loadf<V>((const float*)p, v); return; }
  const uint2 raw = *(const uint2*)p;
  const float2 lo = __bfloat1622float2(*(const __nv_bfloat162*)&raw.x), hi = __bfloat1622float2(*(const __nv_bfloat162*)&raw.y);
  v[0] = lo.x; v[1] = lo.y; v[2 % V] = hi.x; v[3 % V] = hi.y;
}

// A block takes one token and, of gridDim.y parts, a range of key heads with the heads that read them.
template <typename T, int V>
__global__ void __launch_bounds__(256)
hd_prep_kernel(HeadDeltaArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float ys[];          // q and then k of the part's key heads behind the convolution
  const int t = blockIdx.x;
  const int g0 = a.kv_heads * blockIdx.y / gridDim.y, g1 = a.kv_heads * (blockIdx.y + 1) / gridDim.y, rep = a.heads / a.kv_heads;
  const int qk_n = 2 * a.kv_heads * a.d, vn = a.heads * a.dv, C = qk_n + vn;
  const int part_q = (g1 - g0) * a.d, part_n = 2 * part_q + (g1 - g0) * rep * a.dv;
  const int seq = a.tok_seq[t];
  const int q_begin = a.cu_q[seq], q_len = a.cu_q[seq + 1] - q_begin, slot = a.slots[seq];
  const int li = t - q_begin, keep = a.taps_n - 1;
  const T* row = (const T*)a.proj + (size_t)t * a.ld;
  float* st = a.conv_state + (size_t)slot * keep * C;      // not followed when keep is 0
  for (int x = threadIdx.x * V; x < part_n; x += blockDim.x * V) {
    const bool is_v = x >= 2 * part_q;
    const int c = is_v ? qk_n + g0 * rep * a.dv + (x - 2 * part_q) : (x < part_q ? 0 : a.kv_heads * a.d - part_q) + g0 * a.d + x;
    float acc[V] = {}, in[V], w[V];
    if (li >= keep) {                    // every input is one of the step's own: no branch between the loads
      const T* src = row - (size_t)keep * a.ld + c;
#pragma unroll 4
      for (int j = 0; j < a.taps_n; ++j) {
        hd_loadt<T, V>(src + (size_t)j * a.ld, in);
        hd_loadf<V>(a.taps + (size_t)j * C + c, w);
#pragma unroll
        for (int e = 0; e < V; ++e) acc[e] = fmaf(w[e], in[e], acc[e]);
      }
    } else {
      for (int j = 0; j < a.taps_n; ++j) {
        const int back = keep - j;                          // tokens before this one
        if (li >= back) hd_loadt<T, V>(row - (size_t)back * a.ld + c, in);
        else hd_loadf<V>(st + (size_t)(keep + li - back) * C + c, in);
        hd_loadf<V>(a.taps + (size_t)j * C + c, w);
#pragma unroll
        for (int e = 0; e < V; ++e) acc[e] = fmaf(w[e], in[e], acc[e]);
      }
    }
    if (q_len == 1 && keep > 0) {        // this thread is the only one that reads or writes these inputs; `in` is the token's own
      float old[V];
      for (int j = 0; j + 1 < keep; ++j) { hd_loadf<V>(st + (size_t)(j + 1) * C + c, old); hd_storef<V>(st + (size_t)j * C + c, old); }
      hd_storef<V>(st + (size_t)(keep - 1) * C + c, in);
    }
#pragma unroll
    for (int e = 0; e < V; ++e) acc[e] = acc[e] / (1.f + expf(-acc[e]));
    if (is_v) hd_storef<V>(a.o + (size_t)t * vn + (c - qk_n), acc);
    else hd_storef<V>(ys + x, acc);
  }
  for (int h = g0 * rep + threadIdx.x; h < g1 * rep; h += blockDim.x) {
    const float* ab = a.ab + (size_t)t * 2 * a.heads;
    const float decay = expf(-expf(a.a_log[h]) * hd_softplus(ab[h] + a.dt_bias[h]));
    float* dst = a.gb + ((size_t)t * a.heads + h) * 2;
    dst[0] = decay;
    dst[1] = 1.f / (1.f + expf(-ab[a.heads + h]));
  }
  __syncthreads();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
  for (int w = warp; w < 2 * (g1 - g0); w += n_warps) {      // the part's q heads, then its k heads
    const float* src = ys + (size_t)w * a.d;
    float ss = 0.f;
    for (int i = lane; i < a.d; i += 32) ss = fmaf(src[i], src[i], ss);
    ss = warp_sum(ss);
    const bool is_k = w >= g1 - g0;
    const float scale = 1.0f / sqrtf(ss + a.unit_eps) * (is_k ? 1.f : 1.0f / sqrtf((float)a.d));
    float* dst = a.qk + (((size_t)t * a.kv_heads + g0 + (is_k ? w - (g1 - g0) : w)) * 2 + (is_k ? 1 : 0)) * a.d;
    for (int i = lane; i < a.d; i += 32) dst[i] = src[i] * scale;
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
hd_conv_state_kernel(HeadDeltaArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int C = 2 * a.kv_heads * a.d + a.heads * a.dv;
  const int seq = blockIdx.x;
  const int c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= C) return;
  const int q_begin = a.cu_q[seq], q_len = a.cu_q[seq + 1] - q_begin, slot = a.slots[seq];
  if (q_len <= 1) return;                // moved on by prep
  const int keep = a.taps_n - 1;
  float next[HD_MAX_TAPS];
#pragma unroll
  for (int j = 0; j < HD_MAX_TAPS; ++j)
    if (j < keep) next[j] = hd_input<T>(a, C, q_begin, slot, q_len - keep + j, c);
#pragma unroll
  for (int j = 0; j < HD_MAX_TAPS; ++j)
    if (j < keep) a.conv_state[((size_t)slot * keep + j) * C + c] = next[j];
}

__device__ __forceinline__ void hd_cp4(float* dst, const float* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void hd_cp16(float* dst, const float* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void hd_cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void hd_cp_wait_all() { asm volatile("cp.async.wait_group 0;" ::: "memory"); }

// A group's numbers (HD_COEFS floats): beta_i at 0, beta_i G_i at 4, G_i at 8, D_3i at 12, then beta_i D_ij (k_j . k_i) for
// j < i at CK(i, j) and D_ij (k_j . q_i) for j <= i at CQ(i, j).  The group that starts at token t (t - q_begin a multiple
// of 4, four tokens left) lies at slot t / 4: groups share no token, so no two share a slot.
#define CK(i, j) (16 + (i) * ((i) - 1) / 2 + (j))
#define CQ(i, j) (22 + (i) * ((i) + 1) / 2 + (j))

// One warp per (token, key head); the warps of tokens that start no group leave.
__global__ void __launch_bounds__(128)
hd_groups_kernel(HeadDeltaArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float dots[4][20];           // k_j . k_i (the pairs as in CK), then k_j . q_i (as in CQ)
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const long item = (long)blockIdx.x * 4 + warp;
  if (item >= (long)a.n_tokens * a.kv_heads) return;
  const int t = (int)(item / a.kv_heads), kvh = (int)(item % a.kv_heads);
  const int seq = a.tok_seq[t], q_begin = a.cu_q[seq], q_end = a.cu_q[seq + 1];
  if (((t - q_begin) & 3) != 0 || t + 4 > q_end) return;
  const size_t step = (size_t)a.kv_heads * 2 * a.d;
  const float* base = a.qk + (size_t)t * step + (size_t)kvh * 2 * a.d;
  float kk[6] = {}, kq[10] = {};
  for (int e = lane; e < a.d; e += 32) {
    float q[4], k[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) { q[i] = base[i * step + e]; k[i] = base[i * step + a.d + e]; }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
#pragma unroll
      for (int j = 0; j < i; ++j) kk[CK(i, j) - 16] = fmaf(k[i], k[j], kk[CK(i, j) - 16]);
#pragma unroll
      for (int j = 0; j <= i; ++j) kq[CQ(i, j) - 22] = fmaf(q[i], k[j], kq[CQ(i, j) - 22]);
    }
  }
#pragma unroll
  for (int i = 0; i < 6; ++i) { kk[i] = warp_sum(kk[i]); if (lane == 0) dots[warp][i] = kk[i]; }
#pragma unroll
  for (int i = 0; i < 10; ++i) { kq[i] = warp_sum(kq[i]); if (lane == 0) dots[warp][6 + i] = kq[i]; }
  __syncwarp();
  // lane n writes number n: which tokens it is about
  int kind = lane >> 2, i = lane & 3, j = 0;
  if (lane >= 22) { kind = 5; i = lane < 23 ? 0 : (lane < 25 ? 1 : (lane < 28 ? 2 : 3)); j = lane - CQ(i, 0); }
  else if (lane >= 16) { kind = 4; i = lane < 17 ? 1 : (lane < 19 ? 2 : 3); j = lane - CK(i, 0); }
  const int rep = a.heads / a.kv_heads;
  for (int r = 0; r < rep; ++r) {
    const int h = kvh * rep + r;
    float g[4];
#pragma unroll
    for (int m = 0; m < 4; ++m) g[m] = a.gb[((size_t)(t + m) * a.heads + h) * 2];
    const float beta = a.gb[((size_t)(t + i) * a.heads + h) * 2 + 1];
    float G = 1.f, E = 1.f, D = 1.f;                // g_0 .. g_i;  g_(i+1) .. g_3;  g_(j+1) .. g_i
#pragma unroll
    for (int m = 0; m < 4; ++m) {
      if (m <= i) G *= g[m]; else E *= g[m];
      if (m > j && m <= i) D *= g[m];
    }
    float out = beta;
    if (kind == 1) out = beta * G;
    else if (kind == 2) out = G;
    else if (kind == 3) out = E;
    else if (kind == 4) out = beta * D * dots[warp][lane - 16];
    else if (kind == 5) out = D * dots[warp][lane - 16];
    a.coefs[((size_t)(t >> 2) * a.heads + h) * HD_COEFS + lane] = out;
  }
}

// Two floats in one register pair (the packed fp32 operations of sm_100).
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 pack2(float lo, float hi) {
  f32x2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
  return r;
}
__device__ __forceinline__ void unpack2(f32x2 v, float& lo, float& hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v)); }
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
  f32x2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
  f32x2 r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
struct __align__(16) Quad { f32x2 lo, hi; };      // four neighbouring rows

// RS lanes share a column, R rows each (rows 4 (rs + RS j) .. + 3); DP = RS R rows, those beyond d are zero.
template <int RS, int R, int COLS, int TCH>
__global__ void __launch_bounds__(COLS / HD_CPT * RS)
hd_rule_kernel(HeadDeltaArgs a, int vec) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int DP = RS * R, NTH = COLS / HD_CPT * RS, NQ = R / 4, NP = R / 2;
  constexpr int STAGE = TCH * (2 * DP + COLS + 2) + (TCH / 4) * HD_COEFS;
  constexpr int PER_LANE = RS >= 16 ? 1 : 16 / RS;      // of a column pair's 16 sums
  // two stages: qk [TCH][2][DP], v [TCH][COLS], gb [TCH][2], the groups' numbers; then two places for the sums of every
  // column pair
  extern __shared__ __align__(16) float hd_smem[];
  const int seq = blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * COLS;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int rs = tid % RS, col = (tid / RS) * HD_CPT;
  float* sums = hd_smem + 2 * STAGE + (tid / RS) * 32;
  const int q_begin = a.cu_q[seq], q_len = a.cu_q[seq + 1] - q_begin;
  if (q_len <= 0) return;
  const int slot = a.slots[seq], d = a.d, dv = a.dv, kvh = h / (a.heads / a.kv_heads);
  float* S_g = a.state + ((size_t)slot * a.heads + h) * d * dv;
  f32x2 S[HD_CPT][NP];                   // rows 2 p, 2 p + 1 of this lane's R in pair p
  bool live[HD_CPT];
#pragma unroll
  for (int cc = 0; cc < HD_CPT; ++cc) live[cc] = c0 + col + cc < dv;
  const bool pair = (dv & 1) == 0;       // both columns of a thread in one 8-byte access (col is even)
#pragma unroll
  for (int p = 0; p < NP; ++p) {
    float x[2][HD_CPT];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int i = 4 * (rs + RS * (p >> 1)) + 2 * (p & 1) + e;
      const float* src = S_g + (size_t)i * dv + c0 + col;
      if (pair) {
        float2 v = make_float2(0.f, 0.f);
        if (i < d && live[0]) v = *(const float2*)src;
        x[e][0] = v.x; x[e][1] = v.y;
      } else {
#pragma unroll
        for (int cc = 0; cc < HD_CPT; ++cc) x[e][cc] = (i < d && live[cc]) ? src[cc] : 0.f;
      }
    }
#pragma unroll
    for (int cc = 0; cc < HD_CPT; ++cc) S[cc][p] = pack2(x[0][cc], x[1][cc]);
  }
  if (d < DP) {                          // the copies never touch the padding rows
    for (int i = tid; i < 2 * TCH * 2 * (DP - d); i += NTH) {
      const int e = i % (DP - d), rest = i / (DP - d), which = rest & 1, tt = (rest >> 1) % TCH, b = (rest >> 1) / TCH;
      hd_smem[(size_t)b * STAGE + (tt * 2 + which) * DP + d + e] = 0.f;
    }
  }
  auto issue = [&](int chunk) {
    float* buf = hd_smem + (size_t)(chunk & 1) * STAGE;
    const int base = q_begin + chunk * TCH, nt = min(TCH, q_len - chunk * TCH);
    // a warp copies token after token: q and k lie side by side
    for (int tt = warp; tt < nt; tt += NTH / 32) {
      const float* src = a.qk + ((size_t)(base + tt) * a.kv_heads + kvh) * 2 * d;
      float* dst = buf + tt * 2 * DP;
      if (vec) {
        for (int i = 4 * lane; i < d; i += 128) { hd_cp16(dst + i, src + i); hd_cp16(dst + DP + i, src + d + i); }
      } else {
        for (int i = lane; i < d; i += 32) { hd_cp4(dst + i, src + i); hd_cp4(dst + DP + i, src + d + i); }
      }
    }
    float* vs = buf + TCH * 2 * DP;
    for (int i = tid; i < nt * COLS; i += NTH) {
      const int tt = i / COLS, cc = i % COLS;
      if (c0 + cc < dv) hd_cp4(vs + i, a.o + (size_t)(base + tt) * a.heads * dv + (size_t)h * dv + c0 + cc);
      else vs[i] = 0.f;
    }
    float* gs = vs + TCH * COLS;
    if (tid < nt * 2) hd_cp4(gs + tid, a.gb + ((size_t)(base + tid / 2) * a.heads + h) * 2 + (tid & 1));
    float* cf = gs + TCH * 2;
    for (int i = tid; i < nt / 4 * (HD_COEFS / 4); i += NTH) {
      const int grp = i / (HD_COEFS / 4), e = 4 * (i % (HD_COEFS / 4));
      hd_cp16(cf + grp * HD_COEFS + e, a.coefs + ((size_t)((base + 4 * grp) >> 2) * a.heads + h) * HD_COEFS + e);
    }
    hd_cp_commit();
  };

  const int n_chunks = (q_len + TCH - 1) / TCH;
  issue(0);
  for (int chunk = 0; chunk < n_chunks; ++chunk) {
    hd_cp_wait_all();
    __syncthreads();                     // this chunk is there; everybody has left the one before, whose buffer is free
    const int nt = min(TCH, q_len - chunk * TCH);
    if (chunk + 1 < n_chunks) issue(chunk + 1);
    const float* buf = hd_smem + (size_t)(chunk & 1) * STAGE;
    const float* vs = buf + TCH * 2 * DP;
    const float* gs = vs + TCH * COLS;
    const float* cfs = gs + TCH * 2;
    const int groups = nt / 4;
    float* o_row = a.o + (size_t)(q_begin + chunk * TCH) * a.heads * dv + (size_t)h * dv + c0 + col;
    const size_t o_step = (size_t)a.heads * dv;
    auto store = [&](int tt, const float* o) {
      float* dst = o_row + (size_t)tt * o_step;
      if (pair) { if (live[0]) *(float2*)dst = make_float2(o[0], o[1]); }
      else {
#pragma unroll
        for (int cc = 0; cc < HD_CPT; ++cc) if (live[cc]) dst[cc] = o[cc];
      }
    };
    for (int grp = 0; grp < groups; ++grp) {
      const float* tok = buf + grp * 4 * 2 * DP + 4 * rs;
      float part[16];                    // S^T k_i of column cc at 4 cc + i, S^T q_i at 8 + 4 cc + i: this lane's rows
      {
        f32x2 acc[16];
#pragma unroll
        for (int x = 0; x < 16; ++x) acc[x] = 0ull;
#pragma unroll
        for (int j = 0; j < NQ; ++j) {
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const Quad q = *(const Quad*)(tok + i * 2 * DP + 4 * RS * j), k = *(const Quad*)(tok + i * 2 * DP + DP + 4 * RS * j);
#pragma unroll
            for (int cc = 0; cc < HD_CPT; ++cc) {
              acc[4 * cc + i] = fma2(S[cc][2 * j], k.lo, acc[4 * cc + i]);
              acc[4 * cc + i] = fma2(S[cc][2 * j + 1], k.hi, acc[4 * cc + i]);
              acc[8 + 4 * cc + i] = fma2(S[cc][2 * j], q.lo, acc[8 + 4 * cc + i]);
              acc[8 + 4 * cc + i] = fma2(S[cc][2 * j + 1], q.hi, acc[8 + 4 * cc + i]);
            }
          }
        }
#pragma unroll
        for (int x = 0; x < 16; ++x) {
          float lo, hi;
          unpack2(acc[x], lo, hi);
          part[x] = lo + hi;
        }
      }
      // sums over the column's lanes, each lane keeping its share of the 16; all of them through shared memory (two places
      // in turn: a lane that is one group ahead writes the other)
      float* place = sums + (grp & 1) * 16;
      int width = 16;
#pragma unroll
      for (int m = RS >> 1; m > 0; m >>= 1) {
        if (width > 1) {
          width >>= 1;
          const bool upper = (rs & m) != 0;
#pragma unroll
          for (int x = 0; x < 8; ++x)
            if (x < width) {
              const float keep = upper ? part[x + width] : part[x], send = upper ? part[x] : part[x + width];
              part[x] = keep + __shfl_xor_sync(0xffffffffu, send, m);
            }
        } else {
          part[0] += __shfl_xor_sync(0xffffffffu, part[0], m);
        }
      }
      // RS = 32: the last halving added the same sum in both lanes of a pair
      const int first = RS >= 16 ? rs / (RS / 16) : rs * PER_LANE;
#pragma unroll
      for (int x = 0; x < PER_LANE; ++x) place[first + x] = part[x];
      __syncwarp();
      const float* cf = cfs + grp * HD_COEFS;
      const float4 b4 = *(const float4*)cf, bG4 = *(const float4*)(cf + 4), G4 = *(const float4*)(cf + 8), E4 = *(const float4*)(cf + 12);
      const float bi[4] = {b4.x, b4.y, b4.z, b4.w}, bG[4] = {bG4.x, bG4.y, bG4.z, bG4.w}, Gi[4] = {G4.x, G4.y, G4.z, G4.w},
                  Ei[4] = {E4.x, E4.y, E4.z, E4.w};
      float pairs[16];                   // the rest of the numbers, CK(1, 0) first
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const float4 v = *(const float4*)(cf + 16 + 4 * x);
        pairs[4 * x] = v.x; pairs[4 * x + 1] = v.y; pairs[4 * x + 2] = v.z; pairs[4 * x + 3] = v.w;
      }
      float sk[HD_CPT][4], sq[HD_CPT][4], vv[4][HD_CPT], o[4][HD_CPT];
#pragma unroll
      for (int cc = 0; cc < HD_CPT; ++cc) {
        const float4 k = *(const float4*)(place + 4 * cc), q = *(const float4*)(place + 8 + 4 * cc);
        sk[cc][0] = k.x; sk[cc][1] = k.y; sk[cc][2] = k.z; sk[cc][3] = k.w;
        sq[cc][0] = q.x; sq[cc][1] = q.y; sq[cc][2] = q.z; sq[cc][3] = q.w;
      }
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float2 v = *(const float2*)(vs + (grp * 4 + i) * COLS + col);
        vv[i][0] = v.x; vv[i][1] = v.y;
      }
      f32x2 uu[4][HD_CPT];               // D_3i u_i, twice
#pragma unroll
      for (int cc = 0; cc < HD_CPT; ++cc) {
        float u[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          float x = fmaf(-bG[i], sk[cc][i], bi[i] * vv[i][cc]);
          float y = Gi[i] * sq[cc][i];
#pragma unroll
          for (int j = 0; j < i; ++j) {
            x = fmaf(-pairs[CK(i, j) - 16], u[j], x);
            y = fmaf(pairs[CQ(i, j) - 16], u[j], y);
          }
          u[i] = x;
          o[i][cc] = fmaf(pairs[CQ(i, i) - 16], x, y);
          uu[i][cc] = pack2(x * Ei[i], x * Ei[i]);
        }
      }
      if (rs == 0) {
#pragma unroll
        for (int i = 0; i < 4; ++i) store(grp * 4 + i, o[i]);
      }
      const f32x2 GG = pack2(Gi[3], Gi[3]);
#pragma unroll
      for (int j = 0; j < NQ; ++j) {
#pragma unroll
        for (int cc = 0; cc < HD_CPT; ++cc) { S[cc][2 * j] = mul2(S[cc][2 * j], GG); S[cc][2 * j + 1] = mul2(S[cc][2 * j + 1], GG); }
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const Quad k = *(const Quad*)(tok + i * 2 * DP + DP + 4 * RS * j);
#pragma unroll
          for (int cc = 0; cc < HD_CPT; ++cc) {
            S[cc][2 * j] = fma2(k.lo, uu[i][cc], S[cc][2 * j]);
            S[cc][2 * j + 1] = fma2(k.hi, uu[i][cc], S[cc][2 * j + 1]);
          }
        }
      }
    }
    for (int tt = groups * 4; tt < nt; ++tt) {      // the tokens that are left
      const float* tok = buf + tt * 2 * DP + 4 * rs;
      const float g = gs[tt * 2], beta = gs[tt * 2 + 1];
      const f32x2 gg = pack2(g, g);
      f32x2 acc[HD_CPT];
      float dot[HD_CPT], o[HD_CPT];
#pragma unroll
      for (int cc = 0; cc < HD_CPT; ++cc) acc[cc] = 0ull;
#pragma unroll
      for (int j = 0; j < NQ; ++j) {
        const Quad k = *(const Quad*)(tok + DP + 4 * RS * j);
#pragma unroll
        for (int cc = 0; cc < HD_CPT; ++cc) {
          S[cc][2 * j] = mul2(S[cc][2 * j], gg);
          S[cc][2 * j + 1] = mul2(S[cc][2 * j + 1], gg);
          acc[cc] = fma2(S[cc][2 * j], k.lo, acc[cc]);
          acc[cc] = fma2(S[cc][2 * j + 1], k.hi, acc[cc]);
        }
      }
#pragma unroll
      for (int cc = 0; cc < HD_CPT; ++cc) { float lo, hi; unpack2(acc[cc], lo, hi); dot[cc] = lo + hi; acc[cc] = 0ull; }
#pragma unroll
      for (int m = 1; m < RS; m <<= 1)
#pragma unroll
        for (int cc = 0; cc < HD_CPT; ++cc) dot[cc] += __shfl_xor_sync(0xffffffffu, dot[cc], m);
      f32x2 uu[HD_CPT];
#pragma unroll
      for (int cc = 0; cc < HD_CPT; ++cc) {
        const float u = beta * (vs[tt * COLS + col + cc] - dot[cc]);
        uu[cc] = pack2(u, u);
      }
#pragma unroll
      for (int j = 0; j < NQ; ++j) {
        const Quad k = *(const Quad*)(tok + DP + 4 * RS * j), q = *(const Quad*)(tok + 4 * RS * j);
#pragma unroll
        for (int cc = 0; cc < HD_CPT; ++cc) {
          S[cc][2 * j] = fma2(k.lo, uu[cc], S[cc][2 * j]);
          S[cc][2 * j + 1] = fma2(k.hi, uu[cc], S[cc][2 * j + 1]);
          acc[cc] = fma2(S[cc][2 * j], q.lo, acc[cc]);
          acc[cc] = fma2(S[cc][2 * j + 1], q.hi, acc[cc]);
        }
      }
#pragma unroll
      for (int cc = 0; cc < HD_CPT; ++cc) { float lo, hi; unpack2(acc[cc], lo, hi); o[cc] = lo + hi; }
#pragma unroll
      for (int m = 1; m < RS; m <<= 1)
#pragma unroll
        for (int cc = 0; cc < HD_CPT; ++cc) o[cc] += __shfl_xor_sync(0xffffffffu, o[cc], m);
      if (rs == 0) store(tt, o);
    }
  }
#pragma unroll
  for (int p = 0; p < NP; ++p) {
    float x[2][HD_CPT];
#pragma unroll
    for (int cc = 0; cc < HD_CPT; ++cc) unpack2(S[cc][p], x[0][cc], x[1][cc]);
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int i = 4 * (rs + RS * (p >> 1)) + 2 * (p & 1) + e;
      if (i >= d) continue;
      float* dst = S_g + (size_t)i * dv + c0 + col;
      if (pair) { if (live[0]) *(float2*)dst = make_float2(x[e][0], x[e][1]); }
      else {
#pragma unroll
        for (int cc = 0; cc < HD_CPT; ++cc) if (live[cc]) dst[cc] = x[e][cc];
      }
    }
  }
}

// One warp per (token, head).
template <typename T, int V>
__global__ void __launch_bounds__(128)
hd_out_norm_kernel(HeadDeltaArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const long item = (long)blockIdx.x * 4 + (threadIdx.x >> 5);
  if (item >= (long)a.n_tokens * a.heads) return;
  const size_t t = item / a.heads;
  const int h = (int)(item % a.heads);
  const float* o = a.o + item * a.dv;
  const T* gate = (const T*)a.proj + t * a.ld + 2 * a.kv_heads * a.d + a.heads * a.dv + (size_t)h * a.dv;
  T* out = (T*)a.out + item * a.dv;
  float ss = 0.f;
  if (V == 4 && a.dv <= 128) {           // the row in one piece a lane
    const bool in = 4 * lane < a.dv;
    float v[V] = {}, z[V] = {}, w[V] = {};
    if (in) { hd_loadf<V>(o + 4 * lane, v); hd_loadt<T, V>(gate + 4 * lane, z); hd_loadf<V>(a.norm_w + 4 * lane, w); }
#pragma unroll
    for (int e = 0; e < V; ++e) ss = fmaf(v[e], v[e], ss);
    ss = warp_sum(ss);
    const float inv = 1.0f / sqrtf(ss / (float)a.dv + a.eps);
    if (in) {
#pragma unroll
      for (int e = 0; e < V; ++e) v[e] = v[e] * inv * w[e] * (z[e] / (1.f + expf(-z[e])));
      if (sizeof(T) == 4) hd_storef<V>((float*)out + 4 * lane, v);
      else {
        uint2 r;
        *(__nv_bfloat162*)&r.x = __floats2bfloat162_rn(v[0], v[1 % V]);
        *(__nv_bfloat162*)&r.y = __floats2bfloat162_rn(v[2 % V], v[3 % V]);
        *(uint2*)((bf16*)out + 4 * lane) = r;
      }
    }
    return;
  }
  for (int i = lane; i < a.dv; i += 32) ss = fmaf(o[i], o[i], ss);
  ss = warp_sum(ss);
  const float inv = 1.0f / sqrtf(ss / (float)a.dv + a.eps);
  for (int i = lane; i < a.dv; i += 32) {
    const float z = to_f<T>(gate[i]);
    out[i] = from_f<T>(o[i] * inv * a.norm_w[i] * (z / (1.f + expf(-z))));
  }
}

template <int RS, int R, int COLS, int TCH>
static int launch_rule(const HeadDeltaArgs& a, cudaStream_t stream) {
  constexpr int DP = RS * R;
  constexpr size_t smem = sizeof(float) * (2 * ((size_t)TCH * (2 * DP + COLS + 2) + (TCH / 4) * HD_COEFS) + COLS / HD_CPT * 32);
  auto kernel = hd_rule_kernel<RS, R, COLS, TCH>;
  static bool configured = false;
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  const dim3 grid((a.dv + COLS - 1) / COLS, a.heads, a.n_seqs);
  const int vec = a.d % 4 == 0 && ((uintptr_t)a.qk & 15) == 0;
  // Prompts: an ordinary launch.  Started early, while the kernels before still hold the multiprocessors, the few long
  // blocks of a single prompt would be packed several to one and stay there (measured: 2,048 tokens, 16 heads of 128:
  // 1,040 us packed, 440 us spread).
  if (a.max_q_len > 1) {
    kernel<<<grid, dim3(COLS / HD_CPT * RS), smem, stream>>>(a, vec);
    return (int)cudaPeekAtLastError();
  }
  return launch_pdl(kernel, grid, dim3(COLS / HD_CPT * RS), smem, stream, a, vec);
}

// DP rows.  A lane takes 16 of a column's rows and a block 32 columns when that makes two blocks per multiprocessor.  A
// step of one long sequence has nothing else to run beside it, and its time is its tokens' chain of instructions: there
// a lane takes 8 rows and a block 16 columns, and when such blocks leave multiprocessors idle 4 rows (and 8 columns).
// Measured, 2,048 tokens of one sequence, heads of 128 x 128, the whole mixer between its products, us: 16 heads 531 with 8
// rows, 473 with 4; 32 heads 696 and 724; 8 heads 518, 457, and 405 with 8 columns
// (heads of 64 x 64 lose with 8 columns: 419 and 473).
template <int DP, int TCH>
static int launch_rule_form(const HeadDeltaArgs& a, cudaStream_t stream) {
  const long heads = (long)a.heads * a.n_seqs;
  const bool narrow = heads * ((a.dv + 31) / 32) < 2 * 148, few = heads * ((a.dv + 15) / 16) <= 148;
  constexpr int WIDE = DP / 16, NARROW = DP / 8, NARROWEST = DP / 4;
  if constexpr (NARROWEST == 32) {
    if (narrow && few && heads * ((a.dv + 7) / 8) <= 148) return launch_rule<NARROWEST, 4, 8, TCH>(a, stream);
  }
  if constexpr (NARROWEST <= 32 && NARROWEST >= 4) {
    if (narrow && few) return launch_rule<NARROWEST, 4, 16, TCH>(a, stream);
  }
  if constexpr (NARROW <= 32 && NARROW >= 4) {
    if (narrow) return launch_rule<NARROW, 8, 16, TCH>(a, stream);
  }
  if constexpr (WIDE >= 2) return launch_rule<WIDE, 16, 32, TCH>(a, stream);
  else return launch_rule<1, 16, 64, TCH>(a, stream);
}

template <typename T>
static int launch_head_delta(const HeadDeltaArgs& a, cudaStream_t stream) {
  const int C = 2 * a.kv_heads * a.d + a.heads * a.dv;
  // few tokens: a token's heads over several blocks
  const int parts = a.n_tokens >= 296 ? 1 : min(a.kv_heads, (296 + a.n_tokens - 1) / a.n_tokens);
  const size_t smem = sizeof(float) * 2 * (size_t)((a.kv_heads + parts - 1) / parts) * a.d;
  if (smem > 200 * 1024) return ODI_ERR_UNSUPPORTED;
  const bool vec = a.d % 4 == 0 && a.dv % 4 == 0 && a.ld % 4 == 0 &&
                   (((uintptr_t)a.proj | (uintptr_t)a.taps | (uintptr_t)a.conv_state | (uintptr_t)a.o) & 15) == 0;
  auto prep = vec ? hd_prep_kernel<T, 4> : hd_prep_kernel<T, 1>;
  if (smem > 48 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute(prep, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  odi_rc = launch_pdl(prep, dim3(a.n_tokens, parts), dim3(256), smem, stream, a);
  if (odi_rc == 0 && a.taps_n > 1 && a.max_q_len > 1)
    odi_rc = launch_pdl((hd_conv_state_kernel<T>), dim3(a.n_seqs, (C + 255) / 256), dim3(256), 0, stream, a);
  if (odi_rc == 0 && a.max_q_len >= 4)
    odi_rc = launch_pdl(hd_groups_kernel, dim3((unsigned)(((long)a.n_tokens * a.kv_heads + 3) / 4)), dim3(128), 0, stream, a);
  if (odi_rc == 0) {
    if (a.d <= 16) odi_rc = launch_rule_form<16, 16>(a, stream);
    else if (a.d <= 32) odi_rc = launch_rule_form<32, 16>(a, stream);
    else if (a.d <= 64) odi_rc = launch_rule_form<64, 16>(a, stream);
    else if (a.d <= 128) odi_rc = launch_rule_form<128, 16>(a, stream);
    else if (a.d <= 256) odi_rc = launch_rule_form<256, 16>(a, stream);
    else odi_rc = launch_rule_form<512, 8>(a, stream);
  }
  if (odi_rc == 0)
    odi_rc = launch_pdl((vec && ((uintptr_t)a.out | (uintptr_t)a.norm_w) % 16 == 0 ? hd_out_norm_kernel<T, 4> : hd_out_norm_kernel<T, 1>), dim3((unsigned)(((long)a.n_tokens * a.heads + 3) / 4)), dim3(128), 0, stream, a);
  return launch_status();
}

// Kernels launched by one call: 3, one more with a convolution state to move on after a step of several tokens, one more
// when a sequence brings four tokens or more.
extern "C" int odi_head_delta(const HeadDeltaArgs* args, int dtype, cudaStream_t stream) {
  const HeadDeltaArgs a = *args;
  if (a.n_tokens <= 0 || a.n_seqs <= 0) return 0;
  if (a.heads <= 0 || a.kv_heads <= 0 || a.heads % a.kv_heads != 0 || a.d <= 0 || a.dv <= 0 || a.taps_n < 1) return ODI_ERR_ARGUMENT;
  if (a.d > 512 || a.taps_n > HD_MAX_TAPS || a.heads > 65535 || a.n_seqs > 65535) return ODI_ERR_UNSUPPORTED;
  if (a.taps_n > 1 && a.conv_state == nullptr) return ODI_ERR_ARGUMENT;
  return dtype == 0 ? launch_head_delta<float>(a, stream) : launch_head_delta<bf16>(a, stream);
}
