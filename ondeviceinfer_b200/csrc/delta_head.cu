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
//  rule       the recurrence: a block per (sequence, head, block of COLS value columns); a column of S lies in the
//             registers of RS neighbouring lanes, R rows each, two columns a thread; 16 tokens of q, k, v and the
//             decays are staged in shared memory, the next 16 by asynchronous copies meanwhile;
//  out_norm   per (token, head): o / rms(o) (eps inside the root) * weight * silu(gate), rounded once to T.
#include "common.cuh"

#define HD_MAX_TAPS 16
#define HD_CPT 2            // value columns per thread
#define HD_COEFS 40         // floats of a group of four tokens: see group_coefs

struct HeadDeltaArgs {
  const void* proj;       // [n_tokens, ld] in T: q (kv_heads d), k (kv_heads d), v (heads dv), gate (heads dv)
  const float* ab;        // [n_tokens, 2 heads]: a, then b
  const float* taps;      // [C, taps_n], C = 2 kv_heads d + heads dv
  const float* a_log;     // [heads]
  const float* dt_bias;   // [heads]
  const float* norm_w;    // [dv]
  float* conv_state;      // [slots, taps_n - 1, C]; null when taps_n == 1
  float* state;           // [slots, heads, d, dv]
  float* qk;              // [n_tokens, kv_heads, 2, d] scratch: unit q (scaled), unit k
  float* gb;              // [n_tokens, heads, 2] scratch: decay, step size
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

template <typename T>
__global__ void __launch_bounds__(256)
hd_prep_kernel(HeadDeltaArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float ys[];          // [2 kv_heads d]: q and k behind the convolution
  const int t = blockIdx.x;
  const int qk_n = 2 * a.kv_heads * a.d, vn = a.heads * a.dv, C = qk_n + vn;
  const int seq = a.tok_seq[t];
  const int q_begin = a.cu_q[seq], q_len = a.cu_q[seq + 1] - q_begin, slot = a.slots[seq];
  const int li = t - q_begin, keep = a.taps_n - 1;
  for (int c = threadIdx.x; c < C; c += blockDim.x) {
    float acc = 0.f;
    for (int j = 0; j < a.taps_n; ++j) acc = fmaf(a.taps[(size_t)c * a.taps_n + j], hd_input<T>(a, C, q_begin, slot, li - keep + j, c), acc);
    if (q_len == 1 && keep > 0) {        // this thread is the only one that reads or writes these inputs
      float* st = a.conv_state + (size_t)slot * keep * C + c;
      for (int j = 0; j + 1 < keep; ++j) st[(size_t)j * C] = st[(size_t)(j + 1) * C];
      st[(size_t)(keep - 1) * C] = to_f<T>(((const T*)a.proj)[(size_t)t * a.ld + c]);
    }
    const float y = acc / (1.f + expf(-acc));
    if (c < qk_n) ys[c] = y;
    else a.o[(size_t)t * vn + (c - qk_n)] = y;
  }
  for (int h = threadIdx.x; h < a.heads; h += blockDim.x) {
    const float* row = a.ab + (size_t)t * 2 * a.heads;
    const float decay = expf(-expf(a.a_log[h]) * hd_softplus(row[h] + a.dt_bias[h]));
    float* dst = a.gb + ((size_t)t * a.heads + h) * 2;
    dst[0] = decay;
    dst[1] = 1.f / (1.f + expf(-row[a.heads + h]));
  }
  __syncthreads();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
  for (int w = warp; w < 2 * a.kv_heads; w += n_warps) {      // the q heads, then the k heads
    const float* src = ys + (size_t)w * a.d;
    float ss = 0.f;
    for (int i = lane; i < a.d; i += 32) ss = fmaf(src[i], src[i], ss);
    ss = warp_sum(ss);
    const bool is_k = w >= a.kv_heads;
    const float scale = 1.0f / sqrtf(ss + a.unit_eps) * (is_k ? 1.f : 1.0f / sqrtf((float)a.d));
    float* dst = a.qk + (((size_t)t * a.kv_heads + (is_k ? w - a.kv_heads : w)) * 2 + (is_k ? 1 : 0)) * a.d;
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

// Where a group's numbers lie: ck[i][j] = beta_i D_ij (k_j . k_i) at 4 i + j (j < i), cq[i][j] = D_ij (k_j . q_i) at
// 16 + 4 i + j (j <= i), then G_i at 32 + i and D_3i at 36 + i.
// RS lanes share a column, R rows each (rows 4 (rs + RS j) .. + 3); DP = RS R rows, those beyond d are zero.
template <int RS, int R, int COLS, int TCH>
__global__ void __launch_bounds__(COLS / HD_CPT * RS)
hd_rule_kernel(HeadDeltaArgs a, int vec) {
  pdl_launch_dependents();
  pdl_wait();
  constexpr int DP = RS * R, NTH = COLS / HD_CPT * RS, NQ = R / 4;
  constexpr int STAGE = TCH * (2 * DP + COLS + 2);
  extern __shared__ __align__(16) float hd_smem[];      // two stages: qk [TCH][2][DP], v [TCH][COLS], gb [TCH][2]; then the groups' numbers
  float* coefs = hd_smem + 2 * STAGE;                   // [TCH / 4][HD_COEFS]
  const int seq = blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * COLS;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int rs = tid % RS, col = (tid / RS) * HD_CPT;
  const int q_begin = a.cu_q[seq], q_len = a.cu_q[seq + 1] - q_begin;
  if (q_len <= 0) return;
  const int slot = a.slots[seq], d = a.d, dv = a.dv, kvh = h / (a.heads / a.kv_heads);
  float* S_g = a.state + ((size_t)slot * a.heads + h) * d * dv;
  float S[HD_CPT][R];
  bool live[HD_CPT];
#pragma unroll
  for (int cc = 0; cc < HD_CPT; ++cc) live[cc] = c0 + col + cc < dv;
  const bool pair = (dv & 1) == 0;       // both columns of a thread in one 8-byte access (col is even)
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int i = 4 * (rs + RS * (r >> 2)) + (r & 3);
    const float* src = S_g + (size_t)i * dv + c0 + col;
    if (pair) {
      float2 v = make_float2(0.f, 0.f);
      if (i < d && live[0]) v = *(const float2*)src;
      S[0][r] = v.x; S[1][r] = v.y;
    } else {
#pragma unroll
      for (int cc = 0; cc < HD_CPT; ++cc) S[cc][r] = (i < d && live[cc]) ? src[cc] : 0.f;
    }
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
    const int groups = nt / 4;
    // the groups' numbers: a warp per pair (i, j), j <= i, of a group
    for (int p = warp; p < groups * 10; p += NTH / 32) {
      const int grp = p / 10, r = p % 10;
      const int i = r < 1 ? 0 : (r < 3 ? 1 : (r < 6 ? 2 : 3)), j = r - i * (i + 1) / 2;
      const float* ti = buf + (grp * 4 + i) * 2 * DP;
      const float* kj = buf + (grp * 4 + j) * 2 * DP + DP;
      float kk = 0.f, kq = 0.f;
      for (int e = 4 * lane; e < DP; e += 128) {
        const float4 q = *(const float4*)(ti + e), k = *(const float4*)(ti + DP + e), w = *(const float4*)(kj + e);
        kk += k.x * w.x + k.y * w.y + k.z * w.z + k.w * w.w;
        kq += q.x * w.x + q.y * w.y + q.z * w.z + q.w * w.w;
      }
      kk = warp_sum(kk);
      kq = warp_sum(kq);
      if (lane == 0) {
        const float* g = gs + grp * 8;
        float* out = coefs + grp * HD_COEFS;
        float D = 1.f;
        for (int m = j + 1; m <= i; ++m) D *= g[2 * m];
        out[16 + 4 * i + j] = D * kq;
        if (j < i) out[4 * i + j] = g[2 * i + 1] * D * kk;
        else {
          float G = 1.f, E = 1.f;
          for (int m = 0; m <= i; ++m) G *= g[2 * m];
          for (int m = i + 1; m < 4; ++m) E *= g[2 * m];
          out[32 + i] = G;
          out[36 + i] = E;
        }
      }
    }
    __syncthreads();
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
      const float* tok = buf + grp * 4 * 2 * DP;
      const float* cf = coefs + grp * HD_COEFS;
      float sk[4][HD_CPT] = {}, sq[4][HD_CPT] = {};
#pragma unroll
      for (int j = 0; j < NQ; ++j) {
        const int e = 4 * (rs + RS * j);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float4 q = *(const float4*)(tok + i * 2 * DP + e), k = *(const float4*)(tok + i * 2 * DP + DP + e);
#pragma unroll
          for (int cc = 0; cc < HD_CPT; ++cc) {
            const float* s = &S[cc][4 * j];
            sk[i][cc] = fmaf(s[0], k.x, sk[i][cc]); sk[i][cc] = fmaf(s[1], k.y, sk[i][cc]);
            sk[i][cc] = fmaf(s[2], k.z, sk[i][cc]); sk[i][cc] = fmaf(s[3], k.w, sk[i][cc]);
            sq[i][cc] = fmaf(s[0], q.x, sq[i][cc]); sq[i][cc] = fmaf(s[1], q.y, sq[i][cc]);
            sq[i][cc] = fmaf(s[2], q.z, sq[i][cc]); sq[i][cc] = fmaf(s[3], q.w, sq[i][cc]);
          }
        }
      }
#pragma unroll
      for (int m = 1; m < RS; m <<= 1) {
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int cc = 0; cc < HD_CPT; ++cc) {
            sk[i][cc] += __shfl_xor_sync(0xffffffffu, sk[i][cc], m);
            sq[i][cc] += __shfl_xor_sync(0xffffffffu, sq[i][cc], m);
          }
      }
      const float4 G = *(const float4*)(cf + 32), E = *(const float4*)(cf + 36);
      const float Gi[4] = {G.x, G.y, G.z, G.w}, Ei[4] = {E.x, E.y, E.z, E.w};
      float u[4][HD_CPT];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float beta = gs[(grp * 4 + i) * 2 + 1];
        const float2 v = *(const float2*)(vs + (grp * 4 + i) * COLS + col);
        const float vv[2] = {v.x, v.y};
        float o[HD_CPT];
#pragma unroll
        for (int cc = 0; cc < HD_CPT; ++cc) {
          float x = beta * fmaf(-Gi[i], sk[i][cc], vv[cc]);
          float y = Gi[i] * sq[i][cc];
#pragma unroll
          for (int j = 0; j < i; ++j) {
            x = fmaf(-cf[4 * i + j], u[j][cc], x);
            y = fmaf(cf[16 + 4 * i + j], u[j][cc], y);
          }
          u[i][cc] = x;
          o[cc] = fmaf(cf[16 + 5 * i], x, y);
        }
        if (rs == 0) store(grp * 4 + i, o);
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int cc = 0; cc < HD_CPT; ++cc) u[i][cc] *= Ei[i];
#pragma unroll
      for (int j = 0; j < NQ; ++j) {
        const int e = 4 * (rs + RS * j);
        float4 k[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) k[i] = *(const float4*)(tok + i * 2 * DP + DP + e);
#pragma unroll
        for (int cc = 0; cc < HD_CPT; ++cc) {
          float* s = &S[cc][4 * j];
          s[0] *= Gi[3]; s[1] *= Gi[3]; s[2] *= Gi[3]; s[3] *= Gi[3];
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            s[0] = fmaf(k[i].x, u[i][cc], s[0]); s[1] = fmaf(k[i].y, u[i][cc], s[1]);
            s[2] = fmaf(k[i].z, u[i][cc], s[2]); s[3] = fmaf(k[i].w, u[i][cc], s[3]);
          }
        }
      }
    }
    for (int tt = groups * 4; tt < nt; ++tt) {      // the tokens that are left
      const float* tok = buf + tt * 2 * DP;
      const float g = gs[tt * 2], beta = gs[tt * 2 + 1];
      float dot[HD_CPT] = {}, o[HD_CPT] = {};
#pragma unroll
      for (int j = 0; j < NQ; ++j) {
        const float4 k = *(const float4*)(tok + DP + 4 * (rs + RS * j));
#pragma unroll
        for (int cc = 0; cc < HD_CPT; ++cc) {
          float* s = &S[cc][4 * j];
          s[0] *= g; s[1] *= g; s[2] *= g; s[3] *= g;
          dot[cc] += s[0] * k.x + s[1] * k.y + s[2] * k.z + s[3] * k.w;
        }
      }
#pragma unroll
      for (int m = 1; m < RS; m <<= 1)
#pragma unroll
        for (int cc = 0; cc < HD_CPT; ++cc) dot[cc] += __shfl_xor_sync(0xffffffffu, dot[cc], m);
      float u[HD_CPT];
#pragma unroll
      for (int cc = 0; cc < HD_CPT; ++cc) u[cc] = beta * (vs[tt * COLS + col + cc] - dot[cc]);
#pragma unroll
      for (int j = 0; j < NQ; ++j) {
        const float4 k = *(const float4*)(tok + DP + 4 * (rs + RS * j)), q = *(const float4*)(tok + 4 * (rs + RS * j));
#pragma unroll
        for (int cc = 0; cc < HD_CPT; ++cc) {
          float* s = &S[cc][4 * j];
          s[0] = fmaf(k.x, u[cc], s[0]); s[1] = fmaf(k.y, u[cc], s[1]); s[2] = fmaf(k.z, u[cc], s[2]); s[3] = fmaf(k.w, u[cc], s[3]);
          o[cc] += s[0] * q.x + s[1] * q.y + s[2] * q.z + s[3] * q.w;
        }
      }
#pragma unroll
      for (int m = 1; m < RS; m <<= 1)
#pragma unroll
        for (int cc = 0; cc < HD_CPT; ++cc) o[cc] += __shfl_xor_sync(0xffffffffu, o[cc], m);
      if (rs == 0) store(tt, o);
    }
  }
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int i = 4 * (rs + RS * (r >> 2)) + (r & 3);
    if (i >= d) continue;
    float* dst = S_g + (size_t)i * dv + c0 + col;
    if (pair) { if (live[0]) *(float2*)dst = make_float2(S[0][r], S[1][r]); }
    else {
#pragma unroll
      for (int cc = 0; cc < HD_CPT; ++cc) if (live[cc]) dst[cc] = S[cc][r];
    }
  }
}

// One warp per (token, head).
template <typename T>
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
  float ss = 0.f;
  for (int i = lane; i < a.dv; i += 32) ss = fmaf(o[i], o[i], ss);
  ss = warp_sum(ss);
  const float inv = 1.0f / sqrtf(ss / (float)a.dv + a.eps);
  T* out = (T*)a.out + item * a.dv;
  for (int i = lane; i < a.dv; i += 32) {
    const float z = to_f<T>(gate[i]);
    out[i] = from_f<T>(o[i] * inv * a.norm_w[i] * (z / (1.f + expf(-z))));
  }
}

template <int RS, int R, int COLS, int TCH>
static int launch_rule(const HeadDeltaArgs& a, cudaStream_t stream) {
  constexpr int DP = RS * R;
  const size_t smem = sizeof(float) * (2 * (size_t)TCH * (2 * DP + COLS + 2) + (TCH / 4) * HD_COEFS);
  auto kernel = hd_rule_kernel<RS, R, COLS, TCH>;
  static bool configured = false;
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  const dim3 grid((a.dv + COLS - 1) / COLS, a.heads, a.n_seqs);
  const int vec = a.d % 4 == 0 && ((uintptr_t)a.qk & 15) == 0;
  return launch_pdl(kernel, grid, dim3(COLS / HD_CPT * RS), smem, stream, a, vec);
}

// Fewer columns a block make more blocks: a step of one long sequence has nothing else to run beside it.
template <int RS, int R, int TCH>
static int launch_rule_cols(const HeadDeltaArgs& a, cudaStream_t stream) {
  const long heads = (long)a.heads * a.n_seqs;
  if constexpr (RS >= 4) {
    if (heads * ((a.dv + 31) / 32) < 148) return launch_rule<RS, R, 16, TCH>(a, stream);
  }
  if constexpr (RS == 1) return launch_rule<RS, R, 64, TCH>(a, stream);
  else return launch_rule<RS, R, 32, TCH>(a, stream);
}

template <typename T>
static int launch_head_delta(const HeadDeltaArgs& a, cudaStream_t stream) {
  const int C = 2 * a.kv_heads * a.d + a.heads * a.dv;
  const size_t smem = sizeof(float) * 2 * (size_t)a.kv_heads * a.d;
  if (smem > 48 * 1024) {
    if (smem > 200 * 1024) return ODI_ERR_UNSUPPORTED;
    const cudaError_t e = cudaFuncSetAttribute(hd_prep_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  odi_rc = launch_pdl((hd_prep_kernel<T>), dim3(a.n_tokens), dim3(256), smem, stream, a);
  if (odi_rc == 0 && a.taps_n > 1 && a.max_q_len > 1)
    odi_rc = launch_pdl((hd_conv_state_kernel<T>), dim3(a.n_seqs, (C + 255) / 256), dim3(256), 0, stream, a);
  if (odi_rc == 0) {
    if (a.d <= 16) odi_rc = launch_rule_cols<1, 16, 16>(a, stream);
    else if (a.d <= 32) odi_rc = launch_rule_cols<2, 16, 16>(a, stream);
    else if (a.d <= 64) odi_rc = launch_rule_cols<4, 16, 16>(a, stream);
    else if (a.d <= 128) odi_rc = launch_rule_cols<8, 16, 16>(a, stream);
    else if (a.d <= 256) odi_rc = launch_rule_cols<16, 16, 16>(a, stream);
    else odi_rc = launch_rule_cols<32, 16, 8>(a, stream);
  }
  if (odi_rc == 0)
    odi_rc = launch_pdl((hd_out_norm_kernel<T>), dim3((unsigned)(((long)a.n_tokens * a.heads + 3) / 4)), dim3(128), 0, stream, a);
  return launch_status();
}

// Kernels launched by one call: 3, or 4 with a convolution state to move on after a step of several tokens.
extern "C" int odi_head_delta(const HeadDeltaArgs* args, int dtype, cudaStream_t stream) {
  const HeadDeltaArgs a = *args;
  if (a.n_tokens <= 0 || a.n_seqs <= 0) return 0;
  if (a.heads <= 0 || a.kv_heads <= 0 || a.heads % a.kv_heads != 0 || a.d <= 0 || a.dv <= 0 || a.taps_n < 1) return ODI_ERR_ARGUMENT;
  if (a.d > 512 || a.taps_n > HD_MAX_TAPS || a.heads > 65535 || a.n_seqs > 65535) return ODI_ERR_UNSUPPORTED;
  if (a.taps_n > 1 && a.conv_state == nullptr) return ODI_ERR_ARGUMENT;
  return dtype == 0 ? launch_head_delta<float>(a, stream) : launch_head_delta<bf16>(a, stream);
}
