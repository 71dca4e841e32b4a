// Head preparation of an attention whose heads mix their scores before the softmax, one block per token:
//
//  * the RMS norm of the token's whole q projection (all heads' lanes at once) times a weight per lane, and the same of
//    its k projection (optional);
//  * the rotation of the first rot_dim lanes of every q and k head: lane i turns with lane i + rot_dim / 2 (optional);
//  * the mixed queries (with `talk`, a matrix T [nq, nq]): the mixed score of head h, sum_g T[h, g] q_g . k_kv(g), is the
//    dot product of the row [ sum_(g in group j) T[h, g] q_g ]_j with the position's whole key row [ k_j ]_j, so head h's
//    query becomes that row of nkv * lanes lanes; without it the heads' queries as they are;
//  * k and v to the token's row of their cache pages.
//
// fp32 arithmetic throughout, one rounding at the end.  Stored heads have `lanes` (`v_lanes`) lanes, zero behind the
// head's own d (dv).
#include "common.cuh"

struct MixedPrepArgs {
  const void* qkv;        // [n_tokens, nq d + nkv d + nkv dv] in T
  void* q_out;            // [n_tokens, nq, nkv, lanes] with talk, else [n_tokens, nq, lanes]
  void* k_pool;           // [pages, nkv, page_size, lanes]
  void* v_pool;           // [pages, nkv, page_size, v_lanes]
  const float* q_w;       // [nq d], or null: no norm
  const float* k_w;       // [nkv d]
  const float* talk;      // [nq, nq], or null
  const float* cos_t;     // [n_tokens, rot_dim / 2], or null: no rotation
  const float* sin_t;
  const int* tok_seq;
  const int* tok_pos;
  const int* page_start;
  const int* page_ids;
  int n_tokens, nq, nkv, d, dv, lanes, v_lanes, rot_dim, page_size, ring_pages, write_kv;
  float eps;
  int stage_talk, vec;    // set by the launcher: the matrix goes through shared memory; rows in pieces of 16 bytes
};

template <typename T> __device__ __forceinline__ void store4(T* p, const float* v);
template <> __device__ __forceinline__ void store4<float>(float* p, const float* v) { *(float4*)p = make_float4(v[0], v[1], v[2], v[3]); }
template <> __device__ __forceinline__ void store4<bf16>(bf16* p, const float* v) {
  uint2 r;
  *(__nv_bfloat162*)&r.x = __floats2bfloat162_rn(v[0], v[1]);
  *(__nv_bfloat162*)&r.y = __floats2bfloat162_rn(v[2], v[3]);
  *(uint2*)p = r;
}

// Eight neighbouring elements as floats (16-byte accesses; the caller has checked the alignment).
template <typename T> __device__ __forceinline__ void load8(const T* p, float* v);
template <> __device__ __forceinline__ void load8<float>(const float* p, float* v) {
  const float4 a = *(const float4*)p, b = *(const float4*)(p + 4);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
template <> __device__ __forceinline__ void load8<bf16>(const bf16* p, float* v) {
  const uint4 raw = *(const uint4*)p;
  const __nv_bfloat162* h = (const __nv_bfloat162*)&raw;
#pragma unroll
  for (int i = 0; i < 4; ++i) { const float2 f = __bfloat1622float2(h[i]); v[2 * i] = f.x; v[2 * i + 1] = f.y; }
}

// A block takes one token and, of gridDim.y parts, a range of the output's heads (the first part also writes k and v).
// REP: query heads per key head (0: any number, read from shared memory each time).
template <typename T, int REP>
__global__ void __launch_bounds__(256)
mixed_prep_kernel(MixedPrepArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float smem[];
  __shared__ float scratch[33];
  const int d = a.d, nqd = a.nq * d, nkd = a.nkv * d, lanes = a.lanes;
  float* qs = smem;               // [nq, d]
  float* ks = smem + nqd;         // [nkv, d]
  float* ts = smem + (nqd + nkd + 3) / 4 * 4;      // the matrix, when it is staged
  const int t = blockIdx.x, tid = threadIdx.x;
  const T* row = (const T*)a.qkv + (size_t)t * (nqd + nkd + a.nkv * a.dv);
  float sq = 0.f, sk = 0.f;
  if (a.vec) {          // q and k lie side by side; no piece of eight straddles them
#pragma unroll 4
    for (int i = 8 * tid; i < nqd + nkd; i += 8 * blockDim.x) {
      float v[8], ss = 0.f;
      load8<T>(row + i, v);
#pragma unroll
      for (int e = 0; e < 8; ++e) ss = fmaf(v[e], v[e], ss);
      *(float4*)(smem + i) = make_float4(v[0], v[1], v[2], v[3]);
      *(float4*)(smem + i + 4) = make_float4(v[4], v[5], v[6], v[7]);
      if (i < nqd) sq += ss; else sk += ss;
    }
  } else {
    for (int i = tid; i < nqd; i += blockDim.x) { const float v = to_f<T>(row[i]); qs[i] = v; sq = fmaf(v, v, sq); }
    for (int i = tid; i < nkd; i += blockDim.x) { const float v = to_f<T>(row[nqd + i]); ks[i] = v; sk = fmaf(v, v, sk); }
  }
  if (a.stage_talk)
    for (int i = tid; i < a.nq * a.nq; i += blockDim.x) ts[i] = a.talk[i];
  if (a.q_w != nullptr) {
    sq = block_sum(sq, scratch);
    sk = block_sum(sk, scratch);
    const float qi = 1.0f / sqrtf(sq / (float)nqd + a.eps), ki = 1.0f / sqrtf(sk / (float)nkd + a.eps);
    if (a.vec) {        // each thread's own elements
#pragma unroll 4
      for (int i = 8 * tid; i < nqd + nkd; i += 8 * blockDim.x) {
        const bool is_q = i < nqd;
        float w[8];
        load8<float>(is_q ? a.q_w + i : a.k_w + (i - nqd), w);
        const float r = is_q ? qi : ki;
#pragma unroll
        for (int e = 0; e < 8; ++e) smem[i + e] *= r * w[e];
      }
    } else {
      for (int i = tid; i < nqd; i += blockDim.x) qs[i] *= qi * a.q_w[i];
      for (int i = tid; i < nkd; i += blockDim.x) ks[i] *= ki * a.k_w[i];
    }
  }
  __syncthreads();
  if (a.cos_t != nullptr) {
    const int half = a.rot_dim >> 1;
    for (int i = tid; i < (a.nq + a.nkv) * half; i += blockDim.x) {      // q heads, then k heads, lie one after the other
      const int h = i / half, e = i % half;
      float* x = smem + (size_t)h * d + e;
      const float c = a.cos_t[(size_t)t * half + e], s = a.sin_t[(size_t)t * half + e];
      const float u = x[0], v = x[half];
      x[0] = fmaf(-v, s, u * c);
      x[half] = fmaf(u, s, v * c);
    }
    __syncthreads();
  }
  const int h0 = a.nq * blockIdx.y / gridDim.y, h1 = a.nq * (blockIdx.y + 1) / gridDim.y;
  if (a.write_kv && blockIdx.y == 0) {
    const int pos = a.tok_pos[t];
    const int page = a.page_ids[a.page_start[a.tok_seq[t]] + page_slot_of(pos, a.page_size, a.ring_pages)];
    const size_t at = (size_t)page * a.nkv * a.page_size + pos % a.page_size;
    for (int i = tid; i < a.nkv * lanes; i += blockDim.x) {
      const int j = i / lanes, e = i % lanes;
      ((T*)a.k_pool)[(at + (size_t)j * a.page_size) * lanes + e] = from_f<T>(e < d ? ks[j * d + e] : 0.f);
    }
    for (int i = tid; i < a.nkv * a.v_lanes; i += blockDim.x) {
      const int j = i / a.v_lanes, e = i % a.v_lanes;
      ((T*)a.v_pool)[(at + (size_t)j * a.page_size) * a.v_lanes + e] = e < a.dv ? row[nqd + nkd + j * a.dv + e] : from_f<T>(0.f);
    }
  }
  if (a.talk == nullptr) {
    T* out = (T*)a.q_out + (size_t)t * a.nq * lanes;
    for (int i = h0 * lanes + tid; i < h1 * lanes; i += blockDim.x) {
      const int h = i / lanes, e = i % lanes;
      out[i] = from_f<T>(e < d ? qs[h * d + e] : 0.f);
    }
    return;
  }
  // four neighbouring lanes of a key head's query group a thread; its query heads' values stay in registers
  const int width = a.nkv * lanes, rep = REP > 0 ? REP : a.nq / a.nkv;
  T* out = (T*)a.q_out + (size_t)t * a.nq * width;
  // more threads than groups of four lanes: they share the heads out among themselves
  const int spread = max(1, (int)blockDim.x * 4 / width), sub = 4 * tid / width;
  const int begin = spread > 1 ? h0 + (h1 - h0) * sub / spread : h0, end = spread > 1 ? h0 + (h1 - h0) * (sub + 1) / spread : h1;
  if (spread > 1 && sub >= spread) return;
  for (int p = spread > 1 ? 4 * tid - sub * width : 4 * tid; p < width; p += spread > 1 ? width : 4 * blockDim.x) {
    const int j = p / lanes, e = p % lanes;
    const float* src = qs + (size_t)j * rep * d + e;
    float q[REP > 0 ? REP : 1][4];
    if (REP > 0) {
#pragma unroll
      for (int g = 0; g < REP; ++g)
#pragma unroll
        for (int x = 0; x < 4; ++x) q[g][x] = e + x < d ? src[g * d + x] : 0.f;
    }
    const float* T_j = (a.stage_talk ? ts : a.talk) + j * rep;
#pragma unroll 4
    for (int h = begin; h < end; ++h) {
      float s[4] = {0.f, 0.f, 0.f, 0.f};
      if (REP > 0) {
        float w[REP > 0 ? REP : 1];
        if (REP > 0 && REP % 4 == 0) {
#pragma unroll
          for (int g = 0; g < REP; g += 4) {
            const float4 v = *(const float4*)(T_j + (size_t)h * a.nq + g);
            w[g] = v.x; w[(g + 1) % (REP > 0 ? REP : 1)] = v.y; w[(g + 2) % (REP > 0 ? REP : 1)] = v.z; w[(g + 3) % (REP > 0 ? REP : 1)] = v.w;
          }
        } else {
#pragma unroll
          for (int g = 0; g < REP; ++g) w[g] = T_j[(size_t)h * a.nq + g];
        }
#pragma unroll
        for (int g = 0; g < REP; ++g)
#pragma unroll
          for (int x = 0; x < 4; ++x) s[x] = fmaf(w[g], q[g][x], s[x]);
      } else {
        for (int g = 0; g < rep; ++g) {
          const float w = T_j[(size_t)h * a.nq + g];
#pragma unroll
          for (int x = 0; x < 4; ++x) s[x] = fmaf(w, e + x < d ? src[g * d + x] : 0.f, s[x]);
        }
      }
      store4<T>(out + (size_t)h * width + p, s);
    }
  }
}

template <typename T, int REP>
static int launch_mixed_prep(const MixedPrepArgs& a, size_t smem, cudaStream_t stream) {
  if (smem > 48 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute(mixed_prep_kernel<T, REP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  // few tokens: a token's heads over several blocks
  const int parts = a.n_tokens >= 296 ? 1 : min(a.nq, (296 + a.n_tokens - 1) / a.n_tokens);
  return launch_pdl((mixed_prep_kernel<T, REP>), dim3(a.n_tokens, parts), dim3(a.nq * a.d >= 1024 ? 256 : 128), smem, stream, a);
}

extern "C" int odi_mixed_prep(const MixedPrepArgs* args, int dtype, cudaStream_t stream) {
  MixedPrepArgs a = *args;
  if (a.n_tokens <= 0) return 0;
  if (a.nq <= 0 || a.nkv <= 0 || a.nq % a.nkv != 0 || a.d <= 0 || a.dv <= 0 || a.lanes < a.d || a.v_lanes < a.dv || a.lanes % 4 != 0 || ((uintptr_t)a.talk | (uintptr_t)a.q_out) % 16 != 0 ||
      a.rot_dim > a.d || (a.rot_dim & 1) || (a.q_w == nullptr) != (a.k_w == nullptr))
    return ODI_ERR_ARGUMENT;
  a.stage_talk = a.talk != nullptr && a.nq <= 64 && a.n_tokens >= 296;
  a.vec = a.nq * a.d % 8 == 0 && a.nkv * a.d % 8 == 0 && a.nkv * a.dv % 8 == 0 &&
          ((uintptr_t)a.qkv | (uintptr_t)a.q_w | (uintptr_t)a.k_w) % 16 == 0;
  const size_t smem = sizeof(float) * (((size_t)(a.nq + a.nkv) * a.d + 3) / 4 * 4 + (a.stage_talk ? a.nq * a.nq : 0));
  if (smem > 200 * 1024) return ODI_ERR_UNSUPPORTED;
  const int rep = a.nq / a.nkv;
#define ODI_MP(T) \
  do { if (rep == 1) odi_rc = launch_mixed_prep<T, 1>(a, smem, stream); else if (rep == 2) odi_rc = launch_mixed_prep<T, 2>(a, smem, stream); \
       else if (rep == 4) odi_rc = launch_mixed_prep<T, 4>(a, smem, stream); else if (rep == 8) odi_rc = launch_mixed_prep<T, 8>(a, smem, stream); \
       else odi_rc = launch_mixed_prep<T, 0>(a, smem, stream); } while (0)
  if (dtype == 0) ODI_MP(float); else ODI_MP(bf16);
#undef ODI_MP
  return launch_status();
}
