// Parallel residual streams that every sublayer reads as a weighted sum and mixes anew, with the layer norm that follows.
//
// A token's stream row holds S streams of W fp32 lanes side by side.  One kernel, a block per token, does up to two things
// in one pass over the row:
//   update  x_t <- sum_s mix[s, t] x_s + m out[t] y    for all t at once from the old streams (y: a sublayer's fp32 output)
//   read    u = sum_s in[s] x_s (the new streams);  out = cast((u - mean u) / sqrt(var u + eps) * weight + bias)
// with var the mean of the squared deviations (the row of u stays on chip, so they are taken in a pass of their own).
// Null coefficient pointers stand for the identity: mix = I, out = 1, in = 1.
#include "common.cuh"

#define SM_MAX_STREAMS 16

struct StreamMixArgs {
  float* x;               // [rows of the stream, S, W]
  const float* y;         // [n, W], or null: no update
  const float* mix;       // [S, S] (from, to), or null: every stream keeps itself
  const float* out_c;     // [S], or null: ones
  const float* in_c;      // [S], or null: ones
  const float* weight;    // [W]
  const float* bias;      // [W]
  void* out;              // [n, W] in T, or null: no read
  const int* rows;        // null, or n row numbers of x (without an update)
  int n, S, W;
  float m, eps;
};

// V lanes per access; a thread takes lanes V (tid + j blockDim); NV > 0 keeps the row of u in registers (NV accesses a
// thread), NV = 0 in shared memory.  SC > 0: that many streams; 0: any number up to SM_MAX_STREAMS.
template <typename T, int SC, int V, int NV>
__global__ void __launch_bounds__(512)
stream_mix_kernel(StreamMixArgs a) {
  pdl_launch_dependents();
  constexpr int SX = SC > 0 ? SC : SM_MAX_STREAMS;
  __shared__ float scratch[33], coef[SM_MAX_STREAMS * (SM_MAX_STREAMS + 2)];
  extern __shared__ __align__(16) float row_u[];
  const int S = SC > 0 ? SC : a.S, W = a.W, tid = threadIdx.x;
  // coefficients are weights: no earlier kernel of the stream writes them
  for (int i = tid; i < S * (S + 2); i += blockDim.x) {
    float v;
    if (i < S * S) v = a.mix != nullptr ? a.mix[i] : (i / S == i % S ? 1.f : 0.f);
    else if (i < S * (S + 1)) v = a.m * (a.out_c != nullptr ? a.out_c[i - S * S] : 1.f);
    else v = a.in_c != nullptr ? a.in_c[i - S * (S + 1)] : 1.f;
    coef[i] = v;
  }
  pdl_wait();
  __syncthreads();
  const int r = blockIdx.x;
  float* x = a.x + (size_t)(a.rows != nullptr ? a.rows[r] : r) * S * W;
  const float* y = a.y != nullptr ? a.y + (size_t)r * W : nullptr;
  const float* c_out = coef + S * S;
  const float* c_in = c_out + S;
  float keep[NV > 0 ? NV : 1][V];
  float sum = 0.f;
  auto piece = [&](int i, float* u) {            // lanes i .. i + V - 1: update, and u of the new streams
    float v[SX][V], yy[V];
#pragma unroll
    for (int s = 0; s < SX; ++s)
      if (s < S) {
        if (V == 4) { const float4 f = *(const float4*)(x + (size_t)s * W + i); v[s][0] = f.x; v[s][1 % V] = f.y; v[s][2 % V] = f.z; v[s][3 % V] = f.w; }
        else v[s][0] = x[(size_t)s * W + i];
      }
    if (y != nullptr) {
      if (V == 4) { const float4 f = *(const float4*)(y + i); yy[0] = f.x; yy[1 % V] = f.y; yy[2 % V] = f.z; yy[3 % V] = f.w; }
      else yy[0] = y[i];
    }
#pragma unroll
    for (int e = 0; e < V; ++e) u[e] = 0.f;
#pragma unroll
    for (int t = 0; t < SX; ++t)
      if (t < S) {
        float next[V];
        if (y != nullptr) {
#pragma unroll
          for (int e = 0; e < V; ++e) next[e] = c_out[t] * yy[e];
#pragma unroll
          for (int s = 0; s < SX; ++s)
            if (s < S) {
              const float c = coef[s * S + t];
#pragma unroll
              for (int e = 0; e < V; ++e) next[e] = fmaf(c, v[s][e], next[e]);
            }
          if (V == 4) *(float4*)(x + (size_t)t * W + i) = make_float4(next[0], next[1 % V], next[2 % V], next[3 % V]);
          else x[(size_t)t * W + i] = next[0];
        } else {
#pragma unroll
          for (int e = 0; e < V; ++e) next[e] = v[t][e];
        }
#pragma unroll
        for (int e = 0; e < V; ++e) u[e] = fmaf(c_in[t], next[e], u[e]);
      }
  };
  if (NV > 0) {
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const int i = V * (tid + j * blockDim.x);
      if (i < W) piece(i, keep[j]);
      else {
#pragma unroll
        for (int e = 0; e < V; ++e) keep[j][e] = 0.f;
      }
#pragma unroll
      for (int e = 0; e < V; ++e) sum += keep[j][e];
    }
  } else {
    for (int i = V * tid; i < W; i += V * blockDim.x) {
      float u[V];
      piece(i, u);
#pragma unroll
      for (int e = 0; e < V; ++e) { row_u[i + e] = u[e]; sum += u[e]; }
    }
  }
  if (a.out == nullptr) return;
  const float mean = block_sum(sum, scratch) / (float)W;
  float ss = 0.f;
  if (NV > 0) {
#pragma unroll
    for (int j = 0; j < NV; ++j)
      if (V * (tid + j * (int)blockDim.x) < W) {
#pragma unroll
        for (int e = 0; e < V; ++e) { keep[j][e] -= mean; ss = fmaf(keep[j][e], keep[j][e], ss); }
      }
  } else {
    for (int i = V * tid; i < W; i += V * blockDim.x)
#pragma unroll
      for (int e = 0; e < V; ++e) { const float c = row_u[i + e] - mean; row_u[i + e] = c; ss = fmaf(c, c, ss); }
  }
  const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)W + a.eps);
  T* out = (T*)a.out + (size_t)r * W;
  auto write = [&](int i, const float* c) {
    if (V == 4) {
      const float4 w = *(const float4*)(a.weight + i), b = *(const float4*)(a.bias + i);
      const float o0 = fmaf(c[0] * inv, w.x, b.x), o1 = fmaf(c[1 % V] * inv, w.y, b.y), o2 = fmaf(c[2 % V] * inv, w.z, b.z),
                  o3 = fmaf(c[3 % V] * inv, w.w, b.w);
      if (sizeof(T) == 4) *(float4*)((float*)out + i) = make_float4(o0, o1, o2, o3);
      else {
        uint2 p;
        *(__nv_bfloat162*)&p.x = __floats2bfloat162_rn(o0, o1);
        *(__nv_bfloat162*)&p.y = __floats2bfloat162_rn(o2, o3);
        *(uint2*)((bf16*)out + i) = p;
      }
    } else {
      out[i] = from_f<T>(fmaf(c[0] * inv, a.weight[i], a.bias[i]));
    }
  };
  if (NV > 0) {
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const int i = V * (tid + j * blockDim.x);
      if (i < W) write(i, keep[j]);
    }
  } else {
    for (int i = V * tid; i < W; i += V * blockDim.x) write(i, row_u + i);
  }
}

template <typename T, int SC, int V, int NV>
static int launch_stream_mix(const StreamMixArgs& a, int threads, cudaStream_t stream) {
  auto kernel = stream_mix_kernel<T, SC, V, NV>;
  const size_t smem = NV > 0 ? 0 : (size_t)a.W * sizeof(float);
  if (smem > 40 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  return launch_pdl(kernel, dim3(a.n), dim3(threads), smem, stream, a);
}

template <typename T, int SC>
static int launch_streams(const StreamMixArgs& a, cudaStream_t stream) {
  const bool vec = a.W % 4 == 0 && (((uintptr_t)a.x | (uintptr_t)a.y | (uintptr_t)a.weight | (uintptr_t)a.bias | (uintptr_t)a.out) & 15) == 0;
  if (!vec || SC == 0) return launch_stream_mix<T, SC, 1, 0>(a, a.W >= 2048 ? 512 : (a.W >= 512 ? 256 : 128), stream);
  if constexpr (SC > 0) {       // more streams than that: one lane an access, which keeps the registers in bounds
    const int W4 = a.W / 4;
    const int threads = W4 >= 1024 ? 512 : (W4 >= 256 ? 256 : (W4 >= 128 ? 128 : 64));
    const int per = (W4 + threads - 1) / threads;
    if (per <= 1) return launch_stream_mix<T, SC, 4, 1>(a, threads, stream);
    if (per <= 2) return launch_stream_mix<T, SC, 4, 2>(a, threads, stream);
    if (per <= 4) return launch_stream_mix<T, SC, 4, 4>(a, threads, stream);
    return launch_stream_mix<T, SC, 4, 0>(a, threads, stream);
  }
  return ODI_ERR_UNSUPPORTED;
}

extern "C" int odi_stream_mix(const StreamMixArgs* args, int dtype, cudaStream_t stream) {
  const StreamMixArgs a = *args;
  if (a.n <= 0) return 0;
  if (a.S < 1 || a.W < 1 || (a.y == nullptr && a.out == nullptr) || (a.y != nullptr && a.rows != nullptr)) return ODI_ERR_ARGUMENT;
  if (a.out != nullptr && (a.weight == nullptr || a.bias == nullptr)) return ODI_ERR_ARGUMENT;
  if (a.S > SM_MAX_STREAMS || (size_t)a.W * 4 > 200 * 1024) return ODI_ERR_UNSUPPORTED;
#define ODI_SM(T) (a.S == 1 ? launch_streams<T, 1>(a, stream) : a.S == 2 ? launch_streams<T, 2>(a, stream) : \
                   a.S == 3 ? launch_streams<T, 3>(a, stream) : a.S == 4 ? launch_streams<T, 4>(a, stream) : launch_streams<T, 0>(a, stream))
  odi_rc = dtype == 0 ? ODI_SM(float) : ODI_SM(bf16);
#undef ODI_SM
  return launch_status();
}
