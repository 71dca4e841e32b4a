// Causal grouped-query attention over paged cache slots on the CUDA cores, for any
// mixture of sequences: whole prompts, single decoded tokens, or chunks of a few tokens.
// It is the attention of the float32 path and the fallback of the bf16 path (windows,
// head sizes the tensor-core kernels do not take).
//
// Compile with -DODI_HEAD_DIM=<d>, d a multiple of 16 up to 512.
//
// Work item (one block of 4 warps): one sequence, one key/value head, a tile of query
// rows -- `bq` consecutive tokens times up to 16 of the head's query heads -- and, when
// the key range is split, one split.  Keys are streamed 32 at a time through shared
// memory (converted to fp32); each warp owns 4 rows; lane j scores key j of the tile;
// the softmax is the running-maximum form in fp32; the output accumulates in fp32.
// Key j is visible to the query at position p iff j <= p and (window == 0 or j > p - window or j < keep):
// with keep > 0 a windowed layer goes on seeing the first `keep` positions of its sequence.
// With chunk c > 0 (instead of a window) the query at position p sees the keys of its own chunk of c positions only:
// j <= p and j / c == p / c.
// With mixed = 1 a query head has nkv * D lanes, one query of D lanes for every key head, and its score is the sum of
// their dot products with all key heads of the position (heads that mix their scores; the values stay grouped).
// With softcap c > 0 a score s (already times scale) becomes c tanh(s / c) before the softmax.
// With a distance bias its entry for the key's distance is added to the score behind scale and cap.  The output may go to
// rows of its own width, times a constant and a gate (HeadOut).
// With sink = 1 the softmax has one more term, of score 0 and without a value: p_j = e^(s_j) / (1 + sum e^(s_k)).
//
// With splits > 1 every split writes an un-normalised partial (acc[d], max, sum) and
// attention_combine merges them in split order.
//
// Two more build-time options, for attention over a compressed (latent) cache:
//  -DODI_VALUE_DIM=<dv>  the value rows (and the output) are dv wide instead of d (dv <= d when shared);
//  -DODI_SHARED_KV=1     a cached row is key and value at once: the value is its first dv lanes, and
//                        there is no value pool.  With these d may be any multiple of 4 up to 1024.
#include "common.cuh"

#ifndef ODI_HEAD_DIM
#error "compile with -DODI_HEAD_DIM=<head size>"
#endif

#define D ODI_HEAD_DIM
#ifndef ODI_VALUE_DIM
#define ODI_VALUE_DIM ODI_HEAD_DIM
#endif
#ifndef ODI_SHARED_KV
#define ODI_SHARED_KV 0
#endif
#define DV ODI_VALUE_DIM
static_assert(D % 4 == 0, "the key width must be a multiple of 4");
static_assert(!ODI_SHARED_KV || DV <= D, "a shared row cannot hold a value wider than itself");
#define KT 32                 // keys per tile
#define NWARPS 4
#define RW 4                  // rows per warp
#define ROWS (NWARPS * RW)    // rows per block
#define NACC ((DV + 31) / 32)  // output registers per row per lane
#define KSTR (D + 4)          // padded row stride of the key tile (floats)

struct AttnArgs {
  const void* q;        // [n_tokens, nq, D]
  const void* k_pool;   // [pages, nkv, page_size, D]
  const void* v_pool;
  void* out;            // [n_tokens, nq * DV]
  float* partial;       // [n_tokens, nq, splits, DV + 2] when splits > 1
  const int* cu_q;      // [n_seqs + 1] first packed token of each sequence
  const int* past;      // [n_seqs] keys cached before this step
  const int* page_start;
  const int* page_ids;
  int n_seqs, nq, nkv, page_size, ring_pages, window, splits, bq, head_chunks;
  float scale, softcap;
  int sink;             // 1: the softmax has one more term of score 0 and no value (one is added to its denominator)
  int keep;             // > 0 with a window: keys 0..keep-1 stay visible beyond the window
  int chunk;            // > 0: keys of the query's own chunk of this many positions
  int mixed;            // 1: q is [n_tokens, nq, nkv, D]; a score sums over the key heads
  HeadOut ho;
  DistanceBias rel;
};

// 1 / (l + e^-m) for sums l taken relative to the maximum m: the denominator with the sink's term, without overflow.
__device__ __forceinline__ float sink_inverse(float m, float l) {
  if (m == -INFINITY) return 0.f;
  if (m >= 0.f) return 1.f / (l + expf(-m));
  const float e = expf(m);
  return e / fmaf(l, e, 1.f);
}

template <typename T>
__global__ void __launch_bounds__(NWARPS * 32)
attention_simt_kernel(AttnArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) float smem[];
  float* Ks = smem;                    // [KT][KSTR]
  float* Vs = Ks + KT * KSTR;          // [KT][DV]; with shared rows the values are read from Ks
  float* Qs = Vs + (ODI_SHARED_KV ? 0 : KT * DV);   // [ROWS][D]
  float* Ps = Qs + ROWS * D;           // [ROWS][KT]

  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int seq = blockIdx.z;
  const int hk = blockIdx.y / a.head_chunks, chunk = blockIdx.y % a.head_chunks;
  const int qtile = blockIdx.x / a.splits, split = blockIdx.x % a.splits;
  const int g = a.nq / a.nkv;
  const int hpb = min(g - chunk * 16, 16);  // query heads of this block
  const int q_begin = a.cu_q[seq], q_len = a.cu_q[seq + 1] - q_begin;
  const int t0 = qtile * a.bq;
  if (t0 >= q_len) return;
  const int nt = min(a.bq, q_len - t0);     // tokens of this tile
  const int nrows = nt * hpb;
  const int past = a.past[seq];
  const int pos_lo = past + t0, pos_hi = past + t0 + nt - 1;

  // Key range seen by any row of the tile, cut into tiles of KT, then into splits.
  int k_lo = a.window > 0 ? max(0, pos_lo - a.window + 1) : (a.chunk > 0 ? pos_lo - pos_lo % a.chunk : 0);
  k_lo = (k_lo / KT) * KT;
  // the tiles of kept first keys that lie in front of the window's first tile come first in the walk
  const int keep_tiles = a.window > 0 && a.keep > 0 ? min((a.keep + KT - 1) / KT, k_lo / KT) : 0;
  const int n_tiles = keep_tiles + (pos_hi + 1 - k_lo + KT - 1) / KT;
  const int per_split = (n_tiles + a.splits - 1) / a.splits;
  const int tile_begin = split * per_split, tile_end = min(n_tiles, tile_begin + per_split);

  // Stage the query rows (fp32).  Row r: token t0 + r / hpb, head chunk*16 + r % hpb; with mixed heads the part of them
  // that goes with key head kh.
  auto stage_queries = [&](int kh) {
    for (int i = tid; i < ROWS * D; i += NWARPS * 32) {
      const int r = i / D, dd = i % D;
      float v = 0.f;
      if (r < nrows) {
        const int tok = q_begin + t0 + r / hpb;
        const int h = hk * g + chunk * 16 + r % hpb;
        const size_t at = (size_t)tok * a.nq + h;
        v = to_f<T>(((const T*)a.q)[(a.mixed ? at * a.nkv + kh : at) * D + dd]);
      }
      Qs[i] = v;
    }
  };
  if (!a.mixed) stage_queries(0);

  float m[RW], l[RW], acc[RW][NACC];
  int rpos[RW], rold[RW];       // position of the row's query, and the oldest key of its window or chunk
  const float* rrel[RW];        // the row's head in the table of distance biases
#pragma unroll
  for (int r = 0; r < RW; ++r) {
    m[r] = -INFINITY; l[r] = 0.f;
    const int row = warp * RW + r;
    rpos[r] = row < nrows ? past + t0 + row / hpb : -1;
    rold[r] = a.window > 0 ? rpos[r] - a.window + 1 : (a.chunk > 0 && rpos[r] >= 0 ? rpos[r] - rpos[r] % a.chunk : 0);
    rrel[r] = a.rel.table != nullptr && row < nrows ? a.rel.table + (size_t)(hk * g + chunk * 16 + row % hpb) * a.rel.n : nullptr;
#pragma unroll
    for (int i = 0; i < NACC; ++i) acc[r][i] = 0.f;
  }

  const int* pages = a.page_ids + a.page_start[seq];
  for (int tile = tile_begin; tile < tile_end; ++tile) {
    const int kbase = tile < keep_tiles ? tile * KT : k_lo + (tile - keep_tiles) * KT;
    // All KT keys of a tile lie in one page (page_size is a multiple of KT).
    const int page = pages[page_slot_of(kbase, a.page_size, a.ring_pages)];
    const int nkeys = min(KT, pos_hi + 1 - kbase);
    float s[RW];
#pragma unroll
    for (int r = 0; r < RW; ++r) s[r] = 0.f;
    const int kh_first = a.mixed ? 0 : hk, kh_last = a.mixed ? a.nkv - 1 : hk;
    for (int kh = kh_first; kh <= kh_last; ++kh) {
      __syncthreads();  // previous tile fully consumed (also orders the Qs writes)
      if (a.mixed) stage_queries(kh);
      const size_t base = (((size_t)page * a.nkv + kh) * a.page_size + (kbase % a.page_size)) * D;
      const T* kp = (const T*)a.k_pool + base;
      if (D % 8 == 0 && ((uintptr_t)kp % 16) == 0) {
        // eight lanes of a row at a time (16-byte loads of bf16, two of floats)
        for (int i = tid * 8; i < KT * D; i += NWARPS * 32 * 8) {
          const int j = i / D, dd = i % D;
          float v[8];
          if (j < nkeys) {
            if (sizeof(T) == 2) {
              const uint4 raw = *(const uint4*)(kp + i);
              const __nv_bfloat162* h2 = (const __nv_bfloat162*)&raw;
#pragma unroll
              for (int e = 0; e < 4; ++e) { const float2 f = __bfloat1622float2(h2[e]); v[2 * e] = f.x; v[2 * e + 1] = f.y; }
            } else {
              const float4 lo = *(const float4*)(kp + i), hi = *(const float4*)(kp + i + 4);
              v[0] = lo.x; v[1] = lo.y; v[2] = lo.z; v[3] = lo.w; v[4] = hi.x; v[5] = hi.y; v[6] = hi.z; v[7] = hi.w;
            }
          } else {
#pragma unroll
            for (int e = 0; e < 8; ++e) v[e] = 0.f;
          }
          *(float4*)&Ks[j * KSTR + dd] = make_float4(v[0], v[1], v[2], v[3]);
          *(float4*)&Ks[j * KSTR + dd + 4] = make_float4(v[4], v[5], v[6], v[7]);
        }
      } else {
        for (int i = tid; i < KT * D; i += NWARPS * 32) {
          const int j = i / D, dd = i % D;
          Ks[j * KSTR + dd] = j < nkeys ? to_f<T>(kp[i]) : 0.f;
        }
      }
#if !ODI_SHARED_KV
      const T* vp = (const T*)a.v_pool +
                    (((size_t)page * a.nkv + hk) * a.page_size + (kbase % a.page_size)) * DV;
      if (kh == kh_first)
        for (int i = tid; i < KT * DV; i += NWARPS * 32) Vs[i] = i / DV < nkeys ? to_f<T>(vp[i]) : 0.f;
#endif
      __syncthreads();

      // scores: lane = key
      const float* krow = Ks + lane * KSTR;
      const float* qrow = Qs + (warp * RW) * D;
#pragma unroll 4
      for (int dd = 0; dd < D; dd += 4) {
        const float4 kv = *(const float4*)(krow + dd);
#pragma unroll
        for (int r = 0; r < RW; ++r) {
          const float4 qv = *(const float4*)(qrow + r * D + dd);
          s[r] = fmaf(qv.x, kv.x, s[r]); s[r] = fmaf(qv.y, kv.y, s[r]);
          s[r] = fmaf(qv.z, kv.z, s[r]); s[r] = fmaf(qv.w, kv.w, s[r]);
        }
      }
    }
    const int kj = kbase + lane;
    float* prow = Ps + (warp * RW) * KT;
#pragma unroll
    for (int r = 0; r < RW; ++r) {
      const bool vis = rpos[r] >= 0 && kj <= rpos[r] && (kj >= rold[r] || kj < a.keep);
      float sc = s[r] * a.scale;
      if (a.softcap > 0.f) sc = a.softcap * tanhf(sc / a.softcap);
      if (vis && rrel[r] != nullptr) sc += rrel[r][min(rpos[r] - kj, a.rel.n - 1)];
      if (!vis) sc = -INFINITY;
      const float mx = warp_max(sc);
      const float m_new = fmaxf(m[r], mx);
      float p = 0.f, alpha = 1.f;
      if (m_new != -INFINITY) {
        p = vis ? expf(sc - m_new) : 0.f;
        alpha = expf(m[r] - m_new);  // m = -inf gives 0
      }
      l[r] = l[r] * alpha + warp_sum(p);
      m[r] = m_new;
#pragma unroll
      for (int i = 0; i < NACC; ++i) acc[r][i] *= alpha;
      prow[r * KT + lane] = p;
    }
    __syncwarp();
    // output: lane = element of the head
#pragma unroll 4
    for (int j = 0; j < KT; ++j) {
      float vv[NACC];
#pragma unroll
      for (int i = 0; i < NACC; ++i) {
        const int dd = lane + 32 * i;
#if ODI_SHARED_KV
        vv[i] = dd < DV ? Ks[j * KSTR + dd] : 0.f;
#else
        vv[i] = dd < DV ? Vs[j * DV + dd] : 0.f;
#endif
      }
#pragma unroll
      for (int r = 0; r < RW; ++r) {
        const float p = prow[r * KT + j];
#pragma unroll
        for (int i = 0; i < NACC; ++i) acc[r][i] = fmaf(p, vv[i], acc[r][i]);
      }
    }
    __syncwarp();
  }

#pragma unroll
  for (int r = 0; r < RW; ++r) {
    const int row = warp * RW + r;
    if (row >= nrows) continue;
    const int tok = q_begin + t0 + row / hpb;
    const int h = hk * g + chunk * 16 + row % hpb;
    if (a.splits == 1) {
      float inv = l[r] > 0.f ? 1.f / l[r] : 0.f;
      if (a.sink) inv = sink_inverse(m[r], l[r]);
      T* o = (T*)a.out + (size_t)tok * a.ho.out_ld + h * DV;
#pragma unroll
      for (int i = 0; i < NACC; ++i) {
        const int dd = lane + 32 * i;
        if (dd < DV) o[dd] = from_f<T>(acc[r][i] * inv * head_out_factor<T>(a.ho, tok, h, DV, dd));
      }
    } else {
      float* o = a.partial + (((size_t)tok * a.nq + h) * a.splits + split) * (DV + 2);
#pragma unroll
      for (int i = 0; i < NACC; ++i) {
        const int dd = lane + 32 * i;
        if (dd < DV) o[dd] = acc[r][i];
      }
      if (lane == 0) { o[DV] = m[r]; o[DV + 1] = l[r]; }
    }
  }
}

// Merge the partials of one (token, head): out = sum_s e^(m_s - M) acc_s / sum_s e^(m_s - M) l_s.
template <typename T>
__global__ void attention_combine_kernel(const float* __restrict__ partial, T* __restrict__ out, int splits, int sink, int nq, HeadOut ho) {
  pdl_launch_dependents();
  pdl_wait();
  const size_t row = blockIdx.x;  // token * nq + head
  const float* p = partial + row * splits * (DV + 2);
  float M = -INFINITY;
  for (int s = 0; s < splits; ++s) M = fmaxf(M, p[s * (DV + 2) + DV]);
  float denom = 0.f;
  for (int s = 0; s < splits; ++s) {
    const float ms = p[s * (DV + 2) + DV];
    if (ms != -INFINITY) denom += expf(ms - M) * p[s * (DV + 2) + DV + 1];
  }
  float inv = denom > 0.f ? 1.f / denom : 0.f;
  if (sink) inv = sink_inverse(M, denom);
  for (int dd = threadIdx.x; dd < DV; dd += blockDim.x) {
    float v = 0.f;
    for (int s = 0; s < splits; ++s) {
      const float ms = p[s * (DV + 2) + DV];
      if (ms != -INFINITY) v += expf(ms - M) * p[s * (DV + 2) + dd];
    }
    const size_t tok = row / nq;
    const int h = (int)(row % nq);
    out[tok * ho.out_ld + h * DV + dd] = from_f<T>(v * inv * head_out_factor<T>(ho, tok, h, DV, dd));
  }
}

extern "C" int odi_attention_simt_head_dim() { return D; }

// max_q_len: the longest q_len of the batch (sizes the grid); n_tokens: packed tokens.
extern "C" int odi_attention_simt(const AttnArgs* args, int max_q_len, int n_tokens, int dtype,
                                  cudaStream_t stream) {
  AttnArgs a = *args;
  if (a.n_seqs <= 0 || n_tokens <= 0) return 0;
  if (a.nq % a.nkv != 0 || a.page_size % KT != 0 || a.splits < 1 || a.n_seqs > 65535 || a.keep < 0 || a.chunk < 0 ||
      (a.chunk > 0 && (a.window > 0 || a.keep > 0)) || (a.mixed && ODI_SHARED_KV))
    return ODI_ERR_UNSUPPORTED;
  const int g = a.nq / a.nkv;
  const int hpb = g < 16 ? g : 16;
  a.head_chunks = (g + 15) / 16;
  a.bq = ROWS / hpb > 0 ? ROWS / hpb : 1;
  if (a.splits > 1 && a.partial == nullptr) return ODI_ERR_ARGUMENT;
  const int q_tiles = (max_q_len + a.bq - 1) / a.bq;
  dim3 grid(q_tiles * a.splits, a.nkv * a.head_chunks, a.n_seqs);
  if (grid.y > 65535) return ODI_ERR_UNSUPPORTED;
  const size_t smem = sizeof(float) * (KT * KSTR + (ODI_SHARED_KV ? 0 : KT * DV) + ROWS * D + ROWS * KT);
  // The shared-memory opt-in is a property of the function, set once per process.
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(attention_simt_kernel<float>,
                                         cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e == cudaSuccess)
      e = cudaFuncSetAttribute(attention_simt_kernel<bf16>,
                               cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  if (dtype == 0) odi_rc = launch_pdl((attention_simt_kernel<float>), dim3(grid), dim3(NWARPS * 32), smem, stream, a);
  else odi_rc = launch_pdl((attention_simt_kernel<bf16>), dim3(grid), dim3(NWARPS * 32), smem, stream, a);
  int rc = launch_status();
  if (rc != 0 || a.splits == 1) return rc;
  const int rows = n_tokens * a.nq;
  const int threads = DV >= 128 ? 128 : (DV >= 64 ? 64 : 32);
  if (dtype == 0) odi_rc = launch_pdl((attention_combine_kernel<float>), dim3(rows), dim3(threads), 0, stream, a.partial, (float*)a.out, a.splits, a.sink, a.nq, a.ho);
  else odi_rc = launch_pdl((attention_combine_kernel<bf16>), dim3(rows), dim3(threads), 0, stream, a.partial, (bf16*)a.out, a.splits, a.sink, a.nq, a.ho);
  return launch_status();
}
