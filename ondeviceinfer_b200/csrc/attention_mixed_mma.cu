// bf16 causal grouped-query attention inside chunks, with heads that mix their scores, over the paged cache (a ring of
// pages per sequence), on the tensor cores: mma.sync m16n8k16 with fp32 accumulation, fp32 scores and running-maximum
// softmax.
//
//   mixed = 1: q is [n_tokens, nq, nkv, D]; score_h = scale * sum_j q_hj . k_j over all key heads j of the position (the
//              mixing matrix has been folded into the queries: mixed.cu); mixed = 0: q is [n_tokens, nq, D] and
//              score_h = scale * q_h . k_(h / (nq / nkv)).  The values stay grouped either way.
//   key j is visible to the query at position p iff j <= p and (chunk == 0 or j / chunk == p / chunk).
//
// Both kernels walk tiles of 64 positions (one page); a tile's key heads and then its value heads arrive one after the
// other as items of one ring in shared memory (cp.async, rows padded by 16 bytes so that ldmatrix reads are free of bank
// conflicts), so a score tile is accumulated item by item in registers and any number of key heads fits.  One block
// barrier per item: item i + NS - 1 is requested when everybody has left item i - 1, whose place it takes.
//
//  prompts and portions: a block of 8 warps owns 64 consecutive query tokens of one head; a warp takes 16 rows and one half
//    of every tile's keys, with a maximum, sum and accumulator of its own (merged at the end); the rows of all key heads
//    stay in shared memory.
//  single tokens: a block owns up to 16 query heads of one sequence (the rows of its MMAs) and one range of the visible
//    keys; its 4 warps take 16 keys each of every tile, and merge in shared memory.  Rows of different value heads share
//    the accumulator: a value head's product takes the probabilities of its own rows and zero for the others.  With
//    several ranges a combine kernel adds them in order.
//
// Compile with -DODI_HEAD_DIM=<D> -DODI_VALUE_DIM=<DV>, multiples of 16 up to 256.
#include "common.cuh"

#ifndef ODI_HEAD_DIM
#error "compile with -DODI_HEAD_DIM=<key width> -DODI_VALUE_DIM=<value width>"
#endif
#ifndef ODI_VALUE_DIM
#define ODI_VALUE_DIM ODI_HEAD_DIM
#endif
#define D ODI_HEAD_DIM
#define DV ODI_VALUE_DIM
#if (D % 16) != 0 || D > 256 || (DV % 16) != 0 || DV > 256
#error "key and value widths must be multiples of 16, at most 256"
#endif

#define KT 64                       // keys per tile = positions per page
#define ROWB_K (2 * D + 16)         // bytes per shared-memory row of a key tile
#define ROWB_V (2 * DV + 16)
#define STAGE_BYTES (KT * (ROWB_K > ROWB_V ? ROWB_K : ROWB_V))
#define KSTEPS (D / 16)
#define DVTILES (DV / 8)
#define LOG2E 1.4426950408889634f
#define WARPS 4                     // of a single-token block
#define PROMPT_WARPS 8
#define RS (DV + 2)                 // floats of a partial result: weighted values, maximum, sum
#define SMEM_LIMIT 232448

struct MixedAttnArgs {
  const bf16* q;          // [n_tokens, nq, nkv, D] when mixed, else [n_tokens, nq, D]
  const bf16* k_pool;     // [pages, nkv, 64, D]
  const bf16* v_pool;     // [pages, nkv, 64, DV]
  bf16* out;              // [n_tokens, nq * DV]
  float* partial;         // [n_tokens, nq, splits, DV + 2] when splits > 1
  const int* cu_q;
  const int* past;
  const int* page_start;
  const int* page_ids;
  int n_seqs, nq, nkv, ring_pages, chunk, mixed, splits;
  float scale;
};

__device__ __forceinline__ uint32_t smem_addr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_async_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}
__device__ __forceinline__ void ldmatrix_x4(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void mma_bf16(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
  __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *(uint32_t*)&v;
}

// One page tile (64 rows of W bf16, contiguous in global memory) into shared-memory rows of 2 W + 16 bytes.
template <int W, int THREADS>
__device__ __forceinline__ void load_tile(uint32_t dst, const bf16* src, int tid) {
  constexpr int CHUNKS = W / 8;    // 16-byte pieces per row
#pragma unroll 4
  for (int i = tid; i < KT * CHUNKS; i += THREADS) {
    const int r = i / CHUNKS, c = i % CHUNKS;
    cp_async16(dst + r * (2 * W + 16) + c * 16, src + (size_t)i * 8);
  }
}

// The block's query rows into shared memory: row r < rows from src + r * stride, `width` elements each, zeros behind.
template <int THREADS>
__device__ __forceinline__ void load_queries(uint8_t* dst, int rowb, const bf16* src, size_t stride, int rows, int total, int width,
                                             int tid) {
  const int pieces = width / 8;
  for (int i = tid; i < total * pieces; i += THREADS) {
    const int r = i / pieces, c = i % pieces;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (r < rows) v = *(const uint4*)(src + (size_t)r * stride + c * 8);
    *(uint4*)(dst + (size_t)r * rowb + c * 16) = v;
  }
}

template <int NS>
__global__ void __launch_bounds__(PROMPT_WARPS * 32)
attention_mixed_kernel(MixedAttnArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) uint8_t smem[];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  // heads along x, sequences along y, query tiles along z from the last to the first
  const int seq = blockIdx.y, head = blockIdx.x, hk = head / (a.nq / a.nkv);
  const int q_begin = a.cu_q[seq], q_len = a.cu_q[seq + 1] - q_begin;
  const int t0 = (gridDim.z - 1 - blockIdx.z) * 64;
  if (t0 >= q_len) return;
  const int past = a.past[seq];
  const int nt = min(64, q_len - t0), p0 = past + t0;
  const int KH = a.mixed ? a.nkv : 1, width = KH * D, q_rowb = width * 2 + 16, per_tile = KH + 1;
  const int tile_lo = (a.chunk > 0 ? p0 - p0 % a.chunk : 0) / KT, tile_hi = (p0 + nt - 1) / KT;       // inclusive
  const int n_items = (tile_hi - tile_lo + 1) * per_tile;
  const int* pages = a.page_ids + a.page_start[seq];
  uint8_t* ring = smem + 64 * q_rowb;
  const uint32_t ring_addr = smem_addr(ring), q_addr = smem_addr(smem);

  // what item i is: tile tile_lo + i / per_tile, key head i % per_tile, or the values
  int next = 0, next_tile = tile_lo, next_part = 0, next_page = 0;
  auto issue = [&]() {
    if (next < n_items) {
      if (next_part == 0) next_page = pages[page_slot_of_page(next_tile, a.ring_pages)];
      const uint32_t dst = ring_addr + (uint32_t)(next % NS) * STAGE_BYTES;
      if (next_part < KH) {
        const int kh = a.mixed ? next_part : hk;
        load_tile<D, PROMPT_WARPS * 32>(dst, a.k_pool + ((size_t)next_page * a.nkv + kh) * KT * D, tid);
        ++next_part;
      } else {
        load_tile<DV, PROMPT_WARPS * 32>(dst, a.v_pool + ((size_t)next_page * a.nkv + hk) * KT * DV, tid);
        next_part = 0;
        ++next_tile;
      }
      ++next;
    }
    cp_async_commit();                     // one group per item, empty or not
  };
#pragma unroll
  for (int i = 0; i < NS - 1; ++i) issue();
  load_queries<PROMPT_WARPS * 32>(smem, q_rowb, a.q + ((size_t)(q_begin + t0) * a.nq + head) * width, (size_t)a.nq * width, nt, 64, width, tid);

  const int rows0 = (warp & 3) * 16, half = warp >> 2;         // this warp's rows, and its half of a tile's keys
  const int r_lo = rows0 + (lane >> 2), r_hi = r_lo + 8;
  const int pos_lo = p0 + r_lo, pos_hi = p0 + r_hi;
  const int old_lo = a.chunk > 0 ? pos_lo - pos_lo % a.chunk : 0, old_hi = a.chunk > 0 ? pos_hi - pos_hi % a.chunk : 0;
  const int warp_first = p0 + rows0, warp_last = warp_first + 15;
  const int warp_old = a.chunk > 0 ? warp_first - warp_first % a.chunk : 0;
  const bool has_rows = rows0 < nt;
  const float sl2 = a.scale * LOG2E;
  const int mi = lane >> 3, mr = lane & 7;
  // A fragments: (rows 0..7, k 0..7), (rows 8..15, same k), (rows 0..7, k 8..15), (rows 8..15, k 8..15)
  const uint32_t a_base = q_addr + (rows0 + (mi & 1) * 8 + mr) * q_rowb + (mi >> 1) * 16;

  float o[DVTILES][4], s[4][4];
#pragma unroll
  for (int i = 0; i < DVTILES; ++i) { o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f; }
  float m_lo = -INFINITY, m_hi = -INFINITY, l_lo = 0.f, l_hi = 0.f;

  int part = 0, kbase = tile_lo * KT + half * 32;            // the first of this warp's 32 keys
  for (int it = 0; it < n_items; ++it) {
    cp_async_wait<NS - 2>();
    __syncthreads();                       // item `it` is there, item it - 1 has been left
    issue();
    const uint32_t st = ring_addr + (uint32_t)(it % NS) * STAGE_BYTES;
    const bool active = has_rows && kbase <= warp_last && kbase + 32 > warp_old;
    if (part < KH) {
      if (active) {
        if (part == 0) {
#pragma unroll
          for (int i = 0; i < 4; ++i) { s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f; }
        }
        const uint32_t qa = a_base + part * D * 2;
#pragma unroll
        for (int ks = 0; ks < KSTEPS; ++ks) {
          uint32_t qf[4];
          ldmatrix_x4(qa + ks * 32, qf[0], qf[1], qf[2], qf[3]);
#pragma unroll
          for (int np = 0; np < 2; ++np) {
            // matrices: (the half's keys np*16 + 0..7, d ks*16 + 0..7), (same keys, d + 8), (keys + 8, d), (keys + 8, d + 8)
            const int key = half * 32 + np * 16 + (mi >> 1) * 8 + mr, dd = ks * 16 + (mi & 1) * 8;
            uint32_t b0, b1, b2, b3;
            ldmatrix_x4(st + key * ROWB_K + dd * 2, b0, b1, b2, b3);
            mma_bf16(s[np * 2], qf, b0, b1);
            mma_bf16(s[np * 2 + 1], qf, b2, b3);
          }
        }
      }
      ++part;
      continue;
    }
    if (active) {
      float mx_lo = -INFINITY, mx_hi = -INFINITY;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int kj = kbase + i * 8 + (lane & 3) * 2;
        s[i][0] = (kj <= pos_lo && kj >= old_lo) ? s[i][0] * sl2 : -INFINITY;
        s[i][1] = (kj + 1 <= pos_lo && kj + 1 >= old_lo) ? s[i][1] * sl2 : -INFINITY;
        s[i][2] = (kj <= pos_hi && kj >= old_hi) ? s[i][2] * sl2 : -INFINITY;
        s[i][3] = (kj + 1 <= pos_hi && kj + 1 >= old_hi) ? s[i][3] * sl2 : -INFINITY;
        mx_lo = fmaxf(mx_lo, fmaxf(s[i][0], s[i][1]));
        mx_hi = fmaxf(mx_hi, fmaxf(s[i][2], s[i][3]));
      }
      mx_lo = fmaxf(mx_lo, __shfl_xor_sync(0xffffffffu, mx_lo, 1));
      mx_lo = fmaxf(mx_lo, __shfl_xor_sync(0xffffffffu, mx_lo, 2));
      mx_hi = fmaxf(mx_hi, __shfl_xor_sync(0xffffffffu, mx_hi, 1));
      mx_hi = fmaxf(mx_hi, __shfl_xor_sync(0xffffffffu, mx_hi, 2));
      const float mn_lo = fmaxf(m_lo, mx_lo), mn_hi = fmaxf(m_hi, mx_hi);
      // rows with nothing visible yet keep a zero accumulator; avoid (-inf) - (-inf)
      const float ref_lo = mn_lo == -INFINITY ? 0.f : mn_lo, ref_hi = mn_hi == -INFINITY ? 0.f : mn_hi;
      const float al_lo = exp2f(m_lo - ref_lo), al_hi = exp2f(m_hi - ref_hi);
      m_lo = mn_lo; m_hi = mn_hi;
      float sum_lo = 0.f, sum_hi = 0.f;
      uint32_t pf[2][4];                  // P as A fragments for the 2 key steps of 16
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float e0 = exp2f(s[i][0] - ref_lo), e1 = exp2f(s[i][1] - ref_lo);
        const float e2 = exp2f(s[i][2] - ref_hi), e3 = exp2f(s[i][3] - ref_hi);
        sum_lo += e0 + e1; sum_hi += e2 + e3;
        pf[i >> 1][(i & 1) * 2] = pack_bf16(e0, e1);
        pf[i >> 1][(i & 1) * 2 + 1] = pack_bf16(e2, e3);
      }
      l_lo = l_lo * al_lo + sum_lo; l_hi = l_hi * al_hi + sum_hi;
#pragma unroll
      for (int i = 0; i < DVTILES; ++i) { o[i][0] *= al_lo; o[i][1] *= al_lo; o[i][2] *= al_hi; o[i][3] *= al_hi; }
#pragma unroll
      for (int kk = 0; kk < 2; ++kk) {      // 16 keys per step
#pragma unroll
        for (int dp = 0; dp < DVTILES / 2; ++dp) {
          // matrices: (keys kk*16 + 0..7, d dp*16 + 0..7), (keys + 8, same d), (keys, d + 8), (keys + 8, d + 8)
          const int key = half * 32 + kk * 16 + (mi & 1) * 8 + mr, dd = dp * 16 + (mi >> 1) * 8;
          uint32_t b0, b1, b2, b3;
          ldmatrix_x4_trans(st + key * ROWB_V + dd * 2, b0, b1, b2, b3);
          mma_bf16(o[dp * 2], pf[kk], b0, b1);
          mma_bf16(o[dp * 2 + 1], pf[kk], b2, b3);
        }
      }
    }
    part = 0;
    kbase += KT;
  }
  // the row sums live spread over the 4 lanes of a quad
  l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 1); l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 2);
  l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 1); l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 2);
  // the second half's results through the free ring: [row][DV + 2] floats, maxima in the log2 domain
  cp_async_wait<0>();
  __syncthreads();
  const int c = (lane & 3) * 2;
  float* mg_lo = (float*)ring + (size_t)r_lo * RS;
  float* mg_hi = (float*)ring + (size_t)r_hi * RS;
  if (half == 1) {
#pragma unroll
    for (int i = 0; i < DVTILES; ++i) {
      *(float2*)(mg_lo + i * 8 + c) = make_float2(o[i][0], o[i][1]);
      *(float2*)(mg_hi + i * 8 + c) = make_float2(o[i][2], o[i][3]);
    }
    if ((lane & 3) == 0) { mg_lo[DV] = m_lo; mg_lo[DV + 1] = l_lo; mg_hi[DV] = m_hi; mg_hi[DV + 1] = l_hi; }
  }
  __syncthreads();
  if (half == 1) return;
  auto weights = [](float m0, float l0, float m1, float l1, float& w0, float& w1) {
    const float M = fmaxf(m0, m1), ref = M == -INFINITY ? 0.f : M;
    w0 = exp2f(m0 - ref); w1 = exp2f(m1 - ref);
    const float l = w0 * l0 + w1 * l1, inv = l > 0.f ? 1.f / l : 0.f;
    w0 *= inv; w1 *= inv;
  };
  float a_lo, b_lo, a_hi, b_hi;
  weights(m_lo, l_lo, mg_lo[DV], mg_lo[DV + 1], a_lo, b_lo);
  weights(m_hi, l_hi, mg_hi[DV], mg_hi[DV + 1], a_hi, b_hi);
  if (r_lo < nt) {
    bf16* dst = a.out + ((size_t)(q_begin + t0 + r_lo) * a.nq + head) * DV;
#pragma unroll
    for (int i = 0; i < DVTILES; ++i) {
      const float2 v = *(const float2*)(mg_lo + i * 8 + c);
      *(uint32_t*)(dst + i * 8 + c) = pack_bf16(o[i][0] * a_lo + v.x * b_lo, o[i][1] * a_lo + v.y * b_lo);
    }
  }
  if (r_hi < nt) {
    bf16* dst = a.out + ((size_t)(q_begin + t0 + r_hi) * a.nq + head) * DV;
#pragma unroll
    for (int i = 0; i < DVTILES; ++i) {
      const float2 v = *(const float2*)(mg_hi + i * 8 + c);
      *(uint32_t*)(dst + i * 8 + c) = pack_bf16(o[i][2] * a_hi + v.x * b_hi, o[i][3] * a_hi + v.y * b_hi);
    }
  }
}

// ------------------------------------------------------------------------------ single tokens

template <int NS>
__global__ void __launch_bounds__(WARPS * 32)
attention_mixed_decode_kernel(MixedAttnArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ __align__(16) uint8_t smem[];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int split = blockIdx.x, head0 = blockIdx.y * 16, seq = blockIdx.z;
  const int rep = a.nq / a.nkv, heads_here = min(16, a.nq - head0);
  const int tok = a.cu_q[seq], pos = a.past[seq];
  const int first_key = a.chunk > 0 ? pos - pos % a.chunk : 0;
  const int tile_first = first_key / KT, n_tiles = pos / KT + 1 - tile_first;
  const int per_split = (n_tiles + a.splits - 1) / a.splits;
  const int tile_lo = tile_first + split * per_split, tile_end = min(tile_first + n_tiles, tile_lo + per_split);
  if (tile_lo >= tile_end) {
    // nothing to see: say so to the combine kernel (only reached with several splits)
    for (int row = tid; row < heads_here; row += WARPS * 32) {
      float* dst = a.partial + (((size_t)tok * a.nq + head0 + row) * a.splits + split) * RS;
      dst[DV] = -INFINITY; dst[DV + 1] = 0.f;
    }
    return;
  }
  // value heads of these rows; their key heads too when nothing is mixed
  const int v_lo = head0 / rep, n_v = (head0 + heads_here - 1) / rep - v_lo + 1;
  const int k_lo = a.mixed ? 0 : v_lo, KH = a.mixed ? a.nkv : n_v;
  const int width = a.mixed ? a.nkv * D : D, q_rowb = width * 2 + 16, per_tile = KH + n_v;
  const int n_items = (tile_end - tile_lo) * per_tile;
  const int* pages = a.page_ids + a.page_start[seq];
  uint8_t* ring = smem + 16 * q_rowb;
  const uint32_t ring_addr = smem_addr(ring);

  int next = 0, next_tile = tile_lo, next_part = 0, next_page = 0;
  auto issue = [&]() {
    if (next < n_items) {
      if (next_part == 0) next_page = pages[page_slot_of_page(next_tile, a.ring_pages)];
      const uint32_t dst = ring_addr + (uint32_t)(next % NS) * STAGE_BYTES;
      if (next_part < KH)
        load_tile<D, WARPS * 32>(dst, a.k_pool + ((size_t)next_page * a.nkv + k_lo + next_part) * KT * D, tid);
      else
        load_tile<DV, WARPS * 32>(dst, a.v_pool + ((size_t)next_page * a.nkv + v_lo + next_part - KH) * KT * DV, tid);
      if (++next_part == per_tile) { next_part = 0; ++next_tile; }
      ++next;
    }
    cp_async_commit();
  };
#pragma unroll
  for (int i = 0; i < NS - 1; ++i) issue();
  load_queries<WARPS * 32>(smem, q_rowb, a.q + ((size_t)tok * a.nq + head0) * width, width, heads_here, 16, width, tid);

  const int r_lo = lane >> 2, r_hi = r_lo + 8;
  const int g_lo = (head0 + r_lo) / rep, g_hi = (head0 + r_hi) / rep;      // the rows' value heads
  const float sl2 = a.scale * LOG2E;
  const int mi = lane >> 3, mr = lane & 7;
  const uint32_t a_base = smem_addr(smem) + ((mi & 1) * 8 + mr) * q_rowb + (mi >> 1) * 16;
  float o[DVTILES][4], s[2][4];
#pragma unroll
  for (int i = 0; i < DVTILES; ++i) { o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f; }
  float m_lo = -INFINITY, m_hi = -INFINITY, l_lo = 0.f, l_hi = 0.f;
  uint32_t pf[4] = {0u, 0u, 0u, 0u};

  int part = 0, kbase = tile_lo * KT + warp * 16;                          // this warp's 16 keys
  for (int it = 0; it < n_items; ++it) {
    cp_async_wait<NS - 2>();
    __syncthreads();
    issue();
    const uint32_t st = ring_addr + (uint32_t)(it % NS) * STAGE_BYTES;
    const bool active = kbase <= pos && kbase + 15 >= first_key;
    if (active && part < KH) {
      if (part == 0) {
#pragma unroll
        for (int i = 0; i < 2; ++i) { s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f; }
      }
      const uint32_t qa = a_base + (a.mixed ? part * D * 2 : 0);
      const bool mine_lo = a.mixed || g_lo == k_lo + part, mine_hi = a.mixed || g_hi == k_lo + part;
#pragma unroll
      for (int ks = 0; ks < KSTEPS; ++ks) {
        uint32_t qf[4];
        ldmatrix_x4(qa + ks * 32, qf[0], qf[1], qf[2], qf[3]);
        if (!mine_lo) qf[0] = qf[2] = 0u;
        if (!mine_hi) qf[1] = qf[3] = 0u;
        const int key = warp * 16 + (mi >> 1) * 8 + mr, dd = ks * 16 + (mi & 1) * 8;
        uint32_t b0, b1, b2, b3;
        ldmatrix_x4(st + key * ROWB_K + dd * 2, b0, b1, b2, b3);
        mma_bf16(s[0], qf, b0, b1);
        mma_bf16(s[1], qf, b2, b3);
      }
      if (part == KH - 1) {
        // the scores of this warp's keys are complete
        float mx_lo = -INFINITY, mx_hi = -INFINITY;
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const int kj = kbase + i * 8 + (lane & 3) * 2;
          const bool v0 = kj <= pos && kj >= first_key, v1 = kj + 1 <= pos && kj + 1 >= first_key;
          s[i][0] = v0 ? s[i][0] * sl2 : -INFINITY;
          s[i][1] = v1 ? s[i][1] * sl2 : -INFINITY;
          s[i][2] = v0 ? s[i][2] * sl2 : -INFINITY;
          s[i][3] = v1 ? s[i][3] * sl2 : -INFINITY;
          mx_lo = fmaxf(mx_lo, fmaxf(s[i][0], s[i][1]));
          mx_hi = fmaxf(mx_hi, fmaxf(s[i][2], s[i][3]));
        }
        mx_lo = fmaxf(mx_lo, __shfl_xor_sync(0xffffffffu, mx_lo, 1));
        mx_lo = fmaxf(mx_lo, __shfl_xor_sync(0xffffffffu, mx_lo, 2));
        mx_hi = fmaxf(mx_hi, __shfl_xor_sync(0xffffffffu, mx_hi, 1));
        mx_hi = fmaxf(mx_hi, __shfl_xor_sync(0xffffffffu, mx_hi, 2));
        const float mn_lo = fmaxf(m_lo, mx_lo), mn_hi = fmaxf(m_hi, mx_hi);     // finite: one of the 16 keys is visible
        const float al_lo = exp2f(m_lo - mn_lo), al_hi = exp2f(m_hi - mn_hi);
        m_lo = mn_lo; m_hi = mn_hi;
        float sum_lo = 0.f, sum_hi = 0.f;
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const float e0 = exp2f(s[i][0] - mn_lo), e1 = exp2f(s[i][1] - mn_lo);
          const float e2 = exp2f(s[i][2] - mn_hi), e3 = exp2f(s[i][3] - mn_hi);
          sum_lo += e0 + e1; sum_hi += e2 + e3;
          pf[i * 2] = pack_bf16(e0, e1);
          pf[i * 2 + 1] = pack_bf16(e2, e3);
        }
        l_lo = l_lo * al_lo + sum_lo; l_hi = l_hi * al_hi + sum_hi;
#pragma unroll
        for (int i = 0; i < DVTILES; ++i) { o[i][0] *= al_lo; o[i][1] *= al_lo; o[i][2] *= al_hi; o[i][3] *= al_hi; }
      }
    } else if (active) {
      const int vh = v_lo + part - KH;
      uint32_t pv[4];
      pv[0] = g_lo == vh ? pf[0] : 0u; pv[2] = g_lo == vh ? pf[2] : 0u;
      pv[1] = g_hi == vh ? pf[1] : 0u; pv[3] = g_hi == vh ? pf[3] : 0u;
#pragma unroll
      for (int dp = 0; dp < DVTILES / 2; ++dp) {
        const int key = warp * 16 + (mi & 1) * 8 + mr, dd = dp * 16 + (mi >> 1) * 8;
        uint32_t b0, b1, b2, b3;
        ldmatrix_x4_trans(st + key * ROWB_V + dd * 2, b0, b1, b2, b3);
        mma_bf16(o[dp * 2], pv, b0, b1);
        mma_bf16(o[dp * 2 + 1], pv, b2, b3);
      }
    }
    if (++part == per_tile) { part = 0; kbase += KT; }
  }
  cp_async_wait<0>();
  __syncthreads();
  // merge the four warps (each saw a quarter of the keys): [warp][row][DV + 2] floats over the free ring
  l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 1); l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 2);
  l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 1); l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 2);
  float* mg = (float*)ring;
  {
    const int c = (lane & 3) * 2;
    float* lo = mg + ((size_t)warp * 16 + r_lo) * RS;
    float* hi = mg + ((size_t)warp * 16 + r_hi) * RS;
#pragma unroll
    for (int i = 0; i < DVTILES; ++i) {
      lo[i * 8 + c] = o[i][0]; lo[i * 8 + c + 1] = o[i][1];
      hi[i * 8 + c] = o[i][2]; hi[i * 8 + c + 1] = o[i][3];
    }
    if ((lane & 3) == 0) { lo[DV] = m_lo; lo[DV + 1] = l_lo; hi[DV] = m_hi; hi[DV + 1] = l_hi; }
  }
  __syncthreads();
  for (int row = warp; row < heads_here; row += WARPS) {
    float M = -INFINITY;
#pragma unroll
    for (int w = 0; w < WARPS; ++w) M = fmaxf(M, mg[((size_t)w * 16 + row) * RS + DV]);
    float wgt[WARPS], L = 0.f;
#pragma unroll
    for (int w = 0; w < WARPS; ++w) {
      const float mw = mg[((size_t)w * 16 + row) * RS + DV];
      wgt[w] = mw == -INFINITY ? 0.f : exp2f(mw - M);
      L += wgt[w] * mg[((size_t)w * 16 + row) * RS + DV + 1];
    }
    const int head = head0 + row;
    const float inv = a.splits == 1 ? (L > 0.f ? 1.f / L : 0.f) : 1.f;
    float* dst = a.splits == 1 ? nullptr : a.partial + (((size_t)tok * a.nq + head) * a.splits + split) * RS;
    for (int dd = lane; dd < DV; dd += 32) {
      float v = 0.f;
#pragma unroll
      for (int w = 0; w < WARPS; ++w) v += wgt[w] * mg[((size_t)w * 16 + row) * RS + dd];
      if (dst == nullptr) a.out[((size_t)tok * a.nq + head) * DV + dd] = __float2bfloat16_rn(v * inv);
      else dst[dd] = v;
    }
    if (dst != nullptr && lane == 0) { dst[DV] = M; dst[DV + 1] = L; }       // the maximum in the log2 domain
  }
}

// Merge the partials of one (token, head): out = sum_s 2^(m_s - M) acc_s / sum_s 2^(m_s - M) l_s, splits in order.
__global__ void attention_mixed_combine_kernel(const float* __restrict__ partial, bf16* __restrict__ out, int splits) {
  pdl_launch_dependents();
  pdl_wait();
  const size_t row = blockIdx.x;  // token * nq + head
  const float* p = partial + row * splits * RS;
  float M = -INFINITY;
  for (int s = 0; s < splits; ++s) M = fmaxf(M, p[s * RS + DV]);
  float denom = 0.f;
  for (int s = 0; s < splits; ++s) {
    const float ms = p[s * RS + DV];
    if (ms != -INFINITY) denom += exp2f(ms - M) * p[s * RS + DV + 1];
  }
  const float inv = denom > 0.f ? 1.f / denom : 0.f;
  for (int dd = threadIdx.x; dd < DV; dd += blockDim.x) {
    float v = 0.f;
    for (int s = 0; s < splits; ++s) {
      const float ms = p[s * RS + DV];
      if (ms != -INFINITY) v += exp2f(ms - M) * p[s * RS + dd];
    }
    out[row * DV + dd] = __float2bfloat16_rn(v * inv);
  }
}

// ------------------------------------------------------------------------------ launches

static size_t query_bytes(const MixedAttnArgs& a, int rows) { return (size_t)rows * ((a.mixed ? a.nkv : 1) * D * 2 + 16); }
static size_t merge_bytes() { return (size_t)WARPS * 16 * RS * sizeof(float); }

// Whether the kernels' shared memory holds the query rows of these heads.
extern "C" int odi_attention_mixed_fits(int nkv, int mixed) {
  MixedAttnArgs a = {};
  a.nkv = nkv; a.mixed = mixed;
  return query_bytes(a, 64) + 2 * STAGE_BYTES <= SMEM_LIMIT;
}

static int check_args(const MixedAttnArgs& a) {
  if (a.nkv <= 0 || a.nq % a.nkv != 0 || a.n_seqs > 65535 || a.chunk < 0 || a.ring_pages < 0 || a.splits < 1) return ODI_ERR_UNSUPPORTED;
  if (((uintptr_t)a.q | (uintptr_t)a.k_pool | (uintptr_t)a.v_pool | (uintptr_t)a.out) % 16 != 0) return ODI_ERR_UNSUPPORTED;
  if (a.splits > 1 && a.partial == nullptr) return ODI_ERR_ARGUMENT;
  return 0;
}

template <typename K>
static int launch_one(K kernel, int warps, size_t smem, dim3 grid, const MixedAttnArgs& a, cudaStream_t stream) {
  const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return (int)e;
  return launch_pdl(kernel, grid, dim3(warps * 32), smem, stream, a);
}

// max_q_len: the longest q_len of the batch (sizes the grid).
extern "C" int odi_attention_mixed(const MixedAttnArgs* args, int max_q_len, cudaStream_t stream) {
  const MixedAttnArgs a = *args;
  if (a.n_seqs <= 0 || max_q_len <= 0) return 0;
  const int bad = check_args(a);
  if (bad) return bad;
  const int q_tiles = (max_q_len + 63) / 64;
  if (q_tiles > 65535) return ODI_ERR_UNSUPPORTED;
  const dim3 grid(a.nq, a.n_seqs, q_tiles);
  const size_t q = query_bytes(a, 64);
  if (q + 3 * STAGE_BYTES <= SMEM_LIMIT) odi_rc = launch_one(attention_mixed_kernel<3>, PROMPT_WARPS, q + 3 * STAGE_BYTES, grid, a, stream);
  else if (q + 2 * STAGE_BYTES <= SMEM_LIMIT) odi_rc = launch_one(attention_mixed_kernel<2>, PROMPT_WARPS, q + 2 * STAGE_BYTES, grid, a, stream);
  else return ODI_ERR_UNSUPPORTED;
  return launch_status();
}

// One token per sequence; `partial` holds n_seqs * nq * splits * (DV + 2) floats when splits > 1.
extern "C" int odi_attention_mixed_decode(const MixedAttnArgs* args, cudaStream_t stream) {
  const MixedAttnArgs a = *args;
  if (a.n_seqs <= 0) return 0;
  const int bad = check_args(a);
  if (bad) return bad;
  const dim3 grid(a.splits, (a.nq + 15) / 16, a.n_seqs);
  if (grid.y > 65535) return ODI_ERR_UNSUPPORTED;
  const size_t q = query_bytes(a, 16), m = merge_bytes();
  const size_t four = 4 * STAGE_BYTES > m ? 4 * STAGE_BYTES : m, two = 2 * STAGE_BYTES > m ? 2 * STAGE_BYTES : m;
  if (q + four <= SMEM_LIMIT) odi_rc = launch_one(attention_mixed_decode_kernel<4>, WARPS, q + four, grid, a, stream);
  else if (q + two <= SMEM_LIMIT) odi_rc = launch_one(attention_mixed_decode_kernel<2>, WARPS, q + two, grid, a, stream);
  else return ODI_ERR_UNSUPPORTED;
  if (odi_rc == 0 && a.splits > 1) {
    const int threads = DV >= 128 ? 128 : (DV >= 64 ? 64 : 32);
    odi_rc = launch_pdl(attention_mixed_combine_kernel, dim3(a.n_seqs * a.nq), dim3(threads), 0, stream, (const float*)a.partial, a.out, a.splits);
  }
  return launch_status();
}
