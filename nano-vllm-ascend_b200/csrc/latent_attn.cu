// latent_attn.cu -- causal softmax attention over cached latent rows, 16-bit models: every query head of a token reads the
// SAME row [latent (R) | rotated key part] per key, as key (all D columns) and as value (the first R columns).
//
// The rows of a launch are (token, head) pairs of one sequence, so a decode step (one token, H heads), a short portion and
// a whole prompt are the same problem. One CTA = 16 warps = 16 * MT rows against a contiguous share of the keys, 64 at a time:
//   * key rows land in a two-stage shared-memory ring by cp.async (16 bytes per thread and step, zero-filled past the
//     keys and past D), row pitch D + 8 elements so that ldmatrix is free of bank conflicts;
//   * S = Q K^T on mma.sync m16n8k16: the query fragments live in registers for the whole CTA, the inner dimension is
//     split over four groups of warps (each keeps a quarter of the fragments), their partial scores meet in shared
//     memory;
//   * softmax in fp32 with a running maximum, 16 or 32 lanes per row; the weights go to shared memory in the element type;
//   * O += P V: every warp owns R / 16 columns of all rows; V fragments are read from the same key rows (ldmatrix.trans).
// A decode step streams each cached row once: the kernel is bound by HBM, mma.sync has the head room (16 or 32 rows per
// key row). Keys can be split over several CTAs (few rows, many keys): un-normalised fp32 partials, merged by a small
// kernel. window > 0: a row at position i sees the keys j <= i with i - j < window.
#include "seq_common.cuh"

namespace b200 {

constexpr int kLatKeys = 64;                          // keys per tile
constexpr int kLatWarps = 16;
constexpr int kLatThreads = kLatWarps * 32;
constexpr int kLatParts = kLatWarps / 4;              // parts of the inner dimension in S = Q K^T
constexpr int kLatPad = 16 * kLatParts;               // key rows are padded to a multiple of this
constexpr int kLatSPitch = kLatKeys + 4;              // fp32 row of partial scores
constexpr int kLatPPitch = kLatKeys + 8;              // 16-bit row of weights

struct LatentParams {
  const void* q;                                      // [tokens, H, D]
  const void* k;                                      // packed rows [*, D] (row stride k_stride), or the paged cache
  void* out;                                          // [tokens, H, R]
  int64_t k_stride;
  const int *block_tables, *cu_q, *cu_k, *ctx_lens;
  int bt_stride, block_size;
  int H, D, R, window, splits;
  float scale_log2;
  float* part_o;                                      // splits > 1: [tokens * H][splits][R]
  float* part_ml;                                     // splits > 1: [tokens * H][splits][2]
};

template <int MT>
constexpr size_t latent_smem_bytes(int pitch) {
  return (size_t)2 * kLatKeys * pitch * 2 + (size_t)kLatParts * 16 * MT * kLatSPitch * 4 + (size_t)16 * MT * kLatPPitch * 2 +
         (size_t)3 * 16 * MT * 4;
}

// KH: k16 steps of one part of the inner dimension (64 * KH >= D); NT8: 8-wide column tiles per warp (128 * NT8 >= R)
template <typename T, int MT, int KH, int NT8>
__global__ void __launch_bounds__(kLatThreads, 1)
latent_attn_kernel(const LatentParams P) {
  extern __shared__ __align__(16) uint8_t lat_smem[];
  constexpr int ROWS = 16 * MT;
  constexpr int LPR = kLatThreads / ROWS;                     // lanes per row in the softmax
  constexpr int KPL = kLatKeys / LPR;                 // keys per lane
  constexpr int NKT = MT;                             // pairs of 8-key tiles per warp in S = Q K^T
  pdl_wait();
  const SeqSpan sp = seq_span(P.cu_q, P.cu_k, P.ctx_lens, blockIdx.y);
  const int rows = sp.q_len * P.H;
  const int split = (int)blockIdx.x % P.splits;
  const int n_tiles = (int)gridDim.x / P.splits;
  const int r0 = (n_tiles - 1 - (int)blockIdx.x / P.splits) * ROWS;    // late rows (the longest) first
  if (r0 >= rows) return;
  const int D = P.D, R = P.R;
  const int Dp = (D + kLatPad - 1) / kLatPad * kLatPad;
  const int pitch = Dp + 8;                           // elements
  T* sK = reinterpret_cast<T*>(lat_smem);             // [2][kLatKeys][pitch]
  float* sS = reinterpret_cast<float*>(sK + 2 * kLatKeys * pitch);     // [kLatParts][ROWS][kLatSPitch]
  T* sP = reinterpret_cast<T*>(sS + kLatParts * ROWS * kLatSPitch);            // [ROWS][kLatPPitch]
  float* sAlpha = reinterpret_cast<float*>(sP + ROWS * kLatPPitch);    // [ROWS]
  float* sL = sAlpha + ROWS;                          // [ROWS] final sums
  float* sM = sL + ROWS;                              // [ROWS] final maxima (exp2 domain)

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = lane >> 2, t4 = lane & 3;
  const int first_pos = sp.first_pos();

  // ---- this CTA's share of the key tiles
  const int last = min(r0 + ROWS, rows) - 1;
  const int max_pos = first_pos + last / P.H;
  const int lo_key = P.window > 0 ? max(0, first_pos + r0 / P.H - P.window + 1) / kLatKeys * kLatKeys : 0;
  const int tiles = (max_pos - lo_key) / kLatKeys + 1;
  const int j0 = (int)((int64_t)tiles * split / P.splits), j1 = (int)((int64_t)tiles * (split + 1) / P.splits);

  const T* kbase = (const T*)P.k;
  const int* table = P.block_tables != nullptr ? P.block_tables + (int64_t)blockIdx.y * P.bt_stride : nullptr;
  const int64_t packed0 = table == nullptr ? P.cu_k[blockIdx.y] : 0;
  const int vpr = Dp / 8;                             // 16-byte vectors per padded row
  auto load_tile = [&](int j, int stage) {
    const int key0 = lo_key + j * kLatKeys;
    T* dst = sK + (size_t)stage * kLatKeys * pitch;
    // TPR threads per key row: one table lookup each, neighbouring vectors
    constexpr int TPR = kLatThreads / kLatKeys;
    const int r = threadIdx.x / TPR;
    const int key = key0 + r;
    const bool ok = key <= max_pos;
    int64_t row = 0;
    if (ok) row = table != nullptr ? (int64_t)table[key / P.block_size] * P.block_size + key % P.block_size : packed0 + key;
    const T* src = kbase + row * P.k_stride;
    for (int v = threadIdx.x % TPR; v < vpr; v += TPR) {
      const bool in = ok && v * 8 < D;
      cp_async_16(smem_u32(dst + r * pitch + v * 8), in ? src + v * 8 : kbase, in);
    }
    cp_async_commit();
  };
  if (j0 < j1) load_tile(j0, 0);

  // ---- query fragments of this warp: rows of M tile mt_s, k16 steps [part * kh, part * kh + kh)
  const int part = warp % kLatParts, rest = warp / kLatParts;
  const int mt_s = MT == 2 ? rest & 1 : 0;
  const int kg = MT == 2 ? rest >> 1 : rest;          // keys kg * 16 * NKT .. of a tile
  const int kh = Dp / kLatPad;
  uint32_t qf[KH][4];
  {
    const T* qb = (const T*)P.q + (int64_t)sp.q_start * P.H * D;
    const int ra = r0 + mt_s * 16 + g, rb = ra + 8;
    const T* qa = qb + (int64_t)ra * D;
    const T* qc = qb + (int64_t)rb * D;
#pragma unroll
    for (int i = 0; i < KH; ++i) {
      const int c = (part * kh + i) * 16 + 2 * t4;
      const bool in0 = i < kh && c < D, in1 = i < kh && c + 8 < D;
      qf[i][0] = in0 && ra < rows ? *reinterpret_cast<const uint32_t*>(qa + c) : 0u;
      qf[i][1] = in0 && rb < rows ? *reinterpret_cast<const uint32_t*>(qc + c) : 0u;
      qf[i][2] = in1 && ra < rows ? *reinterpret_cast<const uint32_t*>(qa + c + 8) : 0u;
      qf[i][3] = in1 && rb < rows ? *reinterpret_cast<const uint32_t*>(qc + c + 8) : 0u;
    }
  }
  float o[MT][NT8][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < NT8; ++n) o[m][n][0] = o[m][n][1] = o[m][n][2] = o[m][n][3] = 0.f;

  // softmax row of this thread
  const int srow = threadIdx.x / LPR, sub = threadIdx.x % LPR;
  const int spos = r0 + srow < rows ? first_pos + (r0 + srow) / P.H : -1;
  const int slo = P.window > 0 ? spos - P.window + 1 : 0;
  float m_run = -INFINITY, l_run = 0.f;

  for (int j = j0; j < j1; ++j) {
    const int stage = (j - j0) & 1;
    cp_async_wait<0>();
    __syncthreads();                                  // tile j has landed; everyone is done with tile j - 1
    if (j + 1 < j1) load_tile(j + 1, stage ^ 1);
    const uint32_t kb = smem_u32(sK + (size_t)stage * kLatKeys * pitch);
    // ---- partial scores over this warp's part of the inner dimension
    {
      float s[2 * NKT][4];
#pragma unroll
      for (int n = 0; n < 2 * NKT; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
      const int key = kg * 16 * NKT + ((lane >> 4) << 3) + (lane & 7);
      const uint32_t base = kb + (uint32_t)(key * pitch + part * kh * 16 + ((lane >> 3) & 1) * 8) * 2;
#pragma unroll
      for (int i = 0; i < KH; ++i) {
        if (i < kh) {
#pragma unroll
          for (int n = 0; n < NKT; ++n) {
            uint32_t b0, b1, b2, b3;
            ldsm_x4(base + (uint32_t)(n * 16 * pitch + i * 16) * 2, b0, b1, b2, b3);
            mma_16816<T>(s[2 * n], qf[i][0], qf[i][1], qf[i][2], qf[i][3], b0, b1);
            mma_16816<T>(s[2 * n + 1], qf[i][0], qf[i][1], qf[i][2], qf[i][3], b2, b3);
          }
        }
      }
      float* dst = sS + (size_t)part * ROWS * kLatSPitch + (mt_s * 16 + g) * kLatSPitch + kg * 16 * NKT + 2 * t4;
#pragma unroll
      for (int n = 0; n < 2 * NKT; ++n) {
        *reinterpret_cast<float2*>(dst + n * 8) = make_float2(s[n][0], s[n][1]);
        *reinterpret_cast<float2*>(dst + 8 * kLatSPitch + n * 8) = make_float2(s[n][2], s[n][3]);
      }
    }
    __syncthreads();
    // ---- softmax: LPR lanes per row
    {
      const float* a = sS + srow * kLatSPitch;
      const int key0 = lo_key + j * kLatKeys;
      float x[KPL];
      float mx = -INFINITY;
#pragma unroll
      for (int i = 0; i < KPL; ++i) {
        const int c = sub + LPR * i;
        const bool seen = key0 + c <= spos && key0 + c >= slo;
        float s = 0.f;
#pragma unroll
        for (int p = 0; p < kLatParts; ++p) s += a[p * ROWS * kLatSPitch + c];
        x[i] = seen ? s * P.scale_log2 : -INFINITY;
        mx = fmaxf(mx, x[i]);
      }
#pragma unroll
      for (int off = LPR / 2; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
      const float m_new = fmaxf(m_run, mx);
      const float ref = m_new == -INFINITY ? 0.f : m_new;             // nothing visible yet: all weights are zero
      const float alpha = ex2_approx(m_run - ref);
      float sum = 0.f;
#pragma unroll
      for (int i = 0; i < KPL; ++i) {
        const float p = ex2_approx(x[i] - ref);
        sum += p;
        sP[srow * kLatPPitch + sub + LPR * i] = from_f32<T>(p);
      }
#pragma unroll
      for (int off = LPR / 2; off > 0; off >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, off);
      l_run = l_run * alpha + sum;
      m_run = m_new;
      if (sub == 0) sAlpha[srow] = alpha;
    }
    __syncthreads();
    // ---- O = alpha O + P V, this warp's columns
    {
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        const float a0 = sAlpha[m * 16 + g], a1 = sAlpha[m * 16 + g + 8];
        if (__any_sync(0xffffffffu, a0 != 1.f || a1 != 1.f)) {
#pragma unroll
          for (int n = 0; n < NT8; ++n) o[m][n][0] *= a0, o[m][n][1] *= a0, o[m][n][2] *= a1, o[m][n][3] *= a1;
        }
      }
      const uint32_t pb = smem_u32(sP) + (uint32_t)(((lane & 7) + ((lane >> 3) & 1) * 8) * kLatPPitch + (lane >> 4) * 8) * 2;
      const uint32_t vb = kb + (uint32_t)((((lane >> 3) & 1) * 8 + (lane & 7)) * pitch + (lane >> 4) * 8) * 2;
#pragma unroll
      for (int ks = 0; ks < kLatKeys / 16; ++ks) {
        uint32_t pf[MT][4];
#pragma unroll
        for (int m = 0; m < MT; ++m)
          ldsm_x4(pb + (uint32_t)(m * 16 * kLatPPitch + ks * 16) * 2, pf[m][0], pf[m][1], pf[m][2], pf[m][3]);
#pragma unroll
        for (int n = 0; n < NT8 / 2; ++n) {
          const int c = (warp + kLatWarps * n) * 16;
          if (c < R) {
            uint32_t b0, b1, b2, b3;
            ldsm_x4_trans(vb + (uint32_t)(ks * 16 * pitch + c) * 2, b0, b1, b2, b3);
#pragma unroll
            for (int m = 0; m < MT; ++m) {
              mma_16816<T>(o[m][2 * n], pf[m][0], pf[m][1], pf[m][2], pf[m][3], b0, b1);
              mma_16816<T>(o[m][2 * n + 1], pf[m][0], pf[m][1], pf[m][2], pf[m][3], b2, b3);
            }
          }
        }
      }
    }
  }
  if (sub == 0) sL[srow] = l_run, sM[srow] = m_run;
  __syncthreads();
  const int64_t row0 = (int64_t)sp.q_start * P.H + r0;
  if (P.splits > 1 && threadIdx.x < ROWS && r0 + (int)threadIdx.x < rows) {
    float* ml = P.part_ml + ((row0 + threadIdx.x) * P.splits + split) * 2;
    ml[0] = sM[threadIdx.x];
    ml[1] = sL[threadIdx.x];
  }
#pragma unroll
  for (int m = 0; m < MT; ++m) {
#pragma unroll
    for (int e = 0; e < 2; ++e) {                     // rows g and g + 8 of the M tile
      const int r = m * 16 + g + 8 * e;
      if (r0 + r >= rows) continue;
      const float l = sL[r];
      const float inv = l > 0.f ? 1.0f / l : 0.f;
#pragma unroll
      for (int n = 0; n < NT8; ++n) {
        const int c = (warp + kLatWarps * (n >> 1)) * 16 + (n & 1) * 8 + 2 * t4;
        if (c >= R) continue;
        const float x = o[m][n][2 * e], y = o[m][n][2 * e + 1];
        if (P.splits > 1)
          *reinterpret_cast<float2*>(P.part_o + ((row0 + r) * P.splits + split) * R + c) = make_float2(x, y);
        else
          *reinterpret_cast<uint32_t*>((T*)P.out + (row0 + r) * R + c) = pack2<T>(x * inv, y * inv);
      }
    }
  }
}

// merge of the key splits: one warp per (token, head) row
template <typename T>
__global__ void __launch_bounds__(256)
latent_combine_kernel(T* __restrict__ out, const float* __restrict__ part_o, const float* __restrict__ part_ml,
                      const int* __restrict__ ctx_lens, int64_t total, int H, int R, int splits) {
  pdl_wait();
  const int64_t row = (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (row >= total) return;
  if (ctx_lens != nullptr && ctx_lens[row / H] <= 0) return;           // a padded row wrote no partials
  const float* ml = part_ml + row * splits * 2;
  float m = -INFINITY;
  for (int s = 0; s < splits; ++s) m = fmaxf(m, ml[2 * s]);
  float l = 0.f;
  for (int s = 0; s < splits; ++s) l += ml[2 * s] == -INFINITY ? 0.f : ml[2 * s + 1] * ex2_approx(ml[2 * s] - m);
  const float inv = l > 0.f ? 1.0f / l : 0.f;
  for (int c = 2 * lane; c < R; c += 64) {
    float x = 0.f, y = 0.f;
    for (int s = 0; s < splits; ++s) {
      const float ms = ml[2 * s];
      if (ms == -INFINITY) continue;
      const float w = ex2_approx(ms - m);
      const float2 p = *reinterpret_cast<const float2*>(part_o + (row * splits + s) * R + c);
      x += w * p.x, y += w * p.y;
    }
    *reinterpret_cast<uint32_t*>(out + row * R + c) = pack2<T>(x * inv, y * inv);
  }
}

template <typename T, int MT, int KH, int NT8>
static int latent_launch_t(const LatentParams& P, int row_tiles, int num_seqs, cudaStream_t stream) {
  const size_t smem = latent_smem_bytes<MT>((P.D + kLatPad - 1) / kLatPad * kLatPad + 8);
  auto kern = latent_attn_kernel<T, MT, KH, NT8>;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  launch_pdl(kern, dim3(row_tiles * P.splits, num_seqs), dim3(kLatThreads), smem, stream, P);
  return B200_OK;
}

template <typename T, int MT>
static int latent_launch_m(const LatentParams& P, int row_tiles, int num_seqs, cudaStream_t stream) {
  if (P.D <= 128 && P.R <= 256) return latent_launch_t<T, MT, 2, 2>(P, row_tiles, num_seqs, stream);
  if (P.D <= 320 && P.R <= 256) return latent_launch_t<T, MT, 5, 2>(P, row_tiles, num_seqs, stream);
  return latent_launch_t<T, MT, 9, 4>(P, row_tiles, num_seqs, stream);
}

}  // namespace b200

using namespace b200;

// Key splits for a launch of `ctas` row-tile CTAs. Model, in units of one key tile: every CTA costs about three tiles
// (query fragments, pipeline fill, epilogue), a split launch a merge whose cost grows with the splits.
extern "C" int b200_latent_attn_splits(int64_t ctas, int32_t max_keys) {
  const double tiles = (max_keys + kLatKeys - 1) / kLatKeys;
  const int most = max_keys / (2 * kLatKeys) < 16 ? max_keys / (2 * kLatKeys) : 16;
  int best = 1;
  double cost = (double)((ctas + 147) / 148) * (3.0 + tiles);
  for (int s = 2; s <= most; ++s) {
    const double c = (double)((ctas * s + 147) / 148) * (3.0 + tiles / s) + 2.0 + 0.75 * s;
    if (c < cost) cost = c, best = s;
  }
  return best;
}

extern "C" int b200_latent_attn(void* out, const void* q, const void* k, int64_t k_stride, const int32_t* block_tables,
                                int32_t bt_stride, int32_t block_size, const int32_t* cu_q, const int32_t* cu_k,
                                const int32_t* ctx_lens, int32_t num_seqs, int32_t max_q, int32_t total_q,
                                int32_t num_heads, int32_t dim, int32_t rank, float scale, int32_t window, int32_t splits,
                                float* part_o, float* part_ml, int32_t dtype, b200_stream_t stream) {
  B200_RETURN_IF(dtype != B200_DTYPE_BF16 && dtype != B200_DTYPE_F16, B200_ERR_BAD_DTYPE);
  B200_RETURN_IF(num_seqs < 0 || max_q < 0 || total_q < 0 || num_heads <= 0 || rank <= 0 || dim < rank || window < 0 ||
                     splits <= 0 || k_stride < dim, B200_ERR_BAD_SHAPE);
  B200_RETURN_IF(dim % 8 != 0 || rank % 8 != 0 || dim > 576 || rank > 512 || num_seqs > 65535, B200_ERR_UNSUPPORTED);
  if (num_seqs == 0 || max_q == 0) return B200_OK;
  B200_RETURN_IF(!out || !q || !k || (cu_q == nullptr) == (ctx_lens == nullptr) || (cu_q && !cu_k) ||
                     (!block_tables && !cu_q) || (splits > 1 && (!part_o || !part_ml)), B200_ERR_NULL_POINTER);
  B200_RETURN_IF(block_tables && block_size <= 0, B200_ERR_BAD_SHAPE);
  B200_RETURN_IF(!aligned16(q) || !aligned16(k) || !aligned16(out) || k_stride % 8 != 0, B200_ERR_MISALIGNED);
  LatentParams P;
  P.q = q, P.k = k, P.out = out, P.k_stride = k_stride, P.block_tables = block_tables, P.cu_q = cu_q, P.cu_k = cu_k;
  P.ctx_lens = ctx_lens, P.bt_stride = bt_stride, P.block_size = block_size, P.H = num_heads, P.D = dim, P.R = rank;
  P.window = window, P.splits = splits, P.scale_log2 = scale * kLog2e, P.part_o = part_o, P.part_ml = part_ml;
  const int64_t rows = (int64_t)max_q * num_heads;
  const bool two = rows > 16;
  const int64_t row_tiles = two ? (rows + 31) / 32 : 1;
  B200_RETURN_IF(row_tiles * splits > 0x7fffffff, B200_ERR_UNSUPPORTED);
  int rc;
  if (dtype == B200_DTYPE_BF16)
    rc = two ? latent_launch_m<__nv_bfloat16, 2>(P, (int)row_tiles, num_seqs, (cudaStream_t)stream)
             : latent_launch_m<__nv_bfloat16, 1>(P, (int)row_tiles, num_seqs, (cudaStream_t)stream);
  else
    rc = two ? latent_launch_m<__half, 2>(P, (int)row_tiles, num_seqs, (cudaStream_t)stream)
             : latent_launch_m<__half, 1>(P, (int)row_tiles, num_seqs, (cudaStream_t)stream);
  if (rc != B200_OK) return rc;
  if (splits > 1) {
    const int64_t total = (int64_t)total_q * num_heads;
    const dim3 grid((unsigned)((total + 7) / 8));
    if (dtype == B200_DTYPE_BF16)
      launch_pdl(latent_combine_kernel<__nv_bfloat16>, grid, dim3(256), 0, (cudaStream_t)stream, (__nv_bfloat16*)out,
                 (const float*)part_o, (const float*)part_ml, ctx_lens, total, num_heads, rank, splits);
    else
      launch_pdl(latent_combine_kernel<__half>, grid, dim3(256), 0, (cudaStream_t)stream, (__half*)out,
                 (const float*)part_o, (const float*)part_ml, ctx_lens, total, num_heads, rank, splits);
  }
  return finish_launch(splits > 1 ? 2 : 1);
}
