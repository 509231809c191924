// delta_rule.cu -- recurrences with an fp32 state S [kdim x vdim] per head whose decay changes from token to token:
//
//   gated delta rule   S <- diag(g_t) S;   w = beta_t (v_t - S^T k_t);   S <- S + k_t w^T;   o_t = S^T q_t
//                      (the read-out sees the current token's write), with one decay per head and key channel, or one
//                      per head (g_t a number)
//   wkv                o_t = S^T q_t + c_t v_t;   S <- diag(g_t) S + k_t v_t^T   (the read-out comes before the write; the
//                      current token counts through its own coefficient c_t = sum_i q_i u_i k_i)
//
// q, k (unit vectors, per key/value group, for the delta rule), g and beta (wkv: c) arrive in fp32 from delta_prep /
// wkv_prep; v in the model's element type. The state is carried between
// steps in a slot, exactly as the other recurrences: [slots, H, kdim, vdim] fp32; a span that starts at position 0
// ignores what the slot held.
//
// One CTA = 32 NS threads = one (sequence, head) and a band of 32 NC value columns. A thread owns NC neighbouring value
// columns and KPT key rows of S in registers; NS adjacent lanes share the columns, a slice of KPT rows each. Per token the
// delta rule makes two passes over its rows -- decay + the projection S^T k, then the rank-one write + the read-out S^T q --
// and wkv one, with k, q, g read as float4 broadcasts from shared memory; the dot products are finished by xor shuffles
// among the NS lanes. The broadcasts bound the kernel, so a thread uses each of them for NC columns, and the slices of a
// row lie KPT + 4 floats apart: the NS lanes of a column group read different banks. Tokens are staged kDeltaTok at a
// time; where the rows allow 16-byte copies (VEC) the next batch arrives by cp.async in a second set of buffers while the
// current one is consumed, otherwise batches are loaded in place.
#include "seq_common.cuh"

namespace b200 {

constexpr int kDeltaTok = 8;
enum { kDecayPerChannel = 0, kDecayPerHead = 1, kWkv = 2 };

struct DeltaParams {
  const float *q, *k;               // [tokens, groups * kdim]
  const float* g;                   // [tokens, H * kdim]; one decay per head: [tokens, H]
  const float* beta;                // [tokens, H]; wkv: the current token's coefficient
  const void* v;                    // [tokens, H * vdim], element type
  int64_t q_stride, k_stride, v_stride;
  float* out;                       // [tokens, H * vdim] fp32
  float* state;                     // [slots, H, kdim, vdim] fp32 or nullptr
  const int *state_slots, *cu_q, *cu_k, *ctx_lens;
  int H, groups, kdim, vdim;
};

__device__ __forceinline__ void cp_async_4(uint32_t smem_addr, const void* gptr, bool pred) {
  const int bytes = pred ? 4 : 0;
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(smem_addr), "l"(gptr), "r"(bytes) : "memory");
}

template <typename TV, int KPT, int NS, int NC, bool VEC, int MODE>
__global__ void __launch_bounds__(32 * NS)
delta_rule_kernel(const DeltaParams P) {
  extern __shared__ __align__(16) float smem[];
  pdl_wait();
  constexpr int NTH = 32 * NS;
  constexpr int KS = KPT + 4;                        // slice stride: NS lanes, different banks
  constexpr int KP = NS * KS;                        // row of padded keys
  constexpr int CC = 32 * NC;                        // value columns per CTA
  const int s = blockIdx.z, h = blockIdx.y;
  const SeqSpan sp = seq_span(P.cu_q, P.cu_k, P.ctx_lens, s);
  if (sp.q_len == 0) return;
  const int kdim = P.kdim, vdim = P.vdim;
  const int ksl = threadIdx.x % NS, cl = (threadIdx.x / NS) * NC;
  const int c0 = blockIdx.x * CC, col = c0 + cl;
  const int grp = h / (P.H / P.groups);
  constexpr int NB = VEC ? 2 : 1;                    // sets of staging buffers
  constexpr int QK = kDeltaTok * KP;
  constexpr int GT = MODE == kDecayPerHead ? 1 : KP; // decays per token
  float* sq = smem;                                  // [NB][kDeltaTok][KP]
  float* sk = sq + NB * QK;
  float* sg = sk + NB * QK;                          // [NB][kDeltaTok][GT]
  float* sb = sg + NB * kDeltaTok * GT;              // [NB][kDeltaTok]
  float* sx = sb + NB * kDeltaTok;                   // [kDeltaTok][CC] fp32 (in-place form)
  TV* sxr = reinterpret_cast<TV*>(sb + NB * kDeltaTok);   // [2][kDeltaTok][CC] as stored (cp.async form)

  float S[NC][KPT];
  float* slot = P.state != nullptr
                    ? P.state + (((int64_t)P.state_slots[s] * P.H + h) * kdim) * (int64_t)vdim
                    : nullptr;
  const bool carried = slot != nullptr && sp.first_pos() > 0;
#pragma unroll
  for (int r = 0; r < KPT; ++r) {
    const int i = ksl * KPT + r;
#pragma unroll
    for (int c = 0; c < NC; ++c)
      S[c][r] = (carried && col + c < vdim && i < kdim) ? slot[(int64_t)i * vdim + col + c] : 0.f;
  }
  const float* q = P.q + (int64_t)grp * kdim;
  const float* k = P.k + (int64_t)grp * kdim;
  const float* g = P.g + (int64_t)h * (MODE == kDecayPerHead ? 1 : kdim);
  const TV* v = (const TV*)P.v + (int64_t)h * vdim + c0;
  const int vcols = min(CC, vdim - c0);
  const int64_t g_stride = (int64_t)P.H * (MODE == kDecayPerHead ? 1 : kdim);
  auto word = [](int i) { return (i / KPT) * KS + i % KPT; };      // key row i of a token's padded row

  auto issue = [&](int t0, int b) {                  // cp.async form: batch t0 into buffer set b (zero-filled padding)
    const int nt = min(kDeltaTok, sp.q_len - t0);
    const int64_t tok0 = sp.q_start + t0;
    constexpr int K4 = NS * KPT / 4, VE = 16 / (int)sizeof(TV);
    for (int e = threadIdx.x; e < kDeltaTok * K4; e += NTH) {
      const int tt = e / K4, i = (e % K4) * 4;
      const bool ok = tt < nt && i < kdim;
      const int64_t tok = tok0 + (tt < nt ? tt : 0);
      const int ii = ok ? i : 0, at = b * QK + tt * KP + word(i);
      cp_async_16(smem_u32(sq + at), q + tok * P.q_stride + ii, ok);
      cp_async_16(smem_u32(sk + at), k + tok * P.k_stride + ii, ok);
      if constexpr (MODE != kDecayPerHead) cp_async_16(smem_u32(sg + at), g + tok * g_stride + ii, ok);
    }
    for (int e = threadIdx.x; e < kDeltaTok * CC / VE; e += NTH) {
      const int tt = e / (CC / VE), c = (e % (CC / VE)) * VE;
      const bool ok = tt < nt && c < vcols;
      cp_async_16(smem_u32(sxr + (b * kDeltaTok + tt) * CC + c), v + (tok0 + (tt < nt ? tt : 0)) * P.v_stride + (ok ? c : 0), ok);
    }
    if (threadIdx.x < kDeltaTok) {
      const bool ok = (int)threadIdx.x < nt;
      if constexpr (MODE == kDecayPerHead)
        cp_async_4(smem_u32(sg + b * kDeltaTok + threadIdx.x), g + (tok0 + (ok ? threadIdx.x : 0)) * g_stride, ok);
      cp_async_4(smem_u32(sb + b * kDeltaTok + threadIdx.x), P.beta + (tok0 + (ok ? threadIdx.x : 0)) * P.H + h, ok);
    }
    cp_async_commit();
  };
  if (VEC) issue(0, 0);
  int b = 0;
  for (int t0 = 0; t0 < sp.q_len; t0 += kDeltaTok, b ^= (VEC ? 1 : 0)) {
    const int nt = min(kDeltaTok, sp.q_len - t0);
    const int64_t tok0 = sp.q_start + t0;
    if (VEC) {
      cp_async_wait<0>();
      __syncthreads();                               // batch b has landed everywhere; set b ^ 1 has been consumed
      if (t0 + kDeltaTok < sp.q_len) issue(t0 + kDeltaTok, b ^ 1);
    } else {
      __syncthreads();                               // the previous batch has been consumed
      for (int e = threadIdx.x; e < kDeltaTok * NS * KPT; e += NTH) {
        const int tt = e / (NS * KPT), i = e % (NS * KPT), at = tt * KP + word(i);
        const bool ok = tt < nt && i < kdim;
        sq[at] = ok ? q[(tok0 + tt) * P.q_stride + i] : 0.f;
        sk[at] = ok ? k[(tok0 + tt) * P.k_stride + i] : 0.f;
        if constexpr (MODE != kDecayPerHead) sg[at] = ok ? g[(tok0 + tt) * g_stride + i] : 0.f;
      }
      for (int e = threadIdx.x; e < kDeltaTok * CC; e += NTH) {
        const int tt = e / CC, c = e % CC;
        sx[e] = (tt < nt && c < vcols) ? to_f32<TV>(v[(tok0 + tt) * P.v_stride + c]) : 0.f;
      }
      if (threadIdx.x < kDeltaTok) {
        sb[threadIdx.x] = threadIdx.x < nt ? P.beta[(tok0 + threadIdx.x) * P.H + h] : 0.f;
        if constexpr (MODE == kDecayPerHead) sg[threadIdx.x] = threadIdx.x < nt ? g[(tok0 + threadIdx.x) * g_stride] : 0.f;
      }
      __syncthreads();
    }
    float* outp = P.out + tok0 * ((int64_t)P.H * vdim) + (int64_t)h * vdim + col;
    for (int tt = 0; tt < nt; ++tt) {
      const int at = b * QK + tt * KP + ksl * KS;
      const float4* q4 = reinterpret_cast<const float4*>(sq + at);
      const float4* k4 = reinterpret_cast<const float4*>(sk + at);
      const float4* g4 = reinterpret_cast<const float4*>(sg + at);       // (one decay per head: not read)
      const float coef = sb[b * kDeltaTok + tt];
      float x[NC], o[NC][2];                         // two partial sums per column
#pragma unroll
      for (int c = 0; c < NC; ++c) {
        x[c] = VEC ? to_f32<TV>(sxr[(b * kDeltaTok + tt) * CC + cl + c]) : sx[tt * CC + cl + c];
        o[c][0] = o[c][1] = 0.f;
      }
      if constexpr (MODE == kWkv) {
#pragma unroll
        for (int r4 = 0; r4 < KPT / 4; ++r4) {
          const float4 gg = g4[r4], kk = k4[r4], qq = q4[r4];
#pragma unroll
          for (int c = 0; c < NC; ++c) {
            float* Sc = S[c] + r4 * 4;
            o[c][0] += Sc[0] * qq.x;
            Sc[0] = fmaf(Sc[0], gg.x, kk.x * x[c]);
            o[c][1] += Sc[1] * qq.y;
            Sc[1] = fmaf(Sc[1], gg.y, kk.y * x[c]);
            o[c][0] += Sc[2] * qq.z;
            Sc[2] = fmaf(Sc[2], gg.z, kk.z * x[c]);
            o[c][1] += Sc[3] * qq.w;
            Sc[3] = fmaf(Sc[3], gg.w, kk.w * x[c]);
          }
        }
      } else {
        const float g1 = MODE == kDecayPerHead ? sg[b * kDeltaTok + tt] : 0.f;
        float d[NC][2];
#pragma unroll
        for (int c = 0; c < NC; ++c) d[c][0] = d[c][1] = 0.f;
#pragma unroll
        for (int r4 = 0; r4 < KPT / 4; ++r4) {
          const float4 kk = k4[r4];
          const float4 gg = MODE == kDecayPerHead ? make_float4(g1, g1, g1, g1) : g4[r4];
#pragma unroll
          for (int c = 0; c < NC; ++c) {
            float* Sc = S[c] + r4 * 4;
            Sc[0] *= gg.x;
            d[c][0] += Sc[0] * kk.x;
            Sc[1] *= gg.y;
            d[c][1] += Sc[1] * kk.y;
            Sc[2] *= gg.z;
            d[c][0] += Sc[2] * kk.z;
            Sc[3] *= gg.w;
            d[c][1] += Sc[3] * kk.w;
          }
        }
#pragma unroll
        for (int c = 0; c < NC; ++c) {
          float dc = d[c][0] + d[c][1];
#pragma unroll
          for (int off = 1; off < NS; off <<= 1) dc += __shfl_xor_sync(0xffffffffu, dc, off);
          x[c] = coef * (x[c] - dc);                 // what is written
        }
#pragma unroll
        for (int r4 = 0; r4 < KPT / 4; ++r4) {
          const float4 kk = k4[r4], qq = q4[r4];
#pragma unroll
          for (int c = 0; c < NC; ++c) {
            float* Sc = S[c] + r4 * 4;
            Sc[0] += kk.x * x[c];
            o[c][0] += Sc[0] * qq.x;
            Sc[1] += kk.y * x[c];
            o[c][1] += Sc[1] * qq.y;
            Sc[2] += kk.z * x[c];
            o[c][0] += Sc[2] * qq.z;
            Sc[3] += kk.w * x[c];
            o[c][1] += Sc[3] * qq.w;
          }
        }
      }
#pragma unroll
      for (int c = 0; c < NC; ++c) {
        float oc = o[c][0] + o[c][1];
#pragma unroll
        for (int off = 1; off < NS; off <<= 1) oc += __shfl_xor_sync(0xffffffffu, oc, off);
        if (MODE == kWkv) oc += coef * x[c];
        if (ksl == c % NS && col + c < vdim) outp[(int64_t)tt * ((int64_t)P.H * vdim) + c] = oc;
      }
    }
  }
  if (slot != nullptr) {
#pragma unroll
    for (int r = 0; r < KPT; ++r) {
      const int i = ksl * KPT + r;
#pragma unroll
      for (int c = 0; c < NC; ++c)
        if (i < kdim && col + c < vdim) slot[(int64_t)i * vdim + col + c] = S[c][r];
    }
  }
}

template <typename TV, int KPT, int NS, int NC, int MODE>
static void delta_launch_as(const DeltaParams& P, int num_seqs, cudaStream_t stream) {
  constexpr int CC = 32 * NC, KP = NS * (KPT + 4);
  constexpr int VE = 16 / (int)sizeof(TV);
  const dim3 grid((P.vdim + CC - 1) / CC, P.H, num_seqs);
  constexpr int GT = MODE == kDecayPerHead ? 1 : KP;
  const bool vec = P.kdim % 4 == 0 && P.q_stride % 4 == 0 && P.k_stride % 4 == 0 && aligned16(P.q) && aligned16(P.k) &&
                   (MODE == kDecayPerHead || aligned16(P.g)) && P.vdim % VE == 0 && P.v_stride % VE == 0 && aligned16(P.v);
  if (vec) {
    const size_t smem = (size_t)2 * kDeltaTok * (2 * KP + GT + 1) * sizeof(float) + (size_t)2 * kDeltaTok * CC * sizeof(TV);
    static bool configured = false;                   // one flag per instantiation
    if (!configured && smem > 48 * 1024) {
      cudaFuncSetAttribute(delta_rule_kernel<TV, KPT, NS, NC, true, MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                           (int)smem);
      configured = true;
    }
    launch_pdl(delta_rule_kernel<TV, KPT, NS, NC, true, MODE>, grid, dim3(32 * NS), smem, stream, P);
  } else {
    const size_t smem = (size_t)kDeltaTok * (2 * KP + GT + 1 + CC) * sizeof(float);
    launch_pdl(delta_rule_kernel<TV, KPT, NS, NC, false, MODE>, grid, dim3(32 * NS), smem, stream, P);
  }
}

template <typename TV, int MODE>
static int delta_launch(const DeltaParams& P, int num_seqs, cudaStream_t stream) {
  // measured on 16 x 1024-token prompts, us at 8 heads of 128 / 32 heads of 64 (rows x columns per thread): delta rule with
  // a decay per head 64x1 601 / 566, 32x1 871 / 742, 32x2 523 / 480, 16x4 589 / 1035; wkv 64x1 564 / 501, 32x2 589 / 521,
  // 16x4 406 / 755. Decode steps of 256 rows: 32x2 72 / 67, 16x4 120 / 81.
  if (P.kdim <= 16) delta_launch_as<TV, 16, 1, 1, MODE>(P, num_seqs, stream);
  else if (P.kdim <= 32) delta_launch_as<TV, 32, 1, 1, MODE>(P, num_seqs, stream);
  else if (P.kdim <= 64) delta_launch_as<TV, 32, 2, 2, MODE>(P, num_seqs, stream);
  else if (P.kdim <= 128) {
    if (MODE == kWkv && P.cu_q != nullptr) delta_launch_as<TV, 16, 8, 4, MODE>(P, num_seqs, stream);
    else delta_launch_as<TV, 32, 4, 2, MODE>(P, num_seqs, stream);
  } else delta_launch_as<TV, 32, 8, 2, MODE>(P, num_seqs, stream);
  return finish_launch();
}

}  // namespace b200

using namespace b200;

extern "C" int b200_delta_rule(float* out, const float* q, int64_t q_stride, const float* k, int64_t k_stride,
                               const void* v, int64_t v_stride, const float* g, const float* beta, float* state,
                               const int32_t* state_slots, const int32_t* cu_q, const int32_t* cu_k,
                               const int32_t* ctx_lens, int32_t num_seqs, int32_t num_heads, int32_t groups,
                               int32_t kdim, int32_t vdim, int32_t mode, int32_t dtype, b200_stream_t stream) {
  B200_RETURN_IF(num_seqs < 0 || num_heads <= 0 || groups <= 0 || num_heads % groups != 0 || kdim <= 0 || vdim <= 0 ||
                     mode < kDecayPerChannel || mode > kWkv,
                 B200_ERR_BAD_SHAPE);
  B200_RETURN_IF(kdim > 256, B200_ERR_UNSUPPORTED);
  if (num_seqs == 0) return B200_OK;
  B200_RETURN_IF(!out || !q || !k || !v || !g || !beta || (cu_q == nullptr) == (ctx_lens == nullptr) ||
                     (cu_q && !cu_k) || (state && !state_slots), B200_ERR_NULL_POINTER);
  DeltaParams P;
  P.q = q, P.k = k, P.g = g, P.beta = beta, P.v = v, P.q_stride = q_stride, P.k_stride = k_stride;
  P.v_stride = v_stride, P.out = out, P.state = state, P.state_slots = state_slots, P.cu_q = cu_q, P.cu_k = cu_k;
  P.ctx_lens = ctx_lens, P.H = num_heads, P.groups = groups, P.kdim = kdim, P.vdim = vdim;
  B200_DISPATCH_3(dtype, TV, {
    if (mode == kDecayPerHead) return delta_launch<TV, kDecayPerHead>(P, num_seqs, (cudaStream_t)stream);
    if (mode == kWkv) return delta_launch<TV, kWkv>(P, num_seqs, (cudaStream_t)stream);
    return delta_launch<TV, kDecayPerChannel>(P, num_seqs, (cudaStream_t)stream);
  });
  return B200_OK;
}
