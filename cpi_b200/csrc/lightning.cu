// Linear attention with one constant decay per head, a prompt's tokens in chunks on the tensor cores.
//
// Per sequence and head, with a the decay, S the float32 state [N, Dv] and o_t = S_t^T q_t, S_t = a S_{t-1} + k_t v_t^T.
// Over a chunk of C = 64 tokens that starts from S this is, for the local tokens i and j,
//
//     o_i = a^(i+1) S^T q_i + sum_{j <= i} a^(i-j) (q_i . k_j) v_j
//     S  <- a^n S + sum_j k_j (a^(n-1-j) v_j)^T                        (n tokens in the chunk)
//
// that is four products per chunk instead of a chain of 64 rank-one updates.  q, k and v are bfloat16 (projections after
// their activation); everything derived from them is float32: the scores times their powers of the decay, the scaled
// values and the state enter a product as the sum of THREE bfloat16 terms each (8 + 8 + 8 bits of significand: a float32
// number exactly, up to the underflow of the last term), against an operand that is bfloat16 as it is, with float32
// accumulators.  So a product loses no more than a float32 one.
//
// A block owns one sequence, one head and 8 NV columns of the values, and walks over the chunks; its 4 warps split
//   scores          16 query rows a warp; the accumulators become the A operand of the next product in registers
//   outputs         the same 16 rows
//   state           N / 16 row tiles, dealt out to the warps, in registers from the first chunk to the last; its three
//                   terms go through shared memory as the B operand of the next chunk's outputs
// The next chunk's rows are fetched (cp.async, two buffers) while one is computed.  Rows past the sequence's tokens and
// columns past the sizes are zeros.
#include "mma_frag.cuh"

namespace cpi {
namespace lightning {

using namespace frag;

constexpr int C = 64, WARPS = 4, THREADS = 32 * WARPS, TERMS = 3;

struct Params {
  const __nv_bfloat16* qkv; long stride;     // [T, >= H (2 N + Dv)]: q | k | v
  const float* decay;                        // [H]
  float* state;                              // [slots, H, N, Dv]
  float* out; long out_stride;               // [T, H Dv]
  const int* seq_slot; const int* seq_tok0; const int* seq_new;
  int n_heads, n_rows, n_cols;
};

// x as the sum of three bfloat16 numbers
__device__ __forceinline__ void split(float x, float (&t)[TERMS]) {
#pragma unroll
  for (int i = 0; i < TERMS; ++i) {
    t[i] = __bfloat162float(__float2bfloat16_rn(x));
    x -= t[i];
  }
}

// KN: 16-row tiles of the state (its rows padded to 16 KN); NV: 8-column tiles of the block's values
template <int KN, int NV>
struct Shape {
  static constexpr int NP = 16 * KN, LDN = NP + 8, DVS = 8 * NV, LDV = DVS + 8, MT = (KN + WARPS - 1) / WARPS;
  static constexpr size_t bytes = (2 * 2 * C * LDN + 2 * C * LDV + TERMS * C * LDV + TERMS * NP * LDV) * sizeof(__nv_bfloat16) +
                                  (C + 1) * sizeof(float);
};

template <int KN, int NV>
__global__ void __launch_bounds__(THREADS) lightning_chunk_kernel(Params p) {
  using Sh = Shape<KN, NV>;
  constexpr int NP = Sh::NP, LDN = Sh::LDN, DVS = Sh::DVS, LDV = Sh::LDV, MT = Sh::MT;
  extern __shared__ __align__(16) unsigned char smem_raw[];
  __nv_bfloat16* qk_s = reinterpret_cast<__nv_bfloat16*>(smem_raw);       // [buffer][q, k][C][LDN]
  __nv_bfloat16* v_s = qk_s + 2 * 2 * C * LDN;                            // [buffer][C][LDV]
  __nv_bfloat16* vt_s = v_s + 2 * C * LDV;                                // [term][C][LDV] scaled values
  __nv_bfloat16* st_s = vt_s + TERMS * C * LDV;                           // [term][NP][LDV] the state
  float* pw = reinterpret_cast<float*>(st_s + TERMS * NP * LDV);          // [C + 1] powers of the decay
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, lr = lane >> 2, lc = 2 * (lane & 3);
  const int s = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * DVS;
  const int N = p.n_rows, Dv = p.n_cols, H = p.n_heads;
  // (no early launch of the kernel behind it: a prompt's few blocks run long and would share their multiprocessors)
  if (tid <= C) pw[tid] = tid == 0 ? 1.0f : powf(p.decay[h], (float)tid);
  pdl_wait();
  const int n_tok = p.seq_new[s], tok0 = p.seq_tok0[s];

  auto load = [&](int c0, int buf) {
    const __nv_bfloat16* q0 = p.qkv + (size_t)h * N;
    const __nv_bfloat16* v0 = p.qkv + (size_t)2 * H * N + (size_t)h * Dv + col0;
    for (int e = tid; e < 2 * C * (NP / 8); e += THREADS) {
      const int piece = e % (NP / 8), row = e / (NP / 8), which = row / C, j = row % C;
      const bool live = c0 + j < n_tok && 8 * piece < N;
      const __nv_bfloat16* src = live ? q0 + (size_t)(tok0 + c0 + j) * p.stride + (size_t)which * H * N + 8 * piece : p.qkv;
      cp_async16_or_zero(qk_s + ((size_t)(buf * 2 + which) * C + j) * LDN + 8 * piece, src, live);
    }
    for (int e = tid; e < C * NV; e += THREADS) {
      const int piece = e % NV, j = e / NV;
      const bool live = c0 + j < n_tok && col0 + 8 * piece < Dv;
      const __nv_bfloat16* src = live ? v0 + (size_t)(tok0 + c0 + j) * p.stride + 8 * piece : p.qkv;
      cp_async16_or_zero(v_s + ((size_t)buf * C + j) * LDV + 8 * piece, src, live);
    }
    cp_async_commit();
  };

  if (n_tok <= 0) return;
  load(0, 0);
  // this warp's rows of the state: tile warp + WARPS m, rows lr and lr + 8, columns 8 t + lc and + 1
  float* st = p.state + ((size_t)p.seq_slot[s] * H + h) * N * Dv + col0;
  float S[MT][NV][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int t = 0; t < NV; ++t)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int r = 16 * (warp + WARPS * m) + lr + 8 * (i >> 1), c = 8 * t + lc + (i & 1);
        S[m][t][i] = r < N && col0 + c < Dv ? st[(size_t)r * Dv + c] : 0.f;
      }

  int buf = 0;
  for (int c0 = 0; c0 < n_tok; c0 += C, buf ^= 1) {
    const int n = min(C, n_tok - c0);
    cp_async_wait_all();
    __syncthreads();                       // the chunk's rows are here; everybody is done with the chunk before
    if (c0 + C < n_tok) load(c0 + C, buf ^ 1);
    const __nv_bfloat16* q_s = qk_s + (size_t)(buf * 2) * C * LDN;
    const __nv_bfloat16* k_s = q_s + (size_t)C * LDN;
    const __nv_bfloat16* vb_s = v_s + (size_t)buf * C * LDV;
    // the state and the scaled values as three terms
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      if (warp + WARPS * m >= KN) continue;
#pragma unroll
      for (int t = 0; t < NV; ++t)
#pragma unroll
        for (int i = 0; i < 4; i += 2) {
          const int r = 16 * (warp + WARPS * m) + lr + 4 * i;
          float a[TERMS], b[TERMS];
          split(S[m][t][i], a);
          split(S[m][t][i + 1], b);
#pragma unroll
          for (int k = 0; k < TERMS; ++k)
            *reinterpret_cast<uint32_t*>(st_s + ((size_t)k * NP + r) * LDV + 8 * t + lc) = pack_bf16(a[k], b[k]);
        }
    }
    for (int e = tid; e < C * DVS / 2; e += THREADS) {
      const int j = e / (DVS / 2), c = 2 * (e % (DVS / 2));
      const float w = pw[max(n - 1 - j, 0)];                  // (rows past the chunk's tokens hold zeros)
      const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(vb_s + (size_t)j * LDV + c));
      float a[TERMS], b[TERMS];
      split(v.x * w, a);
      split(v.y * w, b);
#pragma unroll
      for (int k = 0; k < TERMS; ++k)
        *reinterpret_cast<uint32_t*>(vt_s + ((size_t)k * C + j) * LDV + c) = pack_bf16(a[k], b[k]);
    }
    __syncthreads();

    // ---- rows 16 warp .. + 15: scores, and what the state answers
    const int i0 = 16 * warp, tiles = 2 * warp + 2;          // key tiles of 8 that these rows may see
    float A[C / 8][4], O1[NV][4], O2[NV][4];
#pragma unroll
    for (int t = 0; t < C / 8; ++t)
#pragma unroll
      for (int i = 0; i < 4; ++i) A[t][i] = 0.f;
#pragma unroll
    for (int t = 0; t < NV; ++t)
#pragma unroll
      for (int i = 0; i < 4; ++i) O1[t][i] = O2[t][i] = 0.f;
#pragma unroll
    for (int k = 0; k < KN; ++k) {
      uint32_t qf[4];
      ldsm_x4(qf, q_s + (size_t)(i0 + (lane & 15)) * LDN + 16 * k + 8 * (lane >> 4));
#pragma unroll
      for (int t = 0; t < C / 8; t += 2) {
        if (t >= tiles) continue;
        uint32_t kf[4];
        ldsm_x4(kf, k_s + (size_t)(8 * t + (lane & 7) + 8 * (lane >> 4)) * LDN + 16 * k + 8 * ((lane >> 3) & 1));
        mma_bf16(A[t], qf, kf[0], kf[1]);
        mma_bf16(A[t + 1], qf, kf[2], kf[3]);
      }
#pragma unroll
      for (int u = 0; u < TERMS; ++u)
#pragma unroll
        for (int t = 0; t < NV; t += 2) {
          uint32_t sf[4];
          ldsm_x4_trans(sf, st_s + ((size_t)u * NP + 16 * k + (lane & 15)) * LDV + 8 * t + 8 * (lane >> 4));
          mma_bf16(O2[t], qf, sf[0], sf[1]);
          mma_bf16(O2[t + 1], qf, sf[2], sf[3]);
        }
    }
    // ---- scores times powers of the decay, times the values
#pragma unroll
    for (int kk = 0; kk < C / 16; ++kk) {
      if (2 * kk >= tiles) continue;
      uint32_t af[TERMS][4];
#pragma unroll
      for (int x = 0; x < 4; ++x) {                          // a fragment's registers: (row, row + 8) of key tile 2 kk, then of 2 kk + 1
        const int t = 2 * kk + (x >> 1), half = x & 1, i = i0 + lr + 8 * half, j = 8 * t + lc;
        float a[TERMS], b[TERMS];
        split(j <= i ? A[t][2 * half] * pw[i - j] : 0.f, a);
        split(j + 1 <= i ? A[t][2 * half + 1] * pw[i - j - 1] : 0.f, b);
#pragma unroll
        for (int u = 0; u < TERMS; ++u) af[u][x] = pack_bf16(a[u], b[u]);
      }
#pragma unroll
      for (int t = 0; t < NV; t += 2) {
        uint32_t vf[4];
        ldsm_x4_trans(vf, vb_s + (size_t)(16 * kk + (lane & 15)) * LDV + 8 * t + 8 * (lane >> 4));
#pragma unroll
        for (int u = 0; u < TERMS; ++u) {
          mma_bf16(O1[t], af[u], vf[0], vf[1]);
          mma_bf16(O1[t + 1], af[u], vf[2], vf[3]);
        }
      }
    }
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int i = i0 + lr + 8 * half;
      if (i >= n) continue;
      const float w = pw[i + 1];
      float* o = p.out + (size_t)(tok0 + c0 + i) * p.out_stride + (size_t)h * Dv + col0;
#pragma unroll
      for (int t = 0; t < NV; ++t)
        if (col0 + 8 * t < Dv)                               // (the columns are a multiple of eight)
          *reinterpret_cast<float2*>(o + 8 * t + lc) = make_float2(fmaf(w, O2[t][2 * half], O1[t][2 * half]),
                                                                   fmaf(w, O2[t][2 * half + 1], O1[t][2 * half + 1]));
    }
    // ---- the state after the chunk
    const float whole = pw[n];
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      if (warp + WARPS * m >= KN) continue;
#pragma unroll
      for (int t = 0; t < NV; ++t)
#pragma unroll
        for (int i = 0; i < 4; ++i) S[m][t][i] *= whole;
    }
#pragma unroll
    for (int kk = 0; kk < C / 16; ++kk) {
      uint32_t kf[MT][4];
#pragma unroll
      for (int m = 0; m < MT; ++m)
        if (warp + WARPS * m < KN)
          ldsm_x4_trans(kf[m], k_s + (size_t)(16 * kk + (lane & 7) + 8 * (lane >> 4)) * LDN + 16 * (warp + WARPS * m) + 8 * ((lane >> 3) & 1));
#pragma unroll
      for (int u = 0; u < TERMS; ++u)
#pragma unroll
        for (int t = 0; t < NV; t += 2) {
          uint32_t vf[4];
          ldsm_x4_trans(vf, vt_s + ((size_t)u * C + 16 * kk + (lane & 15)) * LDV + 8 * t + 8 * (lane >> 4));
#pragma unroll
          for (int m = 0; m < MT; ++m)
            if (warp + WARPS * m < KN) {
              mma_bf16(S[m][t], kf[m], vf[0], vf[1]);
              mma_bf16(S[m][t + 1], kf[m], vf[2], vf[3]);
            }
        }
    }
  }
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int t = 0; t < NV; ++t)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int r = 16 * (warp + WARPS * m) + lr + 8 * (i >> 1), c = 8 * t + lc + (i & 1);
        if (r < N && col0 + c < Dv) st[(size_t)r * Dv + c] = S[m][t][i];
      }
}

template <int KN, int NV>
static int launch(const Params& p, int n_seqs, cudaStream_t stream) {
  using Sh = Shape<KN, NV>;
  static bool attr_set = false;
  if (!attr_set) {
    if (cudaFuncSetAttribute(lightning_chunk_kernel<KN, NV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)Sh::bytes) != cudaSuccess) {
      set_error("lightning_chunks: %zu bytes of shared memory were refused", Sh::bytes);
      return 1;
    }
    attr_set = true;
  }
  const dim3 grid(n_seqs, p.n_heads, (p.n_cols + Sh::DVS - 1) / Sh::DVS);
  cpi::launch_pdl(lightning_chunk_kernel<KN, NV>, grid, dim3(THREADS), Sh::bytes, stream, p);
  return check_launch("lightning_chunks");
}

template <int KN>
static int launch_nv(const Params& p, int n_seqs, cudaStream_t stream) {
  // blocks of 32 columns, or of 16 where 32 would leave multiprocessors idle
  if ((long)n_seqs * p.n_heads * ((p.n_cols + 31) / 32) >= sm_count() || p.n_cols > 16 * 65535) return launch<KN, 4>(p, n_seqs, stream);
  return launch<KN, 2>(p, n_seqs, stream);
}

}  // namespace lightning
}  // namespace cpi

using namespace cpi;

extern "C" int cpi_lightning_chunks_supported(int n_rows, int n_cols) {
  return n_rows >= 8 && n_rows % 8 == 0 && n_rows <= 128 && n_cols >= 8 && n_cols % 8 == 0;
}

extern "C" int cpi_lightning_chunks(const void* qkv, long stride, const float* decay, float* state, float* out,
                                    long out_stride, const int* seq_slot, const int* seq_tok0, const int* seq_new, int n_seqs,
                                    int n_heads, int n_rows, int n_cols, cudaStream_t stream) {
  if (n_seqs == 0) return 0;
  CPI_REQUIRE(cpi_lightning_chunks_supported(n_rows, n_cols), "lightning_chunks: heads of %d and %d elements are not supported "
              "(multiples of eight, keys up to 128)", n_rows, n_cols);
  CPI_REQUIRE(n_heads >= 1 && n_heads <= 65535, "lightning_chunks: %d heads", n_heads);
  CPI_REQUIRE((reinterpret_cast<uintptr_t>(qkv) & 15) == 0 && stride % 8 == 0 && (reinterpret_cast<uintptr_t>(out) & 7) == 0 &&
              out_stride % 2 == 0, "lightning_chunks: rows must start on 16 bytes (outputs on 8)");
  lightning::Params p{reinterpret_cast<const __nv_bfloat16*>(qkv), stride, decay, state, out, out_stride,
                      seq_slot, seq_tok0, seq_new, n_heads, n_rows, n_cols};
  if (n_rows <= 16) return lightning::launch_nv<1>(p, n_seqs, stream);
  if (n_rows <= 32) return lightning::launch_nv<2>(p, n_seqs, stream);
  if (n_rows <= 64) return lightning::launch_nv<4>(p, n_seqs, stream);
  return lightning::launch_nv<8>(p, n_seqs, stream);
}
