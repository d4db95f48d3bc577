// Attention whose values turn with their positions, and the row kernels around it.
//
// A value of position j is rotated by j over all its elements (pair m by j * f_m) before it is cached; a head's output at
// position i, a weighted sum of such values, is turned back by i, so that what reaches it from position j is turned by
// j - i alone.  Queries and keys rotate over their first `rot_dims` elements as usual.
//
//   qkv_conv_rotate   per token, from float32 projection rows [q | k | v]: a causal convolution over time of every
//                     channel (optional; inputs before the step's first token come from the sequence's carried inputs),
//                     the rotation of q and k, the rotation of v (optional), q to its buffer, k and v into the cache
//                     pages.  A thread owns eight columns (four pairs) and walks over a few consecutive tokens of one
//                     sequence with the convolution's last inputs in registers, so every input is read once; the block's
//                     sines and cosines are computed once per (token, pair) for all its heads.  In a step of single
//                     tokens the same launch also updates the carried inputs (nobody else reads or writes those columns).
//   conv_carry_rows   the carried inputs after a step of many tokens.
//   head_turn         per token and head: the output turned back by the token's position, times sigmoid(gate) element by
//                     element, rounded once.
//
// Pairs are (m, m + n / 2) of the n rotated elements, or (2m, 2m + 1) when `interleaved`.
#include "common.cuh"

namespace cpi {

constexpr int QR_THREADS = 128, QR_MAX_TB = 32, QR_MAX_PAIRS = 128, QR_BLOCKS_PER_SM = 4;

struct ConvRotParams {
  const float* qkv; long stride;                   // [T, >= C], C = NH D + NKV D + NKV DV
  const float* conv_wt; int taps;                  // [taps, C] or null
  float* carry; int write_carry;                   // [slots, taps - 1, C]
  const float* inv_freq; int rot_dims;             // [rot_dims / 2] or null
  const float* v_inv_freq;                         // [DV / 2] or null
  int interleaved; float amplitude;
  void* q_out; void* k_cache; void* v_cache;
  const int* page_table; int max_blocks; int page_size;
  const int* token_seq; const int* token_pos; const int* seq_slot; const int* seq_start;
  const int* tile_tok0; const int* tile_rows; int subs;      // null: a tile is one token
  int tb;                                          // tokens of a block
  int n_heads, n_kv_heads, head_dim, v_dim;
};

template <typename TO> __device__ __forceinline__ void store4(TO* p, const float (&v)[8], int at);
template <> __device__ __forceinline__ void store4<float>(float* p, const float (&v)[8], int at) {
  *reinterpret_cast<float4*>(p) = make_float4(v[at], v[at + 1], v[at + 2], v[at + 3]);
}
template <> __device__ __forceinline__ void store4<__nv_bfloat16>(__nv_bfloat16* p, const float (&v)[8], int at) {
  __nv_bfloat162 a = __floats2bfloat162_rn(v[at], v[at + 1]), b = __floats2bfloat162_rn(v[at + 2], v[at + 3]);
  uint2 pk;
  pk.x = *reinterpret_cast<uint32_t*>(&a);
  pk.y = *reinterpret_cast<uint32_t*>(&b);
  *reinterpret_cast<uint2*>(p) = pk;
}

// Turns the four pairs that a thread holds: elements 0..3 with 4..7 (halves), or (0,1) (2,3) ... (interleaved).
__device__ __forceinline__ void turn_pair(float& x, float& y, float c, float s) {
  const float u = x;
  x = u * c - y * s;
  y = y * c + u * s;
}
__device__ __forceinline__ void turn4(float (&v)[8], const float* cs, const float* sn, int interleaved, float sign) {
  if (interleaved) {
#pragma unroll
    for (int i = 0; i < 4; ++i) turn_pair(v[2 * i], v[2 * i + 1], cs[i], sign * sn[i]);
  } else {
#pragma unroll
    for (int i = 0; i < 4; ++i) turn_pair(v[i], v[i + 4], cs[i], sign * sn[i]);
  }
}

// the eight columns of group g within a head of `dim` elements of which the first `rot` turn: two runs of four
__device__ __forceinline__ void group_columns(int g, int rot, int interleaved, int& lo, int& hi, int& pair) {
  const int turning = rot >> 3;
  if (g < turning) {
    pair = 4 * g;
    lo = interleaved ? 8 * g : 4 * g;
    hi = interleaved ? 8 * g + 4 : (rot >> 1) + 4 * g;
  } else {
    pair = -1;
    lo = 8 * g;
    hi = lo + 4;
  }
}

template <typename TO, int TAPS>
__global__ void __launch_bounds__(QR_THREADS, TAPS > 4 ? 2 : QR_BLOCKS_PER_SM) qkv_conv_rotate_kernel(ConvRotParams p) {
  pdl_launch_dependents();
  extern __shared__ float table_s[];               // [tb][pairs] cosines then sines: of q and k, then of v
  __shared__ size_t kv_row_s[QR_MAX_TB];
  const int tid = threadIdx.x, TB = p.tb;
  int tok0, ntok;
  if (p.tile_tok0) {
    const int tile = blockIdx.x / p.subs, off = (blockIdx.x % p.subs) * TB, rows = p.tile_rows[tile];
    if (off >= rows) return;
    tok0 = p.tile_tok0[tile] + off;
    ntok = min(TB, rows - off);
  } else {
    tok0 = blockIdx.x;
    ntok = 1;
  }
  const int D = p.head_dim, DV = p.v_dim;
  const int nq = p.n_heads * D, nk = p.n_kv_heads * D, nv = p.n_kv_heads * DV, C = nq + nk + nv;
  const int rp = p.inv_freq ? p.rot_dims >> 1 : 0, vp = p.v_inv_freq ? DV >> 1 : 0;
  const int c0 = blockIdx.y * QR_THREADS * 8, c1 = min(C, c0 + QR_THREADS * 8);      // the block's columns, as groups of 8
  float* qk_t = table_s;
  float* v_t = table_s + 2 * TB * rp;
  const int seq = p.token_seq[tok0], slot = p.seq_slot[seq];
  // positions and tables are on the device before the step's first kernel: nothing here waits for the projection
  if (c0 < nq + nk)
    for (int i = tid; i < ntok * rp; i += QR_THREADS) {
      const int t = i / rp, m = i % rp;
      float s, c;
      sincosf((float)p.token_pos[tok0 + t] * p.inv_freq[m], &s, &c);
      qk_t[t * rp + m] = c * p.amplitude;
      qk_t[(TB + t) * rp + m] = s * p.amplitude;
    }
  if (c1 > nq + nk)
    for (int i = tid; i < ntok * vp; i += QR_THREADS) {
      const int t = i / vp, m = i % vp;
      float s, c;
      sincosf((float)p.token_pos[tok0 + t] * p.v_inv_freq[m], &s, &c);
      v_t[t * vp + m] = c;
      v_t[(TB + t) * vp + m] = s;
    }
  if (tid < ntok) {
    const int pos = p.token_pos[tok0 + tid];
    const int page = p.page_table[(size_t)slot * p.max_blocks + pos / p.page_size];
    kv_row_s[tid] = (size_t)page * p.n_kv_heads * p.page_size + pos % p.page_size;
  }
  __syncthreads();
  const int col = c0 + tid * 8;
  const bool live = col < C;
  const bool is_q = col < nq, is_v = col >= nq + nk;
  const int dim = is_v ? DV : D, base = is_q ? 0 : is_v ? nq + nk : nq;
  const int head = (col - base) / dim, g = ((col - base) % dim) >> 3;
  int lo, hi, pair;
  group_columns(g, is_v ? 2 * vp : 2 * rp, p.interleaved, lo, hi, pair);
  const int colA = base + head * dim + lo, colB = base + head * dim + hi;
  const float* tab = is_v ? v_t : qk_t;
  const int np = is_v ? vp : rp;
  float w[TAPS][8];
  if (TAPS > 1 && live) {
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      const int jj = j - (TAPS - p.taps);          // fewer taps than registers: the oldest weights are zero
      float4 a = make_float4(0.f, 0.f, 0.f, 0.f), b = a;
      if (jj >= 0) {
        a = *reinterpret_cast<const float4*>(p.conv_wt + (size_t)jj * C + colA);
        b = *reinterpret_cast<const float4*>(p.conv_wt + (size_t)jj * C + colB);
      }
      w[j][0] = a.x; w[j][1] = a.y; w[j][2] = a.z; w[j][3] = a.w;
      w[j][4] = b.x; w[j][5] = b.y; w[j][6] = b.z; w[j][7] = b.w;
    }
  }
  pdl_wait();
  if (!live) return;
  // hist[j]: the input TAPS - 1 - j tokens before the current one
  float hist[TAPS > 1 ? TAPS - 1 : 1][8];
  float* carry = p.carry + (size_t)slot * (p.taps - 1) * C;
  if (TAPS > 1) {
    const int local = p.token_pos[tok0] - p.seq_start[seq];      // tokens of the sequence before tok0 in this step
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) {
      const int back = TAPS - 1 - j;
      float4 a = make_float4(0.f, 0.f, 0.f, 0.f), b = a;
      if (back <= p.taps - 1) {
        const float* src = back <= local ? p.qkv + (size_t)(tok0 - back) * p.stride
                                         : carry + (size_t)(p.taps - 1 - (back - local)) * C;
        a = *reinterpret_cast<const float4*>(src + colA);
        b = *reinterpret_cast<const float4*>(src + colB);
      }
      hist[j][0] = a.x; hist[j][1] = a.y; hist[j][2] = a.z; hist[j][3] = a.w;
      hist[j][4] = b.x; hist[j][5] = b.y; hist[j][6] = b.z; hist[j][7] = b.w;
    }
  }
  // the columns of the next two tokens are asked for before a token's work
  const float* src = p.qkv + (size_t)tok0 * p.stride;
  float4 na[2], nb[2];
#pragma unroll
  for (int u = 0; u < 2; ++u) {
    const float* at = src + (size_t)min(u, ntok - 1) * p.stride;
    na[u] = *reinterpret_cast<const float4*>(at + colA);
    nb[u] = *reinterpret_cast<const float4*>(at + colB);
  }
#pragma unroll 1
  for (int t = 0; t < ntok; ++t) {
    const float in[8] = {na[0].x, na[0].y, na[0].z, na[0].w, nb[0].x, nb[0].y, nb[0].z, nb[0].w};
    na[0] = na[1]; nb[0] = nb[1];
    if (t + 2 < ntok) {
      const float* at = src + (size_t)(t + 2) * p.stride;
      na[1] = *reinterpret_cast<const float4*>(at + colA);
      nb[1] = *reinterpret_cast<const float4*>(at + colB);
    }
    float v[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      if (TAPS > 1) {
        float acc = 0.f;
#pragma unroll
        for (int j = 0; j < TAPS - 1; ++j) acc = fmaf(w[j][i], hist[j][i], acc);
        v[i] = fmaf(w[TAPS - 1][i], in[i], acc);
      } else {
        v[i] = in[i];
      }
    }
    if (TAPS > 1) {
#pragma unroll
      for (int j = 0; j + 1 < TAPS - 1; ++j)
#pragma unroll
        for (int i = 0; i < 8; ++i) hist[j][i] = hist[j + 1][i];
#pragma unroll
      for (int i = 0; i < 8; ++i) hist[TAPS > 1 ? TAPS - 2 : 0][i] = in[i];
    }
    if (pair >= 0) turn4(v, tab + t * np + pair, tab + (TB + t) * np + pair, p.interleaved, 1.0f);
    TO* dst;
    if (is_q) dst = reinterpret_cast<TO*>(p.q_out) + ((size_t)(tok0 + t) * p.n_heads + head) * D;
    else dst = reinterpret_cast<TO*>(is_v ? p.v_cache : p.k_cache) + (kv_row_s[t] + (size_t)head * p.page_size) * dim;
    store4<TO>(dst + lo, v, 0);
    store4<TO>(dst + hi, v, 4);
  }
  if (TAPS > 1 && p.write_carry) {
#pragma unroll
    for (int j = 0; j < TAPS - 1; ++j) {
      const int jj = j - (TAPS - p.taps);
      if (jj >= 0) {
        store4<float>(carry + (size_t)jj * C + colA, hist[j], 0);
        store4<float>(carry + (size_t)jj * C + colB, hist[j], 4);
      }
    }
  }
}

// carry[slot] <- the last taps - 1 inputs of every sequence after this step
__global__ void __launch_bounds__(256) conv_carry_rows_kernel(const float* in, long stride, float* carry, int channels,
                                                              int taps, const int* seq_slot, const int* seq_tok0,
                                                              const int* seq_new) {
  pdl_launch_dependents();
  pdl_wait();
  const int s = blockIdx.x, c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= channels) return;
  const int n = seq_new[s], tok0 = seq_tok0[s], keep = taps - 1;
  float* dst = carry + (size_t)seq_slot[s] * keep * channels + c;
  for (int j = 0; j < keep; ++j) {                 // ascending: an older carried input is read before its place is written
    const int idx = n - keep + j;
    dst[(size_t)j * channels] = idx >= 0 ? in[(size_t)(tok0 + idx) * stride + c] : dst[(size_t)(j + n) * channels];
  }
}

struct HeadTurnParams {
  const void* in; void* out;                       // [T, NH DV]
  const float* gate; long gate_stride;             // [T, >= NH DV] or null
  const float* inv_freq; int interleaved;          // [DV / 2] or null
  const int* token_pos;
  int n_tokens, n_heads, v_dim, tokens_per_block;
};

__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }

__device__ __forceinline__ void load4(const float* p, float (&v)[8], int at) {
  const float4 a = *reinterpret_cast<const float4*>(p);
  v[at] = a.x; v[at + 1] = a.y; v[at + 2] = a.z; v[at + 3] = a.w;
}
__device__ __forceinline__ void load4(const __nv_bfloat16* p, float (&v)[8], int at) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
  v[at] = a.x; v[at + 1] = a.y; v[at + 2] = b.x; v[at + 3] = b.y;
}

template <typename T>
__global__ void __launch_bounds__(QR_THREADS) head_turn_kernel(HeadTurnParams p) {
  pdl_launch_dependents();
  extern __shared__ float table_s[];               // [tokens][pairs] cosines, then sines
  const int tid = threadIdx.x, DV = p.v_dim, vp = p.inv_freq ? DV >> 1 : 0, W = p.n_heads * DV;
  const int t0 = blockIdx.x * p.tokens_per_block, nt = min(p.tokens_per_block, p.n_tokens - t0);
  float* sn_t = table_s + p.tokens_per_block * vp;
  for (int i = tid; i < nt * vp; i += QR_THREADS) {
    float s, c;
    sincosf((float)p.token_pos[t0 + i / vp] * p.inv_freq[i % vp], &s, &c);
    table_s[i] = c;
    sn_t[i] = s;
  }
  __syncthreads();
  pdl_wait();
  const int col = (blockIdx.y * QR_THREADS + tid) * 8;
  if (col >= W) return;
  const int head = col / DV, g = (col % DV) >> 3;
  int lo, hi, pair;
  group_columns(g, 2 * vp, p.interleaved, lo, hi, pair);
  const int a = head * DV + lo, b = head * DV + hi;
#pragma unroll 2
  for (int t = 0; t < nt; ++t) {
    const T* src = reinterpret_cast<const T*>(p.in) + (size_t)(t0 + t) * W;
    float v[8], z[8];
    load4(src + a, v, 0); load4(src + b, v, 4);
    if (p.gate) {
      const float* gr = p.gate + (size_t)(t0 + t) * p.gate_stride;
      load4(gr + a, z, 0); load4(gr + b, z, 4);
    }
    if (pair >= 0) turn4(v, table_s + t * vp + pair, sn_t + t * vp + pair, p.interleaved, -1.0f);
    if (p.gate) {
#pragma unroll
      for (int i = 0; i < 8; ++i) v[i] *= sigmoid_f(z[i]);
    }
    T* dst = reinterpret_cast<T*>(p.out) + (size_t)(t0 + t) * W;
    store4<T>(dst + a, v, 0);
    store4<T>(dst + b, v, 4);
  }
}

// the same for heads of any even size: a thread per pair of one (token, head)
template <typename T>
__global__ void __launch_bounds__(QR_THREADS) head_turn_any_kernel(HeadTurnParams p) {
  pdl_launch_dependents();
  pdl_wait();
  const int DV = p.v_dim, W = p.n_heads * DV, t = blockIdx.x;
  const float pos = (float)p.token_pos[t];
  const T* src = reinterpret_cast<const T*>(p.in) + (size_t)t * W;
  T* dst = reinterpret_cast<T*>(p.out) + (size_t)t * W;
  auto put = [&](int i, float v) {
    dst[i] = from_f32<T>(p.gate ? v * sigmoid_f(p.gate[(size_t)t * p.gate_stride + i]) : v);
  };
  if (!p.inv_freq) {
    for (int i = threadIdx.x; i < W; i += blockDim.x) put(i, to_f32(src[i]));
    return;
  }
  const int half = DV >> 1;
  for (int u = threadIdx.x; u < p.n_heads * half; u += blockDim.x) {
    const int head = u / half, m = u % half;
    const int a = head * DV + (p.interleaved ? 2 * m : m), b = head * DV + (p.interleaved ? 2 * m + 1 : m + half);
    float s, c;
    sincosf(pos * p.inv_freq[m], &s, &c);
    const float x = to_f32(src[a]), y = to_f32(src[b]);
    put(a, x * c + y * s);
    put(b, y * c - x * s);
  }
}

}  // namespace cpi

using namespace cpi;

extern "C" int cpi_qkv_conv_rotate_supported(int head_dim, int v_dim, int rot_dims, int v_turns, int taps) {
  return head_dim % 8 == 0 && v_dim % 8 == 0 && rot_dims % 8 == 0 && rot_dims <= head_dim && rot_dims / 2 <= QR_MAX_PAIRS &&
         (!v_turns || v_dim / 2 <= QR_MAX_PAIRS) && taps >= 1 && taps <= 8;
}

// qkv float32 [T, stride]; conv_wt float32 [taps, C] (null: no convolution, taps 1); carry float32 [slots, taps - 1, C].
// tile_tok0 / tile_rows: runs of at most max_tile_rows consecutive tokens of one sequence; null: every token is the only
// one of its sequence in this step, and the carried inputs are updated too.
extern "C" int cpi_qkv_conv_rotate(const float* qkv, long stride, const float* conv_wt, int taps, float* carry,
                                   const float* inv_freq, int rot_dims, const float* v_inv_freq, int interleaved,
                                   float amplitude, void* q_out, void* k_cache, void* v_cache, int out_dtype,
                                   const int* page_table, int max_blocks, int page_size, const int* token_seq,
                                   const int* token_pos, const int* seq_slot, const int* seq_start, const int* tile_tok0,
                                   const int* tile_rows, int n_tiles, int max_tile_rows, int n_tokens, int n_heads,
                                   int n_kv_heads, int head_dim, int v_dim, cudaStream_t stream) {
  if (n_tokens == 0) return 0;
  CPI_REQUIRE(cpi_qkv_conv_rotate_supported(head_dim, v_dim, inv_freq ? rot_dims : 0, v_inv_freq != nullptr, conv_wt ? taps : 1),
              "qkv_conv_rotate: heads of %d / %d with %d rotated elements and %d taps are not supported", head_dim, v_dim,
              rot_dims, taps);
  CPI_REQUIRE(n_heads > 0 && n_kv_heads > 0 && page_size > 0, "qkv_conv_rotate: bad sizes heads=%d kv=%d page=%d", n_heads,
              n_kv_heads, page_size);
  auto ok16 = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  CPI_REQUIRE(stride % 4 == 0 && ok16(qkv) && ok16(conv_wt) && ok16(carry) && ok16(q_out) && ok16(k_cache) && ok16(v_cache),
              "qkv_conv_rotate: rows must start on 16 bytes");
  CPI_REQUIRE(conv_wt == nullptr || taps == 1 || carry != nullptr, "qkv_conv_rotate: a convolution needs the carried inputs");
  if (!conv_wt) taps = 1;
  const long C = (long)n_heads * head_dim + (long)n_kv_heads * (head_dim + v_dim);
  ConvRotParams p{qkv, stride, conv_wt, taps, carry, tile_tok0 == nullptr, inv_freq, inv_freq ? rot_dims : 0, v_inv_freq,
                  interleaved, amplitude, q_out, k_cache, v_cache, page_table, max_blocks, page_size, token_seq, token_pos,
                  seq_slot, seq_start, tile_tok0, tile_rows, 1, 1, n_heads, n_kv_heads, head_dim, v_dim};
  const int by = (int)((C / 8 + QR_THREADS - 1) / QR_THREADS);
  if (tile_tok0) {
    // tokens of a block: what makes the fewest (waves of blocks) x (tokens, and the inputs before the first one)
    const long slots = (long)sm_count() * QR_BLOCKS_PER_SM;
    long best = -1;
    const long pairs = (inv_freq ? rot_dims / 2 : 0) + (v_inv_freq ? v_dim / 2 : 0);
    for (int tb = 4; tb <= QR_MAX_TB && 2 * tb * pairs * (long)sizeof(float) <= 48 * 1024; ++tb) {      // (four always fit)
      const long blocks = (long)n_tiles * ((max_tile_rows + tb - 1) / tb) * by;
      const long cost = ((blocks + slots - 1) / slots) * (tb + taps + 1);
      if (best < 0 || cost < best) { best = cost; p.tb = tb; }
    }
    p.subs = (max_tile_rows + p.tb - 1) / p.tb;
  }
  const dim3 grid(tile_tok0 ? n_tiles * p.subs : n_tokens, by);
  const size_t smem = 2 * p.tb * ((inv_freq ? rot_dims / 2 : 0) + (v_inv_freq ? v_dim / 2 : 0)) * sizeof(float);
#define CPI_QR(TO, TAPS) cpi::launch_pdl(qkv_conv_rotate_kernel<TO, TAPS>, grid, dim3(QR_THREADS), smem, stream, p)
  // one tap is a product with one weight: it runs as a convolution of four taps with three zeros
  CPI_DISPATCH_DTYPE(out_dtype, TO, {
    if (!conv_wt) CPI_QR(TO, 1);
    else if (taps <= 4) CPI_QR(TO, 4);
    else CPI_QR(TO, 8);
  });
#undef CPI_QR
  return check_launch("qkv_conv_rotate");
}

extern "C" int cpi_conv_carry_rows(const float* in, long stride, float* carry, int channels, int taps,
                                   const int* seq_slot, const int* seq_tok0, const int* seq_new, int n_seqs,
                                   cudaStream_t stream) {
  if (n_seqs == 0 || taps <= 1) return 0;
  cpi::launch_pdl(conv_carry_rows_kernel, dim3(n_seqs, (channels + 255) / 256), dim3(256), 0, stream, in, stride, carry,
                  channels, taps, seq_slot, seq_tok0, seq_new);
  return check_launch("conv_carry_rows");
}

extern "C" int cpi_head_turn(const void* in, void* out, int dtype, const float* gate, long gate_stride,
                             const float* inv_freq, int interleaved, const int* token_pos, int n_tokens, int n_heads,
                             int v_dim, cudaStream_t stream) {
  if (n_tokens == 0) return 0;
  CPI_REQUIRE(n_heads > 0 && v_dim > 0 && (!inv_freq || v_dim % 2 == 0), "head_turn: %d heads of %d values", n_heads, v_dim);
  HeadTurnParams p{in, out, gate, gate_stride, inv_freq, interleaved, token_pos, n_tokens, n_heads, v_dim, 1};
  auto ok16 = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  const bool vec = v_dim % 8 == 0 && (!inv_freq || v_dim / 2 <= QR_MAX_PAIRS) && ok16(in) && ok16(out) && ok16(gate) &&
                   gate_stride % 4 == 0;
  if (vec) {
    const int groups = n_heads * v_dim / 8, by = (groups + QR_THREADS - 1) / QR_THREADS;
    while (p.tokens_per_block < 8 && (long)(n_tokens / (2 * p.tokens_per_block)) * by >= 8 * sm_count()) p.tokens_per_block *= 2;
    const dim3 grid((n_tokens + p.tokens_per_block - 1) / p.tokens_per_block, by);
    const size_t smem = 2 * p.tokens_per_block * (inv_freq ? v_dim / 2 : 0) * sizeof(float);
    CPI_DISPATCH_DTYPE(dtype, T, cpi::launch_pdl(head_turn_kernel<T>, grid, dim3(QR_THREADS), smem, stream, p));
  } else {
    CPI_DISPATCH_DTYPE(dtype, T, cpi::launch_pdl(head_turn_any_kernel<T>, dim3(n_tokens), dim3(QR_THREADS), 0, stream, p));
  }
  return check_launch("head_turn");
}
