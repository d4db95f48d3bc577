// Boundaries between sublayers that are normed on both sides, one pass over a row each:
//
//   norm_step   the norms act element by element (tanh(alpha x) * w + b, no statistics of the row):
//               v = a sublayer's output for token t, given as
//                 - a float32 row y[t], or
//                 - the sum over the token's chosen experts, in the order of its choices: row_of_slot picks the expert's
//                   output row (already weighted), or, for an expert number >= n_real, weight * h_in[t] (an expert whose
//                   output is its input), or
//                 - nothing;
//               x[t] <- x[t] + post(v)   (or x[t] <- post(v) when `add` is off; post may be absent: the sum as it is)
//               h_out[r] = pre(x[rows ? rows[r] : r])   in the activation dtype, when `pre` is given: the next sublayer's
//               input
// so that the norm after a sublayer, the residual sum, the norm before the next sublayer and the combination of the
// experts' outputs are one pass over the row.  Everything is float32; a thread's elements depend on nothing but their own
// column, so a row's result does not depend on the launch.
//
//   rms_step    the same with RMS norms, post(v) = v / sqrt(mean(v^2) + eps) * (offset + w) and pre alike: a block owns a
//               row and keeps it on chip (registers, or shared memory for widths that registers do not take) from the
//               sublayer's output to the next sublayer's input.  The block's size follows from the width alone, so the
//               order of a row's sums does not depend on the other rows.
#include "common.cuh"

namespace cpi {

// a sublayer's output: a row per token, or the sum over a token's chosen experts
struct SublayerRows {
  const float* y; long y_stride;                   // [T, W] or null
  const float* ye; const int* row_of_slot; const int* slot_expert; const float* slot_weight;    // experts or null
  const void* h_in; int h_in_dtype; long h_in_stride;
  int top_k, n_real;
};

struct NormStepParams {
  SublayerRows src;
  float* x; long x_stride; int add;
  int has_post; float post_alpha; const float* post_w; const float* post_b;
  int has_pre; float pre_alpha; const float* pre_w; const float* pre_b;
  void* h_out; int h_out_dtype; long h_out_stride; const int* rows;
  int width;
};

template <int V> struct Vec { float v[V]; };

template <int V> __device__ __forceinline__ Vec<V> loadv(const float* p);
template <> __device__ __forceinline__ Vec<1> loadv<1>(const float* p) { return Vec<1>{{*p}}; }
template <> __device__ __forceinline__ Vec<4> loadv<4>(const float* p) {
  const float4 a = *reinterpret_cast<const float4*>(p);
  return Vec<4>{{a.x, a.y, a.z, a.w}};
}
template <int V> __device__ __forceinline__ Vec<V> loadv(const __nv_bfloat16* p);
template <> __device__ __forceinline__ Vec<1> loadv<1>(const __nv_bfloat16* p) { return Vec<1>{{__bfloat162float(*p)}}; }
template <> __device__ __forceinline__ Vec<4> loadv<4>(const __nv_bfloat16* p) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
  return Vec<4>{{a.x, a.y, b.x, b.y}};
}
template <int V> __device__ __forceinline__ Vec<V> loadv_any(const void* p, int dtype, size_t i) {
  return dtype == kF32 ? loadv<V>(reinterpret_cast<const float*>(p) + i) : loadv<V>(reinterpret_cast<const __nv_bfloat16*>(p) + i);
}

__device__ __forceinline__ void storev(float* p, const Vec<1>& r) { *p = r.v[0]; }
__device__ __forceinline__ void storev(float* p, const Vec<4>& r) {
  *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
}
__device__ __forceinline__ void storev(__nv_bfloat16* p, const Vec<1>& r) { *p = __float2bfloat16_rn(r.v[0]); }
__device__ __forceinline__ void storev(__nv_bfloat16* p, const Vec<4>& r) {
  __nv_bfloat162 a = __floats2bfloat162_rn(r.v[0], r.v[1]), b = __floats2bfloat162_rn(r.v[2], r.v[3]);
  uint2 pk;
  pk.x = *reinterpret_cast<uint32_t*>(&a);
  pk.y = *reinterpret_cast<uint32_t*>(&b);
  *reinterpret_cast<uint2*>(p) = pk;
}
template <int V> __device__ __forceinline__ void storev_any(void* p, int dtype, size_t i, const Vec<V>& r) {
  if (dtype == kF32) storev(reinterpret_cast<float*>(p) + i, r);
  else storev(reinterpret_cast<__nv_bfloat16*>(p) + i, r);
}

// V columns of token t's output, from column c
template <int V>
__device__ __forceinline__ Vec<V> sublayer_row(const SublayerRows& p, int t, int c, int width) {
  if (p.y) return loadv<V>(p.y + (size_t)t * p.y_stride + c);
  Vec<V> v;
#pragma unroll
  for (int i = 0; i < V; ++i) v.v[i] = 0.f;
  for (int k0 = 0; k0 < p.top_k; k0 += 4) {                    // four rows' loads in flight
    Vec<V> e[4];
    float f[4];
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      f[k] = 0.f;
      if (k0 + k < p.top_k) {
        const size_t s = (size_t)t * p.top_k + k0 + k;
        if (p.slot_expert[s] < p.n_real) {
          f[k] = 1.f;
          e[k] = loadv<V>(p.ye + (size_t)p.row_of_slot[s] * width + c);
        } else {
          f[k] = p.slot_weight[s];
          e[k] = loadv_any<V>(p.h_in, p.h_in_dtype, (size_t)t * p.h_in_stride + c);
        }
      }
    }
#pragma unroll
    for (int k = 0; k < 4; ++k)
      if (k0 + k < p.top_k) {
#pragma unroll
        for (int i = 0; i < V; ++i) v.v[i] = fmaf(f[k], e[k].v[i], v.v[i]);
      }
  }
  return v;
}

// V columns a thread (4: every row starts on 16 bytes and the width is a multiple of four)
template <int V>
__global__ void __launch_bounds__(256) norm_step_kernel(NormStepParams p) {
  pdl_launch_dependents();
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
  const bool live = c < p.width;
  // the norms' weights are no kernel's output: they are fetched before the wait on the kernel before this one
  Vec<V> pw, pb, qw, qb;
  if (live && p.has_post) { pw = loadv<V>(p.post_w + c); pb = loadv<V>(p.post_b + c); }
  if (live && p.has_pre) { qw = loadv<V>(p.pre_w + c); qb = loadv<V>(p.pre_b + c); }
  pdl_wait();
  if (!live) return;
  const int r = blockIdx.x, t = p.rows ? p.rows[r] : r;
  float* xp = p.x + (size_t)t * p.x_stride + c;
  Vec<V> x;
  const bool enters = p.src.y != nullptr || p.src.ye != nullptr;
  if (!enters || p.add) x = loadv<V>(xp);
  if (enters) {
    const Vec<V> v = sublayer_row<V>(p.src, t, c, p.width);
#pragma unroll
    for (int i = 0; i < V; ++i) {
      const float n = p.has_post ? fmaf(tanhf(p.post_alpha * v.v[i]), pw.v[i], pb.v[i]) : v.v[i];
      x.v[i] = p.add ? x.v[i] + n : n;
    }
    storev(xp, x);
  }
  if (p.has_pre) {
    Vec<V> h;
#pragma unroll
    for (int i = 0; i < V; ++i) h.v[i] = fmaf(tanhf(p.pre_alpha * x.v[i]), qw.v[i], qb.v[i]);
    storev_any<V>(p.h_out, p.h_out_dtype, (size_t)r * p.h_out_stride + c, h);
  }
}

// ---- RMS norms on both sides ------------------------------------------------------------------------------------
struct RmsStepParams {
  SublayerRows src;
  float* x; long x_stride; int add;
  const void* post_w; int post_dtype; float post_offset, post_eps;           // [W]
  const void* pre_w; int pre_dtype; float pre_offset, pre_eps;               // [W], with h_out
  void* h_out; int h_out_dtype; long h_out_stride;                           // null: no norm before a next sublayer
  int width;
};

constexpr int RMS_THREADS = 256;

// rows of up to PER * 1,024 columns in registers, four columns at a time
template <int PER>
__global__ void __launch_bounds__(RMS_THREADS) rms_step_kernel(RmsStepParams p) {
  pdl_launch_dependents();
  __shared__ float scratch[32];
  const int t = blockIdx.x, groups = p.width >> 2;
  Vec<4> pw[PER], qw[PER];                         // the norms' weights are no kernel's output: fetched before the wait
#pragma unroll
  for (int j = 0; j < PER; ++j) {
    const int g = threadIdx.x + j * RMS_THREADS;
    if (g < groups) {
      pw[j] = loadv_any<4>(p.post_w, p.post_dtype, 4 * (size_t)g);
      if (p.h_out) qw[j] = loadv_any<4>(p.pre_w, p.pre_dtype, 4 * (size_t)g);
    }
  }
  pdl_wait();
  float* xr = p.x + (size_t)t * p.x_stride;
  Vec<4> v[PER], x[PER];
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < PER; ++j) {
    const int g = threadIdx.x + j * RMS_THREADS;
    if (g >= groups) continue;
    if (p.add) x[j] = loadv<4>(xr + 4 * g);
    v[j] = sublayer_row<4>(p.src, t, 4 * g, p.width);
#pragma unroll
    for (int i = 0; i < 4; ++i) ss = fmaf(v[j].v[i], v[j].v[i], ss);
  }
  const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)p.width + p.post_eps);
  ss = 0.f;
#pragma unroll
  for (int j = 0; j < PER; ++j) {
    const int g = threadIdx.x + j * RMS_THREADS;
    if (g >= groups) continue;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float n = v[j].v[i] * inv * (p.post_offset + pw[j].v[i]);
      x[j].v[i] = p.add ? x[j].v[i] + n : n;
      ss = fmaf(x[j].v[i], x[j].v[i], ss);
    }
    storev(xr + 4 * g, x[j]);
  }
  if (!p.h_out) return;
  const float inv2 = 1.0f / sqrtf(block_sum(ss, scratch) / (float)p.width + p.pre_eps);
#pragma unroll
  for (int j = 0; j < PER; ++j) {
    const int g = threadIdx.x + j * RMS_THREADS;
    if (g >= groups) continue;
#pragma unroll
    for (int i = 0; i < 4; ++i) x[j].v[i] = x[j].v[i] * inv2 * (p.pre_offset + qw[j].v[i]);
    storev_any<4>(p.h_out, p.h_out_dtype, (size_t)t * p.h_out_stride + 4 * g, x[j]);
  }
}

// any width and alignment: the row in shared memory (a thread reads back only what it wrote)
__global__ void __launch_bounds__(RMS_THREADS) rms_step_any_kernel(RmsStepParams p) {
  pdl_launch_dependents();
  extern __shared__ float row_s[];
  __shared__ float scratch[32];
  pdl_wait();
  const int t = blockIdx.x;
  float* xr = p.x + (size_t)t * p.x_stride;
  float ss = 0.f;
  for (int c = threadIdx.x; c < p.width; c += RMS_THREADS) {
    const float v = sublayer_row<1>(p.src, t, c, p.width).v[0];
    row_s[c] = v;
    ss = fmaf(v, v, ss);
  }
  const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)p.width + p.post_eps);
  ss = 0.f;
  for (int c = threadIdx.x; c < p.width; c += RMS_THREADS) {
    const float n = row_s[c] * inv * (p.post_offset + load_any(p.post_w, p.post_dtype, c));
    const float x = p.add ? xr[c] + n : n;
    xr[c] = x;
    row_s[c] = x;
    ss = fmaf(x, x, ss);
  }
  if (!p.h_out) return;
  const float inv2 = 1.0f / sqrtf(block_sum(ss, scratch) / (float)p.width + p.pre_eps);
  for (int c = threadIdx.x; c < p.width; c += RMS_THREADS)
    storev_any<1>(p.h_out, p.h_out_dtype, (size_t)t * p.h_out_stride + c,
                  Vec<1>{{row_s[c] * inv2 * (p.pre_offset + load_any(p.pre_w, p.pre_dtype, c))}});
}

}  // namespace cpi

using namespace cpi;

extern "C" int cpi_norm_step(const float* y, long y_stride, const float* ye, const int* row_of_slot,
                             const int* slot_expert, const float* slot_weight, const void* h_in, int h_in_dtype,
                             long h_in_stride, int top_k, int n_real, float* x, long x_stride, int add, int has_post,
                             float post_alpha, const float* post_w, const float* post_b, int has_pre, float pre_alpha,
                             const float* pre_w, const float* pre_b, void* h_out, int h_out_dtype, long h_out_stride,
                             const int* rows, int n_rows, int width, cudaStream_t stream) {
  if (n_rows == 0) return 0;
  CPI_REQUIRE(width >= 1 && x != nullptr, "norm_step: a width of %d", width);
  CPI_REQUIRE(y == nullptr || ye == nullptr, "norm_step: one source, a row or a sum over experts");
  CPI_REQUIRE(ye == nullptr || (row_of_slot && slot_expert && slot_weight && h_in && top_k >= 1),
              "norm_step: a sum over experts needs the lists of the routing and the experts' input");
  CPI_REQUIRE(rows == nullptr || (y == nullptr && ye == nullptr), "norm_step: a row list goes with the norm alone");
  CPI_REQUIRE(!has_post || (post_w && post_b), "norm_step: the norm after a sublayer has a weight and an offset");
  CPI_REQUIRE(!has_pre || (pre_w && pre_b && h_out), "norm_step: the norm before a sublayer has a weight, an offset and an output");
  NormStepParams p{{y, y_stride, ye, row_of_slot, slot_expert, slot_weight, h_in, h_in_dtype, h_in_stride, top_k, n_real},
                   x, x_stride, add, has_post, post_alpha, post_w, post_b, has_pre, pre_alpha, pre_w, pre_b, h_out,
                   h_out_dtype, h_out_stride, rows, width};
  auto ok16 = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  const bool vec = width % 4 == 0 && x_stride % 4 == 0 && y_stride % 4 == 0 && h_in_stride % 4 == 0 && h_out_stride % 4 == 0 &&
                   ok16(x) && ok16(y) && ok16(ye) && ok16(h_in) && ok16(h_out) && ok16(post_w) && ok16(post_b) && ok16(pre_w) &&
                   ok16(pre_b);
  const int cols = vec ? (width + 3) / 4 : width;
  const int threads = cols <= 64 ? 64 : cols <= 128 ? 128 : 256;
  const dim3 grid(n_rows, (cols + threads - 1) / threads);
  if (vec) cpi::launch_pdl(norm_step_kernel<4>, grid, dim3(threads), 0, stream, p);
  else cpi::launch_pdl(norm_step_kernel<1>, grid, dim3(threads), 0, stream, p);
  return check_launch("norm_step");
}

extern "C" int cpi_rms_step(const float* y, long y_stride, const float* ye, const int* row_of_slot, const int* slot_expert,
                            const float* slot_weight, const void* h_in, int h_in_dtype, long h_in_stride, int top_k,
                            int n_real, float* x, long x_stride, int add, const void* post_w, int post_dtype,
                            float post_offset, float post_eps, const void* pre_w, int pre_dtype, float pre_offset,
                            float pre_eps, void* h_out, int h_out_dtype, long h_out_stride, int n_rows, int width,
                            cudaStream_t stream) {
  if (n_rows == 0) return 0;
  constexpr int MOST = 48 * 1024;                  // columns of the kernel that keeps the row in shared memory
  CPI_REQUIRE(width >= 1 && width <= MOST && x != nullptr, "rms_step: a width of %d (1 to %d)", width, MOST);
  CPI_REQUIRE((y == nullptr) != (ye == nullptr), "rms_step: one source, a row or a sum over experts");
  CPI_REQUIRE(ye == nullptr || (row_of_slot && slot_expert && slot_weight && h_in && top_k >= 1),
              "rms_step: a sum over experts needs the lists of the routing and the experts' input");
  CPI_REQUIRE(post_w != nullptr && (h_out == nullptr || pre_w != nullptr), "rms_step: a norm's weight is missing");
  CPI_REQUIRE((h_out_dtype == kF32 || h_out_dtype == kBF16) && (post_dtype == kF32 || post_dtype == kBF16) &&
              (pre_dtype == kF32 || pre_dtype == kBF16) && (h_in_dtype == kF32 || h_in_dtype == kBF16),
              "rms_step: an unknown dtype");
  RmsStepParams p{{y, y_stride, ye, row_of_slot, slot_expert, slot_weight, h_in, h_in_dtype, h_in_stride, top_k, n_real},
                  x, x_stride, add, post_w, post_dtype, post_offset, post_eps, pre_w, pre_dtype, pre_offset, pre_eps,
                  h_out, h_out_dtype, h_out_stride, width};
  auto ok16 = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & 15) == 0; };
  const bool vec = width % 4 == 0 && width <= 8192 && x_stride % 4 == 0 && y_stride % 4 == 0 && h_in_stride % 4 == 0 &&
                   h_out_stride % 4 == 0 && ok16(x) && ok16(y) && ok16(ye) && ok16(h_in) && ok16(h_out) && ok16(post_w) &&
                   ok16(pre_w);
  if (vec) {
    if (width <= 1024) cpi::launch_pdl(rms_step_kernel<1>, dim3(n_rows), dim3(RMS_THREADS), 0, stream, p);
    else if (width <= 2048) cpi::launch_pdl(rms_step_kernel<2>, dim3(n_rows), dim3(RMS_THREADS), 0, stream, p);
    else if (width <= 4096) cpi::launch_pdl(rms_step_kernel<4>, dim3(n_rows), dim3(RMS_THREADS), 0, stream, p);
    else cpi::launch_pdl(rms_step_kernel<8>, dim3(n_rows), dim3(RMS_THREADS), 0, stream, p);
  } else {
    const size_t smem = (size_t)width * sizeof(float);
    static bool attr_set = false;
    if (smem > 40 * 1024 && !attr_set) {
      if (cudaFuncSetAttribute(rms_step_any_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, MOST * (int)sizeof(float)) != cudaSuccess) {
        set_error("rms_step: %zu bytes of shared memory were refused", smem);
        return 1;
      }
      attr_set = true;
    }
    cpi::launch_pdl(rms_step_any_kernel, dim3(n_rows), dim3(RMS_THREADS), smem, stream, p);
  }
  return check_launch("rms_step");
}
