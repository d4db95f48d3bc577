// Boundaries between sublayers whose norms act element by element (tanh(alpha x) * w + b, no statistics of the row):
//
//   norm_step   v = a sublayer's output for token t, given as
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
#include "common.cuh"

namespace cpi {

struct NormStepParams {
  const float* y; long y_stride;                   // [T, W] or null
  const float* ye; const int* row_of_slot; const int* slot_expert; const float* slot_weight;    // experts or null
  const void* h_in; int h_in_dtype; long h_in_stride;
  int top_k, n_real;
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
  const bool enters = p.y != nullptr || p.ye != nullptr;
  if (!enters || p.add) x = loadv<V>(xp);
  if (enters) {
    Vec<V> v;
    if (p.y) {
      v = loadv<V>(p.y + (size_t)t * p.y_stride + c);
    } else {
#pragma unroll
      for (int i = 0; i < V; ++i) v.v[i] = 0.f;
      for (int k0 = 0; k0 < p.top_k; k0 += 4) {                // four rows' loads in flight
        Vec<V> e[4];
        float f[4];
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          f[k] = 0.f;
          if (k0 + k < p.top_k) {
            const size_t s = (size_t)t * p.top_k + k0 + k;
            if (p.slot_expert[s] < p.n_real) {
              f[k] = 1.f;
              e[k] = loadv<V>(p.ye + (size_t)p.row_of_slot[s] * p.width + c);
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
    }
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
  NormStepParams p{y, y_stride, ye, row_of_slot, slot_expert, slot_weight, h_in, h_in_dtype, h_in_stride, top_k, n_real,
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
