// Residual stream steps of decoders that normalise a sublayer's OUTPUT: x' = x + rmsnorm(y) * w.
//
//   kd_embed_rows          x = table[id] (fp32) and its copy in the engine's type, which the first sublayer reads
//   kd_residual_post_norm  x' = x + y / sqrt(mean(y^2) + eps) * w,  y = sum of the split-K partial sums;
//                          h = x', or after the last sublayer h = x' / sqrt(mean(x'^2) + eps) * w_final
// One CTA a row; the row stays in registers between the sum of squares and the update.  x is fp32 throughout.
// Roofline: HBM, one read of x and y and one write of x' and h.
#include "common.cuh"
#include "kernels.cuh"

namespace kd {

namespace {
__device__ __forceinline__ void load4(const void* p, int dt, int64_t at, float (&v)[4]) {
  if (dt == KD_F32) {
    const float4 f = *reinterpret_cast<const float4*>(static_cast<const float*>(p) + at);
    v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
  } else {
    const uint2 u = *reinterpret_cast<const uint2*>(static_cast<const __nv_bfloat16*>(p) + at);
    v[0] = __uint_as_float(u.x << 16); v[1] = __uint_as_float(u.x & 0xffff0000u);
    v[2] = __uint_as_float(u.y << 16); v[3] = __uint_as_float(u.y & 0xffff0000u);
  }
}
__device__ __forceinline__ void store4(void* p, int dt, int64_t at, const float (&v)[4]) {
  if (dt == KD_F32) {
    *reinterpret_cast<float4*>(static_cast<float*>(p) + at) = make_float4(v[0], v[1], v[2], v[3]);
  } else {
    __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    uint2 u;
    u.x = *reinterpret_cast<uint32_t*>(&a);
    u.y = *reinterpret_cast<uint32_t*>(&b);
    *reinterpret_cast<uint2*>(static_cast<__nv_bfloat16*>(p) + at) = u;
  }
}
}  // namespace

__global__ void embed_rows_kernel(const void* __restrict__ table, int dt_table, int64_t vocab, const void* __restrict__ ids, int ids64,
                                  int width, int vec, float* __restrict__ x_out, void* __restrict__ h_out, int dt_h, int* __restrict__ err) {
  pdl_wait();
  pdl_trigger();
  const int64_t row = blockIdx.x;
  const int64_t id = ids64 ? static_cast<const int64_t*>(ids)[row] : (int64_t)static_cast<const int32_t*>(ids)[row];
  const bool ok = id >= 0 && id < vocab;
  if (!ok && threadIdx.x == 0 && atomicCAS(err, 0, 101) == 0) { err[1] = (int)id; err[2] = (int)vocab; }
  if (vec) {
    for (int col = threadIdx.x * 4; col < width; col += blockDim.x * 4) {
      float v[4] = {0.f, 0.f, 0.f, 0.f};
      if (ok) load4(table, dt_table, id * width + col, v);
      store4(x_out, KD_F32, row * width + col, v);
      store4(h_out, dt_h, row * width + col, v);
    }
    return;
  }
  for (int col = threadIdx.x; col < width; col += blockDim.x) {
    const float v = ok ? load_float(table, dt_table, id * width + col) : 0.f;
    x_out[row * width + col] = v;
    store_float(h_out, dt_h, row * width + col, v);
  }
}

struct PostNormParams {
  int64_t rows;
  int width, splits;
  const float* x;
  const void* y;          // [splits, rows, width]
  int dt_y, dt_h;
  float eps;
  const float* w;         // [width]
  const float* w_final;   // [width], or null: h = x'
  float* x_out;
  void* h;
};

// Sum over the CTA; every thread gets it.  `red` [32] may be used again after the next barrier.
__device__ __forceinline__ float block_total(float v, float* red) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
  for (int i = 0; i < (int)(blockDim.x >> 5); ++i) t += red[i];
  return t;
}

// NV chunks of four columns a thread.
template <int NV>
__global__ void __launch_bounds__(256) residual_post_norm_kernel(PostNormParams p) {
  __shared__ float red[2][32];
  pdl_wait();
  pdl_trigger();
  const int64_t row = blockIdx.x;
  float x[NV][4], y[NV][4], ss = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int col = (i * blockDim.x + threadIdx.x) * 4;
    if (col < p.width) {
      load4(p.y, p.dt_y, row * p.width + col, y[i]);
      load4(p.x, KD_F32, row * p.width + col, x[i]);
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e) x[i][e] = y[i][e] = 0.f;
    }
  }
  for (int s = 1; s < p.splits; ++s)
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int col = (i * blockDim.x + threadIdx.x) * 4;
      if (col < p.width) {
        float t[4];
        load4(p.y, p.dt_y, ((int64_t)s * p.rows + row) * p.width + col, t);
#pragma unroll
        for (int e = 0; e < 4; ++e) y[i][e] += t[e];
      }
    }
#pragma unroll
  for (int i = 0; i < NV; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) ss = fmaf(y[i][e], y[i][e], ss);
  float inv = 1.0f / sqrtf(block_total(ss, red[0]) / (float)p.width + p.eps);
  ss = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int col = (i * blockDim.x + threadIdx.x) * 4;
    if (col < p.width) {
      float w[4];
      load4(p.w, KD_F32, col, w);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        x[i][e] = fmaf(y[i][e] * inv, w[e], x[i][e]);
        ss = fmaf(x[i][e], x[i][e], ss);
      }
      store4(p.x_out, KD_F32, row * p.width + col, x[i]);
      if (!p.w_final) store4(p.h, p.dt_h, row * p.width + col, x[i]);
    }
  }
  if (!p.w_final) return;
  inv = 1.0f / sqrtf(block_total(ss, red[1]) / (float)p.width + p.eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int col = (i * blockDim.x + threadIdx.x) * 4;
    if (col < p.width) {
      float w[4];
      load4(p.w_final, KD_F32, col, w);
#pragma unroll
      for (int e = 0; e < 4; ++e) w[e] *= x[i][e] * inv;
      store4(p.h, p.dt_h, row * p.width + col, w);
    }
  }
}

// Any width: the row is read again instead of kept (every thread re-reads what it alone reads and writes).
__global__ void __launch_bounds__(256) residual_post_norm_any_kernel(PostNormParams p) {
  __shared__ float red[2][32];
  pdl_wait();
  pdl_trigger();
  const int64_t row = blockIdx.x;
  auto y_at = [&](int col) {
    float v = 0.f;
    for (int s = 0; s < p.splits; ++s) v += load_float(p.y, p.dt_y, ((int64_t)s * p.rows + row) * p.width + col);
    return v;
  };
  float ss = 0.f;
  for (int col = threadIdx.x; col < p.width; col += blockDim.x) { const float v = y_at(col); ss = fmaf(v, v, ss); }
  float inv = 1.0f / sqrtf(block_total(ss, red[0]) / (float)p.width + p.eps);
  ss = 0.f;
  for (int col = threadIdx.x; col < p.width; col += blockDim.x) {
    const int64_t at = row * p.width + col;
    const float v = fmaf(y_at(col) * inv, p.w[col], p.x[at]);
    ss = fmaf(v, v, ss);
    p.x_out[at] = v;
    if (!p.w_final) store_float(p.h, p.dt_h, at, v);
  }
  if (!p.w_final) return;
  inv = 1.0f / sqrtf(block_total(ss, red[1]) / (float)p.width + p.eps);
  for (int col = threadIdx.x; col < p.width; col += blockDim.x) {
    const int64_t at = row * p.width + col;
    store_float(p.h, p.dt_h, at, p.x_out[at] * inv * p.w_final[col]);
  }
}

}  // namespace kd

using namespace kd;

KD_API int kd_embed_rows(const kd_tensor* table, const kd_tensor* ids, const kd_tensor* x_out, const kd_tensor* h_out) {
  KD_TRY(require_init());
  KD_REQUIRE(table && ids && x_out && h_out, "null tensor");
  KD_REQUIRE(table->ndim == 2 && is_contiguous(table) && (table->dtype == KD_F32 || table->dtype == KD_BF16), "table must be fp32 or bf16 [V,W]");
  KD_REQUIRE((ids->dtype == KD_I32 || ids->dtype == KD_I64) && is_contiguous(ids), "ids must be contiguous int32 or int64");
  const int64_t rows = numel(ids), W = table->shape[1];
  KD_REQUIRE(x_out->dtype == KD_F32 && is_contiguous(x_out) && numel(x_out) == rows * W, "x_out must be contiguous fp32 [T,W]");
  KD_REQUIRE((h_out->dtype == KD_F32 || h_out->dtype == KD_BF16) && is_contiguous(h_out) && numel(h_out) == rows * W, "h_out must be contiguous [T,W]");
  if (rows == 0) return KD_OK;
  void *pt, *pi, *px, *ph;
  KD_TRY(tensor_ptr(table, &pt));
  KD_TRY(tensor_ptr(ids, &pi));
  KD_TRY(tensor_ptr(x_out, &px));
  KD_TRY(tensor_ptr(h_out, &ph));
  const int vec = W % 4 == 0 && ((reinterpret_cast<uintptr_t>(pt) | reinterpret_cast<uintptr_t>(px) | reinterpret_cast<uintptr_t>(ph)) & 15) == 0;
  KD_CUDA_CHECK(launch_ex(embed_rows_kernel, dim3((unsigned)rows), dim3(256), 0, (const void*)pt, (int)table->dtype, table->shape[0], (const void*)pi,
                          (int)(ids->dtype == KD_I64), (int)W, vec, static_cast<float*>(px), ph, (int)h_out->dtype, ctx().error_flag));
  return after_launch("embed_rows_kernel");
}

KD_API int kd_residual_post_norm(const kd_tensor* x, const kd_tensor* y, const kd_tensor* norm_weight, float eps, const kd_tensor* final_weight,
                                 const kd_tensor* x_out, const kd_tensor* h_out) {
  KD_TRY(require_init());
  KD_REQUIRE(x && y && norm_weight && x_out && h_out, "null tensor");
  KD_REQUIRE(x->ndim == 2 && x->dtype == KD_F32 && is_contiguous(x), "x must be contiguous fp32 [T,W]");
  const int64_t rows = x->shape[0], W = x->shape[1];
  KD_REQUIRE(x_out->dtype == KD_F32 && is_contiguous(x_out) && numel(x_out) == rows * W, "x_out must be contiguous fp32 [T,W]");
  KD_REQUIRE((h_out->dtype == KD_F32 || h_out->dtype == KD_BF16) && is_contiguous(h_out) && numel(h_out) == rows * W, "h_out must be contiguous [T,W]");
  KD_REQUIRE(W >= 1 && W < (1ll << 30), "width %lld", (long long)W);
  if (rows == 0) return KD_OK;
  KD_REQUIRE((y->dtype == KD_F32 || y->dtype == KD_BF16) && is_contiguous(y) && numel(y) > 0 && numel(y) % (rows * W) == 0, "y must be contiguous [splits,T,W]");
  PostNormParams p{};
  p.rows = rows; p.width = (int)W;
  p.splits = (int)(numel(y) / (rows * W));
  p.dt_y = y->dtype; p.dt_h = h_out->dtype;
  p.eps = eps;
  uintptr_t all = 0;
  void* q;
  for (const kd_tensor* t : {norm_weight, final_weight}) {
    if (!t) continue;
    KD_REQUIRE(t->dtype == KD_F32 && is_contiguous(t) && numel(t) == W, "norm weights must be contiguous fp32 [%lld]", (long long)W);
    KD_TRY(tensor_ptr(t, &q));
    all |= reinterpret_cast<uintptr_t>(q);
    (t == norm_weight ? p.w : p.w_final) = static_cast<const float*>(q);
  }
  if (final_weight == norm_weight) p.w_final = p.w;
  KD_TRY(tensor_ptr(x, &q)); p.x = static_cast<const float*>(q); all |= reinterpret_cast<uintptr_t>(q);
  KD_TRY(tensor_ptr(y, &q)); p.y = q; all |= reinterpret_cast<uintptr_t>(q);
  KD_TRY(tensor_ptr(x_out, &q)); p.x_out = static_cast<float*>(q); all |= reinterpret_cast<uintptr_t>(q);
  KD_TRY(tensor_ptr(h_out, &q)); p.h = q; all |= reinterpret_cast<uintptr_t>(q);
  auto kernel = residual_post_norm_any_kernel;
  int threads = 256;
  if (W % 4 == 0 && (all & 15) == 0 && W <= 8192) {
    threads = W >= 1024 ? 256 : W >= 512 ? 128 : 64;
    const int64_t chunks = (W / 4 + threads - 1) / threads;
    kernel = chunks <= 1 ? residual_post_norm_kernel<1> : chunks <= 2 ? residual_post_norm_kernel<2> : chunks <= 4 ? residual_post_norm_kernel<4> : residual_post_norm_kernel<8>;
  }
  KD_CUDA_CHECK(launch_ex(kernel, dim3((unsigned)rows), dim3(threads), 0, p));
  return after_launch("residual_post_norm_kernel");
}
