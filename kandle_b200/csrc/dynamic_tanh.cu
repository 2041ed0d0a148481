// Residual stream steps of decoders whose norm is Dynamic Tanh, y = tanh(alpha x) * w + b.
//
// The norm has no statistics, so it is elementwise and rides on whichever kernel last touches the
// residual row:
//   kd_embed_dynamic_tanh     x = table[id] * scale;                        h = norm(x)
//   kd_residual_dynamic_tanh  x' = x + mixer + sum_k weight_k * expert_k;   h = norm(x')
// The residual stays fp32; the expert rows are gathered straight from the grouped GEMM's output, so
// the un-permutation costs no pass of its own.
// Roofline: HBM, one read of every operand and one write of x' and h.
#include "common.cuh"
#include "kernels.cuh"

namespace kd {

template <int V>
__device__ __forceinline__ void load_vec(const void* p, int dt, int64_t idx, float (&v)[V]) {
  if (V == 4) {
    if (dt == KD_F32) {
      const float4 f = *reinterpret_cast<const float4*>(static_cast<const float*>(p) + idx);
      v[0] = f.x; v[1 % V] = f.y; v[2 % V] = f.z; v[3 % V] = f.w;
    } else {
      const uint2 u = *reinterpret_cast<const uint2*>(static_cast<const __nv_bfloat16*>(p) + idx);
      v[0] = __uint_as_float(u.x << 16); v[1 % V] = __uint_as_float(u.x & 0xffff0000u);
      v[2 % V] = __uint_as_float(u.y << 16); v[3 % V] = __uint_as_float(u.y & 0xffff0000u);
    }
  } else {
    v[0] = dt == KD_F32 ? static_cast<const float*>(p)[idx] : __bfloat162float(static_cast<const __nv_bfloat16*>(p)[idx]);
  }
}

template <int V>
__device__ __forceinline__ void store_vec(void* p, int dt, int64_t idx, const float (&v)[V]) {
  if (V == 4) {
    if (dt == KD_F32) {
      *reinterpret_cast<float4*>(static_cast<float*>(p) + idx) = make_float4(v[0], v[1 % V], v[2 % V], v[3 % V]);
    } else {
      __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1 % V]), b = __floats2bfloat162_rn(v[2 % V], v[3 % V]);
      uint2 u;
      u.x = *reinterpret_cast<uint32_t*>(&a);
      u.y = *reinterpret_cast<uint32_t*>(&b);
      *reinterpret_cast<uint2*>(static_cast<__nv_bfloat16*>(p) + idx) = u;
    }
  } else {
    if (dt == KD_F32) static_cast<float*>(p)[idx] = v[0];
    else static_cast<__nv_bfloat16*>(p)[idx] = __float2bfloat16_rn(v[0]);
  }
}

struct DytNorm {
  float alpha;
  const float* w;
  const float* b;
};

template <int V>
__device__ __forceinline__ void dyt_apply(const DytNorm& n, int col, const float (&x)[V], float (&y)[V]) {
#pragma unroll
  for (int i = 0; i < V; ++i) y[i] = fmaf(tanhf(n.alpha * x[i]), __ldg(n.w + col + i), __ldg(n.b + col + i));
}

// grid (rows, column chunks of blockDim * V)
template <int V>
__global__ void embed_dyt_kernel(const void* __restrict__ table, int dt_table, int64_t vocab, const void* __restrict__ ids, int ids64,
                                 float scale, int width, DytNorm n, float* __restrict__ x_out, void* __restrict__ h_out, int dt_h,
                                 int* __restrict__ err) {
  pdl_wait();
  pdl_trigger();
  const int64_t row = blockIdx.x;
  const int64_t id = ids64 ? static_cast<const int64_t*>(ids)[row] : (int64_t)static_cast<const int32_t*>(ids)[row];
  const bool ok = id >= 0 && id < vocab;
  if (!ok && threadIdx.x == 0 && blockIdx.y == 0 && atomicCAS(err, 0, 101) == 0) { err[1] = (int)id; err[2] = (int)vocab; }
  const int col = (blockIdx.y * blockDim.x + threadIdx.x) * V;
  if (col >= width) return;
  float x[V], y[V];
#pragma unroll
  for (int i = 0; i < V; ++i) x[i] = 0.f;
  if (ok) load_vec<V>(table, dt_table, id * width + col, x);
#pragma unroll
  for (int i = 0; i < V; ++i) x[i] *= scale;
  dyt_apply<V>(n, col, x, y);
  store_vec<V>(x_out, KD_F32, row * width + col, x);
  store_vec<V>(h_out, dt_h, row * width + col, y);
}

struct ResidualParams {
  int rows, width;
  const float* x;
  const void* mix;      // [splits][rows][width] partial sums, or NULL
  int dt_mix, splits;
  const void* y;        // expert rows [.., width], or NULL
  int dt_y, top;
  int64_t y_rows;
  const int* slots;     // [rows, top] row of y
  const float* weights; // [rows, top]
  float* x_out;
  void* h_out;
  int dt_h;
  int* err;
};

template <int V>
__global__ void residual_dyt_kernel(ResidualParams p, DytNorm n) {
  pdl_wait();
  pdl_trigger();
  const int64_t row = blockIdx.x;
  const int col = (blockIdx.y * blockDim.x + threadIdx.x) * V;
  if (col >= p.width) return;
  const int64_t at = row * p.width + col;
  float x[V], acc[V], t[V], y[V];
  load_vec<V>(p.x, KD_F32, at, x);
#pragma unroll
  for (int i = 0; i < V; ++i) acc[i] = 0.f;
  if (p.mix) {
    for (int s = 0; s < p.splits; ++s) {
      load_vec<V>(p.mix, p.dt_mix, (int64_t)s * p.rows * p.width + at, t);
#pragma unroll
      for (int i = 0; i < V; ++i) acc[i] += t[i];
    }
  }
  if (p.y) {
#pragma unroll 4
    for (int k = 0; k < p.top; ++k) {
      const int slot = p.slots[row * p.top + k];
      const float w = p.weights[row * p.top + k];
      if (slot < 0 || slot >= p.y_rows) {
        if (col == 0 && atomicCAS(p.err, 0, 111) == 0) { p.err[1] = slot; p.err[2] = (int)p.y_rows; }
        continue;
      }
      load_vec<V>(p.y, p.dt_y, (int64_t)slot * p.width + col, t);
#pragma unroll
      for (int i = 0; i < V; ++i) acc[i] = fmaf(w, t[i], acc[i]);
    }
  }
#pragma unroll
  for (int i = 0; i < V; ++i) x[i] += acc[i];
  dyt_apply<V>(n, col, x, y);
  store_vec<V>(p.x_out, KD_F32, at, x);
  store_vec<V>(p.h_out, p.dt_h, at, y);
}

static int dyt_params(const kd_tensor* w, const kd_tensor* b, float alpha, int64_t width, DytNorm* n) {
  KD_REQUIRE(w && b && w->dtype == KD_F32 && b->dtype == KD_F32 && is_contiguous(w) && is_contiguous(b) && numel(w) == width && numel(b) == width,
             "norm weight and bias must be contiguous fp32 [%lld]", (long long)width);
  void *pw, *pb;
  KD_TRY(tensor_ptr(w, &pw));
  KD_TRY(tensor_ptr(b, &pb));
  n->alpha = alpha;
  n->w = static_cast<const float*>(pw);
  n->b = static_cast<const float*>(pb);
  return KD_OK;
}

static bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

}  // namespace kd

using namespace kd;

KD_API int kd_embed_dynamic_tanh(const kd_tensor* table, const kd_tensor* ids, float scale, float alpha, const kd_tensor* norm_weight,
                                 const kd_tensor* norm_bias, const kd_tensor* x_out, const kd_tensor* h_out) {
  KD_TRY(require_init());
  KD_REQUIRE(table && ids && x_out && h_out, "null tensor");
  KD_REQUIRE(table->ndim == 2 && is_contiguous(table) && (table->dtype == KD_F32 || table->dtype == KD_BF16), "table must be fp32 or bf16 [V,W]");
  KD_REQUIRE((ids->dtype == KD_I32 || ids->dtype == KD_I64) && is_contiguous(ids), "ids must be contiguous int32 or int64");
  const int64_t rows = numel(ids), W = table->shape[1];
  KD_REQUIRE(x_out->dtype == KD_F32 && is_contiguous(x_out) && numel(x_out) == rows * W, "x_out must be contiguous fp32 [T,W]");
  KD_REQUIRE((h_out->dtype == KD_F32 || h_out->dtype == KD_BF16) && is_contiguous(h_out) && numel(h_out) == rows * W, "h_out must be contiguous [T,W]");
  DytNorm n;
  KD_TRY(dyt_params(norm_weight, norm_bias, alpha, W, &n));
  if (rows == 0) return KD_OK;
  void *pt, *pi, *px, *ph;
  KD_TRY(tensor_ptr(table, &pt));
  KD_TRY(tensor_ptr(ids, &pi));
  KD_TRY(tensor_ptr(x_out, &px));
  KD_TRY(tensor_ptr(h_out, &ph));
  const bool v4 = W % 4 == 0 && aligned16(pt) && aligned16(px) && aligned16(ph);
  const int V = v4 ? 4 : 1, threads = 256;
  dim3 grid((unsigned)rows, (unsigned)((W / V + threads - 1) / threads + (W % V ? 1 : 0)));
  auto k = v4 ? embed_dyt_kernel<4> : embed_dyt_kernel<1>;
  KD_CUDA_CHECK(launch_ex(k, grid, dim3(threads), 0, (const void*)pt, (int)table->dtype, table->shape[0], (const void*)pi,
                          (int)(ids->dtype == KD_I64), scale, (int)W, n, static_cast<float*>(px), ph, (int)h_out->dtype, ctx().error_flag));
  return after_launch("embed_dyt_kernel");
}

KD_API int kd_residual_dynamic_tanh(const kd_tensor* x, const kd_tensor* mix, const kd_tensor* y, const kd_tensor* slots,
                                    const kd_tensor* weights, float alpha, const kd_tensor* norm_weight, const kd_tensor* norm_bias,
                                    const kd_tensor* x_out, const kd_tensor* h_out) {
  KD_TRY(require_init());
  KD_REQUIRE(x && x_out && h_out, "null tensor");
  KD_REQUIRE(x->ndim == 2 && x->dtype == KD_F32 && is_contiguous(x), "x must be contiguous fp32 [T,W]");
  const int64_t rows = x->shape[0], W = x->shape[1];
  KD_REQUIRE(x_out->dtype == KD_F32 && is_contiguous(x_out) && numel(x_out) == rows * W, "x_out must be contiguous fp32 [T,W]");
  KD_REQUIRE((h_out->dtype == KD_F32 || h_out->dtype == KD_BF16) && is_contiguous(h_out) && numel(h_out) == rows * W, "h_out must be contiguous [T,W]");
  DytNorm n;
  KD_TRY(dyt_params(norm_weight, norm_bias, alpha, W, &n));
  if (rows == 0) return KD_OK;
  ResidualParams p{};
  p.rows = (int)rows; p.width = (int)W;
  p.dt_h = h_out->dtype;
  p.err = ctx().error_flag;
  void* q;
  bool v4 = W % 4 == 0;
  KD_TRY(tensor_ptr(x, &q)); p.x = static_cast<const float*>(q); v4 = v4 && aligned16(q);
  KD_TRY(tensor_ptr(x_out, &q)); p.x_out = static_cast<float*>(q); v4 = v4 && aligned16(q);
  KD_TRY(tensor_ptr(h_out, &q)); p.h_out = q; v4 = v4 && aligned16(q);
  if (mix) {
    KD_REQUIRE((mix->dtype == KD_F32 || mix->dtype == KD_BF16) && is_contiguous(mix) && numel(mix) % (rows * W) == 0, "mix must be contiguous [splits,T,W]");
    KD_TRY(tensor_ptr(mix, &q)); p.mix = q; v4 = v4 && aligned16(q);
    p.dt_mix = mix->dtype;
    p.splits = (int)(numel(mix) / (rows * W));
  }
  if (y) {
    KD_REQUIRE(slots && weights, "expert rows need slots and weights");
    KD_REQUIRE((y->dtype == KD_F32 || y->dtype == KD_BF16) && is_contiguous(y) && y->ndim == 2 && y->shape[1] == W, "y must be contiguous [R,W]");
    KD_REQUIRE(slots->dtype == KD_I32 && is_contiguous(slots) && numel(slots) % rows == 0, "slots must be contiguous int32 [T,top]");
    KD_REQUIRE(weights->dtype == KD_F32 && is_contiguous(weights) && numel(weights) == numel(slots), "weights must be contiguous fp32 [T,top]");
    KD_TRY(tensor_ptr(y, &q)); p.y = q; v4 = v4 && aligned16(q);
    p.dt_y = y->dtype;
    p.y_rows = y->shape[0];
    KD_TRY(tensor_ptr(slots, &q)); p.slots = static_cast<const int*>(q);
    KD_TRY(tensor_ptr(weights, &q)); p.weights = static_cast<const float*>(q);
    p.top = (int)(numel(slots) / rows);
  }
  const int V = v4 ? 4 : 1, threads = W / V >= 256 ? 256 : 128;
  dim3 grid((unsigned)rows, (unsigned)((W / V + threads - 1) / threads));
  auto k = v4 ? residual_dyt_kernel<4> : residual_dyt_kernel<1>;
  KD_CUDA_CHECK(launch_ex(k, grid, dim3(threads), 0, p, n));
  return after_launch("residual_dyt_kernel");
}
