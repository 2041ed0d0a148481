// Grouped-query attention over a key/value cache with a sliding window: query i sees the keys j with
// 0 <= i - j < window.  Per-head scores may join a sink (exp(sink) in the denominator, no value).
//
//   kd_qk_norm_rope_cache   RMS norm over the whole query (key) projection, rotary positions on the first `rot`
//                           dimensions of a head (entry i paired with i + rot/2); writes the queries and the
//                           cache rows, both padded with zeros to the kernels' head sizes
//   kd_window_attention     prompts and portions: the tcgen05 prefill kernel from the first visible key tile on
//                           (attention_prefill2.cu); one token: the split-KV decode kernel over the window's tiles
//                           (attention_tcgen05.cu).  fp32, and head sizes above 128: the CUDA-core kernel below
// Roofline: prep and decode HBM, prefill tensor cores (4 D flops per visible pair and head).
#include "common.cuh"
#include "kernels.cuh"

namespace kd {

// ----------------------------------------------------------------------------- norm, rotation, cache rows
struct QkPrepParams {
  int S, H, G, dim, vdim, rot, dq, dv, max_s;
  int q_col, k_col, v_col;      // first columns in a projection row (k_col < 0: queries only)
  int64_t ld;
  int64_t kc_b, kc_h, kc_s, vc_b, vc_h, vc_s;
  float eps;
  int vec;                      // 8-column pieces everywhere
  const float* qw;              // [H*dim]
  const float* kw;              // [G*dim]
  const float* cos_t;           // [max_s, rot/2]
  const float* sin_t;
  const int* pos_dev;
  int pos_host;
  int* err;
};

template <typename T> __device__ __forceinline__ float wa_f(T v);
template <> __device__ __forceinline__ float wa_f<float>(float v) { return v; }
template <> __device__ __forceinline__ float wa_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T wa_t(float v);
template <> __device__ __forceinline__ float wa_t<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 wa_t<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

__device__ __forceinline__ uint32_t wa_pack(float a, float b) {
  __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<uint32_t*>(&v);
}

constexpr int QK_THREADS = 128;     // small CTAs: a token is a chain of latencies, so many of them share an SM

// One CTA a token; the query and key rows pass through shared memory as fp32.
template <typename T>
__global__ void __launch_bounds__(QK_THREADS, 8)
qk_prep_kernel(const T* __restrict__ proj, T* __restrict__ q_out, T* __restrict__ k_cache, T* __restrict__ v_cache, QkPrepParams p) {
  extern __shared__ __align__(16) float row_s[];      // [(H + G) * dim] weighted values before the scale
  __shared__ float red[2][QK_THREADS / 32];
  pdl_wait();
  pdl_trigger();
  const int64_t token = blockIdx.x;
  const int b = (int)(token / p.S), si = (int)(token - (int64_t)b * p.S);
  const int pos = (p.pos_dev ? *p.pos_dev : p.pos_host) + si;
  if (pos < 0 || pos >= p.max_s) {    // never outside the tables and the cache; report instead
    if (threadIdx.x == 0 && atomicCAS(p.err, 0, 102) == 0) { p.err[1] = pos; p.err[2] = p.max_s; }
    return;
  }
  const T* row = proj + token * p.ld;
  const int nq = p.H * p.dim, nk = p.k_col >= 0 ? p.G * p.dim : 0, tid = threadIdx.x;
  float sq = 0.f, sk = 0.f;
  if (sizeof(T) == 2 && p.vec) {
    for (int i = tid * 8; i < nq + nk; i += QK_THREADS * 8) {
      const bool is_q = i < nq;
      const uint4 u = *reinterpret_cast<const uint4*>(row + (is_q ? p.q_col + i : p.k_col + i - nq));
      const float* w = is_q ? p.qw + i : p.kw + i - nq;
      const float4 w0 = *reinterpret_cast<const float4*>(w), w1 = *reinterpret_cast<const float4*>(w + 4);
      const float v[8] = {__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xffff0000u), __uint_as_float(u.y << 16), __uint_as_float(u.y & 0xffff0000u),
                          __uint_as_float(u.z << 16), __uint_as_float(u.z & 0xffff0000u), __uint_as_float(u.w << 16), __uint_as_float(u.w & 0xffff0000u)};
      float ss = 0.f;
#pragma unroll
      for (int e = 0; e < 8; ++e) ss = fmaf(v[e], v[e], ss);
      if (is_q) sq += ss; else sk += ss;
      *reinterpret_cast<float4*>(row_s + i) = make_float4(v[0] * w0.x, v[1] * w0.y, v[2] * w0.z, v[3] * w0.w);
      *reinterpret_cast<float4*>(row_s + i + 4) = make_float4(v[4] * w1.x, v[5] * w1.y, v[6] * w1.z, v[7] * w1.w);
    }
  } else {
    for (int i = tid; i < nq + nk; i += QK_THREADS) {
      const bool is_q = i < nq;
      const float v = wa_f<T>(row[is_q ? p.q_col + i : p.k_col + i - nq]);
      if (is_q) sq = fmaf(v, v, sq); else sk = fmaf(v, v, sk);
      row_s[i] = v * (is_q ? p.qw[i] : p.kw[i - nq]);
    }
  }
  sq = warp_sum(sq);
  sk = warp_sum(sk);
  if ((tid & 31) == 0) { red[0][tid >> 5] = sq; red[1][tid >> 5] = sk; }
  __syncthreads();
  sq = sk = 0.f;
#pragma unroll
  for (int w = 0; w < QK_THREADS / 32; ++w) { sq += red[0][w]; sk += red[1][w]; }
  const float iq = 1.0f / sqrtf(sq / (float)nq + p.eps), ik = nk ? 1.0f / sqrtf(sk / (float)nk + p.eps) : 0.f;
  const int n2 = p.rot / 2;
  const float* cs = p.cos_t + (int64_t)pos * n2;
  const float* sn = p.sin_t + (int64_t)pos * n2;
  // entry i of head x (queries first, then keys), normed and rotated
  auto entry = [&](int x, int i) -> float {
    if (i >= p.dim) return 0.f;
    const float inv = x < p.H ? iq : ik;
    const float* r = row_s + x * p.dim;
    if (i < n2) return r[i] * inv * cs[i] - r[i + n2] * inv * sn[i];
    if (i < p.rot) return r[i] * inv * cs[i - n2] + r[i - n2] * inv * sn[i - n2];
    return r[i] * inv;
  };
  const int heads = p.H + (nk ? p.G : 0);
  auto dest = [&](int x) -> T* {
    return x < p.H ? q_out + (token * p.H + x) * p.dq : k_cache + (int64_t)b * p.kc_b + (int64_t)(x - p.H) * p.kc_h + (int64_t)pos * p.kc_s;
  };
  if (sizeof(T) == 2 && p.vec) {
    const int pieces = p.dq / 8;
    for (int i = tid; i < heads * pieces; i += QK_THREADS) {
      const int x = i / pieces, e = (i - x * pieces) * 8;
      float y[8];
      if (p.rot % 16 == 0 && e < p.dim) {       // eight entries lie on one side of every boundary
        const float inv = x < p.H ? iq : ik;
        const float* r = row_s + x * p.dim + e;
        const float4 a = *reinterpret_cast<const float4*>(r), c = *reinterpret_cast<const float4*>(r + 4);
        const float own[8] = {a.x * inv, a.y * inv, a.z * inv, a.w * inv, c.x * inv, c.y * inv, c.z * inv, c.w * inv};
        if (e < p.rot) {
          const bool low = e < n2;
          const float* o = low ? r + n2 : r - n2;
          const float* ct = cs + (low ? e : e - n2);
          const float* st = sn + (low ? e : e - n2);
          const float sign = low ? -inv : inv;
#pragma unroll
          for (int w = 0; w < 2; ++w) {
            const float4 f = *reinterpret_cast<const float4*>(o + 4 * w), co = *reinterpret_cast<const float4*>(ct + 4 * w), si4 = *reinterpret_cast<const float4*>(st + 4 * w);
            y[4 * w + 0] = fmaf(own[4 * w + 0], co.x, sign * f.x * si4.x);
            y[4 * w + 1] = fmaf(own[4 * w + 1], co.y, sign * f.y * si4.y);
            y[4 * w + 2] = fmaf(own[4 * w + 2], co.z, sign * f.z * si4.z);
            y[4 * w + 3] = fmaf(own[4 * w + 3], co.w, sign * f.w * si4.w);
          }
        } else {
#pragma unroll
          for (int w = 0; w < 8; ++w) y[w] = own[w];
        }
      } else {
#pragma unroll
        for (int w = 0; w < 8; ++w) y[w] = entry(x, e + w);
      }
      const uint4 u = make_uint4(wa_pack(y[0], y[1]), wa_pack(y[2], y[3]), wa_pack(y[4], y[5]), wa_pack(y[6], y[7]));
      *reinterpret_cast<uint4*>(dest(x) + e) = u;
    }
    if (!nk) return;
    const int vp = p.dv / 8;
    for (int i = tid; i < p.G * vp; i += QK_THREADS) {
      const int x = i / vp, e = (i - x * vp) * 8;
      const uint4 u = e < p.vdim ? *reinterpret_cast<const uint4*>(row + p.v_col + x * p.vdim + e) : make_uint4(0, 0, 0, 0);
      *reinterpret_cast<uint4*>(v_cache + (int64_t)b * p.vc_b + (int64_t)x * p.vc_h + (int64_t)pos * p.vc_s + e) = u;
    }
    return;
  }
  for (int i = tid; i < heads * p.dq; i += QK_THREADS) {
    const int x = i / p.dq, e = i - x * p.dq;
    dest(x)[e] = wa_t<T>(entry(x, e));
  }
  if (!nk) return;
  for (int i = tid; i < p.G * p.dv; i += QK_THREADS) {
    const int x = i / p.dv, e = i - x * p.dv;
    v_cache[(int64_t)b * p.vc_b + (int64_t)x * p.vc_h + (int64_t)pos * p.vc_s + e] = e < p.vdim ? row[p.v_col + x * p.vdim + e] : wa_t<T>(0.f);
  }
}

// ----------------------------------------------------------------------------- CUDA-core attention
// A warp owns one row (query, head of the group); 16 rows of one key head share each 32-key tile in shared memory.
// Running maximum and sum start at the sink (score sink, no value), so no tile needs a special case.
constexpr int WA_WARPS = 16, WA_KEYS = 32;

struct WindowParams {
  int B, S, H, G, dq, dv, max_s;
  int window;                   // 0: every key up to the query
  int64_t kc_b, kc_h, kc_s, vc_b, vc_h, vc_s;
  float scale;
  const float* sink;            // [H], or null
  const int* pos_dev;
  int pos_host;
};

template <typename T, int VPL>   // value columns a lane: dv <= 32 VPL
__global__ void __launch_bounds__(WA_WARPS * 32)
window_attention_kernel(const T* __restrict__ q, const T* __restrict__ k_cache, const T* __restrict__ v_cache, T* __restrict__ out, WindowParams p) {
  extern __shared__ float smem[];
  float* ks = smem;                                // [WA_KEYS][dq + 1]
  float* vs = ks + WA_KEYS * (p.dq + 1);           // [WA_KEYS][dv]
  float* qs = vs + WA_KEYS * p.dv;                 // [WA_WARPS][dq]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = blockIdx.y, b = blockIdx.z, group = p.H / p.G;
  pdl_wait();
  pdl_trigger();
  const int pos0 = p.pos_dev ? *p.pos_dev : p.pos_host;
  if (pos0 < 0 || pos0 + p.S > p.max_s) return;    // (reported by the kernel that writes the cache rows)
  const int rows = p.S * group, row0 = blockIdx.x * WA_WARPS, row = row0 + warp;
  const bool row_ok = row < rows;
  const int s = min(row, rows - 1) / group, head = g * group + min(row, rows - 1) % group;
  const int me = pos0 + s;                         // this row's position
  const int first = p.window > 0 ? max(0, me - p.window + 1) : 0;
  const int lo = p.window > 0 ? max(0, pos0 + row0 / group - p.window + 1) : 0;      // of all rows of the CTA
  const int hi = pos0 + min(row0 + WA_WARPS - 1, rows - 1) / group + 1;
  const T* qr = q + (((int64_t)b * p.S + s) * p.H + head) * p.dq;
  for (int d = lane; d < p.dq; d += 32) qs[warp * p.dq + d] = wa_f<T>(qr[d]) * p.scale;
  float acc[VPL];
#pragma unroll
  for (int i = 0; i < VPL; ++i) acc[i] = 0.f;
  float m = p.sink ? p.sink[head] : -1e30f, l = p.sink ? 1.f : 0.f;
  const T* kb = k_cache + (int64_t)b * p.kc_b + (int64_t)g * p.kc_h;
  const T* vb = v_cache + (int64_t)b * p.vc_b + (int64_t)g * p.vc_h;
  for (int j0 = lo; j0 < hi; j0 += WA_KEYS) {
    __syncthreads();
    for (int e = threadIdx.x; e < WA_KEYS * p.dq; e += WA_WARPS * 32) {
      const int r = e / p.dq, d = e - r * p.dq;
      ks[r * (p.dq + 1) + d] = j0 + r < hi ? wa_f<T>(kb[(int64_t)(j0 + r) * p.kc_s + d]) : 0.f;
    }
    for (int e = threadIdx.x; e < WA_KEYS * p.dv; e += WA_WARPS * 32) {
      const int r = e / p.dv, d = e - r * p.dv;
      vs[e] = j0 + r < hi ? wa_f<T>(vb[(int64_t)(j0 + r) * p.vc_s + d]) : 0.f;
    }
    __syncthreads();
    const int j = j0 + lane;
    const bool seen = row_ok && j >= first && j <= me;
    if (!__any_sync(0xffffffffu, seen)) continue;
    float sc = -1e30f;
    if (seen) {
      sc = 0.f;
      const float* kr = ks + lane * (p.dq + 1);
      const float* qq = qs + warp * p.dq;
#pragma unroll 8
      for (int d = 0; d < p.dq; ++d) sc = fmaf(qq[d], kr[d], sc);
    }
    const float m_new = fmaxf(m, warp_max(sc)), sf = expf(m - m_new);
    const float pj = seen ? expf(sc - m_new) : 0.f;
    l = l * sf + warp_sum(pj);
#pragma unroll
    for (int i = 0; i < VPL; ++i) acc[i] *= sf;
    for (int jj = 0; jj < WA_KEYS; ++jj) {
      const float pv = __shfl_sync(0xffffffffu, pj, jj);
      if (pv == 0.f) continue;
#pragma unroll
      for (int i = 0; i < VPL; ++i)
        if (lane + 32 * i < p.dv) acc[i] = fmaf(pv, vs[jj * p.dv + lane + 32 * i], acc[i]);
    }
    m = m_new;
  }
  if (!row_ok) return;
  T* o = out + (((int64_t)b * p.S + s) * p.H + head) * p.dv;
#pragma unroll
  for (int i = 0; i < VPL; ++i)
    if (lane + 32 * i < p.dv) o[lane + 32 * i] = wa_t<T>(acc[i] / l);
}

template <typename T, int VPL>
static int launch_window(const void* q, const void* k, const void* v, void* out, const WindowParams& p) {
  const size_t smem = sizeof(float) * (WA_KEYS * (p.dq + 1) + WA_KEYS * p.dv + WA_WARPS * p.dq);
  KD_REQUIRE(smem <= 227 * 1024, "attention: heads of %d and %d are too wide", p.dq, p.dv);
  static bool configured[64] = {false};
  if (!configured[ctx().device & 63]) {
    KD_CUDA_CHECK(cudaFuncSetAttribute(window_attention_kernel<T, VPL>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
    configured[ctx().device & 63] = true;
  }
  const int64_t tiles = ((int64_t)p.S * (p.H / p.G) + WA_WARPS - 1) / WA_WARPS;
  KD_REQUIRE(p.G <= 65535 && p.B <= 65535 && tiles < (1ll << 31), "attention: too many heads, sequences or queries in one call");
  KD_CUDA_CHECK(launch_ex(window_attention_kernel<T, VPL>, dim3((unsigned)tiles, p.G, p.B), dim3(WA_WARPS * 32), smem, (const T*)q, (const T*)k, (const T*)v, (T*)out, p));
  return after_launch("window_attention_kernel");
}

template <typename T>
static int launch_window_size(const void* q, const void* k, const void* v, void* out, const WindowParams& p) {
  if (p.dv <= 64) return launch_window<T, 2>(q, k, v, out, p);
  if (p.dv <= 128) return launch_window<T, 4>(q, k, v, out, p);
  if (p.dv <= 256) return launch_window<T, 8>(q, k, v, out, p);
  if (p.dv <= 512) return launch_window<T, 16>(q, k, v, out, p);
  return fail(KD_ERR_UNSUPPORTED, "attention: values of %d numbers; this path handles up to 512", p.dv);
}

static int scalar_ptr(const kd_tensor* pos, const int** out) {
  *out = nullptr;
  if (!pos) return KD_OK;
  KD_REQUIRE(pos->dtype == KD_I32 && numel(pos) == 1, "position must be a device int32 scalar");
  void* p;
  KD_TRY(tensor_ptr(pos, &p));
  *out = static_cast<const int*>(p);
  return KD_OK;
}

static int norm_ptr(const kd_tensor* t, int64_t n, const char* what, const float** out) {
  KD_REQUIRE(t && t->dtype == KD_F32 && is_contiguous(t) && numel(t) == n, "%s must be contiguous fp32 [%lld]", what, (long long)n);
  void* p;
  KD_TRY(tensor_ptr(t, &p));
  *out = static_cast<const float*>(p);
  return KD_OK;
}

static bool tensor_core_heads(int dtype, int64_t dq, int64_t dv) { return dtype == KD_BF16 && dq == dv && (dq == 64 || dq == 128); }

}  // namespace kd

using namespace kd;

KD_API int kd_attention_head_sizes(int dtype, int dim, int vdim, int* q_size_out, int* v_size_out) {
  KD_REQUIRE(q_size_out && v_size_out && dim >= 1 && vdim >= 1, "bad argument");
  const int widest = dim > vdim ? dim : vdim;
  if (dtype == KD_BF16 && widest <= 128) {
    *q_size_out = *v_size_out = widest <= 64 ? 64 : 128;
    return KD_OK;
  }
  *q_size_out = dim;
  *v_size_out = vdim;
  return KD_OK;
}

KD_API int kd_qk_norm_rope_cache(const kd_tensor* proj, int q_col, int k_col, int v_col, int dim, int vdim, int rot_dim, const kd_tensor* q_norm,
                                 const kd_tensor* k_norm, float eps, const kd_tensor* cos, const kd_tensor* sin, const kd_tensor* k_cache,
                                 const kd_tensor* v_cache, const kd_tensor* pos_dev, int pos_host, const kd_tensor* q_out) {
  KD_TRY(require_init());
  KD_REQUIRE(proj && q_norm && cos && sin && k_cache && v_cache && q_out, "null tensor");
  KD_REQUIRE(proj->ndim == 3 && proj->strides[2] == 1 && proj->strides[0] == proj->strides[1] * proj->shape[1] && (proj->dtype == KD_BF16 || proj->dtype == KD_F32),
             "proj must be [B,S,N] with evenly spaced rows, bf16 or fp32");
  KD_REQUIRE(q_out->ndim == 4 && is_contiguous(q_out) && q_out->dtype == proj->dtype && q_out->shape[0] == proj->shape[0] && q_out->shape[1] == proj->shape[1],
             "q_out must be contiguous [B,S,H,D] of proj's type");
  for (const kd_tensor* t : {k_cache, v_cache})
    KD_REQUIRE(t->ndim == 4 && t->strides[3] == 1 && t->dtype == proj->dtype && t->shape[0] >= proj->shape[0], "caches must be [B,G,maxS,D] of proj's type");
  KD_REQUIRE(v_cache->shape[1] == k_cache->shape[1] && v_cache->shape[2] == k_cache->shape[2], "key and value cache differ");
  QkPrepParams p{};
  p.S = (int)proj->shape[1]; p.H = (int)q_out->shape[2]; p.G = (int)k_cache->shape[1]; p.dim = dim; p.vdim = vdim; p.rot = rot_dim;
  p.dq = (int)q_out->shape[3]; p.dv = (int)v_cache->shape[3]; p.max_s = (int)k_cache->shape[2];
  KD_REQUIRE(dim >= 1 && vdim >= 1 && rot_dim >= 0 && rot_dim % 2 == 0 && rot_dim <= dim, "%d rotated of %d dimensions", rot_dim, dim);
  KD_REQUIRE(p.dq >= dim && p.dv >= vdim && k_cache->shape[3] == p.dq, "heads of %d and %d do not fit rows of %d and %d", dim, vdim, p.dq, p.dv);
  const int64_t N = proj->shape[2];
  KD_REQUIRE(q_col >= 0 && q_col + (int64_t)p.H * dim <= N, "queries exceed the projection row");
  if (k_col >= 0) KD_REQUIRE(k_col + (int64_t)p.G * dim <= N && v_col >= 0 && v_col + (int64_t)p.G * vdim <= N, "keys or values exceed the projection row");
  p.q_col = q_col; p.k_col = k_col; p.v_col = v_col; p.ld = proj->strides[1];
  p.kc_b = k_cache->strides[0]; p.kc_h = k_cache->strides[1]; p.kc_s = k_cache->strides[2];
  p.vc_b = v_cache->strides[0]; p.vc_h = v_cache->strides[1]; p.vc_s = v_cache->strides[2];
  p.eps = eps;
  KD_TRY(norm_ptr(q_norm, (int64_t)p.H * dim, "q_norm", &p.qw));
  if (k_col >= 0) KD_TRY(norm_ptr(k_norm, (int64_t)p.G * dim, "k_norm", &p.kw));
  KD_REQUIRE(cos->dtype == KD_F32 && sin->dtype == KD_F32 && is_contiguous(cos) && is_contiguous(sin) && numel(cos) >= (int64_t)p.max_s * (rot_dim / 2) &&
                 numel(sin) >= (int64_t)p.max_s * (rot_dim / 2), "cos / sin must be fp32 [maxS, rot_dim/2]");
  void* t;
  KD_TRY(tensor_ptr(cos, &t)); p.cos_t = static_cast<const float*>(t);
  KD_TRY(tensor_ptr(sin, &t)); p.sin_t = static_cast<const float*>(t);
  KD_TRY(scalar_ptr(pos_dev, &p.pos_dev));
  p.pos_host = pos_host;
  if (!pos_dev) KD_REQUIRE(pos_host >= 0 && pos_host + p.S <= p.max_s, "Cache overflow: trying to write to position %d-%d, but maxSeqLen is %d", pos_host, pos_host + p.S, p.max_s);
  p.err = ctx().error_flag;
  const int64_t tokens = proj->shape[0] * proj->shape[1];
  if (tokens == 0) return KD_OK;
  void *pp, *pq, *pk, *pv;
  KD_TRY(tensor_ptr(proj, &pp));
  KD_TRY(tensor_ptr(q_out, &pq));
  KD_TRY(tensor_ptr(k_cache, &pk));
  KD_TRY(tensor_ptr(v_cache, &pv));
  const uintptr_t all = reinterpret_cast<uintptr_t>(pp) | reinterpret_cast<uintptr_t>(pq) | reinterpret_cast<uintptr_t>(pk) | reinterpret_cast<uintptr_t>(pv) |
                        reinterpret_cast<uintptr_t>(p.qw) | reinterpret_cast<uintptr_t>(p.kw);
  auto m8 = [](int64_t a, int64_t b, int64_t c, int64_t d) { return (a | b | c | d) % 8 == 0; };
  p.vec = (all & 15) == 0 && m8(dim, vdim, q_col, p.ld) && (k_col < 0 || m8(k_col, v_col, 0, 0)) && m8(p.dq, p.dv, p.kc_b, p.kc_h) && m8(p.kc_s, p.vc_b, p.vc_h, p.vc_s);
  const size_t smem = sizeof(float) * (size_t)(p.H + p.G) * dim;
  KD_REQUIRE(smem <= 200 * 1024, "%d heads of %d are too wide for one token's rows", p.H + p.G, dim);
  static bool configured[64] = {false};
  if (!configured[ctx().device & 63]) {
    KD_CUDA_CHECK(cudaFuncSetAttribute(qk_prep_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    KD_CUDA_CHECK(cudaFuncSetAttribute(qk_prep_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    configured[ctx().device & 63] = true;
  }
  if (proj->dtype == KD_BF16)
    KD_CUDA_CHECK(launch_ex(qk_prep_kernel<__nv_bfloat16>, dim3((unsigned)tokens), dim3(QK_THREADS), smem, (const __nv_bfloat16*)pp, (__nv_bfloat16*)pq, (__nv_bfloat16*)pk, (__nv_bfloat16*)pv, p));
  else
    KD_CUDA_CHECK(launch_ex(qk_prep_kernel<float>, dim3((unsigned)tokens), dim3(QK_THREADS), smem, (const float*)pp, (float*)pq, (float*)pk, (float*)pv, p));
  return after_launch("qk_prep_kernel");
}

KD_API int kd_window_attention(const kd_tensor* q, const kd_tensor* k_cache, const kd_tensor* v_cache, const kd_tensor* sink, float scale, int window,
                               const kd_tensor* pos_dev, int pos_host, const kd_tensor* out) {
  KD_TRY(require_init());
  KD_REQUIRE(q && k_cache && v_cache && out, "null tensor");
  KD_REQUIRE(q->ndim == 4 && is_contiguous(q) && (q->dtype == KD_BF16 || q->dtype == KD_F32), "q must be contiguous [B,S,H,D], bf16 or fp32");
  for (const kd_tensor* t : {k_cache, v_cache})
    KD_REQUIRE(t->ndim == 4 && t->strides[3] == 1 && t->dtype == q->dtype && t->shape[0] >= q->shape[0], "caches must be [B,G,maxS,D] of q's type");
  WindowParams p{};
  p.B = (int)q->shape[0]; p.S = (int)q->shape[1]; p.H = (int)q->shape[2]; p.G = (int)k_cache->shape[1];
  p.dq = (int)q->shape[3]; p.dv = (int)v_cache->shape[3]; p.max_s = (int)k_cache->shape[2];
  KD_REQUIRE(p.G >= 1 && p.H % p.G == 0, "%d query heads over %d key heads", p.H, p.G);
  KD_REQUIRE(k_cache->shape[3] == p.dq && v_cache->shape[1] == p.G && v_cache->shape[2] == p.max_s, "caches and queries do not match");
  KD_REQUIRE(out->dtype == q->dtype && is_contiguous(out) && numel(out) == (int64_t)p.B * p.S * p.H * p.dv, "out must be contiguous [B*S, H*vdim] of q's type");
  KD_REQUIRE(window >= 0, "window %d", window);
  p.window = window;
  p.kc_b = k_cache->strides[0]; p.kc_h = k_cache->strides[1]; p.kc_s = k_cache->strides[2];
  p.vc_b = v_cache->strides[0]; p.vc_h = v_cache->strides[1]; p.vc_s = v_cache->strides[2];
  p.scale = scale;
  if (sink) KD_TRY(norm_ptr(sink, p.H, "sink", &p.sink));
  KD_TRY(scalar_ptr(pos_dev, &p.pos_dev));
  p.pos_host = pos_host;
  if (!pos_dev) KD_REQUIRE(pos_host >= 0 && pos_host + p.S <= p.max_s, "queries at %d-%d exceed the cache of %d rows", pos_host, pos_host + p.S, p.max_s);
  if (p.B == 0 || p.S == 0) return KD_OK;
  void *pq, *pk, *pv, *po;
  KD_TRY(tensor_ptr(q, &pq));
  KD_TRY(tensor_ptr(k_cache, &pk));
  KD_TRY(tensor_ptr(v_cache, &pv));
  KD_TRY(tensor_ptr(out, &po));
  const bool aligned = ((reinterpret_cast<uintptr_t>(pq) | reinterpret_cast<uintptr_t>(pk) | reinterpret_cast<uintptr_t>(pv) | reinterpret_cast<uintptr_t>(po)) & 15) == 0 &&
                       (p.kc_b | p.kc_h | p.kc_s | p.vc_b | p.vc_h | p.vc_s) % 8 == 0;
  if (tensor_core_heads(q->dtype, p.dq, p.dv) && aligned && scale > 0.f && p.H <= 65535 && p.B <= 65535) {
    if (p.S == 1 && p.H / p.G <= 16) {
      WindowDecode d{};
      d.B = p.B; d.H = p.H; d.G = p.G; d.D = p.dq; d.max_s = p.max_s; d.window = window; d.scale = scale; d.sink = p.sink;
      d.pos_dev = p.pos_dev; d.pos_host = pos_host;
      d.kc[0] = p.kc_b; d.kc[1] = p.kc_h; d.kc[2] = p.kc_s; d.vc[0] = p.vc_b; d.vc[1] = p.vc_h; d.vc[2] = p.vc_s;
      return attention_decode_window(pq, pk, pv, po, d);
    }
    if (!p.pos_dev) {
      AttnParams a{};
      a.B = p.B; a.Hq = p.H; a.Hkv = p.G; a.Sq = p.S; a.Skv = pos_host + p.S; a.D = p.dq;
      a.sq[0] = (int64_t)p.S * p.H * p.dq; a.sq[1] = p.dq; a.sq[2] = (int64_t)p.H * p.dq; a.sq[3] = 1;
      a.so[0] = (int64_t)p.S * p.H * p.dv; a.so[1] = p.dv; a.so[2] = (int64_t)p.H * p.dv; a.so[3] = 1;
      a.sk[0] = p.kc_b; a.sk[1] = p.kc_h; a.sk[2] = p.kc_s; a.sk[3] = 1;
      a.sv[0] = p.vc_b; a.sv[1] = p.vc_h; a.sv[2] = p.vc_s; a.sv[3] = 1;
      a.scale = scale;
      a.causal = 1;
      return attention_prefill2_window(pq, pk, pv, po, a, pos_host, window, p.sink);
    }
  }
  if (q->dtype == KD_BF16) return launch_window_size<__nv_bfloat16>(pq, pk, pv, po, p);
  return launch_window_size<float>(pq, pk, pv, po, p);
}
