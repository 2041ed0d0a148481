// Latent attention: keys and values of all heads are linear images of one cached row per token,
// (c, k_rot): a normed latent of kv_rank numbers and one rotated key part shared by all heads.
//
//   kd_latent_prep       RMSNorm of the latent, rotary positions (interleaved pairs) on the shared key
//                        part and, in place, on the rotated part of every query; writes the cache row.
//   kd_latent_absorb     q_abs = (W_uk^T q_unrotated, q_rotated): with it a score is q_abs . (c, k_rot),
//                        so attention runs over the cache rows themselves, all heads sharing one key.
//   kd_latent_attention  split-KV attention over the cache with rows (query, head): partial sums
//                        sum_j p_j c_j, running maxima and sums per split.
//   kd_latent_values     combines the splits (the sink enters the denominator here: exp(sink) with no
//                        key and no value) and applies W_uv per head.  In bf16 both per-head products run
//                        through head_linear_kernel: mma.sync on fragments loaded straight from global
//                        memory, one latency for a decode step's few rows.
// This is the decode path, the path of short portions, and the fp32 path.  Long bf16 prompts expand
// keys and values once and use the tcgen05 prefill kernel (attention_prefill2.cu).
//
// bf16 kernel: a CTA owns 16 (or 32) query-head rows and a range of key tiles.  A key tile (64 cache
// rows) arrives once by TMA (128-byte swizzled slabs of 64 columns, two-stage mbarrier ring) and serves both products: S = Q K^T reads it
// K-major, O += P V reads its first kv_rank columns transposed (ldmatrix.trans).  Warps split S by
// 4 key groups x 2 halves of the depth, and O by columns.  mma.sync is used on purpose: a decode step
// has as many query rows as heads, the tcgen05 tile would be 7/8 padding and its 512-column fp32
// accumulator would fill tensor memory; the kernel is bound by streaming the cache from HBM.
// Roofline for decode: HBM, ctx * (kv_rank + rot_dim) * 2 bytes per sequence.
#include "common.cuh"
#include "kernels.cuh"
#include "sm100.cuh"

namespace kd {

using sm100::smem_u32;

constexpr float LOG2E = 1.4426950408889634f;

template <typename T> __device__ __forceinline__ float to_f(T v);
template <> __device__ __forceinline__ float to_f<float>(float v) { return v; }
template <> __device__ __forceinline__ float to_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

// ----------------------------------------------------------------------------- prep
struct PrepParams {
  int S, H, dim, rot, rank, max_s;
  int q_col, kv_col;            // column of the first query / latent entry in a projection row (kv_col < 0: queries only)
  int64_t ld;                   // projection row stride
  int64_t cache_b, cache_s;     // cache strides: sequence, row
  int64_t ld_dense;             // dense latent rows (0: none)
  float eps;
  const float* norm_w;
  const float* cos_t;           // [max_s, rot/2]
  const float* sin_t;
  const int* pos_dev;
  int pos_host;
  int* err;
};

// One CTA per token.
template <typename T>
__global__ void latent_prep_kernel(T* __restrict__ proj, T* __restrict__ cache, T* __restrict__ dense, PrepParams p) {
  __shared__ float red[8];
  pdl_wait();
  pdl_trigger();
  const int64_t token = blockIdx.x;
  const int b = (int)(token / p.S), s = (int)(token - (int64_t)b * p.S);
  const int pos = (p.pos_dev ? *p.pos_dev : p.pos_host) + s;
  if (pos < 0 || pos >= p.max_s) {    // never read or write outside the tables and the cache; report instead
    if (threadIdx.x == 0 && atomicCAS(p.err, 0, 102) == 0) { p.err[1] = pos; p.err[2] = p.max_s; }
    return;
  }
  T* row = proj + token * p.ld;
  const float* cs = p.cos_t + (int64_t)pos * (p.rot / 2);
  const float* sn = p.sin_t + (int64_t)pos * (p.rot / 2);
  const int half = p.rot / 2;
  for (int i = threadIdx.x; i < p.H * half; i += blockDim.x) {
    const int h = i / half, e = i - h * half;
    T* q = row + p.q_col + (int64_t)h * (p.dim + p.rot) + p.dim + 2 * e;
    const float u = to_f<T>(q[0]), v = to_f<T>(q[1]), c = cs[e], d = sn[e];
    q[0] = from_f<T>(u * c - v * d);
    q[1] = from_f<T>(v * c + u * d);
  }
  if (p.kv_col < 0) return;
  const T* kv = row + p.kv_col;
  T* dst = cache + (int64_t)b * p.cache_b + (int64_t)pos * p.cache_s;
  float ss = 0.f;
  for (int i = threadIdx.x; i < p.rank; i += blockDim.x) { const float v = to_f<T>(kv[i]); ss = fmaf(v, v, ss); }
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  ss = 0.f;
  for (int w = 0; w < (int)(blockDim.x >> 5); ++w) ss += red[w];
  const float inv = 1.0f / sqrtf(ss / (float)p.rank + p.eps);
  for (int i = threadIdx.x; i < p.rank; i += blockDim.x) {
    const T v = from_f<T>(to_f<T>(kv[i]) * inv * p.norm_w[i]);
    dst[i] = v;
    if (p.ld_dense) dense[token * p.ld_dense + i] = v;
  }
  for (int e = threadIdx.x; e < half; e += blockDim.x) {
    const float u = to_f<T>(kv[p.rank + 2 * e]), v = to_f<T>(kv[p.rank + 2 * e + 1]), c = cs[e], d = sn[e];
    dst[p.rank + 2 * e] = from_f<T>(u * c - v * d);
    dst[p.rank + 2 * e + 1] = from_f<T>(v * c + u * d);
  }
}

// ----------------------------------------------------------------------------- absorb
// q_abs[t, h, r] = sum_d q[t, h, d] W_uk[h, d, r]; then the rotated part, then zeros up to the padded width.
constexpr int ABS_TOK = 8;

template <typename T>
__global__ void __launch_bounds__(128)
latent_absorb_kernel(const T* __restrict__ q, int64_t ld, int q_col, const T* __restrict__ wuk, int T_total, int H, int dim, int rot, int rank,
                     int width, T* __restrict__ out) {
  extern __shared__ float qs[];       // [dim][ABS_TOK]
  pdl_wait();
  pdl_trigger();
  const int h = blockIdx.x, t0 = blockIdx.z * ABS_TOK;
  for (int i = threadIdx.x; i < dim * ABS_TOK; i += blockDim.x) {
    const int d = i / ABS_TOK, t = i - d * ABS_TOK;
    qs[i] = t0 + t < T_total ? to_f<T>(q[(int64_t)(t0 + t) * ld + q_col + (int64_t)h * (dim + rot) + d]) : 0.f;
  }
  __syncthreads();
  const int r = blockIdx.y * blockDim.x + threadIdx.x;
  if (r < rank) {
    float acc[ABS_TOK];
#pragma unroll
    for (int t = 0; t < ABS_TOK; ++t) acc[t] = 0.f;
    const T* w = wuk + (int64_t)h * dim * rank + r;
#pragma unroll 8
    for (int d = 0; d < dim; ++d) {
      const float wv = to_f<T>(w[(int64_t)d * rank]);
      const float4 a = *reinterpret_cast<const float4*>(qs + d * ABS_TOK), b = *reinterpret_cast<const float4*>(qs + d * ABS_TOK + 4);
      acc[0] = fmaf(a.x, wv, acc[0]); acc[1] = fmaf(a.y, wv, acc[1]); acc[2] = fmaf(a.z, wv, acc[2]); acc[3] = fmaf(a.w, wv, acc[3]);
      acc[4] = fmaf(b.x, wv, acc[4]); acc[5] = fmaf(b.y, wv, acc[5]); acc[6] = fmaf(b.z, wv, acc[6]); acc[7] = fmaf(b.w, wv, acc[7]);
    }
#pragma unroll
    for (int t = 0; t < ABS_TOK; ++t)
      if (t0 + t < T_total) out[((int64_t)(t0 + t) * H + h) * width + r] = from_f<T>(acc[t]);
  } else if (r < width) {
    for (int t = 0; t < ABS_TOK && t0 + t < T_total; ++t)
      out[((int64_t)(t0 + t) * H + h) * width + r] =
          r < rank + rot ? q[(int64_t)(t0 + t) * ld + q_col + (int64_t)h * (dim + rot) + dim + (r - rank)] : from_f<T>(0.f);
  }
}

// ----------------------------------------------------------------------------- per-head linear (bf16)
__device__ __forceinline__ void mma16816(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

// out[t, h, n] = sum_k x[t, h, k] W[h, n, k] for 32 tokens a CTA, 8 columns a warp group.  The order of k inside
// a product is free as long as both operands agree, so a lane loads eight consecutive k of its row (16 bytes)
// and uses them as the fragments of two k-steps: no shared memory, every load independent of the others.
// KW warps share a column tile and split K.  Columns from N on (q_abs): the rotated part of x, then zeros.
struct HeadLinearParams {
  int T, H, N, K, n_out;
  int64_t x_t, x_h;           // strides of x
  int64_t o_t, o_h;           // strides of out
  int tail_col, tail_len;     // column n >= N of out = x[tail_col + n - N] for n - N < tail_len, else 0
};

constexpr int HL_WARPS = 4;

template <int KW>
__global__ void __launch_bounds__(HL_WARPS * 32)
head_linear_kernel(const __nv_bfloat16* __restrict__ x, const __nv_bfloat16* __restrict__ w, __nv_bfloat16* __restrict__ out, HeadLinearParams p) {
  constexpr int NT = HL_WARPS / KW;            // column tiles per CTA
  __shared__ float red[KW > 1 ? HL_WARPS : 1][32][9];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y, t0 = blockIdx.z * 32;
  const int tile = blockIdx.x * NT + warp / KW, kw = warp % KW;
  const int n0 = tile * 8, g = lane >> 2, q = lane & 3;
  const bool product = n0 < p.N;
  const int per = (p.K / 32 + KW - 1) / KW, k0 = kw * per, k1 = min(p.K / 32, k0 + per);
  pdl_wait();
  pdl_trigger();
  float acc[2][4] = {};
  if (product) {
    const __nv_bfloat16* wr = w + ((int64_t)h * p.N + n0 + g) * p.K + q * 8;
    const __nv_bfloat16* xr[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) xr[i] = x + (int64_t)min(t0 + g + 8 * i, p.T - 1) * p.x_t + (int64_t)h * p.x_h + q * 8;
#pragma unroll 4
    for (int k = k0; k < k1; ++k) {
      const uint4 b = *reinterpret_cast<const uint4*>(wr + k * 32);
      uint4 a[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) a[i] = *reinterpret_cast<const uint4*>(xr[i] + k * 32);
#pragma unroll
      for (int m = 0; m < 2; ++m) {
        mma16816(acc[m], a[2 * m].x, a[2 * m + 1].x, a[2 * m].y, a[2 * m + 1].y, b.x, b.y);
        mma16816(acc[m], a[2 * m].z, a[2 * m + 1].z, a[2 * m].w, a[2 * m + 1].w, b.z, b.w);
      }
    }
  }
  if (KW > 1) {
#pragma unroll
    for (int m = 0; m < 2; ++m)
#pragma unroll
      for (int e = 0; e < 4; ++e) red[warp][m * 16 + g + (e >> 1) * 8][q * 2 + (e & 1)] = acc[m][e];
    __syncthreads();
    if (kw != 0) return;
#pragma unroll
    for (int m = 0; m < 2; ++m)
#pragma unroll
      for (int e = 0; e < 4; ++e)
#pragma unroll
        for (int o = 1; o < KW; ++o) acc[m][e] += red[warp + o][m * 16 + g + (e >> 1) * 8][q * 2 + (e & 1)];
  }
#pragma unroll
  for (int m = 0; m < 2; ++m)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int t = t0 + m * 16 + g + e * 8, n = n0 + q * 2;
      if (t >= p.T || n >= p.n_out) continue;
      __nv_bfloat162 v = __floats2bfloat162_rn(acc[m][2 * e], acc[m][2 * e + 1]);
      if (!product) {
        const __nv_bfloat16* tail = x + (int64_t)t * p.x_t + (int64_t)h * p.x_h + p.tail_col + (n - p.N);
        v.x = n - p.N < p.tail_len ? tail[0] : __float2bfloat16_rn(0.f);
        v.y = n + 1 - p.N < p.tail_len ? tail[1] : __float2bfloat16_rn(0.f);
      }
      *reinterpret_cast<__nv_bfloat162*>(out + (int64_t)t * p.o_t + (int64_t)h * p.o_h + n) = v;
    }
}

template <int KW>
static int launch_head_linear(const void* x, const void* w, void* out, const HeadLinearParams& p) {
  constexpr int NT = HL_WARPS / KW;
  const int64_t z = (p.T + 31) / 32;
  KD_REQUIRE(z <= 65535 && p.H <= 65535, "per-head linear: %d tokens in one call", p.T);
  dim3 grid(((p.n_out + 7) / 8 + NT - 1) / NT, p.H, (unsigned)z);
  KD_CUDA_CHECK(launch_ex(head_linear_kernel<KW>, grid, dim3(HL_WARPS * 32), 0, (const __nv_bfloat16*)x, (const __nv_bfloat16*)w, (__nv_bfloat16*)out, p));
  return after_launch("head_linear_kernel");
}

// ----------------------------------------------------------------------------- attention over cache rows
struct LatAttnParams {
  int B, S, H, rank, width, max_s, splits;
  int rows;                     // S * H
  int64_t cache_b, cache_s;
  float scale_log2;
  const int* pos_dev;
  int pos_host;
  float* part_o;                // [B, rows, splits, rank]
  float* part_ml;               // [B, rows, splits, 2]
  int* err;
};

__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], const void* p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
// row stride of the shared-memory tiles: 16 bytes more than a multiple of 128, so that the eight rows
// of an ldmatrix fall into different banks
__host__ __device__ constexpr int lat_stride(int width) { return (width + 63) / 64 * 64 + 8; }

constexpr int LAT_THREADS = 256;

// MT: 16-row query tiles per CTA; KT: keys per tile; NT: 8-column output tiles per warp (even); QR: k-steps of the
// query tile that a warp keeps in registers (0: it re-reads them from shared memory).
template <int MT, int KT, int NT, int QR>
__global__ void __launch_bounds__(LAT_THREADS, MT == 1 && KT == 32 && NT <= 8 ? 2 : 1)
latent_attention_bf16_kernel(const __nv_bfloat16* __restrict__ q_abs, const __grid_constant__ CUtensorMap tmap, LatAttnParams p) {
  constexpr int ROWS = MT * 16;
  constexpr int KG = KT / 4;                 // keys per warp in S (two warps share a key group, each half of the depth)
  constexpr int TPR = LAT_THREADS / ROWS;    // softmax threads per row
  constexpr int KPT = KT / TPR;              // keys per softmax thread
  constexpr int PST = KT + 8;                // row stride of P
  constexpr int SLAB = KT * 128;             // bytes of a slab: KT rows of 64 columns
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int st = lat_stride(p.width), slabs = (p.width + 63) / 64;
  uint8_t* ks = smem;                                                       // [2][slabs][SLAB]
  __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(smem + 2 * slabs * SLAB);   // [ROWS][st]
  float* ss = reinterpret_cast<float*>(qs + ROWS * st);                     // [2][ROWS][KT]
  __nv_bfloat16* ps = reinterpret_cast<__nv_bfloat16*>(ss + 2 * ROWS * KT); // [ROWS][PST]
  float* al = reinterpret_cast<float*>(ps + ROWS * PST);                    // [ROWS] rescale factors
  uint64_t* full = reinterpret_cast<uint64_t*>(al + ROWS);                  // [2]
  volatile int* abort_flag = reinterpret_cast<volatile int*>(full + 2);

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int b = blockIdx.z, split = blockIdx.x, row0 = blockIdx.y * ROWS;
  pdl_wait();
  pdl_trigger();
  const int pos0 = p.pos_dev ? *p.pos_dev : p.pos_host;
  const int ctx = min(pos0 + p.S, p.max_s);
  // the last row of this CTA sees keys 0 .. pos0 + s_last
  const int s_last = min(row0 + ROWS - 1, p.rows - 1) / p.H;
  const int n_tiles_all = (ctx + KT - 1) / KT;
  const int per_split = (n_tiles_all + p.splits - 1) / p.splits;
  const int t_begin = split * per_split;
  const int t_end = min(min(n_tiles_all, t_begin + per_split), (min(ctx, pos0 + s_last + 1) + KT - 1) / KT);
  const int n_t = t_end - t_begin;

  const int wc = p.width / 8;                // 16-byte chunks per row
  auto load_tile = [&](int t, int buf) {     // one thread
    sm100::mbar_arrive_expect_tx(&full[buf], (uint32_t)(slabs * SLAB));
    for (int i = 0; i < slabs; ++i) sm100::tma_load_3d(ks + (buf * slabs + i) * SLAB, &tmap, &full[buf], i * 64, t * KT, b);
  };
  // address of 8 columns (16 bytes) of a row: chunks of a 128-byte row are permuted by the row's low bits
  auto tile_at = [&](const uint8_t* tile, int row, int col) { return tile + (col >> 6) * SLAB + row * 128 + ((((col >> 3) & 7) ^ (row & 7)) << 4); };
  if (tid == 0) {
    sm100::mbar_init(&full[0], 1);
    sm100::mbar_init(&full[1], 1);
    *abort_flag = 0;
    sm100::fence_mbar_init();
  }
  __syncthreads();
  if (tid == 0 && n_t > 0) {
    load_tile(t_begin, 0);
    if (n_t > 1) load_tile(t_begin + 1, 1);
  }
  for (int i = tid; i < ROWS * wc; i += LAT_THREADS) {
    const int r = i / wc, c = i - r * wc;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (row0 + r < p.rows) v = *reinterpret_cast<const uint4*>(q_abs + ((int64_t)b * p.rows + row0 + r) * p.width + c * 8);
    *reinterpret_cast<uint4*>(qs + r * st + c * 8) = v;
  }
  __syncthreads();

  float o[MT][NT][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[m][n][e] = 0.f;
  const int sr = tid / TPR, sk = (tid % TPR) * KPT;     // softmax: my row, my first key
  const int last_key = row0 + sr < p.rows ? pos0 + (row0 + sr) / p.H : -1;
  float m_run = -1e30f, l_run = 0.f;
  const int kg = warp & 3, kh = warp >> 2;
  const int ksteps = p.width / 16;
  const int ks0 = kh * ((ksteps + 1) / 2), ks1 = kh ? ksteps : (ksteps + 1) / 2;

  uint32_t qr[QR > 0 ? QR : 1][MT][4];
  if (QR > 0) {
#pragma unroll
    for (int k = 0; k < QR; ++k)
      if (k < ks1 - ks0)
#pragma unroll
        for (int m = 0; m < MT; ++m) ldsm4(qr[k][m], qs + (m * 16 + (lane & 15)) * st + (ks0 + k) * 16 + (lane >> 4) * 8);
  }

  int gave_up = -1;
  for (int it = 0; it < n_t; ++it) {
    const int buf = it & 1;
    // (every warp must come to the same answer before it leaves the loop: a wait that ran out ends all of them)
    const bool arrived = sm100::mbar_wait(&full[buf], (uint32_t)((it >> 1) & 1), abort_flag, p.err, 701);
    if (!__syncthreads_and(arrived)) { gave_up = it; break; }
    uint8_t* kt = ks + buf * slabs * SLAB;
    const int valid = ctx - (t_begin + it) * KT;       // rows past the context hold anything: they must not meet P = 0
    if (valid < KT) {
      for (int i = tid; i < (KT - valid) * slabs * 8; i += LAT_THREADS)
        *reinterpret_cast<uint4*>(kt + (i / ((KT - valid) * 8)) * SLAB + valid * 128 + (i % ((KT - valid) * 8)) * 16) = make_uint4(0, 0, 0, 0);
      __syncthreads();
    }
    // S: this warp's keys kg*KG.., depth steps ks0..ks1
    float sacc[MT][KG / 8][4];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int n = 0; n < KG / 8; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) sacc[m][n][e] = 0.f;
    auto score_step = [&](const uint32_t (&a)[MT][4], int k) {
      uint32_t bb[4];
      // lanes 0-7 / 8-15: keys 0-7, depth 0-7 / 8-15; lanes 16-31: keys 8-15 (or, with 8 keys, a repeat)
      const int krow = kg * KG + (lane & 7) + (KG == 16 ? (lane >> 4) * 8 : 0);
      ldsm4(bb, tile_at(kt, krow, k * 16 + ((lane >> 3) & 1) * 8));
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        mma16816(sacc[m][0], a[m][0], a[m][1], a[m][2], a[m][3], bb[0], bb[1]);
        if (KG == 16) mma16816(sacc[m][KG / 8 - 1], a[m][0], a[m][1], a[m][2], a[m][3], bb[2], bb[3]);
      }
    };
    if (QR > 0) {
#pragma unroll
      for (int k = 0; k < QR; ++k)
        if (k < ks1 - ks0) score_step(qr[k], ks0 + k);
    } else if (KG == 8) {
      // two k-steps per key fragment load, a chain of products each
      float odd[MT][4] = {};
#pragma unroll 3
      for (int k = ks0; k < ks1; k += 2) {
        const bool two = k + 1 < ks1;
        uint32_t a[MT][4], c[MT][4], bb[4];
        ldsm4(bb, tile_at(kt, kg * 8 + (lane & 7), (two ? k + (lane >> 4) : k) * 16 + ((lane >> 3) & 1) * 8));
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          const __nv_bfloat16* qrow = qs + (m * 16 + (lane & 15)) * st + k * 16 + (lane >> 4) * 8;
          ldsm4(a[m], qrow);
          ldsm4(c[m], two ? qrow + 16 : qrow);
          mma16816(sacc[m][0], a[m][0], a[m][1], a[m][2], a[m][3], bb[0], bb[1]);
          if (two) mma16816(odd[m], c[m][0], c[m][1], c[m][2], c[m][3], bb[2], bb[3]);
        }
      }
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int e = 0; e < 4; ++e) sacc[m][0][e] += odd[m][e];
    } else {
#pragma unroll 4
      for (int k = ks0; k < ks1; ++k) {
        uint32_t a[MT][4];
#pragma unroll
        for (int m = 0; m < MT; ++m) ldsm4(a[m], qs + (m * 16 + (lane & 15)) * st + k * 16 + (lane >> 4) * 8);
        score_step(a, k);
      }
    }
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int n = 0; n < KG / 8; ++n) {
        const int r = m * 16 + (lane >> 2), c = kg * KG + n * 8 + (lane & 3) * 2;
        *reinterpret_cast<float2*>(ss + (kh * ROWS + r) * KT + c) = make_float2(sacc[m][n][0], sacc[m][n][1]);
        *reinterpret_cast<float2*>(ss + (kh * ROWS + r + 8) * KT + c) = make_float2(sacc[m][n][2], sacc[m][n][3]);
      }
    __syncthreads();
    {
      float v[KPT], mx = -1e30f;
      const int key0 = (t_begin + it) * KT + sk;
#pragma unroll
      for (int i = 0; i < KPT; ++i) {
        v[i] = (ss[sr * KT + sk + i] + ss[(ROWS + sr) * KT + sk + i]) * p.scale_log2;
        if (key0 + i > last_key || key0 + i >= ctx) v[i] = -1e30f;
        mx = fmaxf(mx, v[i]);
      }
#pragma unroll
      for (int off = TPR / 2; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
      const float m_new = fmaxf(m_run, mx);
      const float alpha = exp2f(m_run - m_new);
      float sum = 0.f;
#pragma unroll
      for (int i = 0; i < KPT; ++i) {
        const float e = v[i] > -1e29f ? exp2f(v[i] - m_new) : 0.f;
        sum += e;
        ps[sr * PST + sk + i] = __float2bfloat16_rn(e);
      }
#pragma unroll
      for (int off = TPR / 2; off > 0; off >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, off);
      l_run = l_run * alpha + sum;
      m_run = m_new;
      if (tid % TPR == 0) al[sr] = alpha;
    }
    __syncthreads();
    // O: this warp's columns warp*NT*8 ..
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const float a0 = al[m * 16 + (lane >> 2)], a1 = al[m * 16 + (lane >> 2) + 8];
#pragma unroll
      for (int n = 0; n < NT; ++n) { o[m][n][0] *= a0; o[m][n][1] *= a0; o[m][n][2] *= a1; o[m][n][3] *= a1; }
    }
    // column tile warp NT + n (+ 1 for the upper lanes): for NT <= 8 a warp's tiles lie in one slab and their chunk
    // bits differ by an XOR with n alone
    const uint8_t* vrow = kt + ((warp * NT) >> 3) * SLAB + (lane & 15) * 128;
    const int vx = ((((warp * NT) & 7) | (lane >> 4)) ^ (lane & 7)) << 4;
#pragma unroll
    for (int k = 0; k < KT / 16; ++k) {
      uint32_t a[MT][4];
#pragma unroll
      for (int m = 0; m < MT; ++m) ldsm4(a[m], ps + (m * 16 + (lane & 15)) * PST + k * 16 + (lane >> 4) * 8);
#pragma unroll
      for (int n = 0; n < NT; n += 2) {
        const int col = (warp * NT + n) * 8;
        if (col >= p.rank) break;
        uint32_t bb[4];        // keys 0-7 / 8-15 of 8 columns, then of the next 8
        if (NT <= 8) ldsm4t(bb, vrow + k * 2048 + (vx ^ (n << 4)));
        else ldsm4t(bb, tile_at(kt, k * 16 + (lane & 15), col + (lane >> 4) * 8));
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          mma16816(o[m][n], a[m][0], a[m][1], a[m][2], a[m][3], bb[0], bb[1]);
          mma16816(o[m][n + 1], a[m][0], a[m][1], a[m][2], a[m][3], bb[2], bb[3]);
        }
      }
    }
    __syncthreads();       // every warp is done with the tile: its buffer may be refilled
    if (tid == 0 && it + 2 < n_t) load_tile(t_begin + it + 2, buf);
  }
  if (gave_up >= 0 && tid == 0) {   // let the copies in flight land before the block leaves its shared memory
    for (int t = gave_up; t < min(gave_up + 2, n_t); ++t)
      for (int n = 0; n < (1 << 20) && !sm100::mbar_try_wait(&full[t & 1], (uint32_t)((t >> 1) & 1)); ++n) {}
  }

  if (tid % TPR == 0 && row0 + sr < p.rows) {
    float* ml = p.part_ml + (((int64_t)b * p.rows + row0 + sr) * p.splits + split) * 2;
    ml[0] = m_run;
    ml[1] = l_run;
  }
  if (n_t <= 0) return;       // an empty split: its rows are never read (sum 0)
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = row0 + m * 16 + (lane >> 2) + (e >> 1) * 8, c = (warp * NT + n) * 8 + (lane & 3) * 2 + (e & 1);
        if (r < p.rows && c < p.rank) p.part_o[(((int64_t)b * p.rows + r) * p.splits + split) * p.rank + c] = o[m][n][e];
      }
}

// Exact fp32 form: 8 rows per CTA, 32-key tiles, every product on the CUDA cores.
constexpr int LF_ROWS = 8, LF_KEYS = 32;

__global__ void __launch_bounds__(256)
latent_attention_f32_kernel(const float* __restrict__ q_abs, const float* __restrict__ cache, LatAttnParams p) {
  extern __shared__ float sm[];
  const int st = p.width + 1;
  float* qs = sm;                         // [LF_ROWS][st]
  float* ks = qs + LF_ROWS * st;          // [LF_KEYS][st]
  float* pr = ks + LF_KEYS * st;          // [LF_ROWS][LF_KEYS]
  float* os = pr + LF_ROWS * LF_KEYS;     // [LF_ROWS][rank]
  float* al = os + LF_ROWS * p.rank;      // [LF_ROWS]
  const int tid = threadIdx.x;
  const int b = blockIdx.z, split = blockIdx.x, row0 = blockIdx.y * LF_ROWS;
  pdl_wait();
  pdl_trigger();
  const int pos0 = p.pos_dev ? *p.pos_dev : p.pos_host;
  const int ctx = min(pos0 + p.S, p.max_s);
  const int s_last = min(row0 + LF_ROWS - 1, p.rows - 1) / p.H;
  const int n_all = (ctx + LF_KEYS - 1) / LF_KEYS;
  const int per_split = (n_all + p.splits - 1) / p.splits;
  const int t_begin = split * per_split;
  const int t_end = min(min(n_all, t_begin + per_split), (min(ctx, pos0 + s_last + 1) + LF_KEYS - 1) / LF_KEYS);
  for (int i = tid; i < LF_ROWS * p.width; i += blockDim.x) {
    const int r = i / p.width, c = i - r * p.width;
    qs[r * st + c] = row0 + r < p.rows ? q_abs[((int64_t)b * p.rows + row0 + r) * p.width + c] : 0.f;
  }
  for (int i = tid; i < LF_ROWS * p.rank; i += blockDim.x) os[i] = 0.f;
  const int r = tid >> 5, key = tid & 31;     // one warp per row, one key per lane
  const int last_key = row0 + r < p.rows ? pos0 + (row0 + r) / p.H : -1;
  float m_run = -1e30f, l_run = 0.f;
  for (int t = t_begin; t < t_end; ++t) {
    __syncthreads();
    for (int i = tid; i < LF_KEYS * p.width; i += blockDim.x) {
      const int kr = i / p.width, c = i - kr * p.width;
      ks[kr * st + c] = cache[(int64_t)b * p.cache_b + (int64_t)min(t * LF_KEYS + kr, ctx - 1) * p.cache_s + c];
    }
    __syncthreads();
    float s = 0.f;
    for (int c = 0; c < p.width; ++c) s = fmaf(qs[r * st + c], ks[key * st + c], s);
    s *= p.scale_log2;
    const bool seen = t * LF_KEYS + key <= last_key && t * LF_KEYS + key < ctx;
    if (!seen) s = -1e30f;
    const float m_new = fmaxf(m_run, warp_max(s));
    const float e = seen ? exp2f(s - m_new) : 0.f;
    const float alpha = exp2f(m_run - m_new);
    l_run = l_run * alpha + warp_sum(e);
    m_run = m_new;
    pr[r * LF_KEYS + key] = e;
    if (key == 0) al[r] = alpha;
    __syncthreads();
    for (int i = tid; i < LF_ROWS * p.rank; i += blockDim.x) {
      const int rr = i / p.rank, c = i - rr * p.rank;
      float acc = os[i] * al[rr];
#pragma unroll 8
      for (int k = 0; k < LF_KEYS; ++k) acc = fmaf(pr[rr * LF_KEYS + k], ks[k * st + c], acc);
      os[i] = acc;
    }
  }
  __syncthreads();
  if (key == 0 && row0 + r < p.rows) {
    float* ml = p.part_ml + (((int64_t)b * p.rows + row0 + r) * p.splits + split) * 2;
    ml[0] = m_run;
    ml[1] = l_run;
  }
  if (t_end <= t_begin) return;
  for (int i = tid; i < LF_ROWS * p.rank; i += blockDim.x) {
    const int rr = i / p.rank, c = i - rr * p.rank;
    if (row0 + rr < p.rows) p.part_o[(((int64_t)b * p.rows + row0 + rr) * p.splits + split) * p.rank + c] = os[i];
  }
}

// ----------------------------------------------------------------------------- combine + values
// out[t, h, v] = sum_r W_uvT[h, r, v] (sum_splits ...)[r]; W_uvT [H, rank, vdim].
constexpr int VAL_TOK = 4;

template <typename T>
__global__ void __launch_bounds__(256)
latent_values_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml, const float* __restrict__ sink,
                     const T* __restrict__ wuvt, int T_total, int H, int rank, int vdim, int splits, T* __restrict__ out) {
  extern __shared__ float sm[];
  float* ol = sm;                                   // [rank][VAL_TOK]
  float* wt = ol + rank * VAL_TOK;                  // [VAL_TOK][splits]
  float* red = wt + VAL_TOK * splits;               // [8 warps][VAL_TOK][32]
  pdl_wait();
  pdl_trigger();
  const int h = blockIdx.x, t0 = blockIdx.y * VAL_TOK;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (warp < VAL_TOK) {
    const int t = t0 + warp;
    if (t < T_total) {
      const float* ml = part_ml + ((int64_t)t * H + h) * splits * 2;
      const float sk = sink[h] * LOG2E;
      float m = sk, l = 0.f;
      for (int s = lane; s < splits; s += 32) if (ml[2 * s + 1] > 0.f) m = fmaxf(m, ml[2 * s]);
      m = warp_max(m);
      for (int s = lane; s < splits; s += 32) if (ml[2 * s + 1] > 0.f) l += ml[2 * s + 1] * exp2f(ml[2 * s] - m);
      l = warp_sum(l) + exp2f(sk - m);
      for (int s = lane; s < splits; s += 32) wt[warp * splits + s] = ml[2 * s + 1] > 0.f ? exp2f(ml[2 * s] - m) / l : 0.f;
    } else {
      for (int s = lane; s < splits; s += 32) wt[warp * splits + s] = 0.f;
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < VAL_TOK * rank; i += blockDim.x) {
    const int tt = i / rank, r = i - tt * rank;
    float acc = 0.f;
    if (t0 + tt < T_total) {
      const float* po = part_o + ((int64_t)(t0 + tt) * H + h) * splits * rank + r;
      for (int s = 0; s < splits; ++s) {
        const float w = wt[tt * splits + s];
        if (w != 0.f) acc = fmaf(w, po[(int64_t)s * rank], acc);     // (an empty split's rows are not initialised)
      }
    }
    ol[r * VAL_TOK + tt] = acc;
  }
  __syncthreads();
  const T* w = wuvt + (int64_t)h * rank * vdim;
  for (int v0 = 0; v0 < vdim; v0 += 32) {       // 32 value columns per pass; the eight warps split the latent
    const int v = v0 + lane;
    float acc[VAL_TOK] = {0.f, 0.f, 0.f, 0.f};
    if (v < vdim) {
#pragma unroll 8
      for (int r = warp; r < rank; r += 8) {
        const float wv = to_f<T>(w[(int64_t)r * vdim + v]);
        const float4 a = *reinterpret_cast<const float4*>(ol + r * VAL_TOK);
        acc[0] = fmaf(a.x, wv, acc[0]); acc[1] = fmaf(a.y, wv, acc[1]); acc[2] = fmaf(a.z, wv, acc[2]); acc[3] = fmaf(a.w, wv, acc[3]);
      }
    }
#pragma unroll
    for (int t = 0; t < VAL_TOK; ++t) red[(warp * VAL_TOK + t) * 32 + lane] = acc[t];
    __syncthreads();
    if (warp < VAL_TOK && v < vdim && t0 + warp < T_total) {
      float s = 0.f;
      for (int k = 0; k < 8; ++k) s += red[(k * VAL_TOK + warp) * 32 + lane];
      out[((int64_t)(t0 + warp) * H + h) * vdim + v] = from_f<T>(s);
    }
    __syncthreads();
  }
}

// Combined latents alone, [T*H, rank] bf16: one CTA per (token, head).
__global__ void __launch_bounds__(128)
latent_combine_kernel(const float* __restrict__ part_o, const float* __restrict__ part_ml, const float* __restrict__ sink, int H, int rank,
                      int splits, __nv_bfloat16* __restrict__ out) {
  extern __shared__ float wt[];       // [splits]
  pdl_wait();
  pdl_trigger();
  const int64_t row = blockIdx.x;
  if (threadIdx.x < 32) {
    const int lane = threadIdx.x;
    const float* ml = part_ml + row * splits * 2;
    const float sk = sink[row % H] * LOG2E;
    float m = sk, l = 0.f;
    for (int s = lane; s < splits; s += 32) if (ml[2 * s + 1] > 0.f) m = fmaxf(m, ml[2 * s]);
    m = warp_max(m);
    for (int s = lane; s < splits; s += 32) if (ml[2 * s + 1] > 0.f) l += ml[2 * s + 1] * exp2f(ml[2 * s] - m);
    l = warp_sum(l) + exp2f(sk - m);
    for (int s = lane; s < splits; s += 32) wt[s] = ml[2 * s + 1] > 0.f ? exp2f(ml[2 * s] - m) / l : 0.f;
  }
  __syncthreads();
  for (int r = threadIdx.x * 4; r < rank; r += blockDim.x * 4) {      // rank is a multiple of 32
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
    for (int s = 0; s < splits; ++s) {
      const float w = wt[s];
      if (w == 0.f) continue;                                          // (an empty split's rows are not initialised)
      const float4 v = *reinterpret_cast<const float4*>(part_o + (row * splits + s) * rank + r);
      acc.x = fmaf(w, v.x, acc.x); acc.y = fmaf(w, v.y, acc.y); acc.z = fmaf(w, v.z, acc.z); acc.w = fmaf(w, v.w, acc.w);
    }
    __nv_bfloat162 a = __floats2bfloat162_rn(acc.x, acc.y), c = __floats2bfloat162_rn(acc.z, acc.w);
    uint2 u;
    u.x = *reinterpret_cast<uint32_t*>(&a);
    u.y = *reinterpret_cast<uint32_t*>(&c);
    *reinterpret_cast<uint2*>(out + row * rank + r) = u;
  }
}

// ----------------------------------------------------------------------------- host side
static int pos_ptr(const kd_tensor* pos, const int** out) {
  *out = nullptr;
  if (!pos) return KD_OK;
  KD_REQUIRE(pos->dtype == KD_I32 && numel(pos) == 1, "position must be a device int32 scalar");
  void* p;
  KD_TRY(tensor_ptr(pos, &p));
  *out = static_cast<const int*>(p);
  return KD_OK;
}

template <int MT, int KT, int NT, int QR>
static int launch_lat(const void* q, const CUtensorMap& tmap, const LatAttnParams& p, int smem) {
  static bool configured[64] = {false};
  if (!configured[ctx().device & 63]) {
    KD_CUDA_CHECK(cudaFuncSetAttribute(latent_attention_bf16_kernel<MT, KT, NT, QR>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
    configured[ctx().device & 63] = true;
  }
  dim3 grid(p.splits, (p.rows + MT * 16 - 1) / (MT * 16), p.B);
  KD_CUDA_CHECK(launch_ex(latent_attention_bf16_kernel<MT, KT, NT, QR>, grid, dim3(LAT_THREADS), (size_t)smem, (const __nv_bfloat16*)q, tmap, p));
  return after_launch("latent_attention_bf16_kernel");
}

static int lat_smem(int width, int mt, int kt) {
  const int st = lat_stride(width), rows = mt * 16;
  return 1024 + 2 * ((width + 63) / 64) * kt * 128 + rows * st * 2 + 2 * rows * kt * 4 + rows * (kt + 8) * 2 + rows * 4 + 32;
}

template <int MT, int KT>
static int launch_lat_nt(const void* q, const void* cache_rows, const LatAttnParams& p, int smem) {
  CUtensorMap cache;
  KD_TRY(make_tmap_bf16_3d(&cache, cache_rows, (uint64_t)p.B, (uint64_t)p.max_s, (uint64_t)p.width, (uint64_t)p.cache_b, (uint64_t)p.cache_s, KT, 64));
  // (the depth is split over two warps: 18 k-steps each cover rows of 576 numbers)
  constexpr int QR = MT == 1 && KT == 64 ? 18 : 0;
  const bool qr = QR > 0 && p.width <= 576;
  if (p.rank <= 128) return qr ? launch_lat<MT, KT, 2, QR>(q, cache, p, smem) : launch_lat<MT, KT, 2, 0>(q, cache, p, smem);
  if (p.rank <= 256) return qr ? launch_lat<MT, KT, 4, QR>(q, cache, p, smem) : launch_lat<MT, KT, 4, 0>(q, cache, p, smem);
  if (p.rank <= 512) return qr ? launch_lat<MT, KT, 8, QR>(q, cache, p, smem) : launch_lat<MT, KT, 8, 0>(q, cache, p, smem);
  return launch_lat<MT, KT, 16, 0>(q, cache, p, smem);
}

}  // namespace kd

using namespace kd;

KD_API int kd_latent_prep(const kd_tensor* proj, int q_col, int heads, int dim, int rot_dim, int kv_col, int kv_rank,
                          const kd_tensor* norm_weight, float eps, const kd_tensor* cos, const kd_tensor* sin, const kd_tensor* cache,
                          const kd_tensor* pos_dev, int pos_host, const kd_tensor* dense) {
  KD_TRY(require_init());
  KD_REQUIRE(proj && cos && sin && cache, "null tensor");
  KD_REQUIRE(proj->ndim == 3 && proj->strides[2] == 1 && proj->strides[0] == proj->strides[1] * proj->shape[1] &&
                 (proj->dtype == KD_BF16 || proj->dtype == KD_F32),
             "proj must be [B,S,N] with evenly spaced rows, bf16 or fp32");
  KD_REQUIRE(cache->ndim == 3 && cache->dtype == proj->dtype && cache->strides[2] == 1 && cache->shape[0] >= proj->shape[0], "cache must be [B,maxS,width] of proj's type");
  KD_REQUIRE(heads >= 1 && dim >= 0 && rot_dim >= 0 && rot_dim % 2 == 0, "bad head sizes");
  KD_REQUIRE(q_col >= 0 && q_col + (int64_t)heads * (dim + rot_dim) <= proj->shape[2], "queries exceed the projection row");
  KD_REQUIRE(kv_col < 0 || (kv_rank >= 1 && kv_col + kv_rank + rot_dim <= proj->shape[2] && kv_rank + rot_dim <= cache->shape[2]), "latent exceeds the projection or the cache row");
  PrepParams p{};
  p.S = (int)proj->shape[1]; p.H = heads; p.dim = dim; p.rot = rot_dim; p.rank = kv_rank; p.max_s = (int)cache->shape[1];
  p.q_col = q_col; p.kv_col = kv_col; p.ld = proj->strides[1];
  p.cache_b = cache->strides[0]; p.cache_s = cache->strides[1];
  p.eps = eps;
  KD_REQUIRE(cos->dtype == KD_F32 && sin->dtype == KD_F32 && is_contiguous(cos) && is_contiguous(sin) && numel(cos) >= (int64_t)p.max_s * (rot_dim / 2) &&
                 numel(sin) >= (int64_t)p.max_s * (rot_dim / 2), "cos / sin must be fp32 [maxS, rot_dim/2]");
  KD_TRY(pos_ptr(pos_dev, &p.pos_dev));
  p.pos_host = pos_host;
  if (!pos_dev) KD_REQUIRE(pos_host >= 0 && pos_host + p.S <= p.max_s, "Cache overflow: trying to write to position %d-%d, but maxSeqLen is %d", pos_host, pos_host + p.S, p.max_s);
  p.err = ctx().error_flag;
  void *pp, *pc, *pd = nullptr, *t;
  KD_TRY(tensor_ptr(proj, &pp));
  KD_TRY(tensor_ptr(cache, &pc));
  KD_TRY(tensor_ptr(cos, &t)); p.cos_t = static_cast<const float*>(t);
  KD_TRY(tensor_ptr(sin, &t)); p.sin_t = static_cast<const float*>(t);
  if (kv_col >= 0) {
    KD_REQUIRE(norm_weight && norm_weight->dtype == KD_F32 && is_contiguous(norm_weight) && numel(norm_weight) == kv_rank, "norm weight must be fp32 [kv_rank]");
    KD_TRY(tensor_ptr(norm_weight, &t)); p.norm_w = static_cast<const float*>(t);
    if (dense) {
      KD_REQUIRE(dense->ndim == 2 && dense->dtype == proj->dtype && dense->strides[1] == 1 && dense->shape[0] >= proj->shape[0] * proj->shape[1] && dense->shape[1] >= kv_rank, "dense latent rows must be [B*S, kv_rank]");
      KD_TRY(tensor_ptr(dense, &pd));
      p.ld_dense = dense->strides[0];
    }
  }
  const int64_t tokens = proj->shape[0] * proj->shape[1];
  if (tokens == 0) return KD_OK;
  if (proj->dtype == KD_BF16)
    KD_CUDA_CHECK(launch_ex(latent_prep_kernel<__nv_bfloat16>, dim3((unsigned)tokens), dim3(256), 0, (__nv_bfloat16*)pp, (__nv_bfloat16*)pc, (__nv_bfloat16*)pd, p));
  else
    KD_CUDA_CHECK(launch_ex(latent_prep_kernel<float>, dim3((unsigned)tokens), dim3(256), 0, (float*)pp, (float*)pc, (float*)pd, p));
  return after_launch("latent_prep_kernel");
}

KD_API int kd_latent_absorb(const kd_tensor* proj, int q_col, int rot_dim, const kd_tensor* wuk, const kd_tensor* wuk_t,
                            const kd_tensor* q_abs) {
  KD_TRY(require_init());
  KD_REQUIRE(proj && wuk && q_abs, "null tensor");
  KD_REQUIRE(proj->ndim == 3 && proj->strides[2] == 1 && proj->strides[0] == proj->strides[1] * proj->shape[1], "proj must be [B,S,N] with evenly spaced rows");
  KD_REQUIRE(wuk->ndim == 3 && is_contiguous(wuk) && wuk->dtype == proj->dtype && q_abs->dtype == proj->dtype && is_contiguous(q_abs) &&
                 (proj->dtype == KD_BF16 || proj->dtype == KD_F32), "wuk [H,dim,kv_rank] and q_abs [T,H,width] must be contiguous, bf16 or fp32 like proj");
  const int H = (int)wuk->shape[0], dim = (int)wuk->shape[1], rank = (int)wuk->shape[2];
  const int64_t T = proj->shape[0] * proj->shape[1];
  const int width = (int)q_abs->shape[q_abs->ndim - 1];
  KD_REQUIRE(numel(q_abs) == T * H * width && width >= rank + rot_dim, "q_abs must be [T,H,width >= kv_rank+rot_dim]");
  KD_REQUIRE(q_col >= 0 && q_col + (int64_t)H * (dim + rot_dim) <= proj->shape[2], "queries exceed the projection row");
  KD_REQUIRE(dim * ABS_TOK * 4 <= 48 * 1024, "dim=%d is too large", dim);
  if (T == 0) return KD_OK;
  void *pp, *pw, *pq;
  KD_TRY(tensor_ptr(proj, &pp));
  KD_TRY(tensor_ptr(wuk, &pw));
  KD_TRY(tensor_ptr(q_abs, &pq));
  if (wuk_t) {
    KD_REQUIRE(wuk_t->ndim == 3 && is_contiguous(wuk_t) && wuk_t->dtype == wuk->dtype && wuk_t->shape[0] == H && wuk_t->shape[1] == rank && wuk_t->shape[2] == dim,
               "wuk_t must be [H,kv_rank,dim]");
    void* pt;
    KD_TRY(tensor_ptr(wuk_t, &pt));
    if (proj->dtype == KD_BF16 && dim % 32 == 0 && rank % 8 == 0 && (dim + rot_dim) % 8 == 0 && width % 8 == 0 && q_col % 8 == 0 && proj->strides[1] % 8 == 0 &&
        ((reinterpret_cast<uintptr_t>(pp) | reinterpret_cast<uintptr_t>(pt) | reinterpret_cast<uintptr_t>(pq)) & 15) == 0) {
      HeadLinearParams hp{(int)T, H, rank, dim, width, proj->strides[1], dim + rot_dim, (int64_t)H * width, width, dim, rot_dim};
      return launch_head_linear<1>(static_cast<const __nv_bfloat16*>(pp) + q_col, pt, pq, hp);
    }
  }
  const int64_t zt = (T + ABS_TOK - 1) / ABS_TOK;
  KD_REQUIRE(zt <= 65535, "kd_latent_absorb: %lld tokens in one call", (long long)T);
  dim3 grid(H, (width + 127) / 128, (unsigned)zt);
  const size_t smem = (size_t)dim * ABS_TOK * 4;
  if (proj->dtype == KD_BF16)
    KD_CUDA_CHECK(launch_ex(latent_absorb_kernel<__nv_bfloat16>, grid, dim3(128), smem, (const __nv_bfloat16*)pp, proj->strides[1], q_col, (const __nv_bfloat16*)pw, (int)T, H, dim, rot_dim, rank, width, (__nv_bfloat16*)pq));
  else
    KD_CUDA_CHECK(launch_ex(latent_absorb_kernel<float>, grid, dim3(128), smem, (const float*)pp, proj->strides[1], q_col, (const float*)pw, (int)T, H, dim, rot_dim, rank, width, (float*)pq));
  return after_launch("latent_absorb_kernel");
}

KD_API int kd_latent_attention_splits(int batch, int queries, int heads, int max_seq_len, int* splits_out) {
  KD_TRY(require_init());
  KD_REQUIRE(splits_out && batch >= 1 && queries >= 1 && heads >= 1 && max_seq_len >= 1, "bad argument");
  const int64_t rows = (int64_t)queries * heads, tiles = batch * ((rows + (rows > 16 ? 31 : 15)) / (rows > 16 ? 32 : 16));
  int64_t s = (rows > 16 ? 1 : 2) * ctx().sm_count / tiles, cap = (max_seq_len + 63) / 64;
  if (s > cap) s = cap;
  *splits_out = s < 1 ? 1 : (int)s;
  return KD_OK;
}

KD_API int kd_latent_attention(const kd_tensor* q_abs, const kd_tensor* cache, int kv_rank, float scale, const kd_tensor* pos_dev, int pos_host,
                               const kd_tensor* part_o, const kd_tensor* part_ml) {
  KD_TRY(require_init());
  KD_REQUIRE(q_abs && cache && part_o && part_ml, "null tensor");
  KD_REQUIRE(q_abs->ndim == 4 && is_contiguous(q_abs), "q_abs must be contiguous [B,S,H,width]");
  KD_REQUIRE(cache->ndim == 3 && cache->strides[2] == 1 && cache->dtype == q_abs->dtype && (cache->dtype == KD_BF16 || cache->dtype == KD_F32), "cache must be [B,maxS,width] of q_abs's type");
  LatAttnParams p{};
  p.B = (int)q_abs->shape[0]; p.S = (int)q_abs->shape[1]; p.H = (int)q_abs->shape[2]; p.width = (int)q_abs->shape[3];
  p.rank = kv_rank; p.max_s = (int)cache->shape[1];
  p.rows = p.S * p.H;
  KD_REQUIRE(cache->shape[0] >= p.B && cache->shape[2] == p.width && kv_rank >= 1 && kv_rank <= p.width, "cache and q_abs sizes do not match");
  KD_REQUIRE(part_o->dtype == KD_F32 && is_contiguous(part_o) && part_ml->dtype == KD_F32 && is_contiguous(part_ml), "partial sums must be contiguous fp32");
  KD_REQUIRE(numel(part_ml) > 0 && numel(part_ml) % ((int64_t)p.B * p.rows * 2) == 0, "part_ml must be [B*S*H, splits, 2]");
  p.splits = (int)(numel(part_ml) / ((int64_t)p.B * p.rows * 2));
  KD_REQUIRE(numel(part_o) == (int64_t)p.B * p.rows * p.splits * kv_rank, "part_o must be [B*S*H, splits, kv_rank]");
  p.cache_b = cache->strides[0]; p.cache_s = cache->strides[1];
  p.scale_log2 = scale * LOG2E;
  KD_TRY(pos_ptr(pos_dev, &p.pos_dev));
  p.pos_host = pos_host;
  if (!pos_dev) KD_REQUIRE(pos_host >= 0 && pos_host + p.S <= p.max_s, "queries at %d-%d exceed the cache of %d rows", pos_host, pos_host + p.S, p.max_s);
  p.err = ctx().error_flag;
  void *pq, *pc, *po, *pm;
  KD_TRY(tensor_ptr(q_abs, &pq));
  KD_TRY(tensor_ptr(cache, &pc));
  KD_TRY(tensor_ptr(part_o, &po));
  KD_TRY(tensor_ptr(part_ml, &pm));
  p.part_o = static_cast<float*>(po);
  p.part_ml = static_cast<float*>(pm);
  if (p.B == 0 || p.rows == 0) return KD_OK;
  KD_REQUIRE(p.rows <= 65535 * 8 && p.B <= 65535, "too many query rows");
  if (cache->dtype == KD_F32) {
    const size_t smem = ((size_t)(LF_ROWS + LF_KEYS) * (p.width + 1) + LF_ROWS * LF_KEYS + (size_t)LF_ROWS * p.rank + LF_ROWS) * 4;
    KD_REQUIRE(smem <= 227 * 1024, "latent rows of %d numbers are too wide for the fp32 kernel", p.width);
    static bool configured[64] = {false};
    if (!configured[ctx().device & 63]) {
      KD_CUDA_CHECK(cudaFuncSetAttribute(latent_attention_f32_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
      configured[ctx().device & 63] = true;
    }
    dim3 grid(p.splits, (p.rows + LF_ROWS - 1) / LF_ROWS, p.B);
    KD_CUDA_CHECK(launch_ex(latent_attention_f32_kernel, grid, dim3(256), smem, (const float*)pq, (const float*)pc, p));
    return after_launch("latent_attention_f32_kernel");
  }
  KD_REQUIRE(p.width % 16 == 0 && p.cache_b % 8 == 0 && p.cache_s % 8 == 0 && ((reinterpret_cast<uintptr_t>(pq) | reinterpret_cast<uintptr_t>(pc)) & 15) == 0,
             "bf16 latent rows must be padded to a multiple of 16 and 16-byte aligned");
  KD_REQUIRE(kv_rank <= 1024, "kv_rank=%d; this path handles up to 1024", kv_rank);
  const int limit = 227 * 1024;
  // 32 query rows per CTA when there are that many (every cache tile then serves two row tiles)
  if (p.rows > 16 && kv_rank <= 512) {
    if (lat_smem(p.width, 2, 64) <= limit) return launch_lat_nt<2, 64>(pq, pc, p, lat_smem(p.width, 2, 64));
    if (lat_smem(p.width, 2, 32) <= limit) return launch_lat_nt<2, 32>(pq, pc, p, lat_smem(p.width, 2, 32));
  }
  // 32-key tiles let two CTAs share an SM: one's softmax runs under the other's products
  if (kv_rank <= 512 && 2 * (lat_smem(p.width, 1, 32) + 1024) <= limit) return launch_lat_nt<1, 32>(pq, pc, p, lat_smem(p.width, 1, 32));
  if (lat_smem(p.width, 1, 64) <= limit) return launch_lat_nt<1, 64>(pq, pc, p, lat_smem(p.width, 1, 64));
  KD_REQUIRE(lat_smem(p.width, 1, 32) <= limit, "latent rows of %d numbers are too wide", p.width);
  return launch_lat_nt<1, 32>(pq, pc, p, lat_smem(p.width, 1, 32));
}

KD_API int kd_latent_values(const kd_tensor* part_o, const kd_tensor* part_ml, const kd_tensor* sink, const kd_tensor* wuv_t,
                            const kd_tensor* wuv, const kd_tensor* latents, const kd_tensor* out) {
  KD_TRY(require_init());
  KD_REQUIRE(part_o && part_ml && sink && wuv_t && out, "null tensor");
  KD_REQUIRE(wuv_t->ndim == 3 && is_contiguous(wuv_t) && is_contiguous(out) && out->dtype == wuv_t->dtype && (out->dtype == KD_BF16 || out->dtype == KD_F32),
             "wuv_t [H,kv_rank,vdim] and out [T,H*vdim] must be contiguous, of one type");
  const int H = (int)wuv_t->shape[0], rank = (int)wuv_t->shape[1], vdim = (int)wuv_t->shape[2];
  KD_REQUIRE(sink->dtype == KD_F32 && is_contiguous(sink) && numel(sink) == H, "sink must be fp32 [H]");
  KD_REQUIRE(numel(out) % ((int64_t)H * vdim) == 0, "out must be [T,H*vdim]");
  const int64_t T = numel(out) / ((int64_t)H * vdim);
  if (T == 0) return KD_OK;
  KD_REQUIRE(part_ml->dtype == KD_F32 && is_contiguous(part_ml) && numel(part_ml) % (T * H * 2) == 0, "part_ml must be fp32 [T*H, splits, 2]");
  const int splits = (int)(numel(part_ml) / (T * H * 2));
  KD_REQUIRE(part_o->dtype == KD_F32 && is_contiguous(part_o) && numel(part_o) == T * H * splits * rank, "part_o must be fp32 [T*H, splits, kv_rank]");
  void *po, *pm, *ps, *pw, *pout;
  KD_TRY(tensor_ptr(part_o, &po));
  KD_TRY(tensor_ptr(part_ml, &pm));
  KD_TRY(tensor_ptr(sink, &ps));
  KD_TRY(tensor_ptr(wuv_t, &pw));
  KD_TRY(tensor_ptr(out, &pout));
  if (wuv && latents) {
    KD_REQUIRE(wuv->ndim == 3 && is_contiguous(wuv) && wuv->dtype == out->dtype && wuv->shape[0] == H && wuv->shape[1] == vdim && wuv->shape[2] == rank, "wuv must be [H,vdim,kv_rank]");
    KD_REQUIRE(latents->dtype == out->dtype && is_contiguous(latents) && numel(latents) >= T * H * rank, "latents must be [T*H, kv_rank]");
    void *pl, *pv;
    KD_TRY(tensor_ptr(latents, &pl));
    KD_TRY(tensor_ptr(wuv, &pv));
    if (out->dtype == KD_BF16 && rank % 32 == 0 && vdim % 8 == 0 &&
        ((reinterpret_cast<uintptr_t>(pl) | reinterpret_cast<uintptr_t>(pv) | reinterpret_cast<uintptr_t>(pout) | reinterpret_cast<uintptr_t>(po)) & 15) == 0) {
      KD_CUDA_CHECK(launch_ex(latent_combine_kernel, dim3((unsigned)(T * H)), dim3(128), (size_t)splits * 4, (const float*)po, (const float*)pm, (const float*)ps, H, rank, splits, (__nv_bfloat16*)pl));
      KD_TRY(after_launch("latent_combine_kernel"));
      HeadLinearParams hp{(int)T, H, vdim, rank, vdim, (int64_t)H * rank, rank, (int64_t)H * vdim, vdim, 0, 0};
      return launch_head_linear<4>(pl, pv, pout, hp);
    }
  }
  const size_t smem = ((size_t)rank * VAL_TOK + VAL_TOK * splits + 8 * VAL_TOK * 32) * 4;
  KD_REQUIRE(smem <= 48 * 1024, "kv_rank=%d with %d splits is too large", rank, splits);
  const int64_t yt = (T + VAL_TOK - 1) / VAL_TOK;
  KD_REQUIRE(yt <= 65535, "kd_latent_values: %lld tokens in one call", (long long)T);
  dim3 grid(H, (unsigned)yt);
  if (out->dtype == KD_BF16)
    KD_CUDA_CHECK(launch_ex(latent_values_kernel<__nv_bfloat16>, grid, dim3(256), smem, (const float*)po, (const float*)pm, (const float*)ps, (const __nv_bfloat16*)pw, (int)T, H, rank, vdim, splits, (__nv_bfloat16*)pout));
  else
    KD_CUDA_CHECK(launch_ex(latent_values_kernel<float>, grid, dim3(256), smem, (const float*)po, (const float*)pm, (const float*)ps, (const float*)pw, (int)T, H, rank, vdim, splits, (float*)pout));
  return after_launch("latent_values_kernel");
}
