// Mixture of experts: group-limited sigmoid routing, permutation by expert, grouped linears.
//
//   kd_moe_route   one warp per token: s = sigmoid(logit) in fp32; a group's score is the sum of its
//                  two largest s; the best `keep` groups stay; the `top` largest s among their experts
//                  are chosen (ties: lowest index) and weighted by s / (sum of the chosen s + 1e-20).
//                  The same kernel counts the tokens of every expert and gives every (token, choice)
//                  its rank inside its expert.
//   kd_moe_gather  row of every (token, choice) in expert order = offset[expert] + rank; copies the
//                  token's activation row there.  No sort: the order of an expert's rows is whatever
//                  the counting atomics gave, and no result depends on it (every row of a grouped
//                  linear is computed alone).
//   kd_moe_linear  out[rows of e] = epilogue(x[rows of e] * W[e]^T) for all experts in one launch: on
//                  tcgen05 for bf16 (gemm_tcgen05.cu), on the CUDA cores for fp32 and unaligned sizes.
// Expert rows are laid out without padding; a tensor-core tile that runs over an expert's end computes
// rows of the next expert and does not store them.
#include "common.cuh"
#include "kernels.cuh"

namespace kd {

constexpr int MOE_MAX_EXPERTS = 1024;
constexpr int ROUTE_WARPS = 8;

__global__ void __launch_bounds__(ROUTE_WARPS * 32)
moe_route_kernel(const float* __restrict__ logits, int64_t ld, int T, int E, int top, int groups, int keep,
                 int* __restrict__ ids, float* __restrict__ weights, int* __restrict__ ranks, int* __restrict__ counts) {
  extern __shared__ float sm[];       // [warps][E] scores, [warps][groups] group scores, then int [E] block counts
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* s = sm + warp * (E + groups);
  float* gs = s + E;
  int* cnt = reinterpret_cast<int*>(sm + ROUTE_WARPS * (E + groups));
  for (int e = threadIdx.x; e < E; e += blockDim.x) cnt[e] = 0;
  pdl_wait();
  pdl_trigger();
  __syncthreads();
  const int t = blockIdx.x * ROUTE_WARPS + warp;
  const bool live = t < T;
  int my_e = 0, my_r = 0;             // lane k keeps choice k (top <= 32)
  float my_s = 0.f;
  if (live) {
    for (int e = lane; e < E; e += 32) s[e] = 1.0f / (1.0f + expf(-logits[(int64_t)t * ld + e]));
    __syncwarp();
    const int gsz = E / groups;
    if (keep < groups) {
      for (int g = lane; g < groups; g += 32) {
        float a = -1.f, b = -1.f;     // two largest
        for (int e = g * gsz; e < (g + 1) * gsz; ++e) {
          const float v = s[e];
          if (v > a) { b = a; a = v; } else if (v > b) { b = v; }
        }
        gs[g] = gsz > 1 ? a + b : a;
      }
      __syncwarp();
      // keep the best groups: the ones taken are marked by +4, the rest lose their scores
      for (int i = 0; i < keep; ++i) {
        float best = -1.f;
        int at = groups;
        for (int g = lane; g < groups; g += 32)
          if (gs[g] < 3.f && gs[g] > best) { best = gs[g]; at = g; }
        for (int o = 16; o > 0; o >>= 1) {
          const float v = __shfl_xor_sync(0xffffffffu, best, o);
          const int a = __shfl_xor_sync(0xffffffffu, at, o);
          if (v > best || (v == best && a < at)) { best = v; at = a; }
        }
        if (lane == 0 && at < groups) gs[at] += 4.f;
        __syncwarp();
      }
      for (int e = lane; e < E; e += 32)
        if (gs[e / gsz] < 3.f) s[e] = -1.f;
      __syncwarp();
    }
    float sum = 0.f;
    for (int k = 0; k < top; ++k) {
      float best = -2.f;
      int at = E;
      for (int e = lane; e < E; e += 32)
        if (s[e] > best) { best = s[e]; at = e; }
      for (int o = 16; o > 0; o >>= 1) {
        const float v = __shfl_xor_sync(0xffffffffu, best, o);
        const int a = __shfl_xor_sync(0xffffffffu, at, o);
        if (v > best || (v == best && a < at)) { best = v; at = a; }
      }
      at = min(at, E - 1);                          // (only NaN scores leave nothing to choose)
      __syncwarp();
      if (lane == 0) s[at] = -3.f;
      __syncwarp();
      best = fmaxf(best, 0.f);
      sum += best;
      if (lane == k) { my_e = at; my_s = best; }
    }
    if (lane < top) {
      ids[(int64_t)t * top + lane] = my_e;
      weights[(int64_t)t * top + lane] = my_s / (sum + 1e-20f);
      my_r = atomicAdd(&cnt[my_e], 1);
    }
  }
  __syncthreads();
  for (int e = threadIdx.x; e < E; e += blockDim.x) {
    const int c = cnt[e];
    cnt[e] = c ? atomicAdd(&counts[e], c) : 0;      // base of this block's tokens inside the expert
  }
  __syncthreads();
  if (live && lane < top) ranks[(int64_t)t * top + lane] = cnt[my_e] + my_r;
}

constexpr int GATHER_TOKENS = 4;

// Exclusive prefix of counts over E experts into smem (blockDim 256).
__device__ __forceinline__ void expert_offsets(const int* __restrict__ counts, int E, int* off, int* warp_tot) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  int carry = 0;
  for (int base = 0; base < E; base += blockDim.x) {
    const int e = base + threadIdx.x;
    const int c = e < E ? counts[e] : 0;
    int inc = c;
    for (int o = 1; o < 32; o <<= 1) {
      const int v = __shfl_up_sync(0xffffffffu, inc, o);
      if (lane >= o) inc += v;
    }
    if (lane == 31) warp_tot[warp] = inc;
    __syncthreads();
    int before = carry, all = 0;
    for (int w = 0; w < nw; ++w) { if (w < warp) before += warp_tot[w]; all += warp_tot[w]; }
    if (e < E) off[e] = before + inc - c;
    carry += all;
    __syncthreads();
  }
  if (threadIdx.x == 0) off[E] = carry;
  __syncthreads();
}

__global__ void __launch_bounds__(256)
moe_gather_kernel(const void* __restrict__ h, int row_bytes, int T, int E, int top, const int* __restrict__ ids,
                  const int* __restrict__ ranks, const int* __restrict__ counts, int* __restrict__ slots, int* __restrict__ offsets,
                  void* __restrict__ xp) {
  __shared__ int off[MOE_MAX_EXPERTS + 1];
  __shared__ int warp_tot[8];
  __shared__ int pos[GATHER_TOKENS * 32];
  pdl_wait();
  pdl_trigger();
  expert_offsets(counts, E, off, warp_tot);
  if (blockIdx.x == 0)
    for (int e = threadIdx.x; e <= E; e += blockDim.x) offsets[e] = off[e];
  const int t0 = blockIdx.x * GATHER_TOKENS;
  for (int i = threadIdx.x; i < GATHER_TOKENS * top && t0 * top + i < T * top; i += blockDim.x) {
    const int64_t at = (int64_t)t0 * top + i;
    slots[at] = pos[i] = off[ids[at]] + ranks[at];
  }
  __syncthreads();
  const bool v16 = row_bytes % 16 == 0 && ((reinterpret_cast<uintptr_t>(h) | reinterpret_cast<uintptr_t>(xp)) & 15) == 0;
  for (int i = 0; i < GATHER_TOKENS && t0 + i < T; ++i) {
    const int t = t0 + i;
    const char* src = static_cast<const char*>(h) + (int64_t)t * row_bytes;
    if (v16) {
      for (int c = threadIdx.x; c < row_bytes / 16; c += blockDim.x) {
        const uint4 v = reinterpret_cast<const uint4*>(src)[c];
        for (int k = 0; k < top; ++k) reinterpret_cast<uint4*>(static_cast<char*>(xp) + (int64_t)pos[i * top + k] * row_bytes)[c] = v;
      }
    } else {
      for (int c = threadIdx.x; c < row_bytes / 2; c += blockDim.x) {
        const uint16_t v = reinterpret_cast<const uint16_t*>(src)[c];
        for (int k = 0; k < top; ++k) reinterpret_cast<uint16_t*>(static_cast<char*>(xp) + (int64_t)pos[i * top + k] * row_bytes)[c] = v;
      }
    }
  }
}

// ----------------------------------------------------------------------------- grouped linear, CUDA cores
__device__ __forceinline__ float clamped_glu_exact(float g, float u, float limit) {
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  return g / (1.0f + expf(-1.702f * g)) * (u + 1.0f);
}

// gate and up of one output (epilogue: KD_EPI_SWIGLU, KD_EPI_CLAMPED_GLU or KD_EPI_GEGLU)
__device__ __forceinline__ float glu_exact(float g, float u, int epilogue, float limit) {
  if (epilogue == KD_EPI_CLAMPED_GLU) return clamped_glu_exact(g, u, limit);
  if (epilogue == KD_EPI_SWIGLU) return g / (1.0f + expf(-g)) * u;
  return 0.5f * g * (1.0f + tanhf(0.7978845608028654f * fmaf(0.044715f * g * g, g, g))) * u;
}

constexpr int GL_BM = 32, GL_BN = 32, GL_BK = 32;

// 32 x 32 output tile, 256 threads (4 rows each); with the GLU epilogue two accumulators per output.
template <typename T, bool GLU>
__global__ void __launch_bounds__(256)
moe_linear_kernel(const T* __restrict__ x, const T* __restrict__ w, const int* __restrict__ offsets, int per, int E, int N, int K, int epilogue,
                  float limit, T* __restrict__ out) {
  __shared__ float xs[GL_BM][GL_BK + 1];
  __shared__ float wg[GL_BN][GL_BK + 1];
  __shared__ float wu[GLU ? GL_BN : 1][GL_BK + 1];
  __shared__ int sel[3];
  const int n_out = GLU ? N / 2 : N;
  // blockIdx.y enumerates the 32-row tiles of all experts (without offsets every expert has `per` rows)
  if (threadIdx.x == 0) {
    auto off = [&](int e) { return offsets ? offsets[e] : e * per; };
    int left = blockIdx.y, e = 0;
    for (; e < E; ++e) {
      const int tiles = (off(e + 1) - off(e) + GL_BM - 1) / GL_BM;
      if (left < tiles) break;
      left -= tiles;
    }
    sel[0] = e;
    sel[1] = e < E ? off(e) + left * GL_BM : 0;
    sel[2] = e < E ? off(e + 1) : 0;
  }
  __syncthreads();
  const int e = sel[0], row0 = sel[1], row_end = sel[2];
  if (e >= E) return;
  const int col0 = blockIdx.x * GL_BN;
  const T* we = w + (int64_t)e * N * K;
  const int tx = threadIdx.x & 31, ty = threadIdx.x >> 5;
  float acc[4] = {0.f, 0.f, 0.f, 0.f}, acc2[4] = {0.f, 0.f, 0.f, 0.f};
  for (int k0 = 0; k0 < K; k0 += GL_BK) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = ty + 8 * i, k = k0 + tx;
      xs[r][tx] = (row0 + r < row_end && k < K) ? (float)x[(int64_t)(row0 + r) * K + k] : 0.f;
      const int j = col0 + r;
      const int64_t wr = GLU ? (int64_t)(j >> 4) * 32 + (j & 15) : j;
      wg[r][tx] = (j < n_out && k < K) ? (float)we[wr * K + k] : 0.f;
      if (GLU) wu[r][tx] = (j < n_out && k < K) ? (float)we[(wr + 16) * K + k] : 0.f;
    }
    __syncthreads();
#pragma unroll 8
    for (int k = 0; k < GL_BK; ++k) {
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        acc[i] = fmaf(xs[ty + 8 * i][k], wg[tx][k], acc[i]);
        if (GLU) acc2[i] = fmaf(xs[ty + 8 * i][k], wu[tx][k], acc2[i]);
      }
    }
    __syncthreads();
  }
  const int j = col0 + tx;
  if (j >= n_out) return;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int r = row0 + ty + 8 * i;
    if (r < row_end) out[(int64_t)r * n_out + j] = (T)(GLU ? glu_exact(acc[i], acc2[i], epilogue, limit) : acc[i]);
  }
}

template <typename T>
static void launch_moe_linear(const void* x, const void* w, const int* off, int per, int E, int N, int K, int epi, float limit, void* out, dim3 grid) {
  if (epi != KD_EPI_NONE) moe_linear_kernel<T, true><<<grid, 256, 0, ctx().stream>>>((const T*)x, (const T*)w, off, per, E, N, K, epi, limit, (T*)out);
  else moe_linear_kernel<T, false><<<grid, 256, 0, ctx().stream>>>((const T*)x, (const T*)w, off, per, E, N, K, epi, limit, (T*)out);
}

// Rows of group e (offsets, or R / E rows each) against weight e; tensor cores where the operands allow.
static int grouped_linear(int dtype, const void* x, const void* w, const int* off, int64_t R, int64_t E, int64_t N, int64_t K, int epi, float limit, void* out) {
  const int64_t n_out = epi != KD_EPI_NONE ? N / 2 : N;
  if (dtype == KD_BF16 && K % 8 == 0 && n_out % 8 == 0 && epi != KD_EPI_SWIGLU &&
      ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(w) | reinterpret_cast<uintptr_t>(out)) & 15) == 0) {
    // equal groups of a few rows: stream the weights, where the 128-row weight tiles are enough to fill the GPU
    if (!off && epi == KD_EPI_NONE && R / E <= 64 && E * ((N + 127) / 128) >= ctx().sm_count / 2)
      return gemm_bf16_skinny(x, K, w, K, (int)(R / E), (int)N, (int)K, 1, nullptr, out, 0, 1.0f, nullptr, 0, 0, (int)E);
    return gemm_bf16_grouped(x, w, out, off, (int)R, (int)E, (int)N, (int)K, epi, limit);
  }
  const int64_t tiles = R / GL_BM + (E < R ? E : R) + 1;
  KD_REQUIRE(tiles <= 65535, "grouped linear (CUDA cores): too many row tiles (%lld)", (long long)tiles);
  dim3 grid((unsigned)((n_out + GL_BN - 1) / GL_BN), (unsigned)tiles);
  const int per = (int)(R / E);
  if (dtype == KD_F32) launch_moe_linear<float>(x, w, off, per, (int)E, (int)N, (int)K, epi, limit, out, grid);
  else launch_moe_linear<__nv_bfloat16>(x, w, off, per, (int)E, (int)N, (int)K, epi, limit, out, grid);
  return after_launch("moe_linear_kernel");
}

static int i32_ptr(const kd_tensor* t, int64_t n, const char* what, int** out) {
  KD_REQUIRE(t && t->dtype == KD_I32 && is_contiguous(t) && numel(t) >= n, "%s must be contiguous int32 with at least %lld elements", what, (long long)n);
  void* p;
  KD_TRY(tensor_ptr(t, &p));
  *out = static_cast<int*>(p);
  return KD_OK;
}

}  // namespace kd

using namespace kd;

KD_API int kd_moe_route(const kd_tensor* logits, int top, int groups, int keep, const kd_tensor* ids, const kd_tensor* weights,
                        const kd_tensor* ranks, const kd_tensor* counts) {
  KD_TRY(require_init());
  KD_REQUIRE(logits && weights, "null tensor");
  KD_REQUIRE(logits->dtype == KD_F32 && logits->ndim == 2 && logits->strides[1] == 1, "router logits must be fp32 [T,E]");
  const int64_t T = logits->shape[0], E = logits->shape[1];
  KD_REQUIRE(E >= 1 && E <= MOE_MAX_EXPERTS, "%lld experts; this path handles 1..%d", (long long)E, MOE_MAX_EXPERTS);
  KD_REQUIRE(groups >= 1 && E % groups == 0, "%lld experts do not form %d equal groups", (long long)E, groups);
  KD_REQUIRE(keep >= 1 && keep <= groups, "keep=%d of %d groups", keep, groups);
  KD_REQUIRE(top >= 1 && top <= 32 && top <= keep * (E / groups), "top=%d of %lld selectable experts (at most 32)", top, (long long)(keep * (E / groups)));
  if (T == 0) return KD_OK;
  int *pi, *pr, *pc;
  KD_TRY(i32_ptr(ids, T * top, "ids", &pi));
  KD_TRY(i32_ptr(ranks, T * top, "ranks", &pr));
  KD_TRY(i32_ptr(counts, E, "counts", &pc));
  KD_REQUIRE(weights->dtype == KD_F32 && is_contiguous(weights) && numel(weights) >= T * top, "weights must be contiguous fp32 [T,top]");
  void *pl, *pw;
  KD_TRY(tensor_ptr(logits, &pl));
  KD_TRY(tensor_ptr(weights, &pw));
  const size_t smem = (ROUTE_WARPS * (E + groups)) * sizeof(float) + E * sizeof(int);
  static bool configured[64] = {false};
  if (!configured[ctx().device & 63]) {
    KD_CUDA_CHECK(cudaFuncSetAttribute(moe_route_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 96 * 1024));
    configured[ctx().device & 63] = true;
  }
  KD_CUDA_CHECK(launch_ex(moe_route_kernel, dim3((unsigned)((T + ROUTE_WARPS - 1) / ROUTE_WARPS)), dim3(ROUTE_WARPS * 32), smem,
                          (const float*)pl, logits->strides[0], (int)T, (int)E, top, groups, keep, pi, (float*)pw, pr, pc));
  return after_launch("moe_route_kernel");
}

KD_API int kd_moe_gather(const kd_tensor* h, const kd_tensor* ids, const kd_tensor* ranks, const kd_tensor* counts, int experts,
                         const kd_tensor* slots, const kd_tensor* offsets, const kd_tensor* x_sorted) {
  KD_TRY(require_init());
  KD_REQUIRE(h && ids && x_sorted, "null tensor");
  KD_REQUIRE(h->ndim == 2 && is_contiguous(h) && (h->dtype == KD_BF16 || h->dtype == KD_F32), "h must be contiguous [T,W]");
  const int64_t T = h->shape[0], W = h->shape[1];
  KD_REQUIRE(experts >= 1 && experts <= MOE_MAX_EXPERTS, "%d experts; this path handles 1..%d", experts, MOE_MAX_EXPERTS);
  if (T == 0) return KD_OK;
  KD_REQUIRE(numel(ids) % T == 0, "ids must be [T,top]");
  const int top = (int)(numel(ids) / T);
  KD_REQUIRE(x_sorted->dtype == h->dtype && is_contiguous(x_sorted) && numel(x_sorted) >= T * top * W, "x_sorted must be contiguous [T*top,W]");
  int *pi, *pr, *pc, *ps, *po;
  KD_TRY(i32_ptr(ids, T * top, "ids", &pi));
  KD_TRY(i32_ptr(ranks, T * top, "ranks", &pr));
  KD_TRY(i32_ptr(counts, experts, "counts", &pc));
  KD_TRY(i32_ptr(slots, T * top, "slots", &ps));
  KD_TRY(i32_ptr(offsets, experts + 1, "offsets", &po));
  void *ph, *px;
  KD_TRY(tensor_ptr(h, &ph));
  KD_TRY(tensor_ptr(x_sorted, &px));
  KD_CUDA_CHECK(launch_ex(moe_gather_kernel, dim3((unsigned)((T + GATHER_TOKENS - 1) / GATHER_TOKENS)), dim3(256), 0, (const void*)ph,
                          (int)(W * dtype_size(h->dtype)), (int)T, experts, top, (const int*)pi, (const int*)pr, (const int*)pc, ps, po, px));
  return after_launch("moe_gather_kernel");
}

KD_API int kd_moe_linear(const kd_tensor* x, const kd_tensor* weight, const kd_tensor* offsets, int epilogue, float limit, const kd_tensor* out) {
  KD_TRY(require_init());
  KD_REQUIRE(x && weight && out, "null tensor");
  KD_REQUIRE(epilogue == KD_EPI_NONE || epilogue == KD_EPI_CLAMPED_GLU || epilogue == KD_EPI_GEGLU, "kd_moe_linear: unknown epilogue %d", epilogue);
  KD_REQUIRE(weight->ndim == 3 && is_contiguous(weight) && x->ndim == 2 && is_contiguous(x) && out->ndim == 2 && is_contiguous(out),
             "kd_moe_linear needs contiguous x [R,K], weight [E,N,K], out [R,N]");
  KD_REQUIRE(x->dtype == weight->dtype && x->dtype == out->dtype && (x->dtype == KD_BF16 || x->dtype == KD_F32), "kd_moe_linear: bf16 or fp32, one type");
  const int64_t R = x->shape[0], K = x->shape[1], E = weight->shape[0], N = weight->shape[1];
  const bool glu = epilogue != KD_EPI_NONE;
  const int64_t n_out = glu ? N / 2 : N;
  KD_REQUIRE(weight->shape[2] == K && out->shape[0] == R && out->shape[1] == n_out, "kd_moe_linear: shapes do not match");
  KD_REQUIRE(!glu || N % 32 == 0, "the gated epilogue needs gate and up rows in blocks of 16");
  KD_REQUIRE(E >= 1 && E <= MOE_MAX_EXPERTS && R < (1ll << 30), "kd_moe_linear: %lld experts, %lld rows", (long long)E, (long long)R);
  if (R == 0) return KD_OK;
  int* po = nullptr;
  if (offsets) KD_TRY(i32_ptr(offsets, E + 1, "offsets", &po));
  else KD_REQUIRE(R % E == 0, "kd_moe_linear: %lld rows in %lld equal groups", (long long)R, (long long)E);
  void *px, *pw, *pout;
  KD_TRY(tensor_ptr(x, &px));
  KD_TRY(tensor_ptr(weight, &pw));
  KD_TRY(tensor_ptr(out, &pout));
  return grouped_linear(x->dtype, px, pw, po, R, E, N, K, epilogue, limit, pout);
}

KD_API int kd_linear_glu(const kd_tensor* x, const kd_tensor* weight, int epilogue, const kd_tensor* out) {
  KD_TRY(require_init());
  KD_REQUIRE(x && weight && out, "null tensor");
  KD_REQUIRE(epilogue == KD_EPI_SWIGLU || epilogue == KD_EPI_GEGLU, "kd_linear_glu: unknown epilogue %d", epilogue);
  KD_REQUIRE(x->ndim == 2 && is_contiguous(x) && weight->ndim == 2 && is_contiguous(weight) && out->ndim == 2 && is_contiguous(out),
             "kd_linear_glu needs contiguous x [M,K], weight [2I,K], out [M,I]");
  KD_REQUIRE(x->dtype == weight->dtype && x->dtype == out->dtype && (x->dtype == KD_BF16 || x->dtype == KD_F32), "kd_linear_glu: bf16 or fp32, one type");
  const int64_t M = x->shape[0], K = x->shape[1], N = weight->shape[0];
  KD_REQUIRE(weight->shape[1] == K && N % 32 == 0 && out->shape[0] == M && out->shape[1] == N / 2, "kd_linear_glu: shapes do not match (gate and up rows in blocks of 16)");
  KD_REQUIRE(M < (1ll << 30), "kd_linear_glu: %lld rows", (long long)M);
  if (M == 0) return KD_OK;
  void *px, *pw, *po;
  KD_TRY(tensor_ptr(x, &px));
  KD_TRY(tensor_ptr(weight, &pw));
  KD_TRY(tensor_ptr(out, &po));
  if (x->dtype == KD_BF16 && K % 8 == 0 && ((reinterpret_cast<uintptr_t>(px) | reinterpret_cast<uintptr_t>(pw) | reinterpret_cast<uintptr_t>(po)) & 15) == 0) {
    // a handful of rows: the kernel that streams the weights, where its 128-row tiles are enough to fill the GPU
    if (M <= 64 && N >= 128ll * (ctx().sm_count / 2))
      return gemm_bf16_skinny(px, K, pw, K, (int)M, (int)N, (int)K, 1, nullptr, po, epilogue == KD_EPI_GEGLU ? 2 : 1);
    return gemm_bf16(px, K, pw, K, po, N / 2, 0, nullptr, 0, (int)M, (int)N, (int)K, epilogue);
  }
  return grouped_linear(x->dtype, px, pw, nullptr, M, 1, N, K, epilogue, 0.f, po);
}
