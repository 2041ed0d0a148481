// Gated delta rule with one decay per key channel (a linear-attention layer with an [dim, vdim] fp32
// state per head), prefill and decode in one kernel.
//
// Per head and token:  S <- g S (rows);  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q,
// with q, k, v = silu(short causal convolution of the projections), q and k unit vectors (q also
// times dim^-1/2), g = exp(-exp(A_log) softplus(a + dt_bias)), beta = sigmoid(b).
//
// Why a recurrence and not chunks: everything that enters the recurrence and the state itself is
// fp32, so a chunked form on the tensor cores needs split operands (three products for one), a
// triangular solve per chunk and per-channel decays inside every product.  Counted in instructions
// that is no cheaper than the recurrence itself when the state lives in registers and the arithmetic
// is packed (fma.rn.f32x2: two per lane and instruction).  And the result does not depend on where a
// prompt is cut: every token is computed alone, in order, bit for bit the same in any portion.
//
// Mapping.  A state column (one value channel) never meets another one, so a warp owns 32 / LPC
// groups of 4 columns, and the LPC lanes of a group share its dim rows (32 rows a lane, in quads
// i LPC + j): 128 state registers a lane whatever the size.  Per token a lane reads its 32 entries of
// g, k (twice) and q as broadcast 16-byte shared-memory loads, does 4 packed operations per pair of
// state entries, and the group's S^T k is a butterfly over LPC lanes.
// A CTA is eight consumer warps (one or more heads) and four helper warps.  The helpers prepare the
// next block of tokens (convolution, silu, unit norms, decays, step sizes) in shared memory while the
// consumers walk through the current one.
// Bound: fp32 pipe in prefill (4 dim vdim packed operations / 2 per head and token), HBM in decode
// (the state is read and written once per token: 8 dim vdim bytes per head and sequence).
#include "common.cuh"
#include "kernels.cuh"

namespace kd {

constexpr int DR_CONSUMERS = 8, DR_HELPERS = 4;
constexpr int DR_THREADS = (DR_CONSUMERS + DR_HELPERS) * 32;
constexpr int DR_TB = 8;           // tokens per block
constexpr int DR_MAX_TAPS = 8;

struct DeltaParams {
  int B, S, H, Hk, dim, vdim, taps;
  int dk_pad, dv_pad;              // state [B, H, dk_pad, dv_pad]
  int wpu;                         // warps that cover one head's value columns
  int wpc;                         // of them in one CTA (grid.y tiles the rest)
  int upc;                         // heads per CTA
  int q_col, k_col, v_col, b_col;  // columns of a projection row
  int64_t ld;                      // projection row stride (elements)
  int64_t ld_a;                    // row stride of the decay logits
  float q_scale;
  const float* a;                  // [T, H*dim] decay logits (before dt_bias)
  const float* conv_q;             // [Hk*dim, taps]
  const float* conv_k;
  const float* conv_v;             // [H*vdim, taps]
  const float* neg_rate;           // [H] -exp(A_log)
  const float* dt_bias;            // [H*dim]
  float* state;
  float* o;                        // [T, H*vdim]
};

template <typename T> __device__ __forceinline__ float dr_f(T v);
template <> __device__ __forceinline__ float dr_f<float>(float v) { return v; }
template <> __device__ __forceinline__ float dr_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }

__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
  float2 d;
  asm("{\n\t.reg .b64 a, b, c, d;\n\tmov.b64 a, {%2, %3};\n\tmov.b64 b, {%4, %5};\n\tmov.b64 c, {%6, %7};\n\t"
      "fma.rn.f32x2 d, a, b, c;\n\tmov.b64 {%0, %1}, d;\n\t}"
      : "=f"(d.x), "=f"(d.y) : "f"(a.x), "f"(a.y), "f"(b.x), "f"(b.y), "f"(c.x), "f"(c.y));
  return d;
}
__device__ __forceinline__ float2 mul2(float2 a, float2 b) {
  float2 d;
  asm("{\n\t.reg .b64 a, b, d;\n\tmov.b64 a, {%2, %3};\n\tmov.b64 b, {%4, %5};\n\tmul.rn.f32x2 d, a, b;\n\tmov.b64 {%0, %1}, d;\n\t}"
      : "=f"(d.x), "=f"(d.y) : "f"(a.x), "f"(a.y), "f"(b.x), "f"(b.y));
  return d;
}

// Rounded projections enter through bf16 (FAST: special-function-unit forms, error at fp32 rounding
// level for these arguments); the fp32 mode uses the accurate library functions.
template <bool FAST> __device__ __forceinline__ float dr_sigmoid(float x) {
  return FAST ? __fdividef(1.0f, 1.0f + __expf(-x)) : 1.0f / (1.0f + expf(-x));
}
template <bool FAST> __device__ __forceinline__ float dr_softplus(float x) {
  return FAST ? fmaxf(x, 0.f) + __logf(1.0f + __expf(-fabsf(x))) : fmaxf(x, 0.f) + log1pf(expf(-fabsf(x)));
}
template <bool FAST> __device__ __forceinline__ float dr_exp(float x) { return FAST ? __expf(x) : expf(x); }

// out[t][i] = silu(causal convolution) of tokens t0 .. t0 + n - 1 (n <= DR_TB), channels i < nc; zeros up to
// `pad`.  hist holds the taps - 1 inputs before token 0 of this call, [taps-1][C] for the sequence.  A lane
// keeps the inputs of a channel in registers (four taps, the usual size) or re-reads them (other sizes).
template <typename T, bool FAST>
__device__ __forceinline__ void conv_block(const T* __restrict__ proj, int64_t ld, int64_t row0, int t0, int n, int col, const T* __restrict__ hist,
                                           int64_t hist_ld, const float* __restrict__ taps_w, int taps, int nc, int pad, float* __restrict__ out,
                                           int out_ld, int lane) {
  const int halo = taps - 1;
  auto input = [&](int t, int i) -> float {
    return t >= 0 ? dr_f<T>(proj[(row0 + t) * ld + col + i]) : dr_f<T>(hist[(int64_t)(t + halo) * hist_ld + i]);
  };
#pragma unroll 1
  for (int i = lane; i < nc; i += 32) {
    if (taps == 4) {
      float x[DR_TB + 3];
#pragma unroll
      for (int r = 0; r < DR_TB + 3; ++r) x[r] = r < n + 3 ? input(t0 + r - 3, i) : 0.f;
      const float w0 = taps_w[i * 4], w1 = taps_w[i * 4 + 1], w2 = taps_w[i * 4 + 2], w3 = taps_w[i * 4 + 3];
#pragma unroll
      for (int t = 0; t < DR_TB; ++t) {
        if (t < n) {
          const float y = fmaf(x[t + 3], w3, fmaf(x[t + 2], w2, fmaf(x[t + 1], w1, x[t] * w0)));
          out[t * out_ld + i] = y * dr_sigmoid<FAST>(y);
        }
      }
    } else {
      for (int t = 0; t < n; ++t) {
        float y = 0.f;
        for (int j = 0; j < taps; ++j) y = fmaf(input(t0 + t - halo + j, i), taps_w[(int64_t)i * taps + j], y);
        out[t * out_ld + i] = y * dr_sigmoid<FAST>(y);
      }
    }
  }
#pragma unroll 1
  for (int i = nc + lane; i < pad; i += 32)
    for (int t = 0; t < n; ++t) out[t * out_ld + i] = 0.f;
}

// x[t] <- scale x[t] / sqrt(sum x[t]^2 + 1e-6) over nc channels; a lane touches the channels it wrote itself.
__device__ __forceinline__ void unit_rows(float* x, int ld, int n, int nc, float scale, int lane) {
  for (int t = 0; t < n; ++t) {
    float ss = 0.f;
#pragma unroll 1
    for (int i = lane; i < nc; i += 32) ss = fmaf(x[t * ld + i], x[t * ld + i], ss);
    ss = warp_sum(ss);
    const float inv = scale / sqrtf(ss + 1e-6f);
    for (int i = lane; i < nc; i += 32) x[t * ld + i] *= inv;
  }
}

template <typename T, int LPC>
__global__ void __launch_bounds__(DR_THREADS, 1)
delta_rule_kernel(const T* __restrict__ proj, const T* __restrict__ hist, int64_t hist_b, int64_t hist_ld, DeltaParams p) {
  constexpr bool FAST = sizeof(T) == 2;
  constexpr int DK = 32 * LPC;                 // padded key channels
  constexpr int CPW = 4 * (32 / LPC);          // value columns per warp
  extern __shared__ __align__(16) float sm[];
  const int dvc = p.wpc * CPW;                 // value columns of a head in this CTA
  const int unit_floats = DR_TB * (3 * DK + dvc) + DR_TB;
  // shared memory: [2 stages][upc units]{ q, k, g [TB][DK], v [TB][dvc], beta [TB] }

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int units = p.B * p.H;
  const int unit0 = blockIdx.x * p.upc;
  const int col_tile = blockIdx.y * dvc;       // first value column of this CTA inside its heads
  pdl_wait();
  pdl_trigger();
  const int n_blk = (p.S + DR_TB - 1) / DR_TB;

  // ---- helper: everything token block `blk` needs, into stage `st`
  const int hw = warp - DR_CONSUMERS;
  auto prepare = [&](int blk, int st) {
    const int t0 = blk * DR_TB, n = min(DR_TB, p.S - t0);
    for (int item = hw; item < p.upc * 4; item += DR_HELPERS) {
      const int u = item >> 2, what = item & 3;
      const int unit = unit0 + u;
      if (unit >= units) continue;
      const int b = unit / p.H, h = unit - b * p.H;
      const int hk = h / (p.H / p.Hk);
      const int64_t row0 = (int64_t)b * p.S;
      float* base = sm + (st * p.upc + u) * unit_floats;
      const T* hb = hist + (int64_t)b * hist_b;
      const int kc = p.Hk * p.dim;             // history channels: q, k, v side by side
      if (what == 0) {
        conv_block<T, FAST>(proj, p.ld, row0, t0, n, p.q_col + hk * p.dim, hb + hk * p.dim, hist_ld, p.conv_q + (int64_t)hk * p.dim * p.taps, p.taps,
                            p.dim, DK, base, DK, lane);
        unit_rows(base, DK, n, p.dim, p.q_scale, lane);
      } else if (what == 1) {
        float* k = base + DR_TB * DK;
        conv_block<T, FAST>(proj, p.ld, row0, t0, n, p.k_col + hk * p.dim, hb + kc + hk * p.dim, hist_ld, p.conv_k + (int64_t)hk * p.dim * p.taps, p.taps,
                            p.dim, DK, k, DK, lane);
        unit_rows(k, DK, n, p.dim, 1.0f, lane);
      } else if (what == 2) {
        float* g = base + 2 * DR_TB * DK;
        const float rate = p.neg_rate[h];
#pragma unroll 1
        for (int i = lane; i < DK; i += 32) {
          if (i < p.dim) {
            const float bias = p.dt_bias[h * p.dim + i];
#pragma unroll 4
            for (int t = 0; t < n; ++t)
              g[t * DK + i] = dr_exp<FAST>(rate * dr_softplus<FAST>(p.a[(row0 + t0 + t) * p.ld_a + h * p.dim + i] + bias));
          } else {
            for (int t = 0; t < n; ++t) g[t * DK + i] = 0.f;
          }
        }
      } else {
        float* v = base + 3 * DR_TB * DK;
        const int nc = max(0, min(dvc, p.vdim - col_tile));
        conv_block<T, FAST>(proj, p.ld, row0, t0, n, p.v_col + h * p.vdim + col_tile, hb + 2 * kc + h * p.vdim + col_tile, hist_ld,
                            p.conv_v + ((int64_t)h * p.vdim + col_tile) * p.taps, p.taps, nc, dvc, v, dvc, lane);
        if (lane < n) v[DR_TB * dvc + lane] = dr_sigmoid<FAST>(dr_f<T>(proj[(row0 + t0 + lane) * p.ld + p.b_col + h]));
      }
    }
  };

  auto block_barrier = [] { asm volatile("bar.sync 1, %0;" ::"n"(DR_THREADS) : "memory"); };

  if (warp >= DR_CONSUMERS) {
    asm volatile("setmaxnreg.dec.sync.aligned.u32 88;");
    for (int blk = 0; blk < n_blk; ++blk) {
      prepare(blk, blk & 1);      // (its stage was last read two blocks ago, before the previous barrier)
      block_barrier();
    }
    block_barrier();
    return;
  }
  asm volatile("setmaxnreg.inc.sync.aligned.u32 208;");
  // ---- consumer state: rows (i LPC + j) 4 + e (i < 8, e < 4) of columns col .. col + 3
  const int j = lane % LPC, cg = lane / LPC;
  const int u = warp / p.wpc, uw = warp - u * p.wpc;
  const int unit = unit0 + u;
  const int lcol = uw * CPW + cg * 4;          // column inside the CTA's tile
  const int col = col_tile + lcol;
  const bool active = u < p.upc && unit < units && col < p.dv_pad;
  float2 s[4][16];                             // [column][row pair]
  float* srow = nullptr;
  if (active) {
    srow = p.state + ((int64_t)unit * p.dk_pad + j * 4) * p.dv_pad + col;
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float4 v = *reinterpret_cast<const float4*>(srow + (int64_t)(i * LPC * 4 + e) * p.dv_pad);
        if (e & 1) { s[0][i * 2 + (e >> 1)].y = v.x; s[1][i * 2 + (e >> 1)].y = v.y; s[2][i * 2 + (e >> 1)].y = v.z; s[3][i * 2 + (e >> 1)].y = v.w; }
        else { s[0][i * 2 + (e >> 1)].x = v.x; s[1][i * 2 + (e >> 1)].x = v.y; s[2][i * 2 + (e >> 1)].x = v.z; s[3][i * 2 + (e >> 1)].x = v.w; }
      }
  }
  block_barrier();

  const int b = active ? unit / p.H : 0, h = active ? unit - b * p.H : 0;
  for (int blk = 0; blk < n_blk; ++blk) {
    if (active) {
      const float* base = sm + ((blk & 1) * p.upc + u) * unit_floats;
      const int t0 = blk * DR_TB, n = min(DR_TB, p.S - t0);
      float* orow = p.o + ((int64_t)b * p.S + t0) * p.H * p.vdim + (int64_t)h * p.vdim + col;
      for (int t = 0; t < n; ++t) {
        const float4* q4 = reinterpret_cast<const float4*>(base + t * DK) + j;
        const float4* k4 = reinterpret_cast<const float4*>(base + (DR_TB + t) * DK) + j;
        const float4* g4 = reinterpret_cast<const float4*>(base + (2 * DR_TB + t) * DK) + j;
        const float4 v4 = *reinterpret_cast<const float4*>(base + 3 * DR_TB * DK + t * dvc + lcol);
        const float beta = base[3 * DR_TB * DK + DR_TB * dvc + t];
        float2 acc[4][2];
#pragma unroll
        for (int c = 0; c < 4; ++c) acc[c][0] = acc[c][1] = make_float2(0.f, 0.f);
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          const float4 g = g4[i * LPC], k = k4[i * LPC];
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            s[c][2 * i] = mul2(s[c][2 * i], make_float2(g.x, g.y));
            s[c][2 * i + 1] = mul2(s[c][2 * i + 1], make_float2(g.z, g.w));
            acc[c][0] = fma2(s[c][2 * i], make_float2(k.x, k.y), acc[c][0]);
            acc[c][1] = fma2(s[c][2 * i + 1], make_float2(k.z, k.w), acc[c][1]);
          }
        }
        float pr[4];
#pragma unroll
        for (int c = 0; c < 4; ++c) pr[c] = (acc[c][0].x + acc[c][0].y) + (acc[c][1].x + acc[c][1].y);
#pragma unroll
        for (int o = LPC / 2; o > 0; o >>= 1)
#pragma unroll
          for (int c = 0; c < 4; ++c) pr[c] += __shfl_xor_sync(0xffffffffu, pr[c], o);
        const float uu[4] = {beta * (v4.x - pr[0]), beta * (v4.y - pr[1]), beta * (v4.z - pr[2]), beta * (v4.w - pr[3])};
#pragma unroll
        for (int c = 0; c < 4; ++c) acc[c][0] = acc[c][1] = make_float2(0.f, 0.f);
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          const float4 k = k4[i * LPC], q = q4[i * LPC];
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            const float2 uc = make_float2(uu[c], uu[c]);
            s[c][2 * i] = fma2(make_float2(k.x, k.y), uc, s[c][2 * i]);
            s[c][2 * i + 1] = fma2(make_float2(k.z, k.w), uc, s[c][2 * i + 1]);
            acc[c][0] = fma2(s[c][2 * i], make_float2(q.x, q.y), acc[c][0]);
            acc[c][1] = fma2(s[c][2 * i + 1], make_float2(q.z, q.w), acc[c][1]);
          }
        }
#pragma unroll
        for (int c = 0; c < 4; ++c) pr[c] = (acc[c][0].x + acc[c][0].y) + (acc[c][1].x + acc[c][1].y);
#pragma unroll
        for (int o = LPC / 2; o > 0; o >>= 1)
#pragma unroll
          for (int c = 0; c < 4; ++c) pr[c] += __shfl_xor_sync(0xffffffffu, pr[c], o);
        // the lanes of a group share the store: lane j writes columns j, j + LPC, ...
        float* ot = orow + (int64_t)t * p.H * p.vdim;
#pragma unroll
        for (int c = 0; c < 4; ++c)
          if (c % LPC == j % (LPC < 4 ? LPC : 4) && j < 4 && col + c < p.vdim) ot[c] = pr[c];
      }
    }
    block_barrier();
  }
  if (active) {
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = i * 2 + (e >> 1);
        const float4 v = (e & 1) ? make_float4(s[0][r].y, s[1][r].y, s[2][r].y, s[3][r].y) : make_float4(s[0][r].x, s[1][r].x, s[2][r].x, s[3][r].x);
        *reinterpret_cast<float4*>(srow + (int64_t)(i * LPC * 4 + e) * p.dv_pad) = v;
      }
  }
}

// ----------------------------------------------------------------------------- output gate + convolution history
// out[t, h, :] = o / sqrt(mean(o^2) + eps) * w * sigmoid(gate), one warp per (token, head); the blocks
// behind them move the last taps - 1 convolution inputs of every channel into the history.
struct DeltaOutParams {
  int B, S, H, vdim, taps;
  int channels;                 // history channels, columns conv_col .. of a projection row
  int conv_col;
  int64_t ld, ld_gate, hist_b, hist_ld;
  float eps;
  int out_blocks;
};

template <typename T>
__global__ void __launch_bounds__(256)
delta_out_kernel(const float* __restrict__ o, const T* __restrict__ gate, const float* __restrict__ w, const T* __restrict__ proj,
                 T* __restrict__ hist, T* __restrict__ out, DeltaOutParams p) {
  pdl_wait();
  pdl_trigger();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if ((int)blockIdx.x < p.out_blocks) {
    const int64_t item = (int64_t)blockIdx.x * 8 + warp;
    if (item >= (int64_t)p.B * p.S * p.H) return;
    const int64_t t = item / p.H;
    const int h = (int)(item - t * p.H);
    const float* x = o + item * p.vdim;
    float ss = 0.f;
    for (int i = lane; i < p.vdim; i += 32) ss = fmaf(x[i], x[i], ss);
    ss = warp_sum(ss);
    const float inv = 1.0f / sqrtf(ss / (float)p.vdim + p.eps);
    for (int i = lane; i < p.vdim; i += 32) {
      const float g = dr_sigmoid<false>(dr_f<T>(gate[t * p.ld_gate + h * p.vdim + i]));
      const float y = x[i] * inv * w[i] * g;
      if (sizeof(T) == 2) reinterpret_cast<__nv_bfloat16*>(out)[item * p.vdim + i] = __float2bfloat16_rn(y);
      else reinterpret_cast<float*>(out)[item * p.vdim + i] = y;
    }
    return;
  }
  const int64_t c = (int64_t)(blockIdx.x - p.out_blocks) * blockDim.x + threadIdx.x;
  if (c >= (int64_t)p.B * p.channels) return;
  const int b = (int)(c / p.channels), ch = (int)(c - (int64_t)b * p.channels);
  T* hb = hist + (int64_t)b * p.hist_b + ch;
  const int halo = p.taps - 1;
  for (int r = 0; r < halo; ++r) {      // row r <- input at offset S - halo + r of this call (an old row if that is negative)
    const int t = p.S - halo + r;
    hb[(int64_t)r * p.hist_ld] = t >= 0 ? proj[((int64_t)b * p.S + t) * p.ld + p.conv_col + ch] : hb[(int64_t)(t + halo) * p.hist_ld];
  }
}

static int f32_vec(const kd_tensor* t, int64_t n, const char* what, const float** out) {
  KD_REQUIRE(t && t->dtype == KD_F32 && is_contiguous(t) && numel(t) == n, "%s must be contiguous fp32 with %lld elements", what, (long long)n);
  void* p;
  KD_TRY(tensor_ptr(t, &p));
  *out = static_cast<const float*>(p);
  return KD_OK;
}

template <typename T, int LPC>
static int launch_delta(const void* proj, const void* hist, int64_t hist_b, int64_t hist_ld, DeltaParams p) {
  constexpr int CPW = 4 * (32 / LPC), DK = 32 * LPC;
  const int units = p.B * p.H;
  p.wpu = (p.vdim + CPW - 1) / CPW;
  // enough heads to fill the GPU: whole heads per CTA, several if they fit; otherwise split columns
  int col_tiles = (p.wpu + DR_CONSUMERS - 1) / DR_CONSUMERS;
  const int sms = ctx().sm_count;
  while (col_tiles < p.wpu && units * (col_tiles + 1) <= sms) ++col_tiles;
  p.wpc = (p.wpu + col_tiles - 1) / col_tiles;
  col_tiles = (p.wpu + p.wpc - 1) / p.wpc;
  p.upc = 1;
  while ((p.upc + 1) * p.wpc <= DR_CONSUMERS && units * col_tiles > sms * p.upc) ++p.upc;
  const int dvc = p.wpc * CPW;
  auto smem_of = [&](int upc) { return 2 * upc * (DR_TB * (3 * DK + dvc) + DR_TB) * 4; };
  while (p.upc > 1 && smem_of(p.upc) > 220 * 1024) --p.upc;
  const int smem = smem_of(p.upc);
  KD_REQUIRE(smem <= 227 * 1024, "delta rule: %d x %d heads need too much shared memory", p.dim, p.vdim);
  static bool configured[64] = {false};
  if (!configured[ctx().device & 63]) {
    KD_CUDA_CHECK(cudaFuncSetAttribute(delta_rule_kernel<T, LPC>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
    configured[ctx().device & 63] = true;
  }
  dim3 grid((units + p.upc - 1) / p.upc, col_tiles);
  KD_CUDA_CHECK(launch_ex(delta_rule_kernel<T, LPC>, grid, dim3(DR_THREADS), (size_t)smem, (const T*)proj, (const T*)hist, hist_b, hist_ld, p));
  return after_launch("delta_rule_kernel");
}

template <typename T>
static int launch_delta_lpc(const void* proj, const void* hist, int64_t hist_b, int64_t hist_ld, const DeltaParams& p) {
  if (p.dk_pad == 32) return launch_delta<T, 1>(proj, hist, hist_b, hist_ld, p);
  if (p.dk_pad == 64) return launch_delta<T, 2>(proj, hist, hist_b, hist_ld, p);
  if (p.dk_pad == 128) return launch_delta<T, 4>(proj, hist, hist_b, hist_ld, p);
  return launch_delta<T, 8>(proj, hist, hist_b, hist_ld, p);
}

}  // namespace kd

using namespace kd;

KD_API int kd_delta_state_shape(int dim, int vdim, int* rows_out, int* cols_out) {
  KD_REQUIRE(rows_out && cols_out && dim >= 1 && vdim >= 1, "bad argument");
  KD_REQUIRE(dim <= 256, "delta rule: key heads of %d channels; this path handles up to 256", dim);
  int r = 32;
  while (r < dim) r *= 2;
  *rows_out = r;
  *cols_out = (vdim + 3) / 4 * 4;
  return KD_OK;
}

KD_API int kd_delta_rule(const kd_tensor* proj, int q_col, int k_col, int v_col, int b_col, const kd_tensor* decay, int heads, int kv_heads, int dim,
                         int vdim, const kd_tensor* conv_q, const kd_tensor* conv_k, const kd_tensor* conv_v, const kd_tensor* neg_rate,
                         const kd_tensor* dt_bias, const kd_tensor* history, const kd_tensor* state, const kd_tensor* out) {
  KD_TRY(require_init());
  KD_REQUIRE(proj && decay && conv_q && history && state && out, "null tensor");
  KD_REQUIRE(proj->ndim == 3 && proj->strides[2] == 1 && proj->strides[0] == proj->strides[1] * proj->shape[1] && (proj->dtype == KD_BF16 || proj->dtype == KD_F32),
             "proj must be [B,S,N] with evenly spaced rows, bf16 or fp32");
  KD_REQUIRE(heads >= 1 && kv_heads >= 1 && heads % kv_heads == 0 && dim >= 1 && vdim >= 1, "bad head sizes");
  DeltaParams p{};
  p.B = (int)proj->shape[0]; p.S = (int)proj->shape[1]; p.H = heads; p.Hk = kv_heads; p.dim = dim; p.vdim = vdim;
  p.q_col = q_col; p.k_col = k_col; p.v_col = v_col; p.b_col = b_col;
  p.ld = proj->strides[1];
  const int64_t N = proj->shape[2], C = 2ll * kv_heads * dim + (int64_t)heads * vdim;
  KD_REQUIRE(q_col >= 0 && k_col >= 0 && v_col >= 0 && b_col >= 0 && q_col + kv_heads * dim <= N && k_col + kv_heads * dim <= N &&
                 v_col + heads * vdim <= N && b_col + heads <= N, "columns exceed the projection row");
  KD_REQUIRE(conv_q->ndim == 2, "convolution weights must be [channels, taps]");
  p.taps = (int)conv_q->shape[1];
  KD_REQUIRE(p.taps >= 1 && p.taps <= DR_MAX_TAPS, "%d convolution taps; this path handles 1..%d", p.taps, DR_MAX_TAPS);
  KD_TRY(f32_vec(conv_q, (int64_t)kv_heads * dim * p.taps, "conv_q", &p.conv_q));
  KD_TRY(f32_vec(conv_k, (int64_t)kv_heads * dim * p.taps, "conv_k", &p.conv_k));
  KD_TRY(f32_vec(conv_v, (int64_t)heads * vdim * p.taps, "conv_v", &p.conv_v));
  KD_TRY(f32_vec(neg_rate, heads, "neg_rate", &p.neg_rate));
  KD_TRY(f32_vec(dt_bias, (int64_t)heads * dim, "dt_bias", &p.dt_bias));
  KD_TRY(kd_delta_state_shape(dim, vdim, &p.dk_pad, &p.dv_pad));
  const int64_t T = (int64_t)p.B * p.S;
  KD_REQUIRE(decay->dtype == KD_F32 && decay->ndim == 2 && decay->strides[1] == 1 && decay->shape[0] == T && decay->shape[1] >= (int64_t)heads * dim, "decay must be fp32 [T, heads*dim]");
  p.ld_a = decay->strides[0];
  KD_REQUIRE(history->ndim == 3 && history->dtype == proj->dtype && history->strides[2] == 1 && history->shape[0] >= p.B &&
                 history->shape[1] >= p.taps - 1 && history->shape[2] == C, "history must be [B, taps-1, channels] of proj's type");
  KD_REQUIRE(state->dtype == KD_F32 && is_contiguous(state) && state->ndim == 4 && state->shape[0] >= p.B && state->shape[1] == heads &&
                 state->shape[2] == p.dk_pad && state->shape[3] == p.dv_pad, "state must be fp32 [B,heads,%d,%d]", p.dk_pad, p.dv_pad);
  KD_REQUIRE(out->dtype == KD_F32 && is_contiguous(out) && numel(out) == T * heads * vdim, "out must be fp32 [T, heads*vdim]");
  if (T == 0) return KD_OK;
  p.q_scale = (float)(1.0 / sqrt((double)dim));
  void *pp, *pa, *ph, *ps, *po;
  KD_TRY(tensor_ptr(proj, &pp));
  KD_TRY(tensor_ptr(decay, &pa));
  KD_TRY(tensor_ptr(history, &ph));
  KD_TRY(tensor_ptr(state, &ps));
  KD_TRY(tensor_ptr(out, &po));
  KD_REQUIRE((reinterpret_cast<uintptr_t>(ps) & 15) == 0, "state must be 16-byte aligned");
  p.a = static_cast<const float*>(pa);
  p.state = static_cast<float*>(ps);
  p.o = static_cast<float*>(po);
  if (proj->dtype == KD_BF16) return launch_delta_lpc<__nv_bfloat16>(pp, ph, history->strides[0], history->strides[1], p);
  return launch_delta_lpc<float>(pp, ph, history->strides[0], history->strides[1], p);
}

KD_API int kd_delta_out(const kd_tensor* o, const kd_tensor* gate, const kd_tensor* norm_weight, float eps, const kd_tensor* proj, int conv_col, int taps,
                        const kd_tensor* history, const kd_tensor* out) {
  KD_TRY(require_init());
  KD_REQUIRE(o && gate && norm_weight && proj && history && out, "null tensor");
  KD_REQUIRE(proj->ndim == 3 && proj->strides[2] == 1 && proj->strides[0] == proj->strides[1] * proj->shape[1] && (proj->dtype == KD_BF16 || proj->dtype == KD_F32),
             "proj must be [B,S,N] with evenly spaced rows, bf16 or fp32");
  DeltaOutParams p{};
  p.B = (int)proj->shape[0]; p.S = (int)proj->shape[1]; p.taps = taps;
  p.vdim = (int)numel(norm_weight);
  const int64_t T = (int64_t)p.B * p.S;
  if (T == 0) return KD_OK;
  KD_REQUIRE(o->dtype == KD_F32 && is_contiguous(o) && p.vdim > 0 && numel(o) % (T * p.vdim) == 0, "o must be fp32 [T, heads*vdim]");
  p.H = (int)(numel(o) / (T * p.vdim));
  const float* w;
  KD_TRY(f32_vec(norm_weight, p.vdim, "norm_weight", &w));
  KD_REQUIRE(gate->dtype == proj->dtype && gate->ndim == 2 && gate->strides[1] == 1 && gate->shape[0] == T && gate->shape[1] >= (int64_t)p.H * p.vdim, "gate must be [T, heads*vdim] of proj's type");
  KD_REQUIRE(out->dtype == proj->dtype && is_contiguous(out) && numel(out) == numel(o), "out must be [T, heads*vdim] of proj's type");
  KD_REQUIRE(history->ndim == 3 && history->dtype == proj->dtype && history->strides[2] == 1 && history->shape[0] >= p.B && history->shape[1] >= taps - 1 && taps >= 1, "history must be [B, taps-1, channels]");
  p.channels = (int)history->shape[2];
  p.conv_col = conv_col;
  KD_REQUIRE(conv_col >= 0 && conv_col + p.channels <= proj->shape[2], "columns exceed the projection row");
  p.ld = proj->strides[1]; p.ld_gate = gate->strides[0]; p.hist_b = history->strides[0]; p.hist_ld = history->strides[1];
  p.eps = eps;
  p.out_blocks = (int)((T * p.H + 7) / 8);
  const int hist_blocks = taps > 1 ? (int)(((int64_t)p.B * p.channels + 255) / 256) : 0;
  void *po, *pg, *pp, *ph, *pout;
  KD_TRY(tensor_ptr(o, &po));
  KD_TRY(tensor_ptr(gate, &pg));
  KD_TRY(tensor_ptr(proj, &pp));
  KD_TRY(tensor_ptr(history, &ph));
  KD_TRY(tensor_ptr(out, &pout));
  dim3 grid(p.out_blocks + hist_blocks);
  if (proj->dtype == KD_BF16)
    KD_CUDA_CHECK(launch_ex(delta_out_kernel<__nv_bfloat16>, grid, dim3(256), 0, (const float*)po, (const __nv_bfloat16*)pg, w, (const __nv_bfloat16*)pp, (__nv_bfloat16*)ph, (__nv_bfloat16*)pout, p));
  else
    KD_CUDA_CHECK(launch_ex(delta_out_kernel<float>, grid, dim3(256), 0, (const float*)po, (const float*)pg, w, (const float*)pp, (float*)ph, (float*)pout, p));
  return after_launch("delta_out_kernel");
}
