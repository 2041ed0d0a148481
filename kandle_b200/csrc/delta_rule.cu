// Gated delta rule with one decay per key channel or per head (a linear-attention layer with an
// [dim, vdim] fp32 state per head): one kernel for prompts and portions, one for a single token.
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
// prompt is cut beyond the rounding of the decay products.
//
// Mapping.  A state column (one value channel) never meets another one, so a warp owns 32 / LPC
// groups of 8 columns, and the LPC lanes of a group share its dim rows (16 rows a lane, in quads
// i LPC + j): 128 state registers a lane whatever the size.  Decays are not applied token by token:
// inside a group of four tokens the state is kept divided by the product P of the decays so far, and
// the token's vectors carry the factor (k P and q P to read, k / P to write), so a token costs three
// packed operations per pair of state entries and the group one more.  Where a decay is so small that
// 1 / P could leave the range of fp32 (below 1e-6), it is applied to the state at that token instead.
// S^T k is summed over a group's LPC lanes so that every lane ends with its share of the columns; a
// token's output is summed while the next token's S^T k is, to share the latency.
// A CTA is eight consumer warps (one or more heads) and eight helper warps.  The helpers prepare the
// next block of tokens (convolution, silu, unit norms, decays, step sizes) in shared memory while the
// consumers walk through the current one.
// Bound: fp32 pipe in prefill (3.25 dim vdim multiply-adds per head and token), HBM in decode
// (the state is read and written once per token: 8 dim vdim bytes per head and sequence).
#include "common.cuh"
#include "kernels.cuh"
#include "recurrence.cuh"

namespace kd {

constexpr int DR_CONSUMERS = REC_CONSUMERS, DR_HELPERS = REC_HELPERS;
constexpr int DR_THREADS = REC_THREADS;
constexpr int DR_TB = 16;          // tokens per block
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
  int vec_q, vec_v, vec_a;         // rows allow four-channel vector loads (q and k, v, decay logits)
  int head_decay;                  // one decay per head instead of one per key channel
  const float* a;                  // [T, H*dim] or [T, H] decay logits (before dt_bias)
  const float* conv_q;             // [Hk*dim, taps]
  const float* conv_k;
  const float* conv_v;             // [H*vdim, taps]
  const float* neg_rate;           // [H] -exp(A_log)
  const float* dt_bias;            // [H*dim] or [H]
  float* state;
  float* o;                        // [T, H*vdim]
};

// Shared-memory floats of one head and stage: q, k (read and write side), direct decays [TB][dk], decays left at
// the end of every four tokens [TB/4][dk], v [TB][dv], step sizes and flags [TB].
__host__ __device__ constexpr int delta_unit_floats(int dk, int dv) { return DR_TB * (4 * dk + dv) + (DR_TB / 4) * dk + 2 * DR_TB; }

// exp(rate softplus(x))
template <bool FAST> __device__ __forceinline__ float dr_decay(float rate, float x) {
  if (FAST) {
    const float z = REC_LOG2E * x;
    return ex2f(rate * (fmaxf(z, 0.f) + __log2f(1.0f + ex2f(-fabsf(z)))));
  }
  return expf(rate * (fmaxf(x, 0.f) + log1pf(expf(-fabsf(x)))));
}

// The inputs of one short convolution at four tokens: where they are and how to read them.
template <typename T>
struct ConvSource {
  const T* row0;        // token 0 of the sequence, first channel
  const T* hist;        // the taps - 1 inputs before it
  int64_t ld, hist_ld;
  const float* w;       // [nc, taps]
  int taps, t, S, nc;   // tokens t .. t + 3, those below S
  bool vec;             // vector loads possible, at most four taps
};

// Vector form, first half: seven rows of inputs at channels c .. c + 3, no branch between the loads.
template <typename T>
__device__ __forceinline__ void conv_fetch(const ConvSource<T>& cs, int c, Raw4<T> (&raw)[7]) {
  const int halo = cs.taps - 1, cc = c < cs.nc ? c : 0;
  if (cs.t >= halo && cs.t - halo + 6 < cs.S) {      // all seven rows are rows of this call
    const T* src = cs.row0 + (cs.t - halo) * cs.ld + cc;
#pragma unroll
    for (int r = 0; r < 7; ++r) raw[r].load(src + r * (int)cs.ld);
    return;
  }
#pragma unroll
  for (int r = 0; r < 7; ++r) {
    const int tt = cs.t - halo + r;
    const bool use = r < 3 + cs.taps && tt < cs.S;
    const T* src = !use ? cs.row0 : tt >= 0 ? cs.row0 + (int64_t)tt * cs.ld : cs.hist + (tt + halo) * cs.hist_ld;
    raw[r].load(src + cc);
  }
}

// Vector form, second half: y[token][channel] = silu(conv), zero for channels past nc and tokens past S.
template <typename T, bool FAST>
__device__ __forceinline__ void conv_finish(const ConvSource<T>& cs, int c, const Raw4<T> (&raw)[7], float (&y)[4][4]) {
  float acc[4][4];
#pragma unroll
  for (int q = 0; q < 4; ++q)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[q][e] = 0.f;
  const int cc = c < cs.nc ? c : 0;
  float w[4][4];        // [channel][tap]
  if (cs.taps == 4) {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float4 f = __ldg(reinterpret_cast<const float4*>(cs.w) + cc + e);
      w[e][0] = f.x; w[e][1] = f.y; w[e][2] = f.z; w[e][3] = f.w;
    }
  } else {
#pragma unroll
    for (int e = 0; e < 4; ++e)
#pragma unroll
      for (int k = 0; k < 4; ++k) w[e][k] = k < cs.taps ? __ldg(cs.w + (cc + e) * cs.taps + k) : 0.f;
  }
#pragma unroll
  for (int r = 0; r < 7; ++r) {
    float x[4];
    raw[r].get(x);
    // (rows that no token of this call uses meet a zero weight, or a token past S, whose result is dropped)
#pragma unroll
    for (int q = 0; q < 4; ++q) {
      const int k = r - q;
      if (k >= 0 && k < 4) {
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[q][e] = fmaf(x[e], w[e][k], acc[q][e]);
      }
    }
  }
#pragma unroll
  for (int q = 0; q < 4; ++q)
#pragma unroll
    for (int e = 0; e < 4; ++e) y[q][e] = c < cs.nc && cs.t + q < cs.S ? acc[q][e] * rec_sigmoid<FAST>(acc[q][e]) : 0.f;
}

// Element by element, for sizes or strides that allow no vector loads and for more taps.
template <typename T, bool FAST>
__device__ __forceinline__ void conv_slow(const ConvSource<T>& cs, int c, float (&y)[4][4]) {
  const int halo = cs.taps - 1;
  for (int q = 0; q < 4; ++q)
    for (int e = 0; e < 4; ++e) {
      float acc = 0.f;
      if (c + e < cs.nc && cs.t + q < cs.S)
        for (int k = 0; k < cs.taps; ++k) {
          const int tt = cs.t + q - halo + k;
          acc = fmaf(rec_f<T>(tt >= 0 ? cs.row0[tt * cs.ld + c + e] : cs.hist[(tt + halo) * cs.hist_ld + c + e]), cs.w[(int64_t)(c + e) * cs.taps + k], acc);
        }
      y[q][e] = acc * rec_sigmoid<FAST>(acc);
    }
}

// scale / |y[q]| over the warp's channels (CH passes of 128).
template <bool FAST, int CH>
__device__ __forceinline__ void unit_scale(const float (&y)[CH][4][4], float scale, float (&inv)[4]) {
  float ss[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
  for (int i = 0; i < CH; ++i)
#pragma unroll
    for (int q = 0; q < 4; ++q)
#pragma unroll
      for (int e = 0; e < 4; ++e) ss[q] = fmaf(y[i][q][e], y[i][q][e], ss[q]);
#pragma unroll
  for (int o = 16; o > 0; o >>= 1)
#pragma unroll
    for (int q = 0; q < 4; ++q) ss[q] += __shfl_xor_sync(0xffffffffu, ss[q], o);
#pragma unroll
  for (int q = 0; q < 4; ++q) inv[q] = FAST ? scale * rsqrtf(ss[q] + 1e-6f) : scale / sqrtf(ss[q] + 1e-6f);
}

template <typename T, int LPC>
__global__ void __launch_bounds__(DR_THREADS, 1)
delta_rule_kernel(const T* __restrict__ proj, const T* __restrict__ hist, int64_t hist_b, int64_t hist_ld, DeltaParams p) {
  constexpr bool FAST = sizeof(T) == 2;
  constexpr int DK = 16 * LPC;                 // padded key channels
  constexpr int CH = DK > 128 ? DK / 128 : 1;  // helper passes over the key channels
  constexpr int CPW = 8 * (32 / LPC);          // value columns per warp
  extern __shared__ __align__(16) float sm[];
  const int dvc = p.wpc * CPW;                 // value columns of a head in this CTA
  const int unit_floats = delta_unit_floats(DK, dvc);
  // shared memory: [2 stages][upc units]{ q, kr, kw, d [TB][DK], post [TB/4][DK], v [TB][dvc], (beta, flag) [TB] }

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int units = p.B * p.H;
  const int unit0 = blockIdx.x * p.upc;
  const int col_tile = blockIdx.y * dvc;       // first value column of this CTA inside its heads
  const int n_blk = (p.S + DR_TB - 1) / DR_TB;

  // ---- helper: everything token block `blk` needs, into stage `st`; an item is four tokens of one head
  const int hw = warp - DR_CONSUMERS;
  auto prepare = [&](int blk, int st) {
    for (int item = hw; item < p.upc * (DR_TB / 4); item += DR_HELPERS) {
      const int u = item / (DR_TB / 4), grp = item % (DR_TB / 4);
      const int unit = unit0 + u, t = blk * DR_TB + grp * 4;
      if (unit >= units || t >= p.S) continue;
      const int b = unit / p.H, h = unit - b * p.H;
      const int hk = h / (p.H / p.Hk);
      const T* seq = proj + (int64_t)b * p.S * p.ld;
      const T* hb = hist + (int64_t)b * hist_b;
      const int kc = p.Hk * p.dim;             // history channels: q, k, v side by side
      float* base = sm + (st * p.upc + u) * unit_floats;
      const ConvSource<T> cq{seq + p.q_col + hk * p.dim, hb + hk * p.dim, p.ld, hist_ld, p.conv_q + (int64_t)hk * p.dim * p.taps, p.taps, t, p.S, p.dim, p.vec_q != 0};
      const ConvSource<T> ck{seq + p.k_col + hk * p.dim, hb + kc + hk * p.dim, p.ld, hist_ld, p.conv_k + (int64_t)hk * p.dim * p.taps, p.taps, t, p.S, p.dim, p.vec_q != 0};
      const int at = h * p.vdim + col_tile;
      const ConvSource<T> cv{seq + p.v_col + at, hb + 2 * kc + at, p.ld, hist_ld, p.conv_v + (int64_t)at * p.taps, p.taps, t, p.S,
                             max(0, min(dvc, p.vdim - col_tile)), p.vec_v != 0};
      const int c0 = lane * 4;
      Raw4<T> raw[7];
      float g[CH][4][4];
      const float* a = p.a + ((int64_t)b * p.S + t) * p.ld_a + (p.head_decay ? h : h * p.dim);
      float ah[4] = {0.f, 0.f, 0.f, 0.f};
      if (p.head_decay) {
#pragma unroll
        for (int q = 0; q < 4; ++q) ah[q] = a[(t + q < p.S ? q : 0) * p.ld_a];
      } else
#pragma unroll
      for (int i = 0; i < CH; ++i) {
        const int c = i * 128 + c0;
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          const float* ar = a + (t + q < p.S ? q : 0) * p.ld_a;
          if (p.vec_a) {
            const float4 f = *reinterpret_cast<const float4*>(ar + (c < p.dim ? c : 0));
            g[i][q][0] = f.x; g[i][q][1] = f.y; g[i][q][2] = f.z; g[i][q][3] = f.w;
          } else {
#pragma unroll
            for (int e = 0; e < 4; ++e) g[i][q][e] = c + e < p.dim ? ar[c + e] : 0.f;
          }
        }
      }
      if (CH == 1 && ck.vec) conv_fetch<T>(ck, c0, raw);
      // decays
      const float rate = p.neg_rate[h];
      float least = 1.f;
      if (p.head_decay) {
        const float bias = __ldg(p.dt_bias + h);
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          ah[q] = t + q < p.S ? dr_decay<FAST>(rate, ah[q] + bias) : 1.f;
          least = fminf(least, ah[q]);
#pragma unroll
          for (int i = 0; i < CH; ++i)
#pragma unroll
            for (int e = 0; e < 4; ++e) g[i][q][e] = i * 128 + c0 + e < p.dim ? ah[q] : 1.f;
        }
      } else
#pragma unroll
      for (int i = 0; i < CH; ++i) {
        const int c = i * 128 + c0;
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const bool in = c + e < p.dim;
          const float bias = in ? __ldg(p.dt_bias + h * p.dim + c + e) : 0.f;
#pragma unroll
          for (int q = 0; q < 4; ++q) {
            g[i][q][e] = in && t + q < p.S ? dr_decay<FAST>(rate, g[i][q][e] + bias) : 1.f;
            least = fminf(least, g[i][q][e]);
          }
        }
      }
      // running products of the decays since the last one that was applied directly (or the group's start);
      // g becomes that product, d holds what to multiply the state with where a token is flagged
      bool flag[4] = {false, false, false, false};
      if (__any_sync(0xffffffffu, least < REC_SMALL_DECAY)) {
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          bool small = false;
#pragma unroll
          for (int i = 0; i < CH; ++i)
#pragma unroll
            for (int e = 0; e < 4; ++e) small |= g[i][q][e] < REC_SMALL_DECAY;
          flag[q] = __any_sync(0xffffffffu, small);
        }
      }
      float* dd = base + (3 * DR_TB + grp * 4) * DK;
#pragma unroll
      for (int i = 0; i < CH; ++i) {
        const int c = i * 128 + c0;
        float P[4] = {1.f, 1.f, 1.f, 1.f};
#pragma unroll
        for (int q = 0; q < 4; ++q) {
#pragma unroll
          for (int e = 0; e < 4; ++e) P[e] *= g[i][q][e];
          if (flag[q]) {
            if (c < DK) *reinterpret_cast<float4*>(dd + q * DK + c) = make_float4(P[0], P[1], P[2], P[3]);
#pragma unroll
            for (int e = 0; e < 4; ++e) P[e] = 1.f;
          }
#pragma unroll
          for (int e = 0; e < 4; ++e) g[i][q][e] = P[e];
        }
        if (c < DK) *reinterpret_cast<float4*>(base + (4 * DR_TB + grp) * DK + c) = make_float4(P[0], P[1], P[2], P[3]);
      }
      float y[CH][4][4], inv[4];
      // k: read side k P, write side k / P
      if (CH == 1 && ck.vec) {
        conv_finish<T, FAST>(ck, c0, raw, y[0]);
        conv_fetch<T>(cq, c0, raw);
      } else {
        for (int i = 0; i < CH; ++i) conv_slow<T, FAST>(ck, i * 128 + c0, y[i]);
      }
      unit_scale<FAST, CH>(y, 1.0f, inv);
#pragma unroll
      for (int i = 0; i < CH; ++i) {
        const int c = i * 128 + c0;
        if (c < DK) {
#pragma unroll
          for (int q = 0; q < 4; ++q) {
            float kk[4], r[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              kk[e] = y[i][q][e] * inv[q];
              r[e] = FAST ? rcpf(g[i][q][e]) : 1.0f / g[i][q][e];
            }
            *reinterpret_cast<float4*>(base + (DR_TB + grp * 4 + q) * DK + c) =
                make_float4(kk[0] * g[i][q][0], kk[1] * g[i][q][1], kk[2] * g[i][q][2], kk[3] * g[i][q][3]);
            *reinterpret_cast<float4*>(base + (2 * DR_TB + grp * 4 + q) * DK + c) = make_float4(kk[0] * r[0], kk[1] * r[1], kk[2] * r[2], kk[3] * r[3]);
          }
        }
      }
      if (CH == 1 && cq.vec) {
        conv_finish<T, FAST>(cq, c0, raw, y[0]);
      } else {
        for (int i = 0; i < CH; ++i) conv_slow<T, FAST>(cq, i * 128 + c0, y[i]);
      }
      if (cv.vec && cv.nc > 0) conv_fetch<T>(cv, c0, raw);
      unit_scale<FAST, CH>(y, p.q_scale, inv);
#pragma unroll
      for (int i = 0; i < CH; ++i) {
        const int c = i * 128 + c0;
        if (c < DK) {
#pragma unroll
          for (int q = 0; q < 4; ++q)
            *reinterpret_cast<float4*>(base + (grp * 4 + q) * DK + c) =
                make_float4(y[i][q][0] * inv[q] * g[i][q][0], y[i][q][1] * inv[q] * g[i][q][1], y[i][q][2] * inv[q] * g[i][q][2],
                            y[i][q][3] * inv[q] * g[i][q][3]);
        }
      }
      float* v = base + (4 * DR_TB + DR_TB / 4) * DK;
#pragma unroll 1
      for (int c = c0; c < dvc; c += 128) {
        if (cv.vec && cv.nc > 0) {
          if (c != c0) conv_fetch<T>(cv, c, raw);
          conv_finish<T, FAST>(cv, c, raw, y[0]);
        } else {
          conv_slow<T, FAST>(cv, c, y[0]);
        }
#pragma unroll
        for (int q = 0; q < 4; ++q) *reinterpret_cast<float4*>(v + (grp * 4 + q) * dvc + c) = make_float4(y[0][q][0], y[0][q][1], y[0][q][2], y[0][q][3]);
      }
      if (lane < 4) {
        float* beta = v + DR_TB * dvc;
        beta[2 * (grp * 4 + lane)] = t + lane < p.S ? rec_sigmoid<FAST>(rec_f<T>(seq[(int64_t)(t + lane) * p.ld + p.b_col + h])) : 0.f;
        beta[2 * (grp * 4 + lane) + 1] = (lane == 0 ? flag[0] : lane == 1 ? flag[1] : lane == 2 ? flag[2] : flag[3]) ? 1.f : 0.f;
      }
    }
  };

  auto block_barrier = [] { asm volatile("bar.sync 1, %0;" ::"n"(DR_THREADS) : "memory"); };

  if (warp >= DR_CONSUMERS) {
    asm volatile("setmaxnreg.dec.sync.aligned.u32 80;");
    pdl_wait();
    pdl_trigger();
    for (int blk = 0; blk < n_blk; ++blk) {
      prepare(blk, blk & 1);      // (its stage was last read two blocks ago, before the previous barrier)
      block_barrier();
    }
    block_barrier();
    return;
  }
  asm volatile("setmaxnreg.inc.sync.aligned.u32 176;");
  // ---- consumer state: rows (i LPC + j) 4 + e (i < 4, e < 4) of columns col .. col + 7
  constexpr int OWN = LPC < 8 ? 8 / LPC : 1;   // columns a lane owns after a sum over its group ...
  const int j = lane % LPC, cg = lane / LPC;
  const int own = j * 8 / LPC;                 // ... starting here
  const int u = warp / p.wpc, uw = warp - u * p.wpc;
  const int unit = unit0 + u;
  const int lcol = uw * CPW + cg * 8;          // column inside the CTA's tile
  const int col = col_tile + lcol;
  const bool live = u < p.upc && unit < units;
  const bool active = live && col < p.dv_pad;
  float2 s[8][8];                              // [column][row pair]
  float* srow = nullptr;
  // (the state was last written a whole step ago, before the launch that the grid-dependency wait is for)
  if (active) srow = p.state + ((int64_t)unit * p.dk_pad + j * 4) * p.dv_pad + col;
  state_load<LPC>(s, srow, p.dv_pad);
  pdl_wait();
  pdl_trigger();
  block_barrier();

  const int b = live ? unit / p.H : 0, h = live ? unit - b * p.H : 0;
  float po[8];                                 // this lane's share of the previous token's output
#pragma unroll
  for (int c = 0; c < 8; ++c) po[c] = 0.f;
  const int64_t o_ld = (int64_t)p.H * p.vdim;
  float* orow = p.o + (int64_t)b * p.S * o_ld + (int64_t)h * p.vdim + col + own;
  auto store_out = [&](float* ot, bool any) {
#pragma unroll
    for (int i = 0; i < OWN; ++i)
      if (any && (LPC <= 8 || (j & (LPC / 8 - 1)) == 0) && col + own + i < p.vdim) ot[i] = po[i];
  };
  for (int blk = 0; blk < n_blk; ++blk) {
    // (all lanes of a warp belong to one head; lanes past its columns take part in the shuffles)
    if (live) {
      const float* base = sm + ((blk & 1) * p.upc + u) * unit_floats;
      const float* vb = base + (4 * DR_TB + DR_TB / 4) * DK;
      const int t0 = blk * DR_TB, n = min(DR_TB, p.S - t0);
#pragma unroll 1
      for (int t = 0; t < n; ++t) {
        const float4* q4 = reinterpret_cast<const float4*>(base + t * DK) + j;
        const float4* kr4 = reinterpret_cast<const float4*>(base + (DR_TB + t) * DK) + j;
        const float4* kw4 = reinterpret_cast<const float4*>(base + (2 * DR_TB + t) * DK) + j;
        const float2 bf = *reinterpret_cast<const float2*>(vb + DR_TB * dvc + 2 * t);     // step size, flag
        float v[OWN];
#pragma unroll
        for (int i = 0; i < OWN; ++i) v[i] = vb[t * dvc + lcol + own + i];
        if (bf.y != 0.f) state_scale<LPC>(s, reinterpret_cast<const float4*>(base + (3 * DR_TB + t) * DK) + j);
        float2 acc[8];
#pragma unroll
        for (int c = 0; c < 8; ++c) acc[c] = make_float2(0.f, 0.f);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float4 k = kr4[i * LPC];
#pragma unroll
          for (int c = 0; c < 8; ++c) acc[c] = fma2(s[c][2 * i], make_float2(k.x, k.y), acc[c]);
#pragma unroll
          for (int c = 0; c < 8; ++c) acc[c] = fma2(s[c][2 * i + 1], make_float2(k.z, k.w), acc[c]);
        }
        float pr[8];
#pragma unroll
        for (int c = 0; c < 8; ++c) pr[c] = acc[c].x + acc[c].y;
        // the previous token's output leaves here: its shuffles fill the wait for this token's
        group_sums<LPC>(j, pr, po);
        store_out(orow + (int64_t)(t0 + t - 1) * o_ld, t0 + t > 0);
#pragma unroll
        for (int i = 0; i < OWN; ++i) pr[i] = bf.x * (v[i] - pr[i]);
        float uu[8];
#pragma unroll
        for (int c = 0; c < 8; ++c) uu[c] = __shfl_sync(0xffffffffu, pr[c % OWN], cg * LPC + c * LPC / 8);
#pragma unroll
        for (int c = 0; c < 8; ++c) acc[c] = make_float2(0.f, 0.f);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float4 k = kw4[i * LPC], q = q4[i * LPC];
#pragma unroll
          for (int c = 0; c < 8; ++c) s[c][2 * i] = fma2(make_float2(k.x, k.y), make_float2(uu[c], uu[c]), s[c][2 * i]);
#pragma unroll
          for (int c = 0; c < 8; ++c) s[c][2 * i + 1] = fma2(make_float2(k.z, k.w), make_float2(uu[c], uu[c]), s[c][2 * i + 1]);
#pragma unroll
          for (int c = 0; c < 8; ++c) acc[c] = fma2(s[c][2 * i], make_float2(q.x, q.y), acc[c]);
#pragma unroll
          for (int c = 0; c < 8; ++c) acc[c] = fma2(s[c][2 * i + 1], make_float2(q.z, q.w), acc[c]);
        }
#pragma unroll
        for (int c = 0; c < 8; ++c) po[c] = acc[c].x + acc[c].y;
        if ((t & 3) == 3 || t + 1 == n) state_scale<LPC>(s, reinterpret_cast<const float4*>(base + (4 * DR_TB + (t >> 2)) * DK) + j);
      }
      if (blk + 1 == n_blk) {
        float none[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
        group_sums<LPC>(j, po, none);
        store_out(orow + (int64_t)(p.S - 1) * o_ld, true);
      }
    }
    block_barrier();
  }
  if (active) state_store<LPC>(s, srow, p.dv_pad);
}

// ----------------------------------------------------------------------------- one token (decode)
// The state of a head is read and written once: HBM-bound.  256 threads per (head, 64 value columns): warp r
// holds rows r RPW .. of the state, a lane four columns of every second one; all loads are issued before anything
// is waited for, and three blocks share an SM.
template <typename T, int RPW>
__global__ void __launch_bounds__(256, RPW <= 16 ? 3 : 2)
delta_step_kernel(const T* __restrict__ proj, const T* __restrict__ hist, int64_t hist_b, int64_t hist_ld, DeltaParams p) {
  constexpr bool FAST = sizeof(T) == 2;
  constexpr int DK = 8 * RPW;
  __shared__ __align__(16) float qs[DK], ksm[DK], gs[DK], vs[64];
  __shared__ __align__(16) float part[16][64];
  __shared__ float red[2][8];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int unit = blockIdx.x, b = unit / p.H, h = unit - b * p.H, hk = h / (p.H / p.Hk);
  constexpr int NR = RPW / 2;                 // rows a lane: half a warp covers 64 columns of a row
  const int half = lane >> 4, lcol = (lane & 15) * 4;
  const int col0 = blockIdx.y * 64, col = col0 + lcol;
  const bool cols = col < p.dv_pad;
  float* srow = p.state + ((int64_t)unit * p.dk_pad + warp * RPW + half) * p.dv_pad + (cols ? col : 0);
  float4 s[NR];
  // (written a whole step ago, before the launch that the grid-dependency wait is for)
#pragma unroll
  for (int i = 0; i < NR; ++i) s[i] = *reinterpret_cast<const float4*>(srow + (int64_t)(2 * i) * p.dv_pad);
  pdl_wait();
  pdl_trigger();
  const T* row = proj + (int64_t)b * p.ld;
  const T* hb = hist + (int64_t)b * hist_b;
  const int kc = p.Hk * p.dim, halo = p.taps - 1;
  // (up to four taps: every input and weight is requested before the first is used)
  auto fetch = [&](int column, int channel, const float* w, float (&x)[4], float (&wt)[4]) {
#pragma unroll
    for (int k = 0; k < 4; ++k) {             // k taps back
      x[k] = k == 0 ? rec_f<T>(row[column]) : k <= halo ? rec_f<T>(hb[(int64_t)(halo - k) * hist_ld + channel]) : 0.f;
      wt[k] = k <= halo ? w[halo - k] : 0.f;
    }
  };
  auto finish = [&](int channel, const float* w, const float (&x)[4], const float (&wt)[4]) {
    float y = fmaf(x[3], wt[3], fmaf(x[2], wt[2], fmaf(x[1], wt[1], x[0] * wt[0])));
    for (int k = 4; k <= halo; ++k) y = fmaf(rec_f<T>(hb[(int64_t)(halo - k) * hist_ld + channel]), w[halo - k], y);
    return y * rec_sigmoid<FAST>(y);
  };
  float xq[4], wq[4], xk[4], wk[4], xv[4], wv[4], decay = 0.f, bias = 0.f;
  const int cq = hk * p.dim + tid, cv = h * p.vdim + col0 + tid, ca = p.head_decay ? h : h * p.dim + tid;
  const bool has_v = tid < 64 && col0 + tid < p.vdim;
  if (tid < p.dim) {                          // dim <= 256
    fetch(p.q_col + cq, cq, p.conv_q + (int64_t)cq * p.taps, xq, wq);
    fetch(p.k_col + cq, kc + cq, p.conv_k + (int64_t)cq * p.taps, xk, wk);
    decay = p.a[(int64_t)b * p.ld_a + ca];
    bias = p.dt_bias[ca];
  }
  if (has_v) fetch(p.v_col + cv, 2 * kc + cv, p.conv_v + (int64_t)cv * p.taps, xv, wv);
  const float beta = rec_sigmoid<FAST>(rec_f<T>(row[p.b_col + h]));
  float q = 0.f, k = 0.f;
  if (tid < p.dim) {
    q = finish(cq, p.conv_q + (int64_t)cq * p.taps, xq, wq);
    k = finish(kc + cq, p.conv_k + (int64_t)cq * p.taps, xk, wk);
    gs[tid] = dr_decay<FAST>(p.neg_rate[h], decay + bias);
  } else if (tid < DK) {
    gs[tid] = 0.f;
  }
  if (tid < 64) vs[tid] = has_v ? finish(2 * kc + cv, p.conv_v + (int64_t)cv * p.taps, xv, wv) : 0.f;
  const float sq = warp_sum(q * q), sk = warp_sum(k * k);
  if (lane == 0) { red[0][warp] = sq; red[1][warp] = sk; }
  __syncthreads();
  float nq = 0.f, nk = 0.f;
#pragma unroll
  for (int w = 0; w < 8; ++w) { nq += red[0][w]; nk += red[1][w]; }
  if (tid < DK) {
    qs[tid] = q * (p.q_scale / sqrtf(nq + 1e-6f));
    ksm[tid] = k * (1.0f / sqrtf(nk + 1e-6f));
  }
  __syncthreads();
  float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const float g = gs[warp * RPW + 2 * i + half], kk = ksm[warp * RPW + 2 * i + half];
    s[i].x *= g; s[i].y *= g; s[i].z *= g; s[i].w *= g;
    acc.x = fmaf(s[i].x, kk, acc.x); acc.y = fmaf(s[i].y, kk, acc.y); acc.z = fmaf(s[i].z, kk, acc.z); acc.w = fmaf(s[i].w, kk, acc.w);
  }
  *reinterpret_cast<float4*>(&part[warp * 2 + half][lcol]) = acc;
  __syncthreads();
  float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int w = 0; w < 16; ++w) {
    const float4 x = *reinterpret_cast<const float4*>(&part[w][lcol]);
    u.x += x.x; u.y += x.y; u.z += x.z; u.w += x.w;
  }
  const float4 v = *reinterpret_cast<const float4*>(&vs[lcol]);
  u.x = beta * (v.x - u.x); u.y = beta * (v.y - u.y); u.z = beta * (v.z - u.z); u.w = beta * (v.w - u.w);
  __syncthreads();
  acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const float kk = ksm[warp * RPW + 2 * i + half], qq = qs[warp * RPW + 2 * i + half];
    s[i].x = fmaf(kk, u.x, s[i].x); s[i].y = fmaf(kk, u.y, s[i].y); s[i].z = fmaf(kk, u.z, s[i].z); s[i].w = fmaf(kk, u.w, s[i].w);
    acc.x = fmaf(s[i].x, qq, acc.x); acc.y = fmaf(s[i].y, qq, acc.y); acc.z = fmaf(s[i].z, qq, acc.z); acc.w = fmaf(s[i].w, qq, acc.w);
    if (cols) *reinterpret_cast<float4*>(srow + (int64_t)(2 * i) * p.dv_pad) = s[i];
  }
  *reinterpret_cast<float4*>(&part[warp * 2 + half][lcol]) = acc;
  __syncthreads();
  if (tid < 64 && col0 + tid < p.vdim) {
    float o = 0.f;
#pragma unroll
    for (int w = 0; w < 16; ++w) o += part[w][tid];
    p.o[((int64_t)b * p.H + h) * p.vdim + col0 + tid] = o;
  }
}

template <typename T>
static int launch_delta_step(const void* proj, const void* hist, int64_t hist_b, int64_t hist_ld, const DeltaParams& p) {
  dim3 grid(p.B * p.H, (p.vdim + 63) / 64);
  auto k = p.dk_pad == 32 ? delta_step_kernel<T, 4> : p.dk_pad == 64 ? delta_step_kernel<T, 8> : p.dk_pad == 128 ? delta_step_kernel<T, 16> : delta_step_kernel<T, 32>;
  KD_CUDA_CHECK(launch_ex(k, grid, dim3(256), 0, (const T*)proj, (const T*)hist, hist_b, hist_ld, p));
  return after_launch("delta_step_kernel");
}

// ----------------------------------------------------------------------------- output gate + convolution history
// out[t, h, :] = o / sqrt(mean(o^2) + eps) * w * act(gate), act = sigmoid or silu, one warp per (token, head); the
// blocks behind them move the last taps - 1 convolution inputs of every channel into the history.
struct DeltaOutParams {
  int B, S, H, vdim, taps;
  int channels;                 // history channels, columns conv_col .. of a projection row
  int conv_col;
  int64_t ld, ld_gate, hist_b, hist_ld;
  float eps;
  int out_blocks;
  int gate_silu;                // the gate passes silu instead of sigmoid
  int w_head;                   // norm weights: stride from one head's to the next (0: shared by the heads)
};

// LPH lanes a head (vdim = 4 LPH), 32 / LPH heads a warp; LPH = 0: any size, one head a warp.
template <typename T, int LPH>
__global__ void __launch_bounds__(256)
delta_out_kernel(const float* __restrict__ o, const T* __restrict__ gate, const float* __restrict__ w, const T* __restrict__ proj,
                 T* __restrict__ hist, T* __restrict__ out, DeltaOutParams p) {
  pdl_wait();
  pdl_trigger();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (LPH > 0 && (int)blockIdx.x < p.out_blocks) {
    constexpr int HEADS = LPH > 0 ? 32 / (LPH > 0 ? LPH : 1) : 1;
    const int64_t items = (int64_t)p.B * p.S * p.H, own = ((int64_t)blockIdx.x * 8 + warp) * HEADS + lane / (LPH > 0 ? LPH : 1);
    const int64_t item = own < items ? own : items - 1;      // (lanes without a head join the sums)
    const int64_t t = item / p.H;
    const int h = (int)(item - t * p.H), c = (lane % (LPH > 0 ? LPH : 1)) * 4;
    const float4 x = *reinterpret_cast<const float4*>(o + item * p.vdim + c);
    Raw4<T> graw;
    graw.load(gate + t * p.ld_gate + h * p.vdim + c);
    const float4 wv = *reinterpret_cast<const float4*>(w + h * p.w_head + c);
    float ss = fmaf(x.x, x.x, fmaf(x.y, x.y, fmaf(x.z, x.z, x.w * x.w)));
#pragma unroll
    for (int k = LPH / 2; k > 0; k >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, k);
    if (own >= items) return;
    const float inv = 1.0f / sqrtf(ss / (float)p.vdim + p.eps);
    float z[4];
    graw.get(z);
    const float xs[4] = {x.x, x.y, x.z, x.w}, ws[4] = {wv.x, wv.y, wv.z, wv.w};
    float y[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float g = rec_sigmoid<sizeof(T) == 2>(z[e]);
      y[e] = xs[e] * inv * ws[e] * (p.gate_silu ? z[e] * g : g);
    }
    if constexpr (sizeof(T) == 2) {
      __nv_bfloat162 a = __floats2bfloat162_rn(y[0], y[1]), b = __floats2bfloat162_rn(y[2], y[3]);
      uint2 u;
      u.x = *reinterpret_cast<uint32_t*>(&a);
      u.y = *reinterpret_cast<uint32_t*>(&b);
      *reinterpret_cast<uint2*>(out + item * p.vdim + c) = u;
    } else {
      *reinterpret_cast<float4*>(out + item * p.vdim + c) = make_float4(y[0], y[1], y[2], y[3]);
    }
    return;
  }
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
      const float z = rec_f<T>(gate[t * p.ld_gate + h * p.vdim + i]), g = rec_sigmoid<false>(z);
      const float y = x[i] * inv * w[h * p.w_head + i] * (p.gate_silu ? z * g : g);
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

template <typename T>
static int launch_delta_out(const float* o, const T* gate, const float* w, const T* proj, T* hist, T* out, DeltaOutParams p) {
  const bool vec = p.ld_gate % 4 == 0 && p.w_head % 4 == 0 && reinterpret_cast<uintptr_t>(gate) % (4 * sizeof(T)) == 0 &&
                   ((reinterpret_cast<uintptr_t>(o) | reinterpret_cast<uintptr_t>(w) | reinterpret_cast<uintptr_t>(out)) & 15) == 0;
  const int lph = vec && (p.vdim == 16 || p.vdim == 32 || p.vdim == 64 || p.vdim == 128) ? p.vdim / 4 : 0;
  const int64_t per = lph ? 8 * (32 / lph) : 8;
  p.out_blocks = (int)(((int64_t)p.B * p.S * p.H + per - 1) / per);
  const int hist_blocks = p.taps > 1 ? (int)(((int64_t)p.B * p.channels + 255) / 256) : 0;
  auto k = lph == 4 ? delta_out_kernel<T, 4> : lph == 8 ? delta_out_kernel<T, 8> : lph == 16 ? delta_out_kernel<T, 16> : lph == 32 ? delta_out_kernel<T, 32> : delta_out_kernel<T, 0>;
  KD_CUDA_CHECK(launch_ex(k, dim3(p.out_blocks + hist_blocks), dim3(256), 0, o, gate, w, proj, hist, out, p));
  return after_launch("delta_out_kernel");
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
  constexpr int CPW = 8 * (32 / LPC), DK = 16 * LPC;
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
  auto smem_of = [&](int upc) { return 2 * upc * delta_unit_floats(DK, dvc) * 4; };
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
  if (p.S == 1) return launch_delta_step<T>(proj, hist, hist_b, hist_ld, p);
  if (p.dk_pad == 32) return launch_delta<T, 2>(proj, hist, hist_b, hist_ld, p);
  if (p.dk_pad == 64) return launch_delta<T, 4>(proj, hist, hist_b, hist_ld, p);
  if (p.dk_pad == 128) return launch_delta<T, 8>(proj, hist, hist_b, hist_ld, p);
  return launch_delta<T, 16>(proj, hist, hist_b, hist_ld, p);
}

}  // namespace kd

using namespace kd;

KD_API int kd_delta_state_shape(int dim, int vdim, int* rows_out, int* cols_out) {
  KD_REQUIRE(rows_out && cols_out && dim >= 1 && vdim >= 1, "bad argument");
  KD_REQUIRE(dim <= 256, "delta rule: key heads of %d channels; this path handles up to 256", dim);
  int r = 32;
  while (r < dim) r *= 2;
  *rows_out = r;
  *cols_out = (vdim + 7) / 8 * 8;
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
  // (one decay per head: a bias for every head; with key heads of one channel the two forms are the same)
  p.head_decay = dt_bias && numel(dt_bias) == heads;
  const int64_t decays = p.head_decay ? heads : (int64_t)heads * dim;
  KD_TRY(f32_vec(dt_bias, decays, "dt_bias", &p.dt_bias));
  KD_TRY(kd_delta_state_shape(dim, vdim, &p.dk_pad, &p.dv_pad));
  const int64_t T = (int64_t)p.B * p.S;
  KD_REQUIRE(decay->dtype == KD_F32 && decay->ndim == 2 && decay->strides[1] == 1 && decay->shape[0] == T && decay->shape[1] >= decays, "decay must be fp32 [T, heads*dim] or [T, heads], like dt_bias");
  p.ld_a = decay->strides[0];
  KD_REQUIRE(history->ndim == 3 && history->dtype == proj->dtype && history->strides[2] == 1 && history->shape[0] >= p.B &&
                 history->shape[1] >= p.taps - 1 && history->shape[2] == C, "history must be [B, taps-1, channels] of proj's type");
  KD_REQUIRE(state->dtype == KD_F32 && is_contiguous(state) && state->ndim == 4 && state->shape[0] >= p.B && state->shape[1] == heads &&
                 state->shape[2] == p.dk_pad && state->shape[3] == p.dv_pad, "state must be fp32 [B,heads,%d,%d]", p.dk_pad, p.dv_pad);
  KD_REQUIRE(out->dtype == KD_F32 && is_contiguous(out) && numel(out) == T * heads * vdim, "out must be fp32 [T, heads*vdim]");
  if (T == 0) return KD_OK;
  KD_REQUIRE((int64_t)p.S * p.ld < (1ll << 31), "delta rule: %d tokens of %lld columns in one call", p.S, (long long)p.ld);
  p.q_scale = (float)(1.0 / sqrt((double)dim));
  void *pp, *pa, *ph, *ps, *po;
  KD_TRY(tensor_ptr(proj, &pp));
  KD_TRY(tensor_ptr(decay, &pa));
  KD_TRY(tensor_ptr(history, &ph));
  KD_TRY(tensor_ptr(state, &ps));
  KD_TRY(tensor_ptr(out, &po));
  KD_REQUIRE((reinterpret_cast<uintptr_t>(ps) & 15) == 0, "state must be 16-byte aligned");
  p.a = static_cast<const float*>(pa);
  const int vb = 4 * dtype_size(proj->dtype);
  const bool rows_ok = p.ld % 4 == 0 && history->strides[0] % 4 == 0 && history->strides[1] % 4 == 0 &&
                       reinterpret_cast<uintptr_t>(pp) % vb == 0 && reinterpret_cast<uintptr_t>(ph) % vb == 0;
  p.vec_q = rows_ok && p.taps <= 4 && dim % 4 == 0 && q_col % 4 == 0 && k_col % 4 == 0;
  p.vec_v = rows_ok && p.taps <= 4 && vdim % 4 == 0 && v_col % 4 == 0 && kv_heads * dim % 2 == 0;
  p.vec_a = dim % 4 == 0 && p.ld_a % 4 == 0 && reinterpret_cast<uintptr_t>(pa) % 16 == 0;
  p.state = static_cast<float*>(ps);
  p.o = static_cast<float*>(po);
  if (proj->dtype == KD_BF16) return launch_delta_lpc<__nv_bfloat16>(pp, ph, history->strides[0], history->strides[1], p);
  return launch_delta_lpc<float>(pp, ph, history->strides[0], history->strides[1], p);
}

KD_API int kd_delta_out(const kd_tensor* o, const kd_tensor* gate, const kd_tensor* norm_weight, float eps, int gate_act, const kd_tensor* proj,
                        int conv_col, int taps, const kd_tensor* history, const kd_tensor* out) {
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
  KD_REQUIRE(gate_act == KD_GATE_SIGMOID || gate_act == KD_GATE_SILU, "unknown gate activation %d", gate_act);
  p.gate_silu = gate_act == KD_GATE_SILU;
  void *po, *pg, *pp, *ph, *pout;
  KD_TRY(tensor_ptr(o, &po));
  KD_TRY(tensor_ptr(gate, &pg));
  KD_TRY(tensor_ptr(proj, &pp));
  KD_TRY(tensor_ptr(history, &ph));
  KD_TRY(tensor_ptr(out, &pout));
  if (proj->dtype == KD_BF16)
    return launch_delta_out<__nv_bfloat16>((const float*)po, (const __nv_bfloat16*)pg, w, (const __nv_bfloat16*)pp, (__nv_bfloat16*)ph, (__nv_bfloat16*)pout, p);
  return launch_delta_out<float>((const float*)po, (const float*)pg, w, (const float*)pp, (float*)ph, (float*)pout, p);
}

KD_API int kd_gated_head_norm(const kd_tensor* o, const kd_tensor* gate, const kd_tensor* norm_weight, int heads, float eps, int gate_act,
                              const kd_tensor* out) {
  KD_TRY(require_init());
  KD_REQUIRE(o && gate && norm_weight && out, "null tensor");
  KD_REQUIRE(o->dtype == KD_F32 && o->ndim == 2 && is_contiguous(o) && heads >= 1 && o->shape[1] % heads == 0 && o->shape[1] > 0, "o must be contiguous fp32 [T, heads*vdim]");
  KD_REQUIRE(gate_act == KD_GATE_SIGMOID || gate_act == KD_GATE_SILU, "unknown gate activation %d", gate_act);
  DeltaOutParams p{};
  const int64_t T = o->shape[0];
  p.B = 1; p.S = (int)T; p.H = heads; p.vdim = (int)(o->shape[1] / heads); p.taps = 1;
  p.eps = eps;
  p.gate_silu = gate_act == KD_GATE_SILU;
  p.w_head = numel(norm_weight) == p.vdim ? 0 : p.vdim;
  const float* w;
  KD_TRY(f32_vec(norm_weight, p.w_head ? o->shape[1] : p.vdim, "norm_weight", &w));
  KD_REQUIRE((gate->dtype == KD_BF16 || gate->dtype == KD_F32) && gate->ndim == 2 && gate->strides[1] == 1 && gate->shape[0] == T && gate->shape[1] >= o->shape[1], "gate must be [T, heads*vdim], bf16 or fp32");
  KD_REQUIRE(out->dtype == gate->dtype && is_contiguous(out) && numel(out) == numel(o), "out must be [T, heads*vdim] of gate's type");
  if (T == 0) return KD_OK;
  p.ld_gate = gate->strides[0];
  void *po, *pg, *pout;
  KD_TRY(tensor_ptr(o, &po));
  KD_TRY(tensor_ptr(gate, &pg));
  KD_TRY(tensor_ptr(out, &pout));
  if (gate->dtype == KD_BF16)
    return launch_delta_out<__nv_bfloat16>((const float*)po, (const __nv_bfloat16*)pg, w, nullptr, nullptr, (__nv_bfloat16*)pout, p);
  return launch_delta_out<float>((const float*)po, (const float*)pg, w, nullptr, nullptr, (float*)pout, p);
}
