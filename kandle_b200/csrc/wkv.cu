// WKV recurrence (RWKV-style time mixing): a [dim, dim] fp32 state per head with one decay per key channel and
// token, a bonus for the current token, and the token shift in front of it.
//
//   kd_token_shift  mix_n = h + (h' - h) mu_n for several n at once, h' = the previous token's h
//   kd_wkv          o = S^T r + (sum_i r_i u_i k_i) v;  S <- diag(w) S + k v^T,  w = exp(-exp(logit + w0)):
//                   one kernel for prompts and portions, one for a single token
//
// The same design as delta_rule.cu, without its dependent sum: consumer warps keep the state in registers, helper
// warps prepare the next tokens' vectors in shared memory.  Inside a group of four tokens the state is kept divided
// by the product P of the decays so far (r P to read, k / P to write), so a token costs two packed operations per
// pair of state entries and the group one more; a decay below 1e-6 is applied to the state at that token, between
// its read and its write.  Two tokens' outputs are summed over a group's lanes together.
// Eight consumer warps (208 registers a thread) and four helper warps (88); a helper warp prepares four tokens of a
// head in as many lanes as the head has quads of channels, so a warp takes two groups of tokens of a 64-channel head.
// Bound: fp32 pipe in prefill (2.25 dim^2 multiply-adds per head and token), HBM in decode (the state is read and
// written once per token: 8 dim^2 bytes per head and sequence).
#include "common.cuh"
#include "kernels.cuh"
#include "recurrence.cuh"

namespace kd {

// ----------------------------------------------------------------------------- token shift
constexpr int SHIFT_TOKENS = 4;      // tokens a thread walks through
constexpr int SHIFT_MIXES = 8;

struct ShiftParams {
  int S, width, mixes, chunks;       // chunks: groups of SHIFT_TOKENS tokens per sequence
  int64_t h_b, h_s;                  // strides of h: sequence, token
  int64_t out_m;                     // stride of out: mix
  const float* mu;                   // [mixes, width]
};

template <typename T, int V>
__device__ __forceinline__ void load_row(const T* p, float (&v)[V]) {
  if constexpr (V == 4) {
    Raw4<T> r;
    r.load(p);
    r.get(v);
  } else {
    v[0] = rec_f<T>(p[0]);
  }
}

template <typename T, int V>
__device__ __forceinline__ void store_row(T* p, const float (&v)[V]) {
  if constexpr (V == 4 && sizeof(T) == 2) {
    __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    uint2 u;
    u.x = *reinterpret_cast<uint32_t*>(&a);
    u.y = *reinterpret_cast<uint32_t*>(&b);
    *reinterpret_cast<uint2*>(p) = u;
  } else if constexpr (V == 4) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  } else if constexpr (sizeof(T) == 2) {
    p[0] = __float2bfloat16_rn(v[0]);
  } else {
    p[0] = v[0];
  }
}

// grid (sequence x token chunk, columns); `last` [B, width]: the token before this call, then this call's last one.
// The thread of a sequence's first chunk alone reads and then rewrites it.
template <typename T, int V>
__global__ void __launch_bounds__(128)
token_shift_kernel(const T* h, T* last, T* __restrict__ out, ShiftParams p) {
  pdl_wait();
  pdl_trigger();
  const int b = blockIdx.x / p.chunks, s0 = (blockIdx.x - b * p.chunks) * SHIFT_TOKENS;
  const int col = (blockIdx.y * blockDim.x + threadIdx.x) * V;
  if (col >= p.width) return;
  const T* seq = h + (int64_t)b * p.h_b + col;
  float before[V], cur[SHIFT_TOKENS][V];
  T* kept = last + (int64_t)b * p.width + col;
  if (s0 == 0) {
    float end[V];
    load_row<T, V>(kept, before);
    load_row<T, V>(seq + (int64_t)(p.S - 1) * p.h_s, end);
    store_row<T, V>(kept, end);
  } else {
    load_row<T, V>(seq + (int64_t)(s0 - 1) * p.h_s, before);
  }
#pragma unroll
  for (int i = 0; i < SHIFT_TOKENS; ++i) load_row<T, V>(seq + (int64_t)min(s0 + i, p.S - 1) * p.h_s, cur[i]);
  const int64_t row = (int64_t)b * p.S + s0;
  for (int n = 0; n < p.mixes; ++n) {
    float mu[V];
    load_row<float, V>(p.mu + (int64_t)n * p.width + col, mu);
#pragma unroll
    for (int i = 0; i < SHIFT_TOKENS; ++i) {
      if (s0 + i >= p.S) break;
      float y[V];
#pragma unroll
      for (int e = 0; e < V; ++e) y[e] = fmaf((i ? cur[i ? i - 1 : 0][e] : before[e]) - cur[i][e], mu[e], cur[i][e]);
      store_row<T, V>(out + n * p.out_m + (row + i) * p.width + col, y);
    }
  }
}

// ----------------------------------------------------------------------------- recurrence
struct WkvParams {
  int B, S, H, dim;
  int dk_pad, dv_pad;              // state [B, H, dk_pad, dv_pad]
  int wpu;                         // warps that cover one head's columns
  int wpc;                         // of them in one CTA (grid.y tiles the rest)
  int upc;                         // heads per CTA
  int64_t ld;                      // row stride of r, k and v
  int64_t ld_w;                    // row stride of the decay logits
  int vec;                         // rows allow four-channel vector loads
  const float* logits;             // [T, H*dim]
  const float* w0;                 // [H*dim]
  const float* u;                  // [H*dim]
  float* state;
  float* o;                        // [T, H*dim]
};

// exp(-exp(x))
template <bool FAST> __device__ __forceinline__ float double_exp_decay(float x) {
  return FAST ? ex2f(-REC_LOG2E * ex2f(REC_LOG2E * x)) : expf(-expf(x));
}

// Tokens per block: small heads come several to a CTA.
template <int LPC> constexpr int wkv_tokens() { return LPC <= 4 ? 8 : 16; }
// Shared-memory floats of one head and stage: r, k (write side), direct decays [TB][dk], decays left at the end of every
// four tokens [TB/4][dk], v [TB][dv], bonus factors and flags [TB].
__host__ __device__ constexpr int wkv_unit_floats(int tb, int dk, int dv) { return tb * (3 * dk + dv) + (tb / 4) * dk + 2 * tb; }

constexpr int WKV_HELPERS = 4, WKV_THREADS = (REC_CONSUMERS + WKV_HELPERS) * 32;

template <typename T, int LPC>
__global__ void __launch_bounds__(WKV_THREADS, 1)
wkv_kernel(const T* __restrict__ r_in, const T* __restrict__ k_in, const T* __restrict__ v_in, WkvParams p) {
  constexpr bool FAST = sizeof(T) == 2;
  constexpr int TB = wkv_tokens<LPC>();
  constexpr int DK = 16 * LPC;                 // padded key channels
  constexpr int CH = DK > 128 ? DK / 128 : 1;  // helper passes over the key channels
  constexpr int LANES = DK < 128 ? DK / 4 : 32;                          // helper lanes that share a token's channels
  constexpr int GPI = 32 / LANES < TB / 4 ? 32 / LANES : TB / 4;         // groups of four tokens a helper warp takes at once
  constexpr int CPW = 8 * (32 / LPC);          // columns per warp
  extern __shared__ __align__(16) float sm[];
  const int dvc = p.wpc * CPW;                 // columns of a head in this CTA
  const int unit_floats = wkv_unit_floats(TB, DK, dvc);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int units = p.B * p.H;
  const int unit0 = blockIdx.x * p.upc;
  const int col_tile = blockIdx.y * dvc;       // first column of this CTA inside its heads
  const int n_blk = (p.S + TB - 1) / TB;

  // everything token block `blk` needs, into stage `st`; an item is GPI groups of four tokens of one head
  auto prepare = [&](int blk, int st) {
    constexpr int ITEMS = TB / 4 / GPI;
    const int sub = lane / LANES, c0 = (lane % LANES) * 4;
    const unsigned mine = LANES == 32 ? 0xffffffffu : ((1u << LANES) - 1u) << (sub * LANES);
    for (int item = warp - REC_CONSUMERS; item < p.upc * ITEMS; item += WKV_HELPERS) {
      const int un = item / ITEMS, grp = (item % ITEMS) * GPI + (sub < GPI ? sub : 0);
      const int unit = unit0 + un, t = blk * TB + grp * 4;
      if (unit >= units) continue;
      // (all lanes take part in the sums; those of a group past the end or without a group store nothing)
      const bool stores = sub < GPI && t < p.S;
      const int b = unit / p.H, h = unit - b * p.H;
      float* base = sm + (st * p.upc + un) * unit_floats;
      const int64_t row = (int64_t)b * p.S + (t < p.S ? t : 0);
      const int left = p.S - t;                // tokens of this group that exist
      const int at = h * p.dim, nv = max(0, min(dvc, p.dim - col_tile));
      float g[CH][4][4], bonus[4] = {0.f, 0.f, 0.f, 0.f}, least = 1.f;
      Raw4<T> r[CH][4], k[CH][4], v0[4];
      if (p.vec) {
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          const int64_t rq = row + (q < left ? q : 0);
#pragma unroll
          for (int i = 0; i < CH; ++i) {
            const int cc = at + (i * 128 + c0 < p.dim ? i * 128 + c0 : 0);
            const float4 f = *reinterpret_cast<const float4*>(p.logits + rq * p.ld_w + cc);
            g[i][q][0] = f.x; g[i][q][1] = f.y; g[i][q][2] = f.z; g[i][q][3] = f.w;
            r[i][q].load(r_in + rq * p.ld + cc);
            k[i][q].load(k_in + rq * p.ld + cc);
          }
          v0[q].load(v_in + rq * p.ld + at + (c0 < nv ? col_tile + c0 : 0));
        }
      } else {
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          const int64_t rq = row + (q < left ? q : 0);
#pragma unroll
          for (int i = 0; i < CH; ++i) {
            float rr[4], kk[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const int c = i * 128 + c0 + e, cc = at + (c < p.dim ? c : 0);
              g[i][q][e] = p.logits[rq * p.ld_w + cc];
              rr[e] = rec_f<T>(r_in[rq * p.ld + cc]);
              kk[e] = rec_f<T>(k_in[rq * p.ld + cc]);
            }
            r[i][q].set(rr);
            k[i][q].set(kk);
          }
        }
      }
#pragma unroll
      for (int i = 0; i < CH; ++i) {
        const int c = i * 128 + c0;
        float w0[4], u[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          w0[e] = c + e < p.dim ? __ldg(p.w0 + at + c + e) : 0.f;
          u[e] = c + e < p.dim ? __ldg(p.u + at + c + e) : 0.f;
        }
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          float rr[4], kk[4];
          r[i][q].get(rr);
          k[i][q].get(kk);
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const bool use = c + e < p.dim && q < left;
            g[i][q][e] = use ? double_exp_decay<FAST>(g[i][q][e] + w0[e]) : 1.f;
            least = fminf(least, g[i][q][e]);
            bonus[q] = use ? fmaf(rr[e] * u[e], kk[e], bonus[q]) : bonus[q];
          }
        }
      }
#pragma unroll
      for (int o = LANES / 2; o > 0; o >>= 1)
#pragma unroll
        for (int q = 0; q < 4; ++q) bonus[q] += __shfl_xor_sync(0xffffffffu, bonus[q], o);
      bool flag[4] = {false, false, false, false};
      if (__any_sync(0xffffffffu, least < REC_SMALL_DECAY)) {
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          bool small = false;
#pragma unroll
          for (int i = 0; i < CH; ++i)
#pragma unroll
            for (int e = 0; e < 4; ++e) small |= g[i][q][e] < REC_SMALL_DECAY;
          flag[q] = (__ballot_sync(0xffffffffu, small) & mine) != 0;
        }
      }
      if (!stores) continue;
      // P: product of the decays since the last one that was applied directly (or the group's start)
#pragma unroll
      for (int i = 0; i < CH; ++i) {
        const int c = i * 128 + c0;
        float P[4] = {1.f, 1.f, 1.f, 1.f};
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          float rr[4], kk[4];
          r[i][q].get(rr);
          k[i][q].get(kk);
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const bool use = c + e < p.dim && q < left;
            rr[e] = use ? rr[e] * P[e] : 0.f;
            kk[e] = use ? kk[e] : 0.f;
            P[e] *= g[i][q][e];
          }
          if (flag[q]) {
            *reinterpret_cast<float4*>(base + (2 * TB + grp * 4 + q) * DK + c) = make_float4(P[0], P[1], P[2], P[3]);
#pragma unroll
            for (int e = 0; e < 4; ++e) P[e] = 1.f;
          }
#pragma unroll
          for (int e = 0; e < 4; ++e) kk[e] = FAST ? kk[e] * rcpf(P[e]) : kk[e] / P[e];
          *reinterpret_cast<float4*>(base + (grp * 4 + q) * DK + c) = make_float4(rr[0], rr[1], rr[2], rr[3]);
          *reinterpret_cast<float4*>(base + (TB + grp * 4 + q) * DK + c) = make_float4(kk[0], kk[1], kk[2], kk[3]);
        }
        *reinterpret_cast<float4*>(base + (3 * TB + grp) * DK + c) = make_float4(P[0], P[1], P[2], P[3]);
      }
      float* v = base + (3 * TB + TB / 4) * DK;
#pragma unroll 1
      for (int c = c0; c < dvc; c += LANES * 4) {
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          float y[4] = {0.f, 0.f, 0.f, 0.f};
          if (q < left) {
            const T* src = v_in + (row + q) * p.ld + at + col_tile + c;
            if (p.vec) {
              if (c < nv) {
                if (c != c0) v0[q].load(src);
                v0[q].get(y);
              }
            } else {
#pragma unroll
              for (int e = 0; e < 4; ++e) if (c + e < nv) y[e] = rec_f<T>(src[e]);
            }
          }
          *reinterpret_cast<float4*>(v + (grp * 4 + q) * dvc + c) = make_float4(y[0], y[1], y[2], y[3]);
        }
      }
      if (c0 == 0) {                           // bonus factors, then flags, of the group's four tokens
        float* bf = v + TB * dvc + grp * 8;
        *reinterpret_cast<float4*>(bf) = make_float4(bonus[0], bonus[1], bonus[2], bonus[3]);
        *reinterpret_cast<float4*>(bf + 4) = make_float4(flag[0] ? 1.f : 0.f, flag[1] ? 1.f : 0.f, flag[2] ? 1.f : 0.f, flag[3] ? 1.f : 0.f);
      }
    }
  };
  auto block_barrier = [] { asm volatile("bar.sync 1, %0;" ::"n"(WKV_THREADS) : "memory"); };

  if (warp >= REC_CONSUMERS) {
    // (384 threads were launched with 168 registers each: 256 x 208 + 128 x 88 is the same sum)
    asm volatile("setmaxnreg.dec.sync.aligned.u32 88;");
    pdl_wait();
    pdl_trigger();
    for (int blk = 0; blk < n_blk; ++blk) {
      prepare(blk, blk & 1);      // (its stage was last read two blocks ago, before the previous barrier)
      block_barrier();
    }
    block_barrier();
    return;
  }
  asm volatile("setmaxnreg.inc.sync.aligned.u32 208;");
  constexpr int OWN = LPC < 8 ? 8 / LPC : 1;   // columns a lane owns after a sum over its group ...
  const int j = lane % LPC, cg = lane / LPC;
  const int own = j * 8 / LPC;                 // ... starting here
  const int un = warp / p.wpc, uw = warp - un * p.wpc;
  const int unit = unit0 + un;
  const int lcol = uw * CPW + cg * 8;          // column inside the CTA's tile
  const int col = col_tile + lcol;
  const bool live = un < p.upc && unit < units;
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
  const int64_t o_ld = (int64_t)p.H * p.dim;
  float* orow = p.o + (int64_t)b * p.S * o_ld + (int64_t)h * p.dim + col + own;
  int n_own = 0;                               // columns this lane stores
  if (active && (LPC <= 8 || (j & (LPC / 8 - 1)) == 0)) n_own = max(0, min(OWN, p.dim - col - own));
  for (int blk = 0; blk < n_blk; ++blk) {
    // (all lanes of a warp belong to one head; lanes past its columns take part in the shuffles)
    if (live) {
      const float* base = sm + ((blk & 1) * p.upc + un) * unit_floats;
      const float* vb = base + (3 * TB + TB / 4) * DK + lcol;
      const int t0 = blk * TB, n = min(TB, p.S - t0);
      auto read = [&](int t, float (&po)[8]) {
        const float4* r4 = reinterpret_cast<const float4*>(base + t * DK) + j;
        float2 acc[8];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float4 r = r4[i * LPC];
#pragma unroll
          for (int c = 0; c < 8; ++c) acc[c] = i ? fma2(s[c][2 * i], make_float2(r.x, r.y), acc[c]) : mul2(s[c][0], make_float2(r.x, r.y));
#pragma unroll
          for (int c = 0; c < 8; ++c) acc[c] = fma2(s[c][2 * i + 1], make_float2(r.z, r.w), acc[c]);
        }
#pragma unroll
        for (int c = 0; c < 8; ++c) po[c] = acc[c].x + acc[c].y;
      };
      auto write = [&](int t) {
        const float4* k4 = reinterpret_cast<const float4*>(base + (TB + t) * DK) + j;
        const float4 va = *reinterpret_cast<const float4*>(vb + t * dvc), vc = *reinterpret_cast<const float4*>(vb + t * dvc + 4);
        const float v[8] = {va.x, va.y, va.z, va.w, vc.x, vc.y, vc.z, vc.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float4 k = k4[i * LPC];
#pragma unroll
          for (int c = 0; c < 8; ++c) s[c][2 * i] = fma2(make_float2(k.x, k.y), make_float2(v[c], v[c]), s[c][2 * i]);
#pragma unroll
          for (int c = 0; c < 8; ++c) s[c][2 * i + 1] = fma2(make_float2(k.z, k.w), make_float2(v[c], v[c]), s[c][2 * i + 1]);
        }
      };
      auto finish = [&](int t, float bonus, const float (&po)[8]) {
        float* ot = orow + (int64_t)(t0 + t) * o_ld;
#pragma unroll
        for (int i = 0; i < OWN; ++i)
          if (i < n_own && t < n) ot[i] = fmaf(bonus, vb[t * dvc + own + i], po[i]);
      };
      // (tokens past the end of a group of four hold zeros and decays of one)
#pragma unroll 1
      for (int t = 0; t < n; t += 4) {
        const float* bf = base + (3 * TB + TB / 4) * DK + TB * dvc + t * 2;
        const float4 bonus = *reinterpret_cast<const float4*>(bf), flag = *reinterpret_cast<const float4*>(bf + 4);
        float pa[8], pb[8];
        if (flag.x + flag.y + flag.z + flag.w == 0.f) {
          read(t, pa);
          write(t);
          read(t + 1, pb);
          write(t + 1);
          group_sums<LPC>(j, pa, pb);
          finish(t, bonus.x, pa);
          finish(t + 1, bonus.y, pb);
          read(t + 2, pa);
          write(t + 2);
          read(t + 3, pb);
          write(t + 3);
          group_sums<LPC>(j, pa, pb);
          finish(t + 2, bonus.z, pa);
          finish(t + 3, bonus.w, pb);
        } else {
#pragma unroll 1
          for (int q = 0; q < 4; ++q) {
            read(t + q, pa);
            if (bf[4 + q] != 0.f) state_scale<LPC>(s, reinterpret_cast<const float4*>(base + (2 * TB + t + q) * DK) + j);
            write(t + q);
#pragma unroll
            for (int c = 0; c < 8; ++c) pb[c] = 0.f;
            group_sums<LPC>(j, pa, pb);
            finish(t + q, bf[q], pa);
          }
        }
        state_scale<LPC>(s, reinterpret_cast<const float4*>(base + (3 * TB + (t >> 2)) * DK) + j);
      }
    }
    block_barrier();
  }
  if (active) state_store<LPC>(s, srow, p.dv_pad);
}

// One token: 256 threads per (head, 64 columns), as delta_step_kernel; the state is read and written once.
template <typename T, int RPW>
__global__ void __launch_bounds__(256, RPW <= 16 ? 3 : 2)
wkv_step_kernel(const T* __restrict__ r_in, const T* __restrict__ k_in, const T* __restrict__ v_in, WkvParams p) {
  constexpr bool FAST = sizeof(T) == 2;
  constexpr int DK = 8 * RPW;
  __shared__ __align__(16) float rs[DK], ks[DK], gs[DK], vs[64];
  __shared__ __align__(16) float part[16][64];
  __shared__ float red[8];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int unit = blockIdx.x, b = unit / p.H, h = unit - b * p.H;
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
  const int at = h * p.dim;
  float rk = 0.f;
  if (tid < DK) {                             // dim <= 256
    float r = 0.f, k = 0.f, g = 0.f;
    if (tid < p.dim) {
      r = rec_f<T>(r_in[(int64_t)b * p.ld + at + tid]);
      k = rec_f<T>(k_in[(int64_t)b * p.ld + at + tid]);
      g = double_exp_decay<FAST>(p.logits[(int64_t)b * p.ld_w + at + tid] + p.w0[at + tid]);
      rk = r * p.u[at + tid] * k;
    }
    rs[tid] = r;
    ks[tid] = k;
    gs[tid] = g;
  }
  if (tid < 64) vs[tid] = col0 + tid < p.dim ? rec_f<T>(v_in[(int64_t)b * p.ld + at + col0 + tid]) : 0.f;
  rk = warp_sum(rk);
  if (lane == 0) red[warp] = rk;
  __syncthreads();
  const float4 v = *reinterpret_cast<const float4*>(&vs[lcol]);
  float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int row = warp * RPW + 2 * i + half;
    const float r = rs[row], k = ks[row], g = gs[row];
    acc.x = fmaf(s[i].x, r, acc.x); acc.y = fmaf(s[i].y, r, acc.y); acc.z = fmaf(s[i].z, r, acc.z); acc.w = fmaf(s[i].w, r, acc.w);
    s[i].x = fmaf(k, v.x, s[i].x * g); s[i].y = fmaf(k, v.y, s[i].y * g); s[i].z = fmaf(k, v.z, s[i].z * g); s[i].w = fmaf(k, v.w, s[i].w * g);
    if (cols) *reinterpret_cast<float4*>(srow + (int64_t)(2 * i) * p.dv_pad) = s[i];
  }
  *reinterpret_cast<float4*>(&part[warp * 2 + half][lcol]) = acc;
  __syncthreads();
  if (tid < 64 && col0 + tid < p.dim) {
    float bonus = 0.f, o = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) bonus += red[w];
#pragma unroll
    for (int w = 0; w < 16; ++w) o += part[w][tid];
    p.o[((int64_t)b * p.H + h) * p.dim + col0 + tid] = fmaf(bonus, vs[tid], o);
  }
}

template <typename T, int LPC>
static int launch_wkv(const void* r, const void* k, const void* v, WkvParams p) {
  constexpr int CPW = 8 * (32 / LPC), DK = 16 * LPC, TB = wkv_tokens<LPC>();
  const int units = p.B * p.H;
  p.wpu = (p.dim + CPW - 1) / CPW;
  // enough heads to fill the GPU: whole heads per CTA, several if they fit; otherwise split columns
  int col_tiles = (p.wpu + REC_CONSUMERS - 1) / REC_CONSUMERS;
  const int sms = ctx().sm_count;
  while (col_tiles < p.wpu && units * (col_tiles + 1) <= sms) ++col_tiles;
  p.wpc = (p.wpu + col_tiles - 1) / col_tiles;
  col_tiles = (p.wpu + p.wpc - 1) / p.wpc;
  p.upc = 1;
  while ((p.upc + 1) * p.wpc <= REC_CONSUMERS && units * col_tiles > sms * p.upc) ++p.upc;
  const int dvc = p.wpc * CPW;
  auto smem_of = [&](int upc) { return 2 * upc * wkv_unit_floats(TB, DK, dvc) * 4; };
  while (p.upc > 1 && smem_of(p.upc) > 220 * 1024) --p.upc;
  const int smem = smem_of(p.upc);
  KD_REQUIRE(smem <= 227 * 1024, "wkv: heads of %d need too much shared memory", p.dim);
  static bool configured[64] = {false};
  if (!configured[ctx().device & 63]) {
    KD_CUDA_CHECK(cudaFuncSetAttribute(wkv_kernel<T, LPC>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
    configured[ctx().device & 63] = true;
  }
  dim3 grid((units + p.upc - 1) / p.upc, col_tiles);
  KD_CUDA_CHECK(launch_ex(wkv_kernel<T, LPC>, grid, dim3(WKV_THREADS), (size_t)smem, (const T*)r, (const T*)k, (const T*)v, p));
  return after_launch("wkv_kernel");
}

template <typename T>
static int launch_wkv_size(const void* r, const void* k, const void* v, const WkvParams& p) {
  if (p.S == 1) {
    dim3 grid(p.B * p.H, (p.dim + 63) / 64);
    auto kernel = p.dk_pad == 32 ? wkv_step_kernel<T, 4> : p.dk_pad == 64 ? wkv_step_kernel<T, 8> : p.dk_pad == 128 ? wkv_step_kernel<T, 16> : wkv_step_kernel<T, 32>;
    KD_CUDA_CHECK(launch_ex(kernel, grid, dim3(256), 0, (const T*)r, (const T*)k, (const T*)v, p));
    return after_launch("wkv_step_kernel");
  }
  if (p.dk_pad == 32) return launch_wkv<T, 2>(r, k, v, p);
  if (p.dk_pad == 64) return launch_wkv<T, 4>(r, k, v, p);
  if (p.dk_pad == 128) return launch_wkv<T, 8>(r, k, v, p);
  return launch_wkv<T, 16>(r, k, v, p);
}

static int f32_ptr(const kd_tensor* t, int64_t n, const char* what, const float** out) {
  KD_REQUIRE(t && t->dtype == KD_F32 && is_contiguous(t) && numel(t) == n, "%s must be contiguous fp32 with %lld elements", what, (long long)n);
  void* p;
  KD_TRY(tensor_ptr(t, &p));
  *out = static_cast<const float*>(p);
  return KD_OK;
}

}  // namespace kd

using namespace kd;

KD_API int kd_token_shift(const kd_tensor* h, const kd_tensor* mu, const kd_tensor* last, const kd_tensor* out) {
  KD_TRY(require_init());
  KD_REQUIRE(h && mu && last && out, "null tensor");
  KD_REQUIRE(h->ndim == 3 && h->strides[2] == 1 && (h->dtype == KD_BF16 || h->dtype == KD_F32), "h must be [B,S,W], bf16 or fp32");
  const int64_t B = h->shape[0], S = h->shape[1], W = h->shape[2];
  KD_REQUIRE(mu->ndim == 2 && mu->shape[1] == W && mu->shape[0] >= 1 && mu->shape[0] <= SHIFT_MIXES, "mu must be [mixes <= %d, W]", SHIFT_MIXES);
  ShiftParams p{};
  p.S = (int)S; p.width = (int)W; p.mixes = (int)mu->shape[0];
  KD_TRY(f32_ptr(mu, p.mixes * W, "mu", &p.mu));
  KD_REQUIRE(last->ndim == 2 && last->dtype == h->dtype && is_contiguous(last) && last->shape[0] >= B && last->shape[1] == W, "last must be [B,W] of h's type");
  KD_REQUIRE(out->dtype == h->dtype && is_contiguous(out) && numel(out) == p.mixes * B * S * W, "out must be contiguous [mixes,B*S,W] of h's type");
  if (B * S == 0) return KD_OK;
  p.chunks = (int)((S + SHIFT_TOKENS - 1) / SHIFT_TOKENS);
  p.h_b = h->strides[0]; p.h_s = h->strides[1];
  p.out_m = B * S * W;
  void *ph, *pl, *po;
  KD_TRY(tensor_ptr(h, &ph));
  KD_TRY(tensor_ptr(last, &pl));
  KD_TRY(tensor_ptr(out, &po));
  const bool v4 = W % 4 == 0 && p.h_b % 4 == 0 && p.h_s % 4 == 0 &&
                  ((reinterpret_cast<uintptr_t>(ph) | reinterpret_cast<uintptr_t>(pl) | reinterpret_cast<uintptr_t>(po) | reinterpret_cast<uintptr_t>(p.mu)) & 15) == 0;
  const int V = v4 ? 4 : 1;
  dim3 grid((unsigned)(B * p.chunks), (unsigned)((W + 128 * V - 1) / (128 * V)));
  if (h->dtype == KD_BF16) {
    auto k = v4 ? token_shift_kernel<__nv_bfloat16, 4> : token_shift_kernel<__nv_bfloat16, 1>;
    KD_CUDA_CHECK(launch_ex(k, grid, dim3(128), 0, (const __nv_bfloat16*)ph, (__nv_bfloat16*)pl, (__nv_bfloat16*)po, p));
  } else {
    auto k = v4 ? token_shift_kernel<float, 4> : token_shift_kernel<float, 1>;
    KD_CUDA_CHECK(launch_ex(k, grid, dim3(128), 0, (const float*)ph, (float*)pl, (float*)po, p));
  }
  return after_launch("token_shift_kernel");
}

KD_API int kd_wkv(const kd_tensor* r, const kd_tensor* k, const kd_tensor* v, const kd_tensor* logits, const kd_tensor* w0, const kd_tensor* u,
                  const kd_tensor* state, const kd_tensor* out) {
  KD_TRY(require_init());
  KD_REQUIRE(r && k && v && logits && state && out, "null tensor");
  KD_REQUIRE(state->dtype == KD_F32 && is_contiguous(state) && state->ndim == 4, "state must be contiguous fp32 [B,heads,rows,cols]");
  KD_REQUIRE(r->ndim == 3 && (r->dtype == KD_BF16 || r->dtype == KD_F32) && r->strides[2] == 1 && r->strides[0] == r->strides[1] * r->shape[1],
             "r must be [B,S,heads*dim] with evenly spaced rows, bf16 or fp32");
  for (const kd_tensor* t : {k, v})
    KD_REQUIRE(t->ndim == 3 && t->dtype == r->dtype && t->shape[0] == r->shape[0] && t->shape[1] == r->shape[1] && t->shape[2] == r->shape[2] &&
                   t->strides[0] == r->strides[0] && t->strides[1] == r->strides[1] && t->strides[2] == 1, "k and v must have r's shape, type and strides");
  WkvParams p{};
  p.B = (int)r->shape[0]; p.S = (int)r->shape[1]; p.H = (int)state->shape[1];
  const int64_t N = r->shape[2], T = (int64_t)p.B * p.S;
  KD_REQUIRE(p.H >= 1 && N >= p.H && N % p.H == 0, "%lld columns for %d heads", (long long)N, p.H);
  p.dim = (int)(N / p.H);
  KD_TRY(kd_delta_state_shape(p.dim, p.dim, &p.dk_pad, &p.dv_pad));
  KD_REQUIRE(state->shape[0] >= p.B && state->shape[2] == p.dk_pad && state->shape[3] == p.dv_pad, "state must be fp32 [B,heads,%d,%d]", p.dk_pad, p.dv_pad);
  KD_REQUIRE(logits->dtype == KD_F32 && logits->ndim == 2 && logits->strides[1] == 1 && logits->shape[0] == T && logits->shape[1] >= N, "logits must be fp32 [T, heads*dim]");
  KD_TRY(f32_ptr(w0, N, "w0", &p.w0));
  KD_TRY(f32_ptr(u, N, "u", &p.u));
  KD_REQUIRE(out->dtype == KD_F32 && is_contiguous(out) && numel(out) == T * N, "out must be contiguous fp32 [T, heads*dim]");
  if (T == 0) return KD_OK;
  p.ld = r->strides[1];
  p.ld_w = logits->strides[0];
  void *pr, *pk, *pv, *pl, *ps, *po;
  KD_TRY(tensor_ptr(r, &pr));
  KD_TRY(tensor_ptr(k, &pk));
  KD_TRY(tensor_ptr(v, &pv));
  KD_TRY(tensor_ptr(logits, &pl));
  KD_TRY(tensor_ptr(state, &ps));
  KD_TRY(tensor_ptr(out, &po));
  KD_REQUIRE((reinterpret_cast<uintptr_t>(ps) & 15) == 0, "state must be 16-byte aligned");
  const uintptr_t vb = 4 * dtype_size(r->dtype);
  p.vec = p.dim % 4 == 0 && p.ld % 4 == 0 && p.ld_w % 4 == 0 && reinterpret_cast<uintptr_t>(pl) % 16 == 0 &&
          (reinterpret_cast<uintptr_t>(pr) | reinterpret_cast<uintptr_t>(pk) | reinterpret_cast<uintptr_t>(pv)) % vb == 0;
  p.logits = static_cast<const float*>(pl);
  p.state = static_cast<float*>(ps);
  p.o = static_cast<float*>(po);
  if (r->dtype == KD_BF16) return launch_wkv_size<__nv_bfloat16>(pr, pk, pv, p);
  return launch_wkv_size<float>(pr, pk, pv, p);
}
