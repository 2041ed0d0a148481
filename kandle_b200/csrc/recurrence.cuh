// Shared by the recurrent layers whose state is a [dim, vdim] fp32 matrix per head (delta_rule.cu, wkv.cu):
// elementary functions, packed arithmetic, and the state held in registers.
//
// A warp owns 32 / LPC groups of 8 state columns; the LPC lanes of a group share the rows, 16 a lane: lane j
// holds rows (i LPC + j) 4 + e (i < 4, e < 4), as s[column][row pair].  State in memory is
// [B, heads, rows, columns] with rows = 16 LPC and columns padded to a multiple of 8.
#pragma once
#include "common.cuh"

namespace kd {

constexpr int REC_CONSUMERS = 8, REC_HELPERS = 8;       // warps that hold the state; warps that prepare its inputs
constexpr int REC_THREADS = (REC_CONSUMERS + REC_HELPERS) * 32;
// Decays below this are applied to the state at once; products of four larger ones keep 1 / P in range.
constexpr float REC_SMALL_DECAY = 1e-6f;

template <typename T> __device__ __forceinline__ float rec_f(T v);
template <> __device__ __forceinline__ float rec_f<float>(float v) { return v; }
template <> __device__ __forceinline__ float rec_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }

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

// In bf16 mode (FAST) the elementary functions are the special-function unit's, accurate to a few fp32
// roundings for these arguments; the fp32 mode uses the accurate library functions.
__device__ __forceinline__ float ex2f(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float rcpf(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
constexpr float REC_LOG2E = 1.4426950408889634f;
template <bool FAST> __device__ __forceinline__ float rec_sigmoid(float x) {
  return FAST ? rcpf(1.0f + ex2f(-REC_LOG2E * x)) : 1.0f / (1.0f + expf(-x));
}

// Four consecutive channels of a row as they lie in memory.
template <typename T> struct Raw4;
template <> struct Raw4<__nv_bfloat16> {
  uint2 u;
  __device__ __forceinline__ void load(const __nv_bfloat16* p) { u = *reinterpret_cast<const uint2*>(p); }
  __device__ __forceinline__ void get(float (&v)[4]) const {
    v[0] = __uint_as_float(u.x << 16); v[1] = __uint_as_float(u.x & 0xffff0000u);
    v[2] = __uint_as_float(u.y << 16); v[3] = __uint_as_float(u.y & 0xffff0000u);
  }
  __device__ __forceinline__ void set(const float (&v)[4]) {      // of values that bf16 holds exactly
    u.x = (__float_as_uint(v[0]) >> 16) | (__float_as_uint(v[1]) & 0xffff0000u);
    u.y = (__float_as_uint(v[2]) >> 16) | (__float_as_uint(v[3]) & 0xffff0000u);
  }
};
template <> struct Raw4<float> {
  float4 f;
  __device__ __forceinline__ void load(const float* p) { f = *reinterpret_cast<const float4*>(p); }
  __device__ __forceinline__ void get(float (&v)[4]) const { v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w; }
  __device__ __forceinline__ void set(const float (&v)[4]) { f = make_float4(v[0], v[1], v[2], v[3]); }
};

// Rows of this lane's 8 columns; src points at (row 4 j, first column), null: zeros.
template <int LPC>
__device__ __forceinline__ void state_load(float2 (&s)[8][8], const float* src, int ld) {
#pragma unroll
  for (int c = 0; c < 8; ++c)
#pragma unroll
    for (int r = 0; r < 8; ++r) s[c][r] = make_float2(0.f, 0.f);
  if (!src) return;
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e)
#pragma unroll
      for (int w = 0; w < 2; ++w) {
        const float4 v = *reinterpret_cast<const float4*>(src + (int64_t)(i * LPC * 4 + e) * ld + w * 4);
        const float vv[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          if (e & 1) s[w * 4 + c][i * 2 + (e >> 1)].y = vv[c];
          else s[w * 4 + c][i * 2 + (e >> 1)].x = vv[c];
        }
      }
}

template <int LPC>
__device__ __forceinline__ void state_store(const float2 (&s)[8][8], float* dst, int ld) {
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e)
#pragma unroll
      for (int w = 0; w < 2; ++w) {
        const int r = i * 2 + (e >> 1);
        const float4 v = (e & 1) ? make_float4(s[w * 4][r].y, s[w * 4 + 1][r].y, s[w * 4 + 2][r].y, s[w * 4 + 3][r].y)
                                 : make_float4(s[w * 4][r].x, s[w * 4 + 1][r].x, s[w * 4 + 2][r].x, s[w * 4 + 3][r].x);
        *reinterpret_cast<float4*>(dst + (int64_t)(i * LPC * 4 + e) * ld + w * 4) = v;
      }
}

// Rows times d (quads of the row vector, starting at this lane's).
template <int LPC>
__device__ __forceinline__ void state_scale(float2 (&s)[8][8], const float4* d4) {
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float4 d = d4[i * LPC];
#pragma unroll
    for (int c = 0; c < 8; ++c) {
      s[c][2 * i] = mul2(s[c][2 * i], make_float2(d.x, d.y));
      s[c][2 * i + 1] = mul2(s[c][2 * i + 1], make_float2(d.z, d.w));
    }
  }
}

// Sums x and y over the group's lanes; lane j ends with columns j 8 / LPC .. (8 / LPC of them, at least one) in front.
template <int LPC>
__device__ __forceinline__ void group_sums(int j, float (&x)[8], float (&y)[8]) {
  int n = 8;
#pragma unroll
  for (int m = LPC / 2; m > 0; m >>= 1) {
    if (n > 1) {
      n >>= 1;
      const bool up = j & m;
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (i < n) {
          const float sx = up ? x[i] : x[i + n], kx = up ? x[i + n] : x[i];
          const float sy = up ? y[i] : y[i + n], ky = up ? y[i + n] : y[i];
          x[i] = kx + __shfl_xor_sync(0xffffffffu, sx, m);
          y[i] = ky + __shfl_xor_sync(0xffffffffu, sy, m);
        }
    } else {
      x[0] += __shfl_xor_sync(0xffffffffu, x[0], m);
      y[0] += __shfl_xor_sync(0xffffffffu, y[0], m);
    }
  }
}

}  // namespace kd
