// The hyperbolic tangent of capped scores, for scores that live in registers of the tensor-core kernels.
#pragma once

// tanh(y) = 1 - 2 / (1 + e^2y), with the exponential and the division of the special-function unit.  Its error is a few
// 1e-7 absolute, so a score capped at c is off by a few 1e-7 * c, far below what 16-bit queries and keys leave.
__device__ __forceinline__ float tanh_fast(float y) { return 1.f - __fdividef(2.f, 1.f + __expf(2.f * y)); }

// out * tanh(in * x) for small arguments as a polynomial in x, x * (c0 + c1 x^2 + .. + c5 x^10): the Taylor series of
// the hyperbolic tangent with both factors folded into its coefficients.  Up to |in * x| = 1/2 the terms left out are
// below 5e-7 of `out`.
__device__ __forceinline__ void cap_series(float in, float out, float* c) {
  const float z = in * in;
  float f = in * out;
  c[0] = f;
  c[1] = (f *= z) * (-1.f / 3.f);
  c[2] = (f *= z) * (2.f / 15.f);
  c[3] = (f *= z) * (-17.f / 315.f);
  c[4] = (f *= z) * (62.f / 2835.f);
  c[5] = (f *= z) * (-1382.f / 155925.f);
}

// d = a * b + c and d = a * b on two floats at once (packed f32x2: half the issue slots).
__device__ __forceinline__ float2 cap_fma2(float2 a, float2 b, float c) {
  float2 d;
  asm("{\n\t.reg .b64 ra, rb, rc, rd;\n\t"
      "mov.b64 ra, {%2, %3};\n\tmov.b64 rb, {%4, %5};\n\tmov.b64 rc, {%6, %6};\n\t"
      "fma.rn.f32x2 rd, ra, rb, rc;\n\tmov.b64 {%0, %1}, rd;\n\t}"
      : "=f"(d.x), "=f"(d.y) : "f"(a.x), "f"(a.y), "f"(b.x), "f"(b.y), "f"(c));
  return d;
}
__device__ __forceinline__ float2 cap_mul2(float2 a, float2 b) {
  float2 d;
  asm("{\n\t.reg .b64 ra, rb, rd;\n\t"
      "mov.b64 ra, {%2, %3};\n\tmov.b64 rb, {%4, %5};\n\t"
      "mul.rn.f32x2 rd, ra, rb;\n\tmov.b64 {%0, %1}, rd;\n\t}"
      : "=f"(d.x), "=f"(d.y) : "f"(a.x), "f"(a.y), "f"(b.x), "f"(b.y));
  return d;
}

// 64 scores of every lane of a (converged) warp capped in place: by the series when all of the warp's arguments are
// within its range, else by tanh_fast.
__device__ __forceinline__ void cap64(float* v, float in, float out, const float* c) {
  float far = 0.f;
#pragma unroll
  for (int e = 0; e < 64; ++e) far = fmaxf(far, fabsf(v[e]));
  if (__any_sync(0xffffffffu, !(far * in <= 0.5f))) {
#pragma unroll
    for (int e = 0; e < 64; ++e) v[e] = out * tanh_fast(v[e] * in);
    return;
  }
#pragma unroll
  for (int e = 0; e < 64; e += 2) {
    const float2 x = make_float2(v[e], v[e + 1]), z = cap_mul2(x, x);
    float2 p = cap_fma2(make_float2(c[5], c[5]), z, c[4]);
    p = cap_fma2(p, z, c[3]);
    p = cap_fma2(p, z, c[2]);
    p = cap_fma2(p, z, c[1]);
    p = cap_fma2(p, z, c[0]);
    p = cap_mul2(p, x);
    v[e] = p.x;
    v[e + 1] = p.y;
  }
}
