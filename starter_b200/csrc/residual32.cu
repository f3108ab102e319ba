// A residual stream kept in 32-bit floats whatever the working type, for layers with a norm on both
// sides of each sublayer:
//
//     x <- x + post(sublayer(pre(x)))          pre, post: RMS norms with gains of their own
//
// The sum that closes one sublayer and the norm that opens the next touch the same row, so they are
// ONE kernel (as the residual sum and the norm after it are one kernel in the models whose residual
// has the working type): residual_norm takes the sublayer's output y (working type, with an optional
// float bias that was left for it to add), norms it with the post gain, adds it onto the float row
// in place, and norms the new row with the next sublayer's gain into the working type.  With `rows`
// it does the same for selected rows without writing back: that closes the model.
//
// Norm: y / sqrt(mean(y^2) + eps) * gain, everything in float; the gain arrives as a float vector
// (a gain stored around zero has had its one added when the weights were loaded).
//
// Also here: the embedding gather into such a stream (times a constant), the row [stream | embedding] of a product that
// brings the embedding back into the stream (residual_join), and the bias + activation of a dense feed-forward whose
// projections have biases.
#include "common.cuh"

template <typename T>
__global__ void embed32_kernel(const int* __restrict__ tokens, const T* __restrict__ table,
                               float* __restrict__ out, int hidden, int vocab, float scale, int* status) {
  pdl_wait();      // no early launch_dependents: the successor starts when this kernel's blocks have exited
  SB_BEHIND_WAIT(tokens);
  const int row = blockIdx.x;
  int tok = tokens[row];
  const bool bad = tok < 0 || tok >= vocab;
  if (bad) {
    if (threadIdx.x == 0 && status) atomicOr(status, 1);
    tok = 0;
  }
  const T* src = table + (size_t)tok * hidden;
  float* dst = out + (size_t)row * hidden;
  for (int c = threadIdx.x; c < hidden; c += blockDim.x) dst[c] = bad ? 0.f : to_f<T>(src[c]) * scale;
}

// V neighbouring entries as floats and back (V = 4: one access of 16 bytes for float, 8 for bfloat16; V = 1: any address).
template <int V> __device__ __forceinline__ void row_load(const float* p, float* f) {
  if (V == 1) {
    f[0] = p[0];
  } else {
    const float4 raw = *reinterpret_cast<const float4*>(p);
    f[0] = raw.x; f[1] = raw.y; f[2] = raw.z; f[3] = raw.w;
  }
}
template <int V> __device__ __forceinline__ void row_load(const bf16* p, float* f) {
  if (V == 1) {
    f[0] = to_f<bf16>(p[0]);
  } else {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    f[0] = __uint_as_float(raw.x << 16); f[1] = __uint_as_float(raw.x & 0xffff0000u);
    f[2] = __uint_as_float(raw.y << 16); f[3] = __uint_as_float(raw.y & 0xffff0000u);
  }
}
template <int V> __device__ __forceinline__ void row_store(float* p, const float* f) {
  if (V == 1) p[0] = f[0];
  else *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
}
template <int V> __device__ __forceinline__ void row_store(bf16* p, const float* f) {
  if (V == 1) {
    p[0] = from_f<bf16>(f[0]);
  } else {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(f[0], f[1]), hi = __floats2bfloat162_rn(f[2], f[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
  }
}

// One block per row; the row lives in shared memory (hidden floats) between the passes, each thread on entries of its
// own.  y2 (null: none): a second output that is added as it is (two sublayers side by side).
template <typename T, int V>
__global__ void residual_norm_kernel(float* __restrict__ x, const T* __restrict__ y, const T* __restrict__ y2,
                                     const float* __restrict__ y_bias, const float* __restrict__ post_gain,
                                     const float* __restrict__ next_gain, T* __restrict__ out,
                                     const int* __restrict__ rows, int hidden, float eps_post, float eps) {
  extern __shared__ __align__(16) float row[];
  __shared__ float scratch[33];
  pdl_wait();      // no early launch_dependents: the successor starts when this kernel's blocks have exited
  SB_BEHIND_WAIT(y);
  SB_BEHIND_WAIT(y2);
  SB_BEHIND_WAIT(rows);
  SB_BEHIND_WAIT(x);
  const int out_row = blockIdx.x;
  const int in_row = rows ? rows[out_row] : out_row;
  float* xr = x + (size_t)in_row * hidden;
  const T* yr2 = y2 ? y2 + (size_t)in_row * hidden : nullptr;
  float sq = 0.f, inv_y = 1.f, v[V], d[V], e[V];
  if (y && post_gain) {
    const T* yr = y + (size_t)in_row * hidden;
    float ysq = 0.f;
    for (int c = threadIdx.x * V; c < hidden; c += blockDim.x * V) {
      row_load<V>(yr + c, d);
#pragma unroll
      for (int i = 0; i < V; ++i) {
        if (y_bias) d[i] += y_bias[c + i];
        ysq += d[i] * d[i];
      }
      row_store<V>(row + c, d);
    }
    ysq = block_sum(ysq, scratch);
    inv_y = 1.f / sqrtf(ysq / (float)hidden + eps_post);
  }
  for (int c = threadIdx.x * V; c < hidden; c += blockDim.x * V) {
    row_load<V>(xr + c, v);
    if (y) {
      if (post_gain) {
        row_load<V>(row + c, d);
#pragma unroll
        for (int i = 0; i < V; ++i) d[i] = d[i] * inv_y * post_gain[c + i];
      } else {
        row_load<V>(y + (size_t)in_row * hidden + c, d);
        if (y_bias) {
#pragma unroll
          for (int i = 0; i < V; ++i) d[i] += y_bias[c + i];
        }
      }
      if (yr2) {
        row_load<V>(yr2 + c, e);
#pragma unroll
        for (int i = 0; i < V; ++i) d[i] += e[i];
      }
#pragma unroll
      for (int i = 0; i < V; ++i) v[i] += d[i];
      if (!rows) row_store<V>(xr + c, v);
    }
#pragma unroll
    for (int i = 0; i < V; ++i) sq += v[i] * v[i];
    row_store<V>(row + c, v);
  }
  if (!out) return;
  sq = block_sum(sq, scratch);
  const float inv = 1.f / sqrtf(sq / (float)hidden + eps);
  T* o = out + (size_t)out_row * hidden;
  for (int c = threadIdx.x * V; c < hidden; c += blockDim.x * V) {
    row_load<V>(row + c, v);
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] *= inv * next_gain[c + i];
    row_store<V>(o + c, v);
  }
}

// out[t] = [x[t] + y[t] + y2[t] | table[tokens[t]] * scale] in the working type (y, y2 null: not there): the row a product
// reads that brings the embedding output back into the stream.  The stream itself is left as it was.
template <typename T, int V>
__global__ void residual_join_kernel(const float* __restrict__ x, const T* __restrict__ y, const T* __restrict__ y2,
                                     const int* __restrict__ tokens, const T* __restrict__ table, T* __restrict__ out,
                                     int hidden, int vocab, float scale) {
  pdl_wait();      // no early launch_dependents: the successor starts when this kernel's blocks have exited
  SB_BEHIND_WAIT(x);
  SB_BEHIND_WAIT(y);
  SB_BEHIND_WAIT(y2);
  SB_BEHIND_WAIT(tokens);
  const size_t at = (size_t)blockIdx.x * hidden;
  const int tok = tokens[blockIdx.x];
  const bool bad = tok < 0 || tok >= vocab;      // (reported by the step's embedding, which gave the row zeros)
  const T* embedded = table + (size_t)(bad ? 0 : tok) * hidden;
  T* o = out + 2 * at;
  float v[V], d[V];
  for (int c = threadIdx.x * V; c < hidden; c += blockDim.x * V) {
    row_load<V>(x + at + c, v);
    if (y) {
      row_load<V>(y + at + c, d);
      if (y2) {
        float e[V];
        row_load<V>(y2 + at + c, e);
#pragma unroll
        for (int i = 0; i < V; ++i) d[i] += e[i];
      }
#pragma unroll
      for (int i = 0; i < V; ++i) v[i] += d[i];
    }
    row_store<V>(o + c, v);
    row_load<V>(embedded + c, d);
#pragma unroll
    for (int i = 0; i < V; ++i) d[i] = bad ? 0.f : d[i] * scale;
    row_store<V>(o + hidden + c, d);
  }
}

// y[r, c] = act(x[r, c] + bias[c]); act 0: none, 1: relu, squared; 2: tanh; 3: exp(-exp(.)), the decay
// of a recurrence from its logarithm's logarithm.
template <typename T>
__global__ void bias_act_kernel(const T* __restrict__ x, const float* __restrict__ bias, T* __restrict__ y,
                                int width, size_t total, int act) {
  pdl_wait();      // no early launch_dependents: the successor starts when this kernel's blocks have exited
  SB_BEHIND_WAIT(x);
  size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  const size_t stride = (size_t)gridDim.x * blockDim.x;
  for (; i < total; i += stride) {
    float v = to_f<T>(x[i]);
    if (bias) v += bias[i % width];
    if (act == 1) {
      v = fmaxf(v, 0.f);
      v = v * v;
    } else if (act == 2) {
      v = tanhf(v);
    } else if (act == 3) {
      v = expf(-expf(v));
    }
    y[i] = from_f<T>(v);
  }
}

extern "C" {

// out: float [n_tokens, hidden] = table[token] * scale.  serial != 0: an ordinary launch (the step's
// fence: everything earlier steps wrote is complete before any kernel of this step starts).
int sb_embed32(int dtype, const int* tokens, const void* table, float* out, int n_tokens, int hidden,
               int vocab, float scale, int* status, int serial, cudaStream_t s) {
  if (n_tokens == 0) return 0;
  const int threads = hidden >= 1024 ? 256 : 128;
  if (serial) {
    if (dtype == 0)
      embed32_kernel<float><<<n_tokens, threads, 0, s>>>(tokens, (const float*)table, out, hidden, vocab, scale, status);
    else
      embed32_kernel<bf16><<<n_tokens, threads, 0, s>>>(tokens, (const bf16*)table, out, hidden, vocab, scale, status);
    return SB_LAUNCH_RESULT();
  }
  if (dtype == 0)
    return launch_dependent(embed32_kernel<float>, dim3(n_tokens), dim3(threads), 0, s, tokens, (const float*)table, out, hidden, vocab, scale, status);
  return launch_dependent(embed32_kernel<bf16>, dim3(n_tokens), dim3(threads), 0, s, tokens, (const bf16*)table, out, hidden, vocab, scale, status);
}

// x: float [*, hidden].  y (null: nothing to add) [*, hidden] of the working type; y_bias null or float
// [hidden]; post_gain float [hidden] or null (y is added as it is); y2 null or a second output, added as it is.
// next_gain / out: the norm of the new row into the working type (out null: only the sum).  rows null: every row, x
// updated in place.  eps_post belongs to the norm of y, eps to the norm of the new row.
int sb_residual_norm(int dtype, float* x, const void* y, const void* y2, const float* y_bias, const float* post_gain,
                     const float* next_gain, void* out, const int* rows, int n_rows, int hidden, float eps_post,
                     float eps, cudaStream_t s) {
  if (n_rows == 0) return 0;
  if ((out && !next_gain) || (y2 && !y)) return -2;
  const size_t smem = (size_t)hidden * sizeof(float);
  if (smem > 200 * 1024) return -2;
  const bool wide = hidden % 4 == 0 && (((uintptr_t)x | (uintptr_t)y | (uintptr_t)y2 | (uintptr_t)out) & 15) == 0;
  const int items = wide ? hidden / 4 : hidden;
  const int threads = items >= 1024 ? 512 : items >= 256 ? 256 : 128;
#define NORM_GO(T, V)                                                                                                  \
  {                                                                                                                    \
    if (smem > 48 * 1024)                                                                                              \
      cudaFuncSetAttribute(residual_norm_kernel<T, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);        \
    return launch_dependent(residual_norm_kernel<T, V>, dim3(n_rows), dim3(threads), smem, s, x, (const T*)y,           \
                            (const T*)y2, y_bias, post_gain, next_gain, (T*)out, rows, hidden, eps_post, eps);          \
  }
  if (dtype == 0) {
    if (wide) NORM_GO(float, 4)
    NORM_GO(float, 1)
  }
  if (wide) NORM_GO(bf16, 4)
  NORM_GO(bf16, 1)
#undef NORM_GO
}

// x: float [n_tokens, hidden]; y, y2: null or [n_tokens, hidden]; table: [vocab, hidden]; out: [n_tokens, 2 * hidden].
int sb_residual_join(int dtype, const float* x, const void* y, const void* y2, const int* tokens, const void* table,
                     void* out, int n_tokens, int hidden, int vocab, float scale, cudaStream_t s) {
  if (n_tokens == 0) return 0;
  if (y2 && !y) return -2;
  const bool wide = hidden % 4 == 0 &&
                    (((uintptr_t)x | (uintptr_t)y | (uintptr_t)y2 | (uintptr_t)table | (uintptr_t)out) & 15) == 0;
  const int items = wide ? hidden / 4 : hidden;
  const int threads = items >= 512 ? 256 : 128;
#define JOIN_GO(T, V)                                                                                                  \
  return launch_dependent(residual_join_kernel<T, V>, dim3(n_tokens), dim3(threads), 0, s, x, (const T*)y, (const T*)y2, \
                          tokens, (const T*)table, (T*)out, hidden, vocab, scale)
  if (dtype == 0) {
    if (wide) JOIN_GO(float, 4);
    JOIN_GO(float, 1);
  }
  if (wide) JOIN_GO(bf16, 4);
  JOIN_GO(bf16, 1);
#undef JOIN_GO
}

int sb_bias_act(int dtype, const void* x, const float* bias, void* y, int n_rows, int width, int act,
                cudaStream_t s) {
  const size_t total = (size_t)n_rows * width;
  if (total == 0) return 0;
  size_t blocks = (total + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  if (dtype == 0)
    return launch_dependent(bias_act_kernel<float>, dim3((int)blocks), dim3(256), 0, s, (const float*)x, bias, (float*)y, width, total, act);
  return launch_dependent(bias_act_kernel<bf16>, dim3((int)blocks), dim3(256), 0, s, (const bf16*)x, bias, (bf16*)y, width, total, act);
}

}  // extern "C"
