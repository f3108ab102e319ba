// Grouped-query attention over the paged cache without rotation, whose positions enter through the
// scores and the mask instead:
//
//   score(i, j) = q_i . k_j * scale - r1_h * ln(1 + r2_h * (i - j))        a distance penalty per head
//   visible:      j <= i, and (chunk > 0) floor(i / chunk) == floor(j / chunk), and (window > 0) j > i - window;
//                 chunks are counted from position 0 of the sequence
//   softmax:      the denominator holds one more term exp(sink_h): a key that has no value
//   head output:  times gate[i, h], a number per token and head that arrives as sigmoid(g_h . x_i)
//
//   kept keys:    with a window, the keys j < keep stay visible however far behind they are
//   capped:       a scaled score s becomes cap * tanh(s / cap)
//
// Each of these (penalty, chunk, sink, gate, kept keys, cap) is switched by its pointer or size, so a design may use
// any of them alone.  Keys have `dim` entries, values `vdim`.  Scores, the penalty with its logarithm,
// the running maximum and sum, the accumulator and the gate are float.
//
// The sink is the state the running softmax starts from: maximum = sink, sum = 1, accumulator = 0.
//
// Here: the kernel that files a step's keys and values and forms the gates (sink_prepare), and the plain
// attention kernel, one warp per (token, head), for the 32-bit path and for sizes the tensor-core kernel
// (attention_sink_tc.cu) does not take.
#include "common.cuh"

#define SINK_MAX_D 8  // dim, vdim <= 256

// proj: a row = [q (heads * dim) | k (kv_heads * dim) | v (kv_heads * vdim) | g (heads)]; without `write`
// the row has no k and v.  gate: float [tokens, heads] = sigmoid(g), or null when the row has no g.
template <typename T>
__global__ void sink_prepare_kernel(const T* __restrict__ proj, int proj_width, const int* __restrict__ tok_pos,
                                    const int* __restrict__ tok_slot, const int* __restrict__ block_table,
                                    int table_stride, T* __restrict__ k_store, T* __restrict__ v_store,
                                    float* __restrict__ gate, int heads, int kv_heads, int dim, int vdim, int write,
                                    int vec) {
  pdl_wait();      // no early launch_dependents: the successor starts when this kernel's blocks have exited
  SB_BEHIND_WAIT(proj);
  SB_BEHIND_WAIT(tok_pos);
  SB_BEHIND_WAIT(tok_slot);
  SB_BEHIND_WAIT(block_table);
  const int row = blockIdx.x;
  const T* pr = proj + (size_t)row * proj_width;
  const int q_width = heads * dim;
  int g_at = q_width;
  if (write) {
    const int pos = tok_pos[row];
    const int page = block_table[(size_t)tok_slot[row] * table_stride + pos / SB_PAGE_TOKENS];
    const int off = pos % SB_PAGE_TOKENS;
    const T* k = pr + q_width;
    const T* v = k + kv_heads * dim;
    constexpr int N = 16 / sizeof(T);       // entries of a 16-byte piece
    if (vec) {
      // rows, head sizes and bases in whole 16-byte pieces: a piece a thread
      for (int e = threadIdx.x; e < kv_heads * dim / N; e += blockDim.x) {
        const int h = e / (dim / N), d = (e - h * (dim / N)) * N;
        *reinterpret_cast<uint4*>(k_store + page_row(page, h, off, kv_heads, dim) + d) =
            *reinterpret_cast<const uint4*>(k + h * dim + d);
      }
      for (int e = threadIdx.x; e < kv_heads * vdim / N; e += blockDim.x) {
        const int h = e / (vdim / N), d = (e - h * (vdim / N)) * N;
        *reinterpret_cast<uint4*>(v_store + page_row(page, h, off, kv_heads, vdim) + d) =
            *reinterpret_cast<const uint4*>(v + h * vdim + d);
      }
    } else {
      for (int e = threadIdx.x; e < kv_heads * dim; e += blockDim.x) {
        const int h = e / dim, d = e - h * dim;
        k_store[page_row(page, h, off, kv_heads, dim) + d] = k[e];
      }
      for (int e = threadIdx.x; e < kv_heads * vdim; e += blockDim.x) {
        const int h = e / vdim, d = e - h * vdim;
        v_store[page_row(page, h, off, kv_heads, vdim) + d] = v[e];
      }
    }
    g_at += kv_heads * (dim + vdim);
  }
  if (gate)
    for (int h = threadIdx.x; h < heads; h += blockDim.x)
      gate[(size_t)row * heads + h] = 1.f / (1.f + expf(-to_f<T>(pr[g_at + h])));
}

// The same for a layer whose queries and keys are turned by their positions and whose values may be its keys:
// proj: a row = [q (heads * dim) | k (kv_heads * dim) | v (kv_heads * vdim), absent with v_from_k].  The first
// `rot` entries of every query and key head turn, entry 2i with entry 2i + 1, by the angle whose cos and sin
// stand at [position][i] of the float tables (rot / 2 columns; rot 0: nothing turns).  Queries are turned in
// place; keys go to the cache turned, values as they are; with v_from_k a key/value head's value is its key
// as projected, before the turn (vdim == dim).  A thread a pair of entries; the products are float.
template <typename T>
__global__ void sink_prepare_rot_kernel(T* __restrict__ proj, int proj_width, const int* __restrict__ tok_pos,
                                        const int* __restrict__ tok_slot, const int* __restrict__ block_table,
                                        int table_stride, T* __restrict__ k_store, T* __restrict__ v_store,
                                        const float* __restrict__ cos_t, const float* __restrict__ sin_t, int rot,
                                        int heads, int kv_heads, int dim, int vdim, int v_from_k, int write) {
  pdl_wait();      // no early launch_dependents: the successor starts when this kernel's blocks have exited
  SB_BEHIND_WAIT(proj);
  SB_BEHIND_WAIT(tok_pos);
  SB_BEHIND_WAIT(tok_slot);
  SB_BEHIND_WAIT(block_table);
  const int row = blockIdx.x;
  T* pr = proj + (size_t)row * proj_width;
  const int pos = tok_pos[row];
  const float* cr = cos_t + (size_t)pos * (rot / 2);
  const float* sr = sin_t + (size_t)pos * (rot / 2);
  const int half = (dim + 1) / 2;           // pairs a head (the last may be a single entry)
  for (int e = threadIdx.x; e < heads * half; e += blockDim.x) {
    const int h = e / half, i = e - h * half;
    if (2 * i + 1 >= dim || 2 * i >= rot) continue;
    T* at = pr + (size_t)h * dim + 2 * i;
    const float a = to_f<T>(at[0]), b = to_f<T>(at[1]), c = cr[i], s = sr[i];
    at[0] = from_f<T>(a * c - b * s);
    at[1] = from_f<T>(b * c + a * s);
  }
  if (!write) return;
  const int page = block_table[(size_t)tok_slot[row] * table_stride + pos / SB_PAGE_TOKENS];
  const int off = pos % SB_PAGE_TOKENS;
  const T* k = pr + (size_t)heads * dim;
  const T* v = k + (size_t)kv_heads * dim;
  for (int e = threadIdx.x; e < kv_heads * half; e += blockDim.x) {
    const int h = e / half, i = e - h * half;
    const bool two = 2 * i + 1 < dim;
    const float a = to_f<T>(k[(size_t)h * dim + 2 * i]), b = two ? to_f<T>(k[(size_t)h * dim + 2 * i + 1]) : 0.f;
    T* kd = k_store + page_row(page, h, off, kv_heads, dim) + 2 * i;
    if (two && 2 * i < rot) {
      const float c = cr[i], s = sr[i];
      kd[0] = from_f<T>(a * c - b * s);
      kd[1] = from_f<T>(b * c + a * s);
    } else {
      kd[0] = from_f<T>(a);
      if (two) kd[1] = from_f<T>(b);
    }
    if (v_from_k) {
      T* vd = v_store + page_row(page, h, off, kv_heads, vdim) + 2 * i;
      vd[0] = from_f<T>(a);
      if (two) vd[1] = from_f<T>(b);
    }
  }
  if (!v_from_k)
    for (int e = threadIdx.x; e < kv_heads * vdim; e += blockDim.x) {
      const int h = e / vdim, d = e - h * vdim;
      v_store[page_row(page, h, off, kv_heads, vdim) + d] = v[e];
    }
}

// V consecutive entries as floats and back (V * sizeof(T) == 16: one access; V == 1: any address).
template <typename T, int V> __device__ __forceinline__ void sink_load(const T* p, float* f) {
  if (V == 1) {
    f[0] = to_f<T>(p[0]);
  } else {
    const uint4 raw = *reinterpret_cast<const uint4*>(p);
    const T* e = reinterpret_cast<const T*>(&raw);
#pragma unroll
    for (int i = 0; i < V; ++i) f[i] = to_f<T>(e[i]);
  }
}
template <typename T, int V> __device__ __forceinline__ void sink_store(T* p, const float* f) {
  if (V == 1) {
    p[0] = from_f<T>(f[0]);
  } else {
    uint4 raw;
    T* e = reinterpret_cast<T*>(&raw);
#pragma unroll
    for (int i = 0; i < V; ++i) e[i] = from_f<T>(f[i]);
    *reinterpret_cast<uint4*>(p) = raw;
  }
}

// The same for a layer whose queries and keys may be RMS-normed over their whole projections (q_gain, k_gain: float
// [heads * dim] and [kv_heads * dim], or both null), whose first `rot` entries of a head turn (float tables of rot / 2
// columns; PAIRS false: entry i with entry i + rot / 2; true: entry 2i with entry 2i + 1), and whose values may be
// divided by their root mean square per head (unit_v).  A block a token: the rows' sums of squares, then a piece of V
// entries a thread (with its partner where it turns), queries in place, keys into the cache; a warp a value head.
template <typename T, int V, bool PAIRS>
__global__ void sink_prepare_norm_kernel(T* __restrict__ proj, int proj_width, const int* __restrict__ tok_pos,
                                         const int* __restrict__ tok_slot, const int* __restrict__ block_table,
                                         int table_stride, T* __restrict__ k_store, T* __restrict__ v_store,
                                         const float* __restrict__ cos_t, const float* __restrict__ sin_t, int rot,
                                         const float* __restrict__ q_gain, const float* __restrict__ k_gain, float eps,
                                         int unit_v, int heads, int kv_heads, int dim, int vdim, int write) {
  __shared__ float2 shares[32];
  pdl_wait();      // no early launch_dependents: the successor starts when this kernel's blocks have exited
  SB_BEHIND_WAIT(proj);
  SB_BEHIND_WAIT(tok_pos);
  SB_BEHIND_WAIT(tok_slot);
  SB_BEHIND_WAIT(block_table);
  const int row = blockIdx.x, tid = threadIdx.x;
  T* q = proj + (size_t)row * proj_width;
  T* k = q + (size_t)heads * dim;
  const T* v = k + (size_t)kv_heads * dim;
  const int pos = tok_pos[row], half = rot / 2, pieces = dim / V;
  const float* cr = cos_t + (size_t)pos * half;
  const float* sr = sin_t + (size_t)pos * half;
  const int lane = tid & 31, warp = tid >> 5, warps = blockDim.x >> 5;
  auto squares = [&](const T* x, int n) {                // this thread's share of a row's sum of squares
    float sq = 0.f, f[V];
    for (int c = tid * V; c < n; c += blockDim.x * V) {
      sink_load<T, V>(x + c, f);
#pragma unroll
      for (int i = 0; i < V; ++i) sq += f[i] * f[i];
    }
    return sq;
  };
  // piece c of a head: normed, turned with its partner (which this thread handles too) and stored
  auto turn = [&](const T* from, T* to, const float* gain, float inv, int c) {
    float x[V], y[V], g[V];
    const int at = c * V;
    if (PAIRS && V == 1) {
      if (at < rot && (at & 1)) return;                 // a partner
      x[0] = to_f<T>(from[at]) * (gain ? inv * gain[at] : 1.f);
      if (at >= rot) {
        to[at] = from_f<T>(x[0]);
        return;
      }
      y[0] = to_f<T>(from[at + 1]) * (gain ? inv * gain[at + 1] : 1.f);
      const float co = cr[at / 2], si = sr[at / 2];
      to[at] = from_f<T>(x[0] * co - y[0] * si);
      to[at + 1] = from_f<T>(y[0] * co + x[0] * si);
      return;
    }
    if (PAIRS) {
      sink_load<T, V>(from + at, x);
      if (gain) {
#pragma unroll
        for (int i = 0; i < V; ++i) x[i] *= inv * gain[at + i];
      }
#pragma unroll
      for (int i = 0; i + 1 < V; i += 2) {
        g[i] = x[i];
        g[i + 1] = x[i + 1];
        if (at + i < rot) {
          const float co = cr[(at + i) / 2], si = sr[(at + i) / 2];
          g[i] = x[i] * co - x[i + 1] * si;
          g[i + 1] = x[i + 1] * co + x[i] * si;
        }
      }
      sink_store<T, V>(to + at, g);
      return;
    }
    if (at >= half && at < rot) return;                 // a partner
    sink_load<T, V>(from + at, x);
    if (gain) {
#pragma unroll
      for (int i = 0; i < V; ++i) x[i] *= inv * gain[at + i];
    }
    if (at >= rot) {
      sink_store<T, V>(to + at, x);
      return;
    }
    sink_load<T, V>(from + half + at, y);
    if (gain) {
#pragma unroll
      for (int i = 0; i < V; ++i) y[i] *= inv * gain[half + at + i];
    }
#pragma unroll
    for (int i = 0; i < V; ++i) {
      const float co = cr[at + i], si = sr[at + i];
      g[i] = x[i] * co - y[i] * si;
      y[i] = y[i] * co + x[i] * si;
    }
    sink_store<T, V>(to + at, g);
    sink_store<T, V>(to + half + at, y);
  };
  float q_inv = 1.f, k_inv = 1.f;
  if (q_gain) {
    const float mine_q = warp_sum(squares(q, heads * dim)), mine_k = write ? warp_sum(squares(k, kv_heads * dim)) : 0.f;
    if (lane == 0) shares[warp] = make_float2(mine_q, mine_k);
    __syncthreads();
    float sq = 0.f, sk = 0.f;
    for (int i = 0; i < warps; ++i) {
      sq += shares[i].x;
      sk += shares[i].y;
    }
    q_inv = 1.f / sqrtf(sq / (float)(heads * dim) + eps);
    k_inv = 1.f / sqrtf(sk / (float)(kv_heads * dim) + eps);
  }
  for (int e = tid; e < heads * pieces; e += blockDim.x) {
    const int h = e / pieces, c = e - h * pieces;
    if (!q_gain && c * V >= (PAIRS ? rot : half)) continue;      // queries in place: nothing to do for entries that stay
    turn(q + (size_t)h * dim, q + (size_t)h * dim, q_gain ? q_gain + (size_t)h * dim : nullptr, q_inv, c);
  }
  if (!write) return;
  const int page = block_table[(size_t)tok_slot[row] * table_stride + pos / SB_PAGE_TOKENS];
  const int off = pos % SB_PAGE_TOKENS;
  for (int e = tid; e < kv_heads * pieces; e += blockDim.x) {
    const int h = e / pieces, c = e - h * pieces;
    turn(k + (size_t)h * dim, k_store + page_row(page, h, off, kv_heads, dim), k_gain ? k_gain + (size_t)h * dim : nullptr,
         k_inv, c);
  }
  for (int h = warp; h < kv_heads; h += warps) {
    const T* from = v + (size_t)h * vdim;
    T* to = v_store + page_row(page, h, off, kv_heads, vdim);
    float f[V], inv = 1.f;
    if (unit_v) {
      float sq = 0.f;
      for (int c = lane * V; c < vdim; c += 32 * V) {
        sink_load<T, V>(from + c, f);
#pragma unroll
        for (int i = 0; i < V; ++i) sq += f[i] * f[i];
      }
      inv = 1.f / sqrtf(warp_sum(sq) / (float)vdim + eps);
    }
    for (int c = lane * V; c < vdim; c += 32 * V) {
      sink_load<T, V>(from + c, f);
#pragma unroll
      for (int i = 0; i < V; ++i) f[i] *= inv;
      sink_store<T, V>(to + c, f);
    }
  }
}

template <typename T>
static int sink_prepare_norm(void* proj, int proj_width, const int* tok_pos, const int* tok_slot, const int* block_table,
                             int table_stride, void* k_store, void* v_store, const float* cos_t, const float* sin_t, int rot,
                             const float* q_gain, const float* k_gain, float eps, int unit_v, int n_tokens, int heads,
                             int kv_heads, int dim, int vdim, int write, int pairs, cudaStream_t s) {
  constexpr int N = 16 / sizeof(T);
  const bool wide = proj_width % N == 0 && dim % N == 0 && (pairs || (rot / 2) % N == 0) && vdim % N == 0 &&
                    (((uintptr_t)proj | (uintptr_t)k_store | (uintptr_t)v_store) & 15) == 0;
  const int items = heads * dim / (wide ? N : 1);
  const int threads = items > 512 ? 512 : items > 128 ? 256 : 128;
#define NORM_GO(V, PAIRS)                                                                                              \
  return launch_dependent(sink_prepare_norm_kernel<T, V, PAIRS>, dim3(n_tokens), dim3(threads), 0, s, (T*)proj, proj_width,     \
                          tok_pos, tok_slot, block_table, table_stride, (T*)k_store, (T*)v_store, cos_t, sin_t, rot,    \
                          q_gain, k_gain, eps, unit_v, heads, kv_heads, dim, vdim, write)
  if (pairs) {
    if (wide) NORM_GO(N, true);
    NORM_GO(1, true);
  }
  if (wide) NORM_GO(N, false);
  NORM_GO(1, false);
#undef NORM_GO
}

template <typename T>
__global__ void sink_attention_kernel(const T* __restrict__ q, int q_stride, T* __restrict__ out,
                                      const T* __restrict__ k_store, const T* __restrict__ v_store,
                                      const int* __restrict__ block_table, int table_stride,
                                      const int* __restrict__ tok_slot, const int* __restrict__ tok_pos,
                                      const float* __restrict__ r1, const float* __restrict__ r2,
                                      const float* __restrict__ sink, const float* __restrict__ gate, int n_tokens,
                                      int heads, int kv_heads, int dim, int vdim, float scale, int chunk, int window,
                                      int keep, float cap) {
  pdl_wait();      // no early launch_dependents: the successor starts when this kernel's blocks have exited
  SB_BEHIND_WAIT(q);
  SB_BEHIND_WAIT(k_store);
  SB_BEHIND_WAIT(v_store);
  SB_BEHIND_WAIT(gate);
  SB_BEHIND_WAIT(tok_pos);
  SB_BEHIND_WAIT(tok_slot);
  SB_BEHIND_WAIT(block_table);
  const long long warp = ((long long)blockIdx.x * blockDim.x + threadIdx.x) >> 5;
  const int lane = threadIdx.x & 31;
  if (warp >= (long long)n_tokens * heads) return;
  const int token = (int)(warp / heads);
  const int h = (int)(warp - (long long)token * heads);
  const int kvh = h / (heads / kv_heads);
  const int pos = tok_pos[token];
  const int* pages = block_table + (size_t)tok_slot[token] * table_stride;
  const T* qr = q + (size_t)token * q_stride + (size_t)h * dim;

  float qv[SINK_MAX_D], acc[SINK_MAX_D];
#pragma unroll
  for (int i = 0; i < SINK_MAX_D; ++i) {
    const int d = lane + 32 * i;
    qv[i] = d < dim ? to_f<T>(qr[d]) : 0.f;
    acc[i] = 0.f;
  }
  const float pen1 = r1 ? r1[h] : 0.f, pen2 = r1 ? r2[h] : 0.f;
  float m = sink ? sink[h] : -INFINITY, l = sink ? 1.f : 0.f;
  int first = 0;
  if (chunk > 0) first = pos / chunk * chunk;
  if (window > 0 && pos - window + 1 > first) first = pos - window + 1;

  // the kept keys in front of the first key of the window (or chunk), then everything from there on
  for (int part = keep > 0 && first > 0 ? 0 : 1; part < 2; ++part) {
  const int from = part == 0 ? 0 : first, last = part == 0 ? min(keep, first) - 1 : pos;
  for (int j0 = from; j0 <= last; j0 += 4) {
    float s[4];
    const T* vrow[4];
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      const int j = j0 + u;
      s[u] = 0.f;
      vrow[u] = nullptr;
      if (j <= last) {
        const int page = pages[j / SB_PAGE_TOKENS];
        const T* kr = k_store + page_row(page, kvh, j % SB_PAGE_TOKENS, kv_heads, dim);
        vrow[u] = v_store + page_row(page, kvh, j % SB_PAGE_TOKENS, kv_heads, vdim);
#pragma unroll
        for (int i = 0; i < SINK_MAX_D; ++i) {
          const int d = lane + 32 * i;
          if (d < dim) s[u] += qv[i] * to_f<T>(kr[d]);
        }
      }
    }
    float m_new = m;
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      s[u] = warp_sum(s[u]) * scale;
      if (cap > 0.f) s[u] = cap * tanhf(s[u] / cap);
      if (r1) s[u] -= pen1 * log1pf(pen2 * (float)(pos - (j0 + u)));
      if (j0 + u <= last) m_new = fmaxf(m_new, s[u]);
    }
    const float alpha = expf(m - m_new);
    l *= alpha;
#pragma unroll
    for (int i = 0; i < SINK_MAX_D; ++i) acc[i] *= alpha;
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      if (j0 + u <= last) {
        const float p = expf(s[u] - m_new);
        l += p;
#pragma unroll
        for (int i = 0; i < SINK_MAX_D; ++i) {
          const int d = lane + 32 * i;
          if (d < vdim) acc[i] += p * to_f<T>(vrow[u][d]);
        }
      }
    }
    m = m_new;
  }
  }
  T* orow = out + ((size_t)token * heads + h) * vdim;
  const float inv = (gate ? gate[(size_t)token * heads + h] : 1.f) / l;
#pragma unroll
  for (int i = 0; i < SINK_MAX_D; ++i) {
    const int d = lane + 32 * i;
    if (d < vdim) orow[d] = from_f<T>(acc[i] * inv);
  }
}

extern "C" {

int sb_sink_max_dim() { return 32 * SINK_MAX_D; }

// proj: [n_tokens, proj_width]; k_store [pages, kv_heads, 64, dim], v_store [pages, kv_heads, 64, vdim]
// (ignored when write == 0); gate: float [n_tokens, heads] or null.
int sb_sink_prepare(int dtype, const void* proj, int proj_width, const int* tok_pos, const int* tok_slot,
                    const int* block_table, int table_stride, void* k_store, void* v_store, float* gate, int n_tokens,
                    int heads, int kv_heads, int dim, int vdim, int write, cudaStream_t s) {
  if (n_tokens == 0) return 0;
  if (proj_width < heads * dim + (write ? kv_heads * (dim + vdim) : 0) + (gate ? heads : 0)) return -2;
  const int n = dtype == 0 ? 4 : 8;
  const int vec = write && proj_width % n == 0 && dim % n == 0 && vdim % n == 0 &&
                  (((uintptr_t)proj | (uintptr_t)k_store | (uintptr_t)v_store) & 15) == 0;
  const int threads = write && vec && kv_heads * (dim + vdim) / n > 128 ? 256 : 128;
  if (dtype == 0)
    return launch_dependent(sink_prepare_kernel<float>, dim3(n_tokens), dim3(threads), 0, s, (const float*)proj, proj_width,
                            tok_pos, tok_slot, block_table, table_stride, (float*)k_store, (float*)v_store, gate, heads,
                            kv_heads, dim, vdim, write, vec);
  return launch_dependent(sink_prepare_kernel<bf16>, dim3(n_tokens), dim3(threads), 0, s, (const bf16*)proj, proj_width,
                          tok_pos, tok_slot, block_table, table_stride, (bf16*)k_store, (bf16*)v_store, gate, heads,
                          kv_heads, dim, vdim, write, vec);
}

// proj: [n_tokens, proj_width], its queries turned in place; cos_t, sin_t: float [positions, rot / 2] (unused with
// rot 0); v_from_k: the row has no values and the keys as projected are filed as values (vdim == dim).
int sb_sink_prepare_rot(int dtype, void* proj, int proj_width, const int* tok_pos, const int* tok_slot,
                        const int* block_table, int table_stride, void* k_store, void* v_store, const float* cos_t,
                        const float* sin_t, int rot, int n_tokens, int heads, int kv_heads, int dim, int vdim,
                        int v_from_k, int write, cudaStream_t s) {
  if (n_tokens == 0) return 0;
  if (rot < 0 || rot % 2 || rot > dim || (v_from_k && vdim != dim)) return -2;
  if (proj_width < heads * dim + (write ? kv_heads * (dim + (v_from_k ? 0 : vdim)) : 0)) return -2;
  const int threads = heads * dim > 1024 ? 256 : 128;
  if (dtype == 0)
    return launch_dependent(sink_prepare_rot_kernel<float>, dim3(n_tokens), dim3(threads), 0, s, (float*)proj, proj_width,
                            tok_pos, tok_slot, block_table, table_stride, (float*)k_store, (float*)v_store, cos_t, sin_t,
                            rot, heads, kv_heads, dim, vdim, v_from_k, write);
  return launch_dependent(sink_prepare_rot_kernel<bf16>, dim3(n_tokens), dim3(threads), 0, s, (bf16*)proj, proj_width,
                          tok_pos, tok_slot, block_table, table_stride, (bf16*)k_store, (bf16*)v_store, cos_t, sin_t, rot,
                          heads, kv_heads, dim, vdim, v_from_k, write);
}

// proj: [n_tokens, proj_width] = [q | k | v] (without `write`: [q]), its queries normed and turned in place; keys and
// values go to the cache.  q_gain, k_gain: float [heads * dim], [kv_heads * dim], or null (no norm); cos_t, sin_t: float
// [positions, rot / 2] (unused with rot 0); pairs: entry 2i turns with entry 2i + 1 (else i with i + rot / 2); unit_v:
// values over their root mean square per head.
int sb_sink_prepare_norm(int dtype, void* proj, int proj_width, const int* tok_pos, const int* tok_slot,
                         const int* block_table, int table_stride, void* k_store, void* v_store, const float* cos_t,
                         const float* sin_t, int rot, const float* q_gain, const float* k_gain, float eps, int unit_v,
                         int n_tokens, int heads, int kv_heads, int dim, int vdim, int write, int pairs, cudaStream_t s) {
  if (n_tokens == 0) return 0;
  if (rot < 0 || rot % 2 || rot > dim || (write && (k_gain != nullptr) != (q_gain != nullptr))) return -2;
  if (proj_width < heads * dim + (write ? kv_heads * (dim + vdim) : 0)) return -2;
#define NORM_ARGS proj, proj_width, tok_pos, tok_slot, block_table, table_stride, k_store, v_store, cos_t, sin_t, rot, q_gain, \
                  k_gain, eps, unit_v, n_tokens, heads, kv_heads, dim, vdim, write, pairs, s
  return dtype == 0 ? sink_prepare_norm<float>(NORM_ARGS) : sink_prepare_norm<bf16>(NORM_ARGS);
#undef NORM_ARGS
}

// q: rows of q_stride entries whose first heads * dim are the queries; out: [n_tokens, heads * vdim].
// r1, r2: float [heads] or both null; sink: float [heads] or null; gate: float [n_tokens, heads] or null.
// chunk, window, keep (the first keys a window keeps), cap <= 0: none.
int sb_sink_attention(int dtype, const void* q, int q_stride, void* out, const void* k_store, const void* v_store,
                      const int* block_table, int table_stride, const int* tok_slot, const int* tok_pos,
                      const float* r1, const float* r2, const float* sink, const float* gate, int n_tokens, int heads,
                      int kv_heads, int dim, int vdim, float scale, int chunk, int window, int keep, float cap,
                      cudaStream_t s) {
  if (dim > 32 * SINK_MAX_D || vdim > 32 * SINK_MAX_D || kv_heads <= 0 || heads % kv_heads) return -2;
  if ((r1 == nullptr) != (r2 == nullptr)) return -2;
  const long long warps = (long long)n_tokens * heads;
  if (warps == 0) return 0;
  const int threads = 128;
  const long long blocks = (warps * 32 + threads - 1) / threads;
  if (dtype == 0)
    return launch_dependent(sink_attention_kernel<float>, dim3((unsigned)blocks), dim3(threads), 0, s, (const float*)q,
                            q_stride, (float*)out, (const float*)k_store, (const float*)v_store, block_table,
                            table_stride, tok_slot, tok_pos, r1, r2, sink, gate, n_tokens, heads, kv_heads, dim, vdim,
                            scale, chunk, window, keep, cap);
  return launch_dependent(sink_attention_kernel<bf16>, dim3((unsigned)blocks), dim3(threads), 0, s, (const bf16*)q,
                          q_stride, (bf16*)out, (const bf16*)k_store, (const bf16*)v_store, block_table, table_stride,
                          tok_slot, tok_pos, r1, r2, sink, gate, n_tokens, heads, kv_heads, dim, vdim, scale, chunk,
                          window, keep, cap);
}

}  // extern "C"
