// Row kernels of decoders that keep the residual stream in fp32: embedding lookup into the stream, RMS norm of the
// stream (weight stored either plainly or as an offset from one), the grouped RMS norm with a SiLU gate that follows
// a recurrent mixer (gate applied before or after the normalisation), SiLU * mul over an fp32 gate|up block, and
// the rounding of fp32 rows to the dtype that feeds the next matrix product (with or without a sigmoid gate per element),
// rotary positions on rows that stay in fp32, the norm of the stream with a choice of
// kind (RMS / dynamic tanh / layer norm) and a token shift, the weighted sum of the stored results of earlier layers, and
// the step between two sublayers of hyper-connected streams (update, read, norm).  All arithmetic is fp32; the output
// dtype is bf16 or fp32.  Beside the fp16 / bf16 row kernels of glue.cu (rmsnorm_kernel, silu_mul_kernel), which
// keep a 16-bit residual.
#include "../../include/b200_vllm.h"
#include <algorithm>

#include "seqmix.cuh"

namespace b200 {
using namespace seqmix;

// pos_base > 0: the sinusoidal position vector of the token's position p joins the row: entry 2i is
// sin(p * base^(-2i / width)), entry 2i + 1 the cosine of the same angle (frequency, angle, sine and cosine in fp32)
template <typename T>
__global__ void embed_f32_kernel(float* __restrict__ x, const T* __restrict__ table, const uint32_t* __restrict__ ids,
                                 const int64_t* __restrict__ positions, float pos_base, int width, int vocab,
                                 float scale, T* __restrict__ cast_out) {
  const int t = blockIdx.x;
  uint32_t id = ids[t];
  if (id >= static_cast<uint32_t>(vocab)) id = 0;
  const T* row = table + static_cast<size_t>(id) * width;
  const bool with_pos = pos_base > 0.f && positions != nullptr;
  const float p = with_pos ? static_cast<float>(positions[t]) : 0.f;
  for (int d = threadIdx.x; d < width; d += blockDim.x) {
    float v = ld(row + d) * scale;
    if (with_pos) {
      const float freq = powf(pos_base, -static_cast<float>(d & ~1) / static_cast<float>(width));
      const float ang = p * freq;
      v += (d & 1) ? cosf(ang) : sinf(ang);
    }
    x[static_cast<size_t>(t) * width + d] = v;
    if (cast_out) st(cast_out + static_cast<size_t>(t) * width + d, v);     // the row as the first sublayer reads it
  }
}

// out[r] = x[row(r)] / sqrt(mean(x^2) + eps) * (w_offset + w); rows == nullptr: row(r) = r; ldx: row stride of x
template <typename T>
__global__ void resid_rmsnorm_kernel(T* __restrict__ out, const float* __restrict__ x, size_t ldx,
                                     const float* __restrict__ w, int width, float eps, float w_offset,
                                     const uint32_t* __restrict__ rows) {
  __shared__ float red[33];
  const int r = blockIdx.x;
  const float* xr = x + static_cast<size_t>(rows ? rows[r] : r) * ldx;
  float ss = 0.f;
  for (int d = threadIdx.x; d < width; d += blockDim.x) ss += xr[d] * xr[d];
  ss = block_sum(ss, red);
  const float inv = 1.f / sqrtf(ss / static_cast<float>(width) + eps);
  for (int d = threadIdx.x; d < width; d += blockDim.x)
    st(out + static_cast<size_t>(r) * width + d, xr[d] * inv * (w_offset + w[d]));
}

// One block per (token, group of `group` channels).  gate_first: u = y * act(g), out = u / rms(u) * w;
// otherwise out = y / rms(y) * w * act(g).  w is indexed by (channel % w_period); w == nullptr: no weight.
// act = SiLU (gate_act 0) or the logistic sigmoid (gate_act 1).
template <typename T>
__global__ void gated_group_norm_kernel(T* __restrict__ out, const float* __restrict__ y, int ldy,
                                        const float* __restrict__ gate, int ldg, const float* __restrict__ w,
                                        int w_period, int C, int group, float eps, int gate_first, int gate_act) {
  __shared__ float red[33];
  const int t = blockIdx.x, g0 = blockIdx.y * group;
  const float* yr = y + static_cast<size_t>(t) * ldy + g0;
  const float* gr = gate + static_cast<size_t>(t) * ldg + g0;
  float ss = 0.f;
  for (int d = threadIdx.x; d < group; d += blockDim.x) {
    const float u = gate_first ? yr[d] * (gate_act ? sigmoid_f(gr[d]) : silu_exact(gr[d])) : yr[d];
    ss += u * u;
  }
  ss = block_sum(ss, red);
  const float inv = 1.f / sqrtf(ss / static_cast<float>(group) + eps);
  for (int d = threadIdx.x; d < group; d += blockDim.x) {
    const float s = gate_act ? sigmoid_f(gr[d]) : silu_exact(gr[d]);
    const float wv = w ? w[(g0 + d) % w_period] : 1.f;
    const float v = gate_first ? yr[d] * s * inv * wv : yr[d] * inv * wv * s;
    st(out + static_cast<size_t>(t) * C + g0 + d, v);
  }
}


// x[t] += y[t] / sqrt(mean(y[t]^2) + eps) * (w_offset + w): the norm AFTER a sublayer, folded into the residual sum.
// cast_out (may be NULL): the new row rounded to bf16, for a next sublayer whose input is the un-normed stream.
__global__ void resid_add_rmsnorm_kernel(float* __restrict__ x, const float* __restrict__ y, const float* __restrict__ w,
                                         int width, float eps, float w_offset, __nv_bfloat16* __restrict__ cast_out) {
  __shared__ float red[33];
  const int t = blockIdx.x;
  const float* yr = y + static_cast<size_t>(t) * width;
  float ss = 0.f;
  for (int d = threadIdx.x; d < width; d += blockDim.x) ss += yr[d] * yr[d];
  ss = block_sum(ss, red);
  const float inv = 1.f / sqrtf(ss / static_cast<float>(width) + eps);
  for (int d = threadIdx.x; d < width; d += blockDim.x) {
    const size_t i = static_cast<size_t>(t) * width + d;
    const float v = x[i] + yr[d] * inv * (w_offset + w[d]);
    x[i] = v;
    if (cast_out) cast_out[i] = __float2bfloat16_rn(v);
  }
}

// y[t, d] += scale * bias[d]
__global__ void bias_rows_kernel(float* __restrict__ y, const float* __restrict__ bias, float scale, int n, size_t total) {
  for (size_t i = blockIdx.x * static_cast<size_t>(blockDim.x) + threadIdx.x; i < total;
       i += static_cast<size_t>(gridDim.x) * blockDim.x)
    y[i] += scale * bias[i % n];
}

template <typename T>
__global__ void cast_rows_kernel(T* __restrict__ out, const float* __restrict__ in, int ld_in, int n, size_t total) {
  for (size_t i = blockIdx.x * static_cast<size_t>(blockDim.x) + threadIdx.x; i < total;
       i += static_cast<size_t>(gridDim.x) * blockDim.x) {
    const size_t t = i / n, d = i % n;
    st(out + i, in[t * ld_in + d]);
  }
}

template <typename T>
__global__ void silu_mul_f32_kernel(T* __restrict__ out, const float* __restrict__ gu, int ff, size_t total) {
  for (size_t i = blockIdx.x * static_cast<size_t>(blockDim.x) + threadIdx.x; i < total;
       i += static_cast<size_t>(gridDim.x) * blockDim.x) {
    const size_t t = i / ff, d = i % ff;
    st(out + i, silu_exact(gu[t * 2 * ff + d]) * gu[t * 2 * ff + ff + d]);
  }
}

// Rotary positions on `heads` neighbouring heads of an fp32 row, in place (the queries and keys of a recurrent mixer, which
// go into the scan as they lie in the projection row).  One block per token: cos / sin of the token's angles (angles in
// double) are made once in shared memory and serve every head.  Pairs are (i, i + rot_dims / 2) or interleaved (2i, 2i+1).
__global__ void rotary_rows_kernel(float* __restrict__ x, int ld, const double* __restrict__ rot_freq, float rot_mag,
                                   int rot_half, const int64_t* __restrict__ positions, int heads, int dim,
                                   int rot_dims) {
  extern __shared__ float sm[];          // cos[rot_dims / 2] | sin[rot_dims / 2]
  const int t = blockIdx.x, half = rot_dims / 2;
  float* cs = sm;
  float* sn = sm + half;
  const double pos = static_cast<double>(positions[t]);
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    double s, c;
    sincos(pos * rot_freq[i], &s, &c);
    cs[i] = static_cast<float>(c) * rot_mag;
    sn[i] = static_cast<float>(s) * rot_mag;
  }
  __syncthreads();
  float* row = x + static_cast<size_t>(t) * ld;
  for (int e = threadIdx.x; e < heads * half; e += blockDim.x) {
    const int h = e / half, i = e - h * half;
    float* a = row + static_cast<size_t>(h) * dim + (rot_half ? i : 2 * i);
    float* b = a + (rot_half ? half : 1);
    const float u = *a, v = *b;
    *a = u * cs[i] - v * sn[i];
    *b = v * cs[i] + u * sn[i];
  }
}

// V consecutive fp32 values of a thread (16-byte accesses for V = 4), stored as fp32 or rounded to bf16
template <int V> struct FloatVec;
template <> struct FloatVec<1> {
  float v[1];
  __device__ __forceinline__ void load(const float* p) { v[0] = *p; }
  __device__ __forceinline__ void store(float* p) const { *p = v[0]; }
};
template <> struct FloatVec<4> {
  float v[4];
  __device__ __forceinline__ void load(const float* p) {
    const float4 q = *reinterpret_cast<const float4*>(p);
    v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w;
  }
  __device__ __forceinline__ void store(float* p) const { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
};
template <int V> __device__ __forceinline__ void store_vec(float* p, const FloatVec<V>& f) { f.store(p); }
template <int V> __device__ __forceinline__ void store_vec(__nv_bfloat16* p, const FloatVec<V>& f) {
  if constexpr (V == 4) {
    __nv_bfloat162 q[2] = {__floats2bfloat162_rn(f.v[0], f.v[1]), __floats2bfloat162_rn(f.v[2], f.v[3])};
    *reinterpret_cast<uint2*>(p) = *reinterpret_cast<uint2*>(q);
  } else {
    *p = __float2bfloat16_rn(f.v[0]);
  }
}

// out[t, d] = in[t, d] * sigmoid(gate[t, d]) in the operand dtype; grid.x covers the columns (V per thread), grid.y the rows
template <typename T, int V>
__global__ void gate_rows_kernel(T* __restrict__ out, const float* __restrict__ in, const float* __restrict__ gate,
                                 int ld_gate, int n, int rows) {
  const int d = (blockIdx.x * blockDim.x + threadIdx.x) * V;
  if (d >= n) return;
  for (int t = blockIdx.y; t < rows; t += gridDim.y) {
    FloatVec<V> z, g;
    z.load(in + static_cast<size_t>(t) * n + d);
    g.load(gate + static_cast<size_t>(t) * ld_gate + d);
#pragma unroll
    for (int c = 0; c < V; ++c) z.v[c] *= sigmoid_f(g.v[c]);
    store_vec<V>(out + static_cast<size_t>(t) * n + d, z);
  }
}

// out[t, d] = act(up[t, d] + bias[d]) (* sigmoid(up[t, gate_col]) when gate_col >= 0); ACT 1: relu(.)^2, 2: the exact GELU.
// grid.x covers the columns (V per thread), grid.y the rows
template <typename T, int ACT, int V>
__global__ void ff_act_kernel(T* __restrict__ out, const float* __restrict__ up, int ld, int ff, int gate_col,
                              const float* __restrict__ bias, int rows) {
  const int d = (blockIdx.x * blockDim.x + threadIdx.x) * V;
  if (d >= ff) return;
  FloatVec<V> b;
#pragma unroll
  for (int c = 0; c < V; ++c) b.v[c] = 0.f;
  if (bias) b.load(bias + d);
  for (int t = blockIdx.y; t < rows; t += gridDim.y) {
    const float* row = up + static_cast<size_t>(t) * ld;
    const float g = gate_col >= 0 ? sigmoid_f(row[gate_col]) : 1.f;
    FloatVec<V> z;
    z.load(row + d);
#pragma unroll
    for (int c = 0; c < V; ++c) {
      const float v = z.v[c] + b.v[c], r = fmaxf(v, 0.f);
      z.v[c] = (ACT == 1 ? r * r : 0.5f * v * (1.f + erff(v * 0.70710678118654752f))) * g;
    }
    store_vec<V>(out + static_cast<size_t>(t) * ff + d, z);
  }
}

// One block per output row: a norm of the stream (RMS, layer norm, or the dynamic tanh  tanh(alpha x) w + b  that needs
// no statistics) and, with shift_w, the token shift behind it:  out[t] = n[t] + (n[t-1] - n[t]) * shift_w, where n[t-1] is
// the un-shifted norm of the sequence's previous token -- recomputed from the row above, or, for the first row of a
// portion, read from the sequence's shift state (zeros at position 0).  The block of a sequence's FIRST row also writes
// the state: the un-shifted norm of the sequence's last row of the step.  Every thread reads the state entries it later
// overwrites, so the portion's first row sees the old state whatever the order of the blocks.
template <typename T>
__global__ void stream_norm_kernel(T* __restrict__ out, const float* __restrict__ x, const float* __restrict__ w,
                                   const float* __restrict__ bias, float alpha, int kind, int width, float eps,
                                   float w_offset, const uint32_t* __restrict__ rows, const float* __restrict__ shift_w,
                                   float* __restrict__ shift_state, const int32_t* __restrict__ slots,
                                   const uint32_t* __restrict__ cu, const uint32_t* __restrict__ ctx, int num_seqs) {
  __shared__ float red[33];
  const int r = blockIdx.x;
  const int t = rows ? static_cast<int>(rows[r]) : r;
  const float* xr = x + static_cast<size_t>(t) * width;
  // (mean, inverse root mean square of what is left of the mean) of a row; the RMS kind has no mean
  auto stats = [&](const float* row) {
    float mean = 0.f, ss = 0.f;
    if (kind == B200_NORM_LAYER) {
      for (int d = threadIdx.x; d < width; d += blockDim.x) mean += row[d];
      mean = block_sum(mean, red) / static_cast<float>(width);
    }
    for (int d = threadIdx.x; d < width; d += blockDim.x) ss += (row[d] - mean) * (row[d] - mean);
    ss = block_sum(ss, red);
    return make_float2(mean, 1.f / sqrtf(ss / static_cast<float>(width) + eps));
  };
  auto normed = [&](const float* row, float2 m, int d) {
    const float b = bias ? bias[d] : 0.f;
    return kind == B200_NORM_DYNTANH ? tanhf(alpha * row[d]) * w[d] + b : (row[d] - m.x) * m.y * (w_offset + w[d]) + b;
  };
  const float2 none = make_float2(0.f, 1.f);
  const float2 inv = kind == B200_NORM_DYNTANH ? none : stats(xr);
  if (!shift_w) {
    for (int d = threadIdx.x; d < width; d += blockDim.x) st(out + static_cast<size_t>(r) * width + d, normed(xr, inv, d));
    return;
  }
  const int b = seq_of_row(cu, num_seqs, t);
  const int t0 = static_cast<int>(cu[b]), t1 = static_cast<int>(cu[b + 1]);
  const bool first = t == t0;
  const bool fresh = static_cast<int>(ctx[b]) == t1 - t0;          // the sequence starts in this step
  float* sp = shift_state + static_cast<size_t>(slots[b]) * width;
  const float* xp = xr - width;                                      // the row above (same sequence unless `first`)
  const float* xl = x + static_cast<size_t>(t1 - 1) * width;         // the sequence's last row of the step
  const float2 inv_p = (kind == B200_NORM_DYNTANH || first) ? none : stats(xp);
  const float2 inv_l = (kind == B200_NORM_DYNTANH || !first) ? none : (t1 - 1 == t ? inv : stats(xl));
  for (int d = threadIdx.x; d < width; d += blockDim.x) {
    const float n = normed(xr, inv, d);
    const float prev = first ? (fresh ? 0.f : sp[d]) : normed(xp, inv_p, d);
    st(out + static_cast<size_t>(r) * width + d, n + (prev - n) * shift_w[d]);
    if (first) sp[d] = t1 - 1 == t ? n : normed(xl, inv_l, d);
  }
}

// One block per row: the step between two sublayers of hyper-connected streams (see b200_hyper_step).  A thread owns the
// same columns in every stream, so the streams can be rewritten in place: it reads a column of all S old streams and of
// the sublayer's row, forms every new stream from them, stores it, and keeps only the next sublayer's weighted sum, which
// the block then norms from shared memory (mean first, then the squared deviations from it).  The S x S matrix and the
// weight vectors sit in shared memory.
struct HyperArgs {
  void* out;
  float* x_out;
  size_t out_stride;
  const float* x_in;
  size_t in_stride;
  const float *y, *down;
  const int32_t* slot_of_pair;
  const float* top_w;
  int top;
  const float *mix, *out_w, *in_w, *w, *bias;
  float alpha;
  int kind;
  float eps, w_offset;
  const uint32_t* rows;
  int streams, width;
};
template <typename T, int MS, int V>
__global__ void hyper_step_kernel(const HyperArgs a) {
  // red[36] | mix[S * S] | out_w[S] | in_w[S] | choice weights[top] | choice rows[top] | u[width] (16-byte aligned)
  extern __shared__ __align__(16) float sm[];
  const int S = a.streams, r = blockIdx.x, width = a.width;
  float* red = sm;
  float* mix = red + 36;
  float* ow = mix + S * S;
  float* iw = ow + S;
  float* cw = iw + S;
  int* cr = reinterpret_cast<int*>(cw + a.top);
  float* u = sm + ((36 + S * S + 2 * S + 2 * a.top + 3) & ~3);
  const size_t t = a.rows ? a.rows[r] : r;
  const bool update = a.y != nullptr || a.down != nullptr;
  for (int i = threadIdx.x; i < S * S; i += blockDim.x) {
    const float m = a.mix ? a.mix[i] : (i % (S + 1) == 0 ? 1.f : 0.f);
    mix[i] = update ? m : 0.f;
  }
  for (int i = threadIdx.x; i < S; i += blockDim.x) {
    ow[i] = update ? (a.out_w ? a.out_w[i] : 1.f) : 0.f;
    iw[i] = a.in_w ? a.in_w[i] : 1.f;
  }
  for (int i = threadIdx.x; i < a.top; i += blockDim.x) {
    cw[i] = a.top_w[t * a.top + i];
    cr[i] = a.slot_of_pair[t * a.top + i];
  }
  __syncthreads();
  const float* xr = a.x_in + t * width;
  float sum = 0.f;
  for (int d = threadIdx.x * V; d < width; d += blockDim.x * V) {
    FloatVec<V> x[MS], y, acc;
#pragma unroll
    for (int s = 0; s < MS; ++s) {
      if (s >= S) continue;
      if (s > 0 && a.in_stride == 0) x[s] = x[0];
      else x[s].load(xr + s * a.in_stride + d);
    }
#pragma unroll
    for (int c = 0; c < V; ++c) acc.v[c] = y.v[c] = 0.f;
    if (a.down) {
      for (int j = 0; j < a.top; ++j) {
        FloatVec<V> e;
        e.load(a.down + static_cast<size_t>(cr[j]) * width + d);
#pragma unroll
        for (int c = 0; c < V; ++c) y.v[c] += cw[j] * e.v[c];
      }
    } else if (a.y) {
      y.load(a.y + t * width + d);
    }
#pragma unroll
    for (int k = 0; k < MS; ++k) {
      if (k >= S) continue;
      FloatVec<V> z;
      if (update) {
#pragma unroll
        for (int c = 0; c < V; ++c) z.v[c] = ow[k] * y.v[c];
#pragma unroll
        for (int s = 0; s < MS; ++s) {
          if (s >= S) continue;
          const float m = mix[s * S + k];
#pragma unroll
          for (int c = 0; c < V; ++c) z.v[c] += m * x[s].v[c];
        }
      } else {
        z = x[k];
      }
      if (a.x_out) z.store(a.x_out + k * a.out_stride + t * width + d);
#pragma unroll
      for (int c = 0; c < V; ++c) acc.v[c] += iw[k] * z.v[c];
    }
    if (a.out) {
      acc.store(u + d);
#pragma unroll
      for (int c = 0; c < V; ++c) sum += acc.v[c];
    }
  }
  if (!a.out) return;
  float mean = 0.f, inv = 1.f;
  if (a.kind == B200_NORM_LAYER) mean = block_sum(sum, red) / static_cast<float>(width);
  if (a.kind != B200_NORM_DYNTANH) {
    float ss = 0.f;
    for (int d = threadIdx.x * V; d < width; d += blockDim.x * V) {
      FloatVec<V> f;
      f.load(u + d);
#pragma unroll
      for (int c = 0; c < V; ++c) ss += (f.v[c] - mean) * (f.v[c] - mean);
    }
    ss = block_sum(ss, red);
    inv = 1.f / sqrtf(ss / static_cast<float>(width) + a.eps);
  }
  T* o = reinterpret_cast<T*>(a.out) + static_cast<size_t>(r) * width;
  for (int d = threadIdx.x * V; d < width; d += blockDim.x * V) {      // a thread's own columns: no barrier needed
    FloatVec<V> f, wv, bv;
    f.load(u + d);
    wv.load(a.w + d);
#pragma unroll
    for (int c = 0; c < V; ++c) bv.v[c] = 0.f;
    if (a.bias) bv.load(a.bias + d);
#pragma unroll
    for (int c = 0; c < V; ++c)
      f.v[c] = a.kind == B200_NORM_DYNTANH ? tanhf(a.alpha * f.v[c]) * wv.v[c] + bv.v[c]
                                           : (f.v[c] - mean) * inv * (a.w_offset + wv.v[c]) + bv.v[c];
    store_vec<V>(o + d, f);
  }
}

// out[i] = sum_j w[j] * hist[j * stride + i] (w == nullptr: ones), V floats per thread and step
template <int V>
__global__ void depth_mix_kernel(float* __restrict__ out, const float* __restrict__ hist, size_t stride,
                                 const float* __restrict__ w, int count, size_t n) {
  for (size_t i = blockIdx.x * static_cast<size_t>(blockDim.x) + threadIdx.x; i < n;
       i += static_cast<size_t>(gridDim.x) * blockDim.x) {
    if constexpr (V == 4) {
      float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int j = 0; j < count; ++j) {
        const float wj = w ? w[j] : 1.f;
        const float4 v = *reinterpret_cast<const float4*>(hist + j * stride + i * 4);
        acc.x += wj * v.x; acc.y += wj * v.y; acc.z += wj * v.z; acc.w += wj * v.w;
      }
      *reinterpret_cast<float4*>(out + i * 4) = acc;
    } else {
      float acc = 0.f;
      for (int j = 0; j < count; ++j) acc += (w ? w[j] : 1.f) * hist[j * stride + i];
      out[i] = acc;
    }
  }
}

static int flat_grid(size_t total) {
  const size_t b = (total + 255) / 256;
  return static_cast<int>(b < 1 ? 1 : (b > 148 * 16 ? 148 * 16 : b));
}

void launch_embed_f32(float* x, const void* table, const uint32_t* ids, const int64_t* positions, float pos_base, int T,
                      int width, int vocab, float scale, int dt, void* cast_out, cudaStream_t st_) {
  if (T <= 0) return;
  if (dt)
    embed_f32_kernel<float><<<T, 256, 0, st_>>>(x, (const float*)table, ids, positions, pos_base, width, vocab, scale,
                                                nullptr);
  else
    embed_f32_kernel<__nv_bfloat16><<<T, 256, 0, st_>>>(x, (const __nv_bfloat16*)table, ids, positions, pos_base, width,
                                                        vocab, scale, (__nv_bfloat16*)cast_out);
  B200_CUDA_LAUNCH_CHECK();
}

void launch_resid_rmsnorm(void* out, const float* x, const float* w, int T, int width, float eps, float w_offset,
                          const uint32_t* rows, int dt, cudaStream_t st_, int ldx) {
  if (T <= 0) return;
  if (ldx == 0) ldx = width;
  if (dt)
    resid_rmsnorm_kernel<float><<<T, 256, 0, st_>>>((float*)out, x, ldx, w, width, eps, w_offset, rows);
  else
    resid_rmsnorm_kernel<__nv_bfloat16><<<T, 256, 0, st_>>>((__nv_bfloat16*)out, x, ldx, w, width, eps, w_offset, rows);
  B200_CUDA_LAUNCH_CHECK();
}

void launch_gated_group_norm(void* out, const float* y, int ldy, const float* gate, int ldg, const float* w,
                             int w_period, int T, int C, int group, float eps, int gate_first, int gate_act, int dt,
                             cudaStream_t st_) {
  if (T <= 0) return;
  const dim3 grid(T, C / group);
  const int threads = group >= 256 ? 256 : (group >= 128 ? 128 : 64);
  if (dt)
    gated_group_norm_kernel<float><<<grid, threads, 0, st_>>>((float*)out, y, ldy, gate, ldg, w, w_period, C, group,
                                                              eps, gate_first, gate_act);
  else
    gated_group_norm_kernel<__nv_bfloat16><<<grid, threads, 0, st_>>>((__nv_bfloat16*)out, y, ldy, gate, ldg, w,
                                                                      w_period, C, group, eps, gate_first, gate_act);
  B200_CUDA_LAUNCH_CHECK();
}

void launch_resid_add_rmsnorm(float* x, const float* y, const float* w, int T, int width, float eps, float w_offset,
                              void* cast_out, cudaStream_t st_) {
  if (T <= 0) return;
  resid_add_rmsnorm_kernel<<<T, 256, 0, st_>>>(x, y, w, width, eps, w_offset, (__nv_bfloat16*)cast_out);
  B200_CUDA_LAUNCH_CHECK();
}

void launch_bias_rows(float* y, const float* bias, float scale, int T, int n, cudaStream_t st_) {
  const size_t total = static_cast<size_t>(T) * n;
  if (total == 0) return;
  bias_rows_kernel<<<flat_grid(total), 256, 0, st_>>>(y, bias, scale, n, total);
  B200_CUDA_LAUNCH_CHECK();
}

void launch_cast_rows(void* out, const float* in, int ld_in, int T, int n, int dt, cudaStream_t st_) {
  const size_t total = static_cast<size_t>(T) * n;
  if (total == 0) return;
  if (dt)
    cast_rows_kernel<float><<<flat_grid(total), 256, 0, st_>>>((float*)out, in, ld_in, n, total);
  else
    cast_rows_kernel<__nv_bfloat16><<<flat_grid(total), 256, 0, st_>>>((__nv_bfloat16*)out, in, ld_in, n, total);
  B200_CUDA_LAUNCH_CHECK();
}

void launch_silu_mul_f32(void* out, const float* gate_up, int T, int ff, int dt, cudaStream_t st_) {
  const size_t total = static_cast<size_t>(T) * ff;
  if (total == 0) return;
  if (dt)
    silu_mul_f32_kernel<float><<<flat_grid(total), 256, 0, st_>>>((float*)out, gate_up, ff, total);
  else
    silu_mul_f32_kernel<__nv_bfloat16><<<flat_grid(total), 256, 0, st_>>>((__nv_bfloat16*)out, gate_up, ff, total);
  B200_CUDA_LAUNCH_CHECK();
}

void launch_ff_act(void* out, const float* up, int ld, int T, int ff, int gate_col, const float* bias, int act, int dt,
                   cudaStream_t st_) {
  if (T <= 0 || ff <= 0) return;
  if (act != 1 && act != 2) {
    set_error(1, "ff_act: unknown activation");
    return;
  }
  const bool vec = ff % 4 == 0 && ld % 4 == 0 &&
                   (reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(up) | reinterpret_cast<uintptr_t>(bias)) % 16 == 0;
  const int per_block = 256 * (vec ? 4 : 1);
  const dim3 grid((ff + per_block - 1) / per_block, std::min(T, 32768));
  auto go = [&](auto* o, auto kern) { kern<<<grid, 256, 0, st_>>>(o, up, ld, ff, gate_col, bias, T); };
#define B200_FF_ACT(TYPE)                                                                     \
  if (vec) go((TYPE*)out, act == 1 ? ff_act_kernel<TYPE, 1, 4> : ff_act_kernel<TYPE, 2, 4>);   \
  else go((TYPE*)out, act == 1 ? ff_act_kernel<TYPE, 1, 1> : ff_act_kernel<TYPE, 2, 1>);
  if (dt) { B200_FF_ACT(float) } else { B200_FF_ACT(__nv_bfloat16) }
#undef B200_FF_ACT
  B200_CUDA_LAUNCH_CHECK();
}

void launch_rotary_rows(float* x, int ld, const double* rot_freq, float rot_mag, int rot_half, const int64_t* positions,
                        int T, int heads, int dim, int rot_dims, cudaStream_t st_) {
  if (T <= 0 || heads <= 0 || rot_dims <= 0) return;
  const int pairs = heads * (rot_dims / 2);
  const int threads = pairs >= 1024 ? 512 : (pairs >= 256 ? 256 : 128);
  rotary_rows_kernel<<<T, threads, static_cast<size_t>(rot_dims) * 4, st_>>>(x, ld, rot_freq, rot_mag, rot_half, positions,
                                                                             heads, dim, rot_dims);
  B200_CUDA_LAUNCH_CHECK();
}

void launch_gate_rows(void* out, const float* in, const float* gate, int ld_gate, int T, int n, int dt, cudaStream_t st_) {
  if (T <= 0 || n <= 0) return;
  const bool vec = n % 4 == 0 && ld_gate % 4 == 0 &&
                   (reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(in) | reinterpret_cast<uintptr_t>(gate)) % 16 == 0;
  const int per_block = 256 * (vec ? 4 : 1);
  const dim3 grid((n + per_block - 1) / per_block, std::min(T, 32768));
  auto go = [&](auto* o, auto kern) { kern<<<grid, 256, 0, st_>>>(o, in, gate, ld_gate, n, T); };
  if (dt) go((float*)out, vec ? gate_rows_kernel<float, 4> : gate_rows_kernel<float, 1>);
  else go((__nv_bfloat16*)out, vec ? gate_rows_kernel<__nv_bfloat16, 4> : gate_rows_kernel<__nv_bfloat16, 1>);
  B200_CUDA_LAUNCH_CHECK();
}

void launch_stream_norm(void* out, const float* x, const float* w, const float* bias, float alpha, int kind, float eps,
                        float w_offset, const uint32_t* rows, const float* shift_w, float* shift_state,
                        const int32_t* slots, const uint32_t* cu, const uint32_t* ctx, int num_seqs, int T, int width,
                        int dt, cudaStream_t st_) {
  if (T <= 0) return;
  if (dt)
    stream_norm_kernel<float><<<T, 256, 0, st_>>>((float*)out, x, w, bias, alpha, kind, width, eps, w_offset, rows, shift_w,
                                                  shift_state, slots, cu, ctx, num_seqs);
  else
    stream_norm_kernel<__nv_bfloat16><<<T, 256, 0, st_>>>((__nv_bfloat16*)out, x, w, bias, alpha, kind, width, eps, w_offset,
                                                          rows, shift_w, shift_state, slots, cu, ctx, num_seqs);
  B200_CUDA_LAUNCH_CHECK();
}

template <typename T, int MS>
static void hyper_step_vec(const HyperArgs& a, int rows, bool vec, size_t smem, cudaStream_t st_) {
  auto go = [&](auto kern, int threads) {
    cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    kern<<<rows, threads, smem, st_>>>(a);
  };
  if (vec) go(hyper_step_kernel<T, MS, 4>, a.width >= 1024 ? 256 : (a.width >= 512 ? 128 : 64));
  else go(hyper_step_kernel<T, MS, 1>, 256);
}

void launch_hyper_step(void* out, float* x_out, size_t out_stride, const float* x_in, size_t in_stride, const float* y,
                       const float* down, const int32_t* slot_of_pair, const float* top_w, int top, const float* mix,
                       const float* out_w, const float* in_w, const float* w, const float* bias, float alpha, int kind,
                       float eps, float w_offset, const uint32_t* rows, int streams, int T, int width, int dt,
                       cudaStream_t st_) {
  if (T <= 0) return;
  if (streams < 1 || streams > B200_MAX_STREAMS) {
    set_error(1, "hyper_step: 1 to 16 streams");
    return;
  }
  if (!down) top = 0;
  const HyperArgs a{out, x_out, out_stride, x_in, in_stride, y, down, slot_of_pair, top_w, top, mix, out_w, in_w, w, bias,
                    alpha, kind, eps, w_offset, rows, streams, width};
  const size_t smem = (static_cast<size_t>((36 + streams * streams + 2 * streams + 2 * top + 3) & ~3) + width) * 4;
  if (smem > 220 * 1024) {
    set_error(1, "hyper_step: rows too wide for shared memory");
    return;
  }
  auto al = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
  const bool vec = width % 4 == 0 && in_stride % 4 == 0 && out_stride % 4 == 0 && al(out) && al(x_out) && al(x_in) && al(y) &&
                   al(down) && al(w) && al(bias);
#define B200_HYPER(MS)                                                     \
  if (dt) hyper_step_vec<float, MS>(a, T, vec, smem, st_);                 \
  else hyper_step_vec<__nv_bfloat16, MS>(a, T, vec, smem, st_);
  if (streams == 1) { B200_HYPER(1) }
  else if (streams == 2) { B200_HYPER(2) }
  else if (streams <= 4) { B200_HYPER(4) }
  else if (streams <= 8) { B200_HYPER(8) }
  else { B200_HYPER(16) }
#undef B200_HYPER
  B200_CUDA_LAUNCH_CHECK();
}

void launch_depth_mix(float* out, const float* hist, size_t stride, const float* w, int count, size_t n, cudaStream_t st_) {
  if (n == 0 || count <= 0) return;
  if (n % 4 == 0 && stride % 4 == 0 && (reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(hist)) % 16 == 0)
    depth_mix_kernel<4><<<flat_grid(n / 4), 256, 0, st_>>>(out, hist, stride, w, count, n / 4);
  else
    depth_mix_kernel<1><<<flat_grid(n), 256, 0, st_>>>(out, hist, stride, w, count, n);
  B200_CUDA_LAUNCH_CHECK();
}

}  // namespace b200

extern "C" {
// RMS norm of an fp32 residual stream: out[r] (bf16 when dt == 0, fp32 when dt == 1) = x[r] / sqrt(mean(x[r]^2) + eps)
// * (w_offset + w); w fp32 [width]; w_offset = 1 for weights stored around zero, 0 for plain weights.
void b200_resid_rmsnorm(void* out, const float* x, const float* w, int32_t num_tokens, int32_t width, float eps,
                        float w_offset, int32_t dt, int64_t stream) {
  B200_CHECK_ARG(out && x && w && width > 0 && (dt == 0 || dt == 1), "resid_rmsnorm: bad arguments");
  b200::launch_resid_rmsnorm(out, x, w, num_tokens, width, eps, w_offset, nullptr, dt,
                             reinterpret_cast<cudaStream_t>(stream));
}
// Grouped RMS norm with a SiLU gate over fp32 rows y [T, C] (row stride ldy), gate [T, C] (row stride ldg); groups of
// `group` consecutive channels are normalised separately; w fp32 is indexed by channel % w_period (a per-head weight
// shared by all heads has w_period = group; w NULL: no weight).  gate_first != 0: norm(y * act(gate)) * w; else
// norm(y) * w * act(gate); act = SiLU (gate_act 0) or sigmoid (gate_act 1).
void b200_gated_group_norm(void* out, const float* y, int32_t ldy, const float* gate, int32_t ldg, const float* w,
                           int32_t w_period, int32_t num_tokens, int32_t channels, int32_t group, float eps,
                           int32_t gate_first, int32_t gate_act, int32_t dt, int64_t stream) {
  B200_CHECK_ARG(out && y && gate && group > 0 && channels % group == 0 && w_period > 0 && (dt == 0 || dt == 1),
                 "gated_group_norm: bad arguments");
  b200::launch_gated_group_norm(out, y, ldy, gate, ldg, w, w_period, num_tokens, channels, group, eps, gate_first,
                                gate_act, dt, reinterpret_cast<cudaStream_t>(stream));
}
// x fp32 [T, width] += y / sqrt(mean(y^2) + eps) * (w_offset + w): the norm that follows a sublayer, with its residual sum.
void b200_resid_add_rmsnorm(float* x, const float* y, const float* w, int32_t num_tokens, int32_t width, float eps,
                            float w_offset, int64_t stream) {
  B200_CHECK_ARG(x && y && w && width > 0, "resid_add_rmsnorm: bad arguments");
  b200::launch_resid_add_rmsnorm(x, y, w, num_tokens, width, eps, w_offset, nullptr,
                                 reinterpret_cast<cudaStream_t>(stream));
}
void b200_rmsnorm_rows(void* out, const float* x, int32_t ldx, const float* w, int32_t num_tokens, int32_t n, float eps,
                       float w_offset, int32_t dt, int64_t stream) {
  B200_CHECK_ARG(out && x && w && n > 0 && ldx >= n && (dt == 0 || dt == 1), "rmsnorm_rows: bad arguments");
  b200::launch_resid_rmsnorm(out, x, w, num_tokens, n, eps, w_offset, nullptr, dt, reinterpret_cast<cudaStream_t>(stream), ldx);
}
void b200_rotary_rows(float* x, int32_t ld, const double* rot_freq, float rot_mag, int32_t rot_half,
                      const int64_t* positions, int32_t num_tokens, int32_t heads, int32_t dim, int32_t rot_dims,
                      int64_t stream) {
  B200_CHECK_ARG(x && positions && heads > 0 && dim > 0 && ld >= heads * dim && rot_dims >= 0 && rot_dims <= dim &&
                     rot_dims % 2 == 0 && (rot_dims == 0 || rot_freq),
                 "rotary_rows: bad arguments");
  b200::launch_rotary_rows(x, ld, rot_freq, rot_mag, rot_half, positions, num_tokens, heads, dim, rot_dims,
                           reinterpret_cast<cudaStream_t>(stream));
}
void b200_gate_rows(void* out, const float* in, const float* gate, int32_t ld_gate, int32_t num_tokens, int32_t n,
                    int32_t dt, int64_t stream) {
  B200_CHECK_ARG(out && in && gate && n > 0 && ld_gate >= n && (dt == 0 || dt == 1), "gate_rows: bad arguments");
  b200::launch_gate_rows(out, in, gate, ld_gate, num_tokens, n, dt, reinterpret_cast<cudaStream_t>(stream));
}
void b200_stream_norm(void* out, const float* x, const float* w, const float* bias, float alpha, int32_t kind,
                      float eps, float w_offset, const uint32_t* rows, const float* shift_w, float* shift_state,
                      const int32_t* state_slots, const uint32_t* cu_seqlens_q, const uint32_t* context_lens,
                      int32_t num_seqs, int32_t num_tokens, int32_t width, int32_t dt, int64_t stream) {
  B200_CHECK_ARG(out && x && w && width > 0 && (dt == 0 || dt == 1) && kind >= B200_NORM_RMS && kind <= B200_NORM_LAYER &&
                     (!shift_w || (!rows && shift_state && state_slots && cu_seqlens_q && context_lens && num_seqs > 0)),
                 "stream_norm: bad arguments (a token shift needs the step's sequences and a state, and no row list)");
  b200::launch_stream_norm(out, x, w, bias, alpha, kind, eps, w_offset, rows, shift_w, shift_state, state_slots,
                           cu_seqlens_q, context_lens, num_seqs, num_tokens, width, dt,
                           reinterpret_cast<cudaStream_t>(stream));
}
void b200_hyper_step(void* out, float* x_out, int64_t out_stride, const float* x_in, int64_t in_stride, const float* y,
                     const float* down, const int32_t* slot_of_pair, const float* top_w, int32_t top, const float* mix,
                     const float* out_w, const float* in_w, const float* w, const float* bias, float alpha, int32_t kind,
                     float eps, float w_offset, const uint32_t* rows, int32_t streams, int32_t num_tokens, int32_t width,
                     int32_t dt, int64_t stream) {
  B200_CHECK_ARG((out || x_out) && x_in && width > 0 && (dt == 0 || dt == 1) && in_stride >= 0 && out_stride >= 0 &&
                     (!out || w) && (!down || (slot_of_pair && top_w && top > 0)) &&
                     (!rows || !x_out) && kind >= B200_NORM_RMS && kind <= B200_NORM_LAYER,
                 "hyper_step: bad arguments");
  b200::launch_hyper_step(out, x_out, static_cast<size_t>(out_stride), x_in, static_cast<size_t>(in_stride), y, down,
                          slot_of_pair, top_w, top, mix, out_w, in_w, w, bias, alpha, kind, eps, w_offset, rows, streams,
                          num_tokens, width, dt, reinterpret_cast<cudaStream_t>(stream));
}
void b200_ff_act(void* out, const float* up, int32_t ld, const float* bias, int32_t act, int32_t num_tokens, int32_t n,
                 int32_t dt, int64_t stream) {
  B200_CHECK_ARG(out && up && n > 0 && ld >= n && (act == 1 || act == 2) && (dt == 0 || dt == 1), "ff_act: bad arguments");
  b200::launch_ff_act(out, up, ld, num_tokens, n, -1, bias, act, dt, reinterpret_cast<cudaStream_t>(stream));
}
void b200_depth_mix(float* out, const float* hist, int64_t stride, const float* w, int32_t count, int64_t n,
                    int64_t stream) {
  B200_CHECK_ARG(out && hist && count > 0 && stride >= 0 && n >= 0, "depth_mix: bad arguments");
  b200::launch_depth_mix(out, hist, static_cast<size_t>(stride), w, count, static_cast<size_t>(n),
                         reinterpret_cast<cudaStream_t>(stream));
}
}
