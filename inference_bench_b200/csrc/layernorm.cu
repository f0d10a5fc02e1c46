// Layer norm, with or without a bias, fused with the residual add that precedes it, and the pieces of a block whose sublayers read
// their input through a short causal convolution over time and whose layers are mixed by a depth-weighted average.
// All arithmetic is float32; only a stored activation may be bfloat16.
//
//  * add_layernorm: v = x[t] + scale * (sum_p delta[p][t] + bias)   (scale, bias: per channel, optional; partial sums added in order)
//                   (+ the partial sums of a second contribution, where two sublayers ran side by side on one normed input)
//                   x[t] = v (optional), x_copy[t] = v (optional)
//                   out = w * (v - mean(v)) / sqrt(mean((v - mean)^2) + eps) [+ b]
//    With `halo` > 0 the output rows are laid out for the convolution that follows: segment s (tokens a..b of the flat batch) owns
//    rows a + s * halo .. b + (s + 1) * halo; its first `halo` rows are the request's last `halo` normed rows of earlier steps, copied
//    from its state slot by extra blocks of this kernel, so the convolution reads one array and its state update races with nothing.
//  * causal_conv_rows: out[t] = h[t] + sum_j w[j, :] * h[t - taps + 1 + j] on that layout (w is [taps][channels]: a tap's weights lie together), and the request's new state (the last
//    `halo` = taps - 1 rows of its extended run) written back to its slot.
//  * add_layernorm_conv_single: both of the above in one kernel for a step in which every request brings one token (decoded tokens): a CTA
//    per token norms its row, reads the request's `halo` state rows, writes the convolved row and shifts the state by one row.
//  * depth_average: X = x[t] + scale * (sum_p delta[p][t] + bias); stack[k][t] = X; x[t] = sum_{j <= k} mix[j] * stack[j][t].
//  * scale_values: v *= s (logits times a constant); softcap_values: v = cap tanh(v / cap).
//  * embed_layernorm: the layer norm of a token's row of the embedding table.
//  * shift_mixes: several mixes of every normed row with the row before it (a different weight per channel each), and
//    add_layernorm_mixes_single: the residual add, the norm and the mixes in one kernel for steps of single tokens.
#include <type_traits>

#include "common.cuh"

namespace {

constexpr int kLnThreads = 256;

struct LnExtras {
  const float* wb;   // the norm's bias per channel, or null
  float mult;        // factor on the contribution where there is no per-channel scale
  int early;         // 1: the kernels that follow may be scheduled while this one runs; 0: only when it is done (for the reason given in causal_conv_rows_kernel)
  const float* delta2;   // add_layernorm: a second contribution of P2 partial sums (stride2 apart), added after the first; P2 = 0: none
  int P2;
  size_t stride2;
};

template <typename O>
__global__ void __launch_bounds__(kLnThreads) add_layernorm_kernel(float* __restrict__ x, const float* __restrict__ delta, int P, size_t delta_stride,
                                                                   const float* __restrict__ dscale, const float* __restrict__ dbias,
                                                                   const float* __restrict__ w, O* __restrict__ out, const int* __restrict__ rows, int n_rows,
                                                                   int H, float eps, int write_x, float* __restrict__ x_copy, int halo,
                                                                   const int* __restrict__ seg_of_token, const int* __restrict__ seg_start,
                                                                   const int* __restrict__ seg_slot, const float* __restrict__ state, size_t slot_stride, LnExtras ex) {
  extern __shared__ __align__(16) float row[];
  __shared__ float scratch[32];
  if (ex.early) ib::pdl_launch_dependents();
  ib::pdl_wait();
  const int r = blockIdx.x;
  if (r >= n_rows) {   // a halo row: the request's state of earlier steps, as it is
    const int hb = r - n_rows, s = hb / halo, j = hb % halo;
    const float* src = state + (size_t)seg_slot[s] * slot_stride + (size_t)j * H;
    O* dst = out + ((size_t)seg_start[s] + (size_t)s * halo + j) * H;
    for (int i = threadIdx.x; i < H; i += blockDim.x) dst[i] = ib::from_f32<O>(src[i]);
    return;
  }
  const int t = rows ? rows[r] : r;
  float* xr = x + (size_t)t * H;
  float sum = 0.f;
  for (int i = threadIdx.x; i < H; i += blockDim.x) {
    float v = xr[i];
    if (P > 0 || dbias) {
      float d = dbias ? dbias[i] : 0.f;
      if (P > 0) {
        float a = delta[(size_t)t * H + i];
        for (int p = 1; p < P; p++) a += delta[p * delta_stride + (size_t)t * H + i];
        d = dbias ? a + d : a;
      }
      v = __fmaf_rn(dscale ? dscale[i] : ex.mult, d, v);
    }
    if (ex.P2 > 0) {
      float a = ex.delta2[(size_t)t * H + i];
      for (int p = 1; p < ex.P2; p++) a += ex.delta2[p * ex.stride2 + (size_t)t * H + i];
      v += a;
    }
    if (write_x && (P > 0 || dbias || ex.P2 > 0)) xr[i] = v;
    if (x_copy) x_copy[(size_t)t * H + i] = v;
    row[i] = v;
    sum += v;
  }
  const float mean = ib::block_sum(sum, scratch) / (float)H;
  float sq = 0.f;
  for (int i = threadIdx.x; i < H; i += blockDim.x) {
    const float c = row[i] - mean;
    sq = __fmaf_rn(c, c, sq);
  }
  const float inv = rsqrtf(ib::block_sum(sq, scratch) / (float)H + eps);
  const size_t orow = halo ? (size_t)t + (size_t)(seg_of_token[t] + 1) * halo : (size_t)r;
  O* dst = out + orow * H;
  for (int i = threadIdx.x; i < H; i += blockDim.x) dst[i] = ib::from_f32<O>(__fmaf_rn((row[i] - mean) * inv, w[i], ex.wb ? ex.wb[i] : 0.f));
}

template <typename O>
__global__ void __launch_bounds__(kLnThreads) causal_conv_rows_kernel(const float* __restrict__ ext, const float* __restrict__ w, int taps, O* __restrict__ out,
                                                                      int T, int H, const int* __restrict__ seg_of_token, const int* __restrict__ seg_start,
                                                                      const int* __restrict__ seg_slot, float* __restrict__ state, size_t slot_stride) {
  // This kernel does not let its dependents start early. What follows it is a sublayer's first matrix product, which takes its tensor
  // memory before it waits; the product two kernels back (a mixer's output projection) may itself still be waiting for tensor memory
  // that an attention kernel holds, and a later, smaller request must not be served before it: the later kernel would then hold what
  // the earlier one needs while waiting for it. With no early start here, nothing after this kernel runs before the products before it
  // are done.
  ib::pdl_wait();
  const int halo = taps - 1;
  const int b = blockIdx.x;
  if (b >= T) {   // a halo row of segment s: it stays in the state when the step brought fewer than `halo` tokens
    const int hb = b - T, s = hb / halo, j = hb % halo;
    const int a = seg_start[s], n = seg_start[s + 1] - a;
    if (j < n) return;
    const float* src = ext + ((size_t)a + (size_t)s * halo + j) * H;
    float* dst = state + (size_t)seg_slot[s] * slot_stride + (size_t)(j - n) * H;
    for (int i = threadIdx.x; i < H; i += blockDim.x) dst[i] = src[i];
    return;
  }
  const int t = b, s = seg_of_token[t];
  const int end = seg_start[s + 1];
  const float* cur = ext + ((size_t)t + (size_t)(s + 1) * halo) * H;
  float* keep = end - t <= halo ? state + (size_t)seg_slot[s] * slot_stride + (size_t)(halo - (end - t)) * H : nullptr;
  for (int i = threadIdx.x; i < H; i += blockDim.x) {
    float y = 0.f;
    for (int j = 0; j < taps; j++) y = __fmaf_rn(w[(size_t)j * H + i], cur[(ptrdiff_t)(j - halo) * H + i], y);
    const float h = cur[i];
    out[(size_t)t * H + i] = ib::from_f32<O>(h + y);
    if (keep) keep[i] = h;
  }
}

__global__ void depth_average_kernel(float* __restrict__ x, const float* __restrict__ delta, int P, size_t delta_stride, const float* __restrict__ dscale,
                                     const float* __restrict__ dbias, float* __restrict__ stack, size_t layer_stride, int k, const float* __restrict__ mix, int H) {
  // (no early start of the dependents, for the reason given in causal_conv_rows_kernel: in a layer without a feed-forward this kernel
  // is what stands between a mixer's output projection and the next matrix product)
  ib::pdl_wait();
  const size_t t = blockIdx.y;
  for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < H; i += gridDim.x * blockDim.x) {
    const size_t at = t * H + i;
    float v = x[at];
    if (P > 0) {
      float a = delta[at];
      for (int p = 1; p < P; p++) a += delta[p * delta_stride + at];
      if (dbias) a += dbias[i];
      v = dscale ? __fmaf_rn(dscale[i], a, v) : v + a;
    }
    stack[(size_t)k * layer_stride + at] = v;
    float m = 0.f;
    for (int j = 0; j < k; j++) m = __fmaf_rn(mix[j], stack[(size_t)j * layer_stride + at], m);
    x[at] = __fmaf_rn(mix[k], v, m);
  }
}

// ---- the same three kernels with 16-byte accesses, for rows of a multiple of four values (every sum runs in the order of the scalar forms)
__device__ __forceinline__ float4 ld4(const float* p) { return *(const float4*)p; }
__device__ __forceinline__ void st4(float* p, float4 v) { *(float4*)p = v; }
__device__ __forceinline__ void st4(__nv_bfloat16* p, float4 v) {
  __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
  *(uint2*)p = make_uint2(*(uint32_t*)&lo, *(uint32_t*)&hi);
}
__device__ __forceinline__ float4 add4(float4 a, float4 b) { return make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w); }
__device__ __forceinline__ float4 fma4(float4 a, float4 b, float4 c) {
  return make_float4(__fmaf_rn(a.x, b.x, c.x), __fmaf_rn(a.y, b.y, c.y), __fmaf_rn(a.z, b.z, c.z), __fmaf_rn(a.w, b.w, c.w));
}

template <typename O>
__global__ void __launch_bounds__(kLnThreads) add_layernorm_vec_kernel(float* __restrict__ x, const float* __restrict__ delta, int P, size_t delta_stride,
                                                                       const float* __restrict__ dscale, const float* __restrict__ dbias,
                                                                       const float* __restrict__ w, O* __restrict__ out, const int* __restrict__ rows, int n_rows,
                                                                       int H, float eps, int write_x, float* __restrict__ x_copy, int halo,
                                                                       const int* __restrict__ seg_of_token, const int* __restrict__ seg_start,
                                                                       const int* __restrict__ seg_slot, const float* __restrict__ state, size_t slot_stride, LnExtras ex) {
  extern __shared__ __align__(16) float row[];
  __shared__ float scratch[32];
  if (ex.early) ib::pdl_launch_dependents();
  ib::pdl_wait();
  const int r = blockIdx.x;
  if (r >= n_rows) {
    const int hb = r - n_rows, s = hb / halo, j = hb % halo;
    const float* src = state + (size_t)seg_slot[s] * slot_stride + (size_t)j * H;
    O* dst = out + ((size_t)seg_start[s] + (size_t)s * halo + j) * H;
    for (int i = threadIdx.x * 4; i < H; i += blockDim.x * 4) st4(dst + i, ld4(src + i));
    return;
  }
  const int t = rows ? rows[r] : r;
  float* xr = x + (size_t)t * H;
  float sum = 0.f;
  for (int i = threadIdx.x * 4; i < H; i += blockDim.x * 4) {
    float4 v = ld4(xr + i);
    if (P > 0 || dbias) {
      float4 d = dbias ? ld4(dbias + i) : make_float4(0.f, 0.f, 0.f, 0.f);
      if (P > 0) {
        float4 a = ld4(delta + (size_t)t * H + i);
        for (int p = 1; p < P; p++) a = add4(a, ld4(delta + p * delta_stride + (size_t)t * H + i));
        d = dbias ? add4(a, d) : a;
      }
      v = fma4(dscale ? ld4(dscale + i) : make_float4(ex.mult, ex.mult, ex.mult, ex.mult), d, v);
    }
    if (ex.P2 > 0) {
      float4 a = ld4(ex.delta2 + (size_t)t * H + i);
      for (int p = 1; p < ex.P2; p++) a = add4(a, ld4(ex.delta2 + p * ex.stride2 + (size_t)t * H + i));
      v = add4(v, a);
    }
    if (write_x && (P > 0 || dbias || ex.P2 > 0)) st4(xr + i, v);
    if (x_copy) st4(x_copy + (size_t)t * H + i, v);
    st4(row + i, v);
    sum += (v.x + v.y) + (v.z + v.w);
  }
  const float mean = ib::block_sum(sum, scratch) / (float)H;
  float sq = 0.f;
  for (int i = threadIdx.x * 4; i < H; i += blockDim.x * 4) {
    const float4 v = ld4(row + i);
    const float a = v.x - mean, b = v.y - mean, c = v.z - mean, e = v.w - mean;
    sq = __fmaf_rn(e, e, __fmaf_rn(c, c, __fmaf_rn(b, b, __fmaf_rn(a, a, sq))));
  }
  const float inv = rsqrtf(ib::block_sum(sq, scratch) / (float)H + eps);
  const size_t orow = halo ? (size_t)t + (size_t)(seg_of_token[t] + 1) * halo : (size_t)r;
  O* dst = out + orow * H;
  for (int i = threadIdx.x * 4; i < H; i += blockDim.x * 4) {
    const float4 v = ld4(row + i), g = ld4(w + i), b = ex.wb ? ld4(ex.wb + i) : make_float4(0.f, 0.f, 0.f, 0.f);
    st4(dst + i, fma4(make_float4((v.x - mean) * inv, (v.y - mean) * inv, (v.z - mean) * inv, (v.w - mean) * inv), g, b));
  }
}

template <typename O>
__global__ void __launch_bounds__(kLnThreads) causal_conv_rows_vec_kernel(const float* __restrict__ ext, const float* __restrict__ w, int taps, O* __restrict__ out,
                                                                          int T, int H, const int* __restrict__ seg_of_token, const int* __restrict__ seg_start,
                                                                          const int* __restrict__ seg_slot, float* __restrict__ state, size_t slot_stride) {
  ib::pdl_wait();   // (no early start of the dependents: see causal_conv_rows_kernel)
  const int halo = taps - 1;
  const int b = blockIdx.x;
  if (b >= T) {
    const int hb = b - T, s = hb / halo, j = hb % halo;
    const int a = seg_start[s], n = seg_start[s + 1] - a;
    if (j < n) return;
    const float* src = ext + ((size_t)a + (size_t)s * halo + j) * H;
    float* dst = state + (size_t)seg_slot[s] * slot_stride + (size_t)(j - n) * H;
    for (int i = threadIdx.x * 4; i < H; i += blockDim.x * 4) st4(dst + i, ld4(src + i));
    return;
  }
  const int t = b, s = seg_of_token[t];
  const int end = seg_start[s + 1];
  const float* cur = ext + ((size_t)t + (size_t)(s + 1) * halo) * H;
  float* keep = end - t <= halo ? state + (size_t)seg_slot[s] * slot_stride + (size_t)(halo - (end - t)) * H : nullptr;
  for (int i = threadIdx.x * 4; i < H; i += blockDim.x * 4) {
    float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int j = 0; j < taps; j++) y = fma4(ld4(w + (size_t)j * H + i), ld4(cur + (ptrdiff_t)(j - halo) * H + i), y);
    const float4 h = ld4(cur + i);
    st4(out + (size_t)t * H + i, add4(h, y));
    if (keep) st4(keep + i, h);
  }
}

template <typename O, bool VEC>
__global__ void __launch_bounds__(kLnThreads) add_layernorm_conv_single_kernel(float* __restrict__ x, const float* __restrict__ delta, int P, size_t delta_stride,
                                                                               const float* __restrict__ dscale, const float* __restrict__ dbias,
                                                                               const float* __restrict__ w, float eps, float* __restrict__ x_copy,
                                                                               const float* __restrict__ cw, int taps, O* __restrict__ out, int H,
                                                                               const int* __restrict__ seg_slot, float* __restrict__ state, size_t slot_stride) {
  // Row t is segment t (one token each). As in causal_conv_rows_kernel the dependents do not start early. The row's sums are taken in the
  // order of add_layernorm's kernels (the 16-byte form where that one runs, else the scalar form), so a
  // decoded token's normed row has the same bits whichever kernel made it.
  extern __shared__ __align__(16) float row[];
  __shared__ float scratch[32];
  ib::pdl_wait();
  const int t = blockIdx.x, halo = taps - 1;
  float* xr = x + (size_t)t * H;
  auto value = [&](int i) {
    float v = xr[i];
    if (P > 0 || dbias) {
      float d = dbias ? dbias[i] : 0.f;
      if (P > 0) {
        float a = delta[(size_t)t * H + i];
        for (int p = 1; p < P; p++) a += delta[p * delta_stride + (size_t)t * H + i];
        d = dbias ? a + d : a;
      }
      v = dscale ? __fmaf_rn(dscale[i], d, v) : v + d;
      xr[i] = v;
    }
    if (x_copy) x_copy[(size_t)t * H + i] = v;
    row[i] = v;
    return v;
  };
  float* st = state + (size_t)seg_slot[t] * slot_stride;
  if constexpr (VEC) {   // 16-byte accesses; every sum in the order of add_layernorm_vec_kernel and causal_conv_rows_vec_kernel
    float sum = 0.f;
    for (int i = threadIdx.x * 4; i < H; i += blockDim.x * 4) {
      float4 v = ld4(xr + i);
      if (P > 0 || dbias) {
        float4 d = dbias ? ld4(dbias + i) : make_float4(0.f, 0.f, 0.f, 0.f);
        if (P > 0) {
          float4 a = ld4(delta + (size_t)t * H + i);
          for (int p = 1; p < P; p++) a = add4(a, ld4(delta + p * delta_stride + (size_t)t * H + i));
          d = dbias ? add4(a, d) : a;
        }
        v = dscale ? fma4(ld4(dscale + i), d, v) : add4(v, d);
        st4(xr + i, v);
      }
      if (x_copy) st4(x_copy + (size_t)t * H + i, v);
      st4(row + i, v);
      sum += (v.x + v.y) + (v.z + v.w);
    }
    const float mean = ib::block_sum(sum, scratch) / (float)H;
    float sq = 0.f;
    for (int i = threadIdx.x * 4; i < H; i += blockDim.x * 4) {
      const float4 v = ld4(row + i);
      const float a = v.x - mean, b = v.y - mean, c = v.z - mean, e = v.w - mean;
      sq = __fmaf_rn(e, e, __fmaf_rn(c, c, __fmaf_rn(b, b, __fmaf_rn(a, a, sq))));
    }
    const float inv = rsqrtf(ib::block_sum(sq, scratch) / (float)H + eps);
    for (int i = threadIdx.x * 4; i < H; i += blockDim.x * 4) {
      const float4 v = ld4(row + i), g = ld4(w + i);
      const float4 h = make_float4((v.x - mean) * inv * g.x, (v.y - mean) * inv * g.y, (v.z - mean) * inv * g.z, (v.w - mean) * inv * g.w);
      float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int j = 0; j < halo; j++) {
        const float4 old = ld4(st + (size_t)j * H + i);
        y = fma4(ld4(cw + (size_t)j * H + i), old, y);
        if (j > 0) st4(st + (size_t)(j - 1) * H + i, old);
      }
      y = fma4(ld4(cw + (size_t)halo * H + i), h, y);
      if (halo > 0) st4(st + (size_t)(halo - 1) * H + i, h);
      st4(out + (size_t)t * H + i, add4(h, y));
    }
    return;
  }
  float sum = 0.f;
  for (int i = threadIdx.x; i < H; i += blockDim.x) sum += value(i);
  const float mean = ib::block_sum(sum, scratch) / (float)H;
  float sq = 0.f;
  for (int i = threadIdx.x; i < H; i += blockDim.x) {
    const float c = row[i] - mean;
    sq = __fmaf_rn(c, c, sq);
  }
  const float inv = rsqrtf(ib::block_sum(sq, scratch) / (float)H + eps);
  for (int i = threadIdx.x; i < H; i += blockDim.x) {
    const float h = (row[i] - mean) * inv * w[i];
    float y = 0.f;
    for (int j = 0; j < halo; j++) {
      const float old = st[(size_t)j * H + i];
      y = __fmaf_rn(cw[(size_t)j * H + i], old, y);
      if (j > 0) st[(size_t)(j - 1) * H + i] = old;
    }
    y = __fmaf_rn(cw[(size_t)halo * H + i], h, y);
    if (halo > 0) st[(size_t)(halo - 1) * H + i] = h;
    out[(size_t)t * H + i] = ib::from_f32<O>(h + y);
  }
}


__global__ void depth_average_vec_kernel(float* __restrict__ x, const float* __restrict__ delta, int P, size_t delta_stride, const float* __restrict__ dscale,
                                         const float* __restrict__ dbias, float* __restrict__ stack, size_t layer_stride, int k, const float* __restrict__ mix, int H) {
  ib::pdl_wait();   // (no early start of the dependents: see depth_average_kernel)
  const size_t t = blockIdx.y;
  for (int i = (blockIdx.x * blockDim.x + threadIdx.x) * 4; i < H; i += gridDim.x * blockDim.x * 4) {
    const size_t at = t * H + i;
    float4 v = ld4(x + at);
    if (P > 0) {
      float4 a = ld4(delta + at);
      for (int p = 1; p < P; p++) a = add4(a, ld4(delta + p * delta_stride + at));
      if (dbias) a = add4(a, ld4(dbias + i));
      v = dscale ? fma4(ld4(dscale + i), a, v) : add4(v, a);
    }
    st4(stack + (size_t)k * layer_stride + at, v);
    float4 m = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int j = 0; j < k; j++) {
      const float c = mix[j];
      m = fma4(make_float4(c, c, c, c), ld4(stack + (size_t)j * layer_stride + at), m);
    }
    const float c = mix[k];
    st4(x + at, fma4(make_float4(c, c, c, c), v, m));
  }
}

// v = cap * tanh(v / cap)
__global__ void softcap_values_kernel(float* __restrict__ v, size_t n, float cap) {
  ib::pdl_launch_dependents();
  ib::pdl_wait();
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) v[i] = cap * tanhf(v[i] / cap);
}

// x[t] = layer norm of the token's row of an embedding table, float32 (one CTA a token; sums as in add_layernorm_kernel).
template <typename W>
__global__ void __launch_bounds__(kLnThreads) embed_layernorm_kernel(const W* __restrict__ table, const int* __restrict__ tokens, const float* __restrict__ w,
                                                                     const float* __restrict__ wb, float eps, float* __restrict__ x, int H, int V,
                                                                     unsigned* __restrict__ status) {
  extern __shared__ __align__(16) float row[];
  __shared__ float scratch[32];
  ib::pdl_launch_dependents();
  ib::pdl_wait();
  const int t = blockIdx.x;
  int tok = tokens[t];
  if (tok < 0 || tok >= V) {
    if (threadIdx.x == 0) atomicOr(status, IB_ERR_BAD_TOKEN);
    tok = 0;
  }
  const W* src = table + (size_t)tok * H;
  float sum = 0.f;
  for (int i = threadIdx.x; i < H; i += blockDim.x) {
    const float v = ib::to_f32<W>(src[i]);
    row[i] = v;
    sum += v;
  }
  const float mean = ib::block_sum(sum, scratch) / (float)H;
  float sq = 0.f;
  for (int i = threadIdx.x; i < H; i += blockDim.x) {
    const float c = row[i] - mean;
    sq = __fmaf_rn(c, c, sq);
  }
  const float inv = rsqrtf(ib::block_sum(sq, scratch) / (float)H + eps);
  for (int i = threadIdx.x; i < H; i += blockDim.x) x[(size_t)t * H + i] = __fmaf_rn((row[i] - mean) * inv, w[i], wb ? wb[i] : 0.f);
}

// out[m][t] = h_t + (h_(t-1) - h_t) * mu[m] per channel for M mixes. The row before a segment's first row is the request's state, which
// becomes the segment's last row: the CTA that reads a request's old state (the first row's) is the one that writes the new one.
template <typename O>
__global__ void __launch_bounds__(kLnThreads) shift_mixes_kernel(const float* __restrict__ h, const float* __restrict__ mu, int M, float* __restrict__ state, size_t slot_stride,
                                                                 const int* __restrict__ seg_of_token, const int* __restrict__ seg_start,
                                                                 const int* __restrict__ seg_slot, O* __restrict__ out, int T, int H) {
  ib::pdl_launch_dependents();
  ib::pdl_wait();
  const int t = blockIdx.x;
  const int s = seg_of_token[t], t0 = seg_start[s];
  const bool first = t == t0;
  float* st = state + (size_t)seg_slot[s] * slot_stride;
  const float* prev = first ? st : h + (size_t)(t - 1) * H;
  const float* last = h + (size_t)(seg_start[s + 1] - 1) * H;
  const float* cur = h + (size_t)t * H;
  for (int i = blockIdx.y * blockDim.x + threadIdx.x; i < H; i += gridDim.y * blockDim.x) {
    const float v = cur[i], d = prev[i] - v;
    for (int m = 0; m < M; m++) out[((size_t)m * T + t) * H + i] = ib::from_f32<O>(__fmaf_rn(d, mu[(size_t)m * H + i], v));
    if (first) st[i] = last[i];
  }
}

// The residual add, the layer norm and the mixes in one kernel for a step whose row t is segment t (one token each); sums in the order of
// add_layernorm's kernels, so a decoded token's normed row has the same bits whichever kernel made it.
template <typename O, bool VEC>
__global__ void __launch_bounds__(kLnThreads) add_layernorm_mixes_single_kernel(float* __restrict__ x, const float* __restrict__ delta, int P, size_t delta_stride,
                                                                                const float* __restrict__ w, float eps, const float* __restrict__ mu, int M,
                                                                                O* __restrict__ out, int T, int H, const int* __restrict__ seg_slot,
                                                                                float* __restrict__ state, size_t slot_stride, LnExtras ex) {
  extern __shared__ __align__(16) float row[];
  __shared__ float scratch[32];
  if (ex.early) ib::pdl_launch_dependents();
  ib::pdl_wait();
  const int t = blockIdx.x;
  float* xr = x + (size_t)t * H;
  float* st = state + (size_t)seg_slot[t] * slot_stride;
  constexpr int N = VEC ? 4 : 1;
  float sum = 0.f;
  for (int i = threadIdx.x * N; i < H; i += blockDim.x * N) {
    if constexpr (VEC) {
      float4 v = ld4(xr + i);
      if (P > 0) {
        float4 a = ld4(delta + (size_t)t * H + i);
        for (int p = 1; p < P; p++) a = add4(a, ld4(delta + p * delta_stride + (size_t)t * H + i));
        v = fma4(make_float4(ex.mult, ex.mult, ex.mult, ex.mult), a, v);
        st4(xr + i, v);
      }
      st4(row + i, v);
      sum += (v.x + v.y) + (v.z + v.w);
    } else {
      float v = xr[i];
      if (P > 0) {
        float a = delta[(size_t)t * H + i];
        for (int p = 1; p < P; p++) a += delta[p * delta_stride + (size_t)t * H + i];
        v = __fmaf_rn(ex.mult, a, v);
        xr[i] = v;
      }
      row[i] = v;
      sum += v;
    }
  }
  const float mean = ib::block_sum(sum, scratch) / (float)H;
  float sq = 0.f;
  for (int i = threadIdx.x * N; i < H; i += blockDim.x * N) {
    if constexpr (VEC) {
      const float4 v = ld4(row + i);
      const float a = v.x - mean, b = v.y - mean, c = v.z - mean, e = v.w - mean;
      sq = __fmaf_rn(e, e, __fmaf_rn(c, c, __fmaf_rn(b, b, __fmaf_rn(a, a, sq))));
    } else {
      const float c = row[i] - mean;
      sq = __fmaf_rn(c, c, sq);
    }
  }
  const float inv = rsqrtf(ib::block_sum(sq, scratch) / (float)H + eps);
  for (int i = threadIdx.x * N; i < H; i += blockDim.x * N) {
    if constexpr (VEC) {
      const float4 v = ld4(row + i), b = ex.wb ? ld4(ex.wb + i) : make_float4(0.f, 0.f, 0.f, 0.f), old = ld4(st + i);
      const float4 h = fma4(make_float4((v.x - mean) * inv, (v.y - mean) * inv, (v.z - mean) * inv, (v.w - mean) * inv), ld4(w + i), b);
      const float4 d = make_float4(old.x - h.x, old.y - h.y, old.z - h.z, old.w - h.w);
      st4(st + i, h);
      for (int m = 0; m < M; m++) st4(out + ((size_t)m * T + t) * H + i, fma4(d, ld4(mu + (size_t)m * H + i), h));
    } else {
      const float h = __fmaf_rn((row[i] - mean) * inv, w[i], ex.wb ? ex.wb[i] : 0.f), d = st[i] - h;
      st[i] = h;
      for (int m = 0; m < M; m++) out[((size_t)m * T + t) * H + i] = ib::from_f32<O>(__fmaf_rn(d, mu[(size_t)m * H + i], h));
    }
  }
}

__global__ void scale_values_kernel(float* __restrict__ v, size_t n, float s) {
  ib::pdl_launch_dependents();
  ib::pdl_wait();
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x) v[i] *= s;
}

}  // namespace

extern "C" int ib_add_layernorm(float* x, const float* delta, int P, long long delta_stride, const float* dscale, const float* dbias, const float* w, void* out,
                                int out_dtype, const int* rows, int n_rows, int H, float eps, int write_x, float* x_copy, int halo, const int* seg_of_token,
                                const int* seg_start, const int* seg_slot, int n_segments, const float* state, long long slot_stride, const float* wb,
                                float mult, int early, const float* delta2, int P2, long long stride2, cudaStream_t stream) {
  // delta2, P2, stride2: a second contribution (see LnExtras), P2 = 0 for none
  // wb: the norm's bias per channel, or null; mult: factor on the contribution where dscale is null; early: see LnExtras
  if (n_rows == 0) return 0;
  const LnExtras ex = {wb, mult, early, delta2, P2, (size_t)stride2};
  IB_CHECK_ARG(P2 >= 0 && (P2 == 0 || delta2), "add_layernorm: a second contribution of %d partial sums is missing", P2);
  IB_CHECK_ARG(n_rows > 0 && H > 0 && P >= 0 && halo >= 0, "add_layernorm: bad sizes rows=%d H=%d P=%d halo=%d", n_rows, H, P, halo);
  IB_CHECK_ARG(!(halo && rows), "add_layernorm: gathered rows have no layout for a convolution");
  IB_CHECK_ARG(!halo || (seg_of_token && seg_start && seg_slot && state && n_segments > 0), "add_layernorm: the convolution's layout needs the step's segments and the state");
  const size_t smem = (size_t)H * sizeof(float);
  IB_CHECK_ARG(smem <= 200 * 1024, "add_layernorm: rows of %d values do not fit in shared memory", H);
  const unsigned grid = (unsigned)n_rows + (unsigned)(halo * (halo ? n_segments : 0));
  auto go = [&](auto kernel, auto* o) {
    if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    ib::launch(kernel, grid, kLnThreads, smem, stream, x, delta, P, (size_t)delta_stride, dscale, dbias, w, o, rows, n_rows, H, eps, write_x, x_copy, halo, seg_of_token,
               seg_start, seg_slot, state, (size_t)slot_stride, ex);
  };
  auto al = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
  const bool vec = H % 4 == 0 && al(wb) && al(x) && al(delta) && delta_stride % 4 == 0 && al(dscale) && al(dbias) && al(w) && al(out) && al(x_copy) && al(state) && slot_stride % 4 == 0 &&
                   al(delta2) && stride2 % 4 == 0;
  if (out_dtype != IB_F32 && out_dtype != IB_BF16) return ib_set_error("add_layernorm: unknown output dtype %d", out_dtype);
  if (vec && out_dtype == IB_F32) go(add_layernorm_vec_kernel<float>, (float*)out);
  else if (vec) go(add_layernorm_vec_kernel<__nv_bfloat16>, (__nv_bfloat16*)out);
  else if (out_dtype == IB_F32) go(add_layernorm_kernel<float>, (float*)out);
  else go(add_layernorm_kernel<__nv_bfloat16>, (__nv_bfloat16*)out);
  IB_CHECK_LAUNCH("add_layernorm");
  return 0;
}

extern "C" int ib_add_layernorm_conv_single(float* x, const float* delta, int P, long long delta_stride, const float* dscale, const float* dbias, const float* w,
                                            float eps, float* x_copy, const float* cw, int taps, void* out, int out_dtype, int T, int H, const int* seg_slot, float* state,
                                            long long slot_stride, cudaStream_t stream) {
  if (T == 0) return 0;
  IB_CHECK_ARG(T > 0 && H > 0 && P >= 0 && taps >= 1, "add_layernorm_conv_single: bad sizes T=%d H=%d P=%d taps=%d", T, H, P, taps);
  const size_t smem = (size_t)H * sizeof(float);
  IB_CHECK_ARG(smem <= 200 * 1024, "add_layernorm_conv_single: rows of %d values do not fit in shared memory", H);
  auto go = [&](auto kernel, auto* o) {
    if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    ib::launch(kernel, (unsigned)T, kLnThreads, smem, stream, x, delta, P, (size_t)delta_stride, dscale, dbias, w, eps, x_copy, cw, taps, o, H, seg_slot, state,
               (size_t)slot_stride);
  };
  auto al = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
  const bool vec = H % 4 == 0 && al(x) && al(delta) && delta_stride % 4 == 0 && al(dscale) && al(dbias) && al(w) && al(out) && al(x_copy) && al(state) && slot_stride % 4 == 0 &&
                   al(cw);
  if (out_dtype != IB_F32 && out_dtype != IB_BF16) return ib_set_error("add_layernorm_conv_single: unknown output dtype %d", out_dtype);
  if (vec && out_dtype == IB_F32) go(add_layernorm_conv_single_kernel<float, true>, (float*)out);
  else if (vec) go(add_layernorm_conv_single_kernel<__nv_bfloat16, true>, (__nv_bfloat16*)out);
  else if (out_dtype == IB_F32) go(add_layernorm_conv_single_kernel<float, false>, (float*)out);
  else go(add_layernorm_conv_single_kernel<__nv_bfloat16, false>, (__nv_bfloat16*)out);
  IB_CHECK_LAUNCH("add_layernorm_conv_single");
  return 0;
}

extern "C" int ib_causal_conv_rows(const float* ext, const float* w, int taps, void* out, int out_dtype, int T, int H, const int* seg_of_token, const int* seg_start,
                                   const int* seg_slot, int n_segments, float* state, long long slot_stride, cudaStream_t stream) {
  if (T == 0) return 0;
  IB_CHECK_ARG(T > 0 && H > 0 && taps >= 1 && n_segments > 0, "causal_conv_rows: bad sizes T=%d H=%d taps=%d segments=%d", T, H, taps, n_segments);
  const unsigned grid = (unsigned)T + (unsigned)((taps - 1) * n_segments);
  const bool vec = H % 4 == 0 && ((uintptr_t)ext & 15) == 0 && ((uintptr_t)out & 15) == 0 && ((uintptr_t)state & 15) == 0 && slot_stride % 4 == 0 &&
                   ((uintptr_t)w & 15) == 0;
  if (out_dtype != IB_F32 && out_dtype != IB_BF16) return ib_set_error("causal_conv_rows: unknown output dtype %d", out_dtype);
  auto go = [&](auto kernel, auto* o) { ib::launch(kernel, grid, kLnThreads, 0, stream, ext, w, taps, o, T, H, seg_of_token, seg_start, seg_slot, state, (size_t)slot_stride); };
  if (vec && out_dtype == IB_F32) go(causal_conv_rows_vec_kernel<float>, (float*)out);
  else if (vec) go(causal_conv_rows_vec_kernel<__nv_bfloat16>, (__nv_bfloat16*)out);
  else if (out_dtype == IB_F32) go(causal_conv_rows_kernel<float>, (float*)out);
  else go(causal_conv_rows_kernel<__nv_bfloat16>, (__nv_bfloat16*)out);
  IB_CHECK_LAUNCH("causal_conv_rows");
  return 0;
}

extern "C" int ib_depth_average(float* x, const float* delta, int P, long long delta_stride, const float* dscale, const float* dbias, float* stack, long long layer_stride, int k,
                                const float* mix, int T, int H, cudaStream_t stream) {
  if (T == 0) return 0;
  IB_CHECK_ARG(T > 0 && H > 0 && k >= 1 && P >= 0, "depth_average: bad sizes T=%d H=%d k=%d P=%d", T, H, k, P);
  IB_CHECK_ARG(T <= 65535, "depth_average: T=%d rows exceed the grid limit 65535", T);
  const bool vec = H % 4 == 0 && ((uintptr_t)x & 15) == 0 && ((uintptr_t)delta & 15) == 0 && delta_stride % 4 == 0 && ((uintptr_t)dscale & 15) == 0 &&
                   ((uintptr_t)dbias & 15) == 0 && ((uintptr_t)stack & 15) == 0 && layer_stride % 4 == 0;
  if (vec)
    ib::launch(depth_average_vec_kernel, dim3(min((H / 4 + 255) / 256, 32), T), 256, 0, stream, x, delta, P, (size_t)delta_stride, dscale, dbias, stack, (size_t)layer_stride, k,
               mix, H);
  else
    ib::launch(depth_average_kernel, dim3(min((H + 255) / 256, 32), T), 256, 0, stream, x, delta, P, (size_t)delta_stride, dscale, dbias, stack, (size_t)layer_stride, k, mix, H);
  IB_CHECK_LAUNCH("depth_average");
  return 0;
}

extern "C" int ib_scale_values(float* v, long long n, float s, cudaStream_t stream) {
  if (n <= 0) return 0;
  ib::launch(scale_values_kernel, (unsigned)min((long long)1024, (n + 255) / 256), 256, 0, stream, v, (size_t)n, s);
  IB_CHECK_LAUNCH("scale_values");
  return 0;
}

extern "C" int ib_softcap_values(float* v, long long n, float cap, cudaStream_t stream) {
  if (n <= 0) return 0;
  IB_CHECK_ARG(cap > 0.f, "softcap_values: the cap %g must be positive", (double)cap);
  ib::launch(softcap_values_kernel, (unsigned)min((long long)1024, (n + 255) / 256), 256, 0, stream, v, (size_t)n, cap);
  IB_CHECK_LAUNCH("softcap_values");
  return 0;
}

extern "C" int ib_embed_layernorm(const void* table, int dtype, const int* tokens, const float* w, const float* wb, float eps, float* x, int T, int H, int V, unsigned* status,
                                  cudaStream_t stream) {
  if (T == 0) return 0;
  const size_t smem = (size_t)H * sizeof(float);
  IB_CHECK_ARG(T > 0 && H > 0 && V > 0 && smem <= 200 * 1024, "embed_layernorm: bad sizes T=%d H=%d V=%d", T, H, V);
  auto go = [&](auto kernel, auto* tab) {
    if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    ib::launch(kernel, (unsigned)T, kLnThreads, smem, stream, tab, tokens, w, wb, eps, x, H, V, status);
  };
  if (dtype == IB_F32) go(embed_layernorm_kernel<float>, (const float*)table);
  else if (dtype == IB_BF16) go(embed_layernorm_kernel<__nv_bfloat16>, (const __nv_bfloat16*)table);
  else return ib_set_error("embed_layernorm: unknown table dtype %d", dtype);
  IB_CHECK_LAUNCH("embed_layernorm");
  return 0;
}

// mu float32 [M][H], out [M][T][H].
extern "C" int ib_shift_mixes(const float* h, const float* mu, int M, float* state, long long slot_stride, const int* seg_of_token, const int* seg_start,
                              const int* seg_slot, void* out, int out_dtype, int T, int H, cudaStream_t stream) {
  if (T == 0) return 0;
  IB_CHECK_ARG(T > 0 && H > 0 && M > 0, "shift_mixes: bad sizes T=%d H=%d mixes=%d", T, H, M);
  const dim3 grid((unsigned)T, (unsigned)min((H + kLnThreads - 1) / kLnThreads, 64));
  if (out_dtype == IB_F32) ib::launch(shift_mixes_kernel<float>, grid, kLnThreads, 0, stream, h, mu, M, state, (size_t)slot_stride, seg_of_token, seg_start, seg_slot, (float*)out, T, H);
  else if (out_dtype == IB_BF16)
    ib::launch(shift_mixes_kernel<__nv_bfloat16>, grid, kLnThreads, 0, stream, h, mu, M, state, (size_t)slot_stride, seg_of_token, seg_start, seg_slot, (__nv_bfloat16*)out, T, H);
  else return ib_set_error("shift_mixes: unknown output dtype %d", out_dtype);
  IB_CHECK_LAUNCH("shift_mixes");
  return 0;
}

extern "C" int ib_add_layernorm_mixes_single(float* x, const float* delta, int P, long long delta_stride, float mult, const float* w, const float* wb, float eps,
                                             const float* mu, int M, void* out, int out_dtype, int T, int H, const int* seg_slot, float* state, long long slot_stride,
                                             int early, cudaStream_t stream) {
  if (T == 0) return 0;
  const size_t smem = (size_t)H * sizeof(float);
  IB_CHECK_ARG(T > 0 && H > 0 && P >= 0 && M > 0 && smem <= 200 * 1024, "add_layernorm_mixes_single: bad sizes T=%d H=%d P=%d mixes=%d", T, H, P, M);
  const LnExtras ex = {wb, mult, early, nullptr, 0, 0};
  auto go = [&](auto kernel, auto* o) {
    if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    ib::launch(kernel, (unsigned)T, kLnThreads, smem, stream, x, delta, P, (size_t)delta_stride, w, eps, mu, M, o, T, H, seg_slot, state, (size_t)slot_stride, ex);
  };
  auto al = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
  const bool vec = H % 4 == 0 && al(x) && al(delta) && delta_stride % 4 == 0 && al(w) && al(wb) && al(mu) && al(out) && al(state) && slot_stride % 4 == 0;
  if (out_dtype != IB_F32 && out_dtype != IB_BF16) return ib_set_error("add_layernorm_mixes_single: unknown output dtype %d", out_dtype);
  if (vec && out_dtype == IB_F32) go(add_layernorm_mixes_single_kernel<float, true>, (float*)out);
  else if (vec) go(add_layernorm_mixes_single_kernel<__nv_bfloat16, true>, (__nv_bfloat16*)out);
  else if (out_dtype == IB_F32) go(add_layernorm_mixes_single_kernel<float, false>, (float*)out);
  else go(add_layernorm_mixes_single_kernel<__nv_bfloat16, false>, (__nv_bfloat16*)out);
  IB_CHECK_LAUNCH("add_layernorm_mixes_single");
  return 0;
}
