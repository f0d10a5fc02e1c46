// Routed feed-forward (mixture of experts): the router's choice, the regrouping of the step's tokens by expert,
// the experts' matrix products on the regrouped rows, and the weighted sum back into token order.
//
//  * moe_route: per token, s = softmax(router logits) over all experts in float32 (or, with `score` = 1, s = sigmoid of each logit
//    on its own); experts lie in `n_groups` equal
//    groups of neighbours, a group's score is its largest s (or the sum of its few largest), only the `keep` best groups stay eligible; the `top`
//    eligible experts with the largest s are chosen (ties: the lower index), each weighted s * route_scale, or
//    s / (sum of the chosen s) * route_scale with `renorm`. With a correction, groups and experts are chosen by s + correction[e]
//    and weighted by s alone. With `score` = 2 the experts are chosen by their logits (plus a bias each) and weighted by the softmax over
//    the chosen logits alone.
//  * moe_sort: counts the (token, choice) pairs of every expert, lays the experts' rows out one after the other
//    (offsets[e] .. offsets[e + 1]) and gives every pair a row of its expert's range; tile_start[e] is the first tile of expert e.
//  * moe_route_sort: both in one kernel for a step of few tokens. Experts that every token uses (a shared expert cut into blocks of the routed
//    experts' inner size) may stand behind the routed ones as further choices.
//  * gemm_grouped: out[r] = W[e(r)] x[src(r)] for every regrouped row r: a 64 x 64 tile belongs to one expert; float32
//    FMA chains per output (a row's result does not depend on its place among the rows). With `gated`, W holds gate
//    rows then up rows and the output is silu(gate) * up. With `relu2` the output is the square of max(product, 0).
//  * moe_combine: out[t] = sum_p base[p][t] + sum_k weight[t][k] * y[row(t, k)], in the order of the choices (without weights: the plain sum).
//  * scatter_scaled_rows: out[row(t, k)] = weight[t][k] * x[t]: the step's rows in the experts' order with the router's weight on the
//    expert's input (an expert is not linear, so a weight on its input is not one on its output).
#include <type_traits>

#include "common.cuh"

namespace {

constexpr int kRouteWarps = 4;

// (value, index) argmax over a warp: larger value wins, then the lower index.
__device__ __forceinline__ void warp_argmax(float& v, int& i) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float ov = __shfl_xor_sync(0xffffffffu, v, o);
    const int oi = __shfl_xor_sync(0xffffffffu, i, o);
    if (ov > v || (ov == v && oi < i)) v = ov, i = oi;
  }
}

struct RouteArgs {
  const float* logits;       // float32 partial sums [P][T][row], the experts' are a row's first E
  int P;
  size_t stride_p;
  int T, E, row, n_groups, keep, top;
  float route_scale;
  int renorm, score;
  const float* correction;   // a number per expert added to its score for the choice (of groups and of experts) and left out of the weights, or null
  const float* logit_bias;   // float32 [E] added to the logits, or null
  int group_top;             // a group's score is the sum of its `group_top` largest choice scores (1: its largest)
  int always;                // experts E .. E + always - 1 that every token uses as well: the last entries of its row of choices, weighted by
  int gate_col;              //   the sigmoid of its logit in this column (-1: one)
  int* idx_out;              // [T][top + always]
  float* wt_out;
  __device__ __forceinline__ int row_out() const { return top + always; }
};

// One warp routes token t; `s` holds 2 E + n_groups floats of shared memory of its own. Choice scores may be negative: what cannot be
// chosen counts as minus infinity.
__device__ __forceinline__ void route_token(const RouteArgs& a, int t, float* s, int lane) {
  const int E = a.E;
  float* c = s + E;
  float* g = c + E;
  float mx = -INFINITY;
  for (int e = lane; e < E; e += 32) {
    float z = a.logits[(size_t)t * a.row + e];
    for (int p = 1; p < a.P; p++) z += a.logits[p * a.stride_p + (size_t)t * a.row + e];
    if (a.logit_bias) z += a.logit_bias[e];
    s[e] = z;
    mx = fmaxf(mx, z);
  }
  if (a.score == 1) {   // every expert's own sigmoid
    for (int e = lane; e < E; e += 32) s[e] = 1.f / (1.f + expf(-s[e]));
  } else if (a.score == 0) {
    mx = ib::warp_max(mx);
    float sum = 0.f;
    for (int e = lane; e < E; e += 32) {
      const float v = expf(s[e] - mx);
      s[e] = v;
      sum += v;
    }
    sum = ib::warp_sum(sum);
    const float inv = 1.f / sum;
    for (int e = lane; e < E; e += 32) s[e] *= inv;
  }
  for (int e = lane; e < E; e += 32) c[e] = a.correction ? s[e] + a.correction[e] : s[e];
  __syncwarp();
  if (a.n_groups > 1 && a.keep < a.n_groups) {
    const int per = E / a.n_groups;
    for (int k = lane; k < a.n_groups; k += 32) {
      // the group's `group_top` largest choice scores, found one after the other (ties: the lower index first, which changes no sum)
      float total = 0.f;
      int taken[4] = {-1, -1, -1, -1};
      for (int r = 0; r < a.group_top && r < per; r++) {
        float b = -INFINITY;
        int bi = -1;
        for (int e = k * per; e < (k + 1) * per; e++) {
          if (e == taken[0] || e == taken[1] || e == taken[2] || e == taken[3]) continue;
          if (bi < 0 || c[e] > b) b = c[e], bi = e;
        }
        taken[r] = bi;
        total += b;
      }
      g[k] = total;
    }
    __syncwarp();
    for (int r = 0; r < a.keep; r++) {   // the best groups, one after the other; a kept group is marked in `g` by NaN
      float bv = -INFINITY;
      int bi = 0x7fffffff;
      for (int k = lane; k < a.n_groups; k += 32)
        if (g[k] == g[k] && (bi == 0x7fffffff || g[k] > bv)) bv = g[k], bi = k;
      warp_argmax(bv, bi);
      if (lane == 0 && bi < a.n_groups) g[bi] = __int_as_float(0x7fc00000);
      __syncwarp();
    }
    for (int e = lane; e < E; e += 32)
      if (g[e / per] == g[e / per]) c[e] = -INFINITY;   // its group was not kept
    __syncwarp();
  }
  float chosen_sum = 0.f, chosen_max = 0.f;
  for (int r = 0; r < a.top; r++) {
    float bv = -INFINITY;
    int bi = 0x7fffffff;
    for (int e = lane; e < E; e += 32)
      if (c[e] > bv) bv = c[e], bi = e;
    warp_argmax(bv, bi);
    float w = 0.f;
    if (bi >= E) {   // fewer experts that can be chosen than choices: weight zero
      bi = 0;
    } else if (a.score == 2) {   // the softmax over the chosen logits: the first choice has the largest
      if (r == 0) chosen_max = s[bi];
      w = expf(s[bi] - chosen_max);
    } else {
      w = s[bi];
    }
    if (lane == 0) {
      a.idx_out[(size_t)t * a.row_out() + r] = bi;
      a.wt_out[(size_t)t * a.row_out() + r] = w;
      c[bi] = -INFINITY;
    }
    chosen_sum += w;
    __syncwarp();
  }
  if (lane == 0) {
    const float f = a.renorm ? a.route_scale / (chosen_sum + 1e-20f) : a.route_scale;
    for (int r = 0; r < a.top; r++) a.wt_out[(size_t)t * a.row_out() + r] *= f;
  }
  for (int r = lane; r < a.always; r += 32) {
    float w = 1.f;
    if (a.gate_col >= 0) {
      const float* src = a.logits + (size_t)t * a.row + a.gate_col;
      float z = src[0];
      for (int p = 1; p < a.P; p++) z += src[p * a.stride_p];
      w = 1.f / (1.f + expf(-z));
    }
    a.idx_out[(size_t)t * a.row_out() + a.top + r] = E + r;
    a.wt_out[(size_t)t * a.row_out() + a.top + r] = w;
  }
}

__global__ void moe_route_kernel(RouteArgs a) {
  extern __shared__ float sm[];   // per warp: E scores, E choice scores, then n_groups group scores
  ib::pdl_launch_dependents();
  ib::pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x * kRouteWarps + warp;
  if (t >= a.T) return;
  route_token(a, t, sm + (size_t)warp * (2 * a.E + a.n_groups), lane);
}

constexpr int SM_ = 64;   // rows of a tile of the grouped product

// The regrouping by one CTA; `si` holds 3 E + 1 ints of shared memory.
__device__ __forceinline__ void sort_pairs(const int* idx, int R, int top, int E, int tile_rows, int* __restrict__ offsets, int* __restrict__ tile_start,
                                           int* __restrict__ row_of_pair, int* __restrict__ token_of_row, int* si) {
  int* counts = si;   // counts[E], fill[E], start[E + 1]
  int* fill = si + E;
  int* start = si + 2 * E;
  for (int e = threadIdx.x; e < E; e += blockDim.x) counts[e] = 0, fill[e] = 0;
  __syncthreads();
  for (int r = threadIdx.x; r < R; r += blockDim.x) {
    const int e = idx[r];
    if (e >= 0 && e < E) atomicAdd(&counts[e], 1);
  }
  __syncthreads();
  if (threadIdx.x == 0) {
    int a = 0, tl = 0;
    for (int e = 0; e < E; e++) {
      start[e] = a;
      offsets[e] = a;
      tile_start[e] = tl;
      a += counts[e];
      tl += (counts[e] + tile_rows - 1) / tile_rows;
    }
    start[E] = a;
    offsets[E] = a;
    tile_start[E] = tl;
  }
  __syncthreads();
  // A pair takes the next free row of its expert's range. Which pair gets which row depends on the order threads run in; no result
  // does: every regrouped row is multiplied on its own, and the weighted sum goes back through row_of_pair in the order of the choices.
  for (int r = threadIdx.x; r < R; r += blockDim.x) {
    const int e = idx[r];
    if (e < 0 || e >= E) continue;
    const int row = start[e] + atomicAdd(&fill[e], 1);
    row_of_pair[r] = row;
    token_of_row[row] = r / top;
  }
}

__global__ void __launch_bounds__(1024) moe_sort_kernel(const int* __restrict__ idx, int R, int top, int E, int tile_rows, int* __restrict__ offsets,
                                                        int* __restrict__ tile_start, int* __restrict__ row_of_pair, int* __restrict__ token_of_row) {
  extern __shared__ int si[];
  ib::pdl_launch_dependents();
  ib::pdl_wait();
  sort_pairs(idx, R, top, E, tile_rows, offsets, tile_start, row_of_pair, token_of_row, si);
}

// Both for a step of few tokens: one CTA routes every token (a warp each, in rounds) and regroups the pairs.
__global__ void __launch_bounds__(1024) moe_route_sort_kernel(RouteArgs a, int tile_rows, int* __restrict__ offsets, int* __restrict__ tile_start,
                                                              int* __restrict__ row_of_pair, int* __restrict__ token_of_row) {
  extern __shared__ float sm[];
  ib::pdl_launch_dependents();
  ib::pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
  const int per = 2 * a.E + a.n_groups, E = a.E + a.always;
  for (int t = warp; t < a.T; t += warps) {
    route_token(a, t, sm + (size_t)warp * per, lane);
    __syncwarp();
  }
  __syncthreads();
  // the choices were written by this CTA: they are read as ordinary memory, not through a read-only path
  sort_pairs(a.idx_out, a.T * a.row_out(), a.row_out(), E, tile_rows, offsets, tile_start, row_of_pair, token_of_row, (int*)(sm + (size_t)warps * per));
}

template <typename X, typename W, typename O>
__global__ void __launch_bounds__(256) gemm_grouped_kernel(const X* __restrict__ x, const int* __restrict__ src_row, const W* __restrict__ w,
                                                           O* __restrict__ out, const int* __restrict__ offsets, const int* __restrict__ tile_start, int E,
                                                           int N, int K, int act, const float* __restrict__ limits, float slope) {
  // act: 0 the product, 1 silu(gate) * up (w holds gate rows, then up rows), 2 the square of max(product, 0), 3 as 1 with clamped halves
  // (limits: one an expert, slope: the sigmoid's)
  const bool gated = act == 1 || act == 3;
  constexpr int BK = 16;
  __shared__ float xs[BK][SM_ + 1];
  __shared__ float ws[BK][64 + 1];
  __shared__ float us[BK][64 + 1];
  __shared__ int s_e, s_r0, s_r1;
  ib::pdl_launch_dependents();
  ib::pdl_wait();
  if (threadIdx.x == 0) {
    const int b = blockIdx.y;
    int e = -1;
    if (b < tile_start[E]) {
      int lo = 0, hi = E;   // the last e with tile_start[e] <= b
      while (hi - lo > 1) {
        const int mid = (lo + hi) >> 1;
        if (tile_start[mid] <= b) lo = mid;
        else hi = mid;
      }
      e = lo;
    }
    s_e = e;
    if (e >= 0) {
      s_r0 = offsets[e] + (b - tile_start[e]) * SM_;
      s_r1 = offsets[e + 1];
    }
  }
  __syncthreads();
  const int e = s_e;
  if (e < 0) return;
  const int r0 = s_r0, r1 = s_r1, n0 = blockIdx.x * 64;
  const int rows_w = gated ? 2 * N : N;
  const W* we = w + (size_t)e * rows_w * K;
  const int tid = threadIdx.x, ty = tid / 16, tx = tid % 16;
  float acc[4][4], acu[4][4];
#pragma unroll
  for (int i = 0; i < 4; i++)
#pragma unroll
    for (int j = 0; j < 4; j++) acc[i][j] = 0.f, acu[i][j] = 0.f;
  for (int k0 = 0; k0 < K; k0 += BK) {
#pragma unroll
    for (int q = 0; q < 4; q++) {
      const int idx = tid + q * 256, r = idx / BK, kk = idx % BK, k = k0 + kk;
      const int row = r0 + r, n = n0 + r;
      float xv = 0.f;
      if (row < r1 && k < K) {
        const int src = src_row ? src_row[row] : row;
        xv = ib::to_f32<X>(x[(size_t)src * K + k]);
      }
      xs[kk][r] = xv;
      ws[kk][r] = (n < N && k < K) ? ib::to_f32<W>(we[(size_t)n * K + k]) : 0.f;
      if (gated) us[kk][r] = (n < N && k < K) ? ib::to_f32<W>(we[(size_t)(N + n) * K + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < BK; kk++) {
      float a[4], c[4], u[4];
#pragma unroll
      for (int i = 0; i < 4; i++) a[i] = xs[kk][ty * 4 + i];
#pragma unroll
      for (int j = 0; j < 4; j++) c[j] = ws[kk][tx * 4 + j];
#pragma unroll
      for (int i = 0; i < 4; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) acc[i][j] = fmaf(a[i], c[j], acc[i][j]);
      if (gated) {
#pragma unroll
        for (int j = 0; j < 4; j++) u[j] = us[kk][tx * 4 + j];
#pragma unroll
        for (int i = 0; i < 4; i++)
#pragma unroll
          for (int j = 0; j < 4; j++) acu[i][j] = fmaf(a[i], u[j], acu[i][j]);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; i++) {
    const int row = r0 + ty * 4 + i;
    if (row >= r1) continue;
#pragma unroll
    for (int j = 0; j < 4; j++) {
      const int n = n0 + tx * 4 + j;
      if (n >= N) continue;
      float v = acc[i][j];
      if (gated) {
        v = act == 3 ? ib::clamped_glu<false>(v, acu[i][j], limits[e], slope) : (v / (1.f + expf(-v))) * acu[i][j];
      } else if (act == 2) {
        v = ib::relu2(v);
      }
      out[(size_t)row * N + n] = ib::from_f32<O>(v);
    }
  }
}

// out[r] = x[src_row[r]]: the step's rows in the experts' order (16 bytes a thread; K a multiple of 8).
__global__ void gather_rows_kernel(const uint4* __restrict__ x, const int* __restrict__ src_row, uint4* __restrict__ out, int chunks) {
  ib::pdl_launch_dependents();
  ib::pdl_wait();
  const int r = blockIdx.x;
  const uint4* src = x + (size_t)src_row[r] * chunks;
  for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < chunks; c += gridDim.y * blockDim.x) out[(size_t)r * chunks + c] = src[c];
}

// VEC: 16-byte accesses (H a multiple of 4); an output's sum runs in the same order in both forms.
template <bool VEC>
__global__ void moe_combine_kernel(const float* __restrict__ y, const int* __restrict__ row_of_pair, const float* __restrict__ wt, int top,
                                   const float* __restrict__ base, int P, size_t stride_p, float* __restrict__ out, int H, const float* __restrict__ gate,
                                   int gate_P, size_t gate_stride, int gate_row) {
  // gate: float32 partial sums [gate_P][T][gate_row] offset to one column, or null: `base` counts times the sigmoid of the token's entry there
  ib::pdl_launch_dependents();
  ib::pdl_wait();
  const int t = blockIdx.y;
  float f = 1.f;
  if (gate) {
    const float* gr = gate + (size_t)t * gate_row;
    float z = gr[0];
    for (int p = 1; p < gate_P; p++) z += gr[p * gate_stride];
    f = 1.f / (1.f + expf(-z));
  }
  if constexpr (VEC) {
    for (int i = (blockIdx.x * blockDim.x + threadIdx.x) * 4; i < H; i += gridDim.x * blockDim.x * 4) {
      float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int p = 0; p < P; p++) {
        const float4 b = *(const float4*)(base + p * stride_p + (size_t)t * H + i);
        a.x += b.x, a.y += b.y, a.z += b.z, a.w += b.w;
      }
      if (gate) a.x *= f, a.y *= f, a.z *= f, a.w *= f;
      for (int k0 = 0; k0 < top; k0 += 4) {   // four choices' rows are requested before the first is used
        float4 v[4];
        float c[4];
#pragma unroll
        for (int u = 0; u < 4; u++) {
          if (k0 + u >= top) continue;
          const size_t at = (size_t)t * top + k0 + u;
          c[u] = wt ? wt[at] : 1.f;
          v[u] = *(const float4*)(y + (size_t)row_of_pair[at] * H + i);
        }
#pragma unroll
        for (int u = 0; u < 4; u++) {
          if (k0 + u >= top) continue;
          a.x = fmaf(c[u], v[u].x, a.x), a.y = fmaf(c[u], v[u].y, a.y), a.z = fmaf(c[u], v[u].z, a.z), a.w = fmaf(c[u], v[u].w, a.w);
        }
      }
      *(float4*)(out + (size_t)t * H + i) = a;
    }
    return;
  }
  for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < H; i += gridDim.x * blockDim.x) {
    float a = 0.f;
    for (int p = 0; p < P; p++) a += base[p * stride_p + (size_t)t * H + i];
    if (gate) a *= f;
    if (wt) {
      for (int k = 0; k < top; k++) a = fmaf(wt[(size_t)t * top + k], y[(size_t)row_of_pair[(size_t)t * top + k] * H + i], a);
    } else {
      for (int k = 0; k < top; k++) a += y[(size_t)row_of_pair[(size_t)t * top + k] * H + i];
    }
    out[(size_t)t * H + i] = a;
  }
}

// out[row_of_pair[p]] = wt[p] * x[p / top] for every (token, choice) pair p; the product is taken in float32 and rounded once.
template <typename X>
__global__ void scatter_scaled_rows_kernel(const X* __restrict__ x, const int* __restrict__ row_of_pair, const float* __restrict__ wt, int top, X* __restrict__ out,
                                           int K) {
  ib::pdl_launch_dependents();
  ib::pdl_wait();
  const int p = blockIdx.x;
  const float c = wt[p];
  const X* src = x + (size_t)(p / top) * K;
  X* dst = out + (size_t)row_of_pair[p] * K;
  for (int i = blockIdx.y * blockDim.x + threadIdx.x; i < K; i += gridDim.y * blockDim.x) dst[i] = ib::from_f32<X>(c * ib::to_f32<X>(src[i]));
}

}  // namespace

namespace {
int check_route(const RouteArgs& a, const char* who) {
  IB_CHECK_ARG(a.group_top >= 1 && a.group_top <= 4, "%s: a group's score is the sum of its %d largest scores (1 to 4)", who, a.group_top);
  IB_CHECK_ARG(a.P >= 1 && a.E > 0 && a.top > 0 && a.top <= a.E, "%s: bad sizes P=%d experts=%d top=%d", who, a.P, a.E, a.top);
  IB_CHECK_ARG(a.score >= 0 && a.score <= 2, "%s: score %d is not known (0: softmax, 1: sigmoid, 2: softmax over the chosen logits)", who, a.score);
  IB_CHECK_ARG(a.row >= a.E && a.gate_col < a.row && a.always >= 0, "%s: rows of %d logits do not hold %d experts or column %d", who, a.row, a.E, a.gate_col);
  IB_CHECK_ARG(a.n_groups >= 1 && a.E % a.n_groups == 0 && a.keep >= 1 && a.keep <= a.n_groups, "%s: %d experts in %d groups of which %d stay", who, a.E, a.n_groups, a.keep);
  return 0;
}
RouteArgs route_args(const float* logits, int P, long long stride_p, int T, int E, int n_groups, int keep, int top, float route_scale, int renorm, int* idx_out, float* wt_out,
                     int score, const float* correction, int group_top, int row, const float* logit_bias, int always, int gate_col) {
  RouteArgs a;
  a.logits = logits, a.P = P, a.stride_p = (size_t)stride_p, a.T = T, a.E = E, a.row = row > 0 ? row : E, a.n_groups = n_groups, a.keep = keep, a.top = top;
  a.route_scale = route_scale, a.renorm = renorm || score == 2, a.score = score, a.correction = correction, a.logit_bias = logit_bias, a.group_top = group_top;
  a.always = always, a.gate_col = gate_col, a.idx_out = idx_out, a.wt_out = wt_out;
  return a;
}
}  // namespace

// row: entries of a row of logits (0: E). correction, group_top, logit_bias, always, gate_col: see RouteArgs.
extern "C" int ib_moe_route(const float* logits, int P, long long stride_p, int T, int E, int n_groups, int keep, int top, float route_scale, int renorm,
                            int* idx_out, float* wt_out, int score, const float* correction, int group_top, int row, const float* logit_bias, int always, int gate_col,
                            cudaStream_t stream) {
  if (T == 0) return 0;
  const RouteArgs a = route_args(logits, P, stride_p, T, E, n_groups, keep, top, route_scale, renorm, idx_out, wt_out, score, correction, group_top, row, logit_bias, always, gate_col);
  if (check_route(a, "moe_route")) return 1;
  const size_t smem = (size_t)kRouteWarps * (2 * E + n_groups) * sizeof(float);
  IB_CHECK_ARG(smem <= 48 * 1024, "moe_route: %d experts need %zu bytes of shared memory, more than 48 KiB", E, smem);
  ib::launch(moe_route_kernel, (unsigned)((T + kRouteWarps - 1) / kRouteWarps), kRouteWarps * 32, smem, stream, a);
  IB_CHECK_LAUNCH("moe_route");
  return 0;
}

// ib_moe_route and ib_moe_sort (over E + always experts) in one kernel, for up to 128 tokens; ib_moe_route_sort_fits says whether the sizes allow it.
extern "C" int ib_moe_route_sort_fits(int T, int E, int n_groups, int always) {
  const int warps = T < 32 ? (T > 8 ? T : 8) : 32;
  return T <= 128 && ((size_t)warps * (2 * E + n_groups) + 3 * (E + always) + 1) * 4 <= 48 * 1024;
}
extern "C" int ib_moe_route_sort(const float* logits, int P, long long stride_p, int T, int E, int n_groups, int keep, int top, float route_scale, int renorm,
                                 int* idx_out, float* wt_out, int score, const float* correction, int group_top, int row, const float* logit_bias, int always, int gate_col,
                                 int tile_rows, int* offsets, int* tile_start, int* row_of_pair, int* token_of_row, cudaStream_t stream) {
  if (T == 0) return 0;
  const RouteArgs a = route_args(logits, P, stride_p, T, E, n_groups, keep, top, route_scale, renorm, idx_out, wt_out, score, correction, group_top, row, logit_bias, always, gate_col);
  if (check_route(a, "moe_route_sort")) return 1;
  IB_CHECK_ARG(tile_rows > 0 && ib_moe_route_sort_fits(T, E, n_groups, always), "moe_route_sort: %d tokens, %d experts and tiles of %d rows do not fit one CTA", T, E, tile_rows);
  const int warps = T < 32 ? (T > 8 ? T : 8) : 32;
  const size_t smem = ((size_t)warps * (2 * E + n_groups) + 3 * (E + always) + 1) * 4;
  ib::launch(moe_route_sort_kernel, 1, warps * 32, smem, stream, a, tile_rows, offsets, tile_start, row_of_pair, token_of_row);
  IB_CHECK_LAUNCH("moe_route_sort");
  return 0;
}

extern "C" int ib_moe_tile_rows() { return SM_; }

// tile_rows: the rows of a tile of the product that will run on the regrouped rows (ib_moe_tile_rows() for this file's and the m16n8k16
// kernel; the token tile of the tcgen05 kernel).
extern "C" int ib_moe_sort(const int* idx, int R, int top, int E, int tile_rows, int* offsets, int* tile_start, int* row_of_pair, int* token_of_row,
                           cudaStream_t stream) {
  if (R == 0) return 0;
  IB_CHECK_ARG(R > 0 && top > 0 && E > 0 && tile_rows > 0, "moe_sort: bad sizes pairs=%d top=%d experts=%d tile=%d", R, top, E, tile_rows);
  const size_t smem = (size_t)(3 * E + 1) * sizeof(int);
  IB_CHECK_ARG(smem <= 48 * 1024, "moe_sort: %d experts need %zu bytes of shared memory, more than 48 KiB", E, smem);
  ib::launch(moe_sort_kernel, 1, 1024, smem, stream, idx, R, top, E, tile_rows, offsets, tile_start, row_of_pair, token_of_row);
  IB_CHECK_LAUNCH("moe_sort");
  return 0;
}

extern "C" int ib_gemm_grouped(const void* x, int x_dtype, const int* src_row, const void* w, int w_dtype, void* out, int out_dtype, const int* offsets,
                               const int* tile_start, int R, int E, int N, int K, int act, const float* limits, float slope, cudaStream_t stream) {
  if (R == 0 || N == 0) return 0;
  IB_CHECK_ARG(act >= 0 && act <= 3 && (act != 3 || limits), "gemm_grouped: activation %d is not known (0: none, 1: gated SiLU, 2: squared ReLU, 3: gated, clamped)", act);
  IB_CHECK_ARG(R > 0 && E > 0 && N > 0 && K > 0, "gemm_grouped: bad sizes rows=%d experts=%d N=%d K=%d", R, E, N, K);
  dim3 grid((N + 63) / 64, R / SM_ + E);   // no more tiles than this, whatever the counts
  IB_CHECK_ARG(grid.y <= 65535, "gemm_grouped: %d rows exceed the grid limit", R);
  auto go = [&](auto kernel, auto* xp, auto* wp, auto* op) { ib::launch(kernel, grid, 256, 0, stream, xp, src_row, wp, op, offsets, tile_start, E, N, K, act, limits, slope); };
  using bf = __nv_bfloat16;
  if (x_dtype == IB_F32 && w_dtype == IB_F32 && out_dtype == IB_F32) go(gemm_grouped_kernel<float, float, float>, (const float*)x, (const float*)w, (float*)out);
  else if (x_dtype == IB_BF16 && w_dtype == IB_BF16 && out_dtype == IB_F32) go(gemm_grouped_kernel<bf, bf, float>, (const bf*)x, (const bf*)w, (float*)out);
  else if (x_dtype == IB_BF16 && w_dtype == IB_BF16 && out_dtype == IB_BF16) go(gemm_grouped_kernel<bf, bf, bf>, (const bf*)x, (const bf*)w, (bf*)out);
  else return ib_set_error("gemm_grouped: unsupported dtypes x=%d w=%d out=%d", x_dtype, w_dtype, out_dtype);
  IB_CHECK_LAUNCH("gemm_grouped");
  return 0;
}

extern "C" int ib_moe_combine(const float* y, const int* row_of_pair, const float* wt, int top, const float* base, int P, long long stride_p, float* out, int T,
                              int H, const float* gate, int gate_P, long long gate_stride, int gate_row, cudaStream_t stream) {
  if (T == 0) return 0;
  IB_CHECK_ARG(!gate || (gate_P >= 1 && gate_row >= 1), "moe_combine: a gate of %d parts and rows of %d", gate_P, gate_row);
  IB_CHECK_ARG(T > 0 && H > 0 && top > 0 && P >= 0, "moe_combine: bad sizes T=%d H=%d top=%d P=%d", T, H, top, P);
  IB_CHECK_ARG(T <= 65535, "moe_combine: T=%d rows exceed the grid limit 65535", T);
  const bool vec = H % 4 == 0 && ((uintptr_t)y & 15) == 0 && ((uintptr_t)base & 15) == 0 && ((uintptr_t)out & 15) == 0 && stride_p % 4 == 0;
  const int per = vec ? 1024 : 256;
  dim3 grid(min((H + per - 1) / per, 64), T);
  if (vec) ib::launch(moe_combine_kernel<true>, grid, 256, 0, stream, y, row_of_pair, wt, top, base, P, (size_t)stride_p, out, H, gate, gate_P, (size_t)gate_stride, gate_row);
  else ib::launch(moe_combine_kernel<false>, grid, 256, 0, stream, y, row_of_pair, wt, top, base, P, (size_t)stride_p, out, H, gate, gate_P, (size_t)gate_stride, gate_row);
  IB_CHECK_LAUNCH("moe_combine");
  return 0;
}

extern "C" int ib_gather_rows(const void* x, const int* src_row, void* out, int R, int K, int elem_bytes, cudaStream_t stream) {
  if (R == 0) return 0;
  IB_CHECK_ARG(R > 0 && K > 0 && (K * elem_bytes) % 16 == 0 && ((uintptr_t)x % 16 == 0) && ((uintptr_t)out % 16 == 0), "gather_rows: rows of %d bytes must be multiples of 16, aligned",
               K * elem_bytes);
  const int chunks = K * elem_bytes / 16;
  ib::launch(gather_rows_kernel, dim3(R, min((chunks + 127) / 128, 8)), 128, 0, stream, (const uint4*)x, src_row, (uint4*)out, chunks);
  IB_CHECK_LAUNCH("gather_rows");
  return 0;
}

extern "C" int ib_scatter_scaled_rows(const void* x, int dtype, const int* row_of_pair, const float* wt, int top, void* out, int pairs, int K, cudaStream_t stream) {
  if (pairs == 0) return 0;
  IB_CHECK_ARG(pairs > 0 && K > 0 && top > 0, "scatter_scaled_rows: bad sizes pairs=%d K=%d top=%d", pairs, K, top);
  const dim3 grid((unsigned)pairs, (unsigned)min((K + 255) / 256, 8));
  if (dtype == IB_F32) ib::launch(scatter_scaled_rows_kernel<float>, grid, 256, 0, stream, (const float*)x, row_of_pair, wt, top, (float*)out, K);
  else if (dtype == IB_BF16)
    ib::launch(scatter_scaled_rows_kernel<__nv_bfloat16>, grid, 256, 0, stream, (const __nv_bfloat16*)x, row_of_pair, wt, top, (__nv_bfloat16*)out, K);
  else return ib_set_error("scatter_scaled_rows: unknown dtype %d", dtype);
  IB_CHECK_LAUNCH("scatter_scaled_rows");
  return 0;
}
