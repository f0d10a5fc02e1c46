// Around attention with several score maps over the same values (differential attention): the queries and keys of a head come in `maps`
// parts, each with a softmax of its own, and the outputs are combined per head.
//
//  * map_qkv: the sums of the q/k/v projection's partial products with their biases; every map of every q and k head is turned by the
//    token's angles; keys and values go into the paged cache (a key row holds all maps of a kv head one after the other), and queries are
//    written once per (head, map) as rows as wide as a key row, with zeros outside the map's own part. The product of such a row with a key
//    row is the product of the two maps' parts, so the attention kernels take heads * maps query heads over kv_heads key/value heads and
//    need not know about maps.
//  * diff_combine: out[t, h] = c * u / sqrt(mean(u^2) + eps), u = a[t, h, 0] - lambda a[t, h, 1].
//
// All arithmetic is float32; what is stored may be bfloat16.
#include "kv_view.cuh"

namespace {

constexpr int kWarps = 4;
constexpr int kMaxDim = 512;

template <typename A>
__global__ void __launch_bounds__(kWarps * 32) map_qkv_kernel(const float* __restrict__ proj, int P, size_t stride_p, int R, const float* __restrict__ bias,
                                                              const float* __restrict__ cos_t, const float* __restrict__ sin_t, int rot_half, int interleaved,
                                                              const int* __restrict__ positions, const int* __restrict__ seg_of_token, A* __restrict__ q_out, IbKvView kv,
                                                              int write_kv, int heads, int maps, int dim, int v_dim, int slots, unsigned* __restrict__ status) {
  // A warp takes one slot of a token: a map of a q head, a map of a k head, or a v head, in this order (the projection's row is laid out
  // the same way: [heads * maps * dim | kv_heads * maps * dim | kv_heads * v_dim], the last two only with write_kv).
  __shared__ float vec[kWarps][kMaxDim];
  ib::pdl_launch_dependents();
  ib::pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x, j = blockIdx.y * kWarps + warp;
  if (j >= slots) return;
  const int nq = heads * maps, nk = kv.kv_heads * maps;
  const bool is_q = j < nq, is_v = j >= nq + nk;
  const int n = is_v ? v_dim : dim;
  const int col = is_v ? (nq + nk) * dim + (j - nq - nk) * v_dim : j * dim;
  const float* src = proj + (size_t)t * R + col;
  float* v = vec[warp];
  for (int d = lane; d < n; d += 32) {
    float a = src[d];
    for (int p = 1; p < P; p++) a += src[p * stride_p + d];
    v[d] = bias ? a + bias[col + d] : a;
  }
  __syncwarp();
  if (!is_v) {
    for (int i = lane; i < rot_half; i += 32) {
      const float c = cos_t[(size_t)t * rot_half + i], s = sin_t[(size_t)t * rot_half + i];
      const int a = interleaved ? 2 * i : i, b = interleaved ? 2 * i + 1 : i + rot_half;
      const float x = v[a], y = v[b];
      v[a] = x * c - y * s;
      v[b] = y * c + x * s;
    }
    __syncwarp();
  }
  if (is_q) {
    const int row = maps * dim, d0 = (j % maps) * dim;
    A* dst = q_out + ((size_t)t * nq + j) * row;
    for (int d = lane; d < row; d += 32) dst[d] = ib::from_f32<A>(d >= d0 && d < d0 + dim ? v[d - d0] : 0.f);
    return;
  }
  const int head = is_v ? j - nq - nk : (j - nq) / maps;
  const long long off = ib::kv_offset(kv, seg_of_token[t], positions[t], head);
  if (off < 0) {
    if (lane == 0) atomicOr(status, IB_ERR_BAD_PAGE);
    return;
  }
  A* dst = (A*)kv.base + off + (is_v ? kv.v_offset : (long long)((j - nq) % maps) * dim);
  for (int d = lane; d < n; d += 32) dst[d] = ib::from_f32<A>(v[d]);
}

// A warp per (token, head).
template <typename A>
__global__ void __launch_bounds__(kWarps * 32) diff_combine_kernel(const A* __restrict__ a, float lambda, float eps, float factor, A* __restrict__ out, long long items, int V) {
  ib::pdl_launch_dependents();
  ib::pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long item = (long long)blockIdx.x * kWarps + warp;
  if (item >= items) return;
  const A* a1 = a + item * 2 * V;
  const A* a2 = a1 + V;
  float ss = 0.f;
  for (int d = lane; d < V; d += 32) {
    const float u = __fmaf_rn(-lambda, ib::to_f32<A>(a2[d]), ib::to_f32<A>(a1[d]));
    ss = __fmaf_rn(u, u, ss);
  }
  const float f = factor / sqrtf(ib::warp_sum(ss) / (float)V + eps);
  for (int d = lane; d < V; d += 32) out[item * V + d] = ib::from_f32<A>(__fmaf_rn(-lambda, ib::to_f32<A>(a2[d]), ib::to_f32<A>(a1[d])) * f);
}

}  // namespace

// proj: float32 partial sums [P][T][R] of [q | k | v] (or of q alone without write_kv); bias: float32 [R] or null; cos_t, sin_t: float32 [T][rot_half].
// interleaved: entries 2i and 2i + 1 of a map are turned together (else i and i + rot_half). q_out [T][heads * maps][maps * dim].
extern "C" int ib_map_qkv(const float* proj, int P, long long stride_p, int R, const float* bias, const float* cos_t, const float* sin_t, int rot_half, int interleaved,
                          const int* positions, const int* seg_of_token, void* q_out, int act_dtype, const IbKvView* kv, int write_kv, int T, int heads, int maps, int dim,
                          int v_dim, unsigned* status, cudaStream_t stream) {
  if (T == 0) return 0;
  IB_CHECK_ARG(kv && kv->base && kv->block_table && kv->page_size > 0 && kv->num_pages > 0 && kv->table_stride > 0, "map_qkv: bad cache view");
  IB_CHECK_ARG(P >= 1 && T > 0 && heads > 0 && maps > 0 && dim > 0 && v_dim > 0 && kv->kv_heads > 0 && heads % kv->kv_heads == 0, "map_qkv: bad sizes T=%d heads=%d on %d maps=%d dim=%d v_dim=%d",
               T, heads, kv->kv_heads, maps, dim, v_dim);
  IB_CHECK_ARG(maps * dim <= kv->head_dim && v_dim <= kv->head_dim && dim <= kMaxDim && v_dim <= kMaxDim, "map_qkv: %d maps of %d or values of %d exceed the cache's row of %d (or %d)", maps,
               dim, v_dim, kv->head_dim, kMaxDim);
  IB_CHECK_ARG(rot_half >= 0 && 2 * rot_half <= dim && (rot_half == 0 || (cos_t && sin_t)), "map_qkv: a rotation of %d entries of %d", 2 * rot_half, dim);
  const int need = heads * maps * dim + (write_kv ? kv->kv_heads * (maps * dim + v_dim) : 0);
  IB_CHECK_ARG(R >= need, "map_qkv: rows of %d entries do not hold %d", R, need);
  IB_CHECK_ARG(act_dtype == kv->dtype && (act_dtype == IB_F32 || act_dtype == IB_BF16), "map_qkv: activation dtype %d and cache dtype %d must match", act_dtype, kv->dtype);
  const int slots = heads * maps + (write_kv ? kv->kv_heads * (maps + 1) : 0);
  const dim3 grid((unsigned)T, (unsigned)((slots + kWarps - 1) / kWarps));
  if (act_dtype == IB_F32)
    ib::launch(map_qkv_kernel<float>, grid, kWarps * 32, 0, stream, proj, P, (size_t)stride_p, R, bias, cos_t, sin_t, rot_half, interleaved, positions, seg_of_token, (float*)q_out,
               *kv, write_kv, heads, maps, dim, v_dim, slots, status);
  else
    ib::launch(map_qkv_kernel<__nv_bfloat16>, grid, kWarps * 32, 0, stream, proj, P, (size_t)stride_p, R, bias, cos_t, sin_t, rot_half, interleaved, positions, seg_of_token,
               (__nv_bfloat16*)q_out, *kv, write_kv, heads, maps, dim, v_dim, slots, status);
  IB_CHECK_LAUNCH("map_qkv");
  return 0;
}

// a [T][heads][2][V] -> out [T][heads][V], both of one dtype: factor * u / sqrt(mean(u^2) + eps) with u = a[.., 0, :] - lambda * a[.., 1, :].
extern "C" int ib_diff_combine(const void* a, int dtype, float lambda, float eps, float factor, void* out, long long items, int V, cudaStream_t stream) {
  if (items == 0) return 0;
  IB_CHECK_ARG(items > 0 && V > 0, "diff_combine: bad sizes items=%lld V=%d", items, V);
  const unsigned grid = (unsigned)((items + kWarps - 1) / kWarps);
  if (dtype == IB_F32) ib::launch(diff_combine_kernel<float>, grid, kWarps * 32, 0, stream, (const float*)a, lambda, eps, factor, (float*)out, items, V);
  else if (dtype == IB_BF16)
    ib::launch(diff_combine_kernel<__nv_bfloat16>, grid, kWarps * 32, 0, stream, (const __nv_bfloat16*)a, lambda, eps, factor, (__nv_bfloat16*)out, items, V);
  else return ib_set_error("diff_combine: unknown dtype %d", dtype);
  IB_CHECK_LAUNCH("diff_combine");
  return 0;
}
