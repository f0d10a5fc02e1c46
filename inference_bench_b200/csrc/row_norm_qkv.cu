// Queries, keys and values of an attention whose norms run over a token's whole query and key rows (all heads at once, not head by
// head) and whose values may be mixed with another layer's.
//
//  * row_norm_qkv: a CTA per token adds the partial sums of its projection row [heads x D | kv_heads x D | kv_heads x V] once (several loads in
//    flight) into shared memory, takes the two sums of squares as block sums, and writes: q = w_q q / sqrt(mean(q^2) + eps) and k likewise, both
//    turned (entry i with i + half over each head's first 2 half entries); queries in the activation dtype, keys into the paged cache; values
//    into the cache as they are, or as (1 - c) v + c v_first with c one learned number and v_first another layer's values of the same tokens.
//    Where asked, the token's own values are kept in float32 as the v_first of later layers.
// All arithmetic is float32; sums run in an order that depends on the row's sizes alone.
#include "kv_view.cuh"

namespace {

struct RowNormArgs {
  const float* proj;        // float32 partial sums [P][T][R]
  int P, R;
  size_t stride_p;
  const float* q_w;         // [heads * D]
  const float* k_w;         // [kv_heads * D]
  float eps;
  const float* cos_t;       // [T][half] or null
  const float* sin_t;
  int half;
  const int* positions;
  const int* seg_of_token;
  int heads, D, V;
  const float* mix;         // one number on the device, or null: the values as they are
  const float* first;       // float32 [T][kv_heads * V]: what they are mixed with
  float* keep;              // float32 [T][kv_heads * V] or null: receives the values as projected
  unsigned* status;
};

template <typename A, bool VEC>
__global__ void __launch_bounds__(512) row_norm_qkv_kernel(RowNormArgs p, A* __restrict__ q_out, IbKvView kv) {
  extern __shared__ __align__(16) float row[];
  __shared__ float scratch[32];
  ib::pdl_launch_dependents();
  ib::pdl_wait();
  const int t = blockIdx.x, G = kv.kv_heads, nq = p.heads * p.D, nk = G * p.D, nv = G * p.V, n = nq + nk + nv;
  const float* src = p.proj + (size_t)t * p.R;
  float sq = 0.f, sk = 0.f;
  auto count = [&](int i, float a) {
    if (i < nq) sq = __fmaf_rn(a, a, sq);
    else if (i < nq + nk) sk = __fmaf_rn(a, a, sk);
  };
  if constexpr (VEC) {   // rows and parts of multiples of four values: a group of four lies in one part
    for (int i = threadIdx.x * 4; i < n; i += blockDim.x * 4) {
      float4 a = *(const float4*)(src + i);
#pragma unroll 4
      for (int s = 1; s < p.P; s++) {
        const float4 b = *(const float4*)(src + s * p.stride_p + i);
        a.x += b.x, a.y += b.y, a.z += b.z, a.w += b.w;
      }
      *(float4*)(row + i) = a;
      count(i, a.x), count(i, a.y), count(i, a.z), count(i, a.w);
    }
  } else {
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
      float a = src[i];
#pragma unroll 4
      for (int s = 1; s < p.P; s++) a += src[s * p.stride_p + i];
      row[i] = a;
      count(i, a);
    }
  }
  sq = ib::block_sum(sq, scratch);   // (its barriers also order the row's writes before the reads below)
  sk = ib::block_sum(sk, scratch);
  const float iq = 1.f / sqrtf(sq / (float)nq + p.eps), ik = 1.f / sqrtf(sk / (float)nk + p.eps);
  const long long off = ib::kv_offset(kv, p.seg_of_token[t], p.positions[t], 0);
  if (off < 0 && threadIdx.x == 0) atomicOr(p.status, IB_ERR_BAD_PAGE);
  const long long head_stride = (long long)kv.page_size * kv.head_dim;
  A* k_dst = (A*)kv.base + off;
  A* v_dst = k_dst + kv.v_offset;
  const float* cs = p.cos_t + (size_t)t * p.half;
  const float* sn = p.sin_t + (size_t)t * p.half;
  const int per = p.D - p.half;   // an item is a pair of entries that are turned together, or one that is not
  for (int i = threadIdx.x; i < (p.heads + G) * per; i += blockDim.x) {
    const int h = i / per, w = i - h * per;
    const bool is_q = h < p.heads;
    if (!is_q && off < 0) continue;
    const int d = w < p.half ? w : w + p.half, at = h * p.D + d;    // place in the row [q | k]
    const float* nw = is_q ? p.q_w + at : p.k_w + at - nq;
    const float inv = is_q ? iq : ik;
    A* dst = is_q ? q_out + (size_t)t * nq + at : k_dst + (h - p.heads) * head_stride + d;
    const float a = nw[0] * (row[at] * inv);
    if (w < p.half) {
      const float b = nw[p.half] * (row[at + p.half] * inv), c = cs[w], s = sn[w];
      dst[0] = ib::from_f32<A>(a * c - b * s);
      dst[p.half] = ib::from_f32<A>(b * c + a * s);
    } else {
      dst[0] = ib::from_f32<A>(a);
    }
  }
  const float c = p.mix ? p.mix[0] : 0.f;
  for (int i = threadIdx.x; i < nv; i += blockDim.x) {
    const int h = i / p.V;
    float v = row[nq + nk + i];
    if (p.keep) p.keep[(size_t)t * nv + i] = v;
    if (p.mix) v = __fmaf_rn(c, p.first[(size_t)t * nv + i], (1.f - c) * v);
    if (off >= 0) v_dst[h * head_stride + (i - h * p.V)] = ib::from_f32<A>(v);
  }
}

}  // namespace

// The sizes and pointers are those of RowNormArgs. q_out [T][heads * D] in the cache's dtype.
extern "C" int ib_row_norm_qkv(const float* proj, int P, long long stride_p, int R, const float* q_w, const float* k_w, float eps, const float* cos_t, const float* sin_t,
                               int half, const int* positions, const int* seg_of_token, void* q_out, int act_dtype, const IbKvView* kv, int T, int heads, int D, int V,
                               const float* mix, const float* first, float* keep, unsigned* status, cudaStream_t stream) {
  if (T == 0) return 0;
  IB_CHECK_ARG(kv && kv->base && kv->block_table && kv->kv_heads > 0 && heads > 0 && heads % kv->kv_heads == 0, "row_norm_qkv: bad cache view or %d heads", heads);
  IB_CHECK_ARG(T > 0 && P >= 1 && D > 0 && V > 0 && D <= kv->head_dim && V <= kv->head_dim, "row_norm_qkv: heads of %d and %d do not fit the cache's row of %d", D, V, kv->head_dim);
  IB_CHECK_ARG(half >= 0 && 2 * half <= D && (half == 0 || (cos_t && sin_t)), "row_norm_qkv: %d entries of %d turned", 2 * half, D);
  IB_CHECK_ARG(q_w && k_w && (!mix || first), "row_norm_qkv: a norm's weights or the values to mix with are missing");
  IB_CHECK_ARG(act_dtype == kv->dtype && (act_dtype == IB_F32 || act_dtype == IB_BF16), "row_norm_qkv: activation dtype %d and cache dtype %d must match", act_dtype, kv->dtype);
  const int n = (heads + kv->kv_heads) * D + kv->kv_heads * V;
  const size_t smem = (size_t)n * sizeof(float);
  IB_CHECK_ARG(R >= n && smem <= 200 * 1024, "row_norm_qkv: rows of %d values need %zu bytes of shared memory (at most 200 KiB) and a projection as wide, not %d", n, smem, R);
  RowNormArgs a = {proj, P, R, (size_t)stride_p, q_w, k_w, eps, cos_t, sin_t, half, positions, seg_of_token, heads, D, V, mix, first, keep, status};
  const bool vec = D % 4 == 0 && V % 4 == 0 && R % 4 == 0 && stride_p % 4 == 0 && (uintptr_t)proj % 16 == 0;
  const int threads = n >= 2048 ? 512 : (n >= 512 ? 256 : 128);
  auto go = [&](auto kernel, auto* q) {
    if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    ib::launch(kernel, (unsigned)T, threads, smem, stream, a, q, *kv);
  };
  using bf = __nv_bfloat16;
  if (act_dtype == IB_F32 && vec) go(row_norm_qkv_kernel<float, true>, (float*)q_out);
  else if (act_dtype == IB_F32) go(row_norm_qkv_kernel<float, false>, (float*)q_out);
  else if (vec) go(row_norm_qkv_kernel<bf, true>, (bf*)q_out);
  else go(row_norm_qkv_kernel<bf, false>, (bf*)q_out);
  IB_CHECK_LAUNCH("row_norm_qkv");
  return 0;
}
