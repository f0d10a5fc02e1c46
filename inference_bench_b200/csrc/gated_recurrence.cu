// A gated linear recurrence with a matrix state per head (the HGRN2 form): for head a of a request, with q, f in R^D and v in R^V,
//     S <- diag(f) S + (1 - f) v^T,    o = S^T q,      f = lower + (1 - lower) * sigmoid(z_f + b_f),   q = silu(z_q)
// where z_q, z_f, v are the rows [q | f | v] of one fused projection (float32 partial sums, added in order). The state S [D, V] is
// float32, lives in the request's state slot, starts at zero and is carried from token to token; everything here is float32.
//
//  * gated_recurrence: one CTA per (segment, head, 32 or 16 value columns). A thread owns two neighbouring columns and RPT neighbouring rows of
//    S in registers; the tokens of the segment are walked in order, sixteen at a time: the CTA first turns the sixteen tokens' projections
//    into q, f and 1 - f in shared memory, then every thread updates its rows (the gates and queries of its rows come as 16-byte reads
//    and serve both columns) and adds its share of o, which a shuffle sums over the DS threads of the column pair. The kernel is bound by
//    instruction issue, not by memory: what counts is instructions per FMA. A decoded token is a segment of one: the cost is then the state's trip from memory and back.
//    With `chunks` the same kernel walks chunks of a long segment instead, each from a zero state: it leaves the chunk's own
//    outputs, its closing state and decay, and q_t times the decay from the chunk's start to t; `chunk_carry` then walks a segment's
//    chunks in order (S_in of the next = decay * S_in + the chunk's closing state, elementwise, ending in the request's state) and
//    `chunk_apply` adds (q_t * decay)^T S_in to every output. The three give what the walk over the whole segment gives, up to
//    rounding, with as many CTAs as the segment has chunks; which path a segment takes depends on its own length only.
//  * Other forms of the same walk: a fixed decay per head with a key (form 1: q, k, v behind a SiLU; form 2: q and k turned by the token's
//    angles, the key scaled, v as it is), and a decay per channel and token with a bonus for the current token (form 3:
//    o = (S + diag(u) k v^T)^T r before S <- diag(w) S + k v^T).
//  * Form 4, the matrix memory with exponential gates (mLSTM): log gates i, f per head and token, a running maximum m_t = max(f + m_(t-1), i), and
//    S <- e^(f + m_(t-1) - m_t) S + e^(i - m_t) k v^T. The normaliser n (the same with k alone) is one more column of S whose value is always one,
//    so a head's state is [D][V + 1] and o's last entry is n . q. memory_gates makes the two factors and e^(-m_t) for whole segments (the running
//    maximum is a scan over pairs m -> max(m + a, b), so a CTA takes 256 tokens at a time); in a step of single tokens every CTA of the walk makes
//    its own from the state's m, which memory_out then moves on.
//  * memory_out: o / (max(|n . q|, e^(-m)) + 1e-6), the norm over the head, a weight per channel of all heads, the sigmoid of the gate.
//  * decay_rows: the decays of form 3, exp(-exp(w0 + W2 tanh(low))), from the float32 sums of the low-rank projection.
//  * head_norm_gate: out[t, a, :] = w * o / sqrt(mean(o^2) + eps) * silu(gate), the weight (optional) and the gate per channel of all heads.
//  * head_rmsnorm: out[t, a, :] = w * o[t, a, :] / sqrt(mean(o^2) + eps), into the activation dtype.
#include <type_traits>

#include "common.cuh"

// Where form 4's gates come from: float32 partial sums of the gates' pre-activations (rows of `row` entries, P of them stride apart, offset to the
// first head's column), a bias a head, the cap (cap tanh(z / cap)), and the running maxima float32 [slots][heads], m_stride apart.
struct IbMemoryGates {
  const float* i_src;
  const float* f_src;
  int P, row;
  size_t stride;
  const float* i_bias;
  const float* f_bias;
  float cap;
  float* m_state;
  size_t m_stride;
};

namespace {

constexpr int kChunk = 16;   // tokens prepared at a time
constexpr int kLoads = 4;    // values a thread requests at a time while it prepares tokens
constexpr int kGroup = 8;    // tokens whose outputs are reduced together

// (log input gate, log forget gate) of token t and head a: cap tanh(z / cap), and logsigmoid(cap tanh(z / cap)) = -log(1 + e^(-x)).
__device__ __forceinline__ float2 log_gates(const IbMemoryGates& g, int t, int a) {
  const float* si = g.i_src + (size_t)t * g.row + a;
  const float* sf = g.f_src + (size_t)t * g.row + a;
  float zi = si[0], zf = sf[0];
  for (int p = 1; p < g.P; p++) zi += si[p * g.stride], zf += sf[p * g.stride];
  zi = g.cap * tanhf((zi + g.i_bias[a]) / g.cap);
  zf = g.cap * tanhf((zf + g.f_bias[a]) / g.cap);
  return make_float2(zi, fminf(zf, 0.f) - log1pf(expf(-fabsf(zf))));
}

// RPT: rows of S a thread holds (for each of its two columns); kCols: value columns per CTA (32, or 16 where a thread holds sixteen rows)
struct RecurrenceExtras {
  const float* cos_t;   // form 2: float32 [T][rot_half], the angles of the first 2 * rot_half entries of q and k (entry i with i + rot_half), or null
  const float* sin_t;
  int rot_half;
  float k_scale;        // form 2: factor on the key after the rotation
  const float* decay;   // form 3: float32 [T][heads * D]
  const float2* gates;  // form 4: per token and head (factor on the state, factor on the key), or null: one token a segment, gates made here from
  IbMemoryGates mg;       //   mg and the states' running maxima
};

// FIXED: forms 1 and 2 (one decay a head, kept in a register), BONUS: form 3, both: form 4 (one decay a head and token, in shared memory)
template <int RPT, int kCols, bool FIXED_, bool BONUS_, int MAXT>
__global__ void __launch_bounds__(MAXT, MAXT == 256 && RPT == 8 ? 3 : 1) gated_recurrence_kernel(const float* __restrict__ q_src, const float* __restrict__ f_src, const float* __restrict__ v_src,
                                        int P, size_t stride_p, int R, const float* __restrict__ f_bias,
                                        const float* __restrict__ lower, float* __restrict__ state, size_t slot_stride, const int* __restrict__ seg_start,
                                        const int* __restrict__ seg_slot, float* __restrict__ o_out, int heads, int D, int V, int DS,
                                        const int* __restrict__ seg_list, const int* __restrict__ chunks, float* __restrict__ chunk_state,
                                        float* __restrict__ chunk_decay, float* __restrict__ qa_out, int form, RecurrenceExtras ex) {
  // q_src, f_src, v_src: float32 partial sums of the three parts, rows of R entries, P of them stride_p apart.
  // form 0: the gated form above (q, z_f, v). form 1: a fixed decay per head and a key:
  // S <- lower[a] S + k v^T with q, k, v = silu of q_src, f_src, v_src (f_bias is not read; lower holds one decay a head).
  // form 2: the same with q and k turned by ex's angles, k times ex.k_scale, and no SiLU anywhere.
  // form 4 (GATED): S <- g.x S + g.y k v^T with g = ex.gates[t][a] and q times ex.k_scale; V counts the column of ones, which v_src does not have.
  // form 3 (BONUS): r, k, v as they are, decays ex.decay, lower = u [heads * D]: o = (S + diag(u) k v^T)^T r, then S <- diag(decay) S + k v^T.
  // seg_list: the segments this launch walks (null: all). chunks != null: blockIdx.x is a chunk (first row, rows) that starts from a zero
  // state and leaves its closing state in chunk_state[chunk][head], its decay in chunk_decay[chunk][head] and q * decay in qa_out[row][head].
  constexpr bool GATED = FIXED_ && BONUS_, FIXED = FIXED_, BONUS = BONUS_ && !FIXED_;
  __shared__ float s_keep[GATED ? kChunk : 1], s_take[GATED ? kChunk : 1];
  extern __shared__ float sm[];   // q[kChunk][D], f[kChunk][D], g[kChunk][D], v[kChunk][kCols], running decay [D]
  float* sq = sm;
  float* sf = sq + kChunk * D;
  float* sg = sf + kChunk * D;
  float* sv = sg + kChunk * D;
  float* run = sv + kChunk * kCols;
  ib::pdl_launch_dependents();
  ib::pdl_wait();
  const int a = blockIdx.y, j0 = blockIdx.z * kCols;
  const int tid = threadIdx.x, ds = tid % DS, col = 2 * (tid / DS), j = j0 + col;   // columns j and j + 1, rows ds * RPT .. ds * RPT + RPT - 1
  const int d0 = ds * RPT;
  const bool live = j0 + 2 * ((tid & ~31) / DS) < V;   // (a warp whose columns all lie beyond V only helps to prepare the tokens)
  const bool d4 = D % 4 == 0;
  int t0, t1;
  float* S;
  if (chunks) {
    t0 = chunks[2 * blockIdx.x];
    t1 = t0 + chunks[2 * blockIdx.x + 1];
    S = chunk_state + ((size_t)blockIdx.x * heads + a) * D * V;
    for (int d = tid; d < D; d += blockDim.x) run[d] = 1.f;
  } else {
    const int s = seg_list ? seg_list[blockIdx.x] : blockIdx.x;
    t0 = seg_start[s], t1 = seg_start[s + 1];
    S = state + (size_t)seg_slot[s] * slot_stride + (size_t)a * D * V;
  }
  float st[RPT][2];
#pragma unroll
  for (int r = 0; r < RPT; r++) {
    const int d = d0 + r;
    st[r][0] = (!chunks && d < D && j < V) ? S[(size_t)d * V + j] : 0.f;
    st[r][1] = (!chunks && d < D && j + 1 < V) ? S[(size_t)d * V + j + 1] : 0.f;
  }
  const int v_cols = GATED ? V - 1 : V;   // columns the values' source has
  const int q_off = a * D, v_off = a * v_cols + j0;
  const float fixed = FIXED && !GATED ? lower[a] : 0.f;
  float u[BONUS ? RPT : 1];
  if constexpr (BONUS) {
#pragma unroll
    for (int r = 0; r < RPT; r++) u[r] = d0 + r < D ? lower[a * D + d0 + r] : 0.f;
  }
  for (int c0 = t0; c0 < t1; c0 += kChunk) {
    const int n = min(kChunk, t1 - c0);
    __syncthreads();
    if constexpr (GATED) {
      if (tid < n) {
        if (ex.gates) {
          const float2 g = ex.gates[(size_t)(c0 + tid) * heads + a];
          s_keep[tid] = g.x, s_take[tid] = g.y;
        } else {
          const float m = ex.mg.m_state[(size_t)seg_slot[seg_list ? seg_list[blockIdx.x] : blockIdx.x] * ex.mg.m_stride + a];
          const float2 g = log_gates(ex.mg, c0 + tid, a);
          const float next = fmaxf(g.y + m, g.x);
          s_keep[tid] = expf(g.y + m - next), s_take[tid] = expf(g.x - next);
        }
      }
    }
    // The sixteen tokens' rows into shared memory: every thread requests its values of kLoads items before it uses the first.
    const int step = kLoads * blockDim.x;
    if (FIXED && form == 2) {   // an item is a pair of entries that are turned together, or one that is not
      const int half = ex.rot_half, per = D - half, items = n * per;
      for (int i0 = tid; i0 < items; i0 += step) {
        float zq[kLoads], zk[kLoads], yq[kLoads], yk[kLoads], c[kLoads], sn[kLoads];
#pragma unroll
        for (int e = 0; e < kLoads; e++) {
          const int i = i0 + e * (int)blockDim.x;
          zq[e] = zk[e] = yq[e] = yk[e] = c[e] = sn[e] = 0.f;
          if (i >= items) continue;
          const int tt = i / per, w = i % per;
          const size_t at = (size_t)(c0 + tt) * R + q_off + (w < half ? w : w + half);
          zq[e] = q_src[at], zk[e] = f_src[at];
          if (w < half) {
            yq[e] = q_src[at + half], yk[e] = f_src[at + half];
            c[e] = ex.cos_t[(size_t)(c0 + tt) * half + w], sn[e] = ex.sin_t[(size_t)(c0 + tt) * half + w];
          }
        }
        for (int p = 1; p < P; p++) {
#pragma unroll
          for (int e = 0; e < kLoads; e++) {
            const int i = i0 + e * (int)blockDim.x;
            if (i >= items) continue;
            const int tt = i / per, w = i % per;
            const size_t at = p * stride_p + (size_t)(c0 + tt) * R + q_off + (w < half ? w : w + half);
            zq[e] += q_src[at], zk[e] += f_src[at];
            if (w < half) yq[e] += q_src[at + half], yk[e] += f_src[at + half];
          }
        }
#pragma unroll
        for (int e = 0; e < kLoads; e++) {
          const int i = i0 + e * (int)blockDim.x;
          if (i >= items) continue;
          const int tt = i / per, w = i % per;
          float q = zq[e], k = zk[e];
          if (w < half) {
            sq[tt * D + w + half] = yq[e] * c[e] + zq[e] * sn[e];
            sg[tt * D + w + half] = (yk[e] * c[e] + zk[e] * sn[e]) * ex.k_scale;
            q = zq[e] * c[e] - yq[e] * sn[e], k = zk[e] * c[e] - yk[e] * sn[e];
          }
          const int d = w < half ? w : w + half;
          sq[tt * D + d] = q;
          sg[tt * D + d] = k * ex.k_scale;
        }
      }
    } else {
      const int items = n * D;
      for (int i0 = tid; i0 < items; i0 += step) {
        float zq[kLoads], zf[kLoads], dc[kLoads];
#pragma unroll
        for (int e = 0; e < kLoads; e++) {
          const int i = i0 + e * (int)blockDim.x;
          zq[e] = zf[e] = dc[e] = 0.f;
          if (i >= items) continue;
          const int tt = i / D, d = i % D;
          const size_t at = (size_t)(c0 + tt) * R + q_off + d;
          zq[e] = q_src[at], zf[e] = f_src[at];
          if (BONUS) dc[e] = ex.decay[(size_t)(c0 + tt) * heads * D + q_off + d];
        }
        for (int p = 1; p < P; p++) {
#pragma unroll
          for (int e = 0; e < kLoads; e++) {
            const int i = i0 + e * (int)blockDim.x;
            if (i >= items) continue;
            const size_t at = p * stride_p + (size_t)(c0 + i / D) * R + q_off + i % D;
            zq[e] += q_src[at], zf[e] += f_src[at];
          }
        }
#pragma unroll
        for (int e = 0; e < kLoads; e++) {
          const int i = i0 + e * (int)blockDim.x;
          if (i >= items) continue;
          if constexpr (BONUS) {
            sq[i] = zq[e];
            sg[i] = zf[e];
            sf[i] = dc[e];
          } else if constexpr (GATED) {
            sq[i] = zq[e] * ex.k_scale;
            sg[i] = zf[e];
          } else if constexpr (FIXED) {
            sq[i] = zq[e] / (1.f + expf(-zq[e]));
            sg[i] = zf[e] / (1.f + expf(-zf[e]));
          } else {
            sq[i] = zq[e] / (1.f + expf(-zq[e]));
            const int d = i % D;
            const float z = zf[e] + f_bias[a * D + d];
            const float lo = lower[a * D + d];
            const float sig = 1.f / (1.f + expf(-z));
            const float f = __fmaf_rn(1.f - lo, sig, lo);
            sf[i] = f;
            sg[i] = 1.f - f;
          }
        }
      }
    }
    for (int i0 = tid; i0 < n * kCols; i0 += step) {
      float z[kLoads];
#pragma unroll
      for (int e = 0; e < kLoads; e++) {
        const int i = i0 + e * (int)blockDim.x, c = i % kCols;
        z[e] = (i < n * kCols && j0 + c < v_cols) ? v_src[(size_t)(c0 + i / kCols) * R + v_off + c] : 0.f;
      }
      for (int p = 1; p < P; p++) {
#pragma unroll
        for (int e = 0; e < kLoads; e++) {
          const int i = i0 + e * (int)blockDim.x, c = i % kCols;
          if (i < n * kCols && j0 + c < v_cols) z[e] += v_src[p * stride_p + (size_t)(c0 + i / kCols) * R + v_off + c];
        }
      }
#pragma unroll
      for (int e = 0; e < kLoads; e++) {
        const int i = i0 + e * (int)blockDim.x;
        if (i < n * kCols) sv[i] = GATED ? (j0 + i % kCols == v_cols ? 1.f : z[e]) : FIXED && form == 1 ? z[e] / (1.f + expf(-z[e])) : z[e];
      }
    }
    __syncthreads();
    if (chunks && blockIdx.z == 0) {   // q times the decay since the chunk's start, for the pass that adds the incoming state's share
      for (int d = tid; d < D; d += blockDim.x) {
        float r = run[d];
        for (int tt = 0; tt < n; tt++) {
          if (!BONUS) r *= GATED ? s_keep[GATED ? tt : 0] : FIXED ? fixed : sf[tt * D + d];
          qa_out[((size_t)(c0 + tt) * heads + a) * D + d] = sq[tt * D + d] * r;
          if (BONUS) r *= sf[tt * D + d];   // the current token's decay comes after its output
        }
        run[d] = r;
      }
    }
    // one token: the thread's rows of the state advance, acc0 and acc1 receive its share of o for its two columns
    auto advance = [&](int tt, float& acc0, float& acc1) {
      const float take = GATED ? s_take[GATED ? tt : 0] : 1.f, keep = GATED ? s_keep[GATED ? tt : 0] : fixed;
      const float v0 = GATED ? take * sv[tt * kCols + col] : sv[tt * kCols + col], v1 = GATED ? take * sv[tt * kCols + col + 1] : sv[tt * kCols + col + 1];
      float f[RPT], g[RPT], q[RPT];
      if (d4 && d0 + RPT <= D) {   // this thread's rows are whole groups of four: 16-byte reads
#pragma unroll
        for (int r = 0; r < RPT; r += 4) {
          const float4 b = *(const float4*)(sg + tt * D + d0 + r), c = *(const float4*)(sq + tt * D + d0 + r);
          const float4 a = FIXED ? make_float4(keep, keep, keep, keep) : *(const float4*)(sf + tt * D + d0 + r);
          f[r] = a.x, f[r + 1] = a.y, f[r + 2] = a.z, f[r + 3] = a.w;
          g[r] = b.x, g[r + 1] = b.y, g[r + 2] = b.z, g[r + 3] = b.w;
          q[r] = c.x, q[r + 1] = c.y, q[r + 2] = c.z, q[r + 3] = c.w;
        }
      } else {
#pragma unroll
        for (int r = 0; r < RPT; r++) {
          const int d = d0 + r;
          const bool in = d < D;
          f[r] = FIXED ? keep : in ? sf[tt * D + d] : 0.f, g[r] = in ? sg[tt * D + d] : 0.f, q[r] = in ? sq[tt * D + d] : 0.f;
        }
      }
      acc0 = acc1 = 0.f;
      if constexpr (BONUS) {
        float own = 0.f;   // this thread's rows of r . (u k)
#pragma unroll
        for (int r = 0; r < RPT; r++) {
          own = __fmaf_rn(q[r], u[r] * g[r], own);
          acc0 = __fmaf_rn(st[r][0], q[r], acc0);
          acc1 = __fmaf_rn(st[r][1], q[r], acc1);
          st[r][0] = __fmaf_rn(f[r], st[r][0], g[r] * v0);
          st[r][1] = __fmaf_rn(f[r], st[r][1], g[r] * v1);
        }
        acc0 = __fmaf_rn(own, v0, acc0);
        acc1 = __fmaf_rn(own, v1, acc1);
      } else {
#pragma unroll
        for (int r = 0; r < RPT; r++) {   // rows beyond D have f = g = q = 0: their state stays zero
          st[r][0] = __fmaf_rn(f[r], st[r][0], g[r] * v0);
          st[r][1] = __fmaf_rn(f[r], st[r][1], g[r] * v1);
          acc0 = __fmaf_rn(st[r][0], q[r], acc0);
          acc1 = __fmaf_rn(st[r][1], q[r], acc1);
        }
      }
    };
    int tt = 0;
    // Eight tokens at a time: their sixteen sums per thread are reduced over the DS threads of the column pair together, each exchange halving
    // what a lane still holds (15 shuffles for eight tokens and DS = 16 instead of 64; the pairs that are added, and so the bits, are those of
    // the token-by-token reduction).
    for (; live && tt + kGroup <= n; tt += kGroup) {
      float acc[2 * kGroup];
#pragma unroll
      for (int k = 0; k < kGroup; k++) advance(tt + k, acc[2 * k], acc[2 * k + 1]);
      int o = DS >> 1, first = 0;   // first: number of the sum that acc[0] ends up with
#pragma unroll
      for (int half = kGroup; half >= 1; half >>= 1) {
        if (o > 0) {
          const bool up = ds & o;
#pragma unroll
          for (int i = 0; i < half; i++) {
            const float give = up ? acc[i] : acc[i + half], keep = up ? acc[i + half] : acc[i];
            acc[i] = keep + __shfl_xor_sync(0xffffffffu, give, o);
          }
          first += up ? half : 0;
          o >>= 1;
        }
      }
      for (; o > 0; o >>= 1) acc[0] += __shfl_xor_sync(0xffffffffu, acc[0], o);   // more lanes than sums
      if (DS <= 2 * kGroup || (ds & (DS / (2 * kGroup) - 1)) == 0) {
        const int held = DS >= 2 * kGroup ? 1 : 2 * kGroup / DS;
#pragma unroll
        for (int i = 0; i < kGroup; i++) {   // DS >= 2: at most kGroup sums a lane
          const int m = first + i, c = m & 1;
          if (i < held && j + c < V) o_out[((size_t)(c0 + tt + (m >> 1)) * heads + a) * V + j + c] = acc[i];
        }
      }
    }
    for (; live && tt < n; tt++) {
      float acc0, acc1;
      advance(tt, acc0, acc1);
      for (int o = DS >> 1; o > 0; o >>= 1) {
        acc0 += __shfl_xor_sync(0xffffffffu, acc0, o);
        acc1 += __shfl_xor_sync(0xffffffffu, acc1, o);
      }
      if (ds == 0) {
        float* dst = o_out + ((size_t)(c0 + tt) * heads + a) * V + j;
        if (j < V) dst[0] = acc0;
        if (j + 1 < V) dst[1] = acc1;
      }
    }
  }
#pragma unroll
  for (int r = 0; r < RPT; r++) {
    const int d = d0 + r;
    if (d < D && j < V) S[(size_t)d * V + j] = st[r][0];
    if (d < D && j + 1 < V) S[(size_t)d * V + j + 1] = st[r][1];
  }
  if (chunks && blockIdx.z == 0) {
    __syncthreads();
    for (int d = tid; d < D; d += blockDim.x) chunk_decay[((size_t)blockIdx.x * heads + a) * D + d] = run[d];
  }
}

// One thread per element (d, j) of a head's state walks a long segment's chunks in order: the chunk's place in chunk_state receives
// the state the chunk starts from, and the request's state slot the state after the last chunk.
__global__ void chunk_carry_kernel(const int* __restrict__ long_segs, const int* __restrict__ seg_slot, float* __restrict__ state, size_t slot_stride,
                                   float* __restrict__ chunk_state, const float* __restrict__ chunk_decay, int heads, int D, int V) {
  ib::pdl_launch_dependents();
  ib::pdl_wait();
  const int s = long_segs[3 * blockIdx.x], c_first = long_segs[3 * blockIdx.x + 1], n_chunks = long_segs[3 * blockIdx.x + 2];
  const int a = blockIdx.y;
  float* S = state + (size_t)seg_slot[s] * slot_stride + (size_t)a * D * V;
  for (int e = blockIdx.z * blockDim.x + threadIdx.x; e < D * V; e += gridDim.z * blockDim.x) {
    const int d = e / V;
    float cur = S[e];
    for (int c0 = c_first; c0 < c_first + n_chunks; c0 += 8) {   // eight chunks' values are requested before the first is used
      float own[8], dec[8];
#pragma unroll
      for (int u = 0; u < 8; u++) {
        const int c = c0 + u;
        if (c < c_first + n_chunks) {
          own[u] = chunk_state[((size_t)c * heads + a) * D * V + e];
          dec[u] = chunk_decay[((size_t)c * heads + a) * D + d];
        }
      }
#pragma unroll
      for (int u = 0; u < 8; u++) {
        const int c = c0 + u;
        if (c < c_first + n_chunks) {
          chunk_state[((size_t)c * heads + a) * D * V + e] = cur;
          cur = __fmaf_rn(dec[u], cur, own[u]);
        }
      }
    }
    S[e] = cur;
  }
}

// o[t][j] += sum_d qa[t][d] * S_in[d][j] for the rows of one chunk: a CTA of 256 threads takes 64 rows x 64 columns, 32 values of d at a time; a
// thread owns 4 x 4 outputs, so a value of d costs it two 16-byte reads of shared memory for sixteen FMAs.
__global__ void __launch_bounds__(256) chunk_apply_kernel(const int* __restrict__ chunks, const float* __restrict__ chunk_state, const float* __restrict__ qa,
                                                          float* __restrict__ o_out, int heads, int D, int V) {
  __shared__ __align__(16) float s_in[32][64];
  __shared__ __align__(16) float s_q[32][68];   // [d][row]
  ib::pdl_launch_dependents();
  ib::pdl_wait();
  const int t0 = chunks[2 * blockIdx.x], n = chunks[2 * blockIdx.x + 1];
  const int a = blockIdx.y, j0 = blockIdx.z * 64;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;   // columns 4 tx .., rows 4 ty ..
  const float* Sin = chunk_state + ((size_t)blockIdx.x * heads + a) * D * V;
  float acc[4][4];
#pragma unroll
  for (int r = 0; r < 4; r++)
#pragma unroll
    for (int c = 0; c < 4; c++) acc[r][c] = 0.f;
  for (int d0 = 0; d0 < D; d0 += 32) {
    float in[8], q[8];
#pragma unroll
    for (int e = 0; e < 8; e++) {   // all sixteen values are requested before the first is stored
      const int i = threadIdx.x + e * 256, dd = i >> 6, c = i & 63, tt = i >> 5, qd = i & 31;
      in[e] = (d0 + dd < D && j0 + c < V) ? Sin[(size_t)(d0 + dd) * V + j0 + c] : 0.f;
      q[e] = (tt < n && d0 + qd < D) ? qa[((size_t)(t0 + tt) * heads + a) * D + d0 + qd] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int e = 0; e < 8; e++) {
      const int i = threadIdx.x + e * 256;
      s_in[i >> 6][i & 63] = in[e];
      s_q[i & 31][i >> 5] = q[e];
    }
    __syncthreads();
#pragma unroll 8
    for (int dd = 0; dd < 32; dd++) {
      const float4 v = *(const float4*)&s_in[dd][4 * tx], w = *(const float4*)&s_q[dd][4 * ty];
      const float qv[4] = {w.x, w.y, w.z, w.w}, sv[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
      for (int r = 0; r < 4; r++)
#pragma unroll
        for (int c = 0; c < 4; c++) acc[r][c] = __fmaf_rn(qv[r], sv[c], acc[r][c]);
    }
  }
#pragma unroll
  for (int r = 0; r < 4; r++) {
    const int tt = 4 * ty + r;
    if (tt >= n) continue;
    float* dst = o_out + ((size_t)(t0 + tt) * heads + a) * V + j0 + 4 * tx;
#pragma unroll
    for (int c = 0; c < 4; c++)
      if (j0 + 4 * tx + c < V) dst[c] += acc[r][c];
  }
}

template <typename O>
__global__ void head_rmsnorm_kernel(const float* __restrict__ o, const float* __restrict__ w, float eps, O* __restrict__ out, long long items, int V) {
  ib::pdl_launch_dependents();
  ib::pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long item = (long long)blockIdx.x * (blockDim.x >> 5) + warp;
  if (item >= items) return;
  const float* src = o + item * V;
  float ss = 0.f;
  for (int i = lane; i < V; i += 32) ss = __fmaf_rn(src[i], src[i], ss);
  const float inv = rsqrtf(ib::warp_sum(ss) / (float)V + eps);
  for (int i = lane; i < V; i += 32) out[item * V + i] = ib::from_f32<O>(w[i] * (src[i] * inv));
}

// dec[t][c] = exp(-exp(w0[c] + sum_j w2[j][c] tanh(low[t][j]))): TT tokens and 256 channels a CTA; the tanh values are made once per CTA.
template <int TT>
__global__ void __launch_bounds__(256) decay_rows_kernel(const float* __restrict__ low, int P, size_t stride_p, int rank, const float* __restrict__ w2,
                                                         const float* __restrict__ w0, float* __restrict__ dec, int T, int C) {
  extern __shared__ float th[];   // [rank][TT]
  ib::pdl_launch_dependents();
  ib::pdl_wait();
  const int t0 = blockIdx.y * TT, n = min(TT, T - t0);
  for (int i = threadIdx.x; i < rank * TT; i += blockDim.x) {
    const int tt = i / rank, j = i % rank;
    float z = 0.f;
    if (tt < n) {
      const float* src = low + (size_t)(t0 + tt) * rank + j;
      z = src[0];
      for (int p = 1; p < P; p++) z += src[p * stride_p];
    }
    th[j * TT + tt] = tanhf(z);
  }
  __syncthreads();
  const int c = blockIdx.x * 256 + threadIdx.x;
  if (c >= C) return;
  float acc[TT];
#pragma unroll
  for (int tt = 0; tt < TT; tt++) acc[tt] = 0.f;
  constexpr int U = TT == 1 ? 16 : 8;   // rows of w2 requested before the first is used
  int j = 0;
  for (; j + U <= rank; j += U) {
    float w[U];
#pragma unroll
    for (int e = 0; e < U; e++) w[e] = w2[(size_t)(j + e) * C + c];
#pragma unroll
    for (int e = 0; e < U; e++)
#pragma unroll
      for (int tt = 0; tt < TT; tt++) acc[tt] = __fmaf_rn(w[e], th[(j + e) * TT + tt], acc[tt]);
  }
  for (; j < rank; j++) {
    const float w = w2[(size_t)j * C + c];
#pragma unroll
    for (int tt = 0; tt < TT; tt++) acc[tt] = __fmaf_rn(w, th[j * TT + tt], acc[tt]);
  }
  const float b = w0[c];
#pragma unroll
  for (int tt = 0; tt < TT; tt++)
    if (tt < n) dec[(size_t)(t0 + tt) * C + c] = expf(-expf(acc[tt] + b));
}

// A warp per (token, head): the head's norm, a weight per channel (or none), the gate's SiLU from its float32 partial sums.
template <typename O>
__global__ void head_norm_gate_kernel(const float* __restrict__ o, const float* __restrict__ w, float eps, const float* __restrict__ gate, int gate_P, size_t gate_stride,
                                      int gate_row, O* __restrict__ out, long long items, int heads, int V) {
  ib::pdl_launch_dependents();
  ib::pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long item = (long long)blockIdx.x * (blockDim.x >> 5) + warp;
  if (item >= items) return;
  const long long t = item / heads;
  const int a = (int)(item - t * heads);
  const float* src = o + item * V;
  const float* gr = gate + t * gate_row + a * V;
  float ss = 0.f;
  for (int i = lane; i < V; i += 32) ss = __fmaf_rn(src[i], src[i], ss);
  const float inv = 1.f / sqrtf(ib::warp_sum(ss) / (float)V + eps);
  for (int i = lane; i < V; i += 32) {
    float g = gr[i];
    for (int p = 1; p < gate_P; p++) g += gr[p * gate_stride + i];
    const float y = w ? w[a * V + i] * (src[i] * inv) : src[i] * inv;
    out[item * V + i] = ib::from_f32<O>(y * (g / (1.f + expf(-g))));
  }
}

// The gates of form 4 for whole segments: a CTA per (segment, head) walks its tokens 256 at a time. A token maps m to max(m + f, i); maps compose as
// (a, b) then (a', b') = (a + a', max(b + a', b')), so the running maxima are an inclusive scan (shuffles inside a warp, then over the warps).
// gates[t][head] = (e^(f + m_(t-1) - m_t), e^(i - m_t)), bound[t][head] = e^(-m_t); the state's m becomes the segment's last.
constexpr int kGateTokens = 256;

__global__ void __launch_bounds__(kGateTokens) memory_gates_kernel(IbMemoryGates g, const int* __restrict__ seg_start, const int* __restrict__ seg_slot,
                                                                   float2* __restrict__ gates, float* __restrict__ bound, int heads) {
  __shared__ float2 total[kGateTokens / 32];
  __shared__ float m_all[kGateTokens + 1];
  ib::pdl_launch_dependents();
  ib::pdl_wait();
  const int s = blockIdx.x, a = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int t0 = seg_start[s], t1 = seg_start[s + 1];
  float* m_slot = g.m_state + (size_t)seg_slot[s] * g.m_stride + a;
  float m_in = *m_slot;
  for (int c0 = t0; c0 < t1; c0 += kGateTokens) {
    const int t = c0 + tid;
    const bool in = t < t1;
    const float2 z = in ? log_gates(g, t, a) : make_float2(-INFINITY, 0.f);   // beyond the end: the map that changes nothing
    float A = z.y, B = z.x;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float pa = __shfl_up_sync(0xffffffffu, A, o), pb = __shfl_up_sync(0xffffffffu, B, o);
      if (lane >= o) {
        B = fmaxf(pb + A, B);
        A = pa + A;
      }
    }
    if (lane == 31) total[warp] = make_float2(A, B);
    if (tid == 0) m_all[0] = m_in;
    __syncthreads();
    float m0 = m_in;   // the running maximum before this warp's first token
    for (int w = 0; w < warp; w++) m0 = fmaxf(m0 + total[w].x, total[w].y);
    const float m = fmaxf(m0 + A, B);
    m_all[tid + 1] = m;
    __syncthreads();
    if (in) {
      gates[(size_t)t * heads + a] = make_float2(expf(z.y + m_all[tid] - m), expf(z.x - m));
      bound[(size_t)t * heads + a] = expf(-m);
    }
    m_in = m_all[min(kGateTokens, t1 - c0)];
    __syncthreads();
  }
  if (tid == 0 && t1 > t0) *m_slot = m_in;
}

// A warp per (token, head): o float32 [T][heads][V + 1] with n . q as its last entry. bound: e^(-m) of memory_gates, or null in a step whose row t is
// segment t: m is then moved on here, from the state, as the walk did.
template <typename O>
__global__ void memory_out_kernel(const float* __restrict__ o, const float* __restrict__ bound, IbMemoryGates g, const int* __restrict__ seg_slot,
                                  const float* __restrict__ w, float eps, const float* __restrict__ gate, int gate_P, size_t gate_stride, int gate_row,
                                  O* __restrict__ out, long long items, int heads, int V) {
  ib::pdl_launch_dependents();
  ib::pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long item = (long long)blockIdx.x * (blockDim.x >> 5) + warp;
  if (item >= items) return;
  const long long t = item / heads;
  const int a = (int)(item - t * heads);
  float floor_;
  if (bound) {
    floor_ = bound[item];
  } else {
    float* m_slot = g.m_state + (size_t)seg_slot[t] * g.m_stride + a;
    const float2 z = log_gates(g, (int)t, a);
    const float m = fmaxf(z.y + *m_slot, z.x);
    __syncwarp();
    if (lane == 0) *m_slot = m;
    floor_ = expf(-m);
  }
  const float* src = o + item * (V + 1);
  const float* gr = gate + t * gate_row + a * V;
  const float div = 1.f / (fmaxf(fabsf(src[V]), floor_) + 1e-6f);
  float ss = 0.f;
  for (int i = lane; i < V; i += 32) {
    const float v = src[i] * div;
    ss = __fmaf_rn(v, v, ss);
  }
  const float inv = 1.f / sqrtf(ib::warp_sum(ss) / (float)V + eps);
  for (int i = lane; i < V; i += 32) {
    float z = gr[i];
    for (int p = 1; p < gate_P; p++) z += gr[p * gate_stride + i];
    out[item * V + i] = ib::from_f32<O>(w[a * V + i] * (src[i] * div * inv) / (1.f + expf(-z)));
  }
}

}  // namespace

// seg_list: int32 [n_segments] of the segments to walk (null: segments 0 .. n_segments - 1).
// chunks: null, or int32 [n_segments][2] = (first row, rows <= 64) of chunks that each start from a zero state (n_segments then counts
// chunks); chunk_state float32 [chunks][heads][D][V], chunk_decay float32 [chunks][heads][D] and qa float32 [T][heads][D] receive what
// ib_recurrence_chunks_finish needs.
namespace {
int launch_recurrence(const float* q_src, const float* f_src, const float* v_src, int P, long long stride_p, int R, const float* f_bias, const float* lower, float* state,
                      long long slot_stride, const int* seg_start, const int* seg_slot, int n_segments, float* o_out, int heads, int D, int V, const int* seg_list,
                      const int* chunks, float* chunk_state, float* chunk_decay, float* qa, int form, const RecurrenceExtras& ex, cudaStream_t stream) {
  if (n_segments == 0) return 0;
  IB_CHECK_ARG(!chunks || (chunk_state && chunk_decay && qa), "recurrence: chunks need their state, decay and query buffers");
  IB_CHECK_ARG(n_segments > 0 && P >= 1 && heads > 0 && D > 0 && V > 0, "recurrence: bad sizes segments=%d P=%d heads=%d D=%d V=%d", n_segments, P, heads, D, V);
  IB_CHECK_ARG(D <= 512, "recurrence: a head's key size %d is above 512", D);
  IB_CHECK_ARG(R >= heads * D && R >= heads * V, "recurrence: rows of %d entries do not hold %d heads of %d and %d", R, heads, D, V);
  const int rpt = D <= 256 ? 8 : 16, kCols = D <= 256 ? 32 : 16;
  IB_CHECK_ARG(heads <= 65535 && (V + kCols - 1) / kCols <= 65535, "recurrence: the grid is too large");
  int DS = 1;
  while (DS * rpt < D) DS *= 2;
  if (DS < 2) DS = 2;   // a CTA is a whole warp at least (kCols / 2 column pairs x DS)
  const size_t smem = ((size_t)kChunk * (3 * D + kCols) + D) * sizeof(float);
  const dim3 grid((unsigned)n_segments, (unsigned)heads, (unsigned)((V + kCols - 1) / kCols));
  auto go = [&](auto kernel) {
    if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    ib::launch(kernel, grid, kCols / 2 * DS, smem, stream, q_src, f_src, v_src, P, (size_t)stride_p, R, f_bias, lower, state, (size_t)slot_stride, seg_start, seg_slot, o_out,
               heads, D, V, DS, seg_list, chunks, chunk_state, chunk_decay, qa, form, ex);
  };
  auto pick = [&](auto fixed, auto bonus) {
    constexpr bool F = decltype(fixed)::value, B = decltype(bonus)::value;
    if (rpt == 8 && DS <= 16) go(gated_recurrence_kernel<8, 32, F, B, 256>);
    else if (rpt == 8) go(gated_recurrence_kernel<8, 32, F, B, 512>);
    else go(gated_recurrence_kernel<16, 16, F, B, 256>);
  };
  if (form == 3) pick(std::false_type(), std::true_type());
  else if (form == 4) pick(std::true_type(), std::true_type());
  else if (form == 0) pick(std::false_type(), std::false_type());
  else pick(std::true_type(), std::false_type());
  IB_CHECK_LAUNCH("recurrence");
  return 0;
}
}  // namespace

// The forms with parts of their own (2: turned queries and keys with a fixed decay per head; 3: a decay per channel and token, a bonus for the
// current token): q, k, v float32 partial sums [P][T][row] each, stride_p elements apart. The other arguments as for ib_gated_recurrence.
extern "C" int ib_recurrence_parts(const float* q, const float* k, const float* v, int P, long long stride_p, int row, const float* head_param, float* state,
                                   long long slot_stride, const int* seg_start, const int* seg_slot, int n_segments, float* o_out, int heads, int D, int V,
                                   const int* seg_list, const int* chunks, float* chunk_state, float* chunk_decay, float* qa, int form, const float* cos_t,
                                   const float* sin_t, int rot_half, float k_scale, const float* decay, cudaStream_t stream) {
  if (n_segments == 0) return 0;
  IB_CHECK_ARG(form == 2 || form == 3, "recurrence_parts: form %d is not 2 or 3", form);
  IB_CHECK_ARG(q && k && v && head_param && (form != 3 || decay), "recurrence_parts: a part, the decays or the bonus is missing");
  IB_CHECK_ARG(rot_half >= 0 && 2 * rot_half <= D && (rot_half == 0 || (cos_t && sin_t)), "recurrence_parts: a rotation of %d entries of %d", 2 * rot_half, D);
  RecurrenceExtras ex = {cos_t, sin_t, rot_half, k_scale, decay};
  return launch_recurrence(q, k, v, P, stride_p, row, nullptr, head_param, state, slot_stride, seg_start, seg_slot, n_segments, o_out, heads, D, V, seg_list, chunks, chunk_state,
                           chunk_decay, qa, form, ex, stream);
}

// The matrix memory (form 4). g: see IbMemoryGates; V: a value head's size; state float32 [slots][heads][D][V + 1], o_out [T][heads][V + 1]. gates
// [T][heads][2] from ib_memory_gates, or null where every segment walked here brings one token. q_scale multiplies the queries.
extern "C" int ib_memory_walk(const float* q, const float* k, const float* v, int P, long long stride_p, int row, const IbMemoryGates* g, const float* gates, float q_scale,
                              float* state, long long slot_stride, const int* seg_start, const int* seg_slot, int n_segments, float* o_out, int heads, int D, int V,
                              const int* seg_list, const int* chunks, float* chunk_state, float* chunk_decay, float* qa, cudaStream_t stream) {
  if (n_segments == 0) return 0;
  IB_CHECK_ARG(q && k && v && (gates || (g && !chunks)), "memory_walk: a part or the gates are missing");
  RecurrenceExtras ex = {};
  ex.k_scale = q_scale, ex.gates = (const float2*)gates;
  if (g) ex.mg = *g;
  return launch_recurrence(q, k, v, P, stride_p, row, nullptr, nullptr, state, slot_stride, seg_start, seg_slot, n_segments, o_out, heads, D, V + 1, seg_list, chunks, chunk_state,
                           chunk_decay, qa, 4, ex, stream);
}

extern "C" int ib_memory_gates(const IbMemoryGates* g, const int* seg_start, const int* seg_slot, int n_segments, float* gates, float* bound, int heads, cudaStream_t stream) {
  if (n_segments == 0) return 0;
  IB_CHECK_ARG(n_segments > 0 && heads > 0 && heads <= 65535 && g && g->P >= 1 && g->cap > 0.f, "memory_gates: bad sizes segments=%d heads=%d", n_segments, heads);
  ib::launch(memory_gates_kernel, dim3((unsigned)n_segments, (unsigned)heads), kGateTokens, 0, stream, *g, seg_start, seg_slot, (float2*)gates, bound, heads);
  IB_CHECK_LAUNCH("memory_gates");
  return 0;
}

// gate: float32 partial sums [gate_P][T][gate_row], offset to the first head's first column; out [T][heads * V].
extern "C" int ib_memory_out(const float* o, const float* bound, const IbMemoryGates* g, const int* seg_slot, const float* w, float eps, const float* gate, int gate_P,
                             long long gate_stride, int gate_row, void* out, int out_dtype, int T, int heads, int V, cudaStream_t stream) {
  if (T == 0) return 0;
  IB_CHECK_ARG(T > 0 && heads > 0 && V > 0 && gate && gate_P >= 1 && gate_row >= heads * V && w && g, "memory_out: bad sizes T=%d heads=%d V=%d", T, heads, V);
  const long long items = (long long)T * heads;
  const unsigned grid = (unsigned)((items + 3) / 4);
  if (out_dtype == IB_F32)
    ib::launch(memory_out_kernel<float>, grid, 128, 0, stream, o, bound, *g, seg_slot, w, eps, gate, gate_P, (size_t)gate_stride, gate_row, (float*)out, items, heads, V);
  else if (out_dtype == IB_BF16)
    ib::launch(memory_out_kernel<__nv_bfloat16>, grid, 128, 0, stream, o, bound, *g, seg_slot, w, eps, gate, gate_P, (size_t)gate_stride, gate_row, (__nv_bfloat16*)out, items,
               heads, V);
  else return ib_set_error("memory_out: unknown output dtype %d", out_dtype);
  IB_CHECK_LAUNCH("memory_out");
  return 0;
}

extern "C" int ib_gated_recurrence(const float* proj, int P, long long stride_p, const float* f_bias, const float* lower, float* state, long long slot_stride,
                                   const int* seg_start, const int* seg_slot, int n_segments, float* o_out, int heads, int D, int V, const int* seg_list,
                                   const int* chunks, float* chunk_state, float* chunk_decay, float* qa, int form, int row, int q_col, int f_col, int v_col,
                                   cudaStream_t stream) {
  // form, row, q_col, f_col, v_col: see the kernel; row <= 0 stands for the gated form's own row [q | f | v] with its columns.
  if (n_segments == 0) return 0;
  IB_CHECK_ARG(form == 0 || form == 1, "gated_recurrence: form %d is not known (0: gated, 1: fixed decay with a key)", form);
  int R = 2 * heads * D + heads * V;
  if (row <= 0) q_col = 0, f_col = heads * D, v_col = 2 * heads * D;
  else R = row;
  IB_CHECK_ARG(q_col >= 0 && f_col >= 0 && v_col >= 0 && q_col + heads * D <= R && f_col + heads * D <= R && v_col + heads * V <= R,
               "gated_recurrence: the columns %d, %d, %d do not fit a row of %d", q_col, f_col, v_col, R);
  return launch_recurrence(proj + q_col, proj + f_col, proj + v_col, P, stride_p, R, f_bias, lower, state, slot_stride, seg_start, seg_slot, n_segments, o_out, heads, D, V,
                           seg_list, chunks, chunk_state, chunk_decay, qa, form, RecurrenceExtras{}, stream);
}

// After ib_gated_recurrence on chunks: long_segs int32 [n_long][3] = (segment, its first chunk, its chunks), chunks as above (n_chunks of them).
extern "C" int ib_recurrence_chunks_finish(const int* long_segs, int n_long, const int* chunks, int n_chunks, const int* seg_slot, float* state, long long slot_stride,
                                           float* chunk_state, const float* chunk_decay, const float* qa, float* o_out, int heads, int D, int V, cudaStream_t stream) {
  if (n_long == 0 || n_chunks == 0) return 0;
  IB_CHECK_ARG(n_long > 0 && n_chunks > 0 && heads > 0 && heads <= 65535 && D > 0 && V > 0, "recurrence_chunks_finish: bad sizes");
  ib::launch(chunk_carry_kernel, dim3((unsigned)n_long, (unsigned)heads, (unsigned)min((D * V + 255) / 256, 64)), 256, 0, stream, long_segs, seg_slot, state,
             (size_t)slot_stride, chunk_state, chunk_decay, heads, D, V);
  IB_CHECK_LAUNCH("recurrence chunk_carry");
  ib::launch(chunk_apply_kernel, dim3((unsigned)n_chunks, (unsigned)heads, (unsigned)((V + 63) / 64)), 256, 0, stream, chunks, (const float*)chunk_state, qa, o_out, heads, D, V);
  IB_CHECK_LAUNCH("recurrence chunk_apply");
  return 0;
}

extern "C" int ib_head_rmsnorm(const float* o, const float* w, float eps, void* out, int out_dtype, long long items, int V, cudaStream_t stream) {
  if (items == 0) return 0;
  IB_CHECK_ARG(items > 0 && V > 0, "head_rmsnorm: bad sizes items=%lld V=%d", items, V);
  const unsigned grid = (unsigned)((items + 3) / 4);
  if (out_dtype == IB_F32) ib::launch(head_rmsnorm_kernel<float>, grid, 128, 0, stream, o, w, eps, (float*)out, items, V);
  else if (out_dtype == IB_BF16) ib::launch(head_rmsnorm_kernel<__nv_bfloat16>, grid, 128, 0, stream, o, w, eps, (__nv_bfloat16*)out, items, V);
  else return ib_set_error("head_rmsnorm: unknown output dtype %d", out_dtype);
  IB_CHECK_LAUNCH("head_rmsnorm");
  return 0;
}

extern "C" int ib_decay_rows(const float* low, int P, long long stride_p, int rank, const float* w2, const float* w0, float* dec, int T, int C, cudaStream_t stream) {
  if (T == 0) return 0;
  IB_CHECK_ARG(T > 0 && C > 0 && rank > 0 && P >= 1, "decay_rows: bad sizes T=%d channels=%d rank=%d P=%d", T, C, rank, P);
  auto go = [&](auto kernel, int tt) {
    const size_t smem = (size_t)rank * tt * sizeof(float);
    if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    ib::launch(kernel, dim3((unsigned)((C + 255) / 256), (unsigned)((T + tt - 1) / tt)), 256, smem, stream, low, P, (size_t)stride_p, rank, w2, w0, dec, T, C);
  };
  IB_CHECK_ARG(rank <= 3072 && T <= 65535, "decay_rows: rank %d (at most 3072) or T=%d rows are too large", rank, T);
  if (T >= 256) go(decay_rows_kernel<16>, 16);   // (a channel's sum runs over the rank in the same order in both forms)
  else go(decay_rows_kernel<1>, 1);
  IB_CHECK_LAUNCH("decay_rows");
  return 0;
}

// gate: float32 partial sums [gate_P][T][gate_row], offset to the first head's first column.
extern "C" int ib_head_norm_gate(const float* o, const float* w, float eps, const float* gate, int gate_P, long long gate_stride, int gate_row, void* out, int out_dtype,
                                 int T, int heads, int V, cudaStream_t stream) {
  if (T == 0) return 0;
  IB_CHECK_ARG(T > 0 && heads > 0 && V > 0 && gate && gate_P >= 1 && gate_row >= heads * V, "head_norm_gate: bad sizes T=%d heads=%d V=%d gate rows of %d", T, heads, V, gate_row);
  const long long items = (long long)T * heads;
  const unsigned grid = (unsigned)((items + 3) / 4);
  if (out_dtype == IB_F32) ib::launch(head_norm_gate_kernel<float>, grid, 128, 0, stream, o, w, eps, gate, gate_P, (size_t)gate_stride, gate_row, (float*)out, items, heads, V);
  else if (out_dtype == IB_BF16)
    ib::launch(head_norm_gate_kernel<__nv_bfloat16>, grid, 128, 0, stream, o, w, eps, gate, gate_P, (size_t)gate_stride, gate_row, (__nv_bfloat16*)out, items, heads, V);
  else return ib_set_error("head_norm_gate: unknown output dtype %d", out_dtype);
  IB_CHECK_LAUNCH("head_norm_gate");
  return 0;
}
