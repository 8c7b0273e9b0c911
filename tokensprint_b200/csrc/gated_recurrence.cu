// A gated linear recurrence with one state per channel (a real-gated linear recurrent unit):
//
//   r = sigmoid(pre_r + bias_r),  i = sigmoid(pre_i + bias_i)      the gates; pre_r and pre_i are products of u in
//                                                                  `w / k` diagonal blocks of k channels
//   log a = -c r softplus(lam),   a = exp(log a)                    c: a constant of the design (`decay_scale`)
//   S_t = a S_(t-1) + sqrt(1 - a^2) i u_t                           float32, from the request's state slot
//   out_t = S_t * gelu_tanh(y_t + y_bias)                           y: the second branch of the block
//
// 1 - a^2 is taken as -expm1(2 log a), so that nothing cancels where a channel hardly forgets.  u, y
// and out are in the compute type, everything between is float32.
//
// Two kernels: rglru_scan for portions of any length, rglru_step for steps of one token per sequence.
//
// rglru_scan: a CTA takes 16 channels of one sequence and walks its tokens in rounds.  Inside a round every
// group of lanes takes RG_L consecutive tokens; what they do to the state is one pair (A, B), S -> A S + B.
// The pairs are combined by shuffles inside a warp, then across the warps through shared memory (a warp per
// channel, lanes over the warps), and each group then runs its tokens from the state that enters it.  So
// every input is read once, gates are worked out once, and the dependent chain per round is a handful of
// multiply-adds instead of one per token.  The next round's inputs are fetched before the current
// round is worked on.  No CTA waits for another.
#include "common.cuh"

#define RG_CH 16
#define RG_WARPS 16
#define RG_L 4

struct RgParams {
  const float* pre;         // [T, w / k, 2 k]: per block the r products, then the i products
  const float* bias_r;      // [w]
  const float* bias_i;      // [w]
  const float* lam;         // [w]
  const float* y_bias;      // [w] or null
  float* state;             // [slots, slot_stride], the first w entries of a row
  const int* state_slots;
  const int* cu_seqlens;
  const int* seq_index;
  long long ld_u, ld_y, ld_out, slot_stride;
  float decay_scale;
  int w, k, T;
};

__device__ __forceinline__ float rg_softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float rg_sigmoid(float x) { return 1.f / (1.f + expf(-x)); }

// The step of one token and channel: the factor on the state and what is added to it.
__device__ __forceinline__ void rg_gates(float pr, float pi, float u, float neg_rate, float& a, float& b) {
  const float log_a = neg_rate * rg_sigmoid(pr);
  a = expf(log_a);
  b = sqrtf(-expm1f(2.f * log_a)) * rg_sigmoid(pi) * u;
}

template <typename TA, int VEC>
struct RgRow {
  float u[VEC], y[VEC], pr[VEC], pi[VEC];
};

__device__ __forceinline__ void rg_load(const float* p, float (&v)[1]) { v[0] = *p; }
__device__ __forceinline__ void rg_load(const __nv_bfloat16* p, float (&v)[1]) { v[0] = __bfloat162float(*p); }
__device__ __forceinline__ void rg_load(const float* p, float (&v)[2]) {
  const float2 f = *reinterpret_cast<const float2*>(p);
  v[0] = f.x, v[1] = f.y;
}
__device__ __forceinline__ void rg_load(const __nv_bfloat16* p, float (&v)[2]) {
  const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
  v[0] = f.x, v[1] = f.y;
}
__device__ __forceinline__ void rg_store(float* p, const float (&v)[1]) { *p = v[0]; }
__device__ __forceinline__ void rg_store(__nv_bfloat16* p, const float (&v)[1]) { *p = __float2bfloat16_rn(v[0]); }
__device__ __forceinline__ void rg_store(float* p, const float (&v)[2]) { *reinterpret_cast<float2*>(p) = make_float2(v[0], v[1]); }
__device__ __forceinline__ void rg_store(__nv_bfloat16* p, const float (&v)[2]) {
  *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v[0], v[1]);
}

template <typename TA, int VEC>
__global__ void __launch_bounds__(RG_WARPS * 32, 2) rglru_scan_kernel(RgParams P, const TA* __restrict__ u, const TA* __restrict__ y, TA* __restrict__ out) {
  ts_pdl_prologue();
  constexpr int LANES = RG_CH / VEC, SUB = 32 / LANES, GROUPS = RG_WARPS * SUB, ROUND = GROUPS * RG_L;
  static_assert(RG_WARPS == RG_CH, "a warp per channel combines the warps' pairs");
  __shared__ float sA[RG_WARPS][RG_CH + 1], sB[RG_WARPS][RG_CH + 1], sS[RG_WARPS][RG_CH + 1];
  const int b = blockIdx.y;
  const int t_begin = P.cu_seqlens[b], t_end = P.cu_seqlens[b + 1];
  if (t_end <= t_begin) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int sub = lane / LANES, c_local = (lane % LANES) * VEC;
  const int c = blockIdx.x * RG_CH + c_local;
  const bool on = c < P.w;  // with VEC = 2 the width is even, so both channels exist or neither
  const int block = on ? c / P.k : 0;
  const float* pre_c = P.pre + (on ? (size_t)block * 2 * P.k + (c - block * P.k) : 0);
  const long long ld_pre = 2ll * P.w;
  float rate[VEC], br[VEC], bi[VEC], yb[VEC];
#pragma unroll
  for (int v = 0; v < VEC; ++v) {
    rate[v] = on ? -P.decay_scale * rg_softplus(P.lam[c + v]) : 0.f;
    br[v] = on ? P.bias_r[c + v] : 0.f;
    bi[v] = on ? P.bias_i[c + v] : 0.f;
    yb[v] = on && P.y_bias ? P.y_bias[c + v] : 0.f;
  }
  float* state = P.state + (size_t)P.state_slots[b] * P.slot_stride;
  const int c_own = blockIdx.x * RG_CH + warp;  // the channel whose warps' pairs this warp combines
  float carry = c_own < P.w ? state[c_own] : 0.f;

  RgRow<TA, VEC> row[RG_L];
  auto fetch = [&](int base) {
    const int t0 = base + (warp * SUB + sub) * RG_L;
#pragma unroll
    for (int l = 0; l < RG_L; ++l) {
      const int t = t0 + l;
      if (on && t < t_end) {
        rg_load(u + (size_t)t * P.ld_u + c, row[l].u);
        rg_load(y + (size_t)t * P.ld_y + c, row[l].y);
        rg_load(pre_c + (size_t)t * ld_pre, row[l].pr);
        rg_load(pre_c + (size_t)t * ld_pre + P.k, row[l].pi);
      }
    }
  };
  fetch(t_begin);
  for (int base = t_begin; base < t_end; base += ROUND) {
    const int t0 = base + (warp * SUB + sub) * RG_L;
    float a[RG_L][VEC], x[RG_L][VEC], g[RG_L][VEC];
    float A[VEC], B[VEC];
#pragma unroll
    for (int v = 0; v < VEC; ++v) A[v] = 1.f, B[v] = 0.f;
#pragma unroll
    for (int l = 0; l < RG_L; ++l)
#pragma unroll
      for (int v = 0; v < VEC; ++v) {
        if (on && t0 + l < t_end) {
          rg_gates(row[l].pr[v] + br[v], row[l].pi[v] + bi[v], row[l].u[v], rate[v], a[l][v], x[l][v]);
          g[l][v] = row[l].y[v] + yb[v];
        } else {
          a[l][v] = 1.f, x[l][v] = 0.f, g[l][v] = 0.f;
        }
        A[v] *= a[l][v];
        B[v] = fmaf(a[l][v], B[v], x[l][v]);
      }
    if (base + ROUND < t_end) fetch(base + ROUND);
    // pairs of the groups before this one in the warp, and of the whole warp
#pragma unroll
    for (int d = LANES; d < 32; d <<= 1)
#pragma unroll
      for (int v = 0; v < VEC; ++v) {
        const float pa = __shfl_up_sync(0xffffffffu, A[v], d), pb = __shfl_up_sync(0xffffffffu, B[v], d);
        if (lane >= d) {
          B[v] = fmaf(A[v], pb, B[v]);
          A[v] *= pa;
        }
      }
    float ea[VEC], eb[VEC];  // the pair of everything before this group in the warp
#pragma unroll
    for (int v = 0; v < VEC; ++v) {
      ea[v] = __shfl_up_sync(0xffffffffu, A[v], LANES);
      eb[v] = __shfl_up_sync(0xffffffffu, B[v], LANES);
      if (lane < LANES) ea[v] = 1.f, eb[v] = 0.f;
      if (sub == SUB - 1) {
        sA[warp][c_local + v] = A[v];
        sB[warp][c_local + v] = B[v];
      }
    }
    __syncthreads();
    {  // this warp's channel: states that enter the warps
      const int j = lane & (RG_WARPS - 1);
      float wa = sA[j][warp], wb = sB[j][warp];
#pragma unroll
      for (int d = 1; d < RG_WARPS; d <<= 1) {
        const float pa = __shfl_up_sync(0xffffffffu, wa, d, RG_WARPS), pb = __shfl_up_sync(0xffffffffu, wb, d, RG_WARPS);
        if (j >= d) {
          wb = fmaf(wa, pb, wb);
          wa *= pa;
        }
      }
      const float after = fmaf(wa, carry, wb);  // the state behind warp j
      const float before = __shfl_up_sync(0xffffffffu, after, 1, RG_WARPS);
      if (lane < RG_WARPS) sS[j][warp] = j == 0 ? carry : before;
      carry = __shfl_sync(0xffffffffu, after, RG_WARPS - 1);
    }
    __syncthreads();
    float S[VEC];
#pragma unroll
    for (int v = 0; v < VEC; ++v) S[v] = fmaf(ea[v], sS[warp][c_local + v], eb[v]);
#pragma unroll
    for (int l = 0; l < RG_L; ++l) {
      float o[VEC];
#pragma unroll
      for (int v = 0; v < VEC; ++v) {
        S[v] = fmaf(a[l][v], S[v], x[l][v]);
        o[v] = S[v] * (sizeof(TA) == 2 ? ts_gelu_tanh_fast(g[l][v]) : ts_gelu_tanh(g[l][v]));
      }
      if (on && t0 + l < t_end) rg_store(out + (size_t)(t0 + l) * P.ld_out + c, o);
    }
  }
  if (lane == 0 && c_own < P.w) state[c_own] = carry;
}

// One token per sequence (a decode step; tokens that belong to no sequence get zeros).
template <typename TA>
__global__ void __launch_bounds__(128) rglru_step_kernel(RgParams P, const TA* __restrict__ u, const TA* __restrict__ y, TA* __restrict__ out) {
  ts_pdl_prologue();
  const int t = blockIdx.y, c = blockIdx.x * 128 + threadIdx.x;
  if (c >= P.w) return;
  const int b = P.seq_index[t];
  float o = 0.f;
  if (b >= 0) {
    const int block = c / P.k;
    const float* pre = P.pre + (size_t)t * 2 * P.w + (size_t)block * 2 * P.k + (c - block * P.k);
    float* s = P.state + (size_t)P.state_slots[b] * P.slot_stride + c;
    float a, x;
    rg_gates(pre[0] + P.bias_r[c], pre[P.k] + P.bias_i[c], ts_to_float(u[(size_t)t * P.ld_u + c]), -P.decay_scale * rg_softplus(P.lam[c]), a, x);
    const float S = fmaf(a, *s, x);
    *s = S;
    o = S * ts_gelu_tanh(ts_to_float(y[(size_t)t * P.ld_y + c]) + (P.y_bias ? P.y_bias[c] : 0.f));
  }
  out[(size_t)t * P.ld_out + c] = ts_from_float<TA>(o);
}

template <typename TA>
static int rg_launch(const RgParams& P, const void* u, const void* y, void* out, int first_seq, int num_seqs, bool single, cudaStream_t s) {
  if (single)
    return ts_launch(rglru_step_kernel<TA>, dim3((unsigned)((P.w + 127) / 128), (unsigned)P.T), dim3(128), 0, s, P, (const TA*)u, (const TA*)y,
                     (TA*)out);
  RgParams Q = P;
  Q.cu_seqlens += first_seq;
  Q.state_slots += first_seq;
  const dim3 grid((unsigned)((P.w + RG_CH - 1) / RG_CH), (unsigned)num_seqs), block(RG_WARPS * 32);
  const size_t pair = 2 * sizeof(TA);
  const bool two = P.k % 2 == 0 && P.ld_u % 2 == 0 && P.ld_y % 2 == 0 && P.ld_out % 2 == 0 &&
                   (((uintptr_t)u | (uintptr_t)y | (uintptr_t)out) % pair) == 0 && (uintptr_t)P.pre % 8 == 0;
  if (two) return ts_launch(rglru_scan_kernel<TA, 2>, grid, block, 0, s, Q, (const TA*)u, (const TA*)y, (TA*)out);
  return ts_launch(rglru_scan_kernel<TA, 1>, grid, block, 0, s, Q, (const TA*)u, (const TA*)y, (TA*)out);
}

// u, y, out [T, w] of the compute type (row strides ld_*).  single != 0: every sequence of the step brings at most
// one token and token t is worked out from seq_index[t]; else sequences first_seq .. first_seq + num_seqs - 1 are run.
TS_EXPORT int ts_rglru_scan(const void* u, long long ld_u, const void* y, long long ld_y, int act_dtype, const float* pre, const float* bias_r,
                            const float* bias_i, const float* lam, const float* y_bias, float decay_scale, float* state, long long slot_stride,
                            const int* state_slots, const int* cu_seqlens, const int* seq_index, void* out, long long ld_out, int T, int w,
                            int k, int first_seq, int num_seqs, int single, void* stream) {
  if (T <= 0 || (!single && num_seqs <= 0)) return 0;
  if (w <= 0 || k <= 0 || w % k || ld_u < w || ld_y < w || ld_out < w || slot_stride < w || first_seq < 0) return TS_ERR_BAD_ARGUMENT;
  if (num_seqs > 65535 || (single && T > 65535)) return TS_ERR_UNSUPPORTED_SIZE;
  RgParams P = {pre, bias_r, bias_i, lam, y_bias, state, state_slots, cu_seqlens, seq_index, ld_u, ld_y, ld_out, slot_stride, decay_scale, w, k, T};
  cudaStream_t s = (cudaStream_t)stream;
  if (act_dtype == TS_DTYPE_F32) return rg_launch<float>(P, u, y, out, first_seq, num_seqs, single != 0, s);
  if (act_dtype == TS_DTYPE_BF16) return rg_launch<__nv_bfloat16>(P, u, y, out, first_seq, num_seqs, single != 0, s);
  return TS_ERR_BAD_ARGUMENT;
}
