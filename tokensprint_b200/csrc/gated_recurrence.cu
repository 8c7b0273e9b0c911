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
// Kernels: rglru_scan for portions of any length; rglru_step for steps of one token per sequence, and
// rglru_gate_step, which also works out the gate products.
//
// rglru_scan: a CTA takes 16 channels of one sequence and walks its tokens in rounds.  Inside a round every
// group of lanes takes RG_L consecutive tokens; what they do to the state is one pair (A, B), S -> A S + B.
// The pairs are combined by shuffles inside a warp, then across the warps through shared memory (a warp per
// channel, lanes over the warps), and each group then runs its tokens from the state that enters it.  So
// every input is read once, gates are worked out once, and the dependent chain per round is a handful of
// multiply-adds instead of one per token.  The next round's inputs are asked for as soon as
// this round's gates are worked out.  No CTA waits for another.
#include "common.cuh"

#define RG_CH 16
#define RG_L 2

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

// The step of one token and channel: the factor on the state and what is added to it.  `rate` is
// -decay_scale * softplus(lam).
__device__ __forceinline__ void rg_gates(float pr, float pi, float u, float rate, float& a, float& b) {
  const float log_a = rate * rg_sigmoid(pr);
  a = expf(log_a);
  b = sqrtf(-expm1f(2.f * log_a)) * rg_sigmoid(pi) * u;
}

// The same for u and results in bfloat16, with the fast exponential, division and square root (errors of a few
// units in the last place of float32).  1 - a^2 = 1 - exp(-z) with z = -2 log a: the first terms of its series
// where z is small (so nothing cancels; the next term is below 2e-7 of the sum), the difference elsewhere.
// Both sigmoids come from one division: with A = 1 + exp(-pr), B = 1 + exp(-pi) they are B / (A B) and A / (A B)
// (the gates' arguments are cut at -40, where a sigmoid is 4e-18, so that A B stays finite).
__device__ __forceinline__ void rg_gates_fast(float pr, float pi, float u, float rate, float& a, float& b) {
  const float A = 1.f + __expf(-fmaxf(pr, -40.f)), B = 1.f + __expf(-fmaxf(pi, -40.f));
  const float inv = __fdividef(1.f, A * B);
  const float log_a = rate * (B * inv);
  a = __expf(log_a);
  const float z = -2.f * log_a;
  const float series = z * fmaf(z * -0.5f, fmaf(z * (-1.f / 3.f), fmaf(z * -0.25f, fmaf(z, -0.2f, 1.f), 1.f), 1.f), 1.f);
  const float rest = z < 0.125f ? series : fmaf(-a, a, 1.f);
  float root;
  asm("sqrt.approx.f32 %0, %1;" : "=f"(root) : "f"(rest));
  b = root * (A * inv) * u;
}
__device__ __forceinline__ void rg_gates_of(float, float pr, float pi, float u, float rate, float& a, float& b) { rg_gates(pr, pi, u, rate, a, b); }
__device__ __forceinline__ void rg_gates_of(__nv_bfloat16, float pr, float pi, float u, float rate, float& a, float& b) {
  rg_gates_fast(pr, pi, u, rate, a, b);
}

// One or two neighbouring channels of a row as they lie in memory.
template <typename TA, int VEC>
struct RgRaw;
template <>
struct RgRaw<float, 1> {
  float v;
  __device__ __forceinline__ float get(int) const { return v; }
};
template <>
struct RgRaw<float, 2> {
  float2 v;
  __device__ __forceinline__ float get(int i) const { return i ? v.y : v.x; }
};
template <>
struct RgRaw<__nv_bfloat16, 1> {
  __nv_bfloat16 v;
  __device__ __forceinline__ float get(int) const { return __bfloat162float(v); }
};
template <>
struct RgRaw<__nv_bfloat16, 2> {
  __nv_bfloat162 v;
  __device__ __forceinline__ float get(int i) const { return i ? __high2float(v) : __low2float(v); }
};
template <typename TA, int VEC>
__device__ __forceinline__ RgRaw<TA, VEC> rg_load(const TA* p) {
  return *reinterpret_cast<const RgRaw<TA, VEC>*>(p);
}

__device__ __forceinline__ void rg_store(float* p, const float (&v)[1]) { *p = v[0]; }
__device__ __forceinline__ void rg_store(__nv_bfloat16* p, const float (&v)[1]) { *p = __float2bfloat16_rn(v[0]); }
__device__ __forceinline__ void rg_store(float* p, const float (&v)[2]) { *reinterpret_cast<float2*>(p) = make_float2(v[0], v[1]); }
__device__ __forceinline__ void rg_store(__nv_bfloat16* p, const float (&v)[2]) {
  *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v[0], v[1]);
}

template <typename TA, int VEC, int WARPS>
__global__ void __launch_bounds__(WARPS * 32, 32 / WARPS) rglru_scan_kernel(RgParams P, const TA* __restrict__ u, const TA* __restrict__ y, TA* __restrict__ out) {
  ts_pdl_prologue();
  constexpr int LANES = RG_CH / VEC, SUB = 32 / LANES, GROUPS = WARPS * SUB, ROUND = GROUPS * RG_L;
  static_assert(WARPS >= RG_CH && WARPS <= 32, "a warp per channel combines the warps' pairs, a lane per warp");
  __shared__ float sA[WARPS][RG_CH + 1], sB[WARPS][RG_CH + 1], sS[WARPS][RG_CH + 1];
  const int b = blockIdx.y;
  const int t_begin = P.cu_seqlens[b], t_end = P.cu_seqlens[b + 1];
  if (t_end <= t_begin) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int sub = lane / LANES, c_local = (lane % LANES) * VEC;
  const int c = blockIdx.x * RG_CH + c_local;
  const bool on = c < P.w;  // with VEC = 2 the width is even, so both channels exist or neither
  const int block = on ? c / P.k : 0;
  float rate[VEC], br[VEC], bi[VEC], y_bias[VEC];
#pragma unroll
  for (int v = 0; v < VEC; ++v) {
    rate[v] = on ? -P.decay_scale * rg_softplus(P.lam[c + v]) : 0.f;
    br[v] = on ? P.bias_r[c + v] : 0.f;
    bi[v] = on ? P.bias_i[c + v] : 0.f;
    y_bias[v] = on && P.y_bias ? P.y_bias[c + v] : 0.f;
  }
  float* state = P.state + (size_t)P.state_slots[b] * P.slot_stride;
  const int c_own = blockIdx.x * RG_CH + warp;  // the channel whose warps' pairs this warp combines
  const bool combines = warp < RG_CH && c_own < P.w;
  float carry = combines ? state[c_own] : 0.f;

  // rows are addressed from the portion's first one, in 32 bits (the host refuses longer ones)
  const int n = t_end - t_begin, ld_u = (int)P.ld_u, ld_y = (int)P.ld_y, ld_out = (int)P.ld_out, ld_pre = 2 * P.w;
  const TA* ub = u + (size_t)t_begin * P.ld_u + c;
  const TA* yb = y + (size_t)t_begin * P.ld_y + c;
  TA* ob = out + (size_t)t_begin * P.ld_out + c;
  const float* pb = P.pre + (size_t)t_begin * 2 * P.w + (on ? (size_t)block * 2 * P.k + (c - block * P.k) : 0);
  const int mine = on ? n : 0;  // tokens that this thread's channels have
  RgRaw<TA, VEC> ru[RG_L];
  RgRaw<float, VEC> rr[RG_L], ri[RG_L];
  int t0 = (warp * SUB + sub) * RG_L;  // this group's first token
  auto fetch = [&](int first) {
#pragma unroll
    for (int l = 0; l < RG_L; ++l)
      if (first + l < mine) {
        ru[l] = rg_load<TA, VEC>(ub + (first + l) * ld_u);
        rr[l] = rg_load<float, VEC>(pb + (first + l) * ld_pre);
        ri[l] = rg_load<float, VEC>(pb + (first + l) * ld_pre + P.k);
      }
  };
  fetch(t0);
  for (int base = 0; base < n; base += ROUND, t0 += ROUND) {
    float a[RG_L][VEC], x[RG_L][VEC];
    RgRaw<TA, VEC> g[RG_L];
    float A[VEC], B[VEC];
#pragma unroll
    for (int v = 0; v < VEC; ++v) A[v] = 1.f, B[v] = 0.f;
#pragma unroll
    for (int l = 0; l < RG_L; ++l)
#pragma unroll
      for (int v = 0; v < VEC; ++v) {
        if (t0 + l < mine) {
          rg_gates_of(TA(), rr[l].get(v) + br[v], ri[l].get(v) + bi[v], ru[l].get(v), rate[v], a[l][v], x[l][v]);
        } else {
          a[l][v] = 1.f, x[l][v] = 0.f;
        }
        A[v] *= a[l][v];
        B[v] = fmaf(a[l][v], B[v], x[l][v]);
      }
    // asked for now: the other branch of this round (used behind the barriers), the next round's inputs
#pragma unroll
    for (int l = 0; l < RG_L; ++l)
      if (t0 + l < mine) g[l] = rg_load<TA, VEC>(yb + (t0 + l) * ld_y);
    fetch(t0 + ROUND);
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
    if (warp < RG_CH) {  // this warp's channel: states that enter the warps
      const int j = lane & (WARPS - 1);
      float wa = sA[j][warp], wb = sB[j][warp];
#pragma unroll
      for (int d = 1; d < WARPS; d <<= 1) {
        const float pa = __shfl_up_sync(0xffffffffu, wa, d, WARPS), pb = __shfl_up_sync(0xffffffffu, wb, d, WARPS);
        if (j >= d) {
          wb = fmaf(wa, pb, wb);
          wa *= pa;
        }
      }
      const float after = fmaf(wa, carry, wb);  // the state behind warp j
      const float before = __shfl_up_sync(0xffffffffu, after, 1, WARPS);
      if (lane < WARPS) sS[j][warp] = j == 0 ? carry : before;
      carry = __shfl_sync(0xffffffffu, after, WARPS - 1);
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
        const float z = g[l].get(v) + y_bias[v];
        o[v] = S[v] * (sizeof(TA) == 2 ? ts_gelu_tanh_fast(z) : ts_gelu_tanh(z));
      }
      if (t0 + l < mine) rg_store(ob + (t0 + l) * ld_out, o);
    }
  }
  if (combines && lane == 0) state[c_own] = carry;
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

// One token per sequence with the gate products in the kernel (bfloat16, block widths that are multiples of 8):
// a CTA takes 16 channels of one block and up to 32 tokens.  Its four warps share the block's k inputs in
// chunks of 32 and compute, for r and for i, [16 channels x 32 tokens] partial products on mma.sync (rows: the
// weight rows as they lie in memory, columns: tokens), which meet in shared memory; then every thread works
// out the gates and the step of four (token, channel) pairs.  The products' order of k is free, so a lane
// takes eight consecutive inputs of a row with one 16-byte load and feeds two MMA steps with them.  The first
// chunks' weights are asked for before the kernels ahead are waited for: no kernel writes them.
#define RG_STEP_TOKENS 32
#define RG_STEP_AHEAD 2

__device__ __forceinline__ void rg_mma(float (&c)[4], unsigned a0, unsigned a1, unsigned a2, unsigned a3, unsigned b0, unsigned b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

__global__ void __launch_bounds__(128) rglru_gate_step_kernel(RgParams P, const __nv_bfloat16* __restrict__ u, const __nv_bfloat16* __restrict__ y,
                                                              const __nv_bfloat16* __restrict__ gates, __nv_bfloat16* __restrict__ out) {
  ts_pdl_launch_dependents();
  __shared__ float part[4][2][16][RG_STEP_TOKENS + 1];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, quad = lane >> 2, qi = lane & 3;
  const int k = P.k, tiles = (k + 15) / 16, block = blockIdx.x / tiles, row0 = (blockIdx.x - block * tiles) * 16;
  const int t0 = blockIdx.y * RG_STEP_TOKENS;
  const int chunks = (k + 31) / 32;
  // weight rows of this lane: row0 + quad and row0 + quad + 8, of the r matrix and of the i matrix k rows further
  const bool row_on[2] = {row0 + quad < k, row0 + quad + 8 < k};
  const __nv_bfloat16* wrow = gates + ((size_t)block * 2 * k + row0 + quad) * k + qi * 8;
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  auto weight = [&](int chunk, int gate, int half) {
    const bool there = row_on[half] && chunk < chunks && chunk * 32 + qi * 8 < k;
    return there ? *reinterpret_cast<const uint4*>(wrow + ((size_t)gate * k + half * 8) * k + chunk * 32) : zero;
  };
  uint4 ahead[RG_STEP_AHEAD][2][2];
#pragma unroll
  for (int n = 0; n < RG_STEP_AHEAD; ++n)
#pragma unroll
    for (int g = 0; g < 2; ++g)
#pragma unroll
      for (int h = 0; h < 2; ++h) ahead[n][g][h] = weight(warp + 4 * n, g, h);
  // what the step of this thread's four (token, channel) pairs will need beside the products: threads of a half
  // warp take the 16 channels of one token.  The parameters come before the wait, the rest is asked for right
  // behind it, so that these trips run beside those of the products' inputs.
  const int ch = threadIdx.x & 15, c = block * k + row0 + ch;
  const bool mine = row0 + ch < k;
  float neg_rate = 0.f, br = 0.f, bi = 0.f, yb = 0.f;
  if (mine) {
    neg_rate = -P.decay_scale * rg_softplus(P.lam[c]);
    br = P.bias_r[c];
    bi = P.bias_i[c];
    yb = P.y_bias ? P.y_bias[c] : 0.f;
  }
  ts_pdl_wait();
  float* slot[RG_STEP_TOKENS / 8];
  float old[RG_STEP_TOKENS / 8], uv[RG_STEP_TOKENS / 8], yv[RG_STEP_TOKENS / 8];
#pragma unroll
  for (int i = 0; i < RG_STEP_TOKENS / 8; ++i) {
    const int t = t0 + (threadIdx.x >> 4) + i * 8;
    const int b = mine && t < P.T ? P.seq_index[t] : -1;
    slot[i] = b >= 0 ? P.state + (size_t)P.state_slots[b] * P.slot_stride + c : nullptr;
  }
#pragma unroll
  for (int i = 0; i < RG_STEP_TOKENS / 8; ++i) {
    const int t = t0 + (threadIdx.x >> 4) + i * 8;
    if (slot[i] != nullptr) {
      old[i] = *slot[i];
      uv[i] = __bfloat162float(u[(size_t)t * P.ld_u + c]);
      yv[i] = __bfloat162float(y[(size_t)t * P.ld_y + c]);
    }
  }

  float acc[2][4][4];
#pragma unroll
  for (int g = 0; g < 2; ++g)
#pragma unroll
    for (int n = 0; n < 4; ++n) acc[g][n][0] = acc[g][n][1] = acc[g][n][2] = acc[g][n][3] = 0.f;
  auto multiply = [&](int chunk, const uint4 (&w)[2][2]) {
#pragma unroll
    for (int n = 0; n < 4; ++n) {
      const int t = t0 + n * 8 + quad;
      const uint4 x = t < P.T && chunk * 32 + qi * 8 < k ? *reinterpret_cast<const uint4*>(u + (size_t)t * P.ld_u + (size_t)block * k + chunk * 32 + qi * 8) : zero;
#pragma unroll
      for (int g = 0; g < 2; ++g) {
        rg_mma(acc[g][n], w[g][0].x, w[g][1].x, w[g][0].y, w[g][1].y, x.x, x.y);
        rg_mma(acc[g][n], w[g][0].z, w[g][1].z, w[g][0].w, w[g][1].w, x.z, x.w);
      }
    }
  };
#pragma unroll
  for (int n = 0; n < RG_STEP_AHEAD; ++n)
    if (warp + 4 * n < chunks) multiply(warp + 4 * n, ahead[n]);
  for (int chunk = warp + 4 * RG_STEP_AHEAD; chunk < chunks; chunk += 4) {
    const uint4 w[2][2] = {{weight(chunk, 0, 0), weight(chunk, 0, 1)}, {weight(chunk, 1, 0), weight(chunk, 1, 1)}};
    multiply(chunk, w);
  }
#pragma unroll
  for (int g = 0; g < 2; ++g)
#pragma unroll
    for (int n = 0; n < 4; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) part[warp][g][quad + (e >> 1) * 8][n * 8 + 2 * qi + (e & 1)] = acc[g][n][e];
  __syncthreads();
  if (!mine) return;
#pragma unroll
  for (int i = 0; i < RG_STEP_TOKENS / 8; ++i) {
    const int tt = (threadIdx.x >> 4) + i * 8, t = t0 + tt;
    if (t >= P.T) break;
    float o = 0.f;
    if (slot[i] != nullptr) {
      const float pr = part[0][0][ch][tt] + part[1][0][ch][tt] + (part[2][0][ch][tt] + part[3][0][ch][tt]);
      const float pi = part[0][1][ch][tt] + part[1][1][ch][tt] + (part[2][1][ch][tt] + part[3][1][ch][tt]);
      float a, x;
      rg_gates_fast(pr + br, pi + bi, uv[i], neg_rate, a, x);
      const float S = fmaf(a, old[i], x);
      *slot[i] = S;
      o = S * ts_gelu_tanh_fast(yv[i] + yb);
    }
    out[(size_t)t * P.ld_out + c] = __float2bfloat16_rn(o);
  }
}

template <typename TA>
static int rg_launch(const RgParams& P, const void* u, const void* y, void* out, int first_seq, int num_seqs, bool single, cudaStream_t s) {
  if (single)
    return ts_launch(rglru_step_kernel<TA>, dim3((unsigned)((P.w + 127) / 128), (unsigned)P.T), dim3(128), 0, s, P, (const TA*)u, (const TA*)y,
                     (TA*)out);
  RgParams Q = P;
  Q.cu_seqlens += first_seq;
  Q.state_slots += first_seq;
  const dim3 grid((unsigned)((P.w + RG_CH - 1) / RG_CH), (unsigned)num_seqs);
  const size_t pair = 2 * sizeof(TA);
  const bool two = P.k % 2 == 0 && P.ld_u % 2 == 0 && P.ld_y % 2 == 0 && P.ld_out % 2 == 0 &&
                   (((uintptr_t)u | (uintptr_t)y | (uintptr_t)out) % pair) == 0 && (uintptr_t)P.pre % 8 == 0;
  // as many warps on an SM either way: one CTA of 32 where there is at most one per SM, else two of 16
  const bool wide = (long long)grid.x * grid.y <= 148;
#define RG_CASE(VEC, WARPS) return ts_launch(rglru_scan_kernel<TA, VEC, WARPS>, grid, dim3(WARPS * 32), 0, s, Q, (const TA*)u, (const TA*)y, (TA*)out)
  if (two && wide) RG_CASE(2, 32);
  if (two) RG_CASE(2, 16);
  if (wide) RG_CASE(1, 32);
  RG_CASE(1, 16);
#undef RG_CASE
}

// u, y, out [T, w] of the compute type (row strides ld_*).  single != 0: every sequence of the step brings at most
// one token and token t is worked out from seq_index[t]; else sequences first_seq .. first_seq + num_seqs - 1 are run.
TS_EXPORT int ts_rglru_scan(const void* u, long long ld_u, const void* y, long long ld_y, int act_dtype, const float* pre, const float* bias_r,
                            const float* bias_i, const float* lam, const float* y_bias, float decay_scale, float* state, long long slot_stride,
                            const int* state_slots, const int* cu_seqlens, const int* seq_index, void* out, long long ld_out, int T, int w,
                            int k, int first_seq, int num_seqs, int single, void* stream) {
  if (T <= 0 || (!single && num_seqs <= 0)) return 0;
  if (w <= 0 || k <= 0 || w % k || ld_u < w || ld_y < w || ld_out < w || slot_stride < w || first_seq < 0) return TS_ERR_BAD_ARGUMENT;
  const long long ld_most = max(max(ld_u, ld_y), max(ld_out, 2ll * w));
  if (num_seqs > 65535 || (single && T > 65535) || (T + 4096ll) * ld_most >= (1ll << 31)) return TS_ERR_UNSUPPORTED_SIZE;
  RgParams P = {pre, bias_r, bias_i, lam, y_bias, state, state_slots, cu_seqlens, seq_index, ld_u, ld_y, ld_out, slot_stride, decay_scale, w, k, T};
  cudaStream_t s = (cudaStream_t)stream;
  if (act_dtype == TS_DTYPE_F32) return rg_launch<float>(P, u, y, out, first_seq, num_seqs, single != 0, s);
  if (act_dtype == TS_DTYPE_BF16) return rg_launch<__nv_bfloat16>(P, u, y, out, first_seq, num_seqs, single != 0, s);
  return TS_ERR_BAD_ARGUMENT;
}

// A step in which every sequence brings at most one token, with the gate products worked out here: gates
// [w / k, 2 k, k] bfloat16, per block the r matrix and then the i matrix, both [out, in].
TS_EXPORT int ts_rglru_step(const void* u, long long ld_u, const void* y, long long ld_y, const void* gates, const float* bias_r, const float* bias_i,
                            const float* lam, const float* y_bias, float decay_scale, float* state, long long slot_stride, const int* state_slots,
                            const int* seq_index, void* out, long long ld_out, int T, int w, int k, void* stream) {
  if (T <= 0) return 0;
  if (w <= 0 || k <= 0 || w % k || ld_u < w || ld_y < w || ld_out < w || slot_stride < w) return TS_ERR_BAD_ARGUMENT;
  if (k % 8 || ld_u % 8 || ((uintptr_t)u | (uintptr_t)gates) % 16) return TS_ERR_UNSUPPORTED_SIZE;
  RgParams P = {nullptr, bias_r, bias_i, lam, y_bias, state, state_slots, nullptr, seq_index, ld_u, ld_y, ld_out, slot_stride, decay_scale, w, k, T};
  const dim3 grid((unsigned)((w / k) * ((k + 15) / 16)), (unsigned)((T + RG_STEP_TOKENS - 1) / RG_STEP_TOKENS));
  return ts_launch(rglru_gate_step_kernel, grid, dim3(128), 0, (cudaStream_t)stream, P, (const __nv_bfloat16*)u, (const __nv_bfloat16*)y,
                   (const __nv_bfloat16*)gates, (__nv_bfloat16*)out);
}
