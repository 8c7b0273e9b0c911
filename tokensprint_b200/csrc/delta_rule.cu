// The gated delta rule: per head a state S [d, e] in float32 that is decayed, corrected by what it
// already returns for the new key, and read out, token by token:
//
//   q^ = q / sqrt(sum q^2 + unit_eps) * q_scale,   k^ = k / sqrt(sum k^2 + unit_eps)       (per head)
//   beta = sigmoid(b),   g = exp(-exp(A_log_h) * softplus(a + dt_bias_h))                  (per token and head)
//   S <- g S;   u = beta (v - S^T k^);   S <- S + k^ u^T;   o = S^T q^
//
// The decay may also be one number per key channel (rows of S): g_c = exp(-exp(A_log_h) softplus(a_c + dt_bias_hc)),
// S <- diag(g) S; the decays of long portions are worked out ahead by channel_decay (every CTA of the scan that shares
// a head reads them), those of a step of few tokens in the staging pass.
//
// The kernels also run the plain linear recurrence S <- decay_h S + k v^T, o = S^T q with one constant decay per head and rotated
// q and k (retention, ts_retention_scan): the rule without its correction (u = v), without unit lengths and write strengths.
//
// delta_scan takes the tokens of a portion in blocks of BT (four).  With S the state before a block, Gamma(j..i] the
// product of the decays of tokens j+1 .. i and G_i that of all tokens of the block up to i (all per key channel),
//
//   k~_i = G_i k^_i,   q~_i = G_i q^_i,   k'_j = Gamma(j..last] k^_j
//   A_ij = sum_c k^_i k^_j Gamma(j..i]  (j < i),    B_ij = sum_c q^_i k^_j Gamma(j..i]  (j <= i)
//   u_i  = beta_i (v_i - S^T k~_i - sum_(j<i) A_ij u_j),    o_i = S^T q~_i + sum_(j<=i) B_ij u_j
//   S   <- G_last S + sum_j k'_j u_j^T
//
// which is the rule above written out for the block: one walk over the state gives the 2 BT sums S^T k~ and S^T q~ and
// one round of shuffles adds them up, the u follow one from the other in a handful of multiply-adds, and a second walk
// updates the state.  (Token by token, the chain of two walks and a round of shuffles was met at every token:
// 2,048 tokens at 16 heads of 64 x 128 took 0.66 ms, 0.72 with a decay per channel.)  Decays are only ever multiplied, never
// divided by, so a channel that forgets at once costs no accuracy.
//
// One CTA per (sequence, head, block of value columns).  A thread owns one value column and 4 M key channels of it in
// registers, in fours that interleave with those of the other R - 1 lanes of its column (so that the lanes' 16-byte reads
// of the staged rows fall on consecutive pieces of shared memory); the R lanes add their partial sums by shuffles.  The
// CTA walks its sequence's tokens of the step in order, up to 16 at a time: their q, k, v, beta and decays are staged in shared memory by all
// threads (the next round's rows are asked for before the round's updates begin and wait in registers), then a warp per
// block works out unit lengths, A, B and the block's rows k~, q~, k', G_last, then every thread runs
// the round's blocks from there.  The state is read from the
// request's slot before the first token and written back after the last, so a sequence may be cut
// anywhere, and a token's result depends on nothing but its own sequence and the start of its portion (the grouping of
// the sums: float32 rounding, nothing else).  Steps of one token per sequence run blocks of one.  In the slot the state
// lies value column by value column ([H, e, d]: a thread's channels are then contiguous fours).  A sequence without
// tokens in this step (a padded lane of a fixed-size batch) touches nothing.  q and k heads may be shared by
// groups of value heads (head h reads q/k head h / (H / G)).  Everything is float32.
#include "common.cuh"

#define DR_THREADS 128
#define DR_MAX_KEY_DIM 1024
// Tokens staged at a time: 16 (a portion) or one (steps of one token per sequence), fewer where the padded key width exceeds
// 128 (a round's rows are at most 2,048 entries each, 16 per thread, which wait in registers while the round before is worked
// through).
__host__ __device__ constexpr int dr_round_tokens(int dpad, int bt) { return bt == 1 ? 1 : (dpad <= 128 ? 16 : 2048 / dpad); }

__device__ __forceinline__ float dr_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// The decay of one head (or key channel) and token from its raw row entry: exp(-rate softplus(raw + bias)), rate = exp(A_log_h).
__device__ __forceinline__ float dr_decay(float raw, float bias, float rate) { return expf(-rate * dr_softplus(raw + bias)); }

// Where the write strengths and the decays of a step come from.
struct DrGates {
  const void* beta;       // [T, H] raw write strengths (the sigmoid is taken here), rows ld_beta apart
  const float* decay;     // one entry per (token, head) or, CHANNEL, per (token, head, key channel), rows ld_decay apart
  const float* a_log;     // [H]
  const float* dt_bias;   // [H], or [H * d] with a decay per channel
  long long ld_beta, ld_decay;
  int beta_bf16;          // element type of beta
  int raw;                // 1: decay holds the raw entries; 0: the decays themselves
  const float2* rotation; // DR_LINEAR: [T, half] cosines and sines by which entries i and i + half of q and k turn, or null
  int half;
};

// The recurrences these kernels know.
#define DR_HEAD 0     // the delta rule with one decay per (token, head)
#define DR_CHANNEL 1  // with one per (token, head, key channel)
#define DR_LINEAR 2   // no correction (u = v), q and k as they come but rotated, one constant decay per head (retention)

// The block's sums over the key channels, in the order nk_0.. (squares of k), nq_0.., A_10, A_20, A_21, .., B_00, B_10, B_11, ..
__host__ __device__ constexpr int dr_sums(int bt) { return 2 * bt + bt * bt; }

// Adds up v[0 .. N) over the lanes of a warp; lane l gets the total of v[l] (N <= 32; for N <= 16 of v[l % 16]).
template <int N>
__device__ __forceinline__ float dr_scatter_sum(float (&v)[32], int lane) {
  if (N <= 16) {
#pragma unroll
    for (int i = 0; i < N; ++i) v[i] += __shfl_xor_sync(0xffffffffu, v[i], 16);
  }
#pragma unroll
  for (int o = N <= 16 ? 8 : 16; o > 0; o >>= 1) {
    const bool up = (lane & o) != 0;
#pragma unroll
    for (int i = 0; i < o; ++i) {
      const float give = up ? v[i] : v[i + o], keep = up ? v[i + o] : v[i];
      v[i] = keep + __shfl_xor_sync(0xffffffffu, give, o);
    }
  }
  return v[0];
}

// M fours of key channels per thread, R lanes per value column (4 M R >= d), blocks of BT tokens.
template <int M, int R, int BT, int KIND, typename TX>
__global__ void __launch_bounds__(DR_THREADS) delta_scan_kernel(
    const TX* __restrict__ x, long long ld, int q_off, int k_off, int v_off, DrGates gates, float* __restrict__ state, long long slot_stride,
    const int* __restrict__ state_slots, const int* __restrict__ cu_seqlens, float* __restrict__ out, int H, int G, int d, int e,
    float q_scale, float unit_eps, int vec) {
  ts_pdl_prologue();
  constexpr bool CHANNEL = KIND == DR_CHANNEL, LINEAR = KIND == DR_LINEAR;
  constexpr int COLS = DR_THREADS / R;  // value columns of this CTA
  constexpr int DPAD = 4 * M * R;
  constexpr int TB = dr_round_tokens(DPAD, BT);
  constexpr int NB = TB / BT;           // blocks of a round
  constexpr int PF = (TB * DPAD + DR_THREADS - 1) / DR_THREADS;  // staged entries per thread and round
  constexpr int PFV = (TB * COLS + DR_THREADS - 1) / DR_THREADS;
  constexpr int NA = BT * (BT - 1) / 2, NS = dr_sums(BT);
  static_assert(TB % BT == 0 && PF <= 16 && NS <= 32, "rounds are whole blocks");
  __shared__ __align__(16) float qs[TB * DPAD];  // q as it came, then q~
  __shared__ __align__(16) float ks[TB * DPAD];  // k, then k~
  __shared__ __align__(16) float gs[TB * DPAD];  // the decays (CHANNEL), then k'
  __shared__ __align__(16) float ge[NB * DPAD];  // G_last of every block
  __shared__ float vs[TB * COLS];
  __shared__ float g1[TB], bs[TB], coef[NB][NS - 2 * BT];
  const int b = blockIdx.x, h = blockIdx.y;
  const int t_begin = cu_seqlens[b], t_end = cu_seqlens[b + 1];
  if (t_end <= t_begin) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int r = tid % R, cl = tid / R;
  const int col = blockIdx.z * COLS + cl;
  const bool live = col < e;
  const int hk = h / (H / G);

  float S[4 * M];
  float* sp = state + (size_t)state_slots[b] * slot_stride + ((size_t)h * e + (live ? col : 0)) * d;
  if (vec) {  // d is a multiple of four and every column starts on a 16-byte boundary
#pragma unroll
    for (int m = 0; m < M; ++m) {
      const int i = 4 * (r + R * m);
      const float4 f = live && i < d ? *reinterpret_cast<const float4*>(sp + i) : make_float4(0.f, 0.f, 0.f, 0.f);
      S[4 * m + 0] = f.x, S[4 * m + 1] = f.y, S[4 * m + 2] = f.z, S[4 * m + 3] = f.w;
    }
  } else {
#pragma unroll
    for (int m = 0; m < M; ++m)
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const int i = 4 * (r + R * m) + c;
        S[4 * m + c] = (live && i < d) ? sp[i] : 0.f;
      }
  }
  const float decay_rate = gates.raw ? expf(gates.a_log[h]) : 0.f;
  const float bias_h = gates.raw && !CHANNEL ? gates.dt_bias[h] : 0.f;

  // What a thread fetches of a round: entries tid, tid + 128, ... of the round's [tokens x DPAD] q, k and decay rows and of its
  // [tokens x COLS] values, and (threads 0 .. tokens - 1) the write strength (and decay) of one token.  The next round's values
  // are asked for before this round's updates begin and wait in registers until these are done.
  float pq[PF], pk[PF], pg[CHANNEL ? PF : 1], pv[PFV], pb = 0.f, pa = 0.f;
  auto fetch = [&](int t0) {
    const int nt = min(TB, t_end - t0);
#pragma unroll
    for (int u = 0; u < PF; ++u) {
      const int i = tid + u * DR_THREADS, tt = i / DPAD, c = i - tt * DPAD;
      const bool ok = tt < nt && c < d;
      const TX* row = x + (size_t)(t0 + (ok ? tt : 0)) * ld + hk * d + (ok ? c : 0);
      pq[u] = ok ? ts_to_float(row[q_off]) : 0.f;
      pk[u] = ok ? ts_to_float(row[k_off]) : 0.f;
      if (LINEAR && ok && c < 2 * gates.half) {  // entry c turns with its partner half a rotated width away
        const bool low = c < gates.half;
        const int other = low ? gates.half : -gates.half;
        const float2 cs = gates.rotation[(size_t)(t0 + tt) * gates.half + (low ? c : c - gates.half)];
        const float sn = low ? -cs.y : cs.y;
        pq[u] = pq[u] * cs.x + ts_to_float(row[q_off + other]) * sn;
        pk[u] = pk[u] * cs.x + ts_to_float(row[k_off + other]) * sn;
      }
      if (CHANNEL) pg[u] = ok ? gates.decay[(size_t)(t0 + tt) * gates.ld_decay + (size_t)h * d + c] : 1.f;
    }
#pragma unroll
    for (int u = 0; u < PFV; ++u) {
      const int i = tid + u * DR_THREADS, tt = i / COLS, c = i - tt * COLS;
      const int vc = blockIdx.z * COLS + c;
      const bool ok = tt < nt && vc < e;
      pv[u] = ok ? ts_to_float(x[(size_t)(t0 + tt) * ld + v_off + h * e + vc]) : 0.f;
    }
    if (tid < nt) {
      const size_t at = (size_t)(t0 + tid) * gates.ld_beta + h;
      if (!LINEAR) pb = gates.beta_bf16 ? __bfloat162float(((const __nv_bfloat16*)gates.beta)[at]) : ((const float*)gates.beta)[at];
      if (!CHANNEL) pa = gates.decay[(size_t)(t0 + tid) * gates.ld_decay + h];
    }
  };
  fetch(t_begin);

  for (int t0 = t_begin; t0 < t_end; t0 += TB) {
    const int nt = min(TB, t_end - t0);
    __syncthreads();  // the round before is read out
    // tokens beyond the portion's end write nothing into the state: k = 0, beta = 0, decay 1
#pragma unroll
    for (int u = 0; u < PF; ++u) {
      const int i = tid + u * DR_THREADS;
      if (i < TB * DPAD) {
        qs[i] = pq[u], ks[i] = pk[u];
        if (CHANNEL) {
          const int c = i % DPAD;
          gs[i] = gates.raw && c < d && i / DPAD < nt ? dr_decay(pg[u], gates.dt_bias[h * d + c], decay_rate) : pg[u];
        }
      }
    }
#pragma unroll
    for (int u = 0; u < PFV; ++u) {
      const int i = tid + u * DR_THREADS;
      if (i < TB * COLS) vs[i] = pv[u];
    }
    if (tid < TB) {
      bs[tid] = tid >= nt ? 0.f : LINEAR ? 1.f : 1.f / (1.f + expf(-pb));
      if (!CHANNEL) g1[tid] = tid >= nt ? 1.f : gates.raw ? dr_decay(pa, bias_h, decay_rate) : pa;
    }
    __syncthreads();
    if (t0 + TB < t_end) fetch(t0 + TB);
    // a warp per block: the sums over the key channels, then the block's rows
    for (int blk = warp; blk < NB; blk += DR_THREADS / 32) {
      float* qb = qs + blk * BT * DPAD;
      float* kb = ks + blk * BT * DPAD;
      float* gb = gs + blk * BT * DPAD;
      float sum[32];
#pragma unroll
      for (int i = 0; i < 32; ++i) sum[i] = 0.f;
      float gt[BT];
      if (!CHANNEL) {
#pragma unroll
        for (int i = 0; i < BT; ++i) gt[i] = g1[blk * BT + i];
      }
#pragma unroll(DPAD >= 128 ? 1 : 2)
      for (int c = lane; c < DPAD; c += 32) {
        float k[BT], q[BT];
#pragma unroll
        for (int i = 0; i < BT; ++i) {
          k[i] = kb[i * DPAD + c], q[i] = qb[i * DPAD + c];
          if (CHANNEL) gt[i] = gb[i * DPAD + c];
          sum[i] = fmaf(k[i], k[i], sum[i]);
          sum[BT + i] = fmaf(q[i], q[i], sum[BT + i]);
        }
#pragma unroll
        for (int j = 0; j < BT; ++j) {
          float w = k[j];  // k_j as it has decayed by token i
#pragma unroll
          for (int i = j; i < BT; ++i) {
            if (i > j) {
              w *= gt[i];
              sum[2 * BT + i * (i - 1) / 2 + j] = fmaf(k[i], w, sum[2 * BT + i * (i - 1) / 2 + j]);
            }
            sum[2 * BT + NA + i * (i + 1) / 2 + j] = fmaf(q[i], w, sum[2 * BT + NA + i * (i + 1) / 2 + j]);
          }
        }
      }
      float total = 0.f;
      if (NS > 8) {
        total = dr_scatter_sum<NS>(sum, lane);
      } else {
#pragma unroll
        for (int i = 0; i < NS; ++i) {
          const float w = ts_warp_sum(sum[i]);
          if (lane == i) total = w;
        }
      }
      // lanes 0 .. BT - 1: the factor of k_i, the next BT: of q_i; the others: their entry of A or B times the factors of its rows
      const float own = (lane < BT ? 1.f : q_scale) / sqrtf(!LINEAR && lane < 2 * BT ? total + unit_eps : 1.f);
      int i = 0, j = 0;
      bool of_q = false;
#pragma unroll
      for (int ii = 0; ii < BT; ++ii)
#pragma unroll
        for (int jj = 0; jj <= ii; ++jj) {
          if (jj < ii && lane == 2 * BT + ii * (ii - 1) / 2 + jj) i = ii, j = jj, of_q = false;
          if (lane == 2 * BT + NA + ii * (ii + 1) / 2 + jj) i = ii, j = jj, of_q = true;
        }
      const float f = __shfl_sync(0xffffffffu, own, of_q ? BT + i : i) * __shfl_sync(0xffffffffu, own, j);
      if (lane >= 2 * BT && lane < NS) coef[blk][lane - 2 * BT] = total * f;
      float mk[BT], mq[BT];
#pragma unroll
      for (int ii = 0; ii < BT; ++ii) {
        mk[ii] = __shfl_sync(0xffffffffu, own, ii);
        mq[ii] = __shfl_sync(0xffffffffu, own, BT + ii);
      }
#pragma unroll(DPAD >= 128 ? 1 : 2)
      for (int c = lane; c < DPAD; c += 32) {
        float k[BT], w = 1.f;
#pragma unroll
        for (int ii = 0; ii < BT; ++ii) {
          if (CHANNEL) gt[ii] = gb[ii * DPAD + c];
          w *= gt[ii];
          k[ii] = kb[ii * DPAD + c] * mk[ii];
          kb[ii * DPAD + c] = k[ii] * w;
          qb[ii * DPAD + c] *= mq[ii] * w;
        }
        ge[blk * DPAD + c] = w;
        w = 1.f;
#pragma unroll
        for (int ii = BT - 1; ii >= 0; --ii) {
          gb[ii * DPAD + c] = k[ii] * w;
          w *= gt[ii];
        }
      }
    }
    __syncthreads();
    for (int blk = 0; blk * BT < nt; ++blk) {
      const float4* k4 = reinterpret_cast<const float4*>(ks + blk * BT * DPAD) + r;
      const float4* q4 = reinterpret_cast<const float4*>(qs + blk * BT * DPAD) + r;
      const float4* e4 = reinterpret_cast<const float4*>(gs + blk * BT * DPAD) + r;
      const float4* g4 = reinterpret_cast<const float4*>(ge + blk * DPAD) + r;
      float sk[BT], sq[BT];
#pragma unroll
      for (int i = 0; i < BT; ++i) sk[i] = 0.f, sq[i] = 0.f;
#pragma unroll
      for (int m = 0; m < M; ++m)
#pragma unroll
        for (int i = 0; i < BT; ++i) {
          const float4 qv = q4[i * (DPAD / 4) + R * m];
          sq[i] = fmaf(S[4 * m + 0], qv.x, sq[i]);
          sq[i] = fmaf(S[4 * m + 1], qv.y, sq[i]);
          sq[i] = fmaf(S[4 * m + 2], qv.z, sq[i]);
          sq[i] = fmaf(S[4 * m + 3], qv.w, sq[i]);
          if (!LINEAR) {
            const float4 kv = k4[i * (DPAD / 4) + R * m];
            sk[i] = fmaf(S[4 * m + 0], kv.x, sk[i]);
            sk[i] = fmaf(S[4 * m + 1], kv.y, sk[i]);
            sk[i] = fmaf(S[4 * m + 2], kv.z, sk[i]);
            sk[i] = fmaf(S[4 * m + 3], kv.w, sk[i]);
          }
        }
#pragma unroll
      for (int o = R >> 1; o > 0; o >>= 1)
#pragma unroll
        for (int i = 0; i < BT; ++i) {
          if (!LINEAR) sk[i] += __shfl_xor_sync(0xffffffffu, sk[i], o);
          sq[i] += __shfl_xor_sync(0xffffffffu, sq[i], o);
        }
      float u[BT];
#pragma unroll
      for (int i = 0; i < BT; ++i) {
        float rest = vs[(blk * BT + i) * COLS + cl] - sk[i];
#pragma unroll
        for (int j = 0; j < (LINEAR ? 0 : i); ++j) rest = fmaf(-coef[blk][i * (i - 1) / 2 + j], u[j], rest);
        u[i] = bs[blk * BT + i] * rest;
      }
#pragma unroll
      for (int m = 0; m < M; ++m) {
        const float4 gv = g4[R * m];
        S[4 * m + 0] *= gv.x, S[4 * m + 1] *= gv.y, S[4 * m + 2] *= gv.z, S[4 * m + 3] *= gv.w;
#pragma unroll
        for (int i = 0; i < BT; ++i) {
          const float4 ev = e4[i * (DPAD / 4) + R * m];
          S[4 * m + 0] = fmaf(ev.x, u[i], S[4 * m + 0]);
          S[4 * m + 1] = fmaf(ev.y, u[i], S[4 * m + 1]);
          S[4 * m + 2] = fmaf(ev.z, u[i], S[4 * m + 2]);
          S[4 * m + 3] = fmaf(ev.w, u[i], S[4 * m + 3]);
        }
      }
#pragma unroll
      for (int i = 0; i < BT; ++i) {
        const int t = t0 + blk * BT + i;
        float o = sq[i];
#pragma unroll
        for (int j = 0; j <= i; ++j) o = fmaf(coef[blk][NA + i * (i + 1) / 2 + j], u[j], o);
        if (live && i % R == r && t < t_end) out[(size_t)t * H * e + (size_t)h * e + col] = o;
      }
    }
  }
  if (live) {
    if (vec) {
#pragma unroll
      for (int m = 0; m < M; ++m) {
        const int i = 4 * (r + R * m);
        if (i < d) *reinterpret_cast<float4*>(sp + i) = make_float4(S[4 * m + 0], S[4 * m + 1], S[4 * m + 2], S[4 * m + 3]);
      }
    } else {
#pragma unroll
      for (int m = 0; m < M; ++m)
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          const int i = 4 * (r + R * m) + c;
          if (i < d) sp[i] = S[4 * m + c];
        }
    }
  }
}

template <int M, int R, int BT, int KIND, typename TX>
static int dr_launch(const TX* x, long long ld, int q_off, int k_off, int v_off, const DrGates& gates, float* state, long long slot_stride,
                     const int* state_slots, const int* cu_seqlens, float* out, int B, int H, int G, int d, int e, float q_scale, float unit_eps,
                     cudaStream_t s) {
  constexpr int COLS = DR_THREADS / R;
  const dim3 grid(B, H, (e + COLS - 1) / COLS);
  if (grid.z > 65535) return TS_ERR_UNSUPPORTED_SIZE;
  const int vec = d % 4 == 0 && slot_stride % 4 == 0 && (uintptr_t)state % 16 == 0;
  return ts_launch(delta_scan_kernel<M, R, BT, KIND, TX>, grid, dim3(DR_THREADS), 0, s, x, ld, q_off, k_off, v_off, gates, state, slot_stride,
                   state_slots, cu_seqlens, out, H, G, d, e, q_scale, unit_eps, vec);
}

// The same for portions with key widths up to 128, its two halves side by side: eight warps, of which the last four
// prepare a round (16 tokens, a block of four each) while the first four run the updates of the round before.  A preparing
// warp keeps its block's q, k and decays in registers, its lanes over the key channels: sums, factors and the block's
// rows go to shared memory from there, and the rows of its next block are asked for right behind.  The updating
// threads hold the state, CPT value columns each: a row that is read from shared memory then serves CPT columns (those
// reads, 16 bytes a lane, are what the updates wait for: with one column a thread they kept shared memory busy for more than
// half of the time).  The sums of a block are added up by halving exchanges, so that a lane ends with one of them.  Two
// buffers of shared memory, one barrier a round.
//
// Measured (2,048 tokens, 16 / 32 heads of 64 x 128; 8 x 1,024 tokens, 16 heads): token by token 0.72 / 0.73 ms; blocks of four
// in one kind of thread 0.43 / 0.61, 0.81; the two kinds with one column a thread 0.30 / 0.42, 0.83; two columns, 16
// lanes a column, the loads of two blocks in flight 0.23 / 0.34, 0.61.
#define DP_BT 4
#define DP_NB 4  // blocks of a round: one per preparing warp

template <int M, int R, int CT, int CPT>
struct DpBuffer {
  static constexpr int COLS = CT / R * CPT, DPAD = 4 * M * R;
  float kt[DP_NB][DP_BT][DPAD], qt[DP_NB][DP_BT][DPAD], ke[DP_NB][DP_BT][DPAD], ge[DP_NB][DPAD];
  float4 v[DP_NB][COLS];   // the block's four values of a column
  float4 coef[DP_NB][4];   // A_10 A_20 A_21 A_30 | A_31 A_32 B_00 B_10 | B_11 B_20 B_21 B_22 | B_30 B_31 B_32 B_33
  float4 beta[DP_NB];
};

// Sums of N values over the R >= N lanes of a column: value i ends in the lanes from i * R / N on.
template <int N, int R>
__device__ __forceinline__ float dp_scatter(float (&v)[N], int r) {
  int o = R / 2;
#pragma unroll
  for (int n = N / 2; n >= 1; n >>= 1, o >>= 1) {
    const bool up = (r & o) != 0;
#pragma unroll
    for (int i = 0; i < n; ++i) {
      const float give = up ? v[i] : v[i + n], keep = up ? v[i + n] : v[i];
      v[i] = keep + __shfl_xor_sync(0xffffffffu, give, o);
    }
  }
  float t = v[0];
#pragma unroll
  for (int w = R / N / 2; w > 0; w >>= 1) t += __shfl_xor_sync(0xffffffffu, t, w);
  return t;
}

template <int M, int R, int CT, int CPT, int KIND, typename TX>
__global__ void __launch_bounds__(CT + 128, 2) delta_portion_kernel(
    const TX* __restrict__ x, long long ld, int q_off, int k_off, int v_off, DrGates gates, float* __restrict__ state, long long slot_stride,
    const int* __restrict__ state_slots, const int* __restrict__ cu_seqlens, float* __restrict__ out, int H, int G, int d, int e,
    float q_scale, float unit_eps, int vec) {
  ts_pdl_prologue();
  constexpr bool CHANNEL = KIND == DR_CHANNEL, LINEAR = KIND == DR_LINEAR;
  using Buffer = DpBuffer<M, R, CT, CPT>;
  constexpr int COLS = Buffer::COLS, DPAD = Buffer::DPAD, BT = DP_BT, TB = DP_NB * BT;
  // (LINEAR: an even number of channels, so that the two of a rotated pair sit in one lane)
  constexpr int NCH = LINEAR && DPAD <= 32 ? 2 : (DPAD + 31) / 32, NV = (BT * COLS + 31) / 32;  // channels and values per preparing lane and block
  constexpr int NA = BT * (BT - 1) / 2, NS = dr_sums(BT), SA = 2 * BT + NA, SB = LINEAR ? 0 : SA;  // SB: where B begins among the sums
  extern __shared__ __align__(16) unsigned char dp_smem[];
  Buffer* const buffers = reinterpret_cast<Buffer*>(dp_smem);
  const int b = blockIdx.x, h = blockIdx.y;
  const int t_begin = cu_seqlens[b], t_end = cu_seqlens[b + 1];
  if (t_end <= t_begin) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const bool prepares = warp >= CT / 32;
  const int col0 = blockIdx.z * COLS;
  const int rounds = (t_end - t_begin + TB - 1) / TB;

  // ---- the updating threads' part: CPT columns each, COLS / CPT apart
  const int r = tid % R, cl = (tid % CT) / R;
  float S[CPT][4 * M];
  float* sp[CPT];
  bool live[CPT];
#pragma unroll
  for (int p = 0; p < CPT; ++p) {
    const int col = col0 + cl + p * (COLS / CPT);
    live[p] = !prepares && col < e;
    sp[p] = state + (size_t)state_slots[b] * slot_stride + ((size_t)h * e + (live[p] ? col : 0)) * d;
    if (vec) {  // d is a multiple of four and every column starts on a 16-byte boundary
#pragma unroll
      for (int m = 0; m < M; ++m) {
        const int i = 4 * (r + R * m);
        const float4 f = live[p] && i < d ? *reinterpret_cast<const float4*>(sp[p] + i) : make_float4(0.f, 0.f, 0.f, 0.f);
        S[p][4 * m + 0] = f.x, S[p][4 * m + 1] = f.y, S[p][4 * m + 2] = f.z, S[p][4 * m + 3] = f.w;
      }
    } else {
#pragma unroll
      for (int m = 0; m < M; ++m)
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          const int i = 4 * (r + R * m) + c;
          S[p][4 * m + c] = (live[p] && i < d) ? sp[p][i] : 0.f;
        }
    }
  }
  constexpr int KD = LINEAR ? 0 : BT;       // sums of a block: for every column S^T k~ of the four tokens (not LINEAR), then S^T q~
  constexpr int NC = KD + BT, NVAL = NC * CPT;
  constexpr bool SCATTER = R >= NVAL;
  constexpr int SHARE = SCATTER ? R / NVAL : 1;
  // the column and token whose read-out this lane writes (SCATTER)
  const int w_idx = r / SHARE, w_p = w_idx / NC, w_i = w_idx % NC - KD;
  bool writes = false;
  int w_col = col0;
#pragma unroll
  for (int p = 0; p < CPT; ++p)
    if (p == w_p) writes = live[p] && w_i >= 0 && r % SHARE == 0, w_col = col0 + cl + p * (COLS / CPT);
  const size_t out_row = (size_t)H * e;
  float* const w_out = out + (size_t)(t_begin + (w_i >= 0 ? w_i : 0)) * out_row + (size_t)h * e + w_col;
  auto update = [&](int n) {
    const Buffer& buf = buffers[n & 1];
    const int t0 = n * TB, nt = min(TB, t_end - t_begin - t0);
#pragma unroll 2  // the loads of two blocks in flight
    for (int blk = 0; blk < DP_NB; ++blk) {
      if (blk * BT >= nt) break;
      const float4* k4 = reinterpret_cast<const float4*>(buf.kt[blk][0]) + r;
      const float4* q4 = reinterpret_cast<const float4*>(buf.qt[blk][0]) + r;
      const float4* e4 = reinterpret_cast<const float4*>(buf.ke[blk][0]) + r;
      const float4* g4 = reinterpret_cast<const float4*>(buf.ge[blk]) + r;
      float sums[NVAL];
#pragma unroll
      for (int i = 0; i < NVAL; ++i) sums[i] = 0.f;
#pragma unroll
      for (int m = 0; m < M; ++m)
#pragma unroll
        for (int i = 0; i < BT; ++i) {
          const float4 qv = q4[i * (DPAD / 4) + R * m];
          const float4 kv = LINEAR ? qv : k4[i * (DPAD / 4) + R * m];
#pragma unroll
          for (int p = 0; p < CPT; ++p) {
            float &a = sums[p * NC + i], &z = sums[p * NC + KD + i];
            if (!LINEAR) {
              a = fmaf(S[p][4 * m + 0], kv.x, a);
              a = fmaf(S[p][4 * m + 1], kv.y, a);
              a = fmaf(S[p][4 * m + 2], kv.z, a);
              a = fmaf(S[p][4 * m + 3], kv.w, a);
            }
            z = fmaf(S[p][4 * m + 0], qv.x, z);
            z = fmaf(S[p][4 * m + 1], qv.y, z);
            z = fmaf(S[p][4 * m + 2], qv.z, z);
            z = fmaf(S[p][4 * m + 3], qv.w, z);
          }
        }
      const float4 bb = buf.beta[blk], c0 = buf.coef[blk][0], c1 = buf.coef[blk][1], c2 = buf.coef[blk][2], c3 = buf.coef[blk][3];
      float mine = 0.f;
      if (SCATTER) {
        mine = dp_scatter<SCATTER ? NVAL : 1, R>(reinterpret_cast<float (&)[SCATTER ? NVAL : 1]>(sums), r);
      } else {
#pragma unroll
        for (int o = R >> 1; o > 0; o >>= 1)
#pragma unroll
          for (int i = 0; i < NVAL; ++i) sums[i] += __shfl_xor_sync(0xffffffffu, sums[i], o);
      }
      float u[CPT][BT];
#pragma unroll
      for (int p = 0; p < CPT; ++p) {
        const float4 vv = buf.v[blk][cl + p * (COLS / CPT)];
        float sk[BT];
#pragma unroll
        for (int i = 0; i < BT; ++i) sk[i] = LINEAR ? 0.f : SCATTER ? __shfl_sync(0xffffffffu, mine, (p * NC + i) * SHARE, R) : sums[p * NC + i];
        if (LINEAR) {
          u[p][0] = vv.x, u[p][1] = vv.y, u[p][2] = vv.z, u[p][3] = vv.w;
        } else {
          u[p][0] = bb.x * (vv.x - sk[0]);
          u[p][1] = bb.y * fmaf(-c0.x, u[p][0], vv.y - sk[1]);
          u[p][2] = bb.z * fmaf(-c0.z, u[p][1], fmaf(-c0.y, u[p][0], vv.z - sk[2]));
          u[p][3] = bb.w * fmaf(-c1.y, u[p][2], fmaf(-c1.x, u[p][1], fmaf(-c0.w, u[p][0], vv.w - sk[3])));
        }
      }
#pragma unroll
      for (int m = 0; m < M; ++m) {
        const float4 gv = LINEAR ? make_float4(c0.x, c0.x, c0.x, c0.x) : g4[R * m];
        const float4 a = e4[R * m], f = e4[(DPAD / 4) + R * m], q = e4[2 * (DPAD / 4) + R * m], w = e4[3 * (DPAD / 4) + R * m];
#pragma unroll
        for (int p = 0; p < CPT; ++p) {
          S[p][4 * m + 0] = fmaf(w.x, u[p][3], fmaf(q.x, u[p][2], fmaf(f.x, u[p][1], fmaf(a.x, u[p][0], gv.x * S[p][4 * m + 0]))));
          S[p][4 * m + 1] = fmaf(w.y, u[p][3], fmaf(q.y, u[p][2], fmaf(f.y, u[p][1], fmaf(a.y, u[p][0], gv.y * S[p][4 * m + 1]))));
          S[p][4 * m + 2] = fmaf(w.z, u[p][3], fmaf(q.z, u[p][2], fmaf(f.z, u[p][1], fmaf(a.z, u[p][0], gv.z * S[p][4 * m + 2]))));
          S[p][4 * m + 3] = fmaf(w.w, u[p][3], fmaf(q.w, u[p][2], fmaf(f.w, u[p][1], fmaf(a.w, u[p][0], gv.w * S[p][4 * m + 3]))));
        }
      }
      auto reads = [&](const float (&x)[BT], int i) {
        return i == 0 ? c1.z * x[0]
             : i == 1 ? fmaf(c2.x, x[1], c1.w * x[0])
             : i == 2 ? fmaf(c2.w, x[2], fmaf(c2.z, x[1], c2.y * x[0]))
                      : fmaf(c3.w, x[3], fmaf(c3.z, x[2], fmaf(c3.y, x[1], c3.x * x[0])));
      };
      if (SCATTER) {  // the lane that holds S^T q~_i of a column writes its o_i
        float x[BT];
#pragma unroll
        for (int i = 0; i < BT; ++i) x[i] = CPT == 2 && w_p == 1 ? u[CPT - 1][i] : u[0][i];
        const float o0 = reads(x, 0), o1 = reads(x, 1), o2 = reads(x, 2), o3 = reads(x, 3);
        const float add = w_i == 0 ? o0 : w_i == 1 ? o1 : w_i == 2 ? o2 : o3;
        if (writes && blk * BT + w_i < nt) w_out[(size_t)(t0 + blk * BT) * out_row] = mine + add;
      } else {
#pragma unroll
        for (int p = 0; p < CPT; ++p)
#pragma unroll
          for (int i = 0; i < BT; ++i)
            if (live[p] && i % R == r && blk * BT + i < nt)
              out[(size_t)(t_begin + t0 + blk * BT + i) * out_row + (size_t)h * e + col0 + cl + p * (COLS / CPT)] = sums[p * NC + KD + i] + reads(u[p], i);
      }
    }
  };

  // ---- the preparing warps' part
  const int blk = warp - CT / 32;
  const int hk = h / (H / G);
  const float decay_rate = gates.raw ? expf(gates.a_log[h]) : 0.f;
  // (what is fetched stays as it came until it is used: a conversion would wait for the load)
  TX fq[NCH][BT], fk[NCH][BT], fv[NV];
  float g[CHANNEL ? NCH : 1][BT], pb = 0.f;
  float2 turn[LINEAR ? NCH / 2 : 1][BT];
  // the key channel of a lane's entry n2: lane + 32 n2, or (LINEAR) such that entries 2 m and 2 m + 1 are a rotated pair while there
  // are any left, then the channels behind the rotated ones
  auto channel = [&](int n2) {
    if (!LINEAR) return lane + 32 * n2;
    const int pair = lane + 32 * (n2 >> 1);
    return pair < gates.half ? pair + (n2 & 1) * gates.half : 2 * pair + (n2 & 1);
  };
  auto fetch = [&](int n) {
    const int t0 = t_begin + n * TB + blk * BT;
    // a token beyond the portion's end writes nothing into the state: k = 0, beta = 0, decay 1
#pragma unroll
    for (int i = 0; i < BT; ++i) {
      const bool there = t0 + i < t_end;
      const TX* row = x + (size_t)(there ? t0 + i : t_begin) * ld + hk * d;
      const float* drow = gates.decay + (size_t)(there ? t0 + i : t_begin) * gates.ld_decay + (CHANNEL ? (size_t)h * d : h);
#pragma unroll
      for (int n2 = 0; n2 < NCH; ++n2) {
        const int c = channel(n2);
        const bool ok = there && c < d;
        fq[n2][i] = ok ? row[q_off + c] : TX(0.f);
        fk[n2][i] = ok ? row[k_off + c] : TX(0.f);
        if (LINEAR && n2 % 2 == 0) turn[n2 / 2][i] = ok && c < gates.half ? gates.rotation[(size_t)(t0 + i) * gates.half + c] : make_float2(1.f, 0.f);
        if (CHANNEL) g[n2][i] = ok ? drow[c] : 1.f;
      }
      if (!CHANNEL) g[0][i] = there ? drow[0] : 1.f;
    }
#pragma unroll
    for (int n2 = 0; n2 < NV; ++n2) {
      const int at = lane + 32 * n2, i = at / COLS, c = at % COLS;
      fv[n2] = at < BT * COLS && t0 + i < t_end && col0 + c < e ? x[(size_t)(t0 + i) * ld + v_off + h * e + col0 + c] : TX(0.f);
    }
    if (!LINEAR && lane < BT && t0 + lane < t_end) {
      const size_t at = (size_t)(t0 + lane) * gates.ld_beta + h;
      pb = gates.beta_bf16 ? __bfloat162float(((const __nv_bfloat16*)gates.beta)[at]) : ((const float*)gates.beta)[at];
    }
  };
  auto prepare = [&](int n) {
    Buffer& buf = buffers[n & 1];
    const int t0 = t_begin + n * TB + blk * BT;
    if (t0 >= t_end) return;
    if (gates.raw) {
#pragma unroll
      for (int n2 = 0; n2 < (CHANNEL ? NCH : 1); ++n2) {
        const int c = lane + 32 * n2;
        const float bias = !CHANNEL ? gates.dt_bias[h] : c < d ? gates.dt_bias[h * d + c] : 0.f;
#pragma unroll
        for (int i = 0; i < BT; ++i)
          if (t0 + i < t_end && (!CHANNEL || c < d)) g[n2][i] = dr_decay(g[n2][i], bias, decay_rate);
      }
    }
    float q[NCH][BT], k[NCH][BT];
#pragma unroll
    for (int n2 = 0; n2 < NCH; ++n2)
#pragma unroll
      for (int i = 0; i < BT; ++i) q[n2][i] = ts_to_float(fq[n2][i]), k[n2][i] = ts_to_float(fk[n2][i]);
    if (LINEAR && gates.half > 0) {
#pragma unroll
      for (int n2 = 0; n2 + 1 < NCH; n2 += 2)
#pragma unroll
        for (int i = 0; i < BT; ++i) {
          const float2 cs = turn[LINEAR ? n2 / 2 : 0][i];
          const float qu = q[n2][i], ku = k[n2][i];
          q[n2][i] = qu * cs.x - q[n2 + 1][i] * cs.y, q[n2 + 1][i] = q[n2 + 1][i] * cs.x + qu * cs.y;
          k[n2][i] = ku * cs.x - k[n2 + 1][i] * cs.y, k[n2 + 1][i] = k[n2 + 1][i] * cs.x + ku * cs.y;
        }
    }
    float sum[32];
#pragma unroll
    for (int i = 0; i < 32; ++i) sum[i] = 0.f;
#pragma unroll
    for (int n2 = 0; n2 < NCH; ++n2) {
      const float (&gt)[BT] = g[CHANNEL ? n2 : 0];
#pragma unroll
      for (int i = 0; i < BT; ++i) {
        if (LINEAR) continue;
        sum[i] = fmaf(k[n2][i], k[n2][i], sum[i]);
        sum[BT + i] = fmaf(q[n2][i], q[n2][i], sum[BT + i]);
      }
#pragma unroll
      for (int j = 0; j < BT; ++j) {
        float w = k[n2][j];  // k_j as it has decayed by token i
#pragma unroll
        for (int i = j; i < BT; ++i) {
          if (i > j) {
            w *= gt[i];
            if (!LINEAR) sum[2 * BT + i * (i - 1) / 2 + j] = fmaf(k[n2][i], w, sum[2 * BT + i * (i - 1) / 2 + j]);
          }
          sum[SB + i * (i + 1) / 2 + j] = fmaf(q[n2][i], w, sum[SB + i * (i + 1) / 2 + j]);
        }
      }
    }
    const float total = dr_scatter_sum<LINEAR ? NS - SA : NS>(sum, lane);
    // lanes 0 .. 3: the factor of k_i, 4 .. 7: of q_i; the others: their entry of A or B times the factors of its rows
    const float own = (lane < BT ? 1.f : q_scale) / sqrtf(lane < 2 * BT ? total + unit_eps : 1.f);
    float mk[BT], mq[BT];
#pragma unroll
    for (int i = 0; i < BT; ++i) {
      mk[i] = LINEAR ? 1.f : __shfl_sync(0xffffffffu, own, i);
      mq[i] = LINEAR ? q_scale : __shfl_sync(0xffffffffu, own, BT + i);
    }
    float f = 0.f;
#pragma unroll
    for (int i = 0; i < BT; ++i)
#pragma unroll
      for (int j = 0; j <= i; ++j) {
        if (j < i && lane == 2 * BT + i * (i - 1) / 2 + j) f = mk[i] * mk[j];
        if (lane == 2 * BT + NA + i * (i + 1) / 2 + j) f = mq[i] * mk[j];
      }
    if (LINEAR) {  // no A: its first place takes the block's decay
      if (lane < NS - SA) reinterpret_cast<float*>(buf.coef[blk])[NA + lane] = total * q_scale;
      if (lane == 16) buf.coef[blk][0].x = g[0][0] * g[0][1] * g[0][2] * g[0][3];
    } else if (lane >= 2 * BT && lane < NS) {
      reinterpret_cast<float*>(buf.coef[blk])[lane - 2 * BT] = total * f;
    }
    if (!LINEAR && lane < BT) reinterpret_cast<float*>(&buf.beta[blk])[lane] = t0 + lane < t_end ? 1.f / (1.f + expf(-pb)) : 0.f;
#pragma unroll
    for (int n2 = 0; n2 < NCH; ++n2) {
      const int c = channel(n2);
      const float (&gt)[BT] = g[CHANNEL ? n2 : 0];
      if ((DPAD % 32 == 0 && !LINEAR) || c < DPAD) {
        float w = 1.f, back = 1.f;
#pragma unroll
        for (int i = 0; i < BT; ++i) {
          w *= gt[i];
          k[n2][i] *= mk[i];
          if (!LINEAR) buf.kt[blk][i][c] = k[n2][i] * w;
          buf.qt[blk][i][c] = q[n2][i] * mq[i] * w;
        }
        if (!LINEAR) buf.ge[blk][c] = w;
#pragma unroll
        for (int i = BT - 1; i >= 0; --i) {
          buf.ke[blk][i][c] = k[n2][i] * back;
          back *= gt[i];
        }
      }
    }
#pragma unroll
    for (int n2 = 0; n2 < NV; ++n2) {
      const int at = lane + 32 * n2, i = at / COLS, c = at % COLS;
      if (at < BT * COLS) reinterpret_cast<float*>(&buf.v[blk][c])[i] = ts_to_float(fv[n2]);
    }
  };

  if (prepares) {
    fetch(0);
    prepare(0);
    fetch(1);
  }
  __syncthreads();
  for (int n = 0; n < rounds; ++n) {
    if (!prepares) {
      update(n);
    } else if (n + 1 < rounds) {
      prepare(n + 1);
      fetch(n + 2);
    }
    __syncthreads();
  }
#pragma unroll
  for (int p = 0; p < CPT; ++p) {
    if (!live[p]) continue;
    if (vec) {
#pragma unroll
      for (int m = 0; m < M; ++m) {
        const int i = 4 * (r + R * m);
        if (i < d) *reinterpret_cast<float4*>(sp[p] + i) = make_float4(S[p][4 * m + 0], S[p][4 * m + 1], S[p][4 * m + 2], S[p][4 * m + 3]);
      }
    } else {
#pragma unroll
      for (int m = 0; m < M; ++m)
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          const int i = 4 * (r + R * m) + c;
          if (i < d) sp[p][i] = S[p][4 * m + c];
        }
    }
  }
}

template <int M, int R, int CT, int CPT, int KIND, typename TX>
static int dp_launch(const TX* x, long long ld, int q_off, int k_off, int v_off, const DrGates& gates, float* state, long long slot_stride,
                     const int* state_slots, const int* cu_seqlens, float* out, int B, int H, int G, int d, int e, float q_scale, float unit_eps,
                     cudaStream_t s) {
  constexpr int COLS = CT / R * CPT;
  constexpr size_t smem = 2 * sizeof(DpBuffer<M, R, CT, CPT>);
  const dim3 grid(B, H, (e + COLS - 1) / COLS);
  if (grid.z > 65535) return TS_ERR_UNSUPPORTED_SIZE;
  static bool sized = false;
  if (smem > 48 * 1024 && !sized) {
    const cudaError_t err = cudaFuncSetAttribute(delta_portion_kernel<M, R, CT, CPT, KIND, TX>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (err != cudaSuccess) return (int)err;
    sized = true;
  }
  const int vec = d % 4 == 0 && slot_stride % 4 == 0 && (uintptr_t)state % 16 == 0;
  return ts_launch(delta_portion_kernel<M, R, CT, CPT, KIND, TX>, grid, dim3(CT + 128), smem, s, x, ld, q_off, k_off, v_off, gates, state, slot_stride,
                   state_slots, cu_seqlens, out, H, G, d, e, q_scale, unit_eps, vec);
}

// How the state of one head is cut over threads for key width d: in portions a thread holds 4 or 8 key channels of two value
// columns (of one for narrow keys, in steps of one token 16 channels of one; more where a warp's lanes would not do), and as many
// lanes share a column as that takes: a function of d alone.
template <int KIND, typename TX>
static int dr_dispatch(const TX* x, long long ld, int q_off, int k_off, int v_off, const DrGates& gates, float* state, long long slot_stride,
                       const int* state_slots, const int* cu_seqlens, float* out, int B, int H, int G, int d, int e, float q_scale,
                       float unit_eps, int single, cudaStream_t s) {
#define DR_GO(MM, RR, BB) \
  return dr_launch<MM, RR, BB, KIND, TX>(x, ld, q_off, k_off, v_off, gates, state, slot_stride, state_slots, cu_seqlens, out, B, H, G, d, e, q_scale, unit_eps, s)
  if (single) {
    if (d <= 4) DR_GO(1, 1, 1);
    if (d <= 8) DR_GO(2, 1, 1);
    if (d <= 16) DR_GO(4, 1, 1);
    if (d <= 32) DR_GO(4, 2, 1);
    if (d <= 64) DR_GO(4, 4, 1);
    if (d <= 128) DR_GO(4, 8, 1);
    if (d <= 256) DR_GO(4, 16, 1);
    if (d <= 512) DR_GO(4, 32, 1);
    DR_GO(8, 32, 1);
  }
#define DP_GO(MM, RR, CC, PP) \
  return dp_launch<MM, RR, CC, PP, KIND, TX>(x, ld, q_off, k_off, v_off, gates, state, slot_stride, state_slots, cu_seqlens, out, B, H, G, d, e, q_scale, unit_eps, s)
  if (d <= 8) DP_GO(2, 1, 128, 1);
  if (d <= 16) DP_GO(2, 2, 128, 1);
  if (d <= 32) DP_GO(1, 8, 128, 1);
  if (d <= 64) DP_GO(1, 16, 128, 2);
  if (d <= 128) DP_GO(2, 16, 128, 2);
#undef DP_GO
  if (d <= 256) DR_GO(2, 32, 4);
  if (d <= 512) DR_GO(4, 32, 4);
  DR_GO(8, 32, 2);
#undef DR_GO
}

// beta [T, H] (element type by code, rows ld_beta apart): raw write strengths.  decay: raw entries (raw = 1; a_log and
// dt_bias then make decays of them) or decays (raw = 0), float32, rows ld_decay apart; per_channel = 0: one per
// (token, head), 1: one per (token, head, key channel).  single: every sequence brings one token at most.
TS_EXPORT int ts_delta_scan(const float* x, long long ld, int q_off, int k_off, int v_off, const void* beta, int beta_dtype, long long ld_beta,
                            const float* decay, long long ld_decay, int per_channel, int raw, const float* a_log, const float* dt_bias,
                            float* state, long long slot_stride, const int* state_slots, const int* cu_seqlens, float* out, int B, int H, int G,
                            int d, int e, float q_scale, float unit_eps, int single, void* stream) {
  if (B <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || d <= 0 || e <= 0 || (raw && (a_log == nullptr || dt_bias == nullptr)) ||
      (beta_dtype != TS_DTYPE_F32 && beta_dtype != TS_DTYPE_BF16))
    return TS_ERR_BAD_ARGUMENT;
  if (d > DR_MAX_KEY_DIM || B > 65535 * 16 || H > 65535) return TS_ERR_UNSUPPORTED_SIZE;
  cudaStream_t s = (cudaStream_t)stream;
  const DrGates gates = {beta, decay, a_log, dt_bias, ld_beta, ld_decay, beta_dtype == TS_DTYPE_BF16 ? 1 : 0, raw, nullptr, 0};
  if (per_channel)
    return dr_dispatch<DR_CHANNEL, float>(x, ld, q_off, k_off, v_off, gates, state, slot_stride, state_slots, cu_seqlens, out, B, H, G, d, e, q_scale, unit_eps, single, s);
  return dr_dispatch<DR_HEAD, float>(x, ld, q_off, k_off, v_off, gates, state, slot_stride, state_slots, cu_seqlens, out, B, H, G, d, e, q_scale, unit_eps, single, s);
}

// Retention: S <- decay_h S + k v^T, o = q_scale S^T q per head, with q, k, v columns of x [T, ..] of the compute type, q and k
// rotated as they are read (rotation [T, half, 2] cosines and sines, entry i < half with entry i + half; half = 0: not).
TS_EXPORT int ts_retention_scan(const void* x, int dtype, long long ld, int q_off, int k_off, int v_off, const float* rotation, int half,
                                const float* decay, float* state, long long slot_stride, const int* state_slots, const int* cu_seqlens,
                                float* out, int B, int H, int G, int d, int e, float q_scale, int single, void* stream) {
  if (B <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || d <= 0 || e <= 0 || decay == nullptr || half < 0 || 2 * half > d || (half > 0 && rotation == nullptr))
    return TS_ERR_BAD_ARGUMENT;
  if (d > DR_MAX_KEY_DIM || B > 65535 * 16 || H > 65535) return TS_ERR_UNSUPPORTED_SIZE;
  cudaStream_t s = (cudaStream_t)stream;
  const DrGates gates = {nullptr, decay, nullptr, nullptr, 0, 0, 0, 0, reinterpret_cast<const float2*>(rotation), half};
  if (dtype == TS_DTYPE_F32)
    return dr_dispatch<DR_LINEAR, float>((const float*)x, ld, q_off, k_off, v_off, gates, state, slot_stride, state_slots, cu_seqlens, out, B, H, G, d, e,
                                         q_scale, 0.f, single, s);
  if (dtype == TS_DTYPE_BF16)
    return dr_dispatch<DR_LINEAR, __nv_bfloat16>((const __nv_bfloat16*)x, ld, q_off, k_off, v_off, gates, state, slot_stride, state_slots, cu_seqlens,
                                                 out, B, H, G, d, e, q_scale, 0.f, single, s);
  return TS_ERR_BAD_ARGUMENT;
}

// z[t, h * d + c] <- exp(-exp(a_log[h]) softplus(z[t, h * d + c] + dt_bias[h * d + c])), in place, float32.
__global__ void __launch_bounds__(256) channel_decay_kernel(float* __restrict__ z, long long ld, const float* __restrict__ a_log,
                                                            const float* __restrict__ dt_bias, int T, int H, int d) {
  ts_pdl_prologue();
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= H * d) return;
  const float rate = expf(a_log[c / d]), bias = dt_bias[c];
  for (int t = blockIdx.y; t < T; t += gridDim.y) {
    float* p = z + (size_t)t * ld + c;
    *p = dr_decay(*p, bias, rate);
  }
}

TS_EXPORT int ts_channel_decay(float* z, long long ld, const float* a_log, const float* dt_bias, int T, int H, int d, void* stream) {
  if (T <= 0) return 0;
  if (H <= 0 || d <= 0 || ld < (long long)H * d) return TS_ERR_BAD_ARGUMENT;
  // a few rows per block: a channel's rate and bias are then read once for all of them
  const dim3 grid((H * d + 255) / 256, (unsigned)min((T + 3) / 4, 65535));
  return ts_launch(channel_decay_kernel, grid, dim3(256), 0, (cudaStream_t)stream, z, ld, a_log, dt_bias, T, H, d);
}
