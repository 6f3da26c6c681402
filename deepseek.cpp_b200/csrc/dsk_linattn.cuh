// dsk_linattn.cuh — linear attention with a decayed matrix state per head, in three forms that share their kernels:
//   delta rule (DELTA):  S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q      (g, beta per token and head)
//   plain:               S <- g S + k v^T;  o = S^T q                                       (g fixed per head)
//   mLSTM:               m' = max(f + m, i);  S <- e^(f + m - m') S + e^(i - m') k v^T;  n likewise with k alone (n is one more value
//                        channel whose value is 1);  o = S^T q / (max(|n . q|, e^-m') + 1e-6)         (log gates f, i per token and head)
//
// Portions run it over blocks of kLinBlk tokens (a re-association of the same fp32 sums, no reduced precision).  With S0 the
// state ahead of a block, G_j the product of the decays up to and including token j, and R(j, i) = G_j / G_i:
//   A_ji = beta_j R(j, i) (k_j . k_i)  for i < j,    M_ji = R(j, i) (q_j . k_i)  for i <= j
//   U = (I + A)^-1 W,   w_j = beta_j (v_j - G_j S0^T k_j)            (plain: U = V)
//   o_j = G_j S0^T q_j + sum_i M_ji u_i,    S <- G_end S0 + sum_j R(end, j) k_j u_j^T
// The part that does not depend on the state (A, its inverse, M, the decays) is computed for all blocks of a step at once
// (gdn_prepare / lin_gram / mlstm_gates + mlstm_gram); lin_scan then walks the blocks with the state in registers.  Decay ratios are exponentials of
// sums of the logarithms between the two tokens, so a decay that underflows gives 0 and never 0 / 0, and nothing cancels.
// Steps of up to kLinDecodeTokens tokens run token by token in lin_decode, for the delta rule together with its convolutions,
// unit norms, gates, head norm and output gate.
#pragma once

#include "dsk_hybrid.cuh"

namespace dsk {
namespace hy {

constexpr int kLinBlk = 16;            // tokens per block
constexpr int kLinDecodeTokens = 4;    // steps of at most this many tokens run token by token
constexpr int kConvSpare = 8;          // rows of a convolution history beyond its taps - 1: a step of up to this many tokens writes rows it does not read
// one record per (block, head): inverse, M, and per token G_j, beta_j, R(end, j); then G_end
constexpr int kRecT = 0, kRecM = kLinBlk * kLinBlk, kRecG = 2 * kLinBlk * kLinBlk, kRecB = kRecG + kLinBlk, kRecE = kRecB + kLinBlk, kRecEnd = kRecE + kLinBlk;
constexpr int kRecFloats = kRecEnd + 4;

// value of channel c (of ch, at column off of the rows) at token t after the causal convolution and silu.  hist: ring over
// positions, `ring` rows of ch inputs; positions before the start of the sequence are zero.
__device__ __forceinline__ float conv_silu_at(const float* __restrict__ proj, int ld, int off, int c, int ch, const float* __restrict__ w, int taps,
                                              const float* __restrict__ hist, int ring, int pos0, int t) {
  float acc = 0.f;
  for (int j = 0; j < taps; j++) {
    const int tau = t - (taps - 1) + j;
    float v = 0.f;
    if (tau >= 0) v = proj[(size_t)tau * ld + off + c];
    else if (pos0 + tau >= 0) v = hist[(size_t)((pos0 + tau) % ring) * ch + c];
    acc = fmaf(w[(size_t)c * taps + j], v, acc);
  }
  return silu_f(acc);
}

// stores the step's last taps - 1 inputs in the history ring (steps longer than kConvSpare tokens, after their convolutions)
__global__ void conv_ring_store(const float* __restrict__ proj, int ld, int off, float* __restrict__ hist, int ring, int T, int ch, int taps,
                                const int* __restrict__ ctl) {
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= ch) return;
  for (int tau = max(0, T - (taps - 1)); tau < T; tau++) hist[(size_t)((ctl[0] + tau) % ring) * ch + c] = proj[(size_t)tau * ld + off + c];
}

__device__ __forceinline__ float gdn_log_decay(float a, float A_log, float dt_bias) { return -expf(A_log) * softplus_f(a + dt_bias); }

// k_j . k_i and q_j . k_i of a block: thread (j, i) of 256; rows of `pitch` floats (a multiple of 4, zero beyond the head size)
__device__ __forceinline__ void block_gram(const float* sq, const float* sk, int pitch, int n4, float& kk, float& qk) {
  const int j = threadIdx.x >> 4, i = threadIdx.x & 15;
  const float4* kj = reinterpret_cast<const float4*>(sk + j * pitch);
  const float4* ki = reinterpret_cast<const float4*>(sk + i * pitch);
  const float4* qj = reinterpret_cast<const float4*>(sq + j * pitch);
  float a0 = 0.f, a1 = 0.f, b0 = 0.f, b1 = 0.f;
  for (int n = 0; n < n4; n++) {
    const float4 x = kj[n], y = ki[n], z = qj[n];
    a0 = fmaf(x.x, y.x, a0); a1 = fmaf(x.y, y.y, a1); a0 = fmaf(x.z, y.z, a0); a1 = fmaf(x.w, y.w, a1);
    b0 = fmaf(z.x, y.x, b0); b1 = fmaf(z.y, y.y, b1); b0 = fmaf(z.z, y.z, b0); b1 = fmaf(z.w, y.w, b1);
  }
  kk = a0 + a1; qk = b0 + b1;
}

// ---------------------------------------------------------------------------------------------------------------------
// Delta rule, a step's state-independent part.  Grid (blocks of kLinBlk tokens, G q / k heads + ceil(H P / 256) slices of v).
// A q / k CTA: convolution + silu + unit norm of its head's q and k rows (stored to qn / kn [T][G][NP], zero-padded to NP),
// the block's Gram products, and per value head of the group the record (see above).  A v CTA: convolution + silu of 256 value
// channels (vn [T][H P]).  proj rows hold the raw projections: q at q_off, k and v behind it (the convolution's channels run
// over the three), b at b_off, a at a_off (one number per value head).
// ---------------------------------------------------------------------------------------------------------------------
struct GdnP {
  const float* proj; int ld, q_off, b_off, a_off;
  const float *w, *A_log, *dt_bias;     // w [2 G N + H P][taps]
  float* hist; int ring, taps;
  int T, H, G, N, P;
  const int* ctl;
};
__global__ void __launch_bounds__(256) gdn_prepare(const GdnP D, float* __restrict__ qn, float* __restrict__ kn, float* __restrict__ vn, int NP,
                                                   float* __restrict__ rec) {
  extern __shared__ __align__(16) float sm[];
  const int tid = threadIdx.x, lane = tid & 31, w = tid >> 5, blk = blockIdx.x, t0 = blk * kLinBlk, nt = min(kLinBlk, D.T - t0);
  const int pos0 = D.ctl[0], KD = D.G * D.N, CH = 2 * KD + D.H * D.P;
  if ((int)blockIdx.y >= D.G) {
    const int c = ((int)blockIdx.y - D.G) * 256 + tid;
    if (c < D.H * D.P)
      for (int t = 0; t < nt; t++) vn[(size_t)(t0 + t) * D.H * D.P + c] = conv_silu_at(D.proj, D.ld, D.q_off, 2 * KD + c, CH, D.w, D.taps, D.hist, D.ring, pos0, t0 + t);
    return;
  }
  const int pitch = NP + 4, g = blockIdx.y, rep = D.H / D.G;
  float* sq = sm;                            // [16][pitch]
  float* sk = sq + kLinBlk * pitch;          // [16][pitch]
  float* kk = sk + kLinBlk * pitch;          // [16][16]
  float* qk = kk + kLinBlk * kLinBlk;        // [16][16]
  float* As = qk + kLinBlk * kLinBlk + w * kLinBlk * kLinBlk;   // [8 warps][16][16]
  const float qs = 1.f / sqrtf((float)D.N);
  for (int e = w; e < 2 * kLinBlk; e += 8) {   // a warp per (token, q | k)
    const int t = e >> 1, isk = e & 1;
    float* row = (isk ? sk : sq) + t * pitch;
    float ss = 0.f;
    for (int n = lane; n < pitch; n += 32) {
      const float v = t < nt && n < D.N ? conv_silu_at(D.proj, D.ld, D.q_off, isk * KD + g * D.N + n, CH, D.w, D.taps, D.hist, D.ring, pos0, t0 + t) : 0.f;
      row[n] = v;
      ss = fmaf(v, v, ss);
    }
    const float sc = (isk ? 1.f : qs) / sqrtf(warp_sum(ss) + 1e-6f);
    float* dst = (isk ? kn : qn) + ((size_t)(t0 + t) * D.G + g) * NP;
    for (int n = lane; n < NP; n += 32) {     // the lane that stored an entry scales it
      const float v = row[n] * sc;
      row[n] = v;
      if (t < nt) dst[n] = v;
    }
  }
  __syncthreads();
  float a, b;
  block_gram(sq, sk, pitch, NP >> 2, a, b);
  kk[tid] = a; qk[tid] = b;
  __syncthreads();
  for (int hh = w; hh < rep; hh += 8) {      // a warp per value head of the group
    const int h = g * rep + hh, j = lane & 15;
    float beta = 0.f, raw = 0.f;
    if (j < nt) {
      const float* pr = D.proj + (size_t)(t0 + j) * D.ld;
      beta = sigmoid_f(pr[D.b_off + h]);
      raw = gdn_log_decay(pr[D.a_off + h], D.A_log[h], D.dt_bias[h]);
    }
    float lg = raw;                          // sum over the block's tokens up to j
#pragma unroll
    for (int o = 1; o < kLinBlk; o <<= 1) { const float v = __shfl_up_sync(0xffffffffu, lg, o, kLinBlk); if (j >= o) lg += v; }
    float* R = rec + ((size_t)blk * D.H + h) * kRecFloats;
    float sum = 0.f;                         // lane (half, i): sum of the logarithms behind token i, up to the row
#pragma unroll
    for (int row = 0; row < kLinBlk; row++) {   // lanes 0 .. 15 write M, lanes 16 .. 31 the matrix to invert
      const float lr = __shfl_sync(0xffffffffu, raw, row), br = __shfl_sync(0xffffffffu, beta, row);
      if (row > j) sum += lr;
      const float ratio = j <= row ? expf(sum) : 0.f;
      if (lane < kLinBlk) R[kRecM + row * kLinBlk + j] = ratio * qk[row * kLinBlk + j];
      else As[row * kLinBlk + j] = j < row ? br * ratio * kk[row * kLinBlk + j] : 0.f;
    }
    if (lane < kLinBlk) { R[kRecG + j] = expf(lg); R[kRecB + j] = beta; R[kRecE + j] = expf(sum); }
    if (lane == kLinBlk - 1) R[kRecEnd] = expf(lg);
    __syncwarp();
    if (lane < kLinBlk) {                      // column `lane` of (I + A)^-1 by forward substitution
      float x[kLinBlk];
#pragma unroll
      for (int r = 0; r < kLinBlk; r++) {
        float s = r == lane ? 1.f : 0.f;
#pragma unroll
        for (int m = 0; m < kLinBlk; m++) if (m < r) s = fmaf(-As[r * kLinBlk + m], x[m], s);
        x[r] = s;
        R[kRecT + r * kLinBlk + lane] = s;
      }
    }
    __syncwarp();
  }
}

// Plain form: the records of a step (M and the decays) from q and k as they are.  Grid (blocks, heads).
__global__ void __launch_bounds__(256) lin_gram(const float* __restrict__ q, const float* __restrict__ k, int ld, const float* __restrict__ log_decay,
                                                int T, int H, int N, float* __restrict__ rec) {
  extern __shared__ __align__(16) float sm[];
  const int pitch = ((N + 3) & ~3) + 4, tid = threadIdx.x, t0 = blockIdx.x * kLinBlk, nt = min(kLinBlk, T - t0), h = blockIdx.y;
  float* sq = sm;
  float* sk = sq + kLinBlk * pitch;
  for (int e = tid; e < kLinBlk * pitch; e += 256) {
    const int t = e / pitch, n = e - t * pitch;
    const bool ok = t < nt && n < N;
    sq[e] = ok ? q[(size_t)(t0 + t) * ld + h * N + n] : 0.f;
    sk[e] = ok ? k[(size_t)(t0 + t) * ld + h * N + n] : 0.f;
  }
  __syncthreads();
  float kk, qk;
  block_gram(sq, sk, pitch, (N + 3) >> 2, kk, qk);
  const float ld1 = log_decay[h];
  const int j = tid >> 4, i = tid & 15;
  float* R = rec + ((size_t)blockIdx.x * H + h) * kRecFloats;
  R[kRecM + tid] = i <= j ? expf(ld1 * (float)(j - i)) * qk : 0.f;
  if (tid < kLinBlk) { R[kRecG + tid] = expf(ld1 * (float)(tid + 1)); R[kRecB + tid] = 1.f; R[kRecE + tid] = tid < nt ? expf(ld1 * (float)(nt - 1 - tid)) : 0.f; }
  if (tid == 0) R[kRecEnd] = expf(ld1 * (float)nt);
}

// mLSTM, the gates of a step, one CTA per head: log gates  i = cap tanh(raw / cap),  f = log sigmoid(cap tanh(raw / cap))  of every
// token to gi / gf [H][T], and the running maximum to gm [H][T + 1]: gm[h][0] is the one carried in, m[h] then becomes the last.
// The recurrence m' = max(f + m, i) is a scan of pairs (F, B): m -> max(F + m, B); a thread owns consecutive tokens.
__device__ __forceinline__ float log_sigmoid_f(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
__global__ void __launch_bounds__(256) mlstm_gates(const float* __restrict__ proj, int ld, int i_off, int f_off, float cap, int T, int H,
                                                   float* __restrict__ gi, float* __restrict__ gf, float* __restrict__ gm, float* __restrict__ m) {
  __shared__ float sF[256], sB[256];
  const int h = blockIdx.x, tid = threadIdx.x, per = (T + 255) / 256, t0 = min(T, tid * per), t1 = min(T, t0 + per);
  float F = 0.f, B = -INFINITY;
  for (int t = t0; t < t1; t++) {
    const float a = cap * tanhf(proj[(size_t)t * ld + i_off + h] / cap), f = log_sigmoid_f(cap * tanhf(proj[(size_t)t * ld + f_off + h] / cap));
    gi[(size_t)h * T + t] = a;
    gf[(size_t)h * T + t] = f;
    B = fmaxf(B + f, a);
    F += f;
  }
  sF[tid] = F; sB[tid] = B;
  __syncthreads();
  for (int o = 1; o < 256; o <<= 1) {
    const float pF = tid >= o ? sF[tid - o] : 0.f, pB = tid >= o ? sB[tid - o] : -INFINITY;
    __syncthreads();
    sB[tid] = fmaxf(pB + sF[tid], sB[tid]);
    sF[tid] = pF + sF[tid];
    __syncthreads();
  }
  const float m0 = m[h];
  float cur = tid ? fmaxf(sF[tid - 1] + m0, sB[tid - 1]) : m0;
  __syncthreads();   // every thread has read m[h]
  float* out = gm + (size_t)h * (T + 1);
  if (tid == 0) out[0] = m0;
  for (int t = t0; t < t1; t++) { cur = fmaxf(gf[(size_t)h * T + t] + cur, gi[(size_t)h * T + t]); out[t + 1] = cur; }
  if (t1 == T && t0 < T) m[h] = cur;
}

// mLSTM: the records of a step from q and k as they are (q is scaled by 1 / sqrt(N) here) and the gates above.  Grid (blocks, heads).
__global__ void __launch_bounds__(256) mlstm_gram(const float* __restrict__ q, const float* __restrict__ k, int ld, const float* __restrict__ gi,
                                                  const float* __restrict__ gf, const float* __restrict__ gm, int T, int H, int N, float* __restrict__ rec) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float sf[kLinBlk], si[kLinBlk], sx[kLinBlk + 1];
  const int pitch = ((N + 3) & ~3) + 4, tid = threadIdx.x, t0 = blockIdx.x * kLinBlk, nt = min(kLinBlk, T - t0), h = blockIdx.y;
  float* sq = sm;
  float* sk = sq + kLinBlk * pitch;
  for (int e = tid; e < kLinBlk * pitch; e += 256) {
    const int t = e / pitch, n = e - t * pitch;
    const bool ok = t < nt && n < N;
    sq[e] = ok ? q[(size_t)(t0 + t) * ld + h * N + n] : 0.f;
    sk[e] = ok ? k[(size_t)(t0 + t) * ld + h * N + n] : 0.f;
  }
  if (tid < kLinBlk) {
    sf[tid] = tid < nt ? gf[(size_t)h * T + t0 + tid] : 0.f;
    si[tid] = tid < nt ? gi[(size_t)h * T + t0 + tid] : 0.f;
  }
  if (tid <= kLinBlk) sx[tid] = gm[(size_t)h * (T + 1) + t0 + min(tid, nt)];   // sx[j + 1]: maximum behind token j
  __syncthreads();
  float kk, qk;
  block_gram(sq, sk, pitch, (N + 3) >> 2, kk, qk);
  const float qs = 1.f / sqrtf((float)N);
  const int j = tid >> 4, i = tid & 15;
  float* R = rec + ((size_t)blockIdx.x * H + h) * kRecFloats;
  float lr = si[i] - sx[j + 1];               // logarithm of what token i's write is worth at token j
  for (int l = i + 1; l <= j; l++) lr += sf[l];
  R[kRecM + tid] = i <= j && j < nt ? expf(lr) * (qk * qs) : 0.f;
  if (tid < kLinBlk) {
    float lg = sx[0], le = si[tid] - sx[nt];
    for (int l = 0; l <= tid; l++) lg += sf[l];
    for (int l = tid + 1; l < nt; l++) le += sf[l];
    R[kRecG + tid] = tid < nt ? expf(lg - sx[tid + 1]) * qs : 0.f;
    R[kRecB + tid] = 1.f;
    R[kRecE + tid] = tid < nt ? expf(le) : 0.f;
    if (tid == nt - 1) R[kRecEnd] = expf(lg - sx[nt]);
  }
}

// sums of 32 accumulators over TPC neighbouring lanes, scattered: afterwards a[0 .. 32 / TPC - 1] of a lane hold the totals of
// the entries red_index(..) .. + 32 / TPC - 1
template <int TPC>
__device__ __forceinline__ void reduce_scatter(float (&a)[32], int s) {
#pragma unroll
  for (int o = TPC / 2, n = 16; o >= 1; o >>= 1, n >>= 1) {
    const bool up = (s & o) != 0;
#pragma unroll
    for (int i = 0; i < n; i++) {
      const float mine = up ? a[i + n] : a[i], other = up ? a[i] : a[i + n];
      a[i] = mine + __shfl_xor_sync(0xffffffffu, other, o);
    }
  }
}
template <int TPC>
__device__ __forceinline__ int reduce_index(int s) {
  int idx = 0;
#pragma unroll
  for (int o = TPC / 2, n = 16; o >= 1; o >>= 1, n >>= 1) idx += (s & o) ? n : 0;
  return idx;
}

// ---------------------------------------------------------------------------------------------------------------------
// The walk over the blocks of a step.  CTA = (head, slice of value channels).  A warp owns (32 / TPC) x CPT value channels with the
// whole key dimension: lane (grp, s) holds the rows n = 4 (s + TPC r) + i, r < RQ, of the CPT channels from grp * CPT on in
// registers.  S0^T k and S0^T q of a block are 32 dot products per channel, reduced across the TPC lanes by reduce-scatter;
// everything behind them stays inside the warp (its own shared-memory strip).  The CTA's last kLinStage warps do not compute:
// they bring the blocks' q, k, v and records through three buffers, two blocks ahead (16-byte asynchronous copies where the rows
// allow it, plain loads otherwise), so a block costs the computing warps one barrier.
// q, k: head stride hs (rows of N entries), v: head stride P; head h reads q / k head h / rep.
// nst non-null: one more value channel (index P) whose value is 1 for every token, with its state in nst [H][N] and its output in den [T][H].
// ---------------------------------------------------------------------------------------------------------------------
constexpr int kLinStage = 2;           // staging warps of a CTA
template <bool DELTA, int TPC, int RQ, int CPT>
__global__ void __launch_bounds__(320) lin_scan(const float* __restrict__ q, const float* __restrict__ k, int ldq, int hs, int rep,
                                                const float* __restrict__ v, int ldv, const float* __restrict__ rec, float* __restrict__ state,
                                                float* __restrict__ out, int ldo, int T, int H, int N, int P, int PB, float* __restrict__ nst, float* __restrict__ den) {
  extern __shared__ __align__(16) float sm[];
  constexpr int C = kLinBlk, PITCH = 4 * TPC * RQ, CW = CPT * (32 / TPC), VB = 32 / CPT;
  const int per = 2 * C * PITCH + C * PB + kRecFloats;     // one buffer: k [C][PITCH], q [C][PITCH], v [C][PB], record
  const int tid = threadIdx.x, lane = tid & 31, w = tid >> 5, s = lane & (TPC - 1), grp = lane / TPC;
  const int h = blockIdx.x, p0 = blockIdx.y * PB, hk = h / rep, cw = w * CW;   // cw: the warp's first channel inside the slice
  float* Rw = sm + 3 * per + w * (4 * C * CW);   // [S0^T k | S0^T q][C][CW]
  float* Uw = Rw + 2 * C * CW;                   // [C][CW]  w, then R(end, .) u
  float* Xw = Uw + C * CW;                       // [C][CW]  u
  float S[RQ][4][CPT];                           // [row group][row][channel]
  const int pc = p0 + cw + grp * CPT;              // the lane's first channel of the head
#pragma unroll
  for (int r = 0; r < RQ; r++)
#pragma unroll
    for (int i = 0; i < 4; i++) {
      const int n = 4 * (s + TPC * r) + i;
#pragma unroll
      for (int c = 0; c < CPT; c++) {
        S[r][i][c] = (n < N && pc + c < P && cw + grp * CPT + c < PB) ? state[((size_t)h * N + n) * P + pc + c] : 0.f;
        if (nst && n < N && pc + c == P && cw + grp * CPT + c < PB) S[r][i][c] = nst[(size_t)h * N + n];
      }
    }
  const bool vec = (N & 3) == 0 && (ldq & 3) == 0 && (hs & 3) == 0 && ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k)) & 15) == 0;
  const bool vecv = (P & 3) == 0 && (PB & 3) == 0 && (ldv & 3) == 0 && (reinterpret_cast<uintptr_t>(v) & 15) == 0 && p0 + PB <= P;
  const int nc = (blockDim.x >> 5) - kLinStage;   // computing warps
  for (int e = tid; e < 3 * per; e += blockDim.x) sm[e] = 0.f;   // padding columns stay zero
  __syncthreads();
  const int sw = w - nc, stid = tid - 32 * nc;
  constexpr int ST = 32 * kLinStage;
  auto stage = [&](int buf, int t0) {   // by the staging warps
    float* bk = sm + buf * per;
    float* bq = bk + C * PITCH;
    float* bv = bq + C * PITCH;
    float* br = bv + C * PB;
    const int nt = min(C, T - t0);
    const size_t base = (size_t)t0 * ldq + (size_t)hk * hs;
    if (vec) {
      for (int t = sw; t < C; t += kLinStage) {                   // a warp per row; rows past the end are zero-filled
        const size_t src = base + (size_t)(t < nt ? t : 0) * ldq;
        const int bytes = t < nt ? 16 : 0;
        for (int c = 4 * lane; c < N; c += 128) {
          cp_async_16(bk + t * PITCH + c, k + src + c, bytes);
          cp_async_16(bq + t * PITCH + c, q + src + c, bytes);
        }
      }
    } else {
      for (int t = sw; t < C; t += kLinStage)
        for (int c = lane; c < N; c += 32) {
          bk[t * PITCH + c] = t < nt ? k[base + (size_t)t * ldq + c] : 0.f;
          bq[t * PITCH + c] = t < nt ? q[base + (size_t)t * ldq + c] : 0.f;
        }
    }
    const float* vs = v + (size_t)t0 * ldv + (size_t)h * P + p0;
    if (vecv) {
      const int b4 = PB >> 2;
      for (int e = stid; e < C * b4; e += ST) {
        const int t = e / b4, c = (e - t * b4) * 4;
        cp_async_16(bv + t * PB + c, vs + (size_t)(t < nt ? t : 0) * ldv + c, t < nt ? 16 : 0);
      }
    } else {
      for (int e = stid; e < C * PB; e += ST) {
        const int t = e / PB, c = e - t * PB;
        bv[e] = t < nt && p0 + c < P ? vs[(size_t)t * ldv + c] : nst && t < nt && p0 + c == P ? 1.f : 0.f;
      }
    }
    const float* rs = rec + ((size_t)(t0 / C) * H + h) * kRecFloats;
    for (int e = (DELTA ? 0 : kRecM / 4) + stid; e < kRecFloats / 4; e += ST) cp_async_16(br + 4 * e, rs + 4 * e, 16);
    cp_async_commit();
  };
  const int nb = (T + C - 1) / C;
  if (sw >= 0) {
    stage(0, 0);
    if (nb > 1) { stage(1, C); cp_async_wait<1>(); } else cp_async_wait<0>();
    __syncthreads();                   // block 0 has landed
    for (int b = 0; b < nb; b++) {     // while the others work on block b: start block b + 2, see block b + 1 land
      if (b + 2 < nb) { stage((b + 2) % 3, (b + 2) * C); cp_async_wait<1>(); }
      else cp_async_wait<0>();
      __syncthreads();
    }
    return;
  }
  __syncthreads();
  for (int b = 0; b < nb; b++) {
    const float* bk = sm + (b % 3) * per;
    const float* bq = bk + C * PITCH;
    const float* bv = bq + C * PITCH;
    const float* br = bv + C * PB;
    const int t0 = b * C, nt = min(C, T - t0);
    // S0^T k_j (delta rule) and S0^T q_j: VB tokens x CPT channels per reduction
#pragma unroll
    for (int which = DELTA ? 0 : 1; which < 2; which++) {
      const float* src = which ? bq : bk;
#pragma unroll
      for (int half = 0; half < C; half += VB) {
        float a[32];
#pragma unroll
        for (int e = 0; e < 32; e++) a[e] = 0.f;
#pragma unroll
        for (int t = 0; t < VB; t++)
#pragma unroll
          for (int r = 0; r < RQ; r++) {
            const float4 x = *reinterpret_cast<const float4*>(src + (half + t) * PITCH + 4 * (s + TPC * r));
#pragma unroll
            for (int c = 0; c < CPT; c++) {
              float& acc = a[t * CPT + c];
              acc = fmaf(x.x, S[r][0][c], acc); acc = fmaf(x.y, S[r][1][c], acc);
              acc = fmaf(x.z, S[r][2][c], acc); acc = fmaf(x.w, S[r][3][c], acc);
            }
          }
        reduce_scatter<TPC>(a, s);
        const int idx = reduce_index<TPC>(s);
#pragma unroll
        for (int e = 0; e < 32 / TPC; e++) {
          const int t = (idx + e) / CPT, c = (idx + e) % CPT;
          Rw[which * C * CW + (half + t) * CW + grp * CPT + c] = a[e];
        }
      }
    }
    __syncwarp();
    if (DELTA) {
#pragma unroll
      for (int e = lane; e < C * CW; e += 32) {
        const int j = e / CW, c = e & (CW - 1);
        const float vv = cw + c < PB ? bv[j * PB + cw + c] : 0.f;
        Uw[e] = br[kRecB + j] * fmaf(-br[kRecG + j], Rw[e], vv);
      }
      __syncwarp();
    }
    float u[C * CW / 32];
#pragma unroll
    for (int m = 0; m < C * CW / 32; m++) {
      const int e = lane + 32 * m, j = e / CW, c = e & (CW - 1);
      if (DELTA) {
        float s0 = 0.f, s1 = 0.f;
#pragma unroll
        for (int i = 0; i < C; i += 4) {   // entries above the diagonal of the inverse are zero
          const float4 tt = *reinterpret_cast<const float4*>(br + kRecT + j * C + i);
          s0 = fmaf(tt.x, Uw[i * CW + c], s0); s1 = fmaf(tt.y, Uw[(i + 1) * CW + c], s1);
          s0 = fmaf(tt.z, Uw[(i + 2) * CW + c], s0); s1 = fmaf(tt.w, Uw[(i + 3) * CW + c], s1);
        }
        u[m] = s0 + s1;
      } else u[m] = cw + c < PB ? bv[j * PB + cw + c] : 0.f;
      Xw[e] = u[m];
    }
    __syncwarp();
#pragma unroll
    for (int m = 0; m < C * CW / 32; m++) {
      const int e = lane + 32 * m, j = e / CW, c = e & (CW - 1);
      Uw[e] = br[kRecE + j] * u[m];
      float s0 = br[kRecG + j] * Rw[C * CW + e], s1 = 0.f;
#pragma unroll
      for (int i = 0; i < C; i += 4) {
        const float4 mm = *reinterpret_cast<const float4*>(br + kRecM + j * C + i);
        s0 = fmaf(mm.x, Xw[i * CW + c], s0); s1 = fmaf(mm.y, Xw[(i + 1) * CW + c], s1);
        s0 = fmaf(mm.z, Xw[(i + 2) * CW + c], s0); s1 = fmaf(mm.w, Xw[(i + 3) * CW + c], s1);
      }
      if (j < nt && cw + c < PB && p0 + cw + c < P) out[(size_t)(t0 + j) * ldo + (size_t)h * P + p0 + cw + c] = s0 + s1;
      else if (nst && j < nt && cw + c < PB && p0 + cw + c == P) den[(size_t)(t0 + j) * H + h] = s0 + s1;
    }
    __syncwarp();
    const float ge = br[kRecEnd];
#pragma unroll
    for (int r = 0; r < RQ; r++)
#pragma unroll
      for (int i = 0; i < 4; i++)
#pragma unroll
        for (int c = 0; c < CPT; c++) S[r][i][c] *= ge;
#pragma unroll
    for (int j = 0; j < C; j++) {
      float uu[CPT];
#pragma unroll
      for (int c = 0; c < CPT; c++) uu[c] = Uw[j * CW + grp * CPT + c];
#pragma unroll
      for (int r = 0; r < RQ; r++) {
        const float4 x = *reinterpret_cast<const float4*>(bk + j * PITCH + 4 * (s + TPC * r));
        const float xs[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
        for (int i = 0; i < 4; i++)
#pragma unroll
          for (int c = 0; c < CPT; c++) S[r][i][c] = fmaf(xs[i], uu[c], S[r][i][c]);
      }
    }
    __syncthreads();   // block b's buffer is free, block b + 1 is there
  }
#pragma unroll
  for (int r = 0; r < RQ; r++)
#pragma unroll
    for (int i = 0; i < 4; i++) {
      const int n = 4 * (s + TPC * r) + i;
#pragma unroll
      for (int c = 0; c < CPT; c++) {
        if (n < N && pc + c < P && cw + grp * CPT + c < PB) state[((size_t)h * N + n) * P + pc + c] = S[r][i][c];
        if (nst && n < N && pc + c == P && cw + grp * CPT + c < PB) nst[(size_t)h * N + n] = S[r][i][c];
      }
    }
}
inline size_t lin_scan_smem(int pitch, int PB, int warps, int cw) { return ((size_t)3 * (2 * kLinBlk * pitch + kLinBlk * PB + kRecFloats) + (size_t)warps * 4 * kLinBlk * cw) * 4; }

// ---------------------------------------------------------------------------------------------------------------------
// Steps of up to kLinDecodeTokens tokens, one CTA per value head, the head's state in registers: thread (pl, ng) owns the value
// channels 4 pl .. 4 pl + 3 and the rows ng + NG r, r < RN.  S^T k and S^T q are taken from the state ahead of the token
// (o = g S^T q + (k . q) u), so a token costs one reduction.
// Delta rule: the raw projections come in (GdnP); the convolutions (whose inputs also go into the history ring: rows that no
// CTA of the step reads), silu, unit norms, step size and decay, head norm, output gate and factor are applied here:
//   out[t][h P + p] = alpha rms(o)_p norm_w[p] silu(gate[t][h P + p]).
// Plain form: q, k, v rows of proj (q_off, k and v behind it) as they are, decay[h]; out = o.
// mLSTM: q, k, v likewise, raw gates in columns a_off (forget) and b_off (input), n and m carried in X; head norm with weights [H P], gate:
//   out[t][h P + p] = rms(o)_p norm_w[h P + p] sigmoid(gate[t][h P + p]).
// ---------------------------------------------------------------------------------------------------------------------
constexpr int kLinDecodeThreads = 512;
enum { LIN_PLAIN = 0, LIN_DELTA = 1, LIN_MLSTM = 2 };
struct MlstmP { float cap; float *n, *m; };   // n [H][N], m [H]
template <int MODE, int RN>
__global__ void __launch_bounds__(kLinDecodeThreads) lin_decode(const GdnP D, const float* __restrict__ decay, float* __restrict__ state,
                                                                const float* __restrict__ norm_w, float eps, int gate_off, float alpha,
                                                                float* __restrict__ out, int ldo, const MlstmP X) {
  constexpr bool DELTA = MODE == LIN_DELTA, MLSTM = MODE == LIN_MLSTM;
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[33], gb[5];
  const int N = D.N, P = D.P, h = blockIdx.x, rep = D.H / D.G, g = h / rep, tid = threadIdx.x;
  const int PL = (P + 3) >> 2, NG = min(kLinDecodeThreads / PL, N), pl = tid % PL, ng = tid / PL;
  const bool on = ng < NG;
  float* sq = sm;                    // [N]
  float* sk = sq + N;                // [N]
  float* sv = sk + N;                // [P]   v, then u
  float* so = sv + P;                // [P]
  float* part = so + P + ((4 - ((2 * N + 2 * P) & 3)) & 3);   // [2][NG][4 PL]
  float S[RN][4];
  float* sn = part + 2 * (size_t)NG * 4 * PL;   // [N]  (mLSTM)
  const bool vec = (P & 3) == 0;
  if (MLSTM) {
    for (int n = tid; n < N; n += kLinDecodeThreads) sn[n] = X.n[(size_t)h * N + n];
    if (tid == 0) gb[3] = X.m[h];
  }
#pragma unroll
  for (int r = 0; r < RN; r++) {
    const int n = ng + NG * r;
    const float* src = state + ((size_t)h * N + n) * P + 4 * pl;
    if (on && n < N && vec) {
      const float4 v = *reinterpret_cast<const float4*>(src);
      S[r][0] = v.x; S[r][1] = v.y; S[r][2] = v.z; S[r][3] = v.w;
    } else
#pragma unroll
      for (int c = 0; c < 4; c++) S[r][c] = on && n < N && 4 * pl + c < P ? src[c] : 0.f;
  }
  const int KD = D.G * N, CH = 2 * KD + D.H * P, pos0 = D.ctl[0];
  for (int t = 0; t < D.T; t++) {
    const float* pr = D.proj + (size_t)t * D.ld;
    for (int e = tid; e < 2 * N + P; e += kLinDecodeThreads) {
      const int c = e < N ? g * N + e : e < 2 * N ? KD + g * N + e - N : 2 * KD + h * P + e - 2 * N;   // column behind q_off
      float* dst = e < N ? sq + e : e < 2 * N ? sk + e - N : sv + e - 2 * N;
      const float raw = pr[D.q_off + c];
      if (DELTA) {
        *dst = conv_silu_at(D.proj, D.ld, D.q_off, c, CH, D.w, D.taps, D.hist, D.ring, pos0, t);
        if (D.taps > 1 && (e >= 2 * N || h == g * rep)) D.hist[(size_t)((pos0 + t) % D.ring) * CH + c] = raw;
      } else *dst = raw;
    }
    __syncthreads();
    const int lane = tid & 31, w = tid >> 5;
    if (w < 3) {                     // sums of q^2 (mLSTM: n q), k^2 and q k
      float a = 0.f;
      for (int n = lane; n < N; n += 32) { const float x = w == 1 ? sk[n] : sq[n], y = w == 0 ? (MLSTM ? sn[n] : sq[n]) : sk[n]; a = fmaf(x, y, a); }
      a = warp_sum(a);
      if (lane == 0) red[w] = a;
    } else if (w == 3 && lane == 0) {
      if (DELTA) { gb[0] = expf(gdn_log_decay(pr[D.a_off + h], D.A_log[h], D.dt_bias[h])); gb[1] = sigmoid_f(pr[D.b_off + h]); }
      else if (MLSTM) {
        const float i = X.cap * tanhf(pr[D.b_off + h] / X.cap), f = log_sigmoid_f(X.cap * tanhf(pr[D.a_off + h] / X.cap)), m = fmaxf(f + gb[3], i);
        gb[0] = expf(f + gb[3] - m); gb[1] = expf(i - m); gb[2] = expf(-m); gb[3] = m;
      } else { gb[0] = decay[h]; gb[1] = 1.f; }
    }
    __syncthreads();
    // unit norms as factors on the dot products
    const float fq = DELTA ? 1.f / (sqrtf(red[0] + 1e-6f) * sqrtf((float)N)) : MLSTM ? 1.f / sqrtf((float)N) : 1.f, fk = DELTA ? 1.f / sqrtf(red[1] + 1e-6f) : 1.f, kq = red[2] * fq * fk;
    const float gd = gb[0], beta = gb[1];
    const float inv = MLSTM ? 1.f / (fmaxf(fabsf(fmaf(gd * fq, red[0], beta * kq)), gb[2]) + 1e-6f) : 1.f;
    float ak[4] = {0.f, 0.f, 0.f, 0.f}, aq[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int r = 0; r < RN; r++) {
      const int n = ng + NG * r;
      if (on && n < N) {
        const float x = sk[n], y = sq[n];
#pragma unroll
        for (int c = 0; c < 4; c++) { if (DELTA) ak[c] = fmaf(x, S[r][c], ak[c]); aq[c] = fmaf(y, S[r][c], aq[c]); }
      }
    }
    if (on) {
      float4* pp = reinterpret_cast<float4*>(part);
      if (DELTA) pp[ng * PL + pl] = make_float4(ak[0], ak[1], ak[2], ak[3]);
      pp[(NG + ng) * PL + pl] = make_float4(aq[0], aq[1], aq[2], aq[3]);
    }
    __syncthreads();
    for (int p = tid; p < P; p += kLinDecodeThreads) {
      float rk = 0.f, rq = 0.f;
      for (int i = 0; i < NG; i++) {
        if (DELTA) rk += part[(size_t)i * 4 * PL + p];
        rq += part[(size_t)(NG + i) * 4 * PL + p];
      }
      const float u = DELTA ? beta * fmaf(-gd * fk, rk, sv[p]) : MLSTM ? beta * sv[p] : sv[p];
      so[p] = fmaf(gd * fq, rq, kq * u) * inv;
      sv[p] = u * fk;                 // the update below multiplies the unscaled k
    }
    __syncthreads();
    float uu[4];
#pragma unroll
    for (int c = 0; c < 4; c++) uu[c] = 4 * pl + c < P ? sv[4 * pl + c] : 0.f;
#pragma unroll
    for (int r = 0; r < RN; r++) {
      const int n = ng + NG * r;
      if (on && n < N) {
        const float x = sk[n];
#pragma unroll
        for (int c = 0; c < 4; c++) S[r][c] = fmaf(x, uu[c], gd * S[r][c]);
      }
    }
    if (MLSTM) for (int n = tid; n < N; n += kLinDecodeThreads) sn[n] = fmaf(beta, sk[n], gd * sn[n]);
    if (DELTA || MLSTM) {
      float ss = 0.f;
      for (int p = tid; p < P; p += kLinDecodeThreads) ss = fmaf(so[p], so[p], ss);
      const float sc = alpha / sqrtf(block_sum(ss, red) / (float)P + eps);
      for (int p = tid; p < P; p += kLinDecodeThreads) {
        const float gt = pr[gate_off + h * P + p];
        out[(size_t)t * ldo + (size_t)h * P + p] = MLSTM ? so[p] * sc * norm_w[(size_t)h * P + p] * sigmoid_f(gt) : so[p] * sc * norm_w[p] * silu_f(gt);
      }
    } else
      for (int p = tid; p < P; p += kLinDecodeThreads) out[(size_t)t * ldo + (size_t)h * P + p] = so[p];
    __syncthreads();
  }
  if (MLSTM) {
    for (int n = tid; n < N; n += kLinDecodeThreads) X.n[(size_t)h * N + n] = sn[n];
    if (tid == 0) X.m[h] = gb[3];
  }
#pragma unroll
  for (int r = 0; r < RN; r++) {
    const int n = ng + NG * r;
    if (!(on && n < N)) continue;
    float* dst = state + ((size_t)h * N + n) * P + 4 * pl;
    if (vec) *reinterpret_cast<float4*>(dst) = make_float4(S[r][0], S[r][1], S[r][2], S[r][3]);
    else
#pragma unroll
      for (int c = 0; c < 4; c++) if (4 * pl + c < P) dst[c] = S[r][c];
  }
}
inline size_t lin_decode_smem(int N, int P) {
  const int PL = (P + 3) / 4, NG = kLinDecodeThreads / PL < N ? kLinDecodeThreads / PL : N;
  return ((size_t)3 * N + 2 * P + 4 + (size_t)2 * NG * 4 * PL) * 4;
}

}  // namespace hy
}  // namespace dsk
