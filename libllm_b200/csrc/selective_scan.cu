// The selective state-space recurrence: a diagonal state per channel whose decay, input and read-out depend on the token.
//
//   x_t   = silu(conv bias + sum_j w[c, j] u_(t - taps + 1 + j))           a causal convolution over time per channel
//   dt_t  = softplus(raw dt + dt bias)                                      one number per channel
//   S[c, n] <- exp(dt A[c, n]) S[c, n] + dt x B_n,    A = -exp(A_log)
//   y_c   = sum_n S[c, n] C_n + D_c x_c,    out = y silu(z)
//
// State per sequence: S [slots, inner, N] and the convolution's last taps - 1 inputs [slots, taps - 1, inner], both 32-bit.
// Everything from the products' 32-bit results on is 32-bit; x is rounded to the engine's type once, where the convolution
// hands it to the products and the recurrence alike.
//
//  * short_conv_silu: the convolution, a thread four channels and a run of rows, the last taps values in registers.
//  * selective_scan: a step of any tokens.  A CTA takes 128 / L channels of one sequence, L lanes to a channel, each with NS of its
//    N states in registers (few: what bounds it is how many warps there are to hide one another's latency), and walks the tokens in
//    groups of 32 (8 with many states).  While a group is worked on, the next one's values are on
//    their way into registers; behind it they go, with everything that needs no state already computed (softplus, dt x, D x,
//    silu z), into the other of two buffers in shared memory: one barrier a group.  The only dependence between tokens is the
//    state's fused multiply-add; sixteen tokens' sums over n are joined together, off that chain, by shuffles that leave each lane
//    one token's.  Tokens beyond the sequence's last have dt = 0 and leave the state as it is: no branch in the loop.
//  * selective_step: a step of single tokens, with the product that makes dt (a row of dt_rank values per channel) in the same
//    launch.
// A channel's arithmetic is the same function wherever it is computed and depends on its own sequence alone.
//
// The reference has no such mixer.
#include "common.cuh"
#include <math.h>

LLM_DEFINE_LAST_ERROR(llm_selective_scan_last_error)

namespace {

constexpr float LOG2E = 1.4426950408889634f;

// FAST: for results that are rounded to 16 bits; a few 1e-7 of the value
template <bool FAST = false>
__device__ __forceinline__ float silu_of(float v) {
  return FAST ? __fdividef(v, 1.f + __expf(-v)) : v / (1.f + expf(-v));
}
// log(1 + e^v) without overflow: max(v, 0) + log1p(e^-|v|); FAST: log1p(e) = 2 artanh(e / (2 + e)) by its Taylor series, whose
// argument is a third at most
template <bool FAST = false>
__device__ __forceinline__ float softplus_of(float v) {
  if (!FAST) return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v)));
  const float e = __expf(-fabsf(v)), s = __fdividef(e, 2.f + e), s2 = s * s;
  float p = 1.f / 13.f;
  p = fmaf(p, s2, 1.f / 11.f);
  p = fmaf(p, s2, 1.f / 9.f);
  p = fmaf(p, s2, 1.f / 7.f);
  p = fmaf(p, s2, 1.f / 5.f);
  p = fmaf(p, s2, 1.f / 3.f);
  p = fmaf(p, s2, 1.f);
  return fmaf(2.f * s, p, fmaxf(v, 0.f));
}

// ---------------------------------------------------------------- the short convolution
// u [tokens, ld] 32-bit, weight [taps][channels] 32-bit, bias [channels]; out [tokens, channels].  Rows whose window lies inside
// the step belong to CTAs of a run of SC_ROWS rows (blockIdx.x < n_chunks); the first taps - 1 rows of every sequence, and its
// state, to a CTA of that sequence, whose threads read their channels' old state before they write the new one.
constexpr int SC_THREADS = 128, SC_ROWS = 8, SC_MAX_TAPS = 8;

template <int V>
__device__ __forceinline__ void sc_load(const float *p, float (&x)[V]) {
  if constexpr (V == 4) {
    const float4 v = ld4(p);
    x[0] = v.x, x[1] = v.y, x[2] = v.z, x[3] = v.w;
  } else {
    x[0] = p[0];
  }
}
template <typename T, int V>
__device__ __forceinline__ void sc_store(T *p, const float (&x)[V]) {
  if constexpr (V == 4) st4(p, make_float4(x[0], x[1], x[2], x[3]));
  else p[0] = from_float<T>(x[0]);
}

template <typename T, int V, int TAPS>
__global__ void __launch_bounds__(SC_THREADS)
short_conv_silu_kernel(const float *__restrict__ u, long long ld, const float *__restrict__ weight, const float *__restrict__ bias, int taps,
                       float *__restrict__ state, T *__restrict__ out, long long ldo, int channels, const int *__restrict__ tok_seq,
                       const int *__restrict__ tok_pos, const int *__restrict__ seq_start, const int *__restrict__ seq_past,
                       const int *__restrict__ seq_slot, int n_tokens, int n_chunks) {
  grid_dependents_launch();
  const int c0 = (blockIdx.y * SC_THREADS + threadIdx.x) * V, keep = taps - 1;
  float w[TAPS][V], bs[V], win[TAPS][V], x[V];
  if (c0 < channels) {
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      if (j < taps) sc_load<V>(weight + (size_t)j * channels + c0, w[j]);
      else
#pragma unroll
        for (int e = 0; e < V; ++e) w[j][e] = 0.f;
#pragma unroll
      for (int e = 0; e < V; ++e) win[j][e] = 0.f;
    }
    if (bias) sc_load<V>(bias + c0, bs);
    else
#pragma unroll
      for (int e = 0; e < V; ++e) bs[e] = 0.f;
  }
  grid_dependency_wait();
  unsigned mine = 0;                                     // which rows of a run are its CTA's
  if ((int)blockIdx.x < n_chunks) {
    const int lane = threadIdx.x & 31, row = blockIdx.x * SC_ROWS + lane;
    const bool in = lane < SC_ROWS && row < n_tokens;
    mine = __ballot_sync(0xffffffffu, in && tok_pos[in ? row : 0] - seq_past[tok_seq[in ? row : 0]] >= keep);
  }
  if (c0 >= channels) return;
  auto shift = [&]() {                                   // x becomes the window's last value
#pragma unroll
    for (int j = 0; j < TAPS; ++j)
#pragma unroll
      for (int e = 0; e < V; ++e) {
        if (j < taps - 1) win[j][e] = win[j + 1 < TAPS ? j + 1 : j][e];
        else if (j == taps - 1) win[j][e] = x[e];
      }
  };
  auto take = [&](int row) {
    sc_load<V>(u + (size_t)row * ld + c0, x);
    shift();
  };
  auto place = [&](int row) {
    float y[V];
#pragma unroll
    for (int e = 0; e < V; ++e) {
      y[e] = 0.f;
#pragma unroll
      for (int j = 0; j < TAPS; ++j)
        if (j < taps) y[e] = fmaf(w[j][e], win[j][e], y[e]);
      y[e] = silu_of<sizeof(T) == 2>(y[e] + bs[e]);
    }
    sc_store<T, V>(out + (size_t)row * ldo + c0, y);
  };
  if ((int)blockIdx.x < n_chunks) {
    const int r0 = blockIdx.x * SC_ROWS, r1 = min(n_tokens, r0 + SC_ROWS);
    if (TAPS <= 4 && mine == (1u << SC_ROWS) - 1u) {       // all of them: every row's loads on their way at once
      float in[SC_ROWS + TAPS - 1][V];
#pragma unroll
      for (int i = 0; i < SC_ROWS + TAPS - 1; ++i)
        if (i < SC_ROWS + keep) sc_load<V>(u + (size_t)(r0 - keep + i) * ld + c0, in[i]);
#pragma unroll
      for (int i = 0; i < SC_ROWS + TAPS - 1; ++i)
        if (i < SC_ROWS + keep) {
#pragma unroll
          for (int e = 0; e < V; ++e) x[e] = in[i][e];
          shift();
          if (i >= keep) place(r0 - keep + i);
        }
      return;
    }
    for (int row = r0; row < r1; ++row) {
      if (!((mine >> (row - r0)) & 1u)) continue;
      if (row == r0 || !((mine >> (row - r0 - 1)) & 1u))
        for (int k = keep; k > 0; --k) take(row - k);
      take(row);
      place(row);
    }
    return;
  }
  const int b = blockIdx.x - n_chunks, start = seq_start[b], n = seq_start[b + 1] - start;
  float *st = state + (size_t)seq_slot[b] * keep * channels;
  for (int i = 0; i < keep; ++i) {
    sc_load<V>(st + (size_t)i * channels + c0, x);
    shift();
  }
  for (int i = 0; i < min(n, keep); ++i) {
    take(start + i);
    place(start + i);
  }
  if (n > keep)
    for (int k = keep; k > 0; --k) take(start + n - k);
#pragma unroll
  for (int j = 0; j < TAPS; ++j)
    if (j >= 1 && j < taps) sc_store<float, V>(st + (size_t)(j - 1) * channels + c0, win[j]);
}

// ---------------------------------------------------------------- the recurrence over a step's tokens
constexpr int SCAN_THREADS = 128, SCAN_GROUP = 32;
constexpr int SS_THREADS = 128;                          // of a step of single tokens

// 2^x of a number that is never above nought, in one instruction
__device__ __forceinline__ float decay_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// One token of one state: a = exp2(dt A log2 e), S <- a S + dx B, y += S C.  al2: A log2 e.
__device__ __forceinline__ void scan_state(float &S, float al2, float dt, float dx, float B, float C, float &y) {
  S = fmaf(decay_exp2(dt * al2), S, dx * B);
  y = fmaf(S, C, y);
}
template <int L>
__device__ __forceinline__ float lanes_sum(float v) {
#pragma unroll
  for (int o = 1; o < L; o <<= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

// NT values' sums over L lanes at once, by halving: lane bit k picks the half of what is left after k exchanges, so that a lane ends
// with the sums of NT / L values (of one, where L > NT) from first_of<L, NT>(lane) on, in v[0], v[1], ..
template <int L, int NT>
__device__ __forceinline__ void lanes_sums(float (&v)[NT], int lane) {
#pragma unroll
  for (int o = 1, half = NT / 2; o < L; o <<= 1, half >>= 1) {
    if (half > 0) {
      const bool upper = lane & o;
#pragma unroll
      for (int i = 0; i < NT / 2; ++i)
        if (i < half) {
          const float other = __shfl_xor_sync(0xffffffffu, upper ? v[i] : v[i + half], o);
          v[i] = (upper ? v[i + half] : v[i]) + other;
        }
    } else {
      v[0] += __shfl_xor_sync(0xffffffffu, v[0], o);
    }
  }
}
template <int L, int NT>
__device__ __forceinline__ int first_of(int lane) {
  int at = 0;
#pragma unroll
  for (int o = 1, half = NT / 2; o < L && half > 0; o <<= 1, half >>= 1)
    if (lane & o) at += half;
  return at;
}

// the decays (al2) and values of a lane's states, lane + i L; states beyond N are nought and stay so
template <int L, int NS>
__device__ __forceinline__ void lane_states(const float *__restrict__ a_log, const float *__restrict__ st, int c, int lane, int N, bool in,
                                            float (&al2)[NS], float (&S)[NS]) {
#pragma unroll
  for (int i = 0; i < NS; ++i) {
    const bool has = in && lane + i * L < N;
    al2[i] = has ? fmaxf(-expf(a_log[(size_t)c * N + lane + i * L]) * LOG2E, -3e38f) : 0.f;   // finite: 0 times it is 0
    S[i] = has ? st[(size_t)c * N + lane + i * L] : 0.f;
  }
}

template <typename T, int L, int NS>
__global__ void __launch_bounds__(SCAN_THREADS)
selective_scan_kernel(const T *__restrict__ x, long long ldx, const float *__restrict__ dt_raw, long long ld_dt,
                      const float *__restrict__ dt_bias, const float *__restrict__ bc, long long ld_bc, int off_b, int off_c,
                      const float *__restrict__ z, long long ldz, const float *__restrict__ a_log, const float *__restrict__ skip,
                      float *__restrict__ state, T *__restrict__ out, long long ldo, const int *__restrict__ seq_start,
                      const int *__restrict__ seq_slot, int inner, int N) {
  constexpr int CH = SCAN_THREADS / L, NP = L * NS;      // channels of the CTA, padded states
  constexpr int TG = NP <= 64 ? SCAN_GROUP : 8;          // tokens of a group
  constexpr int PAIRS = (TG * CH + SCAN_THREADS - 1) / SCAN_THREADS, ROWS = SCAN_THREADS / CH;   // (token, channel) pairs a thread brings in
  constexpr int NB = (2 * TG * NP + SCAN_THREADS - 1) / SCAN_THREADS;
  constexpr int NT = TG < 16 ? TG : 16;                  // tokens whose sums over the lanes are made together
  __shared__ __align__(16) float dts[2][CH][TG + 4], dxs[2][CH][TG + 4];   // dt, dt x
  __shared__ __align__(16) float bcs[2][2][TG / 4][NP][4];                 // B, C: four tokens' beside one another
  __shared__ float ys[2][TG][CH];
  grid_dependents_launch();
  const int tid = threadIdx.x, lane = tid % L, ch = tid / L, c = blockIdx.x * CH + ch;
  const int b = blockIdx.y;
  const int lc = tid % CH, lt = tid / CH, gc = blockIdx.x * CH + lc;       // the pairs this thread brings in and stores: tokens lt + i ROWS
  const bool mine = gc < inner;
  const float bias = mine ? dt_bias[gc] : 0.f, dsk = mine ? skip[gc] : 0.f;
  grid_dependency_wait();
  const int start = seq_start[b], n = seq_start[b + 1] - start;
  if (n <= 0) return;
  float *st = state + (size_t)seq_slot[b] * inner * N;
  float al2[NS], S[NS];
  lane_states<L, NS>(a_log, st, c, lane, N, c < inner, al2, S);

  float rx[PAIRS], rd[PAIRS], rz[PAIRS], rb[NB], add[PAIRS], gate[PAIRS];  // on their way; of the group in the works: D x and silu(z)
  auto fetch = [&](int t0) {
#pragma unroll
    for (int i = 0; i < PAIRS; ++i) {
      const int t = lt + i * ROWS;
      const bool in = mine && t < TG && t0 + t < n;
      const size_t row = (size_t)(start + (in ? t0 + t : 0));
      rx[i] = in ? to_float(x[row * ldx + gc]) : 0.f;
      rd[i] = in ? dt_raw[row * ld_dt + gc] : 0.f;
      rz[i] = in ? z[row * ldz + gc] : 0.f;
    }
#pragma unroll
    for (int i = 0; i < NB; ++i) {
      const int k = tid + i * SCAN_THREADS, t = k / (2 * NP), m = k - t * 2 * NP, which = m / NP, s = m - which * NP;
      const bool has = t < TG && t0 + t < n && s < N;
      rb[i] = has ? bc[(size_t)(start + t0 + t) * ld_bc + (which ? off_c : off_b) + s] : 0.f;
    }
  };
  auto leave = [&](int buf, int t0) {
#pragma unroll
    for (int i = 0; i < PAIRS; ++i) {
      const int t = lt + i * ROWS;
      if (t >= TG) continue;
      const float dt = t0 + t < n ? softplus_of<sizeof(T) == 2>(rd[i] + bias) : 0.f;
      dts[buf][lc][t] = dt;
      dxs[buf][lc][t] = dt * rx[i];
    }
#pragma unroll
    for (int i = 0; i < NB; ++i) {
      const int k = tid + i * SCAN_THREADS, t = k / (2 * NP), m = k - t * 2 * NP, which = m / NP, s = m - which * NP;
      if (t < TG) bcs[buf][which][t / 4][s][t % 4] = rb[i];
    }
  };
  auto keep = [&]() {
#pragma unroll
    for (int i = 0; i < PAIRS; ++i) {
      add[i] = dsk * rx[i];
      gate[i] = silu_of<sizeof(T) == 2>(rz[i]);
    }
  };
  fetch(0);
  leave(0, 0);
  keep();
  __syncthreads();
  for (int t0 = 0, g = 0; t0 < n; t0 += TG, ++g) {
    const int buf = g & 1;
    const bool more = t0 + TG < n;
    if (more) fetch(t0 + TG);
#pragma unroll
    for (int q0 = 0; q0 < TG / 4; q0 += NT / 4) {
      float y[NT];
#pragma unroll
      for (int q = 0; q < NT / 4; ++q) {
        const float4 dt = ld4(&dts[buf][ch][4 * (q0 + q)]), dx = ld4(&dxs[buf][ch][4 * (q0 + q)]);
#pragma unroll
        for (int k = 0; k < 4; ++k) y[4 * q + k] = 0.f;
#pragma unroll
        for (int i = 0; i < NS; ++i) {
          const float4 B = ld4(bcs[buf][0][q0 + q][lane + i * L]), C = ld4(bcs[buf][1][q0 + q][lane + i * L]);
          scan_state(S[i], al2[i], dt.x, dx.x, B.x, C.x, y[4 * q]);
          scan_state(S[i], al2[i], dt.y, dx.y, B.y, C.y, y[4 * q + 1]);
          scan_state(S[i], al2[i], dt.z, dx.z, B.z, C.z, y[4 * q + 2]);
          scan_state(S[i], al2[i], dt.w, dx.w, B.w, C.w, y[4 * q + 3]);
        }
      }
      lanes_sums<L, NT>(y, lane);
#pragma unroll
      for (int i = 0; i < (NT > L ? NT / L : 1); ++i)
        if (lane < NT) ys[buf][4 * q0 + first_of<L, NT>(lane) + i][ch] = y[i];
    }
    if (more) leave(buf ^ 1, t0 + TG);
    __syncthreads();
#pragma unroll
    for (int i = 0; i < PAIRS; ++i) {
      const int t = lt + i * ROWS;
      if (mine && t < TG && t0 + t < n)
        out[(size_t)(start + t0 + t) * ldo + gc] = from_float<T>((ys[buf][t][lc] + add[i]) * gate[i]);
    }
    if (more) keep();
  }
#pragma unroll
  for (int i = 0; i < NS; ++i)
    if (c < inner && lane + i * L < N) st[(size_t)c * N + lane + i * L] = S[i];
}

// ---------------------------------------------------------------- a step of single tokens
// Row b is sequence b's token.  low [rows, ..] 32-bit (the sum of low_parts partial products, low_stride floats apart) holds dt_rank
// values, then B and C at their offsets; w_dt [inner, ldw] in the engine's type.
template <typename T, int L, int NS>
__global__ void __launch_bounds__(SS_THREADS)
selective_step_kernel(const T *__restrict__ x, long long ldx, const float *__restrict__ low, long long ld_low, int low_parts,
                      long long low_stride, int rank,
                      const T *__restrict__ w_dt, int ldw, const float *__restrict__ dt_bias, int off_b, int off_c,
                      const float *__restrict__ z, long long ldz, const float *__restrict__ a_log, const float *__restrict__ skip,
                      float *__restrict__ state, T *__restrict__ out, long long ldo, const int *__restrict__ seq_slot, int inner, int N) {
  constexpr int CH = SS_THREADS / L, NP = L * NS;
  extern __shared__ __align__(16) float low_s[];         // B [NP], C [NP], then the dt input [rank]
  grid_dependents_launch();
  const int tid = threadIdx.x, lane = tid % L, c = blockIdx.x * CH + tid / L, b = blockIdx.y;
  const bool in = c < inner;
  const float bias = in ? dt_bias[c] : 0.f, dsk = in ? skip[c] : 0.f;
  float al2[NS], S[NS];
  float *st = state + (size_t)seq_slot[b] * inner * N;
  grid_dependency_wait();
  lane_states<L, NS>(a_log, st, c, lane, N, in, al2, S);
  const float *lr = low + (size_t)b * ld_low;
  for (int i = tid; i < 2 * NP + rank; i += SS_THREADS) {
    const int at = i >= 2 * NP ? i - 2 * NP : i >= NP ? (i - NP < N ? off_c + i - NP : -1) : (i < N ? off_b + i : -1);
    low_s[i] = at >= 0 ? sum_parts(lr + at, low_parts, low_stride) : 0.f;
  }
  const float xv = in ? to_float(x[(size_t)b * ldx + c]) : 0.f, zv = in ? z[(size_t)b * ldz + c] : 0.f;
  __syncthreads();
  float raw = 0.f;
  if (in) {
    const T *w = w_dt + (size_t)c * ldw;
    if (ldw % 4 == 0) {
      for (int r = lane * 4; r < rank; r += L * 4) {     // columns beyond the rank are nought (the matrix is padded to ldw)
        const float4 v = ld4(w + r);
        raw = fmaf(v.x, low_s[2 * NP + r], raw);
        if (r + 1 < rank) raw = fmaf(v.y, low_s[2 * NP + r + 1], raw);
        if (r + 2 < rank) raw = fmaf(v.z, low_s[2 * NP + r + 2], raw);
        if (r + 3 < rank) raw = fmaf(v.w, low_s[2 * NP + r + 3], raw);
      }
    } else {
      for (int r = lane; r < rank; r += L) raw = fmaf(to_float(w[r]), low_s[2 * NP + r], raw);
    }
  }
  const float dt = softplus_of(lanes_sum<L>(raw) + bias);
  float y = 0.f;
#pragma unroll
  for (int i = 0; i < NS; ++i) scan_state(S[i], al2[i], dt, dt * xv, low_s[lane + i * L], low_s[NP + lane + i * L], y);
  y = lanes_sum<L>(y);
#pragma unroll
  for (int i = 0; i < NS; ++i)
    if (in && lane + i * L < N) st[(size_t)c * N + lane + i * L] = S[i];
  if (in && lane == 0) out[(size_t)b * ldo + c] = from_float<T>((y + dsk * xv) * silu_of(zv));
}

}  // namespace

// u [n_tokens, ld] 32-bit -> out [n_tokens, channels] = silu(conv + bias); weight [taps][channels]; state [slots, taps - 1, channels]
// 32-bit (none for one tap).  single_tokens: every sequence brings one token.
LLM_EXPORT int llm_short_conv_silu(int dtype, const float *u, long long ld, const float *weight, const float *bias, int taps, float *state,
                                   void *out, long long ldo, int channels, const int *tok_seq, const int *tok_pos, const int *seq_start,
                                   const int *seq_past, const int *seq_slot, int n_seqs, int n_tokens, int single_tokens, cudaStream_t stream) {
  if (n_tokens == 0) return LLM_OK;
  LLM_REQUIRE(n_tokens > 0 && n_seqs > 0 && channels > 0 && ld >= channels && ldo >= channels && weight, "short_conv_silu: bad sizes");
  LLM_REQUIRE(taps >= 1 && taps <= SC_MAX_TAPS && (taps == 1 || state), "short_conv_silu: %d taps (1 to %d, with their state)", taps, SC_MAX_TAPS);
  const int esz = dtype == LLM_F32 ? 4 : 2;
  const bool vec = channels % 4 == 0 && ld % 4 == 0 && ldo % 4 == 0 && (uintptr_t)u % 16 == 0 && (uintptr_t)weight % 16 == 0 &&
                   (uintptr_t)bias % 16 == 0 && (uintptr_t)state % 16 == 0 && (uintptr_t)out % (4 * esz) == 0;
  const int n_chunks = single_tokens && taps > 1 ? 0 : (n_tokens + SC_ROWS - 1) / SC_ROWS, n_own = taps > 1 ? n_seqs : 0;
  const int units = vec ? channels / 4 : channels;
  const dim3 grid(n_chunks + n_own, (units + SC_THREADS - 1) / SC_THREADS);
  LLM_REQUIRE(grid.y <= 65535, "short_conv_silu: too many channels");
#define SC_GO(T, V, TAPS)                                                                                                      \
  llm_launch(short_conv_silu_kernel<T, V, TAPS>, grid, dim3(SC_THREADS), 0, stream, u, ld, weight, bias, taps, state, (T *)out, ldo, channels, \
             tok_seq, tok_pos, seq_start, seq_past, seq_slot, n_tokens, n_chunks)
#define SC_TAPS(T, V)                  \
  do {                                 \
    if (taps <= 4) SC_GO(T, V, 4);     \
    else SC_GO(T, V, SC_MAX_TAPS);     \
  } while (0)
  if (dtype == LLM_F32 && vec) SC_TAPS(float, 4);
  else if (dtype == LLM_F32) SC_TAPS(float, 1);
  else if (dtype == LLM_BF16 && vec) SC_TAPS(__nv_bfloat16, 4);
  else if (dtype == LLM_BF16) SC_TAPS(__nv_bfloat16, 1);
  else LLM_FAIL("short_conv_silu: unsupported dtype %d", dtype);
#undef SC_TAPS
#undef SC_GO
  LLM_CHECK_LAUNCH("short_conv_silu");
  return LLM_OK;
}

LLM_EXPORT int llm_selective_max_state() { return 256; }

// lanes of a channel and states of a lane for N states per channel: few states a lane over a step's tokens, where the tokens come one
// after another; few lanes in a step of single tokens, whose channels fill the machine
#define SCAN_SHAPES(GO)                   \
  do {                                    \
    if (N <= 16) GO(16, 1);               \
    else if (N <= 32) GO(16, 2);          \
    else if (N <= 64) GO(32, 2);          \
    else if (N <= 128) GO(32, 4);         \
    else GO(32, 8);                       \
  } while (0)
#define STEP_SHAPES(GO)                   \
  do {                                    \
    if (N <= 16) GO(4, 4);                \
    else if (N <= 32) GO(4, 8);           \
    else if (N <= 64) GO(8, 8);           \
    else if (N <= 128) GO(16, 8);         \
    else GO(32, 8);                       \
  } while (0)

// x [n_tokens, inner] in the engine's type (convolved), dt_raw [n_tokens, inner] 32-bit (before its bias), B and C at off_b and off_c
// of the 32-bit rows bc, z [n_tokens, inner] 32-bit; a_log [inner, N], skip (D) [inner], state [slots, inner, N]; out
// [n_tokens, inner] = y silu(z) in the engine's type.
LLM_EXPORT int llm_selective_scan(int dtype, const void *x, long long ldx, const float *dt_raw, long long ld_dt, const float *dt_bias,
                                  const float *bc, long long ld_bc, int off_b, int off_c, const float *z, long long ldz, const float *a_log,
                                  const float *skip, float *state, void *out, long long ldo, const int *seq_start, const int *seq_slot,
                                  int n_seqs, int inner, int N, cudaStream_t stream) {
  if (n_seqs == 0) return LLM_OK;
  LLM_REQUIRE(n_seqs > 0 && n_seqs <= 65535 && inner > 0 && N > 0 && state && a_log && skip && dt_bias, "selective_scan: bad sizes");
  LLM_REQUIRE(N <= llm_selective_max_state(), "selective_scan: %d states a channel are not supported (up to %d)", N, llm_selective_max_state());
#define SS_GO2(T, L, NS)                                                                                                              \
  llm_launch(selective_scan_kernel<T, L, NS>, dim3((inner + SCAN_THREADS / L - 1) / (SCAN_THREADS / L), n_seqs), dim3(SCAN_THREADS), 0, stream,   \
             (const T *)x, ldx, dt_raw, ld_dt, dt_bias, bc, ld_bc, off_b, off_c, z, ldz, a_log, skip, state, (T *)out, ldo, seq_start, seq_slot, \
             inner, N)
#define SS_F32(L, NS) SS_GO2(float, L, NS)
#define SS_BF16(L, NS) SS_GO2(__nv_bfloat16, L, NS)
  if (dtype == LLM_F32) SCAN_SHAPES(SS_F32);
  else if (dtype == LLM_BF16) SCAN_SHAPES(SS_BF16);
  else LLM_FAIL("selective_scan: unsupported dtype %d", dtype);
#undef SS_F32
#undef SS_BF16
#undef SS_GO2
  LLM_CHECK_LAUNCH("selective_scan");
  return LLM_OK;
}

// Single tokens: low [n_seqs, ..] 32-bit rows = the dt input (rank values), B and C at their offsets; w_dt [inner, ldw] in the
// engine's type, columns beyond the rank nought.
LLM_EXPORT int llm_selective_step(int dtype, const void *x, long long ldx, const float *low, long long ld_low, int low_parts,
                                  long long low_stride, int rank, const void *w_dt,
                                  int ldw, const float *dt_bias, int off_b, int off_c, const float *z, long long ldz, const float *a_log,
                                  const float *skip, float *state, void *out, long long ldo, const int *seq_slot, int n_seqs, int inner,
                                  int N, cudaStream_t stream) {
  if (n_seqs == 0) return LLM_OK;
  LLM_REQUIRE(n_seqs > 0 && n_seqs <= 65535 && inner > 0 && N > 0 && rank > 0 && ldw >= rank && state && a_log && skip && dt_bias && w_dt,
              "selective_step: bad sizes");
  LLM_REQUIRE(N <= llm_selective_max_state(), "selective_step: %d states a channel are not supported (up to %d)", N, llm_selective_max_state());
  LLM_REQUIRE(low_parts >= 1 && low_parts <= 64, "selective_step: %d partial products", low_parts);
  LLM_REQUIRE(rank <= 8192, "selective_step: a dt input of %d values is not supported", rank);
  LLM_REQUIRE(ldw % 4 != 0 || (uintptr_t)w_dt % 16 == 0, "selective_step: the dt matrix must start on 16 bytes");
#define SS_GO2(T, L, NS)                                                                                                              \
  llm_launch(selective_step_kernel<T, L, NS>, dim3((inner + SS_THREADS / L - 1) / (SS_THREADS / L), n_seqs), dim3(SS_THREADS),         \
             (size_t)(2 * L * NS + rank) * sizeof(float), stream, (const T *)x, ldx, low, ld_low, low_parts, low_stride, rank, (const T *)w_dt, ldw, dt_bias,  \
             off_b, off_c, z, ldz, a_log, skip, state, (T *)out, ldo, seq_slot, inner, N)
#define SS_F32(L, NS) SS_GO2(float, L, NS)
#define SS_BF16(L, NS) SS_GO2(__nv_bfloat16, L, NS)
  if (dtype == LLM_F32) STEP_SHAPES(SS_F32);
  else if (dtype == LLM_BF16) STEP_SHAPES(SS_BF16);
  else LLM_FAIL("selective_step: unsupported dtype %d", dtype);
#undef SS_F32
#undef SS_BF16
#undef SS_GO2
  LLM_CHECK_LAUNCH("selective_step");
  return LLM_OK;
}

// out [n_rows, cols] bfloat16 = the first n columns of the 32-bit rows `in`, nought beyond them
__global__ void __launch_bounds__(256)
rows_cast_kernel(const float *__restrict__ in, long long ld, int n, __nv_bfloat16 *__restrict__ out, int cols, size_t total) {
  grid_dependents_launch();
  grid_dependency_wait();
  for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (size_t)gridDim.x * blockDim.x) {
    const size_t t = i / cols;
    const int c = (int)(i - t * cols);
    out[i] = __float2bfloat16_rn(c < n ? in[t * ld + c] : 0.f);
  }
}
LLM_EXPORT int llm_rows_cast(const float *in, long long ld, int n, void *out, int n_rows, int cols, cudaStream_t stream) {
  if (n_rows == 0) return LLM_OK;
  LLM_REQUIRE(n_rows > 0 && n > 0 && cols >= n && ld >= n, "rows_cast: bad sizes");
  const size_t total = (size_t)n_rows * cols;
  size_t blocks = (total + 255) / 256;
  if (blocks > (size_t)sm_count() * 16) blocks = (size_t)sm_count() * 16;
  llm_launch(rows_cast_kernel, dim3((unsigned)blocks), dim3(256), 0, stream, in, ld, n, (__nv_bfloat16 *)out, cols, total);
  LLM_CHECK_LAUNCH("rows_cast");
  return LLM_OK;
}
