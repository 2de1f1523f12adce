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
//    N states in registers, and walks the tokens in groups of 16 (8 with many states).  While a group is worked on, the next one's values are on
//    their way into registers; behind it they go, with everything that needs no state already computed (softplus, dt x, D x,
//    silu z), into the other of two buffers in shared memory: one barrier a group.  The only dependence between tokens is the
//    state's fused multiply-add; the sums over n are joined by shuffles off that chain.
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

__device__ __forceinline__ float silu_of(float v) { return v / (1.f + expf(-v)); }
// log(1 + e^v) without overflow: max(v, 0) + log1p(e^-|v|)
__device__ __forceinline__ float softplus_of(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }

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
      y[e] = silu_of(y[e] + bs[e]);
    }
    sc_store<T, V>(out + (size_t)row * ldo + c0, y);
  };
  if ((int)blockIdx.x < n_chunks) {
    const int r0 = blockIdx.x * SC_ROWS, r1 = min(n_tokens, r0 + SC_ROWS);
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
constexpr int SS_THREADS = 128;

// One token of one lane's states: a = exp2(dt A log2 e), S <- a S + dx B, sum += S C.  al2: A log2 e.
template <int NS>
__device__ __forceinline__ float scan_token(float (&S)[NS], const float (&al2)[NS], float dt, float dx, const float *__restrict__ B,
                                            const float *__restrict__ C) {
  float acc = 0.f;
#pragma unroll
  for (int i = 0; i < NS; i += 4) {
    const float4 b = ld4(B + i), c = ld4(C + i);
    const float bb[4] = {b.x, b.y, b.z, b.w}, cc[4] = {c.x, c.y, c.z, c.w};
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      S[i + k] = fmaf(exp2f(dt * al2[i + k]), S[i + k], dx * bb[k]);
      acc = fmaf(S[i + k], cc[k], acc);
    }
  }
  return acc;
}
template <int L>
__device__ __forceinline__ float lanes_sum(float v) {
#pragma unroll
  for (int o = 1; o < L; o <<= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

// a lane's states' decays (al2) and, if wanted, the states themselves; states beyond N are nought and stay so
template <int NS>
__device__ __forceinline__ void lane_states(const float *__restrict__ a_log, const float *__restrict__ st, int c, int n0, int N, bool in,
                                            float (&al2)[NS], float (&S)[NS]) {
#pragma unroll
  for (int i = 0; i < NS; ++i) {
    const bool has = in && n0 + i < N;
    al2[i] = has ? -expf(a_log[(size_t)c * N + n0 + i]) * LOG2E : 0.f;
    S[i] = has ? st[(size_t)c * N + n0 + i] : 0.f;
  }
}

template <typename T, int L, int NS>
__global__ void __launch_bounds__(SS_THREADS)
selective_scan_kernel(const T *__restrict__ x, long long ldx, const float *__restrict__ dt_raw, long long ld_dt,
                      const float *__restrict__ dt_bias, const float *__restrict__ bc, long long ld_bc, int off_b, int off_c,
                      const float *__restrict__ z, long long ldz, const float *__restrict__ a_log, const float *__restrict__ skip,
                      float *__restrict__ state, T *__restrict__ out, long long ldo, const int *__restrict__ seq_start,
                      const int *__restrict__ seq_slot, int inner, int N) {
  constexpr int CH = SS_THREADS / L, NP = L * NS;        // channels of the CTA, padded states
  constexpr int SS_TG = NP <= 128 ? 16 : 8;              // tokens of a group
  constexpr int PER = SS_TG * CH / SS_THREADS;           // (token, channel) pairs a thread brings in (none: some threads bring one)
  constexpr int PAIRS = PER > 0 ? PER : 1;
  constexpr int NB = (2 * SS_TG * NP + SS_THREADS - 1) / SS_THREADS;
  __shared__ __align__(16) float4 tok[2][SS_TG][CH];     // dt, dt x, D x, silu(z)
  __shared__ __align__(16) float bcs[2][SS_TG][2][NP];
  __shared__ float ys[2][SS_TG][CH];
  grid_dependents_launch();
  const int tid = threadIdx.x, lane = tid % L, ch = tid / L, c = blockIdx.x * CH + ch, n0 = lane * NS;
  const int b = blockIdx.y;
  // the pairs this thread brings in: channel lc of tokens lt + i * (SS_THREADS / CH)
  const int lc = tid % CH, lt = tid / CH, gc = blockIdx.x * CH + lc;
  const bool l_in = gc < inner;
  const float bias = l_in ? dt_bias[gc] : 0.f, dsk = l_in ? skip[gc] : 0.f;
  grid_dependency_wait();
  const int start = seq_start[b], n = seq_start[b + 1] - start;
  if (n <= 0) return;
  float *st = state + (size_t)seq_slot[b] * inner * N;
  float al2[NS], S[NS];
  lane_states<NS>(a_log, st, c, n0, N, c < inner, al2, S);

  float rx[PAIRS], rd[PAIRS], rz[PAIRS], rb[NB];
  auto fetch = [&](int t0) {
#pragma unroll
    for (int i = 0; i < PAIRS; ++i) {
      const int t = t0 + lt + i * (SS_THREADS / CH);
      const bool in = l_in && t < n && lt + i * (SS_THREADS / CH) < SS_TG;
      const size_t row = (size_t)(start + (in ? t : 0));
      rx[i] = in ? to_float(x[row * ldx + gc]) : 0.f;
      rd[i] = in ? dt_raw[row * ld_dt + gc] : 0.f;
      rz[i] = in ? z[row * ldz + gc] : 0.f;
    }
#pragma unroll
    for (int i = 0; i < NB; ++i) {
      const int k = tid + i * SS_THREADS, t = k / (2 * NP), m = k - t * 2 * NP, which = m / NP, s = m - which * NP;
      const bool in = t < SS_TG && t0 + t < n && s < N;
      rb[i] = in ? bc[(size_t)(start + t0 + t) * ld_bc + (which ? off_c : off_b) + s] : 0.f;
    }
  };
  auto leave = [&](int buf) {
#pragma unroll
    for (int i = 0; i < PAIRS; ++i) {
      const int t = lt + i * (SS_THREADS / CH);
      if (t >= SS_TG) continue;
      const float dt = softplus_of(rd[i] + bias);
      tok[buf][t][lc] = make_float4(dt, dt * rx[i], dsk * rx[i], silu_of(rz[i]));
    }
#pragma unroll
    for (int i = 0; i < NB; ++i) {
      const int k = tid + i * SS_THREADS;
      if (k < 2 * SS_TG * NP) (&bcs[buf][0][0][0])[k] = rb[i];
    }
  };
  auto store = [&](int t0, int buf) {                    // a finished group's rows
#pragma unroll
    for (int i = 0; i < PAIRS; ++i) {
      const int t = lt + i * (SS_THREADS / CH);
      if (t < SS_TG && t0 + t < n && l_in) out[(size_t)(start + t0 + t) * ldo + gc] = from_float<T>(ys[buf][t][lc]);
    }
  };
  fetch(0);
  leave(0);
  __syncthreads();
  for (int t0 = 0, g = 0; t0 < n; t0 += SS_TG, ++g) {
    const int buf = g & 1;
    const bool more = t0 + SS_TG < n;
    if (more) fetch(t0 + SS_TG);
    const int nt = min(SS_TG, n - t0);
    auto one = [&](int t) {
      const float4 v = tok[buf][t][ch];
      const float y = lanes_sum<L>(scan_token<NS>(S, al2, v.x, v.y, &bcs[buf][t][0][n0], &bcs[buf][t][1][n0]));
      if (lane == 0) ys[buf][t][ch] = (y + v.z) * v.w;
    };
    if (nt == SS_TG) {
#pragma unroll 4
      for (int t = 0; t < SS_TG; ++t) one(t);
    } else {
      for (int t = 0; t < nt; ++t) one(t);
    }
    if (more) leave(buf ^ 1);
    __syncthreads();
    store(t0, buf);
  }
#pragma unroll
  for (int i = 0; i < NS; ++i)
    if (c < inner && n0 + i < N) st[(size_t)c * N + n0 + i] = S[i];
}

// ---------------------------------------------------------------- a step of single tokens
// Row b is sequence b's token.  low [rows, ..] 32-bit holds dt_rank values, then B and C at their offsets; w_dt [inner, ldw] in the
// engine's type.
template <typename T, int L, int NS>
__global__ void __launch_bounds__(SS_THREADS)
selective_step_kernel(const T *__restrict__ x, long long ldx, const float *__restrict__ low, long long ld_low, int rank,
                      const T *__restrict__ w_dt, int ldw, const float *__restrict__ dt_bias, int off_b, int off_c,
                      const float *__restrict__ z, long long ldz, const float *__restrict__ a_log, const float *__restrict__ skip,
                      float *__restrict__ state, T *__restrict__ out, long long ldo, const int *__restrict__ seq_slot, int inner, int N) {
  constexpr int CH = SS_THREADS / L, NP = L * NS;
  extern __shared__ float low_s[];                       // B [NP], C [NP], then the dt input [rank]
  grid_dependents_launch();
  const int tid = threadIdx.x, lane = tid % L, c = blockIdx.x * CH + tid / L, n0 = lane * NS, b = blockIdx.y;
  const bool in = c < inner;
  const float bias = in ? dt_bias[c] : 0.f, dsk = in ? skip[c] : 0.f;
  float al2[NS], S[NS];
  float *st = state + (size_t)seq_slot[b] * inner * N;
  grid_dependency_wait();
  lane_states<NS>(a_log, st, c, n0, N, in, al2, S);
  const float *lr = low + (size_t)b * ld_low;
  for (int i = tid; i < 2 * NP + rank; i += SS_THREADS)
    low_s[i] = i >= 2 * NP ? lr[i - 2 * NP] : i >= NP ? (i - NP < N ? lr[off_c + i - NP] : 0.f) : (i < N ? lr[off_b + i] : 0.f);
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
  const float y = lanes_sum<L>(scan_token<NS>(S, al2, dt, dt * xv, low_s + n0, low_s + NP + n0));
#pragma unroll
  for (int i = 0; i < NS; ++i)
    if (in && n0 + i < N) st[(size_t)c * N + n0 + i] = S[i];
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

// lanes of a channel and states of a lane for N states per channel
#define SS_SHAPES(GO)                     \
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
  llm_launch(selective_scan_kernel<T, L, NS>, dim3((inner + SS_THREADS / L - 1) / (SS_THREADS / L), n_seqs), dim3(SS_THREADS), 0, stream,       \
             (const T *)x, ldx, dt_raw, ld_dt, dt_bias, bc, ld_bc, off_b, off_c, z, ldz, a_log, skip, state, (T *)out, ldo, seq_start, seq_slot, \
             inner, N)
#define SS_F32(L, NS) SS_GO2(float, L, NS)
#define SS_BF16(L, NS) SS_GO2(__nv_bfloat16, L, NS)
  if (dtype == LLM_F32) SS_SHAPES(SS_F32);
  else if (dtype == LLM_BF16) SS_SHAPES(SS_BF16);
  else LLM_FAIL("selective_scan: unsupported dtype %d", dtype);
#undef SS_F32
#undef SS_BF16
#undef SS_GO2
  LLM_CHECK_LAUNCH("selective_scan");
  return LLM_OK;
}

// Single tokens: low [n_seqs, ..] 32-bit rows = the dt input (rank values), B and C at their offsets; w_dt [inner, ldw] in the
// engine's type, columns beyond the rank nought.
LLM_EXPORT int llm_selective_step(int dtype, const void *x, long long ldx, const float *low, long long ld_low, int rank, const void *w_dt,
                                  int ldw, const float *dt_bias, int off_b, int off_c, const float *z, long long ldz, const float *a_log,
                                  const float *skip, float *state, void *out, long long ldo, const int *seq_slot, int n_seqs, int inner,
                                  int N, cudaStream_t stream) {
  if (n_seqs == 0) return LLM_OK;
  LLM_REQUIRE(n_seqs > 0 && n_seqs <= 65535 && inner > 0 && N > 0 && rank > 0 && ldw >= rank && state && a_log && skip && dt_bias && w_dt,
              "selective_step: bad sizes");
  LLM_REQUIRE(N <= llm_selective_max_state(), "selective_step: %d states a channel are not supported (up to %d)", N, llm_selective_max_state());
  LLM_REQUIRE(rank <= 8192, "selective_step: a dt input of %d values is not supported", rank);
  LLM_REQUIRE(ldw % 4 != 0 || (uintptr_t)w_dt % 16 == 0, "selective_step: the dt matrix must start on 16 bytes");
#define SS_GO2(T, L, NS)                                                                                                              \
  llm_launch(selective_step_kernel<T, L, NS>, dim3((inner + SS_THREADS / L - 1) / (SS_THREADS / L), n_seqs), dim3(SS_THREADS),         \
             (size_t)(2 * L * NS + rank) * sizeof(float), stream, (const T *)x, ldx, low, ld_low, rank, (const T *)w_dt, ldw, dt_bias,  \
             off_b, off_c, z, ldz, a_log, skip, state, (T *)out, ldo, seq_slot, inner, N)
#define SS_F32(L, NS) SS_GO2(float, L, NS)
#define SS_BF16(L, NS) SS_GO2(__nv_bfloat16, L, NS)
  if (dtype == LLM_F32) SS_SHAPES(SS_F32);
  else if (dtype == LLM_BF16) SS_SHAPES(SS_BF16);
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
