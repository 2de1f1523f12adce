// Linear recurrences over a matrix of state per head, in three rules that share one scan:
//
//   gated delta   S <- g S;  z = beta (v - S^T k);  S <- S + k z^T;  o = S^T q          (one decay g per head)
//   bonus         o = (S + diag(u) k v^T)^T r;  S <- diag(w) S + k v^T                    (a decay w per key channel)
//   memory        S <- f S + i k v^T;  n <- f n + i k;  o = S^T q, den = n . q            (decay f, input gate i per head)
//
// Each is out = a (S_old^T q) + c z, then S <- W S + k z^T, for a column of S at a time:
//   gated delta   W = a = g, z = beta (v - g S_old^T k), c = k . q
//   bonus         W = w (a vector), a = 1, z = v, c = sum_i r_i u_i k_i
//   memory        W = a = f, z = i v, c = k . q; n is one more column whose v is 1
// so that no result waits for the state it was made with: the two products with the old state are taken side by side.
// What the tokens bring is packed first (the pack kernels below), a head's tokens one behind the other, so that the scan takes
// a run of tokens with one bulk copy for each kind: records of vectors rec [key heads, tokens, k | q (r) | w (bonus)], each
// vector padded with zeros (scan_dmax); scalars scal [heads, tokens, 4] = (a, beta or i, c, spare); values
// vals [heads, slices, tokens, columns of a slice].  state [slots, heads, columns, d]: the d rows of a column together.  A step of single tokens
// has a kernel per rule that does everything between the products of h and the output projection in one launch.
//
// Everything here is 32-bit.  A sequence's result depends on nothing but its own tokens and state: one column belongs
// to a few neighbouring lanes, sums run in a fixed order, no sum crosses sequences.  The reference has no such mixer (its
// one mixer is attention, src/libllm/llama.cc:178-225).
#include "common.cuh"
#include "tc_common.cuh"
#include <math.h>

LLM_DEFINE_LAST_ERROR(llm_state_scan_last_error)

enum Rule { RULE_DELTA = 0, RULE_BONUS = 1, RULE_MEMORY = 2 };

__device__ __forceinline__ float sigmoid32(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float silu32(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float softplus32(float x) { return x > 20.f ? x : log1pf(expf(x)); }
__device__ __forceinline__ float log_sigmoid32(float x) { return fminf(x, 0.f) - log1pf(expf(-fabsf(x))); }
// a vector's place in a record: the head's rows padded with zeros to what the scan's lanes hold
__host__ __device__ constexpr int scan_dmax(int d) { return d <= 16 ? 16 : d <= 32 ? 32 : d <= 64 ? 64 : d <= 128 ? 128 : 256; }

// ---------------------------------------------------------------- the scan over a step's tokens
// CTA (sequence, head, slice of columns): SC_THREADS threads of arithmetic, LANES neighbouring lanes to two columns (lane `sub`
// owns rows 4 (sub + LANES i) .. + 3), and a warp one lane of which brings groups of SC_GROUP tokens into a ring in shared
// memory by bulk copies, several groups ahead of the arithmetic.  Every wait has a time limit (tc_common.cuh).
constexpr int SC_THREADS = 64;
constexpr int SC_GROUP = 8;

__host__ __device__ constexpr int scan_lanes(int dmax) { return dmax <= 64 ? dmax / 8 : dmax / 16; }
// columns of a slice, and slices of a head (memory: one more column, n)
__host__ __device__ constexpr int scan_cols(int d) { return 2 * SC_THREADS / scan_lanes(scan_dmax(d)); }
__host__ __device__ constexpr int scan_slices(int d, int n_cols) { return (n_cols + scan_cols(d) - 1) / scan_cols(d); }

inline int scan_shift(int d) {
  int s = 0;
  while ((1 << s) < scan_cols(d)) ++s;
  return s;
}
// floats of a vector in a record, and of a slice's row of values
LLM_EXPORT int llm_scan_padded(int d) { return scan_dmax(d); }
LLM_EXPORT int llm_scan_columns(int d) { return scan_cols(d); }

__device__ __forceinline__ void bulk_load(unsigned dst, const void *src, unsigned bytes, unsigned bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
               ::"r"(dst), "l"(src), "r"(bytes), "r"(bar) : "memory");
}

// This lane's share of a column: the token's products with the old state, then the new state.  kk, qq, ww point at the
// token's vectors in shared memory; two rows to an instruction (packed 32-bit pairs).
template <int RULE, int LANES, int ROWS>
__device__ __forceinline__ float scan_token(float2 (&S)[ROWS / 2], const float *kk, const float *qq, const float *ww, float4 sc, float v, int sub) {
  float4 k4[ROWS / 4];
  float2 p[2] = {make_float2(0.f, 0.f), make_float2(0.f, 0.f)}, r[2] = {make_float2(0.f, 0.f), make_float2(0.f, 0.f)};
#pragma unroll
  for (int i = 0; i < ROWS / 4; ++i) {
    const int at = 4 * (sub + LANES * i);
    k4[i] = ld4(kk + at);
    const float4 q4 = ld4(qq + at);
    r[0] = __ffma2_rn(make_float2(q4.x, q4.y), S[2 * i], r[0]);
    r[1] = __ffma2_rn(make_float2(q4.z, q4.w), S[2 * i + 1], r[1]);
    if (RULE == RULE_DELTA) {
      p[0] = __ffma2_rn(make_float2(k4[i].x, k4[i].y), S[2 * i], p[0]);
      p[1] = __ffma2_rn(make_float2(k4[i].z, k4[i].w), S[2 * i + 1], p[1]);
    }
  }
  const float2 r2 = __fadd2_rn(r[0], r[1]);
  float rs = r2.x + r2.y, z;
  if (RULE == RULE_DELTA) {
    const float2 p2 = __fadd2_rn(p[0], p[1]);
    float ps = p2.x + p2.y;
#pragma unroll
    for (int o = 1; o < LANES; o <<= 1) ps += __shfl_xor_sync(0xffffffffu, ps, o);
    z = sc.y * fmaf(-sc.x, ps, v);
  } else {
    z = RULE == RULE_BONUS ? v : sc.y * v;
  }
  const float2 z2 = make_float2(z, z), a2 = make_float2(sc.x, sc.x);
#pragma unroll
  for (int i = 0; i < ROWS / 4; ++i) {
    float2 w0 = a2, w1 = a2;
    if (RULE == RULE_BONUS) {
      const float4 w4 = ld4(ww + 4 * (sub + LANES * i));
      w0 = make_float2(w4.x, w4.y);
      w1 = make_float2(w4.z, w4.w);
    }
    S[2 * i] = __ffma2_rn(w0, S[2 * i], __fmul2_rn(make_float2(k4[i].x, k4[i].y), z2));
    S[2 * i + 1] = __ffma2_rn(w1, S[2 * i + 1], __fmul2_rn(make_float2(k4[i].z, k4[i].w), z2));
  }
#pragma unroll
  for (int o = 1; o < LANES; o <<= 1) rs += __shfl_xor_sync(0xffffffffu, rs, o);
  return fmaf(sc.z, z, RULE == RULE_BONUS ? rs : sc.x * rs);
}

// Loads that say they read shared memory, in the order they are written: a token's vectors are asked for a token ahead.
__device__ __forceinline__ float4 shared_ld4(unsigned at) {
  float4 v;
  asm volatile("ld.shared.v4.f32 {%0, %1, %2, %3}, [%4];" : "=f"(v.x), "=f"(v.y), "=f"(v.z), "=f"(v.w) : "r"(at));
  return v;
}
__device__ __forceinline__ float2 shared_ld2(unsigned at) {
  float2 v;
  asm volatile("ld.shared.v2.f32 {%0, %1}, [%2];" : "=f"(v.x), "=f"(v.y) : "r"(at));
  return v;
}

// The same for N tokens in a row and two columns of a lane: the read-outs' sums over the lanes wait until the group is through
// (nothing in it needs them), and a token's vectors are on their way while the token before is worked on.
template <int RULE, int LANES, int ROWS, int REC, int DMAX, int N>
__device__ __forceinline__ void scan_group(float2 (&S)[2][ROWS / 2], unsigned rec, unsigned scal, unsigned vals, unsigned v_step,
                                           float (&out)[2][N]) {
  constexpr int NV = RULE == RULE_BONUS ? 3 : 2;
  float4 x[2][NV][ROWS / 4], sc[2];
  float2 v[2];
  float rs[2][N], cz[2][N];
  auto fetch = [&](int e) {
#pragma unroll
    for (int k = 0; k < NV; ++k)
#pragma unroll
      for (int i = 0; i < ROWS / 4; ++i) x[e & 1][k][i] = shared_ld4(rec + (e * REC + k * DMAX + 4 * LANES * i) * 4);
    sc[e & 1] = shared_ld4(scal + e * 16);
    v[e & 1] = shared_ld2(vals + e * v_step);
  };
  fetch(0);
#pragma unroll
  for (int e = 0; e < N; ++e) {
    if (e + 1 < N) fetch(e + 1);
    __syncwarp();                                     // keeps the loads where they are written: ahead of this token's work
    const float4 (&k4)[ROWS / 4] = x[e & 1][0], (&q4)[ROWS / 4] = x[e & 1][1];
    const float4 s4 = sc[e & 1];
    float z[2];
    if (RULE == RULE_DELTA) {
      float ps[2];
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        float2 p0 = make_float2(0.f, 0.f), p1 = p0;
#pragma unroll
        for (int i = 0; i < ROWS / 4; ++i) {
          p0 = __ffma2_rn(make_float2(k4[i].x, k4[i].y), S[c][2 * i], p0);
          p1 = __ffma2_rn(make_float2(k4[i].z, k4[i].w), S[c][2 * i + 1], p1);
        }
        p0 = __fadd2_rn(p0, p1);
        ps[c] = p0.x + p0.y;
      }
#pragma unroll
      for (int o = 1; o < LANES; o <<= 1)
#pragma unroll
        for (int c = 0; c < 2; ++c) ps[c] += __shfl_xor_sync(0xffffffffu, ps[c], o);
      z[0] = s4.y * fmaf(-s4.x, ps[0], v[e & 1].x);
      z[1] = s4.y * fmaf(-s4.x, ps[1], v[e & 1].y);
    } else {
      z[0] = RULE == RULE_BONUS ? v[e & 1].x : s4.y * v[e & 1].x;
      z[1] = RULE == RULE_BONUS ? v[e & 1].y : s4.y * v[e & 1].y;
    }
#pragma unroll
    for (int c = 0; c < 2; ++c) {
      float2 r0 = make_float2(0.f, 0.f), r1 = r0;
#pragma unroll
      for (int i = 0; i < ROWS / 4; ++i) {
        r0 = __ffma2_rn(make_float2(q4[i].x, q4[i].y), S[c][2 * i], r0);
        r1 = __ffma2_rn(make_float2(q4[i].z, q4[i].w), S[c][2 * i + 1], r1);
      }
      r0 = __fadd2_rn(r0, r1);
      rs[c][e] = RULE == RULE_BONUS ? r0.x + r0.y : s4.x * (r0.x + r0.y);
      cz[c][e] = s4.z * z[c];
      const float2 z2 = make_float2(z[c], z[c]);
      float2 w0 = make_float2(s4.x, s4.x), w1 = w0;
#pragma unroll
      for (int i = 0; i < ROWS / 4; ++i) {
        if constexpr (RULE == RULE_BONUS) {
          w0 = make_float2(x[e & 1][2][i].x, x[e & 1][2][i].y);
          w1 = make_float2(x[e & 1][2][i].z, x[e & 1][2][i].w);
        }
        S[c][2 * i] = __ffma2_rn(w0, S[c][2 * i], __fmul2_rn(make_float2(k4[i].x, k4[i].y), z2));
        S[c][2 * i + 1] = __ffma2_rn(w1, S[c][2 * i + 1], __fmul2_rn(make_float2(k4[i].z, k4[i].w), z2));
      }
    }
  }
#pragma unroll
  for (int o = 1; o < LANES; o <<= 1)
#pragma unroll
    for (int e = 0; e < N; ++e)
#pragma unroll
      for (int c = 0; c < 2; ++c) rs[c][e] += __shfl_xor_sync(0xffffffffu, rs[c][e], o);
#pragma unroll
  for (int e = 0; e < N; ++e)
#pragma unroll
    for (int c = 0; c < 2; ++c) out[c][e] = rs[c][e] + cz[c][e];
}

template <int RULE, int DMAX>
__global__ void __launch_bounds__(SC_THREADS + 32)
state_scan_kernel(const float *__restrict__ rec, const float4 *__restrict__ scal, const float *__restrict__ vals, float *__restrict__ state,
                  float *__restrict__ out, long long ldo, float *__restrict__ den, const int *__restrict__ seq_start,
                  const int *__restrict__ seq_slot, int n_tokens, int n_heads, int n_kv, int d, int dv, int n_groups_ring, int *status) {
  constexpr int NV = RULE == RULE_BONUS ? 3 : 2;
  constexpr int LANES = scan_lanes(DMAX), ROWS = DMAX / LANES, COLS = 2 * SC_THREADS / LANES;
  extern __shared__ __align__(128) unsigned char sc_smem[];
  // a group in the ring: records [tokens][NV * DMAX], values [tokens][COLS], scalars [tokens][4]
  constexpr int rec_f = NV * DMAX, group_f = SC_GROUP * (rec_f + COLS + 4);
  float *ring = reinterpret_cast<float *>(sc_smem);
  unsigned long long *bars = reinterpret_cast<unsigned long long *>(ring + (size_t)n_groups_ring * group_f);
  const unsigned bar_full = smem_u32(bars), bar_empty = smem_u32(bars + n_groups_ring);
  volatile int *abort_flag = reinterpret_cast<volatile int *>(bars + 2 * n_groups_ring);
  const int tid = threadIdx.x;
  if (tid == 0) {
    for (int g = 0; g < n_groups_ring; ++g) {
      mbar_init(bar_full + 8 * g, 1);
      mbar_init(bar_empty + 8 * g, SC_THREADS / 32);
    }
    *abort_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  __syncthreads();
  grid_dependency_wait();
  const int b = blockIdx.x, hd = blockIdx.y, slice = blockIdx.z, kvh = hd / (n_heads / n_kv);
  const int start = seq_start[b], n = seq_start[b + 1] - start;
  const int n_groups = (n + SC_GROUP - 1) / SC_GROUP;
  const int n_cols = dv + (RULE == RULE_MEMORY ? 1 : 0);

  if (tid >= SC_THREADS) {
    const bool leader = elect_one();
    const float *r = rec + ((size_t)kvh * n_tokens + start) * rec_f;
    const float *v = vals + (((size_t)hd * gridDim.z + slice) * n_tokens + start) * COLS;
    const float4 *s = scal + (size_t)hd * n_tokens + start;
    bool ok = true;
    int slot = 0;
    unsigned phase = 0;
    for (int p = 0; p < n_groups && ok; ++p) {
      ok = __all_sync(0xffffffffu, mbar_wait(bar_empty + 8 * slot, phase ^ 1, abort_flag, status, 71));
      if (!ok) break;
      if (leader) {
        const int t0 = p * SC_GROUP, nt = min(SC_GROUP, n - t0);
        const unsigned dst = smem_u32(ring + (size_t)slot * group_f);
        mbar_expect_tx(bar_full + 8 * slot, (unsigned)(nt * (rec_f + COLS + 4) * 4));
        bulk_load(dst, r + (size_t)t0 * rec_f, (unsigned)(nt * rec_f * 4), bar_full + 8 * slot);
        bulk_load(dst + SC_GROUP * rec_f * 4, v + (size_t)t0 * COLS, (unsigned)(nt * COLS * 4), bar_full + 8 * slot);
        bulk_load(dst + SC_GROUP * (rec_f + COLS) * 4, s + t0, (unsigned)(nt * 16), bar_full + 8 * slot);
      }
      __syncwarp();
      if (++slot == n_groups_ring) {
        slot = 0;
        phase ^= 1;
      }
    }
    if (leader && (!ok || *abort_flag)) {             // copies in flight land before the shared memory goes
      const unsigned long long t0 = globaltimer();
      for (int g = 0; g < n_groups_ring; ++g)
        while (!mbar_try(bar_full + 8 * g, 0) && !mbar_try(bar_full + 8 * g, 1) && globaltimer() - t0 < 2000000ull) {
        }
    }
    return;
  }

  const int sub = tid % LANES, col = 2 * (tid / LANES), j = slice * COLS + col;
  float2 S[2][ROWS / 2];
  float *sp = state + ((size_t)seq_slot[b] * n_heads + hd) * n_cols * (size_t)d;
  auto row_of = [&](int i) { return 4 * (sub + LANES * (i / 4)) + i % 4; };
#pragma unroll
  for (int c = 0; c < 2; ++c)
#pragma unroll
    for (int i = 0; i < ROWS; i += 2) {
      const float *column = sp + (size_t)(j + c < n_cols ? j + c : 0) * d;
      S[c][i / 2].x = j + c < n_cols && row_of(i) < d ? column[row_of(i)] : 0.f;
      S[c][i / 2].y = j + c < n_cols && row_of(i + 1) < d ? column[row_of(i + 1)] : 0.f;
    }
  // lane 0 of the columns' lanes writes the first column's results, lane 1 the second's
  const int jw = j + sub;
  const bool writes = sub < 2 && jw < n_cols, to_den = RULE == RULE_MEMORY && jw == dv;
  float *dst = to_den ? den + (size_t)start * n_heads + hd : out + (size_t)start * ldo + (size_t)hd * dv + jw;
  const long long step = to_den ? n_heads : ldo;
  bool ok = true;
  int slot = 0;
  unsigned phase = 0;
  for (int p = 0; p < n_groups; ++p) {
    ok = __all_sync(0xffffffffu, mbar_wait(bar_full + 8 * slot, phase, abort_flag, status, 72));
    if (!ok) break;
    const unsigned g = smem_u32(ring + (size_t)slot * group_f), gr = g + 16 * sub, gv = g + (SC_GROUP * rec_f + col) * 4,
                   gs = g + SC_GROUP * (rec_f + COLS) * 4;
    const int nt = n - p * SC_GROUP;
    if (nt >= SC_GROUP) {
      float o[2][SC_GROUP];
      scan_group<RULE, LANES, ROWS, rec_f, DMAX, SC_GROUP>(S, gr, gs, gv, COLS * 4, o);
#pragma unroll
      for (int e = 0; e < SC_GROUP; ++e) {
        if (writes) *dst = sub ? o[1][e] : o[0][e];
        dst += step;
      }
    } else {
      for (int e = 0; e < nt; ++e) {
        float o[2][1];
        scan_group<RULE, LANES, ROWS, rec_f, DMAX, 1>(S, gr + e * rec_f * 4, gs + e * 16, gv + e * COLS * 4, COLS * 4, o);
        if (writes) *dst = sub ? o[1][0] : o[0][0];
        dst += step;
      }
    }
    __syncwarp();
    if ((tid & 31) == 0) mbar_arrive(bar_empty + 8 * slot);
    if (++slot == n_groups_ring) {
      slot = 0;
      phase ^= 1;
    }
  }
  // only now: this kernel is narrow and runs long, and a dependent let in at its start would sit beside it all that time
  grid_dependents_launch();
#pragma unroll
  for (int c = 0; c < 2; ++c)
#pragma unroll
    for (int i = 0; i < ROWS; ++i)
      if (j + c < n_cols && row_of(i) < d) sp[(size_t)(j + c) * d + row_of(i)] = i % 2 ? S[c][i / 2].y : S[c][i / 2].x;
}

// rec [kv_heads, tokens, 2 or 3, llm_scan_padded(d)], scal [heads, tokens, 4], vals [heads, slices, tokens, columns] (llm_scan_columns), state
// [slots, heads, dv (memory: + 1), d], out [tokens, heads * dv]; den [tokens, heads] (memory).  Launched behind its predecessor.
LLM_EXPORT int llm_state_scan(int rule, const float *rec, const float *scal, const float *vals, float *state, float *out, long long ldo,
                              float *den, const int *seq_start, const int *seq_slot, int n_tokens, int n_seqs, int n_heads, int n_kv, int d,
                              int dv, int *status, cudaStream_t stream) {
  if (n_tokens == 0) return LLM_OK;
  LLM_REQUIRE(rule >= 0 && rule <= 2, "state_scan: rule %d is not known", rule);
  LLM_REQUIRE(n_tokens > 0 && n_seqs > 0 && n_heads > 0 && n_kv > 0 && n_heads % n_kv == 0 && d > 0 && dv > 0, "state_scan: bad sizes");
  LLM_REQUIRE(d <= 256, "state_scan: heads of %d key channels are not supported (up to 256)", d);
  LLM_REQUIRE(n_heads <= 65535, "state_scan: too many heads");
  LLM_REQUIRE((uintptr_t)rec % 16 == 0 && (uintptr_t)scal % 16 == 0 && (uintptr_t)vals % 16 == 0 && (rule != RULE_MEMORY || den), "state_scan: bad pointers");
  const int n_cols = dv + (rule == RULE_MEMORY ? 1 : 0), slices = scan_slices(d, n_cols), dmax = scan_dmax(d);
  LLM_REQUIRE(slices <= 65535, "state_scan: too many value channels");
  const size_t group_bytes = (size_t)SC_GROUP * ((rule == RULE_BONUS ? 3 : 2) * scan_dmax(d) + scan_cols(d) + 4) * sizeof(float);
  int ring = (int)(40 * 1024 / group_bytes);
  ring = ring < 3 ? 3 : ring > 8 ? 8 : ring;
  const size_t smem = ring * group_bytes + 16 * ring + 16;
#define SC_GO(RULE, DMAX)                                                                                                    \
  do {                                                                                                                       \
    LLM_CHECK_CUDA(llm_allow_smem(state_scan_kernel<RULE, DMAX>, smem), "state_scan attribute");                             \
    llm_launch_after(state_scan_kernel<RULE, DMAX>, dim3(n_seqs, n_heads, slices), dim3(SC_THREADS + 32), smem, stream, rec, \
                     (const float4 *)scal, vals, state, out, ldo, den, seq_start, seq_slot, n_tokens, n_heads, n_kv, d, dv, ring, status); \
  } while (0)
#define SC_SIZES(RULE)                   \
  do {                                   \
    if (dmax == 16) SC_GO(RULE, 16);     \
    else if (dmax == 32) SC_GO(RULE, 32); \
    else if (dmax == 64) SC_GO(RULE, 64); \
    else if (dmax == 128) SC_GO(RULE, 128); \
    else SC_GO(RULE, 256);               \
  } while (0)
  if (rule == RULE_DELTA) SC_SIZES(RULE_DELTA);
  else if (rule == RULE_BONUS) SC_SIZES(RULE_BONUS);
  else SC_SIZES(RULE_MEMORY);
#undef SC_SIZES
#undef SC_GO
  LLM_CHECK_LAUNCH("state_scan");
  return LLM_OK;
}

// ---------------------------------------------------------------- what a token brings, packed for the scan
// where value column j of a head's token t lies in vals
struct ValuePlace {
  int cols, slices, shift;                            // cols = 2^shift
  long long n_tokens;
  __device__ __forceinline__ size_t at(int head, long long t, int j) const {
    return ((((size_t)head * slices + (j >> shift)) * n_tokens + t) << shift) + (j & (cols - 1));
  }
};

// Gated delta: rows of the product hold q, k (kv_heads x d) and v (heads x dv) one behind the other.  Each channel through a
// causal convolution over time (weight [channels, taps], nought before the sequence's start) and silu; q and k become unit
// vectors per key head, x / sqrt(sum x^2 + key_eps), q also times q_scale; per head beta = sigmoid(b), g = exp(-exp(a_log) softplus(a +
// dt_bias)), a and b at their offsets of the rows.  A warp takes a key head's q and k, or a head's v, over DP_ROWS rows with
// its channels' window in registers.  The last taps - 1 inputs of every sequence are its state; rows whose window lies in
// the step belong to CTAs of a run of rows, the first taps - 1 rows of a sequence and its state to a CTA of that sequence.
constexpr int DP_MAX_TAPS = 8;

template <int CPL, int TAPS>                          // channels of a lane: lane + 32 e
struct ConvLane {
  float w[TAPS][CPL], win[TAPS][CPL];                 // win[j]: the input at the row's position - taps + 1 + j
  int ch, width, taps;                                // first channel of the head, channels of the head
  __device__ __forceinline__ void init(const float *conv, int first, int n, int n_taps, int lane) {
    ch = first, width = n, taps = n_taps;
#pragma unroll
    for (int e = 0; e < CPL; ++e) {
      const int c = lane + 32 * e;
#pragma unroll
      for (int j = 0; j < TAPS; ++j) {
        w[j][e] = c < n && j < taps ? conv[(size_t)(first + c) * taps + j] : 0.f;
        win[j][e] = 0.f;
      }
    }
  }
  __device__ __forceinline__ void load(const float *row, int lane, float (&x)[CPL]) const {
#pragma unroll
    for (int e = 0; e < CPL; ++e) x[e] = lane + 32 * e < width ? row[ch + lane + 32 * e] : 0.f;
  }
  __device__ __forceinline__ void push(const float (&x)[CPL]) {
#pragma unroll
    for (int e = 0; e < CPL; ++e)
#pragma unroll
      for (int j = 0; j < TAPS; ++j) {
        if (j < taps - 1) win[j][e] = win[j + 1 < TAPS ? j + 1 : j][e];
        else if (j == taps - 1) win[j][e] = x[e];
      }
  }
  __device__ __forceinline__ void result(float (&y)[CPL]) const {
#pragma unroll
    for (int e = 0; e < CPL; ++e) {
      float s = 0.f;
#pragma unroll
      for (int j = 0; j < TAPS; ++j)
        if (j < taps) s = fmaf(w[j][e], win[j][e], s);
      y[e] = silu32(s);
    }
  }
  __device__ __forceinline__ void store(float *st, int channels, int lane) const {
#pragma unroll
    for (int j = 1; j < TAPS; ++j)
      if (j < taps)
#pragma unroll
        for (int e = 0; e < CPL; ++e)
          if (lane + 32 * e < width) st[(size_t)(j - 1) * channels + ch + lane + 32 * e] = win[j][e];
  }
};

template <int CPL, int TAPS, int ROWS>
__global__ void __launch_bounds__(128, CPL <= 2 && TAPS <= 4 ? 4 : CPL <= 4 && TAPS <= 4 ? 3 : 1)
delta_pack_kernel(const float *__restrict__ proj, long long ld, int off_b, int off_a, const float *__restrict__ conv, int taps,
                  float *__restrict__ state, const float *__restrict__ dt_bias, const float *__restrict__ a_log, float key_eps, float q_scale,
                  float *__restrict__ rec, float4 *__restrict__ scal, float *__restrict__ vals, ValuePlace place, const int *__restrict__ tok_seq,
                  const int *__restrict__ tok_pos, const int *__restrict__ seq_start, const int *__restrict__ seq_past,
                  const int *__restrict__ seq_slot, int n_tokens, int n_heads, int n_kv, int d, int dv, int n_chunks) {
  grid_dependents_launch();
  const int lane = threadIdx.x & 31, item = blockIdx.y * 4 + (threadIdx.x >> 5);
  const bool is_v = item >= n_kv;
  const bool idle = item >= n_kv + n_heads;
  const int head = is_v ? item - n_kv : item, group = n_heads / n_kv, dp = scan_dmax(d), keep = taps - 1;
  const int channels = 2 * n_kv * d + n_heads * dv;
  ConvLane<CPL, TAPS> A, B;                            // q and k, or v alone
  if (!idle) {                                         // weights: nothing of the step is read yet
    if (is_v) A.init(conv, 2 * n_kv * d + head * dv, dv, taps, lane);
    else A.init(conv, head * d, d, taps, lane);
    if (!is_v) B.init(conv, (n_kv + head) * d, d, taps, lane);
    else B.width = 0, B.ch = 0, B.taps = taps;
  }
  grid_dependency_wait();
  if (idle) return;
  auto row_out = [&](int t) {
    float y[CPL], k[CPL];
    A.result(y);
    if (is_v) {
#pragma unroll
      for (int e = 0; e < CPL; ++e) {
        const int c = lane + 32 * e;
        if (c < place.cols * place.slices) vals[place.at(head, t, c)] = c < dv ? y[e] : 0.f;
      }
      return;
    }
    B.result(k);
    float qq = 0.f, kk = 0.f, kq = 0.f;
#pragma unroll
    for (int e = 0; e < CPL; ++e) {                    // channels beyond the head are nought
      qq = fmaf(y[e], y[e], qq);
      kk = fmaf(k[e], k[e], kk);
      kq = fmaf(k[e], y[e], kq);
    }
    qq = warp_sum(qq);
    kk = warp_sum(kk);
    kq = warp_sum(kq);
    const float iq = q_scale / sqrtf(qq + key_eps), ik = 1.f / sqrtf(kk + key_eps);
    float *r = rec + ((size_t)head * n_tokens + t) * 2 * dp;
#pragma unroll
    for (int e = 0; e < CPL; ++e) {
      const int c = lane + 32 * e;
      if (c < dp) {
        r[c] = k[e] * ik;
        r[dp + c] = y[e] * iq;
      }
    }
    for (int e = lane; e < group; e += 32) scal[(size_t)(head * group + e) * n_tokens + t].z = kq * iq * ik;
  };
  // the gates of the group's heads for n rows from `first` on, a lane each (rows of `rows` only, a bit per row)
  auto gates = [&](int first, int n, unsigned rows) {
    if (is_v) return;
    for (int e = lane; e < n * group; e += 32) {
      const int i = e / group, h = head * group + e - i * group;
      if (!((rows >> i) & 1u)) continue;
      const float *row = proj + (size_t)(first + i) * ld;
      float4 *dst = scal + (size_t)h * n_tokens + first + i;
      dst->x = expf(-expf(a_log[h]) * softplus32(row[off_a + h] + dt_bias[h]));
      dst->y = sigmoid32(row[off_b + h]);
    }
  };
  auto take = [&](int row) {
    float x[CPL];
    A.load(proj + (size_t)row * ld, lane, x);
    A.push(x);
    if (!is_v) {
      B.load(proj + (size_t)row * ld, lane, x);
      B.push(x);
    }
  };
  if ((int)blockIdx.x < n_chunks) {
    const int r0 = blockIdx.x * ROWS, r1 = min(n_tokens, r0 + ROWS);
    // which rows are this CTA's (bit per row); the others belong to their sequence's own CTA
    const int rl = r0 + lane;
    const unsigned mine = __ballot_sync(0xffffffffu, lane < ROWS && rl < r1 && tok_pos[rl < r1 ? rl : r0] - seq_past[tok_seq[rl < r1 ? rl : r0]] >= keep);
    gates(r0, ROWS, mine);
    if (mine == (1u << ROWS) - 1u) {                   // all of them: the rows' loads do not wait for one another
      constexpr int PRE = CPL <= 2 ? 4 : CPL <= 4 ? 2 : 1;
      for (int k = keep; k > 0; --k) take(r0 - k);
#pragma unroll 1
      for (int i0 = 0; i0 < ROWS; i0 += PRE) {
        float xa[PRE][CPL], xb[PRE][CPL];
#pragma unroll
        for (int i = 0; i < PRE; ++i) {
          A.load(proj + (size_t)(r0 + i0 + i) * ld, lane, xa[i]);
          if (!is_v) B.load(proj + (size_t)(r0 + i0 + i) * ld, lane, xb[i]);
        }
#pragma unroll
        for (int i = 0; i < PRE; ++i) {
          A.push(xa[i]);
          if (!is_v) B.push(xb[i]);
          row_out(r0 + i0 + i);
        }
      }
      return;
    }
    for (int row = r0; row < r1; ++row) {
      if (!((mine >> (row - r0)) & 1u)) continue;
      if (row == r0 || !((mine >> (row - r0 - 1)) & 1u))
        for (int k = keep; k > 0; --k) take(row - k);
      take(row);
      row_out(row);
    }
    return;
  }
  const int b = blockIdx.x - n_chunks, start = seq_start[b], n = seq_start[b + 1] - start;
  float *st = state + (size_t)seq_slot[b] * keep * channels;
  for (int i = 0; i < keep; ++i) {
    float x[CPL];
    A.load(st + (size_t)i * channels, lane, x);
    A.push(x);
    if (!is_v) {
      B.load(st + (size_t)i * channels, lane, x);
      B.push(x);
    }
  }
  gates(start, min(n, keep), 0xffffffffu);
  for (int i = 0; i < min(n, keep); ++i) {
    take(start + i);
    row_out(start + i);
  }
  if (n > keep)
    for (int k = keep; k > 0; --k) take(start + n - k);
  A.store(st, channels, lane);
  if (!is_v) B.store(st, channels, lane);
}

// Rows of `proj` begin with [q | k | v]; conv [channels, taps] (taps 1: one weight per channel), state [slots, taps - 1, channels].
LLM_EXPORT int llm_delta_pack(const float *proj, long long ld, int off_b, int off_a, const float *conv, int taps, float *state,
                              const float *dt_bias, const float *a_log, float key_eps, float q_scale, float *rec, float *scal, float *vals,
                              const int *tok_seq, const int *tok_pos, const int *seq_start, const int *seq_past, const int *seq_slot,
                              int n_tokens, int n_seqs, int n_heads, int n_kv, int d, int dv, int single_tokens, cudaStream_t stream) {
  if (n_tokens == 0) return LLM_OK;
  LLM_REQUIRE(n_tokens > 0 && n_seqs > 0 && n_heads > 0 && n_kv > 0 && n_heads % n_kv == 0 && d > 0 && dv > 0, "delta_pack: bad sizes");
  LLM_REQUIRE(d <= 256 && dv <= 512, "delta_pack: heads of %d and %d channels are not supported (up to 256 and 512)", d, dv);
  LLM_REQUIRE(taps >= 1 && taps <= DP_MAX_TAPS && conv && (taps == 1 || state), "delta_pack: a convolution of %d taps (1 to %d) needs its weight and state",
              taps, DP_MAX_TAPS);
  const ValuePlace place{scan_cols(d), scan_slices(d, dv), scan_shift(d), n_tokens};
  const int widest = scan_dmax(d) > place.cols * place.slices ? scan_dmax(d) : place.cols * place.slices;
  const int n_own = taps > 1 ? n_seqs : 0;
#define DP_GO(CPL, TAPS, ROWS)                                                                                               \
  do {                                                                                                                       \
    const int n_chunks = single_tokens && taps > 1 ? 0 : (n_tokens + ROWS - 1) / ROWS;                                       \
    llm_launch(delta_pack_kernel<CPL, TAPS, ROWS>, dim3(n_chunks + n_own, (n_kv + n_heads + 3) / 4), dim3(128), 0, stream, proj, ld, off_b, \
               off_a, conv, taps, state, dt_bias, a_log, key_eps, q_scale, rec, (float4 *)scal, vals, place, tok_seq, tok_pos, seq_start, \
               seq_past, seq_slot, n_tokens, n_heads, n_kv, d, dv, n_chunks);                                                \
  } while (0)
#define DP_TAPS(CPL, ROWS)                         \
  do {                                             \
    if (taps <= 4) DP_GO(CPL, 4, ROWS);            \
    else DP_GO(CPL, DP_MAX_TAPS, ROWS);            \
  } while (0)
  if (widest <= 32) DP_TAPS(1, 16);
  else if (widest <= 64) DP_TAPS(2, 16);
  else if (widest <= 128) DP_TAPS(4, 16);
  else if (widest <= 256) DP_TAPS(8, 8);
  else DP_TAPS(16, 8);
#undef DP_TAPS
#undef DP_GO
  LLM_CHECK_LAUNCH("delta_pack");
  return LLM_OK;
}

// Bonus: r, k, v and the low-rank decay input x1 (rank values) of every token in rows of their own; per head the decay
// w = exp(-exp(w0 + W2 tanh(x1))) per key channel and c = sum_i r_i u_i k_i.  A CTA takes one head, a warp BP_TT tokens at once: a
// value of W2 serves all of them.  The head's rows of W2 [d, rank] lie in shared memory where they fit (padded by one value).
constexpr int BP_WARPS = 4, BP_TT = 4;

__global__ void __launch_bounds__(BP_WARPS * 32)
bonus_pack_kernel(const float *__restrict__ r, long long ldr, const float *__restrict__ k, long long ldk, const float *__restrict__ v,
                  long long ldv, const float *__restrict__ x1, long long ldx, int rank, const float *__restrict__ w2,
                  const float *__restrict__ w0, const float *__restrict__ u, int n_tokens, int d, int dv, int w2_shared,
                  float *__restrict__ rec, float4 *__restrict__ scal, float *__restrict__ vals, ValuePlace place) {
  extern __shared__ __align__(16) float bp_sm[];      // tanh(x1) [warps][rank][TT], then W2's rows of the head [d][rank + 1]
  grid_dependents_launch();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, hd = blockIdx.y, dp = scan_dmax(d);
  float *th = bp_sm + warp * rank * BP_TT, *w2s = bp_sm + BP_WARPS * rank * BP_TT;
  const float *w2h = w2 + (size_t)hd * d * rank;
  if (w2_shared)
    for (int i = threadIdx.x; i < d * rank; i += BP_WARPS * 32) w2s[(i / rank) * (rank + 1) + i % rank] = w2h[i];
  grid_dependency_wait();
  __syncthreads();
  const int t0 = (blockIdx.x * BP_WARPS + warp) * BP_TT, nt = min(BP_TT, n_tokens - t0);
  if (nt <= 0) return;
  for (int i = lane; i < rank * BP_TT; i += 32) {
    const int tt = i / rank, q = i - tt * rank;
    th[q * BP_TT + tt] = tt < nt ? tanhf(x1[(size_t)(t0 + tt) * ldx + q]) : 0.f;
  }
  // the values, into their slices
  for (int c = lane; c < place.cols * place.slices; c += 32)
#pragma unroll
    for (int tt = 0; tt < BP_TT; ++tt)
      if (tt < nt) vals[place.at(hd, t0 + tt, c)] = c < dv ? v[(size_t)(t0 + tt) * ldv + (size_t)hd * dv + c] : 0.f;
  __syncwarp();
  float c[BP_TT] = {};
  for (int i = lane; i < dp; i += 32) {
    float z[BP_TT], kk[BP_TT], rr[BP_TT];
    const bool in = i < d;
    const float w0i = in ? w0[hd * d + i] : 0.f, ui = in ? u[hd * d + i] : 0.f;
#pragma unroll
    for (int tt = 0; tt < BP_TT; ++tt) {
      z[tt] = w0i;
      kk[tt] = in && tt < nt ? k[(size_t)(t0 + tt) * ldk + (size_t)hd * d + i] : 0.f;
      rr[tt] = in && tt < nt ? r[(size_t)(t0 + tt) * ldr + (size_t)hd * d + i] : 0.f;
    }
    if (in)
      for (int q = 0; q < rank; ++q) {
        const float w = w2_shared ? w2s[i * (rank + 1) + q] : w2h[(size_t)i * rank + q];
        const float4 t4 = ld4(th + q * BP_TT);
        z[0] = fmaf(w, t4.x, z[0]);
        z[1] = fmaf(w, t4.y, z[1]);
        z[2] = fmaf(w, t4.z, z[2]);
        z[3] = fmaf(w, t4.w, z[3]);
      }
#pragma unroll
    for (int tt = 0; tt < BP_TT; ++tt) {
      c[tt] = fmaf(rr[tt] * ui, kk[tt], c[tt]);
      if (tt >= nt) continue;
      float *o = rec + ((size_t)hd * n_tokens + t0 + tt) * 3 * dp;
      o[i] = kk[tt];
      o[dp + i] = rr[tt];
      o[2 * dp + i] = in ? expf(-expf(z[tt])) : 0.f;
    }
  }
#pragma unroll
  for (int tt = 0; tt < BP_TT; ++tt) {
    const float s = warp_sum(c[tt]);
    if (lane == 0 && tt < nt) scal[(size_t)hd * n_tokens + t0 + tt] = make_float4(1.f, 1.f, s, 0.f);
  }
}

LLM_EXPORT int llm_bonus_pack(const float *r, long long ldr, const float *k, long long ldk, const float *v, long long ldv, const float *x1,
                              long long ldx, int rank, const float *w2, const float *w0, const float *u, float *rec, float *scal, float *vals,
                              int n_tokens, int n_heads, int d, int dv, cudaStream_t stream) {
  if (n_tokens == 0) return LLM_OK;
  LLM_REQUIRE(n_tokens > 0 && n_heads > 0 && n_heads <= 65535 && d > 0 && dv > 0 && rank > 0, "bonus_pack: bad sizes");
  const size_t with_w2 = ((size_t)BP_WARPS * rank * BP_TT + (size_t)d * (rank + 1)) * sizeof(float);
  const int w2_shared = with_w2 <= 96 * 1024;
  const size_t smem = w2_shared ? with_w2 : (size_t)BP_WARPS * rank * BP_TT * sizeof(float);
  LLM_REQUIRE(smem <= 96 * 1024, "bonus_pack: a decay input of rank %d is not supported", rank);
  LLM_CHECK_CUDA(llm_allow_smem(bonus_pack_kernel, smem), "bonus_pack attribute");
  const ValuePlace place{scan_cols(d), scan_slices(d, dv), scan_shift(d), n_tokens};
  llm_launch(bonus_pack_kernel, dim3((unsigned)((n_tokens + BP_WARPS * BP_TT - 1) / (BP_WARPS * BP_TT)), n_heads), dim3(BP_WARPS * 32), smem, stream,
             r, ldr, k, ldk, v, ldv, x1, ldx, rank, w2, w0, u, n_tokens, d, dv, w2_shared, rec, (float4 *)scal, vals, place);
  LLM_CHECK_LAUNCH("bonus_pack");
  return LLM_OK;
}

// Memory: the gates of a sequence's tokens in order.  log gates i = cap tanh((x_i + b_i) / cap), f = logsigmoid(cap tanh((x_f +
// b_f) / cap)); with the running maximum m (state [slots, heads], 0 at the start) m_t = max(f + m_(t-1), i):
// scal = (exp(f + m_(t-1) - m_t), exp(i - m_t), room for c, exp(-m_t)).  A CTA per (sequence, head): the logarithms of MG_TOKENS tokens
// side by side, their maxima one after another by one thread out of shared memory, the exponentials side by side.
constexpr int MG_TOKENS = 1024, MG_THREADS = 512;

__device__ __forceinline__ float capped(float x, float cap) { return cap * tanhf(x / cap); }

__global__ void __launch_bounds__(MG_THREADS)
memory_gates_kernel(const float *__restrict__ proj, long long ld, int off_i, int off_f, const float *__restrict__ bias_i,
                    const float *__restrict__ bias_f, float cap, float *__restrict__ state_m, float4 *__restrict__ scal,
                    const int *__restrict__ seq_start, const int *__restrict__ seq_slot, int n_tokens, int n_heads) {
  __shared__ __align__(16) float2 fi[MG_TOKENS];
  __shared__ float m[MG_TOKENS + 1];
  grid_dependents_launch();
  grid_dependency_wait();
  const int b = blockIdx.x, hd = blockIdx.y, tid = threadIdx.x;
  const int start = seq_start[b], n = seq_start[b + 1] - start;
  float *mp = state_m + (size_t)seq_slot[b] * n_heads + hd;
  const float bi = bias_i[hd], bf = bias_f[hd];
  if (tid == 0) m[0] = *mp;
  for (int t0 = 0; t0 < n; t0 += MG_TOKENS) {
    const int nt = min(MG_TOKENS, n - t0);
    for (int e = tid; e < nt; e += MG_THREADS) {
      const float *row = proj + (size_t)(start + t0 + e) * ld;
      const float xi = row[off_i + hd], xf = row[off_f + hd];
      fi[e] = make_float2(log_sigmoid32(capped(xf + bf, cap)), capped(xi + bi, cap));
    }
    __syncthreads();
    if (tid == 0) {
      float run = m[0];
      int e = 0;
      for (; e + 8 <= nt; e += 8) {                    // eight tokens' gates in registers before the chain runs through them
        float4 x[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) x[u] = *reinterpret_cast<const float4 *>(&fi[e + 2 * u]);
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          m[e + 2 * u + 1] = run = fmaxf(x[u].x + run, x[u].y);
          m[e + 2 * u + 2] = run = fmaxf(x[u].z + run, x[u].w);
        }
      }
      for (; e < nt; ++e) m[e + 1] = run = fmaxf(fi[e].x + run, fi[e].y);
    }
    __syncthreads();
    for (int e = tid; e < nt; e += MG_THREADS) {
      const float m0 = m[e], m1 = m[e + 1];
      scal[(size_t)hd * n_tokens + start + t0 + e] = make_float4(expf(fi[e].x + m0 - m1), expf(fi[e].y - m1), 0.f, expf(-m1));
    }
    __syncthreads();
    if (tid == 0) m[0] = m[nt];
  }
  if (tid == 0) *mp = m[0];
}

// Its vectors: k and q (times q_scale) of the product's rows, c = k . q; the values, and 1 in the column of n.  A warp takes
// MP_TT tokens of a head.
constexpr int MP_TT = 4;

__global__ void __launch_bounds__(128)
memory_pack_kernel(const float *__restrict__ proj, long long ld, int off_q, int off_k, int off_v, float q_scale, float *__restrict__ rec,
                   float4 *__restrict__ scal, float *__restrict__ vals, ValuePlace place, int n_tokens, int d, int dv) {
  grid_dependents_launch();
  grid_dependency_wait();
  const int lane = threadIdx.x & 31, dp = scan_dmax(d), hd = blockIdx.y;
  const int t0 = (blockIdx.x * 4 + (threadIdx.x >> 5)) * MP_TT, nt = min(MP_TT, n_tokens - t0);
  if (nt <= 0) return;
  float kq[MP_TT] = {};
  for (int i = lane; i < dp; i += 32) {
    float kk[MP_TT], qq[MP_TT];
#pragma unroll
    for (int tt = 0; tt < MP_TT; ++tt) {
      const float *row = proj + (size_t)(t0 + tt) * ld + (size_t)hd * d + i;
      kk[tt] = i < d && tt < nt ? row[off_k] : 0.f;
      qq[tt] = i < d && tt < nt ? row[off_q] * q_scale : 0.f;
    }
#pragma unroll
    for (int tt = 0; tt < MP_TT; ++tt) {
      kq[tt] = fmaf(kk[tt], qq[tt], kq[tt]);
      if (tt >= nt) continue;
      float *r = rec + ((size_t)hd * n_tokens + t0 + tt) * 2 * dp;
      r[i] = kk[tt];
      r[dp + i] = qq[tt];
    }
  }
  for (int c = lane; c < place.cols * place.slices; c += 32)
#pragma unroll
    for (int tt = 0; tt < MP_TT; ++tt)
      if (tt < nt) vals[place.at(hd, t0 + tt, c)] = c < dv ? proj[(size_t)(t0 + tt) * ld + off_v + (size_t)hd * dv + c] : c == dv ? 1.f : 0.f;
#pragma unroll
  for (int tt = 0; tt < MP_TT; ++tt) {
    const float s = warp_sum(kq[tt]);
    if (lane == 0 && tt < nt) scal[(size_t)hd * n_tokens + t0 + tt].z = s;
  }
}

LLM_EXPORT int llm_memory_pack(const float *proj, long long ld, int off_q, int off_k, int off_v, int off_i, int off_f, const float *bias_i,
                               const float *bias_f, float cap, float q_scale, float *state_m, float *rec, float *scal, float *vals,
                               const int *seq_start, const int *seq_slot, int n_tokens, int n_seqs, int n_heads, int d, int dv,
                               cudaStream_t stream) {
  if (n_tokens == 0) return LLM_OK;
  LLM_REQUIRE(n_tokens > 0 && n_seqs > 0 && n_heads > 0 && n_heads <= 65535 && d > 0 && dv > 0 && cap > 0.f, "memory_pack: bad sizes");
  llm_launch(memory_gates_kernel, dim3(n_seqs, n_heads), dim3(MG_THREADS), 0, stream, proj, ld, off_i, off_f, bias_i, bias_f, cap, state_m,
             (float4 *)scal, seq_start, seq_slot, n_tokens, n_heads);
  LLM_CHECK_LAUNCH("memory_gates");
  const ValuePlace place{scan_cols(d), scan_slices(d, dv + 1), scan_shift(d), n_tokens};
  llm_launch(memory_pack_kernel, dim3((unsigned)((n_tokens + 4 * MP_TT - 1) / (4 * MP_TT)), n_heads), dim3(128), 0, stream, proj, ld, off_q, off_k,
             off_v, q_scale, rec, (float4 *)scal, vals, place, n_tokens, d, dv);
  LLM_CHECK_LAUNCH("memory_pack");
  return LLM_OK;
}

// ---------------------------------------------------------------- behind the scan: norm per head, weight, gate
// y = x / (max(|den|, floor) + 1e-6)   where den is given (memory; floor = scal's fourth value)
// out = y / sqrt(mean(y^2) + eps) * weight * gate * out_scale; weight [heads * dv], or [dv] shared by the heads; gate:
// sigmoid (act 0) or silu (act 1) of 32-bit logits.  LPH lanes to a head, V values of a lane side by side, E times.
template <typename T, int LPH, int V, int E>
__global__ void __launch_bounds__(128)
head_finish_kernel(const float *__restrict__ x, long long ldx, const float *__restrict__ den, const float4 *__restrict__ scal,
                   const float *__restrict__ weight, int shared_weight, const float *__restrict__ gate, long long gate_stride, int act,
                   float eps, float out_scale, int n_tokens, int n_heads, int dv, T *__restrict__ out, long long ldo) {
  grid_dependents_launch();
  const int sub = threadIdx.x % LPH;
  const long long item = (long long)blockIdx.x * (128 / LPH) + threadIdx.x / LPH;
  const bool in = item < (long long)n_tokens * n_heads;          // lanes without a head still take part in the sums
  const int t = in ? (int)(item / n_heads) : 0, hd = in ? (int)(item - (long long)t * n_heads) : 0;
  const float *xr = x + (size_t)t * ldx + (size_t)hd * dv, *gr = gate + (size_t)t * gate_stride + (size_t)hd * dv;
  const float *wr = weight + (shared_weight ? 0 : (size_t)hd * dv);
  T *o = out + (size_t)t * ldo + (size_t)hd * dv;
  float v[E][V], g[E][V], w[E][V];
  auto at = [&](int e) { return (sub + LPH * e) * V; };
  auto load = [&](const float *p, bool ok, float (&y)[V]) {
    if constexpr (V == 4) {
      const float4 f = ok ? ld4(p) : make_float4(0.f, 0.f, 0.f, 0.f);
      y[0] = f.x, y[1] = f.y, y[2] = f.z, y[3] = f.w;
    } else {
      y[0] = ok ? p[0] : 0.f;
    }
  };
#pragma unroll
  for (int e = 0; e < E; ++e) load(wr + at(e), at(e) < dv, w[e]);
  grid_dependency_wait();
#pragma unroll
  for (int e = 0; e < E; ++e) {
    load(xr + at(e), in && at(e) < dv, v[e]);
    load(gr + at(e), in && at(e) < dv, g[e]);
  }
  const float by = den && in ? 1.f / (fmaxf(fabsf(den[item]), scal[(size_t)hd * n_tokens + t].w) + 1e-6f) : 1.f;
  float ss = 0.f;
#pragma unroll
  for (int e = 0; e < E; ++e)
#pragma unroll
    for (int i = 0; i < V; ++i) {
      v[e][i] *= by;
      ss = fmaf(v[e][i], v[e][i], ss);
    }
#pragma unroll
  for (int s = LPH / 2; s > 0; s >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, s);
  const float inv = out_scale / sqrtf(ss / (float)dv + eps);
#pragma unroll
  for (int e = 0; e < E; ++e) {
    if (!in || at(e) >= dv) continue;
#pragma unroll
    for (int i = 0; i < V; ++i) v[e][i] = v[e][i] * inv * w[e][i] * (act ? silu32(g[e][i]) : sigmoid32(g[e][i]));
    if constexpr (V == 4) st4(o + at(e), make_float4(v[e][0], v[e][1], v[e][2], v[e][3]));
    else o[at(e)] = from_float<T>(v[e][0]);
  }
}

LLM_EXPORT int llm_head_finish(const float *x, long long ldx, const float *den, const float *scal, const float *weight, int shared_weight,
                               const float *gate, long long gate_stride, int act, float eps, float out_scale, int n_tokens, int n_heads,
                               int dv, void *out, int out_dtype, long long ldo, cudaStream_t stream) {
  if (n_tokens == 0) return LLM_OK;
  LLM_REQUIRE(n_tokens > 0 && n_heads > 0 && dv > 0 && dv <= 512, "head_finish: heads of %d values are not supported (up to 512)", dv);
  LLM_REQUIRE(act == 0 || act == 1, "head_finish: gate activation %d is not known", act);
  const long long items = (long long)n_tokens * n_heads;
  const int osz = out_dtype == LLM_F32 ? 4 : 2;
  const bool vec = dv % 4 == 0 && ldx % 4 == 0 && ldo % 4 == 0 && gate_stride % 4 == 0 && (uintptr_t)x % 16 == 0 && (uintptr_t)weight % 16 == 0 &&
                   (uintptr_t)gate % 16 == 0 && (uintptr_t)out % (4 * osz) == 0;
#define HF_GO(T, LPH, V, E)                                                                                                   \
  llm_launch(head_finish_kernel<T, LPH, V, E>, dim3((unsigned)((items + 128 / LPH - 1) / (128 / LPH))), dim3(128), 0, stream, x, ldx, den, \
             (const float4 *)scal, weight, shared_weight, gate, gate_stride, act, eps, out_scale, n_tokens, n_heads, dv, (T *)out, ldo)
#define HF_SIZES(T)                              \
  do {                                           \
    if (!vec) HF_GO(T, 32, 1, 16);               \
    else if (dv <= 32) HF_GO(T, 8, 4, 1);        \
    else if (dv <= 64) HF_GO(T, 16, 4, 1);       \
    else if (dv <= 128) HF_GO(T, 32, 4, 1);      \
    else if (dv <= 256) HF_GO(T, 32, 4, 2);      \
    else HF_GO(T, 32, 4, 4);                     \
  } while (0)
  if (out_dtype == LLM_F32) HF_SIZES(float);
  else if (out_dtype == LLM_BF16) HF_SIZES(__nv_bfloat16);
  else LLM_FAIL("head_finish: unknown dtype %d", out_dtype);
#undef HF_SIZES
#undef HF_GO
  LLM_CHECK_LAUNCH("head_finish");
  return LLM_OK;
}

// ---------------------------------------------------------------- a token beside its predecessor
// out[s][t] = h_t + (h_(t-1) - h_t) mu_s for n_mix vectors mu [n_mix, width] (32-bit arithmetic, rounded once); the last row
// of every sequence is its state [slots, width].  A sequence's first row of the step and the state belong to a CTA of
// their sequence (blockIdx.y - n_chunks), whose threads read the old row of their channel before they write the new one.
constexpr int TS_THREADS = 128, TS_ROWS = 8, TS_MIX = 5;

template <typename T, int V>
struct TsVec {
  float x[V];
};
template <typename T, int V>
__device__ __forceinline__ TsVec<T, V> ts_load(const T *p) {
  TsVec<T, V> r;
  if constexpr (V == 1) {
    r.x[0] = to_float(p[0]);
  } else {
    const float4 v = ld4(p);
    r.x[0] = v.x, r.x[1] = v.y, r.x[2] = v.z, r.x[3] = v.w;
  }
  return r;
}
template <typename T, int V>
__device__ __forceinline__ void ts_store(T *p, const TsVec<T, V> &r) {
  if constexpr (V == 1) p[0] = from_float<T>(r.x[0]);
  else st4(p, make_float4(r.x[0], r.x[1], r.x[2], r.x[3]));
}

template <typename T, int V, int N_MIX>
__global__ void __launch_bounds__(TS_THREADS)
token_shift_kernel(const T *__restrict__ h, long long ldh, const float *__restrict__ mu, T *__restrict__ out, long long mix_stride,
                   T *__restrict__ state, const int *__restrict__ tok_seq, const int *__restrict__ tok_pos,
                   const int *__restrict__ seq_start, const int *__restrict__ seq_past, const int *__restrict__ seq_slot, int n_tokens,
                   int width, int n_chunks) {
  grid_dependents_launch();
  const int c = (blockIdx.x * TS_THREADS + threadIdx.x) * V;
  float m[N_MIX][V];                                   // weights: nothing of the step is read yet
  if (c < width)
#pragma unroll
    for (int s = 0; s < N_MIX; ++s)
#pragma unroll
      for (int v = 0; v < V; ++v) m[s][v] = mu[(size_t)s * width + c + v];
  grid_dependency_wait();
  if (c >= width) return;
  auto row_out = [&](int t, const TsVec<T, V> &cur, const TsVec<T, V> &prev) {
#pragma unroll
    for (int s = 0; s < N_MIX; ++s) {
      TsVec<T, V> r;
#pragma unroll
      for (int v = 0; v < V; ++v) r.x[v] = fmaf(prev.x[v] - cur.x[v], m[s][v], cur.x[v]);
      ts_store<T, V>(out + (size_t)s * mix_stride + (size_t)t * width + c, r);
    }
  };
  if ((int)blockIdx.y < n_chunks) {
    const int r0 = blockIdx.y * TS_ROWS, r1 = min(n_tokens, r0 + TS_ROWS);
    TsVec<T, V> x[TS_ROWS + 1];                         // all rows' loads at once; row -1 where there is one
    x[0] = ts_load<T, V>(h + (size_t)(r0 > 0 ? r0 - 1 : 0) * ldh + c);
#pragma unroll
    for (int i = 0; i < TS_ROWS; ++i) x[i + 1] = ts_load<T, V>(h + (size_t)min(r0 + i, n_tokens - 1) * ldh + c);
    bool mine[TS_ROWS];                                // not the first row its sequence brings
#pragma unroll
    for (int i = 0; i < TS_ROWS; ++i) mine[i] = r0 + i < r1 && tok_pos[r0 + i] > seq_past[tok_seq[r0 + i]];
#pragma unroll
    for (int i = 0; i < TS_ROWS; ++i)
      if (mine[i]) row_out(r0 + i, x[i + 1], x[i]);
    return;
  }
  const int b = blockIdx.y - n_chunks, start = seq_start[b], n = seq_start[b + 1] - start;
  if (n <= 0) return;
  T *st = state + (size_t)seq_slot[b] * width + c;
  const TsVec<T, V> old = ts_load<T, V>(st), first = ts_load<T, V>(h + (size_t)start * ldh + c);
  row_out(start, first, old);
  ts_store<T, V>(st, n == 1 ? first : ts_load<T, V>(h + (size_t)(start + n - 1) * ldh + c));
}

LLM_EXPORT int llm_token_shift(int dtype, const void *h, long long ldh, const float *mu, int n_mix, void *out, long long mix_stride,
                               void *state, const int *tok_seq, const int *tok_pos, const int *seq_start, const int *seq_past,
                               const int *seq_slot, int n_tokens, int n_seqs, int width, int single_tokens, cudaStream_t stream) {
  if (n_tokens == 0) return LLM_OK;
  LLM_REQUIRE(n_tokens > 0 && n_seqs > 0 && width > 0 && state, "token_shift: bad arguments");
  LLM_REQUIRE(n_mix == TS_MIX, "token_shift: %d mixes are not built (%d)", n_mix, TS_MIX);
  const int n_chunks = single_tokens ? 0 : (n_tokens + TS_ROWS - 1) / TS_ROWS;
  LLM_REQUIRE(n_chunks + n_seqs <= 65535, "token_shift: too many rows for one launch");
  const int esz = dtype == LLM_F32 ? 4 : 2;
  const bool vec = width % 4 == 0 && ldh % 4 == 0 && mix_stride % 4 == 0 && (uintptr_t)h % (4 * esz) == 0 && (uintptr_t)out % (4 * esz) == 0 &&
                   (uintptr_t)state % (4 * esz) == 0;
  const int v = vec ? 4 : 1;
  const dim3 grid((width + TS_THREADS * v - 1) / (TS_THREADS * v), n_chunks + n_seqs);
#define TS_GO(T, V)                                                                                                            \
  llm_launch(token_shift_kernel<T, V, TS_MIX>, grid, dim3(TS_THREADS), 0, stream, (const T *)h, ldh, mu, (T *)out, mix_stride, (T *)state, \
             tok_seq, tok_pos, seq_start, seq_past, seq_slot, n_tokens, width, n_chunks)
  if (dtype == LLM_F32 && vec) TS_GO(float, 4);
  else if (dtype == LLM_F32) TS_GO(float, 1);
  else if (dtype == LLM_BF16 && vec) TS_GO(__nv_bfloat16, 4);
  else if (dtype == LLM_BF16) TS_GO(__nv_bfloat16, 1);
  else LLM_FAIL("token_shift: unknown dtype %d", dtype);
#undef TS_GO
  LLM_CHECK_LAUNCH("token_shift");
  return LLM_OK;
}

// ---------------------------------------------------------------- a step of single tokens
// One CTA per (sequence, key head): the token's vectors (the convolution included), the heads' state, the norm, its weight
// and the gate, one launch from the products to the input of the output projection.  Eight lanes to a column of the state, 32
// columns at a time; the state of the first columns is on its way while the vectors are made.
constexpr int SS_THREADS = 256, SS_LANES = 8, SS_COLS = SS_THREADS / SS_LANES;

struct StepIn {
  const float *q, *k, *v, *g;            // rows of the products: q (r), k per key head, v per head, gate logits per head
  long long ldq, ldk, ldv, ldg;
  // gated delta
  const float *proj_ab;                  // logits: b at off_b, a at off_a
  long long ld_ab;
  int off_b, off_a;
  const float *dt_bias, *a_log;
  const float *conv;                     // [channels, taps]: q, k, v of all heads one behind the other; taps 1 without
  float *conv_state;                     // [slots, taps - 1, channels]
  int taps;
  float key_eps, q_scale;
  // bonus
  const float *x1, *w2, *w0, *u;
  long long ldx;
  int rank;
  // memory
  const float *x_if, *bias_i, *bias_f;
  long long ld_if;
  int off_i, off_f;
  float cap;
  float *state_m;
};

// a channel's short convolution and silu; the last inputs move on by one
__device__ __forceinline__ float step_conv(const StepIn &in, float x, int ch, int channels, size_t slot) {
  if (in.conv == nullptr) return silu32(x);
  const float *w = in.conv + (size_t)ch * in.taps;
  float *st = in.conv_state + (slot * (in.taps - 1)) * (size_t)channels + ch;
  float s = 0.f;
  for (int j = 0; j < in.taps - 1; ++j) {
    const float o = st[(size_t)j * channels];
    s = fmaf(w[j], o, s);
    if (j > 0) st[(size_t)(j - 1) * channels] = o;
  }
  s = fmaf(w[in.taps - 1], x, s);
  if (in.taps > 1) st[(size_t)(in.taps - 2) * channels] = x;
  return silu32(s);
}

template <int RULE, int DMAX, typename TO>
__global__ void __launch_bounds__(SS_THREADS)
state_step_kernel(const StepIn in, float *__restrict__ state, const float *__restrict__ weight, int shared_weight, int act, float eps,
                  float out_scale, TO *__restrict__ out, long long ldo, const int *__restrict__ seq_slot, int n_heads, int n_kv, int d, int dv) {
  constexpr int ROWS = DMAX / SS_LANES;
  constexpr int R4 = (ROWS + 3) / 4;                  // 16-byte groups of a lane
  constexpr int NC = R4 <= 2 ? 4 : R4 <= 4 ? 2 : 1;     // columns of a lane whose state is fetched at once
  __shared__ __align__(16) float kk[DMAX], qq[DMAX], ww[DMAX];
  __shared__ float red[4];
  extern __shared__ float ss_sm[];                    // v [group * dv], outs [dv + 1], tanh(x1) [rank], scalars [group * 4]
  grid_dependents_launch();
  const int b = blockIdx.x, kvh = blockIdx.y, group = n_heads / n_kv;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, sub = tid % SS_LANES, col = tid / SS_LANES;
  float *vs = ss_sm, *outs = vs + group * dv, *th = outs + dv + 1, *sc = th + (RULE == RULE_BONUS ? in.rank : 0);
  const int n_cols = dv + (RULE == RULE_MEMORY ? 1 : 0);
  for (int i = tid; i < DMAX; i += SS_THREADS) kk[i] = qq[i] = ww[i] = 0.f;
  grid_dependency_wait();
  const size_t slot = (size_t)seq_slot[b];
  float2 S[NC][R4 * 2];
  auto fetch = [&](int h, int j0) {
#pragma unroll
    for (int n = 0; n < NC; ++n) {
      const int j = j0 + n * SS_COLS + col;
      const float *sp = state + ((slot * n_heads + h) * n_cols + (j < n_cols ? j : 0)) * (size_t)d;
#pragma unroll
      for (int i = 0; i < R4; ++i) {
        const int row = 4 * (sub + SS_LANES * i);
        if (d % 4 == 0) {
          const float4 s4 = j < n_cols && row < d ? ld4(sp + row) : make_float4(0.f, 0.f, 0.f, 0.f);
          S[n][2 * i] = make_float2(s4.x, s4.y), S[n][2 * i + 1] = make_float2(s4.z, s4.w);
        } else {
          float x[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) x[e] = j < n_cols && row + e < d ? sp[row + e] : 0.f;
          S[n][2 * i] = make_float2(x[0], x[1]), S[n][2 * i + 1] = make_float2(x[2], x[3]);
        }
      }
    }
  };
  fetch(kvh * group, 0);
  __syncthreads();                                    // the vectors' padding is set
  // ------------------------------------------------------------ the token's vectors
  if (RULE == RULE_DELTA) {
    const int channels = 2 * n_kv * d + n_heads * dv;
    for (int i = tid; i < 2 * d + group * dv; i += SS_THREADS) {
      if (i < d) qq[i] = step_conv(in, in.q[(size_t)b * in.ldq + kvh * d + i], kvh * d + i, channels, slot);
      else if (i < 2 * d) kk[i - d] = step_conv(in, in.k[(size_t)b * in.ldk + kvh * d + i - d], (n_kv + kvh) * d + i - d, channels, slot);
      else vs[i - 2 * d] = step_conv(in, in.v[(size_t)b * in.ldv + kvh * group * dv + i - 2 * d],
                                     2 * n_kv * d + kvh * group * dv + i - 2 * d, channels, slot);
    }
    for (int e = tid; e < group; e += SS_THREADS) {
      const int h = kvh * group + e;
      const float *row = in.proj_ab + (size_t)b * in.ld_ab;
      sc[e * 4] = expf(-expf(in.a_log[h]) * softplus32(row[in.off_a + h] + in.dt_bias[h]));
      sc[e * 4 + 1] = sigmoid32(row[in.off_b + h]);
    }
    __syncthreads();
    if (warp < 3) {                                    // q . q, k . k, k . q: a warp each, lane order then the shuffle tree
      const float *x = warp == 0 ? qq : kk, *y = warp == 1 ? kk : qq;
      float s = 0.f;
      for (int i = lane; i < d; i += 32) s = fmaf(x[i], y[i], s);
      s = warp_sum(s);
      if (lane == 0) red[warp] = s;
    }
    __syncthreads();
    const float iq = in.q_scale / sqrtf(red[0] + in.key_eps), ik = 1.f / sqrtf(red[1] + in.key_eps);
    for (int i = tid; i < d; i += SS_THREADS) {
      qq[i] *= iq;
      kk[i] *= ik;
    }
    for (int e = tid; e < group; e += SS_THREADS) sc[e * 4 + 2] = red[2] * iq * ik;
  } else {
    for (int i = tid; i < d; i += SS_THREADS) {
      qq[i] = in.q[(size_t)b * in.ldq + kvh * d + i] * in.q_scale;
      kk[i] = in.k[(size_t)b * in.ldk + kvh * d + i];
    }
    for (int i = tid; i < dv; i += SS_THREADS) vs[i] = in.v[(size_t)b * in.ldv + (size_t)kvh * dv + i];
    if (RULE == RULE_BONUS)
      for (int i = tid; i < in.rank; i += SS_THREADS) th[i] = tanhf(in.x1[(size_t)b * in.ldx + i]);
    if (RULE == RULE_MEMORY && tid == 0) {
      const float *row = in.x_if + (size_t)b * in.ld_if;
      const float li = capped(row[in.off_i + kvh] + in.bias_i[kvh], in.cap);
      const float lf = log_sigmoid32(capped(row[in.off_f + kvh] + in.bias_f[kvh], in.cap));
      float *mp = in.state_m + slot * n_heads + kvh;
      const float m0 = *mp, m1 = fmaxf(lf + m0, li);
      *mp = m1;
      sc[0] = expf(lf + m0 - m1);
      sc[1] = expf(li - m1);
      sc[3] = expf(-m1);
    }
    __syncthreads();
    if (RULE == RULE_BONUS) {
      // a channel's decay by eight lanes: W2's row in strides, then the shuffle tree
      for (int i0 = 0; i0 < d; i0 += SS_COLS) {
        const int i = i0 + col;
        float z = 0.f;
        if (i < d) {
          const float *w2r = in.w2 + ((size_t)kvh * d + i) * in.rank;
          for (int q = sub; q < in.rank; q += SS_LANES) z = fmaf(w2r[q], th[q], z);
        }
#pragma unroll
        for (int o = 1; o < SS_LANES; o <<= 1) z += __shfl_xor_sync(0xffffffffu, z, o);
        if (i < d && sub == 0) ww[i] = expf(-expf(z + in.w0[(size_t)kvh * d + i]));
      }
    }
    if (warp == 7) {                                   // c
      float s = 0.f;
      for (int i = lane; i < d; i += 32) s = fmaf(RULE == RULE_BONUS ? qq[i] * in.u[(size_t)kvh * d + i] : qq[i], kk[i], s);
      s = warp_sum(s);
      if (lane == 0) {
        sc[2] = s;
        if (RULE == RULE_BONUS) sc[0] = sc[1] = 1.f;
      }
    }
  }
  __syncthreads();
  // ------------------------------------------------------------ the heads' state
  for (int e = 0; e < group; ++e) {
    const int h = kvh * group + e;
    const float4 s4 = make_float4(sc[e * 4], sc[e * 4 + 1], sc[e * 4 + 2], sc[e * 4 + 3]);
    for (int j0 = 0; j0 < n_cols; j0 += NC * SS_COLS) {
      if (e > 0 || j0 > 0) fetch(h, j0);
#pragma unroll
      for (int n = 0; n < NC; ++n) {
        const int j = j0 + n * SS_COLS + col;
        const float v = j < dv ? vs[e * dv + j] : 1.f;
        const float o = scan_token<RULE, SS_LANES, R4 * 4>(S[n], kk, qq, ww, s4, v, sub);
        if (j >= n_cols) continue;
        float *sp = state + ((slot * n_heads + h) * n_cols + j) * (size_t)d;
#pragma unroll
        for (int i = 0; i < R4; ++i) {
          const int row = 4 * (sub + SS_LANES * i);
          if (d % 4 == 0) {
            if (row < d) st4(sp + row, make_float4(S[n][2 * i].x, S[n][2 * i].y, S[n][2 * i + 1].x, S[n][2 * i + 1].y));
          } else {
            const float x[4] = {S[n][2 * i].x, S[n][2 * i].y, S[n][2 * i + 1].x, S[n][2 * i + 1].y};
#pragma unroll
            for (int f = 0; f < 4; ++f)
              if (row + f < d) sp[row + f] = x[f];
          }
        }
        if (sub == 0) outs[j] = o;
      }
    }
    __syncthreads();
    const float by = RULE == RULE_MEMORY ? 1.f / (fmaxf(fabsf(outs[dv]), s4.w) + 1e-6f) : 1.f;
    if (warp == 0) {
      float s = 0.f;
      for (int i = lane; i < dv; i += 32) s = fmaf(outs[i] * by, outs[i] * by, s);
      s = warp_sum(s);
      if (lane == 0) red[3] = out_scale / sqrtf(s / (float)dv + eps);
    }
    __syncthreads();
    for (int i = tid; i < dv; i += SS_THREADS) {
      const float g = in.g[(size_t)b * in.ldg + (size_t)h * dv + i];
      out[(size_t)b * ldo + (size_t)h * dv + i] =
          from_float<TO>(outs[i] * by * red[3] * weight[shared_weight ? i : h * dv + i] * (act ? silu32(g) : sigmoid32(g)));
    }
    if (e + 1 < group) __syncthreads();                // the next head's results take the place
  }
}

// 1 if a step of single tokens with heads of these sizes has this kernel.
LLM_EXPORT int llm_state_step_supports(int d, int dv, int group, int rank) {
  return d <= 256 && ((long long)group * dv + dv + 1 + rank + 4 * group) * 4 <= 40 * 1024;
}

template <int RULE>
static int launch_state_step(const StepIn &in, float *state, const float *weight, int shared_weight, int act, float eps, float out_scale,
                             void *out, int out_dtype, long long ldo, const int *seq_slot, int n_seqs, int n_heads, int n_kv, int d, int dv,
                             cudaStream_t stream) {
  if (n_seqs == 0) return LLM_OK;
  const int group = n_kv > 0 ? n_heads / n_kv : 0;
  LLM_REQUIRE(n_seqs > 0 && n_heads > 0 && n_kv > 0 && n_heads % n_kv == 0 && n_kv <= 65535 && d > 0 && dv > 0, "state_step: bad sizes");
  LLM_REQUIRE(llm_state_step_supports(d, dv, group, RULE == RULE_BONUS ? in.rank : 0), "state_step: heads of %d and %d channels are not supported", d, dv);
  const size_t smem = ((size_t)group * dv + dv + 1 + (RULE == RULE_BONUS ? in.rank : 0) + 4 * group) * sizeof(float);
#define SS_GO(DMAX, TO)                                                                                                       \
  llm_launch(state_step_kernel<RULE, DMAX, TO>, dim3(n_seqs, n_kv), dim3(SS_THREADS), smem, stream, in, state, weight, shared_weight, act, \
             eps, out_scale, (TO *)out, ldo, seq_slot, n_heads, n_kv, d, dv)
#define SS_SIZES(TO)                   \
  do {                                 \
    if (d <= 32) SS_GO(32, TO);        \
    else if (d <= 64) SS_GO(64, TO);   \
    else if (d <= 128) SS_GO(128, TO); \
    else SS_GO(256, TO);               \
  } while (0)
  if (out_dtype == LLM_F32) SS_SIZES(float);
  else if (out_dtype == LLM_BF16) SS_SIZES(__nv_bfloat16);
  else LLM_FAIL("state_step: unknown dtype %d", out_dtype);
#undef SS_SIZES
#undef SS_GO
  LLM_CHECK_LAUNCH("state_step");
  return LLM_OK;
}

// Rows of `proj` (32-bit): q, k (kv_heads x d), v, gate (heads x dv), b and a (heads) at their offsets.
LLM_EXPORT int llm_delta_gated_step(const float *proj, long long ld, int off_q, int off_k, int off_v, int off_g, int off_b, int off_a,
                                    const float *conv, float *conv_state, int taps, const float *dt_bias, const float *a_log, float key_eps,
                                    float q_scale, float *state, const float *weight, int shared_weight, int act, float eps, float out_scale,
                                    void *out, int out_dtype, long long ldo, const int *seq_slot, int n_seqs, int n_heads, int n_kv, int d,
                                    int dv, cudaStream_t stream) {
  LLM_REQUIRE(taps >= 1 && (conv == nullptr || taps == 1 || conv_state != nullptr), "delta_gated_step: a convolution needs its state");
  StepIn in = {};
  in.q = proj + off_q, in.k = proj + off_k, in.v = proj + off_v, in.g = proj + off_g;
  in.ldq = in.ldk = in.ldv = in.ldg = in.ld_ab = ld;
  in.proj_ab = proj, in.off_b = off_b, in.off_a = off_a, in.dt_bias = dt_bias, in.a_log = a_log;
  in.conv = conv, in.conv_state = conv_state, in.taps = taps, in.key_eps = key_eps, in.q_scale = q_scale;
  return launch_state_step<RULE_DELTA>(in, state, weight, shared_weight, act, eps, out_scale, out, out_dtype, ldo, seq_slot, n_seqs, n_heads,
                                       n_kv, d, dv, stream);
}

LLM_EXPORT int llm_bonus_step(const float *r, long long ldr, const float *k, long long ldk, const float *v, long long ldv, const float *g,
                              long long ldg, const float *x1, long long ldx, int rank, const float *w2, const float *w0, const float *u,
                              float *state, const float *weight, int act, float eps, float out_scale, void *out, int out_dtype,
                              long long ldo, const int *seq_slot, int n_seqs, int n_heads, int d, int dv, cudaStream_t stream) {
  StepIn in = {};
  in.q = r, in.k = k, in.v = v, in.g = g, in.ldq = ldr, in.ldk = ldk, in.ldv = ldv, in.ldg = ldg;
  in.x1 = x1, in.ldx = ldx, in.rank = rank, in.w2 = w2, in.w0 = w0, in.u = u, in.q_scale = 1.f;
  return launch_state_step<RULE_BONUS>(in, state, weight, 0, act, eps, out_scale, out, out_dtype, ldo, seq_slot, n_seqs, n_heads, n_heads, d,
                                       dv, stream);
}

// Rows of `proj`: q, k (heads x d), v, gate (heads x dv), i and f (heads).
LLM_EXPORT int llm_memory_step(const float *proj, long long ld, int off_q, int off_k, int off_v, int off_g, int off_i, int off_f,
                               const float *bias_i, const float *bias_f, float cap, float q_scale, float *state_m, float *state,
                               const float *weight, int act, float eps, float out_scale, void *out, int out_dtype, long long ldo,
                               const int *seq_slot, int n_seqs, int n_heads, int d, int dv, cudaStream_t stream) {
  StepIn in = {};
  in.q = proj + off_q, in.k = proj + off_k, in.v = proj + off_v, in.g = proj + off_g;
  in.ldq = in.ldk = in.ldv = in.ldg = in.ld_if = ld;
  in.x_if = proj, in.off_i = off_i, in.off_f = off_f, in.bias_i = bias_i, in.bias_f = bias_f, in.cap = cap, in.state_m = state_m;
  in.q_scale = q_scale;
  return launch_state_step<RULE_MEMORY>(in, state, weight, 0, act, eps, out_scale, out, out_dtype, ldo, seq_slot, n_seqs, n_heads, n_heads, d,
                                        dv, stream);
}
