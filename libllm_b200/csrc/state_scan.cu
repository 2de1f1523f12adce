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
// What a token brings is packed first (the pack kernels below): a record of vectors per (token, key head),
// [k | q (r)] or [k | r | w], each padded with zeros to a multiple of 4 floats, and four scalars per (token, head),
// (a, beta or i, c, spare).  state [slots, heads, columns, d]: the d rows of a column together.  A step of single tokens
// has a kernel per rule that does everything between the products of h and the output projection in one launch.
//
// Everything here is 32-bit.  A sequence's result depends on nothing but its own tokens and state: one column belongs
// to a few neighbouring lanes, sums run in a fixed order, no sum crosses sequences.  The reference has no such mixer (its
// one mixer is attention, src/libllm/llama.cc:178-225).
#include "common.cuh"
#include <math.h>

LLM_DEFINE_LAST_ERROR(llm_state_scan_last_error)

enum Rule { RULE_DELTA = 0, RULE_BONUS = 1, RULE_MEMORY = 2 };

__device__ __forceinline__ float sigmoid32(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float silu32(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float softplus32(float x) { return x > 20.f ? x : log1pf(expf(x)); }
__device__ __forceinline__ float log_sigmoid32(float x) { return fminf(x, 0.f) - log1pf(expf(-fabsf(x))); }
__host__ __device__ constexpr int pad4(int d) { return (d + 3) / 4 * 4; }

// ---------------------------------------------------------------- the scan over a step's tokens
// CTA (sequence, head, run of columns): SC_THREADS threads of arithmetic, LANES neighbouring lanes to a column (lane `sub`
// owns rows 4 (sub + LANES i) .. + 3), and a warp that copies the tokens' records into a ring in shared memory, some
// tokens ahead of the arithmetic.
constexpr int SC_THREADS = 64;
constexpr int SC_STAGES = 16;                        // tokens of the ring, in four groups with a barrier each

__device__ __forceinline__ void sc_copy16(void *smem, const void *gmem) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((unsigned)__cvta_generic_to_shared(smem)), "l"(gmem));
}
__device__ __forceinline__ void sc_copy4(void *smem, const void *gmem) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((unsigned)__cvta_generic_to_shared(smem)), "l"(gmem));
}
__device__ __forceinline__ void sc_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void sc_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// This lane's share of a column: the token's products with the old state, then the new state.  kk, qq, ww point at the
// token's vectors (each DMAX floats apart in shared memory).
template <int RULE, int LANES, int ROWS>
__device__ __forceinline__ float scan_token(float (&S)[ROWS], const float *kk, const float *qq, const float *ww, float4 sc, float v, int sub) {
  float4 k4[ROWS / 4];
  float p[4] = {0.f, 0.f, 0.f, 0.f}, r[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
  for (int i = 0; i < ROWS / 4; ++i) {
    const int at = 4 * (sub + LANES * i);
    k4[i] = ld4(kk + at);
    const float4 q4 = ld4(qq + at);
    r[0] = fmaf(q4.x, S[4 * i], r[0]);
    r[1] = fmaf(q4.y, S[4 * i + 1], r[1]);
    r[2] = fmaf(q4.z, S[4 * i + 2], r[2]);
    r[3] = fmaf(q4.w, S[4 * i + 3], r[3]);
    if (RULE == RULE_DELTA) {
      p[0] = fmaf(k4[i].x, S[4 * i], p[0]);
      p[1] = fmaf(k4[i].y, S[4 * i + 1], p[1]);
      p[2] = fmaf(k4[i].z, S[4 * i + 2], p[2]);
      p[3] = fmaf(k4[i].w, S[4 * i + 3], p[3]);
    }
  }
  float rs = (r[0] + r[1]) + (r[2] + r[3]), z;
  if (RULE == RULE_DELTA) {
    float ps = (p[0] + p[1]) + (p[2] + p[3]);
#pragma unroll
    for (int o = 1; o < LANES; o <<= 1) {
      ps += __shfl_xor_sync(0xffffffffu, ps, o);
      rs += __shfl_xor_sync(0xffffffffu, rs, o);
    }
    z = sc.y * (v - sc.x * ps);
  } else {
#pragma unroll
    for (int o = 1; o < LANES; o <<= 1) rs += __shfl_xor_sync(0xffffffffu, rs, o);
    z = RULE == RULE_BONUS ? v : sc.y * v;
  }
#pragma unroll
  for (int i = 0; i < ROWS / 4; ++i) {
    float4 w4 = make_float4(sc.x, sc.x, sc.x, sc.x);
    if (RULE == RULE_BONUS) w4 = ld4(ww + 4 * (sub + LANES * i));
    S[4 * i] = fmaf(w4.x, S[4 * i], k4[i].x * z);
    S[4 * i + 1] = fmaf(w4.y, S[4 * i + 1], k4[i].y * z);
    S[4 * i + 2] = fmaf(w4.z, S[4 * i + 2], k4[i].z * z);
    S[4 * i + 3] = fmaf(w4.w, S[4 * i + 3], k4[i].w * z);
  }
  return (RULE == RULE_BONUS ? rs : sc.x * rs) + sc.z * z;
}

template <int RULE, int DMAX, int LANES>
__global__ void __launch_bounds__(SC_THREADS + 32)
state_scan_kernel(const float *__restrict__ rec, const float4 *__restrict__ scal, const float *__restrict__ v, long long ldv,
                  float *__restrict__ state, float *__restrict__ out, long long ldo, float *__restrict__ den,
                  const int *__restrict__ seq_start, const int *__restrict__ seq_slot, int n_heads, int n_kv, int d, int dv) {
  constexpr int NV = RULE == RULE_BONUS ? 3 : 2;
  constexpr int ROWS = DMAX / LANES;
  constexpr int COLS = SC_THREADS / LANES;
  constexpr int SLOT = NV * DMAX + 4 + COLS;         // vectors, scalars, the CTA's columns of v
  constexpr int STAGES = SC_STAGES * SLOT * 4 <= 48 * 1024 ? SC_STAGES : SC_STAGES / 2;
  constexpr int G = STAGES / 4, GROUPS = 4;
  constexpr int PER = (NV * DMAX / 4 + 1 + 31) / 32;  // 16-byte copies of a loader lane per token
  __shared__ __align__(16) float ring[STAGES][SLOT];
  grid_dependency_wait();
  const int b = blockIdx.x, hd = blockIdx.y, kvh = hd / (n_heads / n_kv);
  const int tid = threadIdx.x;
  const int j0 = blockIdx.z * COLS;
  const int start = seq_start[b], n = seq_start[b + 1] - start;
  const int n_groups = (n + G - 1) / G;
  const int n_cols = dv + (RULE == RULE_MEMORY ? 1 : 0);
  const int dp = pad4(d);
  // what is never copied stays as it is set here: rows beyond the padded size are nought, the column of n has v = 1
  for (int i = tid; i < STAGES * SLOT; i += SC_THREADS + 32) {
    const int at = i % SLOT - (NV * DMAX + 4);
    (&ring[0][0])[i] = RULE == RULE_MEMORY && at >= 0 && j0 + at == dv ? 1.f : 0.f;
  }
  __syncthreads();

  if (tid >= SC_THREADS) {
    const int lane = tid - SC_THREADS;
    const int per_vec = dp / 4, n16 = NV * per_vec;
    int from[PER], to[PER];
#pragma unroll
    for (int e = 0; e < PER; ++e) {
      const int idx = lane + e * 32;
      from[e] = to[e] = -1;
      if (idx < n16) {
        from[e] = idx * 4;
        to[e] = (idx / per_vec) * DMAX + (idx % per_vec) * 4;
      } else if (idx == n16) {
        from[e] = -2;                                 // the scalars
        to[e] = NV * DMAX;
      }
    }
    auto fetch_group = [&](int p) {
      for (int t = G * p; t < min(n, G * p + G); ++t) {
        float *dst = ring[t % STAGES];
        const size_t tok = (size_t)(start + t);
        const float *r = rec + (tok * n_kv + kvh) * (size_t)(NV * dp);
#pragma unroll
        for (int e = 0; e < PER; ++e)
          if (to[e] >= 0) sc_copy16(dst + to[e], from[e] >= 0 ? (const void *)(r + from[e]) : (const void *)(scal + tok * n_heads + hd));
        for (int c = lane; c < COLS; c += 32)
          if (j0 + c < dv) sc_copy4(dst + NV * DMAX + 4 + c, v + tok * (size_t)ldv + (size_t)hd * dv + j0 + c);
      }
      sc_commit();
    };
    for (int p = 0; p < GROUPS - 1; ++p) fetch_group(p);
    for (int p = 0; p < n_groups; ++p) {
      sc_wait<GROUPS - 2>();                          // group p has arrived
      __syncthreads();                                // everyone may read it, and is done with group p - 1
      fetch_group(p + GROUPS - 1);                    // ... whose place these copies take
    }
    sc_wait<0>();
    return;
  }

  const int sub = tid % LANES, col = tid / LANES, j = j0 + col;
  const bool live = j < n_cols;
  float S[ROWS];
  float *sp = state + (((size_t)seq_slot[b] * n_heads + hd) * n_cols + (live ? j : 0)) * d;
#pragma unroll
  for (int i = 0; i < ROWS; ++i) {
    const int row = 4 * (sub + LANES * (i / 4)) + i % 4;
    S[i] = live && row < d ? sp[row] : 0.f;
  }
  auto token = [&](int t) {
    const float *slot = ring[t % STAGES];
    const float4 sc = ld4(slot + NV * DMAX);
    const float o = scan_token<RULE, LANES, ROWS>(S, slot, slot + DMAX, slot + 2 * DMAX, sc, slot[NV * DMAX + 4 + col], sub);
    if (live && sub == 0) {
      const size_t tok = (size_t)(start + t);
      if (RULE == RULE_MEMORY && j == dv) den[tok * n_heads + hd] = o;
      else out[tok * (size_t)ldo + (size_t)hd * dv + j] = o;
    }
  };
  for (int p = 0; p < n_groups; ++p) {
    __syncthreads();
    if (G * p + G <= n) {
#pragma unroll
      for (int g = 0; g < G; ++g) token(G * p + g);
    } else {
      for (int t = G * p; t < n; ++t) token(t);
    }
  }
  // only now: this kernel is narrow and runs long, and a dependent let in at its start would sit beside it all that time
  grid_dependents_launch();
  if (live)
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
      const int row = 4 * (sub + LANES * (i / 4)) + i % 4;
      if (row < d) sp[row] = S[i];
    }
}

// rec [tokens, kv_heads, 2 or 3, pad4(d)], scal [tokens, heads, 4], v rows [tokens, >= heads * dv], state [slots, heads,
// dv (memory: + 1), d], out [tokens, heads * dv]; den [tokens, heads] (memory).  Launched behind its predecessor.
LLM_EXPORT int llm_state_scan(int rule, const float *rec, const float *scal, const float *v, long long ldv, float *state, float *out,
                              long long ldo, float *den, const int *seq_start, const int *seq_slot, int n_tokens, int n_seqs,
                              int n_heads, int n_kv, int d, int dv, cudaStream_t stream) {
  if (n_tokens == 0) return LLM_OK;
  LLM_REQUIRE(rule >= 0 && rule <= 2, "state_scan: rule %d is not known", rule);
  LLM_REQUIRE(n_tokens > 0 && n_seqs > 0 && n_heads > 0 && n_kv > 0 && n_heads % n_kv == 0 && d > 0 && dv > 0, "state_scan: bad sizes");
  LLM_REQUIRE(d <= 256, "state_scan: heads of %d key channels are not supported (up to 256)", d);
  LLM_REQUIRE(n_heads <= 65535, "state_scan: too many heads");
  LLM_REQUIRE((uintptr_t)rec % 16 == 0 && (uintptr_t)scal % 16 == 0 && (rule != RULE_MEMORY || den), "state_scan: bad pointers");
  const int n_cols = dv + (rule == RULE_MEMORY ? 1 : 0);
#define SC_GO(RULE, DMAX, LANES)                                                                                             \
  llm_launch_after(state_scan_kernel<RULE, DMAX, LANES>, dim3(n_seqs, n_heads, (n_cols + SC_THREADS / LANES - 1) / (SC_THREADS / LANES)), \
                   dim3(SC_THREADS + 32), 0, stream, rec, (const float4 *)scal, v, ldv, state, out, ldo, den, seq_start, seq_slot, \
                   n_heads, n_kv, d, dv)
#define SC_SIZES(RULE)                         \
  do {                                         \
    if (d <= 16) SC_GO(RULE, 16, 2);           \
    else if (d <= 32) SC_GO(RULE, 32, 2);      \
    else if (d <= 64) SC_GO(RULE, 64, 4);      \
    else if (d <= 128) SC_GO(RULE, 128, 8);    \
    else SC_GO(RULE, 256, 16);                 \
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
// Gated delta: rows `cv` [q (kv_heads x d) | k (kv_heads x d) | v] as the short convolution left them; q and k become unit
// vectors per key head, x / sqrt(sum x^2 + key_eps), q also times q_scale; per head beta = sigmoid(b), g =
// exp(-exp(a_log) softplus(a + dt_bias)), a and b at their offsets of the product's rows.  A warp per (token, key head).
__global__ void __launch_bounds__(128)
delta_pack_kernel(const float *__restrict__ cv, long long ldc, const float *__restrict__ proj, long long ld, int off_b, int off_a,
                  const float *__restrict__ dt_bias, const float *__restrict__ a_log, float key_eps, float q_scale,
                  float *__restrict__ rec, float4 *__restrict__ scal, int n_tokens, int n_heads, int n_kv, int d) {
  grid_dependents_launch();
  grid_dependency_wait();
  const int lane = threadIdx.x & 31;
  const long long item = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
  if (item >= (long long)n_tokens * n_kv) return;
  const int t = (int)(item / n_kv), kvh = (int)(item - (long long)t * n_kv), dp = pad4(d), group = n_heads / n_kv;
  const float *q = cv + (size_t)t * ldc + (size_t)kvh * d, *k = q + (size_t)n_kv * d;
  float qq = 0.f, kk = 0.f, kq = 0.f;
  for (int i = lane; i < d; i += 32) {
    qq = fmaf(q[i], q[i], qq);
    kk = fmaf(k[i], k[i], kk);
    kq = fmaf(k[i], q[i], kq);
  }
  qq = warp_sum(qq);
  kk = warp_sum(kk);
  kq = warp_sum(kq);
  const float iq = q_scale / sqrtf(qq + key_eps), ik = 1.f / sqrtf(kk + key_eps);
  float *r = rec + (size_t)item * 2 * dp;
  for (int i = lane; i < dp; i += 32) {
    r[i] = i < d ? k[i] * ik : 0.f;
    r[dp + i] = i < d ? q[i] * iq : 0.f;
  }
  for (int e = lane; e < group; e += 32) {
    const int h = kvh * group + e;
    const float *row = proj + (size_t)t * ld;
    const float g = expf(-expf(a_log[h]) * softplus32(row[off_a + h] + dt_bias[h]));
    scal[(size_t)t * n_heads + h] = make_float4(g, sigmoid32(row[off_b + h]), kq * iq * ik, 0.f);
  }
}

LLM_EXPORT int llm_delta_pack(const float *cv, long long ldc, const float *proj, long long ld, int off_b, int off_a, const float *dt_bias,
                              const float *a_log, float key_eps, float q_scale, float *rec, float *scal, int n_tokens, int n_heads,
                              int n_kv, int d, cudaStream_t stream) {
  if (n_tokens == 0) return LLM_OK;
  LLM_REQUIRE(n_tokens > 0 && n_heads > 0 && n_kv > 0 && n_heads % n_kv == 0 && d > 0, "delta_pack: bad sizes");
  const long long items = (long long)n_tokens * n_kv;
  llm_launch(delta_pack_kernel, dim3((unsigned)((items + 3) / 4)), dim3(128), 0, stream, cv, ldc, proj, ld, off_b, off_a, dt_bias, a_log,
             key_eps, q_scale, rec, (float4 *)scal, n_tokens, n_heads, n_kv, d);
  LLM_CHECK_LAUNCH("delta_pack");
  return LLM_OK;
}

// Bonus: r, k and the low-rank decay input x1 (rank values) of every token in rows of their own; per head the decay
// w = exp(-exp(w0 + W2 tanh(x1))) per key channel and c = sum_i r_i u_i k_i.  A CTA takes one head and a run of tokens, a warp a
// token at a time; the head's rows of W2 [d, rank] lie in shared memory where they fit (padded by one value).
constexpr int BP_WARPS = 4, BP_TOKENS = 32;

__global__ void __launch_bounds__(BP_WARPS * 32)
bonus_pack_kernel(const float *__restrict__ r, long long ldr, const float *__restrict__ k, long long ldk, const float *__restrict__ x1,
                  long long ldx, int rank, const float *__restrict__ w2, const float *__restrict__ w0, const float *__restrict__ u,
                  int n_tokens, int n_heads, int d, int w2_shared, float *__restrict__ rec, float4 *__restrict__ scal) {
  extern __shared__ float bp_sm[];                   // tanh(x1) [warps][rank], then W2's rows of the head [d][rank + 1]
  grid_dependents_launch();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, hd = blockIdx.y, dp = pad4(d);
  float *th = bp_sm + warp * rank, *w2s = bp_sm + BP_WARPS * rank;
  const float *w2h = w2 + (size_t)hd * d * rank;
  if (w2_shared)
    for (int i = threadIdx.x; i < d * rank; i += BP_WARPS * 32) w2s[(i / rank) * (rank + 1) + i % rank] = w2h[i];
  grid_dependency_wait();
  __syncthreads();
  const int t1 = min(n_tokens, (int)(blockIdx.x + 1) * BP_TOKENS);
  for (int t = blockIdx.x * BP_TOKENS + warp; t < t1; t += BP_WARPS) {
    const float *rr = r + (size_t)t * ldr + (size_t)hd * d, *kr = k + (size_t)t * ldk + (size_t)hd * d;
    __syncwarp();
    for (int q = lane; q < rank; q += 32) th[q] = tanhf(x1[(size_t)t * ldx + q]);
    __syncwarp();
    float *o = rec + ((size_t)t * n_heads + hd) * 3 * dp;
    float c = 0.f;
    for (int i0 = 0; i0 < dp; i0 += 128) {            // four channels of a lane at a time: four chains of sums
      float z[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int i = i0 + lane + 32 * e;
        z[e] = i < d ? w0[hd * d + i] : 0.f;
      }
      for (int q = 0; q < rank; ++q) {
        const float tq = th[q];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int i = i0 + lane + 32 * e;
          if (i < d) z[e] = fmaf(w2_shared ? w2s[i * (rank + 1) + q] : w2h[(size_t)i * rank + q], tq, z[e]);
        }
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int i = i0 + lane + 32 * e;
        if (i >= dp) continue;
        const float ki = i < d ? kr[i] : 0.f, ri = i < d ? rr[i] : 0.f;
        if (i < d) c = fmaf(ri * u[hd * d + i], ki, c);
        o[i] = ki;
        o[dp + i] = ri;
        o[2 * dp + i] = i < d ? expf(-expf(z[e])) : 0.f;
      }
    }
    c = warp_sum(c);
    if (lane == 0) scal[(size_t)t * n_heads + hd] = make_float4(1.f, 1.f, c, 0.f);
  }
}

LLM_EXPORT int llm_bonus_pack(const float *r, long long ldr, const float *k, long long ldk, const float *x1, long long ldx, int rank,
                              const float *w2, const float *w0, const float *u, float *rec, float *scal, int n_tokens, int n_heads, int d,
                              cudaStream_t stream) {
  if (n_tokens == 0) return LLM_OK;
  LLM_REQUIRE(n_tokens > 0 && n_heads > 0 && n_heads <= 65535 && d > 0 && rank > 0, "bonus_pack: bad sizes");
  const size_t with_w2 = ((size_t)BP_WARPS * rank + (size_t)d * (rank + 1)) * sizeof(float);
  const int w2_shared = with_w2 <= 96 * 1024;
  const size_t smem = w2_shared ? with_w2 : (size_t)BP_WARPS * rank * sizeof(float);
  LLM_REQUIRE(smem <= 96 * 1024, "bonus_pack: a decay input of rank %d is not supported", rank);
  LLM_CHECK_CUDA(llm_allow_smem(bonus_pack_kernel, smem), "bonus_pack attribute");
  llm_launch(bonus_pack_kernel, dim3((unsigned)((n_tokens + BP_TOKENS - 1) / BP_TOKENS), n_heads), dim3(BP_WARPS * 32), smem, stream, r, ldr,
             k, ldk, x1, ldx, rank, w2, w0, u, n_tokens, n_heads, d, w2_shared, rec, (float4 *)scal);
  LLM_CHECK_LAUNCH("bonus_pack");
  return LLM_OK;
}

// Memory: the gates of a sequence's tokens in order.  log gates i = cap tanh((x_i + b_i) / cap), f = logsigmoid(cap tanh((x_f +
// b_f) / cap)); with the running maximum m (state [slots, heads], 0 at the start) m_t = max(f + m_(t-1), i):
// scal = (exp(f + m_(t-1) - m_t), exp(i - m_t), room for c, exp(-m_t)).  A CTA per (sequence, head): the logarithms of 128 tokens
// side by side, their maxima one after another by one thread out of shared memory, the exponentials side by side.
constexpr int MG_TOKENS = 128;

__device__ __forceinline__ float capped(float x, float cap) { return cap * tanhf(x / cap); }

__global__ void __launch_bounds__(MG_TOKENS)
memory_gates_kernel(const float *__restrict__ proj, long long ld, int off_i, int off_f, const float *__restrict__ bias_i,
                    const float *__restrict__ bias_f, float cap, float *__restrict__ state_m, float4 *__restrict__ scal,
                    const int *__restrict__ seq_start, const int *__restrict__ seq_slot, int n_heads) {
  __shared__ float li[MG_TOKENS], lf[MG_TOKENS], m[MG_TOKENS + 1];
  grid_dependents_launch();
  grid_dependency_wait();
  const int b = blockIdx.x, hd = blockIdx.y, tid = threadIdx.x;
  const int start = seq_start[b], n = seq_start[b + 1] - start;
  float *mp = state_m + (size_t)seq_slot[b] * n_heads + hd;
  if (tid == 0) m[0] = *mp;
  for (int t0 = 0; t0 < n; t0 += MG_TOKENS) {
    const int t = t0 + tid, nt = min(MG_TOKENS, n - t0);
    if (t < n) {
      const float *row = proj + (size_t)(start + t) * ld;
      li[tid] = capped(row[off_i + hd] + bias_i[hd], cap);
      lf[tid] = log_sigmoid32(capped(row[off_f + hd] + bias_f[hd], cap));
    }
    __syncthreads();
    if (tid == 0) {
      float run = m[0];
#pragma unroll 8
      for (int e = 0; e < nt; ++e) m[e + 1] = run = fmaxf(lf[e] + run, li[e]);
    }
    __syncthreads();
    if (t < n)
      scal[(size_t)(start + t) * n_heads + hd] =
          make_float4(expf(lf[tid] + m[tid] - m[tid + 1]), expf(li[tid] - m[tid + 1]), 0.f, expf(-m[tid + 1]));
    __syncthreads();
    if (tid == 0) m[0] = m[nt];
  }
  if (tid == 0) *mp = m[0];
}

// Its vectors: k and q (times q_scale) of the product's rows, c = k . q.  A warp per (token, head).
__global__ void __launch_bounds__(128)
memory_pack_kernel(const float *__restrict__ proj, long long ld, int off_q, int off_k, float q_scale, float *__restrict__ rec,
                   float4 *__restrict__ scal, int n_tokens, int n_heads, int d) {
  grid_dependents_launch();
  grid_dependency_wait();
  const int lane = threadIdx.x & 31, dp = pad4(d);
  const long long item = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
  if (item >= (long long)n_tokens * n_heads) return;
  const int t = (int)(item / n_heads), hd = (int)(item - (long long)t * n_heads);
  const float *q = proj + (size_t)t * ld + off_q + (size_t)hd * d, *k = proj + (size_t)t * ld + off_k + (size_t)hd * d;
  float *r = rec + (size_t)item * 2 * dp;
  float kq = 0.f;
  for (int i = lane; i < dp; i += 32) {
    const float ki = i < d ? k[i] : 0.f, qi = i < d ? q[i] * q_scale : 0.f;
    kq = fmaf(ki, qi, kq);
    r[i] = ki;
    r[dp + i] = qi;
  }
  kq = warp_sum(kq);
  if (lane == 0) scal[item].z = kq;
}

LLM_EXPORT int llm_memory_pack(const float *proj, long long ld, int off_q, int off_k, int off_i, int off_f, const float *bias_i,
                               const float *bias_f, float cap, float q_scale, float *state_m, float *rec, float *scal,
                               const int *seq_start, const int *seq_slot, int n_tokens, int n_seqs, int n_heads, int d,
                               cudaStream_t stream) {
  if (n_tokens == 0) return LLM_OK;
  LLM_REQUIRE(n_tokens > 0 && n_seqs > 0 && n_heads > 0 && n_heads <= 65535 && d > 0 && cap > 0.f, "memory_pack: bad sizes");
  llm_launch(memory_gates_kernel, dim3(n_seqs, n_heads), dim3(MG_TOKENS), 0, stream, proj, ld, off_i, off_f, bias_i, bias_f, cap, state_m,
             (float4 *)scal, seq_start, seq_slot, n_heads);
  LLM_CHECK_LAUNCH("memory_gates");
  const long long items = (long long)n_tokens * n_heads;
  llm_launch(memory_pack_kernel, dim3((unsigned)((items + 3) / 4)), dim3(128), 0, stream, proj, ld, off_q, off_k, q_scale, rec,
             (float4 *)scal, n_tokens, n_heads, d);
  LLM_CHECK_LAUNCH("memory_pack");
  return LLM_OK;
}

// ---------------------------------------------------------------- behind the scan: norm per head, weight, gate
// y = x / (max(|den|, floor) + 1e-6)   where den is given (memory; floor = scal's fourth value)
// out = y / sqrt(mean(y^2) + eps) * weight * gate * out_scale; weight [heads * dv], or [dv] shared by the heads; gate:
// sigmoid (act 0) or silu (act 1) of 32-bit logits.  A warp per (token, head), the head in registers (up to 512 values).
constexpr int HF_MAX = 16;

template <typename T>
__global__ void __launch_bounds__(128)
head_finish_kernel(const float *__restrict__ x, long long ldx, const float *__restrict__ den, const float4 *__restrict__ scal,
                   const float *__restrict__ weight, int shared_weight, const float *__restrict__ gate, long long gate_stride, int act,
                   float eps, float out_scale, int n_tokens, int n_heads, int dv, T *__restrict__ out, long long ldo) {
  grid_dependents_launch();
  grid_dependency_wait();
  const int lane = threadIdx.x & 31;
  const long long item = (long long)blockIdx.x * 4 + (threadIdx.x >> 5);
  if (item >= (long long)n_tokens * n_heads) return;
  const int t = (int)(item / n_heads), hd = (int)(item - (long long)t * n_heads);
  const float *xr = x + (size_t)t * ldx + (size_t)hd * dv, *gr = gate + (size_t)t * gate_stride + (size_t)hd * dv;
  const float *wr = weight + (shared_weight ? 0 : (size_t)hd * dv);
  T *o = out + (size_t)t * ldo + (size_t)hd * dv;
  const float by = den ? 1.f / (fmaxf(fabsf(den[item]), scal[item].w) + 1e-6f) : 1.f;
  float v[HF_MAX], ss = 0.f;
#pragma unroll
  for (int e = 0; e < HF_MAX; ++e) {
    const int i = lane + 32 * e;
    v[e] = i < dv ? xr[i] * by : 0.f;
    ss = fmaf(v[e], v[e], ss);
  }
  const float inv = out_scale / sqrtf(warp_sum(ss) / (float)dv + eps);
#pragma unroll
  for (int e = 0; e < HF_MAX; ++e) {
    const int i = lane + 32 * e;
    if (i < dv) {
      const float g = gr[i];
      o[i] = from_float<T>(v[e] * inv * wr[i] * (act ? silu32(g) : sigmoid32(g)));
    }
  }
}

LLM_EXPORT int llm_head_finish(const float *x, long long ldx, const float *den, const float *scal, const float *weight, int shared_weight,
                               const float *gate, long long gate_stride, int act, float eps, float out_scale, int n_tokens, int n_heads,
                               int dv, void *out, int out_dtype, long long ldo, cudaStream_t stream) {
  if (n_tokens == 0) return LLM_OK;
  LLM_REQUIRE(n_tokens > 0 && n_heads > 0 && dv > 0 && dv <= 32 * HF_MAX, "head_finish: heads of %d values are not supported (up to %d)", dv,
              32 * HF_MAX);
  LLM_REQUIRE(act == 0 || act == 1, "head_finish: gate activation %d is not known", act);
  const dim3 grid((unsigned)(((long long)n_tokens * n_heads + 3) / 4));
#define HF_GO(T)                                                                                                              \
  llm_launch(head_finish_kernel<T>, grid, dim3(128), 0, stream, x, ldx, den, (const float4 *)scal, weight, shared_weight, gate, \
             gate_stride, act, eps, out_scale, n_tokens, n_heads, dv, (T *)out, ldo)
  if (out_dtype == LLM_F32) HF_GO(float);
  else if (out_dtype == LLM_BF16) HF_GO(__nv_bfloat16);
  else LLM_FAIL("head_finish: unknown dtype %d", out_dtype);
#undef HF_GO
  LLM_CHECK_LAUNCH("head_finish");
  return LLM_OK;
}

// ---------------------------------------------------------------- a token beside its predecessor
// out[s][t] = h_t + (h_(t-1) - h_t) mu_s for n_mix vectors mu [n_mix, width] (32-bit arithmetic, rounded once); the last row
// of every sequence is its state [slots, width].  A sequence's first row of the step and the state belong to a CTA of
// their sequence (blockIdx.y - n_chunks), whose threads read the old row of their channel before they write the new one.
constexpr int TS_THREADS = 128, TS_ROWS = 8;

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

template <typename T, int V>
__global__ void __launch_bounds__(TS_THREADS)
token_shift_kernel(const T *__restrict__ h, long long ldh, const float *__restrict__ mu, int n_mix, T *__restrict__ out, long long mix_stride,
                   T *__restrict__ state, const int *__restrict__ tok_seq, const int *__restrict__ tok_pos,
                   const int *__restrict__ seq_start, const int *__restrict__ seq_past, const int *__restrict__ seq_slot, int n_tokens,
                   int width, int n_chunks) {
  grid_dependents_launch();
  grid_dependency_wait();
  const int c = (blockIdx.x * TS_THREADS + threadIdx.x) * V;
  if (c >= width) return;
  auto row_out = [&](int t, const TsVec<T, V> &cur, const TsVec<T, V> &prev) {
    for (int s = 0; s < n_mix; ++s) {
      TsVec<T, V> r;
#pragma unroll
      for (int v = 0; v < V; ++v) r.x[v] = fmaf(prev.x[v] - cur.x[v], mu[(size_t)s * width + c + v], cur.x[v]);
      ts_store<T, V>(out + (size_t)s * mix_stride + (size_t)t * width + c, r);
    }
  };
  if ((int)blockIdx.y < n_chunks) {
    const int r0 = blockIdx.y * TS_ROWS, r1 = min(n_tokens, r0 + TS_ROWS);
    for (int t = r0; t < r1; ++t)
      if (tok_pos[t] > seq_past[tok_seq[t]]) row_out(t, ts_load<T, V>(h + (size_t)t * ldh + c), ts_load<T, V>(h + (size_t)(t - 1) * ldh + c));
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
  LLM_REQUIRE(n_tokens > 0 && n_seqs > 0 && width > 0 && n_mix > 0 && state, "token_shift: bad arguments");
  const int n_chunks = single_tokens ? 0 : (n_tokens + TS_ROWS - 1) / TS_ROWS;
  LLM_REQUIRE(n_chunks + n_seqs <= 65535, "token_shift: too many rows for one launch");
  const int esz = dtype == LLM_F32 ? 4 : 2;
  const bool vec = width % 4 == 0 && ldh % 4 == 0 && mix_stride % 4 == 0 && (uintptr_t)h % (4 * esz) == 0 && (uintptr_t)out % (4 * esz) == 0 &&
                   (uintptr_t)state % (4 * esz) == 0;
  const int v = vec ? 4 : 1;
  const dim3 grid((width + TS_THREADS * v - 1) / (TS_THREADS * v), n_chunks + n_seqs);
#define TS_GO(T, V)                                                                                                            \
  llm_launch(token_shift_kernel<T, V>, grid, dim3(TS_THREADS), 0, stream, (const T *)h, ldh, mu, n_mix, (T *)out, mix_stride, (T *)state, \
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
  float S[NC][R4 * 4];
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
          S[n][4 * i] = s4.x, S[n][4 * i + 1] = s4.y, S[n][4 * i + 2] = s4.z, S[n][4 * i + 3] = s4.w;
        } else {
#pragma unroll
          for (int e = 0; e < 4; ++e) S[n][4 * i + e] = j < n_cols && row + e < d ? sp[row + e] : 0.f;
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
            if (row < d) st4(sp + row, make_float4(S[n][4 * i], S[n][4 * i + 1], S[n][4 * i + 2], S[n][4 * i + 3]));
          } else {
#pragma unroll
            for (int f = 0; f < 4; ++f)
              if (row + f < d) sp[row + f] = S[n][4 * i + f];
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
