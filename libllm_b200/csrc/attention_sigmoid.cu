// Attention whose weights stand each for itself: a visible key's weight is sigmoid(cap tanh(s temp[h] / cap) + bias[h]) of
// its score s (cap 0: no bound), not normalised over the keys, so that runs of keys simply add.  bfloat16 operands over the
// paged cache, scores, weights and sums in 32-bit.  Causal, optionally a window; values of a width of their own.
//
// Prompt steps (tcgen05): the structure of attention_prefill_tc.cu's first form without what a softmax needs.  A CTA takes 128
// query rows of one head of one sequence:
//   warp 8     brings the Q tile once and then, page by page, K and V tiles (a page of the cache is one key tile) by TMA;
//   warp 9     issues S = Q K^T into one of two score buffers in tensor memory;
//   warp 10    issues O += P V, P the A operand straight from tensor memory, V the MN-major B operand; O stays in tensor memory;
//   warps 0-7  two threads per query row, each with half of the tile's keys: scores out of tensor memory, weights, and P as
//              packed bfloat16 over the half's own score columns.  Nothing passes between the partners, no row is rescaled.
// Heads that are no multiple of 64 channels are padded by TMA: channels of K and V beyond the head read as zeros, what the Q
// tile holds there (the next head's) meets zeros.  Every wait has a time limit (tc_common.cuh).
//
// The weight's two exponentials and two reciprocals: with r = 1 / (1 + 2^(s c1)) the bounded score is cap (1 - 2 r), and the
// weight 1 / (1 + 2^(A + B r)).  A pair of scores shares one reciprocal (1/x = y / (x y), exponents bounded to keep the product
// finite), so that a score costs three special-function instructions, not four.
//
// Single tokens (mma.sync): a CTA per (run of pages, kv head, sequence), the group's heads as the rows of a 16-row tile; K and V
// pages through shared memory, two in flight.  The four warps share out a page's keys for S, leave P in shared memory, and
// share out the value channels for O.  Runs are added, in order, by the CTA that finishes last.
//
// The reference has no such attention (its own: src/flint/cuda/flash_attn.cc:101-186).
#include "common.cuh"
#include "mma_tiles.cuh"
#include "tc_common.cuh"
#include <math.h>

LLM_DEFINE_LAST_ERROR(llm_attention_sigmoid_last_error)

namespace {

constexpr float LOG2E = 1.4426950408889634f;
constexpr float MAX_EXP = 60.f;             // 2^60 stands for infinity: its reciprocal is nought beside any rounding

__device__ __forceinline__ float sg_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float sg_rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

struct Weigh {
  float c1, a, b;                           // bounded: r = 1 / (1 + 2^(s c1)), weight 1 / (1 + 2^(a + b r)); else 1 / (1 + 2^(a + b s))
  bool bounded;
};
// scale, temperature, bound and bias as the constants above
__device__ __forceinline__ Weigh weigh_of(float scale, float temp, float cap, float bias) {
  Weigh w;
  w.bounded = cap > 0.f;
  if (w.bounded) {
    w.c1 = 2.f * LOG2E * scale * temp / cap;
    w.a = -(cap + bias) * LOG2E;
    w.b = 2.f * cap * LOG2E;
  } else {
    w.c1 = 0.f;
    w.a = -bias * LOG2E;
    w.b = -scale * temp * LOG2E;
  }
  return w;
}
// 1 / (1 + 2^x) and 1 / (1 + 2^y)
__device__ __forceinline__ float2 inverse_pair(float x, float y) {
  const float p = 1.f + sg_exp2(fminf(x, MAX_EXP)), q = 1.f + sg_exp2(fminf(y, MAX_EXP));
  const float i = sg_rcp(p * q);
  return make_float2(q * i, p * i);
}
template <bool BOUNDED>
__device__ __forceinline__ float2 weights_of(const Weigh &w, float s0, float s1) {
  float2 r = make_float2(s0, s1);
  if (BOUNDED) r = inverse_pair(s0 * w.c1, s1 * w.c1);
  return inverse_pair(fmaf(w.b, r.x, w.a), fmaf(w.b, r.y, w.a));
}

// ------------------------------------------------------------------ prompt steps
constexpr int SA_THREADS = 384, SA_BM = 128, SA_BN = 64;

template <int KB, int VB>                   // blocks of 64 channels of a key and of a value
struct SaShape {
  static constexpr int Q_BYTES = SA_BM * KB * 128;
  static constexpr int K_BYTES = SA_BN * KB * 128, V_BYTES = SA_BN * VB * 128, KV_BYTES = K_BYTES + V_BYTES;
  static constexpr int TMEM_COLS = 2 * SA_BN + 64 * VB <= 256 ? 256 : 512;
  static constexpr int CTAS = TMEM_COLS == 256 ? 2 : 1;     // per SM
  static constexpr int BUDGET = CTAS == 2 ? 108 * 1024 : 200 * 1024;
  static constexpr int STAGES_FIT = (BUDGET - Q_BYTES) / KV_BYTES;
  static constexpr int STAGES = STAGES_FIT > 4 ? 4 : STAGES_FIT;
  static constexpr size_t SMEM = Q_BYTES + (size_t)STAGES * KV_BYTES + 256;
  static constexpr int REGS_LAUNCH = CTAS == 2 ? 80 : 168, REGS_FEW = CTAS == 2 ? 48 : 56, REGS_MANY = CTAS == 2 ? 96 : 216;
  static_assert(STAGES >= 2, "two tiles in flight");
  static_assert(128 * REGS_FEW + 256 * REGS_MANY <= SA_THREADS * REGS_LAUNCH, "register moves must balance within the CTA");
};

template <int KB, int VB, bool BOUNDED>
__global__ void __launch_bounds__(SA_THREADS, SaShape<KB, VB>::CTAS)
sigmoid_prefill_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                       const __grid_constant__ CUtensorMap map_v, __nv_bfloat16 *__restrict__ out, long long out_stride,
                       const int *__restrict__ seq_start, const int *__restrict__ seq_past, const int *__restrict__ page_table,
                       int pt_stride, int n_heads, int n_kv, int d, int dv, int window, float scale, const float *__restrict__ temp,
                       const float *__restrict__ bias, float cap, float out_scale, int *status) {
  using S = SaShape<KB, VB>;
  constexpr int STAGES = S::STAGES;
  extern __shared__ __align__(1024) unsigned char smem[];
  unsigned char *sQ = smem, *sKV = smem + S::Q_BYTES;
  unsigned long long *bars = (unsigned long long *)(sKV + (size_t)STAGES * S::KV_BYTES);
  // full[STAGES], empty[STAGES], q_full, then one per score buffer: s_full[2], p_full[2], pv_done[2]; last
  const unsigned bar_full = smem_u32(bars), bar_empty = smem_u32(bars + STAGES), bar_q = smem_u32(bars + 2 * STAGES),
                 bar_sfull = bar_q + 8, bar_pfull = bar_q + 24, bar_pvdone = bar_q + 40, bar_last = bar_q + 56;
  unsigned *tmem_slot = (unsigned *)(bars + 2 * STAGES + 8);
  volatile int *abort_flag = (volatile int *)(tmem_slot + 1);

  const int warp = __shfl_sync(0xffffffffu, threadIdx.x >> 5, 0), lane = threadIdx.x & 31;
  grid_dependents_launch();
  if (threadIdx.x == 0) {
    tma_prefetch_map(&map_q);
    tma_prefetch_map(&map_k);
    tma_prefetch_map(&map_v);
  }
  if (smem_u32(smem) & 1023u) {                               // swizzled tiles need 1024-byte alignment
    if (threadIdx.x == 0 && status) atomicCAS(status, 0, 61);
    return;
  }
  if (threadIdx.x == 0) {
    for (int s = 0; s < STAGES; ++s) {
      mbar_init(bar_full + 8 * s, 1);
      mbar_init(bar_empty + 8 * s, 1);
    }
    mbar_init(bar_q, 1);
    for (int x = 0; x < 2; ++x) {
      mbar_init(bar_sfull + 8 * x, 1);
      mbar_init(bar_pfull + 8 * x, 8);
      mbar_init(bar_pvdone + 8 * x, 1);
    }
    mbar_init(bar_last, 1);
    *abort_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 9) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)),
                 "r"((unsigned)S::TMEM_COLS) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const unsigned tmem_base = *tmem_slot;
  const unsigned tmem_s = tmem_base, tmem_o = tmem_base + 2 * SA_BN;

  grid_dependency_wait();
  // [heads, sequences, query tiles]: every head's longest (last) tile is handed out first
  const int b = blockIdx.y, h = blockIdx.x;
  const int q0 = seq_start[b], n_q = seq_start[b + 1] - q0, past = seq_past[b];
  const int r0 = (gridDim.z - 1 - blockIdx.z) * SA_BM;
  const bool active = r0 < n_q;
  const int rows = active ? min(SA_BM, n_q - r0) : 0;
  const int kvh = h / (n_heads / n_kv);
  const int last_tile = active ? (past + r0 + rows - 1) / SA_BN : -1;
  const int first_tile = (window > 0 ? max(0, past + r0 - window + 1) : 0) / SA_BN;
  const int n_tiles = last_tile - first_tile + 1;             // <= 0: nothing to do
  const int *pt = page_table + (size_t)b * pt_stride;

  if (warp >= 8) {
  asm volatile("setmaxnreg.dec.sync.aligned.u32 %0;" ::"n"(S::REGS_FEW));
  if (warp == 8) {
    // ------------------------------------------------------------ loader
    const bool leader = elect_one();
    if (n_tiles > 0) {
      if (leader) {
        mbar_expect_tx(bar_q, S::Q_BYTES);
        for (int kb = 0; kb < KB; ++kb) {
          tma_load_2d(smem_u32(sQ) + kb * (SA_BM * 128), &map_q, h * d + kb * 64, q0 + r0, bar_q);
          tma_load_2d(smem_u32(sQ) + kb * (SA_BM * 128) + 64 * 128, &map_q, h * d + kb * 64, q0 + r0 + 64, bar_q);
        }
      }
      int stage = 0;
      unsigned phase = 0;
      bool ok = true;
      for (int j = 0; j < n_tiles && ok; ++j) {
        ok = __all_sync(0xffffffffu, mbar_wait(bar_empty + 8 * stage, phase ^ 1, abort_flag, status, 51));
        if (!ok) break;
        const int row = (pt[first_tile + j] * n_kv + kvh) * SA_BN;
        const unsigned dk = smem_u32(sKV + (size_t)stage * S::KV_BYTES), dvv = dk + S::K_BYTES;
        if (leader) {
          mbar_expect_tx(bar_full + 8 * stage, S::KV_BYTES);
          for (int kb = 0; kb < KB; ++kb) tma_load_2d(dk + kb * (SA_BN * 128), &map_k, kb * 64, row, bar_full + 8 * stage);
          for (int kb = 0; kb < VB; ++kb) tma_load_2d(dvv + kb * (SA_BN * 128), &map_v, kb * 64, row, bar_full + 8 * stage);
        }
        if (++stage == STAGES) {
          stage = 0;
          phase ^= 1;
        }
      }
      if (leader && (!ok || *abort_flag)) {
        const unsigned long long t0 = globaltimer();
        for (int s = 0; s < STAGES; ++s)
          while (!mbar_try(bar_full + 8 * s, 0) && !mbar_try(bar_full + 8 * s, 1) && globaltimer() - t0 < 2000000ull) {
          }
      }
    }
  } else if (warp == 9) {
    // ------------------------------------------------------------ tensor-core issue: scores
    const bool leader = elect_one();
    if (n_tiles > 0) {
      constexpr unsigned IDESC_S = instr_desc(SA_BM, SA_BN);
      bool ok = __all_sync(0xffffffffu, mbar_wait(bar_q, 0, abort_flag, status, 52));
      for (int j = 0; j < n_tiles && ok; ++j) {
        const int stage = j % STAGES;
        ok = mbar_wait(bar_full + 8 * stage, (j / STAGES) & 1, abort_flag, status, 53);
        // buffer j & 1 last held tile j - 2's scores and weights, which the other warp's product has to have read
        if (ok && j >= 2) ok = mbar_wait(bar_pvdone + 8 * (j & 1), ((j >> 1) - 1) & 1, abort_flag, status, 54);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        tc_fence_after();
        const unsigned ka = smem_u32(sKV + (size_t)stage * S::KV_BYTES);
        if (leader) {
#pragma unroll
          for (int kb = 0; kb < KB; ++kb)
#pragma unroll
            for (int kk = 0; kk < 4; ++kk)
              tc_mma(tmem_s + (j & 1) * SA_BN, smem_desc(smem_u32(sQ) + kb * (SA_BM * 128) + kk * 32),
                     smem_desc(ka + kb * (SA_BN * 128) + kk * 32), IDESC_S, (kb > 0 || kk > 0) ? 1u : 0u);
          tc_commit(bar_sfull + 8 * (j & 1));
        }
        __syncwarp();
      }
    }
  } else if (warp == 10) {
    // ------------------------------------------------------------ tensor-core issue: output
    const bool leader = elect_one();
    if (n_tiles > 0) {
      constexpr unsigned IDESC_O = instr_desc(SA_BM, 64 * VB) | (1u << 16);      // V lies [key][channel]: MN-major
      bool ok = true;
      for (int j = 0; j < n_tiles && ok; ++j) {
        const int stage = j % STAGES;
        ok = mbar_wait(bar_full + 8 * stage, (j / STAGES) & 1, abort_flag, status, 55) &&
             mbar_wait(bar_pfull + 8 * (j & 1), (j >> 1) & 1, abort_flag, status, 56);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        tc_fence_after();
        const unsigned va = smem_u32(sKV + (size_t)stage * S::KV_BYTES) + S::K_BYTES;
        // 16 keys to a product; the second half of the keys has its weights 32 columns further on
        if (leader) {
#pragma unroll
          for (int kk = 0; kk < SA_BN / 16; ++kk)
            tc_mma_ts(tmem_o, tmem_s + (j & 1) * SA_BN + (kk >> 1) * 32 + (kk & 1) * 8, smem_desc_lbo(va + kk * 2048, SA_BN * 128), IDESC_O,
                      (j > 0 || kk > 0) ? 1u : 0u);
          tc_commit(bar_pvdone + 8 * (j & 1));
          tc_commit(bar_empty + 8 * stage);
          if (j + 1 == n_tiles) tc_commit(bar_last);
        }
        __syncwarp();
      }
    }
  }
  } else {
    // ------------------------------------------------------------ two threads per query row
    asm volatile("setmaxnreg.inc.sync.aligned.u32 %0;" ::"n"(S::REGS_MANY));
    const int quarter = warp & 3, half = warp >> 2;
    const int row = quarter * 32 + lane;                       // row of the tile = lane of tensor memory
    const unsigned lane_addr = (unsigned)(quarter * 32) << 16;
    const int pos = past + r0 + row;
    const Weigh w = weigh_of(scale, temp[h], cap, bias[h]);
    const int vis_lo = window > 0 ? pos - window + 1 : 0;
    bool ok = n_tiles > 0;
    for (int j = 0; j < n_tiles && ok; ++j) {
      ok = __all_sync(0xffffffffu, mbar_wait(bar_sfull + 8 * (j & 1), (j >> 1) & 1, abort_flag, status, 58));
      if (!ok) break;
      const unsigned s_addr = tmem_s + (j & 1) * SA_BN + lane_addr + half * 32;
      const int k0 = (first_tile + j) * SA_BN + half * 32;    // this thread's first key
      float own[2][16];
      tc_fence_after();
      tc_ld16_issue(s_addr, own[0]);
      tc_ld16_issue(s_addr + 16, own[1]);
      tc_ld_wait();
      tc_ld_ready(own[0]);
      tc_ld_ready(own[1]);
      const bool edge = (k0 + 31 > past + r0) || (window > 0 && k0 <= past + r0 + SA_BM - 1 - window);
      unsigned pk[16];                                        // two keys to a column
#pragma unroll
      for (int c = 0; c < 2; ++c)
#pragma unroll
        for (int i = 0; i < 16; i += 2) {
          float2 p = weights_of<BOUNDED>(w, own[c][i], own[c][i + 1]);
          if (edge) {
            const int key = k0 + c * 16 + i;
            if (key > pos || key < vis_lo) p.x = 0.f;
            if (key + 1 > pos || key + 1 < vis_lo) p.y = 0.f;
          }
          pk[c * 8 + (i >> 1)] = pack_bf16(p.x, p.y);
        }
      tc_st16(s_addr, pk);
      tc_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(bar_pfull + 8 * (j & 1));
    }
    if (ok) ok = __all_sync(0xffffffffu, mbar_wait(bar_last, 0, abort_flag, status, 60));
    if (ok) {
      tc_fence_after();
      constexpr int HD = 32 * VB;                             // this thread's channels of the output row
      const unsigned o_addr = tmem_o + lane_addr + half * HD;
      __nv_bfloat16 *dst = out + (size_t)(q0 + r0 + row) * out_stride + (size_t)h * dv + half * HD;
#pragma unroll
      for (int c0 = 0; c0 < HD; c0 += 16) {
        float t[16];
        tc_ld16(o_addr + c0, t);
        if (row < rows) {
#pragma unroll
          for (int h8 = 0; h8 < 2; ++h8) {
            if (half * HD + c0 + h8 * 8 >= dv) continue;      // heads of a multiple of 8 channels
            uint4 v;
            v.x = pack_bf16(t[h8 * 8] * out_scale, t[h8 * 8 + 1] * out_scale);
            v.y = pack_bf16(t[h8 * 8 + 2] * out_scale, t[h8 * 8 + 3] * out_scale);
            v.z = pack_bf16(t[h8 * 8 + 4] * out_scale, t[h8 * 8 + 5] * out_scale);
            v.w = pack_bf16(t[h8 * 8 + 6] * out_scale, t[h8 * 8 + 7] * out_scale);
            *reinterpret_cast<uint4 *>(dst + c0 + h8 * 8) = v;
          }
        }
      }
      tc_fence_before();
    }
  }

  tc_fence_before();
  __syncthreads();
  if (warp == 9) {
    tc_fence_after();
    __syncwarp();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"((unsigned)S::TMEM_COLS)
                 : "memory");
  }
}

template <int KB, int VB>
int launch_sigmoid_prefill(const CUtensorMap &map_q, const CUtensorMap &map_k, const CUtensorMap &map_v, void *out, long long out_stride,
                           const int *seq_start, const int *seq_past, const int *page_table, int pt_stride, int n_seqs, int max_q_len,
                           int n_heads, int n_kv, int d, int dv, int window, float scale, const float *temp, const float *bias, float cap,
                           float out_scale, int *status, cudaStream_t stream) {
  using S = SaShape<KB, VB>;
  auto kern = cap > 0.f ? sigmoid_prefill_kernel<KB, VB, true> : sigmoid_prefill_kernel<KB, VB, false>;
  LLM_CHECK_CUDA(llm_allow_smem(kern, S::SMEM), "attention_sigmoid attribute");
  dim3 grid(n_heads, n_seqs, (max_q_len + SA_BM - 1) / SA_BM);
  LLM_CHECK_CUDA(llm_launch(kern, grid, dim3(SA_THREADS), S::SMEM, stream, map_q, map_k, map_v, (__nv_bfloat16 *)out, out_stride, seq_start,
                            seq_past, page_table, pt_stride, n_heads, n_kv, d, dv, window, scale, temp, bias, cap, out_scale, status),
                 "attention_sigmoid launch");
  return LLM_OK;
}

}  // namespace

// 1 if heads of d key and dv value channels have the prompt kernel with pages of that size, else 0.
LLM_EXPORT int llm_sigmoid_prefill_supports(int d, int dv, int page_size) {
  return page_size == SA_BN && d >= 8 && d <= 128 && d % 8 == 0 && dv >= 8 && dv <= 256 && dv % 8 == 0;
}

// q [n_tokens, heads * d] bfloat16 (rotated), out [n_tokens, heads * dv], caches [n_pages, kv_heads, 64, d | dv]; sequence b owns
// rows seq_start[b] .. at positions seq_past[b] ..; temp, bias [heads]; `status` receives a code if a wait ran out of time.
LLM_EXPORT int llm_sigmoid_prefill(const void *q, long long q_stride, long long n_tokens, void *out, long long out_stride, const void *kc,
                                   const void *vc, long long n_pages, const int *seq_start, const int *seq_past, const int *page_table,
                                   int pt_stride, int n_seqs, int max_q_len, int n_heads, int n_kv, int d, int dv, int page_size, int window,
                                   float scale, const float *temp, const float *bias, float cap, float out_scale, int *status,
                                   cudaStream_t stream) {
  if (n_seqs == 0 || max_q_len == 0) return LLM_OK;
  LLM_REQUIRE(n_seqs > 0 && n_seqs <= 65535 && n_heads > 0 && n_heads <= 65535 && n_kv > 0 && n_heads % n_kv == 0,
              "sigmoid_prefill: bad sizes (%d sequences, %d heads, %d kv heads)", n_seqs, n_heads, n_kv);
  LLM_REQUIRE(max_q_len > 0 && max_q_len <= 65535 * 128, "sigmoid_prefill: %d tokens of one sequence in a step", max_q_len);
  LLM_REQUIRE(llm_sigmoid_prefill_supports(d, dv, page_size),
              "sigmoid_prefill: heads of %d / %d channels with pages of %d tokens are not built", d, dv, page_size);
  LLM_REQUIRE(q_stride % 8 == 0 && (uintptr_t)q % 16 == 0 && (uintptr_t)kc % 16 == 0 && (uintptr_t)vc % 16 == 0 && out_stride % 8 == 0 &&
                  (uintptr_t)out % 16 == 0,
              "sigmoid_prefill: rows must be 16-byte aligned");
  LLM_REQUIRE(window >= 0 && cap >= 0.f && temp && bias, "sigmoid_prefill: bad window, bound or head constants");
  LLM_REQUIRE(n_pages * n_kv * SA_BN < (1ll << 31), "sigmoid_prefill: the cache has too many rows for one tensor map");
  CUtensorMap map_q, map_k, map_v;
  int rc = get_map(q, n_tokens, (long long)n_heads * d, q_stride, 64, &map_q);
  if (rc != LLM_OK) return rc;
  rc = get_map(kc, n_pages * n_kv * SA_BN, d, d, 64, &map_k);
  if (rc != LLM_OK) return rc;
  rc = get_map(vc, n_pages * n_kv * SA_BN, dv, dv, 64, &map_v);
  if (rc != LLM_OK) return rc;
#define SA_GO(KB, VB)                                                                                                          \
  if ((d + 63) / 64 == KB && (dv + 63) / 64 == VB)                                                                             \
    return launch_sigmoid_prefill<KB, VB>(map_q, map_k, map_v, out, out_stride, seq_start, seq_past, page_table, pt_stride, n_seqs, \
                                          max_q_len, n_heads, n_kv, d, dv, window, scale, temp, bias, cap, out_scale, status, stream);
  SA_GO(1, 1) SA_GO(1, 2) SA_GO(1, 3) SA_GO(1, 4) SA_GO(2, 1) SA_GO(2, 2) SA_GO(2, 3) SA_GO(2, 4)
#undef SA_GO
  LLM_FAIL("sigmoid_prefill: no kernel for heads of %d / %d channels", d, dv);
}

// ------------------------------------------------------------------ single tokens
constexpr int SD_WARPS = 4, SD_BN = 64;

template <int VT>                           // 16-channel groups of the value a warp owns at most
__global__ void __launch_bounds__(SD_WARPS * 32)
sigmoid_decode_kernel(const __nv_bfloat16 *__restrict__ q, long long q_stride, const __nv_bfloat16 *__restrict__ kc,
                      const __nv_bfloat16 *__restrict__ vc, const int *__restrict__ tok_pos, const int *__restrict__ page_table, int pt_stride,
                      int n_heads, int n_kv, int d, int dv, int window, float scale, const float *__restrict__ temp,
                      const float *__restrict__ bias, float cap, float out_scale, int n_splits, float *__restrict__ ws,
                      int *__restrict__ counters, __nv_bfloat16 *__restrict__ out, long long out_stride) {
  extern __shared__ __align__(16) unsigned char smem_raw[];
  const int ldk = d + 8, ldv = dv + 8;
  constexpr int LDP = SD_BN + 8;
  __nv_bfloat16 *sQ = reinterpret_cast<__nv_bfloat16 *>(smem_raw);         // [16][ldk]
  __nv_bfloat16 *sP = sQ + 16 * ldk;                                       // [2][16][LDP]
  __nv_bfloat16 *sK = sP + 2 * 16 * LDP;                                   // [2][64][ldk]
  __nv_bfloat16 *sV = sK + 2 * SD_BN * ldk;                                // [2][64][ldv]
  __shared__ int s_last;
  grid_dependents_launch();
  const int split = blockIdx.x, kvh = blockIdx.y, b = blockIdx.z;
  const int group = n_heads / n_kv;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  // positions and page tables come from the step's descriptor, complete before the step's first kernel
  const int pos = tok_pos[b], kstart = window > 0 ? max(0, pos - window + 1) : 0;
  const int page0 = kstart / SD_BN, n_pages = pos / SD_BN - page0 + 1, per = (n_pages + n_splits - 1) / n_splits;
  const int it0 = split * per, it1 = min(n_pages, it0 + per);
  const int live = (n_pages + per - 1) / per;                              // runs that hold pages
  const int *pt = page_table + (size_t)b * pt_stride + page0;
  const int kch = d / 8, vch = dv / 8;
  Weigh w[2];
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int h = g + 8 * r < group ? kvh * group + g + 8 * r : kvh * group;
    w[r] = weigh_of(scale, temp[h], cap, bias[h]);
  }
  grid_dependency_wait();
  auto load = [&](int it, int stage) {
    const size_t base = ((size_t)pt[it] * n_kv + kvh) * SD_BN;
    __nv_bfloat16 *tk = sK + stage * SD_BN * ldk, *tv = sV + stage * SD_BN * ldv;
    for (int c = tid; c < SD_BN * kch; c += SD_WARPS * 32) cp_async16(tk + (c / kch) * ldk + (c % kch) * 8, kc + base * d + (size_t)c * 8, true);
    for (int c = tid; c < SD_BN * vch; c += SD_WARPS * 32) cp_async16(tv + (c / vch) * ldv + (c % vch) * 8, vc + base * dv + (size_t)c * 8, true);
  };
  float o[VT][2][4];
#pragma unroll
  for (int i = 0; i < VT; ++i)
#pragma unroll
    for (int e = 0; e < 8; ++e) o[i][e >> 2][e & 3] = 0.f;
  if (it0 < it1) {
    for (int c = tid; c < 16 * kch; c += SD_WARPS * 32) {
      const int r = c / kch, ch = c % kch;
      cp_async16(sQ + r * ldk + ch * 8, q + (size_t)b * q_stride + (size_t)(kvh * group + (r < group ? r : 0)) * d + ch * 8, r < group);
    }
    load(it0, 0);
  }
  cp_async_commit();
  for (int it = it0; it < it1; ++it) {
    const int stage = (it - it0) & 1;
    cp_async_wait<0>();
    __syncthreads();                                 // the page has arrived; everyone is done with the page before
    if (it + 1 < it1) load(it + 1, stage ^ 1);
    cp_async_commit();
    const __nv_bfloat16 *tk = sK + stage * SD_BN * ldk, *tv = sV + stage * SD_BN * ldv;
    __nv_bfloat16 *pp = sP + stage * 16 * LDP;
    // S: 16 heads x this warp's 16 keys
    float s[2][4];
#pragma unroll
    for (int e = 0; e < 8; ++e) s[e >> 2][e & 3] = 0.f;
    for (int ks = 0; ks < d / 16; ++ks) {
      unsigned qf[4], kb[4];
      ldmatrix_x4(qf, sQ + (lane & 15) * ldk + ks * 16 + (lane >> 4) * 8);
      ldmatrix_x4(kb, tk + (warp * 16 + (lane & 7) + (lane >> 4) * 8) * ldk + ks * 16 + ((lane >> 3) & 1) * 8);
      mma16816(s[0], qf, kb[0], kb[1]);
      mma16816(s[1], qf, kb[2], kb[3]);
    }
    const int k0 = (page0 + it) * SD_BN + warp * 16;
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        float2 p = w[r].bounded ? weights_of<true>(w[r], s[n][2 * r], s[n][2 * r + 1]) : weights_of<false>(w[r], s[n][2 * r], s[n][2 * r + 1]);
        const int key = k0 + n * 8 + 2 * t;
        if (key > pos || key < kstart) p.x = 0.f;
        if (key + 1 > pos || key + 1 < kstart) p.y = 0.f;
        *reinterpret_cast<unsigned *>(pp + (g + 8 * r) * LDP + warp * 16 + n * 8 + 2 * t) = pack_bf16(p.x, p.y);
      }
    __syncthreads();
    // O: 16 heads x this warp's groups of 16 channels, over the page's keys
#pragma unroll
    for (int kk = 0; kk < SD_BN / 16; ++kk) {
      unsigned pa[4];
      ldmatrix_x4(pa, pp + (lane & 15) * LDP + kk * 16 + (lane >> 4) * 8);
#pragma unroll
      for (int i = 0; i < VT; ++i) {
        const int c16 = warp + SD_WARPS * i;
        if (c16 * 16 >= dv) continue;
        unsigned vb[4];
        ldmatrix_x4_trans(vb, tv + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * ldv + c16 * 16 + (lane >> 4) * 8);
        mma16816(o[i][0], pa, vb[0], vb[1]);
        mma16816(o[i][1], pa, vb[2], vb[3]);
      }
    }
  }
  cp_async_wait<0>();
  // every (row, pair of channels) of this thread: where its sums go
  auto each = [&](auto fn) {
#pragma unroll
    for (int i = 0; i < VT; ++i) {
      const int c16 = warp + SD_WARPS * i;
      if (c16 * 16 >= dv) continue;
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int r = 0; r < 2; ++r)
          if (g + 8 * r < group) fn(g + 8 * r, c16 * 16 + n * 8 + 2 * t, o[i][n][2 * r], o[i][n][2 * r + 1]);
    }
  };
  __nv_bfloat16 *orow = out + (size_t)b * out_stride + (size_t)kvh * group * dv;
  if (live == 1) {
    if (split == 0)
      each([&](int r, int c, float x, float y) {
        *reinterpret_cast<unsigned *>(orow + (size_t)r * dv + c) = pack_bf16(x * out_scale, y * out_scale);
      });
    return;
  }
  if (split >= live) return;
  float *mine = ws + (((size_t)b * n_kv + kvh) * n_splits + split) * (size_t)(group * dv);
  each([&](int r, int c, float x, float y) { *reinterpret_cast<float2 *>(mine + (size_t)r * dv + c) = make_float2(x, y); });
  __threadfence();
  __syncthreads();
  int *counter = counters + b * n_kv + kvh;
  if (tid == 0) s_last = atomicAdd(counter, 1) == live - 1;
  __syncthreads();
  if (!s_last) return;
  __threadfence();
  const float *all = ws + ((size_t)b * n_kv + kvh) * n_splits * (size_t)(group * dv);
  for (int i = tid * 2; i < group * dv; i += SD_WARPS * 64) {
    float2 sum = make_float2(0.f, 0.f);
    for (int s0 = 0; s0 < live; s0 += 8) {           // eight runs' loads on their way at once, added in order
      float2 v[8];
#pragma unroll
      for (int e = 0; e < 8; ++e)
        if (s0 + e < live) v[e] = __ldcg(reinterpret_cast<const float2 *>(all + (size_t)(s0 + e) * (group * dv) + i));
#pragma unroll
      for (int e = 0; e < 8; ++e)
        if (s0 + e < live) {
          sum.x += v[e].x;
          sum.y += v[e].y;
        }
    }
    *reinterpret_cast<unsigned *>(orow + i) = pack_bf16(sum.x * out_scale, sum.y * out_scale);
  }
  if (tid == 0) *counter = 0;                        // as it was found
}

static size_t sigmoid_decode_smem(int d, int dv) {
  return ((size_t)(16 + 2 * SD_BN) * (d + 8) + 2 * 16 * (SD_BN + 8) + (size_t)2 * SD_BN * (dv + 8)) * sizeof(__nv_bfloat16);
}
LLM_EXPORT int llm_sigmoid_decode_supports(int d, int dv, int group, int page_size) {
  return page_size == SD_BN && d >= 16 && d <= 256 && d % 16 == 0 && dv >= 16 && dv <= 256 && dv % 16 == 0 && group >= 1 && group <= 16;
}
// CTAs of the kernel that fit on one SM
LLM_EXPORT int llm_sigmoid_decode_ctas_per_sm(int d, int dv) {
  const int n = (int)((size_t)220 * 1024 / (sigmoid_decode_smem(d, dv) + 1024));
  return n < 1 ? 1 : n > 8 ? 8 : n;
}

// One query token per sequence, q [sequences, heads * d]; ws: sequences * heads * dv * n_splits floats and counters (sequences *
// kv_heads ints, nought, left so) when n_splits > 1.
LLM_EXPORT int llm_sigmoid_decode(const void *q, long long q_stride, void *out, long long out_stride, const void *kc, const void *vc,
                                  const int *tok_pos, const int *page_table, int pt_stride, int n_seqs, int n_heads, int n_kv, int d, int dv,
                                  int page_size, int window, float scale, const float *temp, const float *bias, float cap, float out_scale,
                                  int n_splits, float *ws, int *counters, cudaStream_t stream) {
  if (n_seqs == 0) return LLM_OK;
  LLM_REQUIRE(n_seqs > 0 && n_seqs <= 65535 && n_kv > 0 && n_kv <= 65535 && n_heads % n_kv == 0 && n_splits >= 1, "sigmoid_decode: bad sizes");
  LLM_REQUIRE(llm_sigmoid_decode_supports(d, dv, n_heads / n_kv, page_size), "sigmoid_decode: heads of %d / %d channels, %d to a kv head, are not built",
              d, dv, n_heads / n_kv);
  LLM_REQUIRE(n_splits == 1 || (ws && counters), "sigmoid_decode: several runs need scratch memory and counters");
  LLM_REQUIRE(q_stride % 8 == 0 && (uintptr_t)q % 16 == 0 && (uintptr_t)kc % 16 == 0 && (uintptr_t)vc % 16 == 0 && out_stride % 2 == 0 &&
                  (uintptr_t)out % 4 == 0 && temp && bias && cap >= 0.f && window >= 0,
              "sigmoid_decode: bad arguments");
  const size_t smem = sigmoid_decode_smem(d, dv);
#define SD_GO(VT)                                                                                                              \
  do {                                                                                                                         \
    LLM_CHECK_CUDA(llm_allow_smem(sigmoid_decode_kernel<VT>, smem), "sigmoid_decode attribute");                               \
    llm_launch(sigmoid_decode_kernel<VT>, dim3(n_splits, n_kv, n_seqs), dim3(SD_WARPS * 32), smem, stream, (const __nv_bfloat16 *)q, q_stride, \
               (const __nv_bfloat16 *)kc, (const __nv_bfloat16 *)vc, tok_pos, page_table, pt_stride, n_heads, n_kv, d, dv, window, scale, \
               temp, bias, cap, out_scale, n_splits, ws, counters, (__nv_bfloat16 *)out, out_stride);                          \
  } while (0)
  if (dv <= 64) SD_GO(1);
  else if (dv <= 128) SD_GO(2);
  else SD_GO(4);
#undef SD_GO
  LLM_CHECK_LAUNCH("sigmoid_decode");
  return LLM_OK;
}
