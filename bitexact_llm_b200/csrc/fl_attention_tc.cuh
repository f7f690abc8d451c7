// Attention over a paged cache on the tensor cores (bf16 cache, fp32 scores and softmax), one kernel for prompts and decoding.
//
// A tile is up to 128 query rows = (consecutive tokens of one sequence) x (heads of one group): all of them read the same
// cache rows, so a block of 64 rows is staged once for 128 queries. Scores Q K^T: A = Q tile [128 x W], B = the rows' keys,
// both K-major. P V: the values are staged row by row like the keys and read as an MN-major B operand (their rows are the
// contraction index), so nothing is transposed; in latent attention they are the first R entries of the staged keys
// themselves and nothing is loaded twice. A = P comes from TMEM, where
// the softmax warps leave it as bf16 in place of the scores. TMEM: two score buffers of 64 columns, then the output
// accumulator (256 columns; a wider latent is cut into value slices over blockIdx.z).
//
// Warp 0 = TMA, warp 1 = MMA, the others = softmax: a query row is shared by PARTS threads (one per warp of its TMEM lane
// quarter), 64 / PARTS of the 64 keys each; a decoding tile fills one quarter only, and a single warp per row would be bound
// by its own latency. PARTS = 4: one CTA per SM. PARTS = 2 for values of up to 128 entries: half the TMEM and half the threads,
// so that two CTAs share an SM and the scores -> softmax -> values chain of one tile runs beside the other's. The running maximum starts at the sink (denominator 1); the accumulator is rescaled only when the maximum
// grows by more than 2^8 since the last time. Few tiles (decoding): the keys of a tile are split over blockIdx.y, and a
// second kernel joins the parts.
#pragma once

#include "fl_attention.cuh"
#include "fl_gemm.cuh"

namespace bxf {

constexpr int LT_KEYS = 64, LT_MAX_STAGES = 4, LT_MAX_SPLIT = 8, LT_VCOLS = 256;
constexpr int LT_O = 2 * LT_KEYS;                        // first TMEM column of the output accumulator
constexpr float LT_LOG2E = 1.4426950408889634f;
constexpr float LT_GROWTH = 8.0f;

struct LatentTc {
  int cols, kcols, vbox;                                 // 64-entry column blocks of a staged row, of its key; first one of its value
  int stages, qrows;                                     // key stages of the ring, rows of the Q box
  int row_blocks, vsplit;                                // blockIdx.z = (group * vsplit + value slice) * row_blocks + row block
  int splits;
  float* part;                                           // splits > 1: [splits][M G H][R] accumulators, then [splits][M G H][2]
};

struct LatentShared {
  uint64_t q_full, o_done;
  uint64_t full[LT_MAX_STAGES], empty[LT_MAX_STAGES];
  uint64_t s_full[2], p_full[2], pv_done[2];
  float row_max[2][4][128], row_den[4][128];
  uint32_t tmem_base, abort_flag;
};

__device__ __forceinline__ float exp2_fast(float v) {
  float r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(v));
  return r;
}

// The PARTS warps of a lane quarter.
template <int PARTS>
__device__ __forceinline__ void quarter_barrier(int quarter) {
  asm volatile("bar.sync %0, %1;" ::"r"(1 + quarter), "n"(32 * PARTS) : "memory");
}
__host__ __device__ constexpr int lt_threads(int parts) { return 64 + 128 * parts; }

// D (+)= A[tmem] * B[smem]; A: bf16 pairs, one row per lane.
__device__ __forceinline__ void umma_bf16_ts(uint32_t d_tmem, uint32_t a_tmem, uint64_t b_desc, uint32_t idesc,
                                             uint32_t accumulate) {
  asm volatile(
      "{\n\t"
      ".reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t"
      "}\n" ::"r"(d_tmem),
      "r"(a_tmem), "l"(b_desc), "r"(idesc), "r"(accumulate)
      : "memory");
}

// MN-major operand in 128-byte-swizzled boxes of 64 entries x LT_KEYS rows: 8 contraction rows are 1024 bytes apart, the
// next 64 entries one box further on.
__device__ __forceinline__ uint64_t umma_desc_mn(uint32_t addr) {
  uint64_t d = umma_desc_sw128(addr);
  d &= ~(static_cast<uint64_t>(0x3FFF) << 16);
  return d | static_cast<uint64_t>((LT_KEYS * 128) >> 4) << 16;
}

template <int PARTS>
__global__ void __launch_bounds__(lt_threads(PARTS), PARTS == 2 ? 2 : 1)
fl_paged_attention_tc_kernel(const __grid_constant__ CUtensorMap mq, const __grid_constant__ CUtensorMap mc,
                             const PagedAttn a, const LatentTc c) {
  constexpr int TCOLS = PARTS == 2 ? 256 : 512;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* qs = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int q_box = c.qrows * 128;                       // bytes of a column block of the queries
  uint8_t* ring = qs + c.kcols * q_box;
  const int stage_bytes = c.cols * LT_KEYS * 128;
  LatentShared* sh = reinterpret_cast<LatentShared*>(ring + c.stages * stage_bytes);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

  wait_previous();

  // ---- the tile ----
  int tok0, ntok;
  i64 seq;
  if (a.tiles) {
    const int* t = a.tiles + (i64)blockIdx.x * 3;
    seq = t[0];
    tok0 = t[1];
    ntok = t[2];
  } else {
    tok0 = blockIdx.x;
    ntok = 1;
    seq = a.seq[tok0];
  }
  const int row0 = (blockIdx.z % c.row_blocks) * 128, rows = min(128, ntok * a.H - row0);
  const int slice = blockIdx.z / c.row_blocks, group = slice / c.vsplit;
  const int v0 = slice % c.vsplit * LT_VCOLS, vn = min(LT_VCOLS, a.R - v0);
  const i64 limit = (i64)a.nblk * a.bs - 1;
  const i64 p_first = min(a.pos[tok0], limit), p_last = min(a.pos[tok0 + ntok - 1], limit);
  const int b_lo = a.first_key(p_first) / LT_KEYS, b_hi = (int)(p_last / LT_KEYS) + 1;
  const int b0 = b_lo + (b_hi - b_lo) * (int)blockIdx.y / c.splits, b1 = b_lo + (b_hi - b_lo) * ((int)blockIdx.y + 1) / c.splits;
  const int nb = b1 - b0;
  if (rows <= 0) return;
  const int quarters = (rows + 31) / 32;                 // TMEM lane quarters in use

  if (threadIdx.x == 0) {
    mbar_init(&sh->q_full, 1);
    mbar_init(&sh->o_done, 1);
    for (int i = 0; i < c.stages; ++i) {
      mbar_init(&sh->full[i], 1);
      mbar_init(&sh->empty[i], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&sh->s_full[i], 1);
      mbar_init(&sh->p_full[i], PARTS * quarters);
      mbar_init(&sh->pv_done[i], 1);
    }
    sh->abort_flag = *reinterpret_cast<volatile int*>(&g_wait_timeouts) != 0;
    fence_barrier_init();
    tma_prefetch_desc(&mq);
    tma_prefetch_desc(&mc);
  }
  __syncthreads();
  if (warp == 1) {
    tmem_alloc(&sh->tmem_base, TCOLS);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  launch_next();                                         // after the TMEM allocation
  const uint32_t tmem = sh->tmem_base;
  const bool dead = sh->abort_flag != 0;
  __syncthreads();

  auto fail = [&] {
    atomicAdd(&g_wait_timeouts, 1);
    *reinterpret_cast<volatile uint32_t*>(&sh->abort_flag) = 1;
  };

  if (dead) {
  } else if (warp == 0) {
    // ---- TMA: the queries once, then the key blocks in boxes that lie in one page. The warp reads the block table for 32
    //      boxes at a time; one lane issues the copies ----
    if (nb > 0) {
      if (lane == 0) {
        mbar_arrive_expect_tx(&sh->q_full, c.kcols * q_box);
        for (int j = 0; j < c.kcols; ++j)
          tma_load_3d(qs + j * q_box, &mq, &sh->q_full, j * 64, tok0 * a.H + row0, group);
      }
      const int box = min(a.bs, LT_KEYS), boxes = LT_KEYS / box;
      int i = 0, held = 0;
      bool ok = true;
      for (; i < nb; ++i) {
        const int s = i % c.stages, round = i / c.stages;
        if (round > 0) ok = mbar_wait(&sh->empty[s], (round - 1) & 1);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        uint8_t* st = ring + s * stage_bytes;
        if (lane == 0) mbar_arrive_expect_tx(&sh->full[s], stage_bytes);
        for (int p = 0; p < boxes; ++p) {
          const int nth = i * boxes + p;                             // box of this CTA
          if ((nth & 31) == 0) {
            const int page = (b0 * LT_KEYS + (nth + lane) * box) / a.bs;
            held = (int)a.page_of(seq, min(page, a.nblk - 1)) * a.G + group;
          }
          const int page = __shfl_sync(0xffffffffu, held, nth & 31);
          if (lane == 0)
            for (int j = 0; j < c.cols; ++j)
              tma_load_3d(st + j * LT_KEYS * 128 + p * box * 128, &mc, &sh->full[s],
                          j < c.kcols ? j * 64 : a.voff + (j - c.kcols) * 64, (b0 * LT_KEYS + nth * box) % a.bs, page);
        }
      }
      if (!ok && lane == 0) {
        fail();
        mbar_wait(&sh->q_full, 0);
        for (int k = i > c.stages ? i - c.stages : 0; k < i; ++k) mbar_wait(&sh->full[k % c.stages], (k / c.stages) & 1);
      }
    }
  } else if (warp == 1) {
    if (lane == 0 && nb > 0) {
      // ---- MMA: scores of block i + 1 are issued before the values of block i. A query box of fewer than 128 rows is
      //      read on into what follows it in shared memory: those accumulator lanes belong to no query ----
      constexpr uint32_t ID_S = umma_idesc_bf16(LT_KEYS);
      const uint32_t id_v = umma_idesc_bf16((vn + 15) / 16 * 16, true);
      auto scores = [&](int i) {
        const int s = i % c.stages, buf = i & 1;
        if (!mbar_wait(&sh->full[s], (i / c.stages) & 1)) return false;
        if (i >= 2 && !mbar_wait(&sh->pv_done[buf], ((i >> 1) - 1) & 1)) return false;   // P of block i - 2 is read
        tc_fence_after();
        const uint32_t qa = smem_u32(qs), ka = smem_u32(ring + s * stage_bytes);
        for (int j = 0; j < c.kcols; ++j)
#pragma unroll
          for (int ks = 0; ks < 4; ++ks)
            umma_bf16(tmem + buf * LT_KEYS, umma_desc_sw128(qa + j * q_box + ks * 32),
                      umma_desc_sw128(ka + j * LT_KEYS * 128 + ks * 32), ID_S, (j | ks) != 0);
        umma_commit(&sh->s_full[buf]);
        return true;
      };
      bool ok = mbar_wait(&sh->q_full, 0) && scores(0);
      for (int i = 0; i < nb && ok; ++i) {
        const int s = i % c.stages, buf = i & 1;
        if (c.stages > 1 && i + 1 < nb && !(ok = scores(i + 1))) break;
        if (!(ok = mbar_wait(&sh->p_full[buf], (i >> 1) & 1))) break;
        tc_fence_after();
        const uint32_t va = smem_u32(ring + s * stage_bytes) + (c.vbox + v0 / 64) * LT_KEYS * 128;
#pragma unroll
        for (int ks = 0; ks < LT_KEYS / 16; ++ks)
          umma_bf16_ts(tmem + LT_O, tmem + buf * LT_KEYS + ks * 8, umma_desc_mn(va + ks * 2048), id_v, (i | ks) != 0);
        umma_commit(&sh->pv_done[buf]);
        umma_commit(&sh->empty[s]);
        if (c.stages == 1 && i + 1 < nb) ok = scores(i + 1);             // one stage: nothing to run ahead into
      }
      if (ok) umma_commit(&sh->o_done);
      else fail();
    }
  } else if ((warp & 3) < quarters) {
    // ---- softmax. A wait that gives up is remembered and the loop goes on (the quarter's barriers count every warp) ----
    constexpr int KW = LT_KEYS / PARTS;
    const int quarter = warp & 3, part = (warp - 2) >> 2, r = quarter * 32 + lane;
    const bool live = r < rows;
    const int flat = row0 + (live ? r : 0), token = tok0 + flat / a.H, head = group * a.H + flat % a.H;
    const i64 pos = min(a.pos[token], limit);
    const int lo = a.first_key(pos), hi = (int)pos;
    const float scale = a.scale * LT_LOG2E;
    float ref = a.sink ? a.sink[head] * LT_LOG2E : -INFINITY;
    float den = a.sink && blockIdx.y == 0 && part == 0 ? 1.0f : 0.0f;
    const uint32_t lanes = (uint32_t)(quarter * 32) << 16;
    bool ok = true;
    for (int i = 0; i < nb; ++i) {
      const int buf = i & 1;
      ok = ok && mbar_wait(&sh->s_full[buf], (i >> 1) & 1);
      __syncwarp();
      tc_fence_after();
      uint32_t u[KW];
#pragma unroll
      for (int k = 0; k < KW; k += 16) tmem_ld16(tmem + lanes + buf * LT_KEYS + part * KW + k, *reinterpret_cast<uint32_t(*)[16]>(u + k));
      tmem_ld_wait();
      const int k0 = (b0 + i) * LT_KEYS + part * KW;
      float s[KW], mx = -INFINITY;
      if (k0 >= lo && k0 + KW - 1 <= hi) {
#pragma unroll
        for (int k = 0; k < KW; ++k) {
          s[k] = __uint_as_float(u[k]) * scale;
          mx = fmaxf(mx, s[k]);
        }
      } else {
#pragma unroll
        for (int k = 0; k < KW; ++k) {
          s[k] = k0 + k >= lo && k0 + k <= hi ? __uint_as_float(u[k]) * scale : -INFINITY;
          mx = fmaxf(mx, s[k]);
        }
      }
      sh->row_max[buf][part][r] = mx;
      tc_fence_before();
      quarter_barrier<PARTS>(quarter);                     // the quarter's scores are in registers: P may replace them
      tc_fence_after();
#pragma unroll
      for (int k = 0; k < PARTS; ++k) mx = fmaxf(mx, sh->row_max[buf][k][r]);
      float f = 1.0f;
      if (mx > ref + LT_GROWTH || ref == -INFINITY) {
        f = ref == -INFINITY ? 0.0f : exp2_fast(ref - mx);
        ref = mx;
      }
      if (__any_sync(0xffffffffu, f != 1.0f && live)) {    // the same in the four warps of the quarter
        den *= f;
        if (i > 0) {
          // the accumulator may be touched once the values of block i - 1 are in
          ok = ok && mbar_wait(&sh->pv_done[buf ^ 1], ((i - 1) >> 1) & 1);
          __syncwarp();
          tc_fence_after();
          for (int q = part * 16; q < vn; q += 16 * PARTS) {
            uint32_t o[16];
            tmem_ld16(tmem + lanes + LT_O + q, o);
            tmem_ld_wait();
#pragma unroll
            for (int k = 0; k < 16; ++k) o[k] = __float_as_uint(__uint_as_float(o[k]) * f);
            tmem_st16(tmem + lanes + LT_O + q, o);
          }
        }
      }
      const float base = ref == -INFINITY ? 0.0f : ref;    // no visible key yet: every weight is 0
      float d0 = 0.0f, d1 = 0.0f;
      uint32_t w[KW / 2];
#pragma unroll
      for (int k = 0; k < KW / 2; ++k) {
        const float e0 = exp2_fast(s[2 * k] - base), e1 = exp2_fast(s[2 * k + 1] - base);
        d0 += e0;
        d1 += e1;
        w[k] = pack_bf16(e0, e1);
      }
      den += d0 + d1;
#pragma unroll
      for (int k = 0; k < KW / 2; k += 8)
        tmem_st8(tmem + lanes + buf * LT_KEYS + part * (KW / 2) + k, *reinterpret_cast<const uint32_t(*)[8]>(w + k));
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&sh->p_full[buf]);
    }
    if (nb > 0) ok = ok && mbar_wait(&sh->o_done, 0);
    ok = __all_sync(0xffffffffu, ok);
    sh->row_den[part][r] = den;
    quarter_barrier<PARTS>(quarter);
    den = 0.0f;
#pragma unroll
    for (int k = 0; k < PARTS; ++k) den += sh->row_den[k][r];
    if (!ok) {
      if (lane == 0) fail();
    } else {
      tc_fence_after();
      const i64 n = (i64)a.M * a.H * a.G, at = (i64)token * a.H * a.G + head;
      const float inv = 1.0f / den;
      float* acc = c.part + (blockIdx.y * n + at) * a.R + v0;
      bf16* out = static_cast<bf16*>(a.out) + token * a.out_tok + head * a.out_head + v0;
      for (int q = part * 16; q < vn; q += 16 * PARTS) {
        uint32_t u[16] = {};
        if (nb > 0) {
          tmem_ld16(tmem + lanes + LT_O + q, u);
          tmem_ld_wait();
        }
        if (!live) continue;
        const int cnt = min(16, vn - q);
        float v[16];
#pragma unroll
        for (int k = 0; k < 16; ++k) v[k] = __uint_as_float(u[k]) * (c.splits == 1 ? inv : 1.0f);
        if (c.splits == 1) store_run(out + q, v, cnt);
        else store_run(acc + q, v, cnt);
      }
      if (c.splits > 1 && live && v0 == 0 && part == 0) {
        float* ml = c.part + c.splits * n * a.R + (blockIdx.y * n + at) * 2;
        ml[0] = ref;
        ml[1] = den;
      }
    }
  }

  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    __syncwarp();
    tc_fence_after();
    tmem_dealloc(tmem, TCOLS);
  }
}

// Joins the key splits: one CTA per query row (token, head).
__global__ void __launch_bounds__(128) fl_attention_join_kernel(const PagedAttn a, const float* part, int splits) {
  launch_next();
  wait_previous();
  const i64 at = blockIdx.x, heads = a.H * a.G, n = a.M * heads;
  const float* ml = part + splits * n * a.R;
  float mx = -INFINITY, f[LT_MAX_SPLIT], den = 0.0f;
  for (int s = 0; s < splits; ++s)
    if (ml[(s * n + at) * 2 + 1] > 0.0f) mx = fmaxf(mx, ml[(s * n + at) * 2]);
#pragma unroll
  for (int s = 0; s < LT_MAX_SPLIT; ++s) {
    f[s] = s < splits && ml[(s * n + at) * 2 + 1] > 0.0f ? exp2f(ml[(s * n + at) * 2] - mx) : 0.0f;
    if (f[s] > 0.0f) den += f[s] * ml[(s * n + at) * 2 + 1];
  }
  const float inv = 1.0f / den;
  bf16* out = static_cast<bf16*>(a.out) + at / heads * a.out_tok + at % heads * a.out_head;
  for (int d = threadIdx.x; d < a.R; d += 128) {
    float o = 0.0f;
#pragma unroll
    for (int s = 0; s < LT_MAX_SPLIT; ++s)
      if (f[s] > 0.0f) o += f[s] * part[(s * n + at) * a.R + d];
    st(out + d, o * inv);
  }
}

}  // namespace bxf
