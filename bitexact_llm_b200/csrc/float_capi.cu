// C ABI of libbitexact_float.so (declared in include/bitexact_float.h): argument contracts, tensor maps, tile choice and
// launches of the float-model kernels. One translation unit, so the device status word is shared by every kernel.
#include <cuda.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "../../include/bitexact_float.h"
#include "host_util.cuh"
#include "fl_attention.cuh"
#include "fl_attention_tc.cuh"
#include "fl_gemm.cuh"
#include "fl_gemm_simt.cuh"
#include "fl_recurrence_chunks.cuh"
#include "fl_stages.cuh"
#include "fl_streams.cuh"

namespace {

using namespace bxf;

static_assert(sizeof(bxf_epilogue) == 136 && sizeof(bxf_gru) == 56 && sizeof(bxf_streams_step) == 112 &&
                  sizeof(bxf_gqa_rows) == 120 && sizeof(bxf_conv) == 72 && sizeof(bxf_recurrence_rows) == 160 &&
                  sizeof(bxf_gate_rows) == 152 && sizeof(bxf_chunk_table) == 48,
              "layouts of the callers' structs");

inline cudaStream_t stream_of(void* s) { return static_cast<cudaStream_t>(s); }
inline bool dtype_ok(int d) { return d == BXF_BF16 || d == BXF_F32; }
inline int ceil_div(int a, int b) { return (a + b - 1) / b; }

// bf16 [planes, rows, K] (leading dimension ld, plane stride gs) -> 3-D map, box (64 elements, box_rows, box_planes),
// 128-byte swizzle; everything outside the extents reads as zero.
bool make_map_bf16(CUtensorMap* m, const void* base, i64 K, i64 rows, i64 planes, i64 ld, i64 gs, uint32_t box_rows,
                   uint32_t box_planes) {
  EncodeTiledFn fn = encode_fn();
  if (!fn) return false;
  cuuint64_t dims[3] = {(cuuint64_t)K, (cuuint64_t)rows, (cuuint64_t)planes};
  cuuint64_t strides[2] = {(cuuint64_t)ld * 2, (cuuint64_t)(planes > 1 ? gs : rows * ld) * 2};
  cuuint32_t box[3] = {64, box_rows, box_planes};
  cuuint32_t estr[3] = {1, 1, 1};
  return fn(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, estr,
            CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
            CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

// Launch with the permission to start before the previous kernel of the stream has ended (every kernel launched this way
// calls wait_previous before it touches dependent memory).
template <class... P, class... A>
int launch_chained(void (*kernel)(P...), dim3 grid, int threads, int smem, cudaStream_t st, int cluster, A&&... args) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = dim3(threads, 1, 1);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = st;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  attr[1].id = cudaLaunchAttributeClusterDimension;
  attr[1].val.clusterDim.x = cluster;
  attr[1].val.clusterDim.y = 1;
  attr[1].val.clusterDim.z = 1;
  cfg.attrs = attr;
  cfg.numAttrs = cluster > 0 ? 2 : 1;
  if (cudaLaunchKernelEx(&cfg, kernel, static_cast<P>(args)...) != cudaSuccess) return BX_ELAUNCH;
  return launched(1);
}

struct Operands {
  const void *w, *x;
  i64 ldw, gsw, ldx, gsx;
};

template <class Epi>
int launch_simt(const Operands& o, GemmShape s, const typename Epi::Params& ep, cudaStream_t st) {
  constexpr int stash = Epi::stash_bytes(SIMT_TA);
  static PerDevice configured;
  if (once_per_device(configured, [] {
        return cudaFuncSetAttribute(fl_gemm_simt_kernel<Epi>, cudaFuncAttributeMaxDynamicSharedMemorySize, stash);
      }) != BX_OK)
    return BX_ELAUNCH;
  s.n_tiles = ceil_div(s.N, NROWS);
  s.m_tiles = s.counts ? s.M / SIMT_TA + (s.groups < s.M ? s.groups : s.M) : ceil_div(s.M, SIMT_TA);
  const i64 grid = (i64)s.n_tiles * s.m_tiles * (s.counts || Epi::PLANES > 1 ? 1 : s.groups);
  fl_gemm_simt_kernel<Epi><<<(unsigned)grid, EPI_THREADS, stash, st>>>(
      static_cast<const float*>(o.w), o.ldw, o.gsw, static_cast<const float*>(o.x), o.ldx, o.gsx, s, ep);
  return launched(1);
}

// Token tiles of `rows` rows: exact for dense lists, an upper bound for ragged ones (the sizes are on the device).
int token_tiles(const GemmShape& s, int rows) {
  return s.counts ? s.M / rows + (s.groups < s.M ? s.groups : s.M) : ceil_div(s.M, rows);
}

// ---- which kernel and tile: the estimated cycles of the slowest SM ----
struct Plan {
  int tile;                    // token rows (16, 32, 64: fl_gemm_kernel) or weight rows (128, 256: persistent kernel)
  int split;                   // CTAs that share K
  double cycles;
};

// Expected token tiles; experts' sizes vary, so their tiles are counted at 1.3 times the mean size.
double expected_tiles(const GemmShape& s, int rows) {
  if (!s.counts) return ceil_div(s.M, rows);
  const int used = s.groups < s.M ? s.groups : s.M;
  return (double)used * ceil_div((int)(1.3 * s.M / used + 0.5), rows);
}

// Clusters of `split` CTAs of the tile kernels that the device holds at a time (a cluster lies within one group of SMs, so
// fewer than SMs / split), cached per device.
int resident_clusters(int split, int sms);

// A K block of a tile of R + C rows moves (R + C) x 128 bytes into shared memory and reads them once for the MMAs, at 128
// bytes a cycle; the constants are the measured prologue, epilogue and cluster exchange.
Plan tile_plan(const GemmShape& s, int planes, int ta, int max_split, int sms) {
  const double tiles = expected_tiles(s, ta) * ceil_div(s.N, NROWS) * (s.counts || planes > 1 ? 1 : s.groups);
  const int nkb = ceil_div(s.K, KE);
  Plan best = {ta, 1, 1e300};
  for (int split = 1; split <= max_split && (split == 1 || nkb >= 2 * split); split *= 2) {
    const int slots = split == 1 ? sms : resident_clusters(split, sms);
    const double waves = (double)(i64)((tiles + slots - 1) / slots);
    const double per = ceil_div(nkb, split) * 2.3 * (planes * NROWS + ta) + 3000 + 20.0 * planes * ta + (split > 1 ? 1800 : 0);
    if (waves * per < best.cycles) best = {ta, split, waves * per};
  }
  return best;
}

Plan persistent_plan(const GemmShape& s, int tn, int sms) {
  const double tiles = expected_tiles(s, NROWS) * ceil_div(s.N, tn) * (s.counts ? 1 : s.groups);
  const double waves = (double)(i64)((tiles + sms - 1) / sms);
  const double loop = ceil_div(s.K, KE) * 2.3 * (NROWS + tn), epilogue = 25.0 * tn;
  return {tn, 1, waves * (loop > epilogue ? loop : epilogue) + 3000 + epilogue};
}

Plan plan_linear(const GemmShape& s, int sms) {
  Plan best = tile_plan(s, 1, 16, FL_SPLIT_MAX, sms);
  const auto consider = [&](const Plan& p) {
    if (p.cycles < best.cycles) best = p;
  };
  consider(tile_plan(s, 1, 32, FL_SPLIT_MAX, sms));
  consider(tile_plan(s, 1, 64, FL_SPLIT_MAX, sms));
  consider(persistent_plan(s, 128, sms));
  consider(persistent_plan(s, 256, sms));
  return best;
}

int resident_clusters(int split, int sms) {
  static PerDevice cache[2];
  const int dev = current_device();
  if (dev < 0) return sms / split;
  std::atomic<int>& slot = cache[split == 2 ? 0 : 1].v[dev];
  int n = slot.load(std::memory_order_acquire);
  if (n > 0) return n;
  using Cfg = FlCfg<3, 64>;                              // one CTA per SM
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(4 * 148, 1, 1);
  cfg.blockDim = dim3(64 + 32 * GruEpi::warps(64), 1, 1);
  cfg.dynamicSmemBytes = Cfg::SMEM_BYTES;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = split;
  attr[0].val.clusterDim.y = 1;
  attr[0].val.clusterDim.z = 1;
  cfg.attrs = attr;
  cfg.numAttrs = 1;
  if (cudaFuncSetAttribute(fl_gemm_kernel<64, GruEpi>, cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg::SMEM_BYTES) !=
          cudaSuccess ||
      cudaOccupancyMaxActiveClusters(&n, fl_gemm_kernel<64, GruEpi>, &cfg) != cudaSuccess || n <= 0) {
    cudaGetLastError();
    return sms / split;
  }
  slot.store(n, std::memory_order_release);
  return n;
}

// One tile per cluster of `split` CTAs.
template <int TA, class Epi>
int launch_tiles(const Operands& o, GemmShape s, const typename Epi::Params& ep, int split, cudaStream_t st) {
  constexpr int NP = Epi::PLANES;
  using Cfg = FlCfg<NP, TA, Epi::ctas(TA)>;
  static PerDevice configured;
  if (once_per_device(configured, [] {
        return cudaFuncSetAttribute(fl_gemm_kernel<TA, Epi>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                    Cfg::SMEM_BYTES);
      }) != BX_OK)
    return BX_ELAUNCH;
  s.n_tiles = ceil_div(s.N, NROWS);
  s.m_tiles = token_tiles(s, TA);
  CUtensorMap mw, mx;
  if (!make_map_bf16(&mw, o.w, s.K, s.N, NP > 1 ? NP : s.groups, o.ldw, o.gsw, NROWS, NP) ||
      !make_map_bf16(&mx, o.x, s.K, s.M, NP > 1 || s.counts ? 1 : s.groups, o.ldx, o.gsx, TA, 1))
    return BX_ELAUNCH;
  const i64 tiles = (i64)s.n_tiles * s.m_tiles * (s.counts || NP > 1 ? 1 : s.groups);
  if (tiles > (1 << 24)) return BX_ELIMIT;
  if (Cfg::PARTIAL_BYTES + Epi::stash_bytes(TA) > Cfg::RING_BYTES) split = 1;
  return launch_chained(fl_gemm_kernel<TA, Epi>, dim3((unsigned)(tiles * split)), 64 + 32 * Epi::warps(TA), Cfg::SMEM_BYTES,
                        st, split, mw, mx, s, ep);
}

template <int TN, class Epi>
int launch_persistent(const Operands& o, GemmShape s, const typename Epi::Params& ep, int sms, cudaStream_t st) {
  using Cfg = FlCfg<1, TN>;
  static PerDevice configured;
  if (once_per_device(configured, [] {
        return cudaFuncSetAttribute(fl_gemm_persistent_kernel<TN, Epi>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                    Cfg::SMEM_BYTES);
      }) != BX_OK)
    return BX_ELAUNCH;
  s.n_tiles = ceil_div(s.N, TN);
  s.m_tiles = token_tiles(s, NROWS);
  CUtensorMap mw, mx;
  if (!make_map_bf16(&mw, o.w, s.K, s.N, s.groups, o.ldw, o.gsw, TN, 1) ||
      !make_map_bf16(&mx, o.x, s.K, s.M, s.counts ? 1 : s.groups, o.ldx, o.gsx, NROWS, 1))
    return BX_ELAUNCH;
  const i64 tiles = (i64)s.n_tiles * s.m_tiles * (s.counts ? 1 : s.groups);
  if (tiles > (1 << 24)) return BX_ELIMIT;
  return launch_chained(fl_gemm_persistent_kernel<TN, Epi>, dim3((unsigned)(tiles < sms ? tiles : sms)), GEMM_THREADS,
                        Cfg::SMEM_BYTES, st, 0, mw, mx, s, ep);
}

bool operand_ok(const void* p, i64 ld, i64 gs, bool grouped, int K, int dtype) {
  if (!p || ld < K) return false;
  return dtype == BXF_F32 || (aligned16(p) && ld % 8 == 0 && (!grouped || gs % 8 == 0));
}

int run_bf16(const Operands& o, const GemmShape& s, const bxf_epilogue& ep, int tile, cudaStream_t st) {
  const int sms = device_sms();
  if (sms <= 0) return BX_ELAUNCH;
  Plan p = {tile, 1, 0};
  if (tile == 0) p = plan_linear(s, sms);
  else if (tile <= 64) p = tile_plan(s, 1, tile, FL_SPLIT_MAX, sms);
  switch (p.tile) {
    case 16: return launch_tiles<16, StageEpi>(o, s, ep, p.split, st);
    case 32: return launch_tiles<32, StageEpi>(o, s, ep, p.split, st);
    case 64: return launch_tiles<64, StageEpi>(o, s, ep, p.split, st);
    case 128: return launch_persistent<128, StageEpi>(o, s, ep, sms, st);
    case 256: return launch_persistent<256, StageEpi>(o, s, ep, sms, st);
    default: return BX_EARG;
  }
}

// The tensor-core attention kernel takes pages of 8, 16, .. keys, rows of at most 9 column blocks (shared memory).
bool paged_tc_fits(int dtype, const PagedAttn& a) {
  const int cols = ceil_div(a.W, 64) + (a.voff > 0 ? ceil_div(a.R, 64) : 0);
  return dtype == BXF_BF16 && a.bs >= 8 && (a.bs & (a.bs - 1)) == 0 && cols <= 9 && aligned16(a.q) && aligned16(a.cache) &&
         a.ldq % 8 == 0 && a.ldc % 8 == 0 && a.voff % 8 == 0;
}

// Two CTAs per SM: values in half of the TMEM columns, two key stages in half of the shared memory.
constexpr int LT_PAIR_SMEM = 113 * 1024;

bool paged_pair_fits(const PagedAttn& a) {
  const int kcols = ceil_div(a.W, 64), cols = kcols + (a.voff > 0 ? ceil_div(a.R, 64) : 0);
  const int rows = (a.tiles ? bxf_latent_attention_tile(a.H) : 1) * a.H, qrows = rows >= 128 ? 128 : ceil_div(rows, 8) * 8;
  return a.R <= 128 && 1024 + kcols * qrows * 128 + (int)sizeof(LatentShared) + 2 * cols * LT_KEYS * 128 <= LT_PAIR_SMEM;
}

size_t attention_scratch(i64 rows, int R, int splits) { return (size_t)splits * rows * (R + 2) * sizeof(float); }

// Key splits only happen while the query tiles leave SMs idle (148 of them).
size_t attention_scratch_for(int M, int groups, int heads, int R) {
  if (M < 1 || groups < 1 || heads < 1 || R < 1 || (i64)M * groups > 148) return 0;
  const int free = 148 / (M * groups), splits = free < 2 ? 2 : free > LT_MAX_SPLIT ? LT_MAX_SPLIT : free;
  return attention_scratch((i64)M * groups * heads, R, splits);
}

template <int PARTS>
int launch_paged_tc(const PagedAttn& a, void* scratch, size_t scratch_bytes, cudaStream_t st) {
  constexpr int SMEM_MAX = PARTS == 2 ? LT_PAIR_SMEM : 227 * 1024;
  static PerDevice configured;
  if (once_per_device(configured, [] {
        return cudaFuncSetAttribute(fl_paged_attention_tc_kernel<PARTS>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM_MAX);
      }) != BX_OK)
    return BX_ELAUNCH;
  LatentTc c = {};
  c.kcols = ceil_div(a.W, 64);
  c.vbox = a.voff > 0 ? c.kcols : 0;
  c.cols = c.kcols + (a.voff > 0 ? ceil_div(a.R, 64) : 0);
  const int tokens = a.tiles ? bxf_latent_attention_tile(a.H) : 1, tiles = a.tiles ? a.ntiles : a.M;
  const int rows = tokens * a.H;
  c.qrows = rows >= 128 ? 128 : ceil_div(rows, 8) * 8;
  const int fixed = 1024 + c.kcols * c.qrows * 128 + (int)sizeof(LatentShared);
  c.stages = (SMEM_MAX - fixed) / (c.cols * LT_KEYS * 128);
  if (c.stages > LT_MAX_STAGES) c.stages = LT_MAX_STAGES;
  c.row_blocks = ceil_div(rows, 128);
  c.vsplit = ceil_div(a.R, LT_VCOLS);
  c.splits = 1;
  const i64 span = a.window > 0 && a.window + tokens < (i64)a.nblk * a.bs ? a.window + tokens : (i64)a.nblk * a.bs;
  const i64 blocks = span / LT_KEYS + 1, ctas = (i64)tiles * c.row_blocks * c.vsplit * a.G;
  if ((i64)c.row_blocks * c.vsplit * a.G > 65535) return BX_ELIMIT;
  const int sms = device_sms();
  if (sms <= 0) return BX_ELAUNCH;
  while (c.splits < LT_MAX_SPLIT && ctas * c.splits * 2 <= sms && blocks >= c.splits * 4 && scratch &&
         scratch_bytes >= attention_scratch((i64)a.M * a.H * a.G, a.R, c.splits * 2))
    c.splits *= 2;
  c.part = static_cast<float*>(scratch);
  CUtensorMap mq, mc;
  if (!make_map_bf16(&mq, a.q, a.W, (i64)a.M * a.H, a.G, a.ldq, (i64)a.M * a.H * a.ldq, c.qrows, 1) ||
      !make_map_bf16(&mc, a.cache, a.voff > 0 ? a.voff + a.R : a.W, a.bs, (i64)a.nb * a.G, a.ldc, (i64)a.bs * a.ldc,
                     a.bs < LT_KEYS ? a.bs : LT_KEYS, 1))
    return BX_ELAUNCH;
  const dim3 grid(tiles, c.splits, c.row_blocks * c.vsplit * a.G);
  const int rc = launch_chained(fl_paged_attention_tc_kernel<PARTS>, grid, lt_threads(PARTS), fixed + c.stages * c.cols * LT_KEYS * 128, st,
                                0, mq, mc, a, c);
  if (rc != BX_OK || c.splits == 1) return rc;
  return launch_chained(fl_attention_join_kernel, dim3((unsigned)(a.M * a.H * a.G)), 128, 0, st, 0, a, c.part, c.splits);
}

int run_attention(int dtype, const PagedAttn& a, void* scratch, size_t scratch_bytes, int variant, cudaStream_t st) {
  if (a.R > LA_MAX_R || a.W > 8192 || (i64)a.H * a.G > 65535) return BX_ELIMIT;
  if (g_status_seen.load() != 0) return BX_EDEVICE;
  if (a.M == 0) return BX_OK;
  if (variant == 2 && !paged_tc_fits(dtype, a)) return BX_ELIMIT;
  if (variant != 1 && paged_tc_fits(dtype, a) && (!a.tiles || a.ntiles > 0))
    return paged_pair_fits(a) ? launch_paged_tc<2>(a, scratch, scratch_bytes, st) : launch_paged_tc<4>(a, scratch, scratch_bytes, st);
  const dim3 grid(a.M, a.H * a.G);
  if (dtype == BXF_F32) fl_paged_attention_kernel<float><<<grid, LA_THREADS, a.W * 4, st>>>(a);
  else fl_paged_attention_kernel<bf16><<<grid, LA_THREADS, a.W * 4, st>>>(a);
  return launched(1);
}

bool gru_ok(const bxf_gru* g, int M, int width) {
  return g && M >= 0 && width >= 1 && g->bias_z && g->bias_x && g->state && g->flags && g->seq && g->out && g->ldo >= width;
}

template <class T>
int launch_streams(const bxf_streams_step& p, int M, bool vec, cudaStream_t st) {
  const int S = p.streams;
  auto* kernel = S <= 2 ? (vec ? fl_streams_kernel<T, 2, 4> : fl_streams_kernel<T, 2, 1>)
               : S <= 4 ? (vec ? fl_streams_kernel<T, 4, 4> : fl_streams_kernel<T, 4, 1>)
                        : (vec ? fl_streams_kernel<T, BXF_MAX_STREAMS, 4> : fl_streams_kernel<T, BXF_MAX_STREAMS, 1>);
  const int smem = p.h ? p.D * 4 : 0;
  if (smem > 40 * 1024 && cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess)
    return BX_ELAUNCH;
  return launch_chained(kernel, dim3(M), NORM_THREADS, smem, st, 0, p);
}

bool conv_ok(const bxf_conv* c) {
  return c && c->u && c->w && c->b && c->state && c->flags && c->seq && c->pos && c->channels >= 1 && c->taps >= 1 &&
         c->taps <= BXF_MAX_TAPS && c->ldu >= c->channels;
}

bool recurrence_ok(const bxf_recurrence_rows* p) {
  if (!p || !p->y || !p->side || !p->state || !p->flags || !p->seq || !p->out || p->heads < 1 || p->groups < 1 ||
      p->heads % p->groups || p->K < 1 || p->V < 1 || p->ldo < (i64)p->heads * p->V)
    return false;
  if (p->kind == BXF_DECAY_CHANNEL) return p->rank >= 1 && p->a2 && p->a2_b && p->groups == p->heads;
  return p->kind == BXF_DECAY_HEAD && p->A_log && p->skip;
}

template <class T, bool CHANNEL, int CW, int KR, int ROWS>
int launch_recurrence_rows(const bxf_recurrence_rows& p, int M, cudaStream_t st) {
  const int smem = recurrence_smem(p.K, CW, CHANNEL, ROWS);
  static PerDevice configured;
  if (once_per_device(configured, [] {
        return cudaFuncSetAttribute(fl_recurrence_kernel<T, CHANNEL, CW, KR, ROWS>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                    recurrence_smem(REC_THREADS / CW * KR, CW, CHANNEL, ROWS));
      }) != BX_OK)
    return BX_ELAUNCH;
  return launch_chained(fl_recurrence_kernel<T, CHANNEL, CW, KR, ROWS>, dim3(M, p.heads, ceil_div(p.V, 4 * CW)), REC_THREADS,
                        smem, st, 0, p, M);
}

template <class T, bool CHANNEL, int CW, int KR>
int launch_recurrence_as(const bxf_recurrence_rows& p, int M, cudaStream_t st) {
  if (std::is_same<T, bf16>::value && p.batch == 1) return launch_recurrence_rows<T, CHANNEL, CW, KR, 1>(p, M, st);
  return launch_recurrence_rows<T, CHANNEL, CW, KR, REC_ROWS>(p, M, st);
}

template <class T>
int launch_recurrence(const bxf_recurrence_rows& p, int M, cudaStream_t st) {
  auto go = [&](auto channel) {
    constexpr bool C = decltype(channel)::value;
    if (p.V >= 64 && p.K <= 128 && (i64)M * p.heads * ceil_div(p.V, 64) >= 4 * 148)
      return p.K <= 64 ? launch_recurrence_as<T, C, 16, 4>(p, M, st) : launch_recurrence_as<T, C, 16, 8>(p, M, st);
    const int kr = ceil_div(p.K, 32);
    if (kr <= 1) return launch_recurrence_as<T, C, 8, 1>(p, M, st);
    if (kr <= 2) return launch_recurrence_as<T, C, 8, 2>(p, M, st);
    if (kr <= 4) return launch_recurrence_as<T, C, 8, 4>(p, M, st);
    if (kr <= 8) return launch_recurrence_as<T, C, 8, 8>(p, M, st);
    return launch_recurrence_as<T, C, 8, 16>(p, M, st);
  };
  return p.kind == BXF_DECAY_CHANNEL ? go(std::true_type{}) : go(std::false_type{});
}

// The chunk kernel takes bf16 rows whose key and value sizes are multiples of 8.
bool chunks_fit(int dtype, int K, int V) { return dtype == BXF_BF16 && K % 8 == 0 && V % 8 == 0 && K <= RC_MAX_K; }

struct ChunkScratch {
  size_t planes, edge, masks, states, decays, bytes;     // sizes, in this order
};

ChunkScratch chunk_scratch(int kind, int M, int chunks, int segments, int heads, int K, int V) {
  const auto up = [](size_t n) { return (n + 255) / 256 * 256; };
  const size_t channel = kind == BXF_DECAY_CHANNEL ? 1 : 0;
  ChunkScratch s;
  s.planes = up(channel * 4 * M * heads * K * 2);
  s.edge = up(channel * M * heads * K * 4);
  s.masks = up(channel * chunks * heads * 8);
  s.states = up((size_t)segments * heads * K * V * 4);
  s.decays = up((size_t)segments * heads * K * 4);
  s.bytes = s.planes + s.edge + s.masks + s.states + s.decays;
  return s;
}

template <bool CHANNEL, int KT, int NW, ChunkPass PASS>
int launch_chunk_pass(const bxf_recurrence_rows& p, const ChunkArgs& a, int n, cudaStream_t st) {
  using Cfg = ChunkCfg<CHANNEL, KT, NW, PASS>;
  static PerDevice configured;
  if (once_per_device(configured, [] {
        return cudaFuncSetAttribute(fl_recurrence_chunk_kernel<CHANNEL, KT, NW, PASS>,
                                    cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg::SMEM);
      }) != BX_OK)
    return BX_ELAUNCH;
  return launch_chained(fl_recurrence_chunk_kernel<CHANNEL, KT, NW, PASS>, dim3(n, p.heads, ceil_div(p.V, Cfg::VS)), 32 * NW,
                        Cfg::SMEM, st, 0, p, a);
}

// nsegs = 0: every CTA walks a whole run.
template <bool CHANNEL, int KT>
int launch_chunks_as(const bxf_recurrence_rows& p, ChunkArgs a, int nruns, const int* segs, int nsegs, const int* spans,
                     cudaStream_t st) {
  if (nsegs == 0) return launch_chunk_pass<CHANNEL, KT, 4, WHOLE_RUN>(p, a, nruns, st);
  a.runs = segs;
  int rc = launch_chunk_pass<CHANNEL, KT, 4, CONTRIBUTION>(p, a, nsegs, st);
  if (rc != BX_OK) return rc;
  rc = launch_chained(fl_recurrence_chain_kernel, dim3(nruns, p.heads, ceil_div(p.K * p.V, 1024)), 256, 0, st, 0, p, spans, a.states,
                      a.decays);
  return rc != BX_OK ? rc : launch_chunk_pass<CHANNEL, KT, 4, OUTPUTS>(p, a, nsegs, st);
}

template <bool CHANNEL>
int launch_chunks(const bxf_recurrence_rows& p, const ChunkArgs& a, int nruns, const int* segs, int nsegs, const int* spans,
                  cudaStream_t st) {
  const int kt = ceil_div(p.K, 16);
  if (kt <= 2) return launch_chunks_as<CHANNEL, 2>(p, a, nruns, segs, nsegs, spans, st);
  if (kt <= 4) return launch_chunks_as<CHANNEL, 4>(p, a, nruns, segs, nsegs, spans, st);
  if (kt <= 8) return launch_chunks_as<CHANNEL, 8>(p, a, nruns, segs, nsegs, spans, st);
  return launch_chunks_as<CHANNEL, 16>(p, a, nruns, segs, nsegs, spans, st);
}

template <class T>
int launch_gated_norm(const bxf_gate_rows& p, int M, cudaStream_t st) {
  const int size = p.n / p.parts;
  const bool vec = size % 8 == 0 && p.wn % 8 == 0 && p.ldo % 8 == 0 && p.ldz % 8 == 0 && p.ldout % 8 == 0 && aligned16(p.o) &&
                   aligned16(p.z) && aligned16(p.out) && aligned16(p.w);
  const bool warp = size <= 512;                         // a warp per part, or a CTA
  const int part_ctas = warp ? ceil_div(p.parts, GATE_THREADS / 32) : p.parts;
  if (part_ctas >= 65535) return BX_ELIMIT;
  const dim3 grid(M, part_ctas + (p.conv.w && p.conv.taps > 1 ? 1 : 0));
  auto* kernel = warp ? (vec ? fl_gated_norm_kernel<T, true, 8> : fl_gated_norm_kernel<T, true, 1>)
                      : (vec ? fl_gated_norm_kernel<T, false, 8> : fl_gated_norm_kernel<T, false, 1>);
  return launch_chained(kernel, grid, GATE_THREADS, 0, st, 0, p, part_ctas);
}

// Rows of a scan chunk: short ones while there are few rows to spread over the SMs.
int gru_chunk(int M) { return M <= 512 ? 16 : 64; }

}  // namespace

extern "C" {

int bxf_version(void) { return 1; }
long long bxf_launch_count(void) { return g_launches; }
int bxf_device_status(void) { return status_read(); }
int bxf_clear_device_status(void) { return status_clear(); }
int bxf_set_device_status(int value) { return status_write(value); }

int bxf_linear(int dtype, const void* w, int64_t ldw, int64_t gsw, const void* x, int64_t ldx, int64_t gsx, int groups,
               int M, int N, int K, const int* counts, const bxf_epilogue* epi, int tile, void* stream) {
  if (!dtype_ok(dtype) || !epi || groups < 1 || M < 0 || N < 1 || K < 1) return BX_EARG;
  if (!operand_ok(w, ldw, gsw, groups > 1, K, dtype) || !operand_ok(x, ldx, gsx, groups > 1 && !counts, K, dtype))
    return BX_EARG;
  if (epi->kind < BXF_EPI_STORE || epi->kind > BXF_EPI_GLU || !epi->out) return BX_EARG;
  if (epi->kind == BXF_EPI_STORE && epi->n_main < N && (!epi->side || groups > 1)) return BX_EARG;
  if (epi->kind == BXF_EPI_GATE && !epi->gate) return BX_EARG;
  if (epi->kind == BXF_EPI_GLU && (N % 2 || groups > 1)) return BX_EARG;
  if (epi->kind == BXF_EPI_ROPE &&
      (!epi->rot_out || !epi->cs || epi->rot_dim < 2 || epi->rot_dim % 2 || epi->n_main % 8 || groups > 1))
    return BX_EARG;
  if (g_status_seen.load() != 0) return BX_EDEVICE;
  if (M == 0) return BX_OK;
  const Operands o{w, x, ldw, gsw, ldx, gsx};
  const GemmShape s{M, N, K, groups, 0, 0, counts};
  if (dtype == BXF_F32) return launch_simt<StageEpi>(o, s, *epi, stream_of(stream));
  return run_bf16(o, s, *epi, tile, stream_of(stream));
}

int bxf_gru_rows(int dtype) { return dtype == BXF_F32 ? SIMT_TA : 64; }
int bxf_gru_chunks(int M) { return ceil_div(M, gru_chunk(M)); }

int bxf_gru_linear(int dtype, const void* w, int64_t ldw, const void* x, int64_t ldx, int M, int width, int K,
                   const bxf_gru* gru, void* stream) {
  if (!dtype_ok(dtype) || !gru_ok(gru, M, width) || K < 1 || M > bxf_gru_rows(dtype)) return BX_EARG;
  if (!operand_ok(w, ldw, (i64)width * ldw, true, K, dtype) || !operand_ok(x, ldx, 0, false, K, dtype)) return BX_EARG;
  if (g_status_seen.load() != 0) return BX_EDEVICE;
  if (M == 0) return BX_OK;
  const Operands o{w, x, ldw, (i64)width * ldw, ldx, 0};
  const GemmShape s{M, width, K, 1, 0, 0, nullptr};
  cudaStream_t st = stream_of(stream);
  if (dtype == BXF_F32) return launch_simt<GruEpi>(o, s, *gru, st);
  const int sms = device_sms();
  if (sms <= 0) return BX_ELAUNCH;
  const int tile = M <= 16 ? 16 : 64;
  const int split = tile_plan(s, 3, tile, FL_SPLIT_MAX, sms).split;
  return tile == 16 ? launch_tiles<16, GruEpi>(o, s, *gru, split, st) : launch_tiles<64, GruEpi>(o, s, *gru, split, st);
}

int bxf_gru_scan(int dtype, float* y, float* fold, int M, int width, const bxf_gru* gru, void* stream) {
  if (!dtype_ok(dtype) || !gru_ok(gru, M, width) || !y || !fold) return BX_EARG;
  if (M == 0) return BX_OK;
  const int chunk = gru_chunk(M);
  if (ceil_div(M, chunk) > 65535) return BX_ELIMIT;
  const dim3 grid(ceil_div(width, 128), ceil_div(M, chunk));
  float2* f = reinterpret_cast<float2*>(fold);
  const int rc = launch_chained(dtype == BXF_F32 ? fl_gru_fold_kernel<float> : fl_gru_fold_kernel<bf16>, grid, 128, 0,
                                stream_of(stream), 0, *gru, y, f, M, width, chunk);
  if (rc != BX_OK) return rc;
  return launch_chained(dtype == BXF_F32 ? fl_gru_apply_kernel<float> : fl_gru_apply_kernel<bf16>, grid, 128, 0,
                        stream_of(stream), 0, *gru, y, f, M, width, chunk);
}

int bxf_row_flags(const int64_t* seq, const int64_t* slot, const int64_t* pos, int* flags, int M, void* stream) {
  if (!seq || !slot || !pos || !flags || M < 0) return BX_EARG;
  if (M == 0) return BX_OK;
  return launch_chained(fl_row_flags_kernel, dim3(ceil_div(M, 256)), 256, 0, stream_of(stream), 0,
                        reinterpret_cast<const i64*>(seq), reinterpret_cast<const i64*>(slot),
                        reinterpret_cast<const i64*>(pos), flags, M);
}

int bxf_norm(int dtype, float* x, const int64_t* ids, const void* embed, int64_t V, const float* y, const int* place,
             const float* weight, int top, const float* w, const float* b, float eps, void* h, int64_t ldh, int* zero,
             int nzero, int M, int D, void* stream) {
  if (!dtype_ok(dtype) || !x || M < 0 || D < 1 || D > 32768 || top < 0 || nzero < 0) return BX_EARG;
  if ((ids && (!embed || V < 1)) || (top > 0 && (!y || !place || !weight)) || (h && (!w || !b || ldh < D)) ||
      (nzero > 0 && !zero))
    return BX_EARG;
  if (M == 0) return BX_OK;
  const int smem = D * 4;
  const i64* ids_ = reinterpret_cast<const i64*>(ids);
  auto go = [&](auto* kernel, auto* typed, PerDevice& configured) {
    using T = std::remove_pointer_t<decltype(typed)>;
    if (once_per_device(configured, [&] {
          return cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 32768 * 4);
        }) != BX_OK)
      return BX_ELAUNCH;
    return launch_chained(kernel, dim3(M), NORM_THREADS, smem, stream_of(stream), 0, x, ids_, static_cast<const T*>(embed), V,
                          y, place, weight, top, w, b, eps, static_cast<T*>(h), ldh, zero, nzero, D);
  };
  static PerDevice conf16, conf32;
  return dtype == BXF_F32 ? go(fl_norm_kernel<float>, (float*)nullptr, conf32) : go(fl_norm_kernel<bf16>, (bf16*)nullptr, conf16);
}

int bxf_route(const float* logits, int64_t ldl, int experts, int top, int* chosen, float* weight, int* rank, int* counts,
              int M, void* stream) {
  if (!logits || !chosen || !weight || !rank || !counts || M < 0) return BX_EARG;
  if (experts < 1 || experts > BXF_MAX_EXPERTS || top < 1 || top > BXF_MAX_TOP || top > experts) return BX_ELIMIT;
  if (M == 0) return BX_OK;
  return launch_chained(fl_route_kernel, dim3(ceil_div(M, 8)), 256, 0, stream_of(stream), 0, logits, ldl, experts, top, chosen,
                        weight, rank, counts, M);
}

int bxf_gather(int dtype, const void* h, int64_t ldh, int D, const int* chosen, const int* rank, const int* counts,
               int experts, int top, void* hp, int* place, int M, void* stream) {
  if (!dtype_ok(dtype) || !h || !chosen || !rank || !counts || !hp || !place || M < 0 || D < 1 || ldh < D) return BX_EARG;
  if (experts < 1 || experts > BXF_MAX_EXPERTS || top < 1 || top > BXF_MAX_TOP) return BX_ELIMIT;
  if (M == 0) return BX_OK;
  if (dtype == BXF_F32)
    return launch_chained(fl_gather_kernel<float>, dim3(M * top), 128, 0, stream_of(stream), 0, static_cast<const float*>(h),
                          ldh, D, chosen, rank, counts, top, static_cast<float*>(hp), place);
  return launch_chained(fl_gather_kernel<bf16>, dim3(M * top), 128, 0, stream_of(stream), 0, static_cast<const bf16*>(h), ldh,
                        D, chosen, rank, counts, top, static_cast<bf16*>(hp), place);
}

int bxf_latent_prepare(int dtype, const float* y, int64_t ldy, int q_rank, int kv_rank, int rot_dim, int heads,
                       const float* wq, const float* wkv, float eps, const float* freq, const int64_t* pos,
                       const int64_t* slot, void* cq, int64_t ldcq, void* cache, int64_t ldc, float* cs, float* gate,
                       int M, void* stream) {
  if (!dtype_ok(dtype) || !y || !wq || !wkv || !freq || !pos || !slot || !cq || !cache || !cs || !gate || M < 0)
    return BX_EARG;
  if (q_rank < 1 || kv_rank < 1 || rot_dim < 0 || rot_dim % 2 || heads < 1 || ldy < q_rank + kv_rank + rot_dim + heads ||
      ldcq < q_rank || ldc < kv_rank + rot_dim)
    return BX_EARG;
  if (M == 0) return BX_OK;
  const i64 *pos_ = reinterpret_cast<const i64*>(pos), *slot_ = reinterpret_cast<const i64*>(slot);
  if (dtype == BXF_F32)
    return launch_chained(fl_latent_prepare_kernel<float>, dim3(M), PREP_THREADS, 0, stream_of(stream), 0, y, ldy, q_rank,
                          kv_rank, rot_dim, heads, wq, wkv, eps, freq, pos_, slot_, static_cast<float*>(cq), ldcq,
                          static_cast<float*>(cache), ldc, cs, gate);
  return launch_chained(fl_latent_prepare_kernel<bf16>, dim3(M), PREP_THREADS, 0, stream_of(stream), 0, y, ldy, q_rank,
                        kv_rank, rot_dim, heads, wq, wkv, eps, freq, pos_, slot_, static_cast<bf16*>(cq), ldcq,
                        static_cast<bf16*>(cache), ldc, cs, gate);
}

size_t bxf_latent_attention_scratch(int M, int heads, int kv_rank) { return attention_scratch_for(M, 1, heads, kv_rank); }

int bxf_latent_attention_tile(int heads) { return heads >= 128 ? 1 : 128 / (heads < 1 ? 1 : heads); }

int bxf_latent_attention(int dtype, const void* q, int64_t ldq, int M, int heads, int kv_rank, int rot_dim,
                         const void* cache, int64_t ldc, int bs, int nb, const void* bt, int bt_is64, int64_t bt_stride,
                         int nblk, const int64_t* seq, const int64_t* pos, const int* tiles, int ntiles, int window,
                         const float* sink, float scale, void* out, int64_t ldo, void* scratch, size_t scratch_bytes,
                         int variant, void* stream) {
  if (!dtype_ok(dtype) || !q || !cache || !bt || !seq || !pos || !out || M < 0 || heads < 1) return BX_EARG;
  if (kv_rank < 1 || rot_dim < 0 || ldq < kv_rank + rot_dim || ldc < kv_rank + rot_dim || ldo < kv_rank || bs < 1 || nb < 1 ||
      nblk < 1 || window < 0 || heads > 65535)
    return BX_EARG;
  const PagedAttn a{q, ldq, M, heads, 1, kv_rank + rot_dim, kv_rank, 0, cache, ldc, bs, nb, bt, bt_is64, bt_stride, nblk,
                    reinterpret_cast<const i64*>(seq), reinterpret_cast<const i64*>(pos), tiles, ntiles, window, sink,
                    scale, out, heads * ldo, ldo};
  return run_attention(dtype, a, scratch, scratch_bytes, variant, stream_of(stream));
}

int bxf_angles(const double* freq, int half, const int64_t* pos, float* cs, int M, void* stream) {
  if (!freq || !pos || !cs || half < 1 || M < 0) return BX_EARG;
  if (M == 0) return BX_OK;
  const i64 n = (i64)M * half;
  return launch_chained(fl_angles_kernel, dim3((unsigned)((n + 255) / 256)), 256, 0, stream_of(stream), 0, freq, half,
                        reinterpret_cast<const i64*>(pos), cs, n);
}

int bxf_gqa_prepare(int dtype, const bxf_gqa_rows* p, int M, void* stream) {
  if (!dtype_ok(dtype) || !p || M < 0) return BX_EARG;
  if (p->heads < 1 || p->kv_heads < 1 || p->heads % p->kv_heads || p->dim < 1 || p->vdim < 1 || p->rot_dims < 0 ||
      p->rot_dims % 2 || p->rot_dims > p->dim || (p->rot_dims > 0 && !p->cs) || !p->y || !p->slot || !p->q || !p->cache ||
      p->page < 1)
    return BX_EARG;
  const i64 nq = (i64)p->heads * p->dim, nk = (i64)p->kv_heads * p->dim, nv = (i64)p->kv_heads * p->vdim;
  if (p->ldy < nq + nk + nv || p->ldq < p->dim || p->voff < p->dim || p->ldc < p->voff + p->vdim) return BX_EARG;
  if (M == 0) return BX_OK;
  const bool vec = p->dim % 8 == 0 && p->vdim % 8 == 0 && p->rot_dims % 16 == 0 && p->ldy % 8 == 0 && p->ldq % 8 == 0 &&
                   p->ldc % 8 == 0 && p->voff % 8 == 0 && aligned16(p->y) && aligned16(p->q) && aligned16(p->cache);
  cudaStream_t st = stream_of(stream);
  if (dtype == BXF_F32)
    return launch_chained(fl_gqa_prepare_kernel<float, 1>, dim3(M), PREP_THREADS, 0, st, 0, *p, M);
  return launch_chained(vec ? fl_gqa_prepare_kernel<bf16, 8> : fl_gqa_prepare_kernel<bf16, 1>, dim3(M), PREP_THREADS, 0, st, 0,
                        *p, M);
}

size_t bxf_gqa_attention_scratch(int M, int heads, int kv_heads, int vdim) {
  return kv_heads < 1 ? 0 : attention_scratch_for(M, kv_heads, heads / kv_heads, vdim);
}

int bxf_gqa_attention(int dtype, const void* q, int64_t ldq, int M, int heads, int kv_heads, int dim, int vdim,
                      const void* cache, int64_t ldc, int64_t voff, int bs, int nb, const void* bt, int bt_is64,
                      int64_t bt_stride, int nblk, const int64_t* seq, const int64_t* pos, const int* tiles, int ntiles,
                      int window, const float* sink, float scale, void* out, int64_t ldo, void* scratch,
                      size_t scratch_bytes, int variant, void* stream) {
  if (!dtype_ok(dtype) || !q || !cache || !bt || !seq || !pos || !out || M < 0 || heads < 1 || kv_heads < 1) return BX_EARG;
  if (heads % kv_heads || dim < 1 || vdim < 1 || ldq < dim || voff < dim || ldc < voff + vdim ||
      ldo < (int64_t)heads * vdim || bs < 1 || nb < 1 || nblk < 1 || window < 0)
    return BX_EARG;
  const PagedAttn a{q, ldq, M, heads / kv_heads, kv_heads, dim, vdim, (int)voff, cache, ldc, bs, nb, bt, bt_is64, bt_stride,
                    nblk, reinterpret_cast<const i64*>(seq), reinterpret_cast<const i64*>(pos), tiles, ntiles, window, sink,
                    scale, out, ldo, vdim};
  return run_attention(dtype, a, scratch, scratch_bytes, variant, stream_of(stream));
}

int bxf_streams(int dtype, const bxf_streams_step* p, int M, void* stream) {
  if (!dtype_ok(dtype) || !p || M < 0 || !p->x || p->streams < 1 || p->streams > BXF_MAX_STREAMS || p->D < 1 || p->D > 32768)
    return BX_EARG;
  if ((p->ids && (!p->embed || p->vocab < 1)) || (p->y && (!p->out || !p->mix)) || (p->h && (!p->w || p->ldh < p->D)) ||
      (!p->h && !p->sum))
    return BX_EARG;
  if (M == 0) return BX_OK;
  const bool vec = p->D % 4 == 0 && (!p->h || p->ldh % 4 == 0);
  return dtype == BXF_F32 ? launch_streams<float>(*p, M, vec, stream_of(stream)) : launch_streams<bf16>(*p, M, vec, stream_of(stream));
}

int bxf_causal_conv(int dtype, const bxf_conv* c, void* out, int64_t ldo, int M, void* stream) {
  if (!dtype_ok(dtype) || !conv_ok(c) || !out || ldo < c->channels || M < 0) return BX_EARG;
  if (M == 0) return BX_OK;
  if (ceil_div(M, CONV_ROWS) > 65535) return BX_ELIMIT;
  const dim3 grid(ceil_div(c->channels, 2 * CONV_THREADS), ceil_div(M, CONV_ROWS));
  cudaStream_t st = stream_of(stream);
  if (dtype == BXF_F32)
    return launch_chained(fl_causal_conv_kernel<float>, grid, CONV_THREADS, 0, st, 0, *c, static_cast<float*>(out), ldo, M);
  if (c->taps >= 2 && c->taps <= 4 && c->channels % 8 == 0 && c->ldu % 8 == 0 && ldo % 8 == 0 && aligned16(c->u) &&
      aligned16(out) && aligned16(c->state) && aligned16(c->w) && aligned16(c->b)) {
    const int rows = M <= 64 ? 1 : M <= 1024 ? CONV_BATCH : CONV_ROWS;
    const dim3 wide(ceil_div(c->channels, 8 * CONV_THREADS), ceil_div(M, rows));
    return launch_chained(c->taps == 2 ? fl_causal_conv_rows_kernel<2> : c->taps == 3 ? fl_causal_conv_rows_kernel<3>
                                                                                      : fl_causal_conv_rows_kernel<4>,
                          wide, CONV_THREADS, 0, st, 0, *c, static_cast<bf16*>(out), ldo, M, rows);
  }
  return launch_chained(fl_causal_conv_kernel<bf16>, grid, CONV_THREADS, 0, st, 0, *c, static_cast<bf16*>(out), ldo, M);
}

int bxf_recurrence(int dtype, const bxf_recurrence_rows* p, int M, void* stream) {
  if (!dtype_ok(dtype) || !recurrence_ok(p) || M < 0) return BX_EARG;
  if (p->K > BXF_MAX_STATE || p->heads > 65535 || ceil_div(p->V, 32) > 65535) return BX_ELIMIT;
  if (p->kind == BXF_DECAY_CHANNEL && !p->decays) return BX_EARG;
  if (M == 0) return BX_OK;
  if (p->kind == BXF_DECAY_CHANNEL) {
    const int rows = M <= 64 ? 1 : DECAY_ROWS;
    if (ceil_div(M, rows) > 65535) return BX_ELIMIT;
    const int rc = launch_chained(fl_decay_rows_kernel, dim3(ceil_div(p->heads * p->K, 256), ceil_div(M, rows)), 256, 0,
                                  stream_of(stream), 0, *p, M, rows);
    if (rc != BX_OK) return rc;
  }
  return dtype == BXF_F32 ? launch_recurrence<float>(*p, M, stream_of(stream)) : launch_recurrence<bf16>(*p, M, stream_of(stream));
}

int bxf_recurrence_chunk_rows(int dtype, int K, int V) { return chunks_fit(dtype, K, V) ? RC_ROWS : 0; }

size_t bxf_recurrence_chunk_scratch(int kind, int M, int chunks, int segments, int heads, int K, int V) {
  if (M < 1 || chunks < 1 || segments < 0 || heads < 1 || K < 1 || V < 1) return 0;
  return chunk_scratch(kind, M, chunks, segments, heads, K, V).bytes;
}

int bxf_recurrence_chunks(int dtype, const bxf_recurrence_rows* p, const bxf_chunk_table* t, void* scratch,
                          size_t scratch_bytes, int M, void* stream) {
  if (!recurrence_ok(p) || !t || M < 0 || !t->runs || !t->chunks || t->nruns < 0 || t->nchunks < t->nruns || t->nsegments < 0 ||
      (t->nsegments > 0 && (!t->segments || !t->spans)))
    return BX_EARG;
  if (!chunks_fit(dtype, p->K, p->V) || p->heads > 65535 || ceil_div(p->K * p->V, 1024) > 65535) return BX_ELIMIT;
  if (p->ldy % 8 || p->q0 % 8 || p->k0 % 8 || p->v0 % 8 || p->ldo % 2 || !aligned16(p->y) || !aligned16(p->state)) return BX_EARG;
  if (M == 0 || t->nruns == 0) return BX_OK;
  const ChunkScratch s = chunk_scratch(p->kind, M, t->nchunks, t->nsegments, p->heads, p->K, p->V);
  if (s.bytes > 0 && (!scratch || !aligned16(scratch) || scratch_bytes < s.bytes)) return BX_EARG;
  uint8_t* at = static_cast<uint8_t*>(scratch);
  const auto take = [&](size_t bytes) {
    uint8_t* r = at;
    at += bytes;
    return r;
  };
  bf16* planes = reinterpret_cast<bf16*>(take(s.planes));
  float* edge = reinterpret_cast<float*>(take(s.edge));
  auto* masks = reinterpret_cast<unsigned long long*>(take(s.masks));
  float* states = reinterpret_cast<float*>(take(s.states));
  float* decays = reinterpret_cast<float*>(take(s.decays));
  const ChunkArgs a{t->runs, planes, edge, masks, states, decays, M};
  cudaStream_t st = stream_of(stream);
  if (p->kind == BXF_DECAY_HEAD) return launch_chunks<false>(*p, a, t->nruns, t->segments, t->nsegments, t->spans, st);
  const int smem = decay_prepare_smem(p->K, p->rank);
  if (smem > 200 * 1024) return BX_ELIMIT;
  static PerDevice configured;
  if (once_per_device(configured, [] {
        return cudaFuncSetAttribute(fl_decay_prepare_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
      }) != BX_OK)
    return BX_ELAUNCH;
  const int rc = launch_chained(fl_decay_prepare_kernel, dim3(t->nchunks, p->heads), RP_THREADS, smem, st, 0, *p, t->chunks, planes,
                                edge, masks, M);
  return rc != BX_OK ? rc : launch_chunks<true>(*p, a, t->nruns, t->segments, t->nsegments, t->spans, st);
}

int bxf_gated_norm(int dtype, const bxf_gate_rows* p, int M, void* stream) {
  if (!dtype_ok(dtype) || !p || M < 0 || !p->o || !p->z || !p->w || !p->out || p->n < 1 || p->parts < 1 || p->n % p->parts ||
      p->wn < 1 || p->ldo < p->n || p->ldz < p->n || p->ldout < p->n)
    return BX_EARG;
  if (p->conv.w && !conv_ok(&p->conv)) return BX_EARG;
  if (M == 0) return BX_OK;
  return dtype == BXF_F32 ? launch_gated_norm<float>(*p, M, stream_of(stream)) : launch_gated_norm<bf16>(*p, M, stream_of(stream));
}

}  // extern "C"
