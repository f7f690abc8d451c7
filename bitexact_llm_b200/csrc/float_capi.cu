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
#include "fl_stages.cuh"

namespace {

using namespace bxf;

static_assert(sizeof(bxf_epilogue) == 128 && sizeof(bxf_gru) == 80, "layouts of the callers' structs");

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

template <int TA, class Epi>
int maps_for(const Operands& o, const GemmShape& s, CUtensorMap* mw, CUtensorMap* mx) {
  constexpr int NP = Epi::PLANES;
  const bool ok = make_map_bf16(mw, o.w, s.K, s.N, NP > 1 ? NP : s.groups, o.ldw, o.gsw, NROWS, NP) &&
                  make_map_bf16(mx, o.x, s.K, s.M, NP > 1 || s.counts ? 1 : s.groups, o.ldx, o.gsx, TA, 1);
  return ok ? BX_OK : BX_ELAUNCH;
}

template <int TA, class Epi>
void tile_counts(GemmShape& s) {
  s.n_tiles = ceil_div(s.N, NROWS);
  s.m_tiles = s.counts ? s.M / TA + (s.groups < s.M ? s.groups : s.M) : ceil_div(s.M, TA);
}

// One tile per cluster; K is split while the tile list leaves most SMs idle and every slice keeps a few K blocks.
template <int TA, class Epi>
int launch_tiles(const Operands& o, GemmShape s, const typename Epi::Params& ep, cudaStream_t st) {
  using Cfg = FlCfg<Epi::PLANES, TA>;
  static PerDevice configured;
  if (once_per_device(configured, [] {
        return cudaFuncSetAttribute(fl_gemm_kernel<TA, Epi>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                    Cfg::SMEM_BYTES);
      }) != BX_OK)
    return BX_ELAUNCH;
  tile_counts<TA, Epi>(s);
  CUtensorMap mw, mx;
  if (int rc = maps_for<TA, Epi>(o, s, &mw, &mx)) return rc;
  const i64 tiles = (i64)s.n_tiles * s.m_tiles * (s.counts || Epi::PLANES > 1 ? 1 : s.groups);
  const int sms = device_sms(), nkb = ceil_div(s.K, KE);
  if (sms <= 0 || tiles > (1 << 24)) return BX_ELAUNCH;
  int split = 1;
  if (Cfg::PARTIAL_BYTES + Epi::stash_bytes(TA) <= Cfg::RING_BYTES)
    while (split < FL_SPLIT_MAX && tiles * split * 2 <= sms && nkb >= split * 4) split *= 2;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3((unsigned)(tiles * split), 1, 1);
  cfg.blockDim = dim3(GEMM_THREADS, 1, 1);
  cfg.dynamicSmemBytes = Cfg::SMEM_BYTES;
  cfg.stream = st;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = split;
  attr[0].val.clusterDim.y = 1;
  attr[0].val.clusterDim.z = 1;
  cfg.attrs = attr;
  cfg.numAttrs = 1;
  if (cudaLaunchKernelEx(&cfg, fl_gemm_kernel<TA, Epi>, mw, mx, s, ep) != cudaSuccess) return BX_ELAUNCH;
  return launched(1);
}

template <int TA, class Epi>
int launch_persistent(const Operands& o, GemmShape s, const typename Epi::Params& ep, cudaStream_t st) {
  using Cfg = FlCfg<Epi::PLANES, TA>;
  static PerDevice configured;
  if (once_per_device(configured, [] {
        return cudaFuncSetAttribute(fl_gemm_persistent_kernel<TA, Epi>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                    Cfg::SMEM_BYTES);
      }) != BX_OK)
    return BX_ELAUNCH;
  tile_counts<TA, Epi>(s);
  CUtensorMap mw, mx;
  if (int rc = maps_for<TA, Epi>(o, s, &mw, &mx)) return rc;
  const i64 tiles = (i64)s.n_tiles * s.m_tiles * (s.counts ? 1 : s.groups);
  const int sms = device_sms();
  if (sms <= 0 || tiles > (1 << 24)) return BX_ELAUNCH;
  fl_gemm_persistent_kernel<TA, Epi><<<(unsigned)(tiles < sms ? tiles : sms), GEMM_THREADS, Cfg::SMEM_BYTES, st>>>(mw, mx,
                                                                                                                s, ep);
  return launched(1);
}

bool operand_ok(const void* p, i64 ld, i64 gs, bool grouped, int K, int dtype) {
  if (!p || ld < K) return false;
  return dtype == BXF_F32 || (aligned16(p) && ld % 8 == 0 && (!grouped || gs % 8 == 0));
}

// Rows of a token tile when the caller leaves it open: the smallest that holds a group's rows (for experts: twice the
// mean, their sizes vary).
int pick_tile(const GemmShape& s) {
  const int rows = s.counts ? ceil_div(2 * s.M, s.groups) : s.M;
  return rows <= 16 ? 16 : rows <= 32 ? 32 : rows <= 64 ? 64 : rows <= 128 ? 128 : 256;
}

template <class Epi>
int run_bf16(const Operands& o, const GemmShape& s, const typename Epi::Params& ep, int ta, cudaStream_t st) {
  switch (ta ? ta : pick_tile(s)) {
    case 16: return launch_tiles<16, Epi>(o, s, ep, st);
    case 32: return launch_tiles<32, Epi>(o, s, ep, st);
    case 64: return launch_tiles<64, Epi>(o, s, ep, st);
    case 128: return launch_persistent<128, Epi>(o, s, ep, st);
    case 256: return launch_persistent<256, Epi>(o, s, ep, st);
    default: return BX_EARG;
  }
}

// The tensor-core attention kernel takes pages of 8, 16, .. keys, rows of at most 9 column blocks (shared memory).
bool latent_tc_fits(int dtype, const LatentAttn& a) {
  return dtype == BXF_BF16 && a.bs >= 8 && (a.bs & (a.bs - 1)) == 0 && ceil_div(a.R + a.rot, 64) <= 9 && aligned16(a.q) &&
         aligned16(a.cache) && aligned16(a.out) && a.ldq % 8 == 0 && a.ldc % 8 == 0 && a.ldo % 8 == 0;
}

size_t latent_scratch(i64 rows, int R, int splits) { return (size_t)splits * rows * (R + 2) * sizeof(float); }

int launch_latent_tc(const LatentAttn& a, void* scratch, size_t scratch_bytes, cudaStream_t st) {
  constexpr int SMEM_MAX = 227 * 1024;
  static PerDevice configured;
  if (once_per_device(configured, [] {
        return cudaFuncSetAttribute(fl_latent_attention_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM_MAX);
      }) != BX_OK)
    return BX_ELAUNCH;
  LatentTc c = {};
  const int W = a.R + a.rot;
  c.cols = ceil_div(W, 64);
  const int fixed = 1024 + c.cols * 128 * 128 + (int)sizeof(LatentShared);
  c.stages = (SMEM_MAX - fixed) / (c.cols * LT_KEYS * 128);
  if (c.stages > LT_MAX_STAGES) c.stages = LT_MAX_STAGES;
  const int tokens = a.tiles ? bxf_latent_attention_tile(a.H) : 1, tiles = a.tiles ? a.ntiles : a.M;
  const int rows = tokens * a.H;
  c.qrows = rows >= 128 ? 128 : ceil_div(rows, 8) * 8;
  c.row_blocks = ceil_div(rows, 128);
  c.vsplit = ceil_div(a.R, LT_VCOLS);
  c.splits = 1;
  const i64 span = a.window > 0 && a.window + tokens < (i64)a.nblk * a.bs ? a.window + tokens : (i64)a.nblk * a.bs;
  const i64 blocks = span / LT_KEYS + 1, ctas = (i64)tiles * c.row_blocks * c.vsplit;
  const int sms = device_sms();
  if (sms <= 0) return BX_ELAUNCH;
  while (c.splits < LT_MAX_SPLIT && ctas * c.splits * 2 <= sms && blocks >= c.splits * 4 && scratch &&
         scratch_bytes >= latent_scratch((i64)a.M * a.H, a.R, c.splits * 2))
    c.splits *= 2;
  c.part = static_cast<float*>(scratch);
  CUtensorMap mq, mc;
  if (!make_map_bf16(&mq, a.q, W, (i64)a.M * a.H, 1, a.ldq, 0, c.qrows, 1) ||
      !make_map_bf16(&mc, a.cache, W, a.bs, a.nb, a.ldc, (i64)a.bs * a.ldc, a.bs < LT_KEYS ? a.bs : LT_KEYS, 1))
    return BX_ELAUNCH;
  const dim3 grid(tiles, c.splits, c.row_blocks * c.vsplit);
  fl_latent_attention_tc_kernel<<<grid, LT_THREADS, fixed + c.stages * c.cols * LT_KEYS * 128, st>>>(mq, mc, a, c);
  if (c.splits == 1) return launched(1);
  fl_latent_join_kernel<<<(unsigned)(a.M * a.H), 128, 0, st>>>(a, c.part, c.splits);
  return launched(2);
}

constexpr int GRU_TILE = 64, GRU_LONG_TILE = 128;        // bf16; the 32-bit kernel has tiles of SIMT_TA rows

}  // namespace

extern "C" {

int bxf_version(void) { return 1; }
long long bxf_launch_count(void) { return g_launches; }
int bxf_device_status(void) { return status_read(); }
int bxf_clear_device_status(void) { return status_clear(); }
int bxf_set_device_status(int value) { return status_write(value); }

int bxf_linear(int dtype, const void* w, int64_t ldw, int64_t gsw, const void* x, int64_t ldx, int64_t gsx, int groups,
               int M, int N, int K, const int* counts, const bxf_epilogue* epi, int tile_rows, void* stream) {
  if (!dtype_ok(dtype) || !epi || groups < 1 || M < 0 || N < 1 || K < 1) return BX_EARG;
  if (!operand_ok(w, ldw, gsw, groups > 1, K, dtype) || !operand_ok(x, ldx, gsx, groups > 1 && !counts, K, dtype))
    return BX_EARG;
  if (epi->kind < BXF_EPI_STORE || epi->kind > BXF_EPI_GATE || !epi->out) return BX_EARG;
  if (epi->kind == BXF_EPI_STORE && epi->n_main < N && (!epi->side || groups > 1)) return BX_EARG;
  if (epi->kind == BXF_EPI_GATE && !epi->gate) return BX_EARG;
  if (epi->kind == BXF_EPI_ROPE &&
      (!epi->rot_out || !epi->cs || epi->rot_dim < 2 || epi->rot_dim % 2 || epi->n_main % 2 || groups > 1))
    return BX_EARG;
  if (g_status_seen.load() != 0) return BX_EDEVICE;
  if (M == 0) return BX_OK;
  const Operands o{w, x, ldw, gsw, ldx, gsx};
  const GemmShape s{M, N, K, groups, 0, 0, counts};
  if (dtype == BXF_F32) return launch_simt<StageEpi>(o, s, *epi, stream_of(stream));
  return run_bf16<StageEpi>(o, s, *epi, tile_rows, stream_of(stream));
}

int bxf_gru_tile_rows(int dtype) { return dtype == BXF_F32 ? SIMT_TA : GRU_TILE; }
int bxf_gru_long_tile(int dtype) { return dtype == BXF_F32 ? SIMT_TA : GRU_LONG_TILE; }

int bxf_gru_linear(int dtype, const void* w, int64_t ldw, const void* x, int64_t ldx, int M, int width, int K,
                   const bxf_gru* gru, void* stream) {
  if (!dtype_ok(dtype) || !gru || M < 0 || width < 1 || K < 1) return BX_EARG;
  if (!operand_ok(w, ldw, (i64)width * ldw, true, K, dtype) || !operand_ok(x, ldx, 0, false, K, dtype)) return BX_EARG;
  if (!gru->bias_z || !gru->bias_x || !gru->state || !gru->flags || !gru->seq || !gru->out) return BX_EARG;
  if (gru->mode == 0 ? M > bxf_gru_tile_rows(dtype) : (gru->mode != 1 || !gru->decay || !gru->local)) return BX_EARG;
  if (g_status_seen.load() != 0) return BX_EDEVICE;
  if (M == 0) return BX_OK;
  const Operands o{w, x, ldw, (i64)width * ldw, ldx, 0};
  const GemmShape s{M, width, K, 1, 0, 0, nullptr};
  cudaStream_t st = stream_of(stream);
  if (dtype == BXF_F32) return launch_simt<GruEpi>(o, s, *gru, st);
  if (gru->mode == 1) return launch_tiles<GRU_LONG_TILE, GruEpi>(o, s, *gru, st);
  if (M <= 16) return launch_tiles<16, GruEpi>(o, s, *gru, st);
  return launch_tiles<GRU_TILE, GruEpi>(o, s, *gru, st);
}

int bxf_gru_finish(int dtype, int M, int width, const bxf_gru* gru, void* stream) {
  if (!dtype_ok(dtype) || !gru || gru->mode != 1 || M < 0 || width < 1 || !gru->decay || !gru->local || !gru->out)
    return BX_EARG;
  if (M == 0) return BX_OK;
  const int tile = bxf_gru_long_tile(dtype);
  const dim3 grid(ceil_div(width, 128), ceil_div(M, tile), tile / 16);
  if (dtype == BXF_F32) fl_gru_finish_kernel<float><<<grid, 128, 0, stream_of(stream)>>>(*gru, M, width, tile);
  else fl_gru_finish_kernel<bf16><<<grid, 128, 0, stream_of(stream)>>>(*gru, M, width, tile);
  return launched(1);
}

int bxf_row_flags(const int64_t* seq, const int64_t* slot, const int64_t* pos, int* flags, int M, void* stream) {
  if (!seq || !slot || !pos || !flags || M < 0) return BX_EARG;
  if (M == 0) return BX_OK;
  fl_row_flags_kernel<<<ceil_div(M, 256), 256, 0, stream_of(stream)>>>(
      reinterpret_cast<const i64*>(seq), reinterpret_cast<const i64*>(slot), reinterpret_cast<const i64*>(pos), flags, M);
  return launched(1);
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
    kernel<<<M, NORM_THREADS, smem, stream_of(stream)>>>(x, ids_, static_cast<const T*>(embed), V, y, place, weight, top, w,
                                                         b, eps, static_cast<T*>(h), ldh, zero, nzero, D);
    return launched(1);
  };
  static PerDevice conf16, conf32;
  return dtype == BXF_F32 ? go(fl_norm_kernel<float>, (float*)nullptr, conf32) : go(fl_norm_kernel<bf16>, (bf16*)nullptr, conf16);
}

int bxf_route(const float* logits, int64_t ldl, int experts, int top, int* chosen, float* weight, int* rank, int* counts,
              int M, void* stream) {
  if (!logits || !chosen || !weight || !rank || !counts || M < 0) return BX_EARG;
  if (experts < 1 || experts > BXF_MAX_EXPERTS || top < 1 || top > BXF_MAX_TOP || top > experts) return BX_ELIMIT;
  if (M == 0) return BX_OK;
  fl_route_kernel<<<ceil_div(M, 8), 256, 0, stream_of(stream)>>>(logits, ldl, experts, top, chosen, weight, rank, counts, M);
  return launched(1);
}

int bxf_gather(int dtype, const void* h, int64_t ldh, int D, const int* chosen, const int* rank, const int* counts,
               int experts, int top, void* hp, int* place, int M, void* stream) {
  if (!dtype_ok(dtype) || !h || !chosen || !rank || !counts || !hp || !place || M < 0 || D < 1 || ldh < D) return BX_EARG;
  if (experts < 1 || experts > BXF_MAX_EXPERTS || top < 1 || top > BXF_MAX_TOP) return BX_ELIMIT;
  if (M == 0) return BX_OK;
  if (dtype == BXF_F32)
    fl_gather_kernel<float><<<M * top, 128, 0, stream_of(stream)>>>(static_cast<const float*>(h), ldh, D, chosen, rank,
                                                                    counts, top, static_cast<float*>(hp), place);
  else
    fl_gather_kernel<bf16><<<M * top, 128, 0, stream_of(stream)>>>(static_cast<const bf16*>(h), ldh, D, chosen, rank, counts,
                                                                   top, static_cast<bf16*>(hp), place);
  return launched(1);
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
    fl_latent_prepare_kernel<float><<<M, PREP_THREADS, 0, stream_of(stream)>>>(
        y, ldy, q_rank, kv_rank, rot_dim, heads, wq, wkv, eps, freq, pos_, slot_, static_cast<float*>(cq), ldcq,
        static_cast<float*>(cache), ldc, cs, gate);
  else
    fl_latent_prepare_kernel<bf16><<<M, PREP_THREADS, 0, stream_of(stream)>>>(
        y, ldy, q_rank, kv_rank, rot_dim, heads, wq, wkv, eps, freq, pos_, slot_, static_cast<bf16*>(cq), ldcq,
        static_cast<bf16*>(cache), ldc, cs, gate);
  return launched(1);
}

// Key splits only happen while the query tiles leave SMs idle.
size_t bxf_latent_attention_scratch(int M, int heads, int kv_rank) {
  if (M < 1 || heads < 1 || kv_rank < 1 || M > 148) return 0;
  return latent_scratch((i64)M * heads, kv_rank, LT_MAX_SPLIT);
}

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
  if (kv_rank > LA_MAX_R || kv_rank + rot_dim > 8192) return BX_ELIMIT;
  if (g_status_seen.load() != 0) return BX_EDEVICE;
  if (M == 0) return BX_OK;
  const LatentAttn a{q, ldq, M, heads, kv_rank, rot_dim, cache, ldc, bs, nb, bt, bt_is64, bt_stride, nblk,
                     reinterpret_cast<const i64*>(seq), reinterpret_cast<const i64*>(pos), tiles, ntiles, window, sink,
                     scale, out, ldo};
  if (variant == 2 && !latent_tc_fits(dtype, a)) return BX_ELIMIT;
  if (variant != 1 && latent_tc_fits(dtype, a) && (!tiles || ntiles > 0))
    return launch_latent_tc(a, scratch, scratch_bytes, stream_of(stream));
  const dim3 grid(M, heads);
  const int smem = (kv_rank + rot_dim) * 4;
  if (dtype == BXF_F32) fl_latent_attention_kernel<float><<<grid, LA_THREADS, smem, stream_of(stream)>>>(a);
  else fl_latent_attention_kernel<bf16><<<grid, LA_THREADS, smem, stream_of(stream)>>>(a);
  return launched(1);
}

}  // extern "C"
