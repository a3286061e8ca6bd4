// LinearTc: Y[r][n] = act(sum_k X[r][k] W[n][k] + bias[n]) for many rows, bf16 operands, fp32 sums, on
// the 5th-generation tensor cores: operands by TMA (128-byte swizzle) into a ring of stages, products
// by tcgen05.mma kind::f16 with the weights as the M operand (128 output features per tile) and the
// activation rows as the N operand (`nt` of them, 16..256), accumulators in tensor memory, two buffers,
// so that a tile's epilogue overlaps the next tile's products.
//
// LinearTc: one block per SM walks tiles. Roles: warp 0 lane 0 issues the copies, warp 1 lane 0 the
// products, warps 4..7 read the accumulators (a lane = one output feature, so a warp stores 32
// consecutive features of a row at a time).
//
// LinearTcGrouped: the same over the rows of a mixture's experts, sorted by expert: W [E][N][K] as one
// map of E N rows, tiles (expert, first row, rows) and their number from memory.
//
// LinearTcSplit2 / 4 / 8, for few tiles: a cluster of that many blocks shares one tile (nt <= 128), each
// block a part of K. The blocks exchange their fp32 partials through distributed shared memory, every
// block summing its share of the rows in block order.
//
// Every wait is bounded: one that runs out stores a code in the host-visible fault word, after which
// the block's other waits return at once and the kernel ends (copies in flight awaited, tensor memory
// freed).
#include <cuda.h>
#include <cuda_bf16.h>

#include "weight_ring.cuh"

namespace ainfer {

struct LinearTcArgs {
  CUtensorMap Wm;        // [N][K], box 64 x 128
  CUtensorMap Xm;        // [rows][K], box 64 x nt
  const float *Bias;     // [N] or null
  void *Y;               // [rows][ldy]
  int32_t rows, N, K, nt, ldy, act, out16;
  float cap;
};

struct LinearTcGroupedArgs {
  CUtensorMap Wm;        // [E N][K], box 64 x 128
  CUtensorMap Xm;        // [places][K], box 64 x nt
  void *Y;               // [places][ldy]
  const int4 *Tiles;     // (expert, first place, places <= nt, 0)
  const int32_t *Count;  // tiles
  int32_t N, K, nt, ldy, act, out16;
};

constexpr int kLtThreads = 256, kLtBudget = 200 * 1024;
constexpr uint32_t kLtSpin = 1u << 22;
__host__ __device__ inline uint32_t lt_stage_bytes(int nt) { return (128u + (uint32_t)nt) * 128u; }
__host__ __device__ inline uint32_t lt_stages(int nt) {
  const uint32_t s = (uint32_t)kLtBudget / lt_stage_bytes(nt);
  return s > 8 ? 8 : s;
}

__device__ __forceinline__ uint64_t lt_desc(uint32_t addr) {
  // K-major operand, 128-byte swizzle: rows of 128 bytes in groups of eight (1024 bytes apart)
  return (uint64_t)((addr >> 4) & 0x3FFFu) | (1ull << 16) | ((uint64_t)(1024u >> 4) << 32) | (1ull << 46) | (2ull << 61);
}
__device__ __forceinline__ void lt_mma(uint32_t d, uint64_t da, uint64_t db, uint32_t idesc, uint32_t acc) {
  asm volatile(
      "{\n\t.reg .pred p;\n\tsetp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}" ::"r"(d), "l"(da), "l"(db), "r"(idesc), "r"(acc)
      : "memory");
}
__device__ __forceinline__ void lt_commit(uint32_t bar) {
  asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(bar) : "memory");
}
__device__ __forceinline__ void lt_tma(uint32_t dst, const CUtensorMap *m, uint32_t bar, int x, int y) {
  asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4}], [%2];" ::"r"(dst),
               "l"(reinterpret_cast<uint64_t>(m)), "r"(bar), "r"(x), "r"(y)
               : "memory");
}
__device__ __forceinline__ void lt_ld16(uint32_t taddr, uint32_t (&v)[16]) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15}, [%16];"
      : "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3]), "=r"(v[4]), "=r"(v[5]), "=r"(v[6]), "=r"(v[7]), "=r"(v[8]), "=r"(v[9]), "=r"(v[10]),
        "=r"(v[11]), "=r"(v[12]), "=r"(v[13]), "=r"(v[14]), "=r"(v[15])
      : "r"(taddr)
      : "memory");
}
__device__ __forceinline__ void lt_ld_wait() { asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory"); }
__device__ __forceinline__ float lt_act(float v, int act, float cap) {
  if (act == 1) { v = v > 0.0f ? v : 0.0f; return v * v; }
  if (act == 2) return cap * tanhf(v / cap);
  return v;
}
// One accumulator lane (an output feature) over nr rows: y points at the feature in the tile's first
// row. No branch depends on data, so the columns of a load overlap; the next columns' load is in flight
// while these are stored.
template <int ACT, typename T>
__device__ __forceinline__ void lt_store16(const uint32_t (&v)[16], T *y, size_t ldy, float bias, float cap, bool in, int left) {
#pragma unroll
  for (int i = 0; i < 16; ++i) {
    const float r = lt_act(__uint_as_float(v[i]) + bias, ACT, cap);
    if (in && i < left) {
      if constexpr (sizeof(T) == 2) y[i * ldy] = __float2bfloat16_rn(r);
      else y[i * ldy] = r;
    }
  }
}
template <int ACT, typename T>
__device__ __forceinline__ void lt_epilogue(uint32_t taddr, int nr, T *y, int ld, float bias, float cap, bool in) {
  const size_t ldy = (size_t)ld;
  uint32_t a[16], b[16];
  lt_ld16(taddr, a);
  for (int c = 0; c < nr; c += 32) {
    lt_ld_wait();
    if (c + 16 < nr) lt_ld16(taddr + (uint32_t)c + 16u, b);
    lt_store16<ACT, T>(a, y + (size_t)c * ldy, ldy, bias, cap, in, nr - c);
    if (c + 16 >= nr) break;
    lt_ld_wait();
    if (c + 32 < nr) lt_ld16(taddr + (uint32_t)c + 32u, a);
    lt_store16<ACT, T>(b, y + (size_t)(c + 16) * ldy, ldy, bias, cap, in, nr - c - 16);
  }
}

struct LtShared {
  unsigned long long full[8], empty[8], acc_full[2], acc_empty[2], drain;
  uint32_t tmem, fail;
};
__device__ __forceinline__ bool lt_wait(LtShared *s, unsigned long long *b, uint32_t parity) {
  if (mbar_try(b, parity)) return true;
  for (uint32_t i = 0; i < kLtSpin; ++i) {
    if (mbar_try(b, parity)) return true;
    if (*reinterpret_cast<volatile uint32_t *>(&s->fail)) return false;
  }
  *reinterpret_cast<volatile uint32_t *>(&s->fail) = 1;
  if (g_stream_fault_word) *reinterpret_cast<volatile unsigned int *>(g_stream_fault_word) = 1;
  return false;
}

// What a tile is: its first row of the weights' map, first output feature, first row and rows.
struct LtTile { int w0, n0, r0, nr; };
__device__ __forceinline__ LtTile lt_tile(const LinearTcArgs &a, int u, int n_tiles) {
  const int n0 = (u % n_tiles) * 128, r0 = (u / n_tiles) * a.nt;
  return LtTile{n0, n0, r0, min(a.nt, a.rows - r0)};
}
__device__ __forceinline__ LtTile lt_tile(const LinearTcGroupedArgs &a, int u, int n_tiles) {
  const int4 t = a.Tiles[u / n_tiles];
  const int n0 = (u % n_tiles) * 128;
  return LtTile{t.x * a.N + n0, n0, t.y, t.z};
}
__device__ __forceinline__ int lt_tiles(const LinearTcArgs &a, int n_tiles) { return n_tiles * ((a.rows + a.nt - 1) / a.nt); }
__device__ __forceinline__ int lt_tiles(const LinearTcGroupedArgs &a, int n_tiles) { return n_tiles * a.Count[0]; }
__device__ __forceinline__ float lt_bias(const LinearTcArgs &a, int n) { return a.Bias && n < a.N ? a.Bias[n] : 0.0f; }
__device__ __forceinline__ float lt_bias(const LinearTcGroupedArgs &, int) { return 0.0f; }
__device__ __forceinline__ float lt_cap(const LinearTcArgs &a) { return a.cap; }
__device__ __forceinline__ float lt_cap(const LinearTcGroupedArgs &) { return 0.0f; }

template <typename Args>
__device__ __forceinline__ void linear_tc_body(const Args &a) {
  extern __shared__ __align__(1024) unsigned char lt_smem_raw[];
  __shared__ LtShared sh;
  pdl_launch_dependents();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const uint32_t base = (smem_addr(lt_smem_raw) + 1023u) & ~1023u;
  const int nt = a.nt, nst = (int)lt_stages(nt);
  const uint32_t stage_bytes = lt_stage_bytes(nt);
  const int n_tiles = (a.N + 127) / 128;
  const int kb = (a.K + 63) / 64;
  uint32_t cols = 32;
  while (cols < 2u * (uint32_t)nt) cols <<= 1;
  if (tid == 0) {
    for (int i = 0; i < nst; ++i) { mbar_init(&sh.full[i], 1); mbar_init(&sh.empty[i], 1); }
    for (int i = 0; i < 2; ++i) { mbar_init(&sh.acc_full[i], 1); mbar_init(&sh.acc_empty[i], 128); }
    mbar_init(&sh.drain, 1);
    sh.fail = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    asm volatile("prefetch.tensormap [%0];" ::"l"(reinterpret_cast<uint64_t>(&a.Wm)) : "memory");
    asm volatile("prefetch.tensormap [%0];" ::"l"(reinterpret_cast<uint64_t>(&a.Xm)) : "memory");
  }
  if (warp == 2) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_addr(&sh.tmem)), "r"(cols) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
  const uint32_t tmem = sh.tmem;
  pdl_wait();
  const int tiles = lt_tiles(a, n_tiles);

  if (warp == 0 && lane == 0) {
    // ---- copies ----
    uint32_t st = 0, ph = 1, issued = 0;
    for (int u = blockIdx.x; u < tiles; u += gridDim.x) {
      const LtTile t = lt_tile(a, u, n_tiles);
      for (int k = 0; k < kb; ++k) {
        if (!lt_wait(&sh, &sh.empty[st], ph)) break;
        const uint32_t dst = base + st * stage_bytes, bar = smem_addr(&sh.full[st]);
        mbar_arrive_expect(&sh.full[st], stage_bytes);
        lt_tma(dst, &a.Wm, bar, k * 64, t.w0);
        lt_tma(dst + 128u * 128u, &a.Xm, bar, k * 64, t.r0);
        ++issued;
        if (++st == (uint32_t)nst) { st = 0; ph ^= 1; }
      }
      if (*reinterpret_cast<volatile uint32_t *>(&sh.fail)) break;
    }
    if (*reinterpret_cast<volatile uint32_t *>(&sh.fail)) {
      // await every copy still in flight (each stage's last use) before the block may end
      for (int i = 0; i < nst && (uint32_t)i < issued; ++i) {
        const uint32_t uses = (issued - (uint32_t)i + (uint32_t)nst - 1) / (uint32_t)nst;
        for (uint32_t s = 0; s < kLtSpin && !mbar_try(&sh.full[i], (uses - 1) & 1); ++s) {}
      }
    }
  } else if (warp == 1 && lane == 0) {
    // ---- products ----
    const uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(nt >> 3) << 17) | ((128u >> 4) << 24);
    uint32_t st = 0, ph = 0, buf = 0, aph = 1;
    for (int u = blockIdx.x; u < tiles; u += gridDim.x) {
      if (!lt_wait(&sh, &sh.acc_empty[buf], aph)) break;
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      const uint32_t d = tmem + buf * (uint32_t)nt;
      bool ok = true;
      for (int k = 0; k < kb; ++k) {
        ok = lt_wait(&sh, &sh.full[st], ph);
        if (!ok) break;
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        const uint64_t da = lt_desc(base + st * stage_bytes), db = lt_desc(base + st * stage_bytes + 128u * 128u);
#pragma unroll
        for (int q = 0; q < 4; ++q) lt_mma(d, da + (uint64_t)(2 * q), db + (uint64_t)(2 * q), idesc, k > 0 || q > 0 ? 1u : 0u);
        lt_commit(smem_addr(&sh.empty[st]));
        if (++st == (uint32_t)nst) { st = 0; ph ^= 1; }
      }
      if (!ok) break;
      lt_commit(smem_addr(&sh.acc_full[buf]));
      if (++buf == 2) { buf = 0; aph ^= 1; }
    }
    if (*reinterpret_cast<volatile uint32_t *>(&sh.fail)) {   // await the products already issued
      lt_commit(smem_addr(&sh.drain));
      for (uint32_t s = 0; s < kLtSpin && !mbar_try(&sh.drain, 0); ++s) {}
    }
  } else if (warp >= 4) {
    // ---- epilogue ----
    const int lw = (warp & 3) * 32 + lane;
    uint32_t buf = 0, ph = 0;
    for (int u = blockIdx.x; u < tiles; u += gridDim.x) {
      const LtTile t = lt_tile(a, u, n_tiles);
      const int n = t.n0 + lw, nr = t.nr;
      const float bias = lt_bias(a, n), cap = lt_cap(a);
      lt_wait(&sh, &sh.acc_full[buf], ph);
      __syncwarp();
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      const uint32_t taddr = tmem + buf * (uint32_t)nt + ((uint32_t)((warp & 3) * 32) << 16);
      const bool in = n < a.N;
      const size_t o = (size_t)t.r0 * a.ldy + n;
      if (a.out16) {
        __nv_bfloat16 *y = reinterpret_cast<__nv_bfloat16 *>(a.Y) + o;
        if (a.act == 1) lt_epilogue<1>(taddr, nr, y, a.ldy, bias, cap, in);
        else if (a.act == 2) lt_epilogue<2>(taddr, nr, y, a.ldy, bias, cap, in);
        else lt_epilogue<0>(taddr, nr, y, a.ldy, bias, cap, in);
      } else {
        float *y = reinterpret_cast<float *>(a.Y) + o;
        if (a.act == 1) lt_epilogue<1>(taddr, nr, y, a.ldy, bias, cap, in);
        else if (a.act == 2) lt_epilogue<2>(taddr, nr, y, a.ldy, bias, cap, in);
        else lt_epilogue<0>(taddr, nr, y, a.ldy, bias, cap, in);
      }
      asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
      mbar_arrive(&sh.acc_empty[buf]);
      if (++buf == 2) { buf = 0; ph ^= 1; }
    }
  }
  __syncwarp();
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  if (warp == 2) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(cols) : "memory");
}
__global__ void __launch_bounds__(kLtThreads, 1) LinearTc(const __grid_constant__ LinearTcArgs a) { linear_tc_body(a); }
__global__ void __launch_bounds__(kLtThreads, 1) LinearTcGrouped(const __grid_constant__ LinearTcGroupedArgs a) { linear_tc_body(a); }
static uint32_t linear_tc_smem(const void *args) {
  const int nt = ((const LinearTcArgs *)args)->nt;
  return lt_stages(nt) * lt_stage_bytes(nt) + 1024;
}
static uint32_t linear_tc_grouped_smem(const void *args) {
  const int nt = ((const LinearTcGroupedArgs *)args)->nt;
  return lt_stages(nt) * lt_stage_bytes(nt) + 1024;
}

// ---- K split over a cluster ----
// Half of an SM's shared memory, so that the next launch's blocks (or a second one of this) fit beside.
__host__ __device__ inline uint32_t lts_stages(int nt) {
  const uint32_t s = ((uint32_t)kLtBudget / 2 + 8192 - (uint32_t)nt * 512u) / lt_stage_bytes(nt);
  return s > 8 ? 8 : s;
}
__device__ __forceinline__ void cluster_sync_all() {
  asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
  asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
}
template <int CL>
__device__ __forceinline__ void linear_tc_split(const LinearTcArgs &a) {
  extern __shared__ __align__(1024) unsigned char lt_smem_raw[];
  __shared__ LtShared sh;
  pdl_launch_dependents();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const uint32_t base = (smem_addr(lt_smem_raw) + 1023u) & ~1023u;
  const int nt = a.nt, nst = (int)lts_stages(nt), rpo = nt / CL;   // rows of the tile that a block sums
  const uint32_t stage_bytes = lt_stage_bytes(nt), red = base + (uint32_t)nst * stage_bytes;
  float *red_p = reinterpret_cast<float *>(lt_smem_raw + (red - smem_addr(lt_smem_raw)));   // [CL][rpo][128]
  const int n_tiles = (a.N + 127) / 128, tile = blockIdx.x / CL, kb = (a.K + 63) / 64;
  uint32_t rank;
  asm volatile("mov.u32 %0, %%cluster_ctarank;" : "=r"(rank));
  const int n0 = (tile % n_tiles) * 128, r0 = (tile / n_tiles) * nt, nr = min(nt, a.rows - r0);
  const int k_lo = kb * (int)rank / CL, k_hi = kb * ((int)rank + 1) / CL;
  uint32_t cols = 32;
  while (cols < (uint32_t)nt) cols <<= 1;
  if (tid == 0) {
    for (int i = 0; i < nst; ++i) { mbar_init(&sh.full[i], 1); mbar_init(&sh.empty[i], 1); }
    mbar_init(&sh.acc_full[0], 1);
    mbar_init(&sh.drain, 1);
    sh.fail = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    asm volatile("prefetch.tensormap [%0];" ::"l"(reinterpret_cast<uint64_t>(&a.Wm)) : "memory");
    asm volatile("prefetch.tensormap [%0];" ::"l"(reinterpret_cast<uint64_t>(&a.Xm)) : "memory");
  }
  if (warp == 2) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_addr(&sh.tmem)), "r"(cols) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
  const uint32_t tmem = sh.tmem;
  cluster_sync_all();   // every block of the cluster runs: its shared memory may be written
  int pre = 0;          // stages whose weights travel before the dependency wait (they do not depend on it)
  if (warp == 0 && lane == 0)
    for (; pre < nst && k_lo + pre < k_hi; ++pre) {
      mbar_arrive_expect(&sh.full[pre], stage_bytes);
      lt_tma(base + (uint32_t)pre * stage_bytes, &a.Wm, smem_addr(&sh.full[pre]), (k_lo + pre) * 64, n0);
    }
  pdl_wait();

  if (warp == 0 && lane == 0) {
    uint32_t st = 0, ph = 1, issued = 0;
    for (int k = k_lo; k < k_hi; ++k) {
      const uint32_t dst = base + st * stage_bytes, bar = smem_addr(&sh.full[st]);
      if (k - k_lo >= pre) {
        if (!lt_wait(&sh, &sh.empty[st], ph)) break;
        mbar_arrive_expect(&sh.full[st], stage_bytes);
        lt_tma(dst, &a.Wm, bar, k * 64, n0);
      }
      lt_tma(dst + 128u * 128u, &a.Xm, bar, k * 64, r0);
      ++issued;
      if (++st == (uint32_t)nst) { st = 0; ph ^= 1; }
    }
    if (*reinterpret_cast<volatile uint32_t *>(&sh.fail)) {
      for (int i = 0; i < nst && (uint32_t)i < issued; ++i) {
        const uint32_t uses = (issued - (uint32_t)i + (uint32_t)nst - 1) / (uint32_t)nst;
        for (uint32_t s = 0; s < kLtSpin && !mbar_try(&sh.full[i], (uses - 1) & 1); ++s) {}
      }
    }
  } else if (warp == 1 && lane == 0) {
    const uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(nt >> 3) << 17) | ((128u >> 4) << 24);
    uint32_t st = 0, ph = 0;
    bool ok = true;
    for (int k = k_lo; k < k_hi; ++k) {
      ok = lt_wait(&sh, &sh.full[st], ph);
      if (!ok) break;
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      const uint64_t da = lt_desc(base + st * stage_bytes), db = lt_desc(base + st * stage_bytes + 128u * 128u);
#pragma unroll
      for (int q = 0; q < 4; ++q) lt_mma(tmem, da + (uint64_t)(2 * q), db + (uint64_t)(2 * q), idesc, k > k_lo || q > 0 ? 1u : 0u);
      lt_commit(smem_addr(&sh.empty[st]));
      if (++st == (uint32_t)nst) { st = 0; ph ^= 1; }
    }
    lt_commit(smem_addr(ok ? &sh.acc_full[0] : &sh.drain));
    if (!ok)
      for (uint32_t s = 0; s < kLtSpin && !mbar_try(&sh.drain, 0); ++s) {}
  } else if (warp >= 4) {
    const int lw = (warp & 3) * 32 + lane;
    lt_wait(&sh, &sh.acc_full[0], 0);
    __syncwarp();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const uint32_t taddr = tmem + ((uint32_t)((warp & 3) * 32) << 16);
    const uint32_t mine = red + ((uint32_t)rank * (uint32_t)rpo * 128u + (uint32_t)lw) * 4u;
    const int lg = 31 - __clz(rpo);   // nt and the cluster size are powers of two
    for (int c = 0; c < nr; c += 16) {
      uint32_t v[16];
      lt_ld16(taddr + (uint32_t)c, v);
      asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        const int col = c + i;
        if (col < nr) {
          uint32_t peer;
          asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(peer) : "r"(mine + (uint32_t)(col & (rpo - 1)) * 512u), "r"(col >> lg));
          asm volatile("st.shared::cluster.u32 [%0], %1;" ::"r"(peer), "r"(v[i]) : "memory");
        }
      }
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  }
  __syncwarp();
  cluster_sync_all();
  const int n = n0 + (tid & 127);
  if (n < a.N) {
    const float bias = a.Bias ? a.Bias[n] : 0.0f;
    for (int r = tid >> 7; r < rpo; r += 2) {
      const int row = (int)rank * rpo + r;
      if (row >= nr) break;
      float v = 0.0f;
#pragma unroll
      for (int s = 0; s < CL; ++s) v += red_p[(s * rpo + r) * 128 + (tid & 127)];
      v = lt_act(v + bias, a.act, a.cap);
      const size_t o = (size_t)(r0 + row) * a.ldy + n;
      if (a.out16) reinterpret_cast<uint16_t *>(a.Y)[o] = f32_to_bf16(v);
      else reinterpret_cast<float *>(a.Y)[o] = v;
    }
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  if (warp == 2) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(cols) : "memory");
}
__global__ void __cluster_dims__(2, 1, 1) __launch_bounds__(kLtThreads, 2) LinearTcSplit2(const __grid_constant__ LinearTcArgs a) { linear_tc_split<2>(a); }
__global__ void __cluster_dims__(4, 1, 1) __launch_bounds__(kLtThreads, 2) LinearTcSplit4(const __grid_constant__ LinearTcArgs a) { linear_tc_split<4>(a); }
__global__ void __cluster_dims__(8, 1, 1) __launch_bounds__(kLtThreads, 2) LinearTcSplit8(const __grid_constant__ LinearTcArgs a) { linear_tc_split<8>(a); }
static uint32_t linear_tc_split_smem(const void *args) {
  const int nt = ((const LinearTcArgs *)args)->nt;
  return lts_stages(nt) * lt_stage_bytes(nt) + (uint32_t)nt * 512u + 1024;
}

#define F(f) AINFER_ARG(LinearTcArgs, f)
#define LT_FIELDS F(Wm), F(Xm), F(Bias), F(Y), F(rows), F(N), F(K), F(nt), F(ldy), F(act), F(out16), F(cap)
AINFER_REGISTER(LinearTc, LinearTcArgs, kLtThreads, 0, 0, linear_tc_smem, LT_FIELDS);
AINFER_REGISTER(LinearTcSplit2, LinearTcArgs, kLtThreads, 2, 0, linear_tc_split_smem, LT_FIELDS);
AINFER_REGISTER(LinearTcSplit4, LinearTcArgs, kLtThreads, 4, 0, linear_tc_split_smem, LT_FIELDS);
AINFER_REGISTER(LinearTcSplit8, LinearTcArgs, kLtThreads, 8, 0, linear_tc_split_smem, LT_FIELDS);
#undef F

#define F(f) AINFER_ARG(LinearTcGroupedArgs, f)
AINFER_REGISTER(LinearTcGrouped, LinearTcGroupedArgs, kLtThreads, 0, 0, linear_tc_grouped_smem, F(Wm), F(Xm), F(Y), F(Tiles), F(Count), F(N), F(K),
                F(nt), F(ldy), F(act), F(out16));
#undef F

AINFER_EARLY_LAUNCH(LinearTcGrouped);
AINFER_EARLY_LAUNCH(LinearTc);
AINFER_EARLY_LAUNCH(LinearTcSplit2);
AINFER_EARLY_LAUNCH(LinearTcSplit4);
AINFER_EARLY_LAUNCH(LinearTcSplit8);

}  // namespace ainfer
