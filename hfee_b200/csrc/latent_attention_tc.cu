// Latent attention for prompt portions on the 5th-generation tensor cores: softmax attention of many query heads over ONE
// cached vector per token ([latent | shared rotated part]) whose leading dimensions are also the values.
//
// A CTA serves one request and a tile of 128 (token, head) rows (tokens_per_tile tokens of all heads), for up to
// LT_VALUES value columns (more are split among CTAs, which then compute the scores each for itself: the outputs fill
// the tensor memory).  Keys go in blocks of 64; a block is loaded once and is both the keys (K-major operand of the
// scores) and the values (MN-major operand of the outputs):
//   warp 0      TMA producer   the query tile once, 64 dimensions (a slab) per load; per block the slabs of 64 keys
//                              through the block table into a ring of stages
//   warp 1      MMA issuer     S_(j+1) = Q K_(j+1)^T into the one of two S buffers that is free, then, once the softmax
//                              warps have left P_j in tensor memory, O += P_j V_j; so the tensor core works on the next
//                              block's scores while this block's weights are computed (with room for one stage only the
//                              order is O += P_j V_j, then S_(j+1))
//   warps 4..7  softmax        one row per thread: S from tensor memory once, mask / max / exp2 / sum in registers, P
//                              back to one of two P buffers as packed bfloat16
// O stays in tensor memory for the whole key loop.  The running maximum is moved only when it grew by more than 2^8 in the
// exponent (then the warp rescales its O rows); the old one is kept otherwise, which cancels in O / sum.  The sink is one
// more term exp(sink[h]) of the sum, added at the end.  Rows of positions behind the tile's last token are cleared in the
// last block before it serves as values, so that nothing an earlier owner of the page left there (also a NaN) meets an
// MMA.  Pages of at least 64 tokens; other shapes use the mma.sync kernel.  Every barrier wait is bounded.
#include "tcgen05.cuh"

namespace {

using namespace tc;

constexpr int LT_ROWS = 128;                 // query rows per tile
constexpr int LT_KEYS = 64;                  // keys per block
constexpr int LT_VALUES = 256;               // value columns per CTA
constexpr int LT_Q_SLAB = LT_ROWS * 128;     // bytes of 64 dimensions of the query tile
constexpr int LT_K_SLAB = LT_KEYS * 128;     // bytes of 64 dimensions of a key block
constexpr int LT_MAX_STAGES = 4;
constexpr int LT_BAR_BYTES = 256;
constexpr int LT_SMEM_MAX = 227 * 1024;
constexpr float LT_RESCALE_LOG2 = 8.f;
// tensor memory columns: two S buffers of 64, two P buffers of 32 (64 packed bfloat16), O
constexpr uint32_t LT_S_COL = 0, LT_P_COL = 2 * LT_KEYS, LT_O_COL = LT_P_COL + LT_KEYS, LT_TMEM_COLS = 512;
static_assert(LT_O_COL + LT_VALUES <= LT_TMEM_COLS, "tensor memory");

struct LatentTcParams {
  __nv_bfloat16* out; long long ld_o;
  const int* block_table; int max_pages, page_shift, page_size;
  const int* cu_tokens; const int* slots; const int* context_before;
  int heads, dk, dv, slabs, stages;
  float scale_log2;
  int window, tokens_per_tile, q_tiles;
  const float* sink;
};

__device__ __forceinline__ void lt_load_3d(void* dst, const CUtensorMap* map, int c0, int c1, int c2, uint64_t* bar) {
  asm volatile(
      "cp.async.bulk.tensor.3d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5}], [%2];"
      ::"r"(smem_u32(dst)), "l"(reinterpret_cast<uint64_t>(map)), "r"(smem_u32(bar)), "r"(c0), "r"(c1), "r"(c2)
      : "memory");
}
// MN-major operand tile in the 128-byte swizzle: rows (the K index) of 64 contiguous MN elements, 8-row groups 1024 bytes apart.
__device__ __forceinline__ uint64_t lt_desc_mn(uint32_t smem_addr) {
  return (uint64_t)((smem_addr & 0x3FFFF) >> 4) | ((uint64_t)(16 >> 4) << 16) | ((uint64_t)(1024 >> 4) << 32) | (1ull << 46) | (2ull << 61);
}
// D[tmem] (+)= A[tmem] * B[smem]
__device__ __forceinline__ void lt_mma_ts(uint32_t tmem_d, uint32_t tmem_a, uint64_t desc_b, uint32_t idesc, uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t}"
      ::"r"(tmem_d), "r"(tmem_a), "l"(desc_b), "r"(idesc), "r"(accumulate) : "memory");
}
__device__ __forceinline__ void lt_st32(uint32_t taddr, const uint32_t (&v)[32]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], "
      "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16, "
      "%17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31, %32};"
      ::"r"(taddr), "r"(v[0]), "r"(v[1]), "r"(v[2]), "r"(v[3]), "r"(v[4]), "r"(v[5]), "r"(v[6]), "r"(v[7]),
        "r"(v[8]), "r"(v[9]), "r"(v[10]), "r"(v[11]), "r"(v[12]), "r"(v[13]), "r"(v[14]), "r"(v[15]),
        "r"(v[16]), "r"(v[17]), "r"(v[18]), "r"(v[19]), "r"(v[20]), "r"(v[21]), "r"(v[22]), "r"(v[23]),
        "r"(v[24]), "r"(v[25]), "r"(v[26]), "r"(v[27]), "r"(v[28]), "r"(v[29]), "r"(v[30]), "r"(v[31])
      : "memory");
}
__device__ __forceinline__ void lt_wait_st() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }
__device__ __forceinline__ float lt_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

__global__ void __launch_bounds__(256, 1)
latent_attention_tc_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k, LatentTcParams p,
                           int* __restrict__ status) {
  // no static shared memory: tiles first (1024-byte aligned for the swizzle), barriers behind them
  extern __shared__ __align__(1024) unsigned char smem_dyn[];
  const int slabs = p.slabs, ST = p.stages;
  const int stage_bytes = slabs * LT_K_SLAB;
  unsigned char* q_s = smem_dyn;                                // [slab][128 rows][64]
  unsigned char* kv_s = q_s + slabs * LT_Q_SLAB;                // [stage][slab][64 keys][64]
  uint64_t* q_full = reinterpret_cast<uint64_t*>(kv_s + ST * stage_bytes);
  uint64_t* k_full = q_full + 1;               // [LT_MAX_STAGES]
  uint64_t* kv_empty = k_full + LT_MAX_STAGES; // [LT_MAX_STAGES]
  uint64_t* s_full = kv_empty + LT_MAX_STAGES; // [2]  S_j is in buffer j & 1
  uint64_t* s_free = s_full + 2;               // [2]  the softmax threads hold S_j in registers
  uint64_t* p_full = s_free + 2;               // [2]  P_j is in buffer j & 1 (and O rescaled if it had to be)
  uint64_t* o_done = p_full + 2;               // [2]  the MMAs O += P_j V_j have completed
  uint64_t* v_clean = o_done + 2;              //      the last block's rows behind the last position are cleared
  uint32_t& tmem_base_slot = *reinterpret_cast<uint32_t*>(v_clean + 1);
  int& abort_flag = *reinterpret_cast<int*>(reinterpret_cast<uint32_t*>(v_clean + 1) + 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

  // the heaviest tiles (latest positions) first, the light ones fill the gaps at the end
  const int tile = p.q_tiles - 1 - (int)blockIdx.y, r = blockIdx.z, v0 = blockIdx.x * LT_VALUES;
  const int value_slabs = min(LT_VALUES, p.dv - v0) / 64;
  const int tok0 = p.cu_tokens[r], n_new = p.cu_tokens[r + 1] - tok0;
  const int t_first = tile * p.tokens_per_tile;
  if (t_first >= n_new) return;
  const int t_count = min(p.tokens_per_tile, n_new - t_first);
  const int slot = p.slots[r], pos_first = p.context_before[r] + t_first, pos_last = pos_first + t_count - 1;
  const int key_lo = (p.window > 0 && pos_first + 1 > p.window) ? pos_first + 1 - p.window : 0;
  const int b_lo = key_lo / LT_KEYS, nb = pos_last / LT_KEYS - b_lo + 1;

  if (threadIdx.x == 0) {
    abort_flag = (smem_u32(smem_dyn) & 1023u) != 0 ? 1 : 0;       // misaligned tiles would corrupt the swizzle
    mbar_init(q_full, 1);
    for (int s = 0; s < ST; ++s) { mbar_init(&k_full[s], 1); mbar_init(&kv_empty[s], 1); }
    for (int b = 0; b < 2; ++b) { mbar_init(&s_full[b], 1); mbar_init(&s_free[b], 4); mbar_init(&p_full[b], 4); mbar_init(&o_done[b], 1); }
    mbar_init(v_clean, 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_base_slot)), "r"(LT_TMEM_COLS) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = tmem_base_slot;
  pdl_wait();                       // queries and this step's cached vectors come from the previous kernels
  pdl_launch_dependents();

  if (warp == 0) {
    if (lane == 0) {
      // a query box is tokens_per_tile x heads rows; the rows left over of the 128 are never read back
      mbar_expect_tx(q_full, (uint32_t)(p.tokens_per_tile * p.heads * 128 * slabs));
      for (int h = 0; h < slabs; ++h) lt_load_3d(q_s + h * LT_Q_SLAB, &map_q, h * 64, 0, tok0 + t_first, q_full);
      bool ok = true;
#pragma unroll 1
      for (int j = 0; j < nb && ok; ++j) {
        const int s = j % ST;
        ok = mbar_wait(&kv_empty[s], ((j / ST) & 1u) ^ 1u, &abort_flag);
        if (!ok) break;
        const int key0 = (b_lo + j) * LT_KEYS;
        // a block beyond the pages the request holds reads page -1: out of range, zero-filled
        const int page = (key0 >> p.page_shift) < p.max_pages ? p.block_table[(long long)slot * p.max_pages + (key0 >> p.page_shift)] : -1;
        const int in_page = key0 & (p.page_size - 1);
        mbar_expect_tx(&k_full[s], (uint32_t)stage_bytes);
        for (int h = 0; h < slabs; ++h) lt_load_3d(kv_s + s * stage_bytes + h * LT_K_SLAB, &map_k, h * 64, in_page, page, &k_full[s]);
      }
    }
    __syncwarp();
    {
      const int j = nb - 1, s = j % ST;
      int done = lane == 0 ? (int)mbar_wait(&k_full[s], (j / ST) & 1u, &abort_flag) : 0;
      done = __shfl_sync(0xffffffffu, done, 0);
      const int first_row = pos_last - (b_lo + j) * LT_KEYS + 1;      // 1..64
      if (done && first_row < LT_KEYS) {
        unsigned char* v_dst = kv_s + s * stage_bytes + (v0 / 64) * LT_K_SLAB;
        const int per_slab = (LT_KEYS - first_row) * 8;               // 16-byte pieces
        for (int i = lane; i < per_slab * value_slabs; i += 32) {
          const int h = i / per_slab, o = i - h * per_slab;
          *reinterpret_cast<uint4*>(v_dst + h * LT_K_SLAB + first_row * 128 + o * 16) = make_uint4(0, 0, 0, 0);
        }
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
      }
      __syncwarp();
      if (lane == 0 && done) mbar_arrive(v_clean);
    }
  } else if (warp == 1) {
    // the whole warp walks the loop; one elected lane issues the MMAs and commits
    constexpr uint32_t idesc_s = make_idesc(LT_ROWS, LT_KEYS);               // A, B K-major
    constexpr uint32_t idesc_o = make_idesc(LT_ROWS, 64) | (1u << 16);       // B (values) MN-major, 64 columns per MMA
    bool ok = true;
    auto wait = [&](uint64_t* bar, uint32_t parity) {
      if (ok) ok = __all_sync(0xffffffffu, mbar_wait(bar, parity, &abort_flag));
      return ok;
    };
    const uint64_t q_desc = make_desc(smem_u32(q_s)), k_desc = make_desc(smem_u32(kv_s)), v_desc = lt_desc_mn(smem_u32(kv_s + (v0 / 64) * LT_K_SLAB));
    const int k_steps = p.dk / 16;
    auto issue_s = [&](int j) {
      const int s = j % ST, b = j & 1;
      if (j >= 2 && !wait(&s_free[b], ((j - 2) >> 1) & 1u)) return;
      if (!wait(&k_full[s], (j / ST) & 1u)) return;
      tc_fence_after();
      if (elect_one()) {
        const uint64_t dk = k_desc + (uint64_t)(s * (stage_bytes >> 4));         // descriptor addresses count 16-byte units
        for (int ks = 0; ks < k_steps; ++ks) {
          // 16 dimensions = 32 bytes further along a slab's rows; the next slab after four of them
          const uint32_t in_slab = 2 * (ks & 3);
          tc_mma(tmem_base + LT_S_COL + b * LT_KEYS, q_desc + (uint64_t)((ks >> 2) * (LT_Q_SLAB >> 4) + in_slab),
                 dk + (uint64_t)((ks >> 2) * (LT_K_SLAB >> 4) + in_slab), idesc_s, ks != 0);
        }
        tc_commit(&s_full[b]);
      }
      __syncwarp();
    };
    auto issue_pv = [&](int j) {
      const int s = j % ST, b = j & 1;
      if (!wait(&p_full[b], (j >> 1) & 1u)) return;
      if (j == nb - 1 && !wait(v_clean, 0)) return;
      tc_fence_after();
      if (elect_one()) {
        const uint64_t dv = v_desc + (uint64_t)(s * (stage_bytes >> 4));
#pragma unroll
        for (int kk = 0; kk < LT_KEYS / 16; ++kk)
          // P: 16 keys = 8 columns of packed bfloat16 further; values: 16 keys = two 8-row groups of 1024 bytes
          for (int h = 0; h < value_slabs; ++h)
            lt_mma_ts(tmem_base + LT_O_COL + h * 64, tmem_base + LT_P_COL + b * (LT_KEYS / 2) + kk * 8,
                      dv + (uint64_t)(h * (LT_K_SLAB >> 4) + kk * (2048 >> 4)), idesc_o, (j > 0 || kk != 0) ? 1u : 0u);
        tc_commit(&o_done[b]);
        tc_commit(&kv_empty[s]);
      }
      __syncwarp();
    };
    if (wait(q_full, 0)) issue_s(0);
#pragma unroll 1
    for (int j = 0; j < nb && ok; ++j) {
      if (ST > 1 && j + 1 < nb) issue_s(j + 1);
      if (ok) issue_pv(j);
      if (ST == 1 && j + 1 < nb && ok) issue_s(j + 1);
    }
  } else if (warp >= 4) {
    const int quad = warp & 3;                              // the 32 lanes of tensor memory this warp may touch
    const int row = quad * 32 + lane;                       // tile row = lane of tensor memory
    const bool valid = row < t_count * p.heads;
    const int tk = valid ? row / p.heads : t_count - 1;     // rows past the tile's tokens compute like its last one and are never stored
    const int head = valid ? row - tk * p.heads : 0;
    const int pos = pos_first + tk;
    const uint32_t lane_addr = tmem_base + ((uint32_t)(quad * 32) << 16);
    const uint32_t o_addr = lane_addr + LT_O_COL;
    const float c_log2 = p.scale_log2;
    const int key_min = p.window > 0 ? pos - p.window + 1 : -(1 << 30);
    float m_run = -INFINITY, l_run = 0.f;
    bool ok = true;
    auto wait_all = [&](uint64_t* bar, uint32_t parity) {   // every lane of a warp takes the same path, also when a wait gives up
      return __all_sync(0xffffffffu, mbar_wait(bar, parity, &abort_flag)) != 0;
    };
#pragma unroll 1
    for (int j = 0; j < nb && ok; ++j) {
      const int key0 = (b_lo + j) * LT_KEYS, b = j & 1;
      ok = wait_all(&s_full[b], (j >> 1) & 1u);
      if (!ok) break;
      tc_fence_after();
      float v[LT_KEYS];
#pragma unroll
      for (int ch = 0; ch < LT_KEYS / 32; ++ch)
        tc_ld32(lane_addr + LT_S_COL + b * LT_KEYS + ch * 32, *reinterpret_cast<uint32_t(*)[32]>(&v[ch * 32]));
      tc_wait_ld();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&s_free[b]);
      if (__any_sync(0xffffffffu, key0 + LT_KEYS - 1 > pos || key0 < key_min)) {
        const int hi = pos - key0, lo = key_min - key0;
#pragma unroll
        for (int i = 0; i < LT_KEYS; ++i) v[i] = (i <= hi && i >= lo) ? v[i] : -INFINITY;
      }
      float mx[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int i = 0; i < LT_KEYS; i += 4)
#pragma unroll
        for (int e = 0; e < 4; ++e) mx[e] = fmaxf(mx[e], v[i + e]);
      // (a negative scale would turn the largest score into the smallest exponent; the launcher refuses it)
      const float m_new = fmaxf(fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3])), m_run);
      const bool grow = (m_new - m_run) * c_log2 > LT_RESCALE_LOG2;          // always from -inf to a number
      if (__any_sync(0xffffffffu, grow)) {
        const float m_use = m_new == -INFINITY ? 0.f : m_new;
        const float alpha = lt_exp2((m_run - m_use) * c_log2);               // 0 from -inf
        m_run = m_new;
        l_run *= alpha;
        if (j > 0) {                                        // O holds the blocks before this one: rescale its rows
          ok = wait_all(&o_done[b ^ 1], ((j - 1) >> 1) & 1u);
          if (!ok) break;
          tc_fence_after();
          for (int ch = 0; ch < 2 * value_slabs; ++ch) {
            uint32_t o[32];
            tc_ld32(o_addr + ch * 32, o);
            tc_wait_ld();
#pragma unroll
            for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * alpha);
            lt_st32(o_addr + ch * 32, o);
          }
        }
      }
      if (j >= 2) {                                         // the MMAs that read this P buffer must be through with it
        ok = wait_all(&o_done[b], ((j - 2) >> 1) & 1u);
        if (!ok) break;
        tc_fence_after();
      }
      const float neg_mc = m_run == -INFINITY ? 0.f : -m_run * c_log2;
      float ls[2] = {0.f, 0.f};
      uint32_t packed[32];
#pragma unroll
      for (int i = 0; i < LT_KEYS; i += 2) {
        const float e0 = lt_exp2(fmaf(v[i], c_log2, neg_mc)), e1 = lt_exp2(fmaf(v[i + 1], c_log2, neg_mc));
        ls[0] += e0;
        ls[1] += e1;
        const __nv_bfloat162 w = __floats2bfloat162_rn(e0, e1);
        packed[i / 2] = *reinterpret_cast<const uint32_t*>(&w);
      }
      lt_st32(lane_addr + LT_P_COL + b * (LT_KEYS / 2), packed);
      l_run += ls[0] + ls[1];
      lt_wait_st();                                         // P (and a rescaled O) must have landed before the MMA is told
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_full[b]);
    }
    if (ok) {
      ok = wait_all(&o_done[(nb - 1) & 1], ((nb - 1) >> 1) & 1u);
      tc_fence_after();
    }
    if (ok) {
      float inv;
      if (p.sink != nullptr) {                              // against the larger of the two exponents
        const float m2 = m_run * c_log2, s2 = p.sink[head] * 1.4426950408889634f, top = fmaxf(m2, s2);
        const float shrink = lt_exp2(m2 - top);
        inv = shrink / fmaf(l_run, shrink, lt_exp2(s2 - top));
      } else {
        inv = l_run > 0.f ? 1.f / l_run : 0.f;
      }
      __nv_bfloat16* dst = p.out + (long long)(tok0 + t_first + tk) * p.ld_o + (long long)head * p.dv + v0;
      for (int ch = 0; ch < 2 * value_slabs; ++ch) {
        uint32_t o[32];
        tc_ld32(o_addr + ch * 32, o);
        tc_wait_ld();
        if (valid) {
#pragma unroll
          for (int d = 0; d < 32; d += 8) {
            uint32_t w[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const __nv_bfloat162 t2 = __floats2bfloat162_rn(__uint_as_float(o[d + 2 * e]) * inv, __uint_as_float(o[d + 2 * e + 1]) * inv);
              w[e] = *reinterpret_cast<const uint32_t*>(&t2);
            }
            *reinterpret_cast<uint4*>(dst + ch * 32 + d) = make_uint4(w[0], w[1], w[2], w[3]);
          }
        }
      }
    }
  }

  tc_fence_before();
  __syncthreads();
  if (abort_flag) {                                         // let copies in flight land before the shared memory goes
#pragma unroll 1
    for (int i = 0; i < 400; ++i) __nanosleep(1000);
    if (threadIdx.x == 0 && status != nullptr) atomicExch(status, 2);
    __syncthreads();
  }
  if (warp == 1) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(LT_TMEM_COLS) : "memory");
  }
}

int lt_stages(int slabs) {
  const int room = (LT_SMEM_MAX - LT_BAR_BYTES - slabs * LT_Q_SLAB) / (slabs * LT_K_SLAB);
  return room > LT_MAX_STAGES ? LT_MAX_STAGES : room;
}

int lt_map(CUtensorMap* map, const void* base, const cuuint64_t (&dims)[3], const cuuint64_t (&strides)[2], const cuuint32_t (&box)[3]) {
  EncodeTiledFn fn = encode_fn();
  if (!fn) return hfee_fail(HFEE_ERR_CUDA, "latent_attention_tc: the driver has no cuTensorMapEncodeTiled");
  cuuint32_t elem[3] = {1, 1, 1};
  CUresult rc = fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, elem,
                   CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                   CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  if (rc != CUDA_SUCCESS) return hfee_fail(HFEE_ERR_CUDA, "latent_attention_tc: cuTensorMapEncodeTiled failed with %d", (int)rc);
  return HFEE_OK;
}

}  // namespace

// 1 if the kernel takes these sizes: at most 128 heads, a key size that is a multiple of 16 and leaves room for a key block
// beside the query tile, a value size that is a multiple of 64 and at most the key size, power-of-two pages of 64 and more.
HFEE_API int hfee_latent_attention_tc_supports(int heads, int dk, int dv, int page_size) {
  if (heads < 1 || heads > LT_ROWS || dk < 16 || dk % 16 != 0 || dv < 64 || dv % 64 != 0 || dv > dk) return 0;
  if (page_size < LT_KEYS || (page_size & (page_size - 1)) != 0) return 0;
  return lt_stages((dk + 63) / 64) >= 1 ? 1 : 0;
}

// Arguments as hfee_latent_attention_mma's; scale must be positive.
HFEE_API int hfee_latent_attention_tc(const void* q, long long ld_q, const void* pool, int num_pages, const int* block_table,
                                      int max_pages, int page_size, const int* cu_tokens, const int* slots,
                                      const int* context_before, void* out, long long ld_o, int n_tokens, int requests, int max_new,
                                      int heads, int dk, int dv, float scale, int window, const float* sink, int* status,
                                      cudaStream_t stream) {
  if (requests == 0 || max_new == 0 || n_tokens == 0) return HFEE_OK;
  HFEE_REQUIRE(hfee_latent_attention_tc_supports(heads, dk, dv, page_size), "latent_attention_tc: sizes %d heads, %d key, %d value dimensions, pages of %d are not taken", heads, dk, dv, page_size);
  HFEE_REQUIRE(ld_q % 8 == 0 && ld_o % 8 == 0 && (uintptr_t)q % 16 == 0 && (uintptr_t)out % 16 == 0 && (uintptr_t)pool % 16 == 0,
               "latent_attention_tc: queries, cache and outputs must be 16-byte aligned");
  HFEE_REQUIRE(requests <= 65535 && max_new > 0 && num_pages > 0 && window >= 0 && scale > 0.f && status != nullptr, "latent_attention_tc: bad batch, window or scale");
  LatentTcParams p{};
  p.out = (__nv_bfloat16*)out; p.ld_o = ld_o;
  p.block_table = block_table; p.max_pages = max_pages; p.page_size = page_size;
  while ((1 << p.page_shift) < page_size) ++p.page_shift;
  p.cu_tokens = cu_tokens; p.slots = slots; p.context_before = context_before;
  p.heads = heads; p.dk = dk; p.dv = dv;
  p.slabs = (dk + 63) / 64;
  p.stages = lt_stages(p.slabs);
  p.scale_log2 = scale * 1.4426950408889634f;
  p.window = window;
  p.tokens_per_tile = LT_ROWS / heads;
  p.q_tiles = (max_new + p.tokens_per_tile - 1) / p.tokens_per_tile;
  p.sink = sink;
  HFEE_REQUIRE(p.q_tiles <= 65535, "latent_attention_tc: a portion of %d tokens exceeds one launch", max_new);
  CUtensorMap mq, mk;
  {
    const cuuint64_t dims[3] = {(cuuint64_t)dk, (cuuint64_t)heads, (cuuint64_t)n_tokens};
    const cuuint64_t strides[2] = {(cuuint64_t)dk * 2, (cuuint64_t)ld_q * 2};
    const cuuint32_t box[3] = {64, (cuuint32_t)heads, (cuuint32_t)p.tokens_per_tile};
    const int rc = lt_map(&mq, q, dims, strides, box);
    if (rc != HFEE_OK) return rc;
  }
  {
    const cuuint64_t dims[3] = {(cuuint64_t)dk, (cuuint64_t)page_size, (cuuint64_t)num_pages};
    const cuuint64_t strides[2] = {(cuuint64_t)dk * 2, (cuuint64_t)page_size * dk * 2};
    const cuuint32_t box[3] = {64, 64, 1};
    const int rc = lt_map(&mk, pool, dims, strides, box);
    if (rc != HFEE_OK) return rc;
  }
  const size_t smem = (size_t)p.slabs * LT_Q_SLAB + (size_t)p.stages * p.slabs * LT_K_SLAB + LT_BAR_BYTES;
  static bool configured = false;
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(latent_attention_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, LT_SMEM_MAX);
    if (e != cudaSuccess) return hfee_fail(HFEE_ERR_CUDA, "latent_attention_tc: cannot get %d bytes of shared memory: %s", LT_SMEM_MAX, cudaGetErrorString(e));
    configured = true;
  }
  hfee_launch(latent_attention_tc_kernel, dim3((unsigned)((dv + LT_VALUES - 1) / LT_VALUES), (unsigned)p.q_tiles, (unsigned)requests), dim3(256),
              smem, stream, mq, mk, p, status);
  return hfee_check_launch("latent_attention_tc");
}
