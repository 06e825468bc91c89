// The state-space scan with one decay per head and token (see gated_recurrence.cu, "step sizes") for prompt portions, on
// mma.sync tiles: bfloat16 x, B and C, float32 step sizes, decays and states.
//
//   S_t = e^(a_t) S_(t-1) + dt_t B_t x_t^T,   y_t = S_t^T C_t + D x_t,   dt_t = softplus(step_t + bias), a_t = -exp(A_log) dt_t
//
// A request's tokens go in runs of HS_T.  With s_t the sum of a over the run's tokens up to t, a run of n tokens is
//
//   y_t   = e^(s_t) S_in^T C_t + sum_(u <= t) e^(s_t - s_u) dt_u (C_t . B_u) x_u + D x_t
//   S_out = e^(s_n) S_in + sum_u e^(s_n - s_u) dt_u B_u x_u^T
//
// which is the recurrence written out; every exponent is at most zero, so nothing overflows and a strong decay becomes zero.
// Three kernels: (1) head_scan_gates: dt_t and s_t (in log2 units) of every token and head; (2) head_scan_states: per
// (request, head, 32 columns of x) the walk over the runs with the state in the MMA accumulators; the state in front of
// every run goes to the workspace, the state behind the last one to the request's slot; (3) head_scan_outputs: all runs at
// once.  C . B is shared by the heads of a group, so a block of (3) takes several heads of one.
//
// x, B and C enter the products as they are.  What is float32 (the weighted x, the weights times C . B, the state) enters as
// the sum of two bfloat16 numbers, the value rounded and what the rounding left, each with a product of its own; sums are
// float32.  (2) computes S transposed, so that its accumulators, packed in pairs, are the very B fragments that (3) wants:
// the workspace holds them in that order, one 16-byte piece (two halves, high and low) per lane.
#include "common.cuh"
#include "mma_tiles.cuh"

namespace {

constexpr int HS_T = 64;            // tokens of a run
constexpr int HS_WARPS = 8;         // of a block of outputs
constexpr int HS_THREADS = HS_WARPS * 32;
constexpr int HS_COLS_STATES = 32;  // columns of x per block of the walk
constexpr int HS_COLS_OUT = 64;     // and of the outputs
constexpr int HS_PAD = 8;
constexpr float HS_LOG2E = 1.4426950408889634f;

struct HeadScanArgs {
  const bf16* x; const bf16* b; const bf16* c;
  long long ld;
  const bf16* step;
  long long ld_step;
  const float* dt_bias; const float* a_log; const float* d_skip;
  float* state;                 // [slots, heads, n_state, vdim]
  const int* cu_tokens; const int* slots;
  float* out;
  long long ld_o;
  float* gate_s; float* gate_dt;          // [heads][n_tokens]
  uint4* carried;                         // [runs][heads][tiles of 16 state entries][tiles of 8 columns][32 lanes]
  int requests, n_tokens, heads, groups, n_state, vdim, ctiles, write_state, heads_per_block;
};

__device__ __forceinline__ int hs_runs(int count) { return (count + HS_T - 1) / HS_T; }

__device__ __forceinline__ bool hs_find_run(const int* __restrict__ cu_tokens, int requests, int number, int* req, int* run) {
  int base = 0;
  for (int r = 0; r < requests; ++r) {
    const int c = hs_runs(cu_tokens[r + 1] - cu_tokens[r]);
    if (number < base + c) { *req = r; *run = number - base; return true; }
    base += c;
  }
  return false;
}

__device__ __forceinline__ float hs_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void hs_copy16(void* smem, const void* gmem, bool valid) {
  const unsigned s = (unsigned)__cvta_generic_to_shared(smem);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(s), "l"(gmem), "r"(valid ? 16 : 0));
}
__device__ __forceinline__ void hs_copy4(void* smem, const void* gmem, bool valid) {
  const unsigned s = (unsigned)__cvta_generic_to_shared(smem);
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;\n" ::"r"(s), "l"(gmem), "r"(valid ? 4 : 0));
}
__device__ __forceinline__ void hs_commit() { asm volatile("cp.async.commit_group;\n" ::); }
__device__ __forceinline__ void hs_wait_all() { asm volatile("cp.async.wait_group 0;\n" ::); }

// a pair of float32 numbers as two packed pairs of bfloat16: rounded, and what the rounding left
__device__ __forceinline__ void split_pair(float a, float b, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  const __nv_bfloat162 l = __floats2bfloat162_rn(a - __bfloat162float(h.x), b - __bfloat162float(h.y));
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}

// ------------------------------------------------------------------------------------------ (1) gates
constexpr int HS_GATE_HEADS = 8;    // heads per block, one per warp

__global__ void __launch_bounds__(HS_GATE_HEADS * 32)
head_scan_gates_kernel(HeadScanArgs p) {
  __shared__ float dt_s[HS_T][HS_GATE_HEADS + 1];
  int req = 0, run = 0;
  const bool mine = hs_find_run(p.cu_tokens, p.requests, blockIdx.y, &req, &run);
  const int h0 = blockIdx.x * HS_GATE_HEADS, lane = threadIdx.x & 31, j = threadIdx.x >> 5;
  const int own = h0 + (threadIdx.x % HS_GATE_HEADS);
  const float bias = own < p.heads ? p.dt_bias[own] : 0.f;
  const float rate = h0 + j < p.heads ? -expf(p.a_log[h0 + j]) * HS_LOG2E : 0.f;
  pdl_wait();
  pdl_launch_dependents();
  if (!mine) return;
  const int begin = p.cu_tokens[req] + run * HS_T, n = min(HS_T, p.cu_tokens[req + 1] - begin);
#pragma unroll
  for (int i = 0; i < HS_T / 32; ++i) {
    const int t = threadIdx.x / HS_GATE_HEADS + i * 32;
    float dt = 0.f;
    if (t < n && own < p.heads) {
      const float z = __bfloat162float(p.step[(long long)(begin + t) * p.ld_step + own]) + bias;
      dt = fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)));
    }
    dt_s[t][threadIdx.x % HS_GATE_HEADS] = dt;
  }
  __syncthreads();
  if (h0 + j >= p.heads) return;
  const float d0 = dt_s[2 * lane][j], d1 = dt_s[2 * lane + 1][j];
  const float a0 = rate * d0, a1 = rate * d1;
  float sum = a0 + a1;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float before = __shfl_up_sync(0xffffffffu, sum, o);
    if (lane >= o) sum += before;
  }
  float front = __shfl_up_sync(0xffffffffu, sum, 1);
  if (lane == 0) front = 0.f;
  const long long at = (long long)(h0 + j) * p.n_tokens + begin + 2 * lane;
  if (2 * lane < n) { p.gate_s[at] = front + a0; p.gate_dt[at] = d0; }
  if (2 * lane + 1 < n) { p.gate_s[at + 1] = front + a0 + a1; p.gate_dt[at + 1] = d1; }
}

// ------------------------------------------------------------------------------------------ (2) states
// Warps 0..7 keep the state (transposed) and multiply: warp w has the columns 16 (w & 1) .. + 15 of the block's 32 and a
// quarter of the state entries.  Warps 8..11 bring the runs in (three in flight) and weigh the next run's x while this
// run is multiplied; one barrier a run.
constexpr int HS_MUL_WARPS = 8, HS_IN_WARPS = 4, HS_IN = HS_IN_WARPS * 32;
constexpr int HS_STATES_THREADS = (HS_MUL_WARPS + HS_IN_WARPS) * 32;

template <int NP> struct StatesCfg {
  static constexpr int TILES = NP / 16;                    // tiles of 16 state entries
  static constexpr int MINE = TILES >= 4 ? TILES / 4 : 1;  // per warp
  static constexpr int LDB = NP + HS_PAD, LDX = HS_COLS_STATES + HS_PAD;
  static constexpr int STAGE = HS_T * (LDB + LDX) * 2 + 2 * HS_T * 4;     // bytes: B, x, s, dt of one run
  static constexpr int SMEM = 3 * STAGE + 4 * HS_T * LDX * 2;             // + the weighted x of two runs, high and low
};

template <int NP>
__global__ void __launch_bounds__(HS_STATES_THREADS)
head_scan_states_kernel(HeadScanArgs p) {
  using C = StatesCfg<NP>;
  extern __shared__ __align__(16) unsigned char smem_raw[];
  const int head = blockIdx.x, req = blockIdx.y, c0 = blockIdx.z * HS_COLS_STATES;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int begin = p.cu_tokens[req], count = p.cu_tokens[req + 1] - begin;
  const int slot = p.slots[req];
  int first_run = 0;
  for (int r = 0; r < req; ++r) first_run += hs_runs(p.cu_tokens[r + 1] - p.cu_tokens[r]);
  const int group = head / (p.heads / p.groups);
  pdl_wait();
  pdl_launch_dependents();
  if (count <= 0) return;
  bf16* wx = reinterpret_cast<bf16*>(smem_raw + 3 * C::STAGE);            // [2 runs][high, low][HS_T][LDX]
  auto b_of = [&](int run) { return reinterpret_cast<bf16*>(smem_raw + (run % 3) * C::STAGE); };
  auto x_of = [&](int run) { return b_of(run) + HS_T * C::LDB; };
  auto s_of = [&](int run) { return reinterpret_cast<float*>(x_of(run) + HS_T * C::LDX); };
  auto wx_of = [&](int run, int low) { return wx + ((run & 1) * 2 + low) * HS_T * C::LDX; };
  const int runs = hs_runs(count);
  const int tid = threadIdx.x - HS_MUL_WARPS * 32;         // among the warps that bring the runs in

  auto load = [&](int run) {                               // always a group, also when there is no such run
    if (run < runs) {
      const int row0 = begin + run * HS_T, n = min(HS_T, count - run * HS_T);
      bf16* bd = b_of(run);
      bf16* xd = x_of(run);
      float* sd = s_of(run);
#pragma unroll
      for (int e = tid; e < HS_T * (NP / 8); e += HS_IN) {
        const int s = e / (NP / 8), k = (e % (NP / 8)) * 8;
        const bool ok = s < n && k < p.n_state;
        hs_copy16(bd + s * C::LDB + k, ok ? p.b + (long long)(row0 + s) * p.ld + group * p.n_state + k : p.b, ok);
      }
#pragma unroll
      for (int e = tid; e < HS_T * (HS_COLS_STATES / 8); e += HS_IN) {
        const int s = e / (HS_COLS_STATES / 8), c = (e % (HS_COLS_STATES / 8)) * 8;
        const bool ok = s < n && c0 + c < p.vdim;
        hs_copy16(xd + s * C::LDX + c, ok ? p.x + (long long)(row0 + s) * p.ld + (long long)head * p.vdim + c0 + c : p.x, ok);
      }
      const int s = tid % HS_T;
      const float* src = (tid < HS_T ? p.gate_s : p.gate_dt) + (long long)head * p.n_tokens + row0;
      hs_copy4(sd + tid, s < n ? src + s : p.gate_s, s < n);              // s first, dt behind it
    }
    hs_commit();
  };
  auto weigh = [&](int run) {
    if (run >= runs) return;
    const int n = min(HS_T, count - run * HS_T);
    const float* ss = s_of(run);
    const float* sdt = ss + HS_T;
    const bf16* xs = x_of(run);
    const float s_last = ss[n - 1];
#pragma unroll
    for (int e = tid; e < HS_T * (HS_COLS_STATES / 8); e += HS_IN) {
      const int s = e / (HS_COLS_STATES / 8), c = (e % (HS_COLS_STATES / 8)) * 8;
      const float w = s < n ? hs_exp2(s_last - ss[s]) * sdt[s] : 0.f;
      const uint4 raw = *reinterpret_cast<const uint4*>(xs + s * C::LDX + c);
      const uint32_t in[4] = {raw.x, raw.y, raw.z, raw.w};
      uint32_t hi[4], lo[4];
#pragma unroll
      for (int i = 0; i < 4; ++i)
        split_pair(__uint_as_float(in[i] << 16) * w, __uint_as_float(in[i] & 0xffff0000u) * w, hi[i], lo[i]);
      *reinterpret_cast<uint4*>(wx_of(run, 0) + s * C::LDX + c) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
      *reinterpret_cast<uint4*>(wx_of(run, 1) + s * C::LDX + c) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
    }
  };
  auto landed = [&]() {                                    // all copies but the newest run's, of every thread that copies
    asm volatile("cp.async.wait_group 1;\n" ::);
    asm volatile("bar.sync 1, %0;" ::"n"(HS_IN) : "memory");
  };

  if (warp >= HS_MUL_WARPS) {
    load(0);
    load(1);
    landed();
    weigh(0);
    __syncthreads();
    for (int run = 0; run < runs; ++run) {
      load(run + 2);                                       // its place was used up before the last barrier
      landed();
      weigh(run + 1);
      __syncthreads();
    }
    hs_wait_all();
    return;
  }

  const int m0 = (warp & 1) * 16, tile0 = (warp >> 1) * C::MINE;
  const bool active = tile0 < C::TILES;
  float acc[2 * C::MINE][4];                               // [8 state entries]: S transposed, 16 columns
  float* S_g = p.state + ((long long)slot * p.heads + head) * p.n_state * p.vdim;
#pragma unroll
  for (int j = 0; j < 2 * C::MINE; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int c = c0 + m0 + g + (i >= 2 ? 8 : 0), k = tile0 * 16 + j * 8 + 2 * t + (i & 1);
      acc[j][i] = active && c < p.vdim && k < p.n_state ? S_g[(long long)k * p.vdim + c] : 0.f;
    }
  __syncthreads();
  for (int run = 0; run < runs; ++run) {
    if (active) {
      const int n = min(HS_T, count - run * HS_T);
      const float decay = hs_exp2(s_of(run)[n - 1]);
      // the state in front of the run, as B fragments
      uint4* dst = p.carried + ((long long)(first_run + run) * p.heads + head) * (C::TILES * p.ctiles * 32) + lane;
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int ct = (c0 + m0) / 8 + half;
        if (ct >= p.ctiles) continue;
#pragma unroll
        for (int j = 0; j < C::MINE; ++j) {
          uint4 f;
          split_pair(acc[2 * j][2 * half], acc[2 * j][2 * half + 1], f.x, f.z);
          split_pair(acc[2 * j + 1][2 * half], acc[2 * j + 1][2 * half + 1], f.y, f.w);
          dst[((tile0 + j) * p.ctiles + ct) * 32] = f;
        }
      }
#pragma unroll
      for (int j = 0; j < 2 * C::MINE; ++j)
#pragma unroll
        for (int i = 0; i < 4; ++i) acc[j][i] *= decay;
      const bf16* bs = b_of(run);
#pragma unroll
      for (int ks = 0; ks < HS_T / 16; ++ks) {
        uint32_t ah[4], al[4];
        load_a_trans(ah, wx_of(run, 0), C::LDX, m0, ks * 16, lane);
        load_a_trans(al, wx_of(run, 1), C::LDX, m0, ks * 16, lane);
#pragma unroll
        for (int j = 0; j < C::MINE; ++j) {
          uint32_t b[4];
          load_b_pair_trans(b, bs, C::LDB, (tile0 + j) * 16, ks * 16, lane);
          mma_bf16(acc[2 * j], ah, b[0], b[1]);
          mma_bf16(acc[2 * j + 1], ah, b[2], b[3]);
          mma_bf16(acc[2 * j], al, b[0], b[1]);
          mma_bf16(acc[2 * j + 1], al, b[2], b[3]);
        }
      }
    }
    __syncthreads();
  }
  if (!p.write_state || !active) return;
#pragma unroll
  for (int j = 0; j < 2 * C::MINE; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int c = c0 + m0 + g + (i >= 2 ? 8 : 0), k = tile0 * 16 + j * 8 + 2 * t + (i & 1);
      if (c < p.vdim && k < p.n_state) S_g[(long long)k * p.vdim + c] = acc[j][i];
    }
}

// ------------------------------------------------------------------------------------------ (3) outputs
// C . B and the weights made of it: warp w has the run's tokens 16 (w & 3) .. + 15 against every second tile of 16 tokens
// in front of them (from w >> 2 on); they meet in shared memory.  Outputs: warp w has the columns 16 (w & 3) .. + 15 of two
// of the run's four tiles of 16 tokens, the outer ones or the inner ones (as many tiles in front of them either way).
template <int NP> struct OutCfg {
  static constexpr int TILES = NP / 16;
  static constexpr int LDB = NP + HS_PAD, LDX = HS_COLS_OUT + HS_PAD, LDP = HS_T + HS_PAD;
  static constexpr int X_STAGE = HS_T * LDX * 2 + 2 * HS_T * 4;           // bytes: x, s, dt of one head
  static constexpr int B_BYTES = HS_T * LDB * 2, P_BYTES = 2 * HS_T * LDP * 2;
  static constexpr int SHARED = B_BYTES > P_BYTES ? B_BYTES : P_BYTES;    // B, later the weights (high and low)
  static constexpr int SMEM = HS_T * LDB * 2 + SHARED + 2 * X_STAGE;
};

constexpr int HS_OUT_BLOCKS = 2;     // resident per SM

template <int NP>
__global__ void __launch_bounds__(HS_THREADS, HS_OUT_BLOCKS)
head_scan_outputs_kernel(HeadScanArgs p) {
  using C = OutCfg<NP>;
  extern __shared__ __align__(16) unsigned char smem_raw[];
  const int head0 = blockIdx.y * p.heads_per_block, c0 = blockIdx.z * HS_COLS_OUT;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  int req = 0, run = 0;
  const bool mine = hs_find_run(p.cu_tokens, p.requests, blockIdx.x, &req, &run);
  pdl_wait();
  pdl_launch_dependents();
  if (!mine) return;
  const int begin = p.cu_tokens[req] + run * HS_T, n = min(HS_T, p.cu_tokens[req + 1] - begin);
  const int group = head0 / (p.heads / p.groups);
  bf16* cs = reinterpret_cast<bf16*>(smem_raw);            // [HS_T][LDB]
  bf16* bs = cs + HS_T * C::LDB;                           // [HS_T][LDB]
  bf16* w_hi = bs;                                         // [HS_T][LDP], once C . B is known
  bf16* w_lo = w_hi + HS_T * C::LDP;
  unsigned char* stages = smem_raw + HS_T * C::LDB * 2 + C::SHARED;
  auto x_of = [&](int st) { return reinterpret_cast<bf16*>(stages + st * C::X_STAGE); };
  auto s_of = [&](int st) { return reinterpret_cast<float*>(x_of(st) + HS_T * C::LDX); };
  auto load_head = [&](int head, int st) {
    bf16* xd = x_of(st);
    float* sd = s_of(st);
#pragma unroll
    for (int e = tid; e < HS_T * (HS_COLS_OUT / 8); e += HS_THREADS) {
      const int s = e / (HS_COLS_OUT / 8), c = (e % (HS_COLS_OUT / 8)) * 8;
      const bool ok = s < n && c0 + c < p.vdim;
      hs_copy16(xd + s * C::LDX + c, ok ? p.x + (long long)(begin + s) * p.ld + (long long)head * p.vdim + c0 + c : p.x, ok);
    }
    if (tid < 2 * HS_T) {
      const int s = tid % HS_T;
      const float* src = (tid < HS_T ? p.gate_s : p.gate_dt) + (long long)head * p.n_tokens + begin;
      hs_copy4(sd + tid, s < n ? src + s : p.gate_s, s < n);
    }
    hs_commit();
  };
#pragma unroll
  for (int e = tid; e < HS_T * (NP / 8); e += HS_THREADS) {
    const int s = e / (NP / 8), k = (e % (NP / 8)) * 8;
    const bool ok = s < n && k < p.n_state;
    const long long at = (long long)(begin + s) * p.ld + group * p.n_state + k;
    hs_copy16(cs + s * C::LDB + k, ok ? p.c + at : p.c, ok);
    hs_copy16(bs + s * C::LDB + k, ok ? p.b + at : p.b, ok);
  }
  load_head(head0, 0);
  hs_wait_all();
  __syncthreads();

  // C . B, for all heads of the block
  const int quarter = warp & 3, side = warp >> 2;
  const int r0 = quarter * 16;
  float cb[2][2][4];                                       // tiles side and side + 2 of 16 tokens, by 8
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int q = 0; q < 2; ++q) cb[i][q][0] = cb[i][q][1] = cb[i][q][2] = cb[i][q][3] = 0.f;
#pragma unroll
  for (int kk = 0; kk < C::TILES; ++kk) {
    uint32_t a[4];
    load_a(a, cs, C::LDB, r0, kk * 16, lane);
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int kt = side + 2 * i;
      if (kt <= quarter) {
        uint32_t b[4];
        load_b_pair(b, bs, C::LDB, kt * 16, kk * 16, lane);
        mma_bf16(cb[i][0], a, b[0], b[1]);
        mma_bf16(cb[i][1], a, b[2], b[3]);
      }
    }
  }
  __syncthreads();                                         // B is used up: its place takes the weights
  const int ct0 = c0 / 8 + 2 * quarter;                    // the warp's two tiles of 8 columns
  const int cts = min(2, p.ctiles - ct0);                  // 0 or less: none of them exists
  const int row_tile[2] = {side, 3 - side};
  for (int hh = 0; hh < p.heads_per_block; ++hh) {
    const int head = head0 + hh, st = hh & 1;
    if (hh + 1 < p.heads_per_block) load_head(head + 1, st ^ 1);
    // the state in front of the run: requested before the weights are computed
    const uint4* S = p.carried + ((long long)(blockIdx.x) * p.heads + head) * (C::TILES * p.ctiles * 32) + ct0 * 32 + lane;
    constexpr int AHEAD = C::TILES < 4 ? C::TILES : 4;
    uint4 f[AHEAD][2];
#pragma unroll
    for (int kk = 0; kk < AHEAD; ++kk)
#pragma unroll
      for (int j = 0; j < 2; ++j)
        if (j < cts) f[kk][j] = S[(kk * p.ctiles + j) * 32];
    const float* ss = s_of(st);
    const float* sdt = ss + HS_T;
    const bf16* xs = x_of(st);
    // weights e^(s_t - s_u) dt_u (C_t . B_u)
    const float s_lo = ss[r0 + g], s_hi = ss[r0 + g + 8];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int kt = side + 2 * i;
      if (kt <= quarter) {
#pragma unroll
        for (int q = 0; q < 2; ++q) {
          const int u = kt * 16 + q * 8 + 2 * t;
          const float2 su = *reinterpret_cast<const float2*>(ss + u), du = *reinterpret_cast<const float2*>(sdt + u);
          const int lo_row = r0 + g, hi_row = r0 + g + 8;
          const float w0 = u <= lo_row ? cb[i][q][0] * (hs_exp2(s_lo - su.x) * du.x) : 0.f;
          const float w1 = u + 1 <= lo_row ? cb[i][q][1] * (hs_exp2(s_lo - su.y) * du.y) : 0.f;
          const float w2 = u <= hi_row ? cb[i][q][2] * (hs_exp2(s_hi - su.x) * du.x) : 0.f;
          const float w3 = u + 1 <= hi_row ? cb[i][q][3] * (hs_exp2(s_hi - su.y) * du.y) : 0.f;
          uint32_t hi, lo;
          split_pair(w0, w1, hi, lo);
          *reinterpret_cast<uint32_t*>(w_hi + lo_row * C::LDP + u) = hi;
          *reinterpret_cast<uint32_t*>(w_lo + lo_row * C::LDP + u) = lo;
          split_pair(w2, w3, hi, lo);
          *reinterpret_cast<uint32_t*>(w_hi + hi_row * C::LDP + u) = hi;
          *reinterpret_cast<uint32_t*>(w_lo + hi_row * C::LDP + u) = lo;
        }
      }
    }
    __syncthreads();
    if (cts > 0) {
      float acc[2][2][4];
#pragma unroll
      for (int r = 0; r < 2; ++r)
#pragma unroll
        for (int j = 0; j < 2; ++j) acc[r][j][0] = acc[r][j][1] = acc[r][j][2] = acc[r][j][3] = 0.f;
      // what the state in front of the run gives
#pragma unroll
      for (int kk = 0; kk < C::TILES; ++kk) {
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          uint32_t a[4];
          load_a(a, cs, C::LDB, row_tile[r] * 16, kk * 16, lane);
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            mma_bf16(acc[r][j], a, f[kk % AHEAD][j].x, f[kk % AHEAD][j].y);
            mma_bf16(acc[r][j], a, f[kk % AHEAD][j].z, f[kk % AHEAD][j].w);
          }
        }
        if (kk + AHEAD < C::TILES) {
#pragma unroll
          for (int j = 0; j < 2; ++j)
            if (j < cts) f[kk % AHEAD][j] = S[((kk + AHEAD) * p.ctiles + j) * 32];
        }
      }
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const float e_lo = hs_exp2(ss[row_tile[r] * 16 + g]), e_hi = hs_exp2(ss[row_tile[r] * 16 + g + 8]);
#pragma unroll
        for (int j = 0; j < 2; ++j) { acc[r][j][0] *= e_lo; acc[r][j][1] *= e_lo; acc[r][j][2] *= e_hi; acc[r][j][3] *= e_hi; }
      }
      // what the run's own tokens give
#pragma unroll
      for (int kt = 0; kt < HS_T / 16; ++kt) {
        if (kt > row_tile[1]) continue;                    // row_tile[1] is the later of the two
        uint32_t b[4];
        load_b_pair_trans(b, xs, C::LDX, quarter * 16, kt * 16, lane);
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          if (kt > row_tile[r]) continue;
          uint32_t ah[4], al[4];
          load_a(ah, w_hi, C::LDP, row_tile[r] * 16, kt * 16, lane);
          load_a(al, w_lo, C::LDP, row_tile[r] * 16, kt * 16, lane);
          mma_bf16(acc[r][0], ah, b[0], b[1]);
          mma_bf16(acc[r][1], ah, b[2], b[3]);
          mma_bf16(acc[r][0], al, b[0], b[1]);
          mma_bf16(acc[r][1], al, b[2], b[3]);
        }
      }
      const float skip = p.d_skip[head];
#pragma unroll
      for (int r = 0; r < 2; ++r) {
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          if (j >= cts) continue;
          const int x_col = quarter * 16 + j * 8 + 2 * t, c = c0 + x_col;
#pragma unroll
          for (int half = 0; half < 2; ++half) {
            const int row = row_tile[r] * 16 + g + 8 * half;
            if (row >= n) continue;
            const __nv_bfloat162 xv = *reinterpret_cast<const __nv_bfloat162*>(xs + row * C::LDX + x_col);
            *reinterpret_cast<float2*>(p.out + (long long)(begin + row) * p.ld_o + (long long)head * p.vdim + c) =
                make_float2(fmaf(skip, __bfloat162float(xv.x), acc[r][j][2 * half]), fmaf(skip, __bfloat162float(xv.y), acc[r][j][2 * half + 1]));
          }
        }
      }
    }
    hs_wait_all();
    __syncthreads();
  }
}

int padded_state(int n_state) { return n_state <= 32 ? 32 : n_state <= 64 ? 64 : n_state <= 128 ? 128 : 256; }

template <int NP>
int launch_head_scan(HeadScanArgs p, int max_runs, cudaStream_t stream) {
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(head_scan_states_kernel<NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, StatesCfg<NP>::SMEM);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(head_scan_outputs_kernel<NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, OutCfg<NP>::SMEM);
    if (e != cudaSuccess) return hfee_fail(HFEE_ERR_CUDA, "head_scan_mma: cannot get its shared memory: %s", cudaGetErrorString(e));
    configured = true;
  }
  hfee_launch(head_scan_gates_kernel, dim3((p.heads + HS_GATE_HEADS - 1) / HS_GATE_HEADS, max_runs), dim3(HS_GATE_HEADS * 32), 0, stream, p);
  int rc = hfee_check_launch("head_scan_gates");
  if (rc != HFEE_OK) return rc;
  hfee_launch(head_scan_states_kernel<NP>, dim3(p.heads, p.requests, (p.vdim + HS_COLS_STATES - 1) / HS_COLS_STATES), dim3(HS_STATES_THREADS),
              StatesCfg<NP>::SMEM, stream, p);
  rc = hfee_check_launch("head_scan_states");
  if (rc != HFEE_OK) return rc;
  const int tiles = (p.vdim + HS_COLS_OUT - 1) / HS_COLS_OUT;
  // Several heads of a group per block share its C . B, if the blocks still fill the GPU well: about one head's work for the
  // shared part and one for each head, times the rounds that the blocks make.
  const long long slots = HS_OUT_BLOCKS * (long long)hfee_sm_count();
  long long best = 0;
  for (int h : {1, 2, 4}) {
    if ((p.heads / p.groups) % h != 0) continue;
    const long long cost = ((long long)max_runs * (p.heads / h) * tiles + slots - 1) / slots * (h + 1);
    if (best == 0 || cost < best) { best = cost; p.heads_per_block = h; }
  }
  hfee_launch(head_scan_outputs_kernel<NP>, dim3(max_runs, p.heads / p.heads_per_block, tiles), dim3(HS_THREADS), OutCfg<NP>::SMEM, stream, p);
  return hfee_check_launch("head_scan_outputs");
}

}  // namespace

// 1 if hfee_head_scan_mma takes these sizes (bfloat16 is implied).
HFEE_API int hfee_head_scan_mma_supports(int state_dim, int vdim) {
  return state_dim > 0 && state_dim <= 256 && state_dim % 8 == 0 && vdim > 0 && vdim % 8 == 0 ? 1 : 0;
}

// Floats of workspace for steps of at most n_tokens tokens of at most `requests` requests.
HFEE_API long long hfee_head_scan_mma_workspace(int requests, int n_tokens, int heads, int state_dim, int vdim) {
  const long long runs = n_tokens / HS_T + requests;
  return runs * heads * (padded_state(state_dim) / 16) * ((vdim + 7) / 8) * 128 + 2ll * heads * n_tokens;
}

// Arguments as hfee_head_scan (all activations bfloat16); the workspace must start on 16 bytes.
HFEE_API int hfee_head_scan_mma(const void* x, const void* bmat, const void* cmat, long long ld, const void* step, long long ld_step,
                                const float* dt_bias, const float* a_log, const float* d_skip, float* state, const int* cu_tokens,
                                const int* slots, float* out, long long ld_o, int requests, int n_tokens, int heads, int groups,
                                int state_dim, int vdim, int write_state, float* workspace, long long workspace_floats,
                                cudaStream_t stream) {
  if (requests == 0 || n_tokens == 0) return HFEE_OK;
  HFEE_REQUIRE(hfee_head_scan_mma_supports(state_dim, vdim), "head_scan_mma: state size %d and vdim %d must be multiples of 8, the former at most 256",
               state_dim, vdim);
  HFEE_REQUIRE(heads > 0 && groups > 0 && heads % groups == 0, "head_scan_mma: heads %d must be a multiple of groups %d", heads, groups);
  HFEE_REQUIRE(ld % 8 == 0 && (uintptr_t)x % 16 == 0 && (uintptr_t)bmat % 16 == 0 && (uintptr_t)cmat % 16 == 0 && ld_o % 2 == 0 &&
               (uintptr_t)out % 8 == 0, "head_scan_mma: rows must start on 16 bytes (the output's on 8)");
  HFEE_REQUIRE(ld_o >= (long long)heads * vdim && ld_step >= heads, "head_scan_mma: a row stride is too small");
  HFEE_REQUIRE(workspace != nullptr && (uintptr_t)workspace % 16 == 0 &&
               workspace_floats >= hfee_head_scan_mma_workspace(requests, n_tokens, heads, state_dim, vdim), "head_scan_mma: the workspace is too small");
  const int max_runs = n_tokens / HS_T + requests;
  HFEE_REQUIRE(max_runs <= 65535 && requests <= 65535 && heads <= 65535, "head_scan_mma: too many runs or heads for one grid");
  const int np = padded_state(state_dim), ctiles = (vdim + 7) / 8;
  HeadScanArgs p{(const bf16*)x, (const bf16*)bmat, (const bf16*)cmat, ld, (const bf16*)step, ld_step, dt_bias, a_log, d_skip, state,
                 cu_tokens, slots, out, ld_o, nullptr, nullptr, (uint4*)workspace, requests, n_tokens, heads, groups, state_dim, vdim, ctiles,
                 write_state, 1};
  p.gate_s = workspace + (long long)max_runs * heads * (np / 16) * ctiles * 128;
  p.gate_dt = p.gate_s + (long long)heads * n_tokens;
  switch (np) {
    case 32: return launch_head_scan<32>(p, max_runs, stream);
    case 64: return launch_head_scan<64>(p, max_runs, stream);
    case 128: return launch_head_scan<128>(p, max_runs, stream);
    default: return launch_head_scan<256>(p, max_runs, stream);
  }
}
