// The gated delta rule with a decay per key channel.  Per request and head, with S [dim, vdim] float32 carried from
// step to step:
//
//     S <- diag(g_t) S;   u = beta_t (v_t - S^T k_t);   S <- S + k_t u^T;   o_t = S^T q_t
//
// q and k are first made unit vectors (x / sqrt(sum x^2 + 1e-6); q also times dim^-1/2), beta_t = sigmoid(b_t) and
// g_t = exp(-exp(A_log) softplus(z_t + dt_bias)) per key channel, all float32.  `qk_heads` query/key heads serve `heads`
// value heads; the decays belong to the value head.
//
// hfee_channel_delta, a step of single tokens: the recurrence itself, a block per (32 state columns, head, request).
//
// A step with longer portions: tiles of CD_TILE tokens.  With G_t the product of the decays of the tile's tokens up to t
// (per channel), S_0 the state in front of the tile and `*` element by element over key channels,
//
//     u_t = beta_t (v_t - S_0^T (G_t * k_t) - sum_{j<t} A[t][j] u_j)       A[t][j] = k_t . (G_t / G_j * k_j)
//     o_t = S_0^T (G_t * q_t) + sum_{j<=t} B[t][j] u_j                      B[t][j] = q_t . (G_t / G_j * k_j)
//     S   = diag(G_last) S_0 + sum_j (G_last / G_j * k_j) u_j^T
//
// The first line is a triangular system with the same matrix for every column, so `channel_delta_prepare` solves it once
// per tile and head for the right-hand sides that do not involve the state: u = U - W S_0 and o = O + P S_0 with
//
//     (I + diag(beta) A) [W | U] = diag(beta) [G * k | v]      P = G * q - B W      O = B U
//
// for all tiles at once, and `channel_delta_walk` goes through a request's tiles with three small products per tile.
// The ratios G_t / G_j are running products of decays from j on (never a quotient of two products, which could be 0 / 0),
// so strong decays underflow to zero and nothing overflows.  The result depends on how a prompt was cut only through the
// order of float32 sums.
//
// A tile's part of the workspace (its place: (first token of the tile) / 16 + request, different for any two tiles of a
// step), per head, rows of DP = dim rounded up to 32 floats:  W [16] | P [16] | Khat [16] (= G_last / G_j * k_j) | G_last,
// and behind all of them, per head and group of CW_COLS columns, U [16][CW_COLS] | O [16][CW_COLS].
#include "tcgen05.cuh"

namespace {

constexpr int CD_TILE = 16;
constexpr int CD_MAX_DIM = 256;
constexpr int CD_THREADS = 128;
constexpr int CD_COLS = 32;                  // state columns per block of the one-token kernel

struct ChannelDeltaArgs {
  long long ld_qkv, ld_b, ld_z, ld_out;
  int q_off, k_off, v_off;
  int heads, qk_heads, dim, vdim;
  int write_state;
  int vec;                     // rows of q, k, z and dt_bias can be fetched four channels at a time
};

__device__ __forceinline__ float softplus_cd(float z) { return z > 20.f ? z : log1pf(expf(z)); }
// the decay of one key channel; the bfloat16 instances take the fast exponential (relative error of some 1e-6)
template <typename T> __device__ __forceinline__ float channel_decay(float rate, float z);
template <> __device__ __forceinline__ float channel_decay<float>(float rate, float z) { return expf(-rate * softplus_cd(z)); }
template <> __device__ __forceinline__ float channel_decay<__nv_bfloat16>(float rate, float z) {
  return __expf(-rate * (fmaxf(z, 0.f) + log1pf(__expf(-fabsf(z)))));
}
template <typename T> __device__ __forceinline__ float4 load4(const T* p);
template <> __device__ __forceinline__ float4 load4<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <> __device__ __forceinline__ float4 load4<__nv_bfloat16>(const __nv_bfloat16* p) {
  const uint2 r = *reinterpret_cast<const uint2*>(p);
  return make_float4(__uint_as_float(r.x << 16), __uint_as_float(r.x & 0xffff0000u), __uint_as_float(r.y << 16), __uint_as_float(r.y & 0xffff0000u));
}

// Two float32 numbers side by side, multiplied and added as a pair.
__device__ __forceinline__ uint64_t pair_of(float lo, float hi) {
  uint64_t r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
  return r;
}
__device__ __forceinline__ float2 unpair(uint64_t v) {
  float2 r;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
  return r;
}
__device__ __forceinline__ uint64_t fma_pair(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ uint64_t mul_pair(uint64_t a, uint64_t b) {
  uint64_t r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ uint64_t add_pair(uint64_t a, uint64_t b) {
  uint64_t r;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}


// ---------------------------------------------------------------------------------------------------------------
// One token per request.  A thread keeps RPT rows of VEC neighbouring columns in registers; 32 / VEC threads side by
// side make a row of CD_COLS columns.
template <typename T, int VEC, int RPT>
__global__ void __launch_bounds__(CD_THREADS)
channel_delta_token_kernel(const T* __restrict__ qkv, const T* __restrict__ b, const float* __restrict__ z,
                           const float* __restrict__ a_log, const float* __restrict__ dt_bias, float* __restrict__ state,
                           const int* __restrict__ cu_tokens, const int* __restrict__ slots, float* __restrict__ out,
                           ChannelDeltaArgs p) {
  constexpr int LANES = CD_COLS / VEC, RG = CD_THREADS / LANES;        // threads of a row, rows taken side by side
  __shared__ float k_s[CD_MAX_DIM], q_s[CD_MAX_DIM], g_s[CD_MAX_DIM];
  __shared__ float sums_s[3][CD_THREADS / 32];
  __shared__ float part_s[2][CD_THREADS / 32][CD_COLS];
  const int h = blockIdx.y, req = blockIdx.z;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int cl = tid % LANES, rg = tid / LANES;
  const int col = blockIdx.x * CD_COLS + cl * VEC;
  const int dim = p.dim, vdim = p.vdim, kh = h / (p.heads / p.qk_heads);
  const int slot = slots[req], tok = cu_tokens[req];
  const float rate = expf(a_log[h]);
  pdl_wait();
  pdl_launch_dependents();
  float* sp = state + ((long long)slot * p.heads + h) * (long long)dim * vdim;
  float S[RPT][VEC];
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int d = rg + RG * i;
    const bool in = d < dim && col < vdim;
    if constexpr (VEC == 4) {
      const float4 t = in ? *reinterpret_cast<const float4*>(sp + (long long)d * vdim + col) : make_float4(0.f, 0.f, 0.f, 0.f);
      S[i][0] = t.x; S[i][1] = t.y; S[i][2] = t.z; S[i][3] = t.w;
    } else {
      S[i][0] = in ? sp[(long long)d * vdim + col] : 0.f;
    }
  }
  const T* row = qkv + (long long)tok * p.ld_qkv;
  float sk = 0.f, sq = 0.f, kq = 0.f;
  for (int d = tid; d < dim; d += CD_THREADS) {
    const float kv = to_f32<T>(row[p.k_off + (long long)kh * dim + d]), qv = to_f32<T>(row[p.q_off + (long long)kh * dim + d]);
    const float zz = z[(long long)tok * p.ld_z + (long long)h * dim + d] + dt_bias[(long long)h * dim + d];
    k_s[d] = kv;
    q_s[d] = qv;
    g_s[d] = channel_decay<T>(rate, zz);
    sk = fmaf(kv, kv, sk);
    sq = fmaf(qv, qv, sq);
    kq = fmaf(kv, qv, kq);
  }
  sk = warp_sum(sk); sq = warp_sum(sq); kq = warp_sum(kq);
  if (lane == 0) { sums_s[0][warp] = sk; sums_s[1][warp] = sq; sums_s[2][warp] = kq; }
  __syncthreads();
  sk = sq = kq = 0.f;
#pragma unroll
  for (int w = 0; w < CD_THREADS / 32; ++w) { sk += sums_s[0][w]; sq += sums_s[1][w]; kq += sums_s[2][w]; }
  const float k_scale = 1.0f / sqrtf(sk + 1e-6f), q_scale = (1.0f / sqrtf((float)dim)) / sqrtf(sq + 1e-6f);
  kq *= k_scale * q_scale;
  float pk[VEC], pq[VEC];
#pragma unroll
  for (int e = 0; e < VEC; ++e) pk[e] = pq[e] = 0.f;
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int d = rg + RG * i;
    const float g = d < dim ? g_s[d] : 0.f, kk = d < dim ? k_s[d] : 0.f, qq = d < dim ? q_s[d] : 0.f;
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      S[i][e] *= g;
      pk[e] = fmaf(S[i][e], kk, pk[e]);
      pq[e] = fmaf(S[i][e], qq, pq[e]);
    }
  }
#pragma unroll
  for (int o = 16; o >= LANES; o >>= 1)
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      pk[e] += __shfl_xor_sync(0xffffffffu, pk[e], o);
      pq[e] += __shfl_xor_sync(0xffffffffu, pq[e], o);
    }
  if (lane < LANES)
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      part_s[0][warp][cl * VEC + e] = pk[e];
      part_s[1][warp][cl * VEC + e] = pq[e];
    }
  __syncthreads();
  const float beta = 1.f / (1.f + expf(-to_f32<T>(b[(long long)tok * p.ld_b + h])));
  float u[VEC], o[VEC];
#pragma unroll
  for (int e = 0; e < VEC; ++e) {
    float sum_k = 0.f, sum_q = 0.f;
#pragma unroll
    for (int w = 0; w < CD_THREADS / 32; ++w) { sum_k += part_s[0][w][cl * VEC + e]; sum_q += part_s[1][w][cl * VEC + e]; }
    const float v = col + e < vdim ? to_f32<T>(row[p.v_off + (long long)h * vdim + col + e]) : 0.f;
    u[e] = beta * (v - sum_k * k_scale);
    o[e] = fmaf(kq, u[e], sum_q * q_scale);
  }
  if (rg == 0)
#pragma unroll
    for (int e = 0; e < VEC; ++e)
      if (col + e < vdim) out[(long long)tok * p.ld_out + (long long)h * vdim + col + e] = o[e];
  if (!p.write_state) return;
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int d = rg + RG * i;
    if (d >= dim || col >= vdim) continue;
    const float kk = k_s[d] * k_scale;
    if constexpr (VEC == 4) {
      *reinterpret_cast<float4*>(sp + (long long)d * vdim + col) =
          make_float4(fmaf(kk, u[0], S[i][0]), fmaf(kk, u[1], S[i][1]), fmaf(kk, u[2], S[i][2]), fmaf(kk, u[3], S[i][3]));
    } else {
      sp[(long long)d * vdim + col] = fmaf(kk, u[0], S[i][0]);
    }
  }
}

// ---------------------------------------------------------------------------------------------------------------
constexpr int CW_COLS = 16;                                         // state columns per block of the walk
constexpr int CW_STAGES = 3;

__host__ __device__ inline int cd_pad(int dim) { return (dim + 31) / 32 * 32; }
__host__ __device__ inline long long cd_head_floats(int dim) { return (3ll * CD_TILE + 1) * cd_pad(dim); }
__host__ __device__ inline int cd_col_tiles(int vdim) { return (vdim + CW_COLS - 1) / CW_COLS; }
constexpr int CD_UO = 2 * CD_TILE * CW_COLS;

// NI: float4 per lane of a row (a row of DP = 32 * NI floats shared by 8 lanes)
template <typename T, int NI>
__global__ void __launch_bounds__(CD_THREADS, NI <= 4 ? 6 : 3)
channel_delta_prepare_kernel(const T* __restrict__ qkv, const T* __restrict__ b, const float* __restrict__ z,
                             const float* __restrict__ a_log, const float* __restrict__ dt_bias,
                             const int* __restrict__ cu_tokens, float* __restrict__ ws_head, float* __restrict__ ws_uo,
                             ChannelDeltaArgs p) {
  constexpr int DP = 32 * NI;
  extern __shared__ __align__(128) float smem[];
  float* k_s = smem;                         // [16][DP]
  float* q_s = k_s + CD_TILE * DP;
  float* g_s = q_s + CD_TILE * DP;
  __shared__ __align__(16) float2 A_s[CD_TILE][CD_TILE], B_s[CD_TILE][CD_TILE];      // -A and B, every number twice: operands of pairs
  __shared__ float beta_s[CD_TILE];
  const int req = blockIdx.z, h = blockIdx.y, tile0 = blockIdx.x * CD_TILE;
  const int begin = cu_tokens[req], count = cu_tokens[req + 1] - begin;
  pdl_wait();
  // the walk's few blocks are let in only when this kernel's last ones are done: let in earlier they would all settle on
  // the first SMs with room
  if (tile0 >= count) return;
  const int tt = min(CD_TILE, count - tile0);
  const long long tok0 = begin + tile0, place = tok0 / CD_TILE + req;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int dim = p.dim, vdim = p.vdim, kh = h / (p.heads / p.qk_heads);
  // work of the last part: pairs of columns of the triangular system (key channels, then values), then pairs of key
  // channels once more
  const int value_cols = cd_col_tiles(vdim) * CW_COLS, items = DP + value_cols / 2;
  float* v_s = g_s + CD_TILE * DP;           // [16][value_cols]
  const float b_own = tid < tt ? to_f32<T>(b[(tok0 + tid) * p.ld_b + h]) : 0.f;
  const float rate = expf(a_log[h]);
  // a missing token is the identity: no write, no decay
  if (p.vec) {
#pragma unroll
    for (int n = 0; n < NI; ++n) {
      const int e = tid + n * CD_THREADS, t = e / (DP / 4), d = (e - t * (DP / 4)) * 4;
      float4 kv = make_float4(0.f, 0.f, 0.f, 0.f), qv = kv, g = make_float4(1.f, 1.f, 1.f, 1.f);
      if (t < tt && d < dim) {
        const T* row = qkv + (tok0 + t) * p.ld_qkv + (long long)kh * dim + d;
        kv = load4<T>(row + p.k_off);
        qv = load4<T>(row + p.q_off);
        const float4 zz = *reinterpret_cast<const float4*>(z + (tok0 + t) * p.ld_z + (long long)h * dim + d);
        const float4 bb = *reinterpret_cast<const float4*>(dt_bias + (long long)h * dim + d);
        g = make_float4(channel_decay<T>(rate, zz.x + bb.x), channel_decay<T>(rate, zz.y + bb.y), channel_decay<T>(rate, zz.z + bb.z),
                        channel_decay<T>(rate, zz.w + bb.w));
      }
      reinterpret_cast<float4*>(k_s)[e] = kv;
      reinterpret_cast<float4*>(q_s)[e] = qv;
      reinterpret_cast<float4*>(g_s)[e] = g;
    }
  } else {
    for (int e = tid; e < CD_TILE * DP; e += CD_THREADS) {
      const int t = e / DP, d = e - t * DP;
      float kv = 0.f, qv = 0.f, g = 1.f;
      if (t < tt && d < dim) {
        const T* row = qkv + (tok0 + t) * p.ld_qkv + (long long)kh * dim + d;
        kv = to_f32<T>(row[p.k_off]);
        qv = to_f32<T>(row[p.q_off]);
        g = channel_decay<T>(rate, z[(tok0 + t) * p.ld_z + (long long)h * dim + d] + dt_bias[(long long)h * dim + d]);
      }
      k_s[e] = kv;
      q_s[e] = qv;
      g_s[e] = g;
    }
  }
  if (p.vec && vdim % 4 == 0) {
    for (int e = tid; e < CD_TILE * value_cols / 4; e += CD_THREADS) {
      const int t = e / (value_cols / 4), c = (e - t * (value_cols / 4)) * 4;
      reinterpret_cast<float4*>(v_s)[e] = t < tt && c < vdim ? load4<T>(qkv + (tok0 + t) * p.ld_qkv + p.v_off + (long long)h * vdim + c)
                                                             : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  } else {
    for (int e = tid; e < CD_TILE * value_cols; e += CD_THREADS) {
      const int t = e / value_cols, c = e - t * value_cols;
      v_s[e] = t < tt && c < vdim ? to_f32<T>(qkv[(tok0 + t) * p.ld_qkv + p.v_off + (long long)h * vdim + c]) : 0.f;
    }
  }
  if (tid < CD_TILE) beta_s[tid] = tid < tt ? 1.f / (1.f + expf(-b_own)) : 0.f;
  __syncthreads();
  const float q_unit = 1.0f / sqrtf((float)dim);
#pragma unroll
  for (int half = 0; half < 2; ++half) {       // eight lanes per vector: 16 keys, then 16 queries
    float4* vec = reinterpret_cast<float4*>(half ? q_s : k_s) + (tid >> 3) * (DP / 4) + (tid & 7);
    float4 x[NI];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      x[i] = vec[8 * i];
      ss = fmaf(x[i].x, x[i].x, ss); ss = fmaf(x[i].y, x[i].y, ss); ss = fmaf(x[i].z, x[i].z, ss); ss = fmaf(x[i].w, x[i].w, ss);
    }
#pragma unroll
    for (int o = 4; o >= 1; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const float scale = (half ? q_unit : 1.f) / sqrtf(ss + 1e-6f);
#pragma unroll
    for (int i = 0; i < NI; ++i) vec[8 * i] = make_float4(x[i].x * scale, x[i].y * scale, x[i].z * scale, x[i].w * scale);
  }
  __syncthreads();
  {
    // the tables: eight lanes per row j, each with its share of the channels of G_t / G_j * k_j as t runs on from j
    const int j = tid >> 3, sl = tid & 7;
    const ulonglong2* k4 = reinterpret_cast<const ulonglong2*>(k_s);
    const ulonglong2* q4 = reinterpret_cast<const ulonglong2*>(q_s);
    const ulonglong2* g4 = reinterpret_cast<const ulonglong2*>(g_s);
    ulonglong2 w[NI];
#pragma unroll
    for (int i = 0; i < NI; ++i) w[i] = k4[j * (DP / 4) + sl + 8 * i];
    const int j_first = (warp * 4);            // smallest j of this warp: earlier tokens concern none of its rows
    for (int t = j_first; t < tt; ++t) {
      uint64_t a2 = 0, c2 = 0;                 // pairs of zeros
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const int at = t * (DP / 4) + sl + 8 * i;
        const ulonglong2 kk = k4[at], qq = q4[at];
        if (t > j) {
          const ulonglong2 g = g4[at];
          w[i].x = mul_pair(w[i].x, g.x);
          w[i].y = mul_pair(w[i].y, g.y);
        }
        a2 = fma_pair(w[i].x, kk.x, a2); a2 = fma_pair(w[i].y, kk.y, a2);
        c2 = fma_pair(w[i].x, qq.x, c2); c2 = fma_pair(w[i].y, qq.y, c2);
      }
      const float2 af = unpair(a2), cf = unpair(c2);
      float a = af.x + af.y, c = cf.x + cf.y;
#pragma unroll
      for (int o = 4; o >= 1; o >>= 1) {
        a += __shfl_xor_sync(0xffffffffu, a, o);
        c += __shfl_xor_sync(0xffffffffu, c, o);
      }
      if (sl == 0) {
        A_s[t][j] = t > j ? make_float2(-a, -a) : make_float2(0.f, 0.f);
        B_s[t][j] = t >= j ? make_float2(c, c) : make_float2(0.f, 0.f);
      }
    }
    if (sl == 0) {                             // what the loop did not reach
      for (int t = 0; t < CD_TILE; ++t)
        if (t < j_first || t >= tt) A_s[t][j] = B_s[t][j] = make_float2(0.f, 0.f);
    }
  }
  __syncthreads();
  float* wh = ws_head + (place * p.heads + h) * cd_head_floats(dim);
  float* wuo = ws_uo + (place * p.heads + h) * (long long)value_cols * 2 * CD_TILE;
  const ulonglong2* A2 = reinterpret_cast<const ulonglong2*>(A_s);      // [t][j / 2]
  const ulonglong2* B2 = reinterpret_cast<const ulonglong2*>(B_s);
  for (int item = tid; item < items; item += CD_THREADS) {
    if (item >= DP / 2 + value_cols / 2) {     // a pair of key channels: what a token's write is worth at the tile's end
      const int c = 2 * (item - DP / 2 - value_cols / 2);
      uint64_t after = pair_of(1.f, 1.f);
#pragma unroll
      for (int t = CD_TILE - 1; t >= 0; --t) {
        const uint64_t k = *reinterpret_cast<const uint64_t*>(k_s + t * DP + c), g = *reinterpret_cast<const uint64_t*>(g_s + t * DP + c);
        *reinterpret_cast<uint64_t*>(wh + (2 * CD_TILE + t) * DP + c) = mul_pair(after, k);
        after = mul_pair(after, g);
      }
      *reinterpret_cast<uint64_t*>(wh + 3 * CD_TILE * DP + c) = after;
      continue;
    }
    // two columns of the triangular system side by side, the second product behind it
    const bool key = item < DP / 2;
    const int c = key ? 2 * item : 2 * (item - DP / 2);
    float* dst = key ? wh + c : wuo + (c / CW_COLS) * CD_UO + c % CW_COLS;
    const int ld = key ? DP : CW_COLS;
    uint64_t x[CD_TILE], run = pair_of(1.f, 1.f);
#pragma unroll
    for (int t = 0; t < CD_TILE; ++t) {
      asm volatile("" ::: "memory");           // or all the tokens' loads would be moved up here and overflow the registers
      uint64_t r, second;
      if (key) {
        run = mul_pair(run, *reinterpret_cast<const uint64_t*>(g_s + t * DP + c));
        r = mul_pair(run, *reinterpret_cast<const uint64_t*>(k_s + t * DP + c));
        second = mul_pair(run, *reinterpret_cast<const uint64_t*>(q_s + t * DP + c));
      } else {
        r = *reinterpret_cast<const uint64_t*>(v_s + t * value_cols + c);
        second = 0;
      }
#pragma unroll
      for (int j = 0; j < t; j += 2) {         // A holds -A, and zero from the diagonal on
        const ulonglong2 m = A2[t * (CD_TILE / 2) + j / 2];
        r = fma_pair(m.x, x[j], r);
        if (j + 1 < t) r = fma_pair(m.y, x[j + 1], r);
      }
      const float bt = beta_s[t];
      x[t] = mul_pair(pair_of(bt, bt), r);
      *reinterpret_cast<uint64_t*>(dst + t * ld) = x[t];
      uint64_t o = 0;
#pragma unroll
      for (int j = 0; j <= t; j += 2) {
        const ulonglong2 m = B2[t * (CD_TILE / 2) + j / 2];
        o = fma_pair(m.x, x[j], o);
        if (j + 1 <= t) o = fma_pair(m.y, x[j + 1], o);
      }
      *reinterpret_cast<uint64_t*>(dst + (CD_TILE + t) * ld) = key ? fma_pair(o, pair_of(-1.f, -1.f), second) : o;
    }
  }
}

// A block walks the tiles of one request and head for CW_COLS state columns; the tiles' parts of the workspace come in
// through a ring of bulk copies.  A warp owns C neighbouring columns.  Lane (dg, cg), dg < 8 and cg < 4, holds the rows
// 4 dg + 32 i + (0..3) of all C of them (the four lanes of a dg hold copies): for the products with W and P it takes the
// rows t = 4 r + cg, r < 8, of the two matrices, so that a row is read from shared memory once per warp, and eight
// lanes' partial sums leave lane (dg, cg) with those of t = 4 dg + cg: rows of W in the lanes with dg < 4, of P in the
// others.  For the update it takes the tokens 4 r + cg, and the four partial sums meet by exchanges across cg, in an
// order that gives every copy the same bits.
template <int NI, int C>
__global__ void __launch_bounds__(CW_COLS / C * 32, 1)
channel_delta_walk_kernel(const float* __restrict__ ws_head, const float* __restrict__ ws_uo, float* __restrict__ state,
                          const int* __restrict__ cu_tokens, const int* __restrict__ slots, float* __restrict__ out,
                          int* __restrict__ status, ChannelDeltaArgs p) {
  constexpr int DP = 32 * NI;
  constexpr int HEAD = (3 * CD_TILE + 1) * DP, STAGE = HEAD + CD_UO;      // floats of a tile
  extern __shared__ __align__(128) float smem[];                          // [CW_STAGES][STAGE]
  __shared__ __align__(8) uint64_t full[CW_STAGES];
  __shared__ int abort_flag;
  const int req = blockIdx.z, h = blockIdx.y, tile_col = blockIdx.x;
  const int begin = cu_tokens[req], count = cu_tokens[req + 1] - begin;
  const int slot = slots[req];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int dg = lane & 7, cg = lane >> 3;
  const int in_tile = warp * C, col = tile_col * CW_COLS + in_tile;
  const int dim = p.dim, vdim = p.vdim, tiles = (count + CD_TILE - 1) / CD_TILE;
  if (tid == 0) {
    abort_flag = 0;
    for (int s = 0; s < CW_STAGES; ++s) tc::mbar_init(&full[s], 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  __syncthreads();
  pdl_wait();
  pdl_launch_dependents();
  if (count <= 0) return;
  const int col_tiles = cd_col_tiles(vdim);
  auto bulk = [](float* dst, const float* src, uint32_t bytes, uint64_t* bar) {
    asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
                 ::"r"(tc::smem_u32(dst)), "l"(src), "r"(bytes), "r"(tc::smem_u32(bar)) : "memory");
  };
  auto fetch = [&](int tile) {
    const int s = tile % CW_STAGES;
    const long long place = (begin + tile * CD_TILE) / CD_TILE + req, at = place * p.heads + h;
    tc::mbar_expect_tx(&full[s], STAGE * 4u);
    bulk(smem + s * STAGE, ws_head + at * HEAD, HEAD * 4u, &full[s]);
    bulk(smem + s * STAGE + HEAD, ws_uo + (at * col_tiles + tile_col) * CD_UO, CD_UO * 4u, &full[s]);
  };
  if (tid == 0)
    for (int t = 0; t < CW_STAGES - 1 && t < tiles; ++t) fetch(t);
  float* sp = state + ((long long)slot * p.heads + h) * (long long)dim * vdim + col;
  uint64_t S[NI][C][2];                                       // rows (0, 1) and (2, 3) of the lane's four, per column
#pragma unroll
  for (int i = 0; i < NI; ++i)
#pragma unroll
    for (int c = 0; c < C; ++c)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int d = 32 * i + 4 * dg + 2 * e;
        S[i][c][e] = pair_of((d < dim && col + c < vdim) ? sp[(long long)d * vdim + c] : 0.f,
                             (d + 1 < dim && col + c < vdim) ? sp[(long long)(d + 1) * vdim + c] : 0.f);
      }
  const bool wide = C == 4 && vdim % 4 == 0 && p.ld_out % 4 == 0 && (uintptr_t)out % 16 == 0;
  bool ok = true;
  for (int tile = 0; tile < tiles; ++tile) {
    const int s = tile % CW_STAGES;
    ok = tc::mbar_wait(&full[s], (tile / CW_STAGES) & 1u, &abort_flag);
    if (!__syncthreads_and(ok)) { ok = false; break; }        // also: every warp is done with the tile before
    if (tid == 0 && tile + CW_STAGES - 1 < tiles) fetch(tile + CW_STAGES - 1);
    const ulonglong2* M = reinterpret_cast<const ulonglong2*>(smem + s * STAGE) + dg;
    float val[8 * C];                                         // [r][c]
#pragma unroll
    for (int r = 0; r < 8; ++r) {
      uint64_t acc[C];
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const ulonglong2 m = M[(4 * r + cg) * (DP / 4) + 8 * i];
#pragma unroll
        for (int c = 0; c < C; ++c) {
          acc[c] = i == 0 ? mul_pair(m.x, S[i][c][0]) : fma_pair(m.x, S[i][c][0], acc[c]);
          acc[c] = fma_pair(m.y, S[i][c][1], acc[c]);
        }
      }
#pragma unroll
      for (int c = 0; c < C; ++c) {
        const float2 f = unpair(acc[c]);
        val[r * C + c] = f.x + f.y;
      }
    }
#pragma unroll
    for (int off = 4; off >= 1; off >>= 1) {
      const bool upper = (lane & off) != 0;
#pragma unroll
      for (int i = 0; i < off * C; ++i) {
        const float send = upper ? val[i] : val[i + off * C], keep = upper ? val[i + off * C] : val[i];
        val[i] = keep + __shfl_xor_sync(0xffffffffu, send, off);
      }
    }
    const int t = 4 * dg + cg;                                // below 16: u of token t, else o of token t - 16
    const float* uo = smem + s * STAGE + HEAD + t * CW_COLS + in_tile;
    float x[C];
#pragma unroll
    for (int c = 0; c < C; ++c) x[c] = uo[c] + (dg < 4 ? -val[c] : val[c]);
    if (dg >= 4 && tile * CD_TILE + t - CD_TILE < count) {
      float* o = out + (long long)(begin + tile * CD_TILE + t - CD_TILE) * p.ld_out + (long long)h * vdim + col;
      if (wide && C == 4) {
        if (col < vdim) *reinterpret_cast<float4*>(o) = make_float4(x[0], x[1 % C], x[2 % C], x[3 % C]);
      } else {
#pragma unroll
        for (int c = 0; c < C; ++c)
          if (col + c < vdim) o[c] = x[c];
      }
    }
    uint64_t u[4][C];                                         // of the tokens 4 r + cg, twice side by side
#pragma unroll
    for (int r = 0; r < 4; ++r)
#pragma unroll
      for (int c = 0; c < C; ++c) {
        const float v = __shfl_sync(0xffffffffu, x[c], (lane & 24) + r);
        u[r][c] = pair_of(v, v);
      }
    const ulonglong2* K = M + 2 * CD_TILE * (DP / 4);
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      uint64_t d[C][2];
#pragma unroll
      for (int r = 0; r < 4; ++r) {
        const ulonglong2 k = K[(4 * r + cg) * (DP / 4) + 8 * i];
#pragma unroll
        for (int c = 0; c < C; ++c) {
          d[c][0] = r == 0 ? mul_pair(k.x, u[r][c]) : fma_pair(k.x, u[r][c], d[c][0]);
          d[c][1] = r == 0 ? mul_pair(k.y, u[r][c]) : fma_pair(k.y, u[r][c], d[c][1]);
        }
      }
#pragma unroll
      for (int off = 8; off <= 16; off <<= 1)
#pragma unroll
        for (int c = 0; c < C; ++c)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const float2 f = unpair(d[c][e]);
            d[c][e] = add_pair(d[c][e], pair_of(__shfl_xor_sync(0xffffffffu, f.x, off), __shfl_xor_sync(0xffffffffu, f.y, off)));
          }
      const ulonglong2 g = K[CD_TILE * (DP / 4) + 8 * i];
#pragma unroll
      for (int c = 0; c < C; ++c) {
        S[i][c][0] = fma_pair(g.x, S[i][c][0], d[c][0]);
        S[i][c][1] = fma_pair(g.y, S[i][c][1], d[c][1]);
      }
    }
  }
  if (!ok) {                                                  // a copy never arrived: say so; copies in flight get a while to end
    if (tid == 0) *status = 1;
    for (int s = 0; s < CW_STAGES; ++s)
      for (int i = 0; i < 64; ++i)
        if (tc::mbar_try(&full[s], 0) || tc::mbar_try(&full[s], 1)) break;
    return;
  }
  if (p.write_state && cg == 0)
#pragma unroll
    for (int i = 0; i < NI; ++i)
#pragma unroll
      for (int c = 0; c < C; ++c)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int d = 32 * i + 4 * dg + 2 * e;
          const float2 f = unpair(S[i][c][e]);
          if (d < dim && col + c < vdim) sp[(long long)d * vdim + c] = f.x;
          if (d + 1 < dim && col + c < vdim) sp[(long long)(d + 1) * vdim + c] = f.y;
        }
}

template <typename T, int VEC, int RPT>
int launch_token_r(const void* qkv, const void* b, const float* z, const float* a_log, const float* dt_bias, float* state,
                   const int* cu_tokens, const int* slots, float* out, const ChannelDeltaArgs& p, int requests, cudaStream_t stream) {
  hfee_launch(channel_delta_token_kernel<T, VEC, RPT>, dim3((unsigned)((p.vdim + CD_COLS - 1) / CD_COLS), (unsigned)p.heads, (unsigned)requests),
              dim3(CD_THREADS), 0, stream, (const T*)qkv, (const T*)b, z, a_log, dt_bias, state, cu_tokens, slots, out, p);
  return hfee_check_launch("channel_delta_token");
}

template <typename T>
int launch_token(const void* qkv, const void* b, const float* z, const float* a_log, const float* dt_bias, float* state,
                 const int* cu_tokens, const int* slots, float* out, const ChannelDeltaArgs& p, int requests, cudaStream_t stream) {
#define HFEE_CD(V, R) return launch_token_r<T, V, R>(qkv, b, z, a_log, dt_bias, state, cu_tokens, slots, out, p, requests, stream)
  if (p.vdim % 4 == 0 && (uintptr_t)state % 16 == 0) {       // 16 rows side by side
    if (p.dim <= 32) HFEE_CD(4, 2);
    if (p.dim <= 64) HFEE_CD(4, 4);
    if (p.dim <= 128) HFEE_CD(4, 8);
    HFEE_CD(4, 16);
  }
  if (p.dim <= 64) HFEE_CD(1, 16);                           // 4 rows side by side
  HFEE_CD(1, 64);
#undef HFEE_CD
}

template <typename T, int NI>
int launch_tiles_n(const void* qkv, const void* b, const float* z, const float* a_log, const float* dt_bias, float* state,
                   const int* cu_tokens, const int* slots, float* out, const ChannelDeltaArgs& p, int requests, int max_new,
                   float* ws_head, float* ws_uo, int* status, cudaStream_t stream) {
  constexpr int C = NI <= 4 ? 4 : 2;                          // columns per warp of the walk: what its registers hold
  const size_t prep = (size_t)CD_TILE * (3 * 32 * NI + cd_col_tiles(p.vdim) * CW_COLS) * sizeof(float);
  HFEE_REQUIRE(prep <= 200 * 1024, "channel_delta: values of %d numbers per head do not fit shared memory", p.vdim);
  const size_t walk = (size_t)CW_STAGES * ((3 * CD_TILE + 1) * 32 * NI + CD_UO) * sizeof(float);
  if (prep > 40 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(channel_delta_prepare_kernel<T, NI>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)prep);
    if (e != cudaSuccess) return hfee_fail(HFEE_ERR_CUDA, "channel_delta_prepare: %s", cudaGetErrorString(e));
  }
  if (walk > 40 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(channel_delta_walk_kernel<NI, C>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)walk);
    if (e != cudaSuccess) return hfee_fail(HFEE_ERR_CUDA, "channel_delta_walk: %s", cudaGetErrorString(e));
  }
  hfee_launch(channel_delta_prepare_kernel<T, NI>, dim3((unsigned)((max_new + CD_TILE - 1) / CD_TILE), (unsigned)p.heads, (unsigned)requests),
              dim3(CD_THREADS), prep, stream, (const T*)qkv, (const T*)b, z, a_log, dt_bias, cu_tokens, ws_head, ws_uo, p);
  const int rc = hfee_check_launch("channel_delta_prepare");
  if (rc != HFEE_OK) return rc;
  hfee_launch(channel_delta_walk_kernel<NI, C>, dim3((unsigned)cd_col_tiles(p.vdim), (unsigned)p.heads, (unsigned)requests),
              dim3(CW_COLS / C * 32), walk, stream, ws_head, ws_uo, state, cu_tokens, slots, out, status, p);
  return hfee_check_launch("channel_delta_walk");
}

template <typename T>
int launch_tiles(const void* qkv, const void* b, const float* z, const float* a_log, const float* dt_bias, float* state,
                 const int* cu_tokens, const int* slots, float* out, const ChannelDeltaArgs& p, int requests, int max_new,
                 float* ws_head, float* ws_uo, int* status, cudaStream_t stream) {
#define HFEE_CT(N) case N: return launch_tiles_n<T, N>(qkv, b, z, a_log, dt_bias, state, cu_tokens, slots, out, p, requests, max_new, ws_head, ws_uo, status, stream)
  switch (cd_pad(p.dim) / 32) {
    HFEE_CT(1); HFEE_CT(2); HFEE_CT(3); HFEE_CT(4); HFEE_CT(5); HFEE_CT(6); HFEE_CT(7);
    default: return launch_tiles_n<T, 8>(qkv, b, z, a_log, dt_bias, state, cu_tokens, slots, out, p, requests, max_new, ws_head, ws_uo, status, stream);
  }
#undef HFEE_CT
}

long long cd_places(int requests, int n_tokens) { return n_tokens / CD_TILE + requests + 1; }

}  // namespace

// Floats of workspace for a step of n_tokens tokens in `requests` requests that has a portion of several tokens.
HFEE_API long long hfee_channel_delta_workspace(int requests, int n_tokens, int heads, int dim, int vdim) {
  return cd_places(requests, n_tokens) * heads * (cd_head_floats(dim) + (long long)cd_col_tiles(vdim) * CD_UO);
}

// qkv rows (dtype): head g's query at q_off + g * dim, its key at k_off + g * dim (g < qk_heads; head h of `heads` uses
// g = h / (heads / qk_heads)), head h's value at v_off + h * vdim.  b rows (dtype): one number per head.  z rows
// (float32): heads * dim.  dt_bias: [heads * dim].  state: [slots, heads, dim, vdim] float32.  out: float32 [n, heads *
// vdim].  max_new: the longest portion of the step; 1 takes the one-token kernel, more takes the workspace.
HFEE_API int hfee_channel_delta(const void* qkv, long long ld_qkv, int q_off, int k_off, int v_off, const void* b, long long ld_b,
                                const float* z, long long ld_z, int dtype, const float* a_log, const float* dt_bias, float* state,
                                const int* cu_tokens, const int* slots, float* out, long long ld_out, int requests, int heads,
                                int qk_heads, int dim, int vdim, int write_state, int n_tokens, int max_new, float* workspace,
                                long long workspace_floats, int* status, cudaStream_t stream) {
  if (requests == 0 || max_new == 0) return HFEE_OK;
  HFEE_REQUIRE(heads > 0 && qk_heads > 0 && heads % qk_heads == 0, "channel_delta: heads %d must be a multiple of %d", heads, qk_heads);
  HFEE_REQUIRE(dim > 0 && dim <= CD_MAX_DIM && vdim > 0, "channel_delta: key size %d is outside 1..%d", dim, CD_MAX_DIM);
  HFEE_REQUIRE(requests <= 65535 && heads <= 65535, "channel_delta: too many requests or heads");
  HFEE_REQUIRE(dtype == HFEE_F32 || dtype == HFEE_BF16, "channel_delta: unknown dtype %d", dtype);
  const int vec = dim % 4 == 0 && ld_qkv % 4 == 0 && ld_z % 4 == 0 && q_off % 4 == 0 && k_off % 4 == 0 && v_off % 4 == 0 &&
                  (uintptr_t)qkv % (dtype == HFEE_F32 ? 16 : 8) == 0 && (uintptr_t)z % 16 == 0 && (uintptr_t)dt_bias % 16 == 0;
  const ChannelDeltaArgs p{ld_qkv, ld_b, ld_z, ld_out, q_off, k_off, v_off, heads, qk_heads, dim, vdim, write_state, vec};
  if (max_new == 1) {
    if (dtype == HFEE_F32) return launch_token<float>(qkv, b, z, a_log, dt_bias, state, cu_tokens, slots, out, p, requests, stream);
    return launch_token<__nv_bfloat16>(qkv, b, z, a_log, dt_bias, state, cu_tokens, slots, out, p, requests, stream);
  }
  HFEE_REQUIRE(workspace != nullptr && workspace_floats >= hfee_channel_delta_workspace(requests, n_tokens, heads, dim, vdim) &&
               (uintptr_t)workspace % 16 == 0 && status != nullptr, "channel_delta: the workspace is missing, too small or not 16-byte aligned");
  float* ws_head = workspace;
  float* ws_uo = workspace + cd_places(requests, n_tokens) * heads * cd_head_floats(dim);
  if (dtype == HFEE_F32)
    return launch_tiles<float>(qkv, b, z, a_log, dt_bias, state, cu_tokens, slots, out, p, requests, max_new, ws_head, ws_uo, status, stream);
  return launch_tiles<__nv_bfloat16>(qkv, b, z, a_log, dt_bias, state, cu_tokens, slots, out, p, requests, max_new, ws_head, ws_uo, status, stream);
}
