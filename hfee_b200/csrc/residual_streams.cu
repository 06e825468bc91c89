// Several residual streams beside one another (hyper-connections): everything between two sublayers in one pass.
//
// A token has `streams` float32 rows X_1 .. X_s.  A sublayer with coefficients a, M, b reads u = sum_s a[s] X_s through
// an RMS norm in groups (each of `groups` equal consecutive parts of the row divided by its own root mean square, then
// a weight per column), and its output y goes back as X_t <- sum_s M[s][t] X_s + b[t] y.  hfee_stream_step does, per
// token: the second half of the sublayer before (if there is one: y not null), the first half of the next, the norm and,
// optionally, the token shift h_t + (h_(t-1) - h_t) * mu on the normed row, and stores the row in the dtype the matrix
// products read.
//
// The row in front of a portion's first token belongs to the request (`shift_state`, one float32 row per slot: the
// normed row before its shift).  A block takes `run` consecutive tokens and keeps the row before in shared memory; it
// computes the row in front of its first token again unless that token is its request's first in the step.  The streams
// go to another buffer than they are read from, so a block may read any token at any time.  The block that reads a
// request's state is also the one that renews it, from the request's last token, which it computes again if it lies
// outside its run: no other block touches that slot, so one launch does it all.
//
// Float32 arithmetic; the order of the sums depends on the sizes only.
#include "common.cuh"

namespace {

constexpr int ST_WARPS = 8;
constexpr int ST_THREADS = ST_WARPS * 32;
constexpr int ST_MAX_STREAMS = 64;

struct StreamArgs {
  const float* x; long long token_stride, stream_stride;      // streams in front of the update (stream stride 0: all equal)
  const float* y; long long ld_y;                             // output of the sublayer before, or null: nothing to update
  const float* mix; const float* out_w;                       // its M [from][to] and b (y not null)
  float* x_out;                                               // [n][streams][width], or null (the streams end here)
  const float* in_w;                                          // the next sublayer's a, or null: the plain sum
  const float* norm_w; float eps; int groups;
  const float* shift_w; float* shift_state; int write_state;  // mu and the per-request rows, or null
  const int* slot_of_token; const int* cu_tokens; int requests;
  const int* rows;                                            // tokens to take (no shift, no x_out), or null: all
  long long ld_h;
  int n, width, streams, run;
};

template <int VEC> struct Pack;
template <> struct Pack<1> {
  float v[1];
  __device__ __forceinline__ void load(const float* p) { v[0] = *p; }
  __device__ __forceinline__ void store(float* p) const { *p = v[0]; }
};
template <> struct Pack<4> {
  float v[4];
  __device__ __forceinline__ void load(const float* p) { const float4 t = *reinterpret_cast<const float4*>(p); v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w; }
  __device__ __forceinline__ void store(float* p) const { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
};
template <typename T, int VEC> __device__ __forceinline__ void store_row(T* p, const Pack<VEC>& a) {
#pragma unroll
  for (int e = 0; e < VEC; ++e) p[e] = from_f32<T>(a.v[e]);
}
template <> __device__ __forceinline__ void store_row<float, 4>(float* p, const Pack<4>& a) { a.store(p); }
template <> __device__ __forceinline__ void store_row<__nv_bfloat16, 4>(__nv_bfloat16* p, const Pack<4>& a) {
  const __nv_bfloat162 lo = __floats2bfloat162_rn(a.v[0], a.v[1]), hi = __floats2bfloat162_rn(a.v[2], a.v[3]);
  uint2 r;
  r.x = *reinterpret_cast<const uint32_t*>(&lo);
  r.y = *reinterpret_cast<const uint32_t*>(&hi);
  *reinterpret_cast<uint2*>(p) = r;
}

// S: number of streams, or 0 for any number (the streams are then read again for every output stream).
template <typename T, int S, int VEC>
__global__ void __launch_bounds__(ST_THREADS, S > 0 ? 3 : 2)
stream_step_kernel(StreamArgs p, T* __restrict__ h_out) {
  extern __shared__ __align__(16) float row_s[];       // [width]: u of the token in work; with a shift [width]: the row before
  __shared__ float coef_s[ST_MAX_STREAMS * 2 + (S > 0 ? S * S : ST_MAX_STREAMS * ST_MAX_STREAMS)];
  __shared__ float red_s[2][ST_WARPS];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int streams = S > 0 ? S : p.streams;
  float* in_s = coef_s;
  float* out_s = coef_s + ST_MAX_STREAMS;
  float* mix_s = coef_s + 2 * ST_MAX_STREAMS;
  for (int e = tid; e < streams; e += ST_THREADS) {    // weights: no kernel writes them
    in_s[e] = p.in_w != nullptr ? p.in_w[e] : 1.f;
    out_s[e] = p.y != nullptr ? p.out_w[e] : 0.f;
  }
  if (p.y != nullptr)
    for (int e = tid; e < streams * streams; e += ST_THREADS) mix_s[e] = p.mix[e];
  float* u_s = row_s;
  float* prev_s = row_s + p.width;
  const int i0 = blockIdx.x * p.run, i1 = min(i0 + p.run, p.n);
  // warps share the groups out: a team of warps per group, or several groups per warp
  const int teams = min(p.groups, ST_WARPS), per_team = ST_WARPS / teams;
  const int team = warp / per_team, in_team = warp - team * per_team;
  const int part = p.width / p.groups, vecs = part / VEC;
  __syncthreads();
  pdl_wait();
  pdl_launch_dependents();

  int turn = 0;
  // The normed row of token i, element by element to `use(column, values)`; store: its streams go to x_out.
  auto normed = [&](int i, bool store, auto&& use) {
    const long long src = p.rows != nullptr ? p.rows[i] : i;
    const float* xr = p.x + src * p.token_stride;
    const float* yr = p.y != nullptr ? p.y + src * p.ld_y : nullptr;
    float* xo = (store && p.x_out != nullptr) ? p.x_out + src * (long long)streams * p.width : nullptr;
    for (int g = team; g < p.groups && team < teams; g += teams) {
      float ss = 0.f;
      for (int j = in_team * 32 + lane; j < vecs; j += per_team * 32) {
        const int c = g * part + j * VEC;
        Pack<VEC> u;
#pragma unroll
        for (int e = 0; e < VEC; ++e) u.v[e] = 0.f;
        if constexpr (S > 0) {
          Pack<VEC> xs[S], yv;
#pragma unroll
          for (int s = 0; s < S; ++s) xs[s].load(xr + s * p.stream_stride + c);
          if (yr != nullptr) {
            yv.load(yr + c);
#pragma unroll
            for (int t = 0; t < S; ++t) {
              Pack<VEC> a;
              const float b = out_s[t], w = in_s[t];
#pragma unroll
              for (int e = 0; e < VEC; ++e) a.v[e] = b * yv.v[e];
#pragma unroll
              for (int s = 0; s < S; ++s) {
                const float m = mix_s[s * S + t];
#pragma unroll
                for (int e = 0; e < VEC; ++e) a.v[e] = fmaf(m, xs[s].v[e], a.v[e]);
              }
              if (xo != nullptr) a.store(xo + (long long)t * p.width + c);
#pragma unroll
              for (int e = 0; e < VEC; ++e) u.v[e] = fmaf(w, a.v[e], u.v[e]);
            }
          } else {
#pragma unroll
            for (int s = 0; s < S; ++s) {
              const float w = in_s[s];
#pragma unroll
              for (int e = 0; e < VEC; ++e) u.v[e] = fmaf(w, xs[s].v[e], u.v[e]);
            }
          }
        } else {
          Pack<VEC> yv, xv;
          if (yr != nullptr) yv.load(yr + c);
          for (int t = 0; t < streams; ++t) {
            Pack<VEC> a;
            if (yr != nullptr) {
#pragma unroll
              for (int e = 0; e < VEC; ++e) a.v[e] = out_s[t] * yv.v[e];
              for (int s = 0; s < streams; ++s) {
                xv.load(xr + s * p.stream_stride + c);
                const float m = mix_s[s * streams + t];
#pragma unroll
                for (int e = 0; e < VEC; ++e) a.v[e] = fmaf(m, xv.v[e], a.v[e]);
              }
              if (xo != nullptr) a.store(xo + (long long)t * p.width + c);
            } else {
              a.load(xr + t * p.stream_stride + c);
            }
#pragma unroll
            for (int e = 0; e < VEC; ++e) u.v[e] = fmaf(in_s[t], a.v[e], u.v[e]);
          }
        }
        u.store(u_s + c);                              // read back by the same thread only
#pragma unroll
        for (int e = 0; e < VEC; ++e) ss = fmaf(u.v[e], u.v[e], ss);
      }
      ss = warp_sum(ss);
      if (per_team > 1) {                              // then every team has exactly one group
        if (lane == 0) red_s[turn][warp] = ss;
        asm volatile("bar.sync %0, %1;" ::"r"(1 + team), "r"(per_team * 32) : "memory");
        ss = 0.f;
        for (int w = 0; w < per_team; ++w) ss += red_s[turn][team * per_team + w];
      }
      const float scale = 1.0f / sqrtf(ss / (float)part + p.eps);
      for (int j = in_team * 32 + lane; j < vecs; j += per_team * 32) {
        const int c = g * part + j * VEC;
        Pack<VEC> u, w;
        u.load(u_s + c);
        w.load(p.norm_w + c);
#pragma unroll
        for (int e = 0; e < VEC; ++e) u.v[e] = u.v[e] * scale * w.v[e];
        use(c, u);
      }
    }
    turn ^= 1;                                         // the next token's sums go to the other half of red_s
  };

  const bool shift = p.shift_w != nullptr;
  bool reads_state = false;                            // the request in work has its first token of the step in this block
  auto first_of_request = [&](int i) { return i == 0 || p.slot_of_token[i - 1] != p.slot_of_token[i]; };
  // the run, behind the token in front of it if that is needed, and in front of the last request's last token likewise
  int i = shift && !first_of_request(i0) ? i0 - 1 : i0;
  for (; i < i1; ++i) {
    const bool own = i >= i0, first = shift && own && first_of_request(i);
    reads_state = reads_state || first;
    float* state = shift ? p.shift_state + (long long)p.slot_of_token[i] * p.width : nullptr;
    const bool renew = shift && own && reads_state && p.write_state && (i + 1 == p.n || p.slot_of_token[i + 1] != p.slot_of_token[i]);
    normed(i, own, [&](int c, const Pack<VEC>& h) {
      Pack<VEC> out = h;
      if (shift && own) {
        Pack<VEC> before, mu;
        before.load((first ? state : prev_s) + c);
        mu.load(p.shift_w + c);
#pragma unroll
        for (int e = 0; e < VEC; ++e) out.v[e] = fmaf(before.v[e] - h.v[e], mu.v[e], h.v[e]);
        if (renew) h.store(state + c);
      }
      if (own) store_row<T, VEC>(h_out + (long long)i * p.ld_h + c, out);
      if (shift) h.store(prev_s + c);
    });
  }
  if (reads_state && p.write_state && i1 < p.n && p.slot_of_token[i1] == p.slot_of_token[i1 - 1]) {
    int lo = 0, hi = p.requests;                       // the request that holds token i1 - 1: cu[lo] <= i1 - 1 < cu[lo + 1]
    while (hi - lo > 1) {
      const int mid = (lo + hi) >> 1;
      if (p.cu_tokens[mid] <= i1 - 1) lo = mid;
      else hi = mid;
    }
    float* state = p.shift_state + (long long)p.slot_of_token[i1 - 1] * p.width;
    normed(p.cu_tokens[lo + 1] - 1, false, [&](int c, const Pack<VEC>& h) { h.store(state + c); });
  }
}

template <typename T, int S, int VEC>
int launch_stream_step(const StreamArgs& p, void* h_out, cudaStream_t stream) {
  const size_t smem = (size_t)p.width * sizeof(float) * (p.shift_w != nullptr ? 2 : 1);
  HFEE_REQUIRE(smem <= 160 * 1024, "stream_step: a row of %d columns does not fit shared memory", p.width);
  if (smem > 32 * 1024) {                              // the static part may take some 17 KB beside it
    cudaError_t e = cudaFuncSetAttribute(stream_step_kernel<T, S, VEC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return hfee_fail(HFEE_ERR_CUDA, "stream_step: %s", cudaGetErrorString(e));
  }
  hfee_launch(stream_step_kernel<T, S, VEC>, dim3((unsigned)((p.n + p.run - 1) / p.run)), dim3(ST_THREADS), smem, stream, p, (T*)h_out);
  return hfee_check_launch("stream_step");
}

template <typename T>
int launch_stream_step_t(const StreamArgs& p, bool vec, void* h_out, cudaStream_t stream) {
  if (!vec) return launch_stream_step<T, 0, 1>(p, h_out, stream);
  switch (p.streams) {
    case 1: return launch_stream_step<T, 1, 4>(p, h_out, stream);
    case 2: return launch_stream_step<T, 2, 4>(p, h_out, stream);
    case 3: return launch_stream_step<T, 3, 4>(p, h_out, stream);
    case 4: return launch_stream_step<T, 4, 4>(p, h_out, stream);
    default: return launch_stream_step<T, 0, 4>(p, h_out, stream);
  }
}

}  // namespace

// x: n tokens (or, with rows, any number) of `streams` float32 rows; h_out [n, width] in `dtype`.  See StreamArgs.
HFEE_API int hfee_stream_step(const float* x, long long token_stride, long long stream_stride, const float* y, long long ld_y,
                              const float* mix, const float* out_w, float* x_out, const float* in_w, const float* norm_w,
                              float eps, int groups, const float* shift_w, float* shift_state, int write_state,
                              const int* slot_of_token, const int* cu_tokens, int requests, const int* rows, void* h_out,
                              long long ld_h, int dtype, int n, int width, int streams, cudaStream_t stream) {
  if (n == 0) return HFEE_OK;
  HFEE_REQUIRE(n > 0 && width > 0 && streams > 0 && streams <= ST_MAX_STREAMS, "stream_step: %d streams are outside 1..%d", streams, ST_MAX_STREAMS);
  HFEE_REQUIRE(groups > 0 && width % groups == 0, "stream_step: width %d does not form %d equal groups", width, groups);
  HFEE_REQUIRE(y == nullptr || (mix != nullptr && out_w != nullptr), "stream_step: a sublayer's output comes with its coefficients");
  HFEE_REQUIRE(x_out == nullptr || (y != nullptr && x_out != x), "stream_step: updated streams go to a buffer of their own");
  HFEE_REQUIRE(shift_w == nullptr || (shift_state != nullptr && slot_of_token != nullptr && cu_tokens != nullptr && requests > 0 && rows == nullptr),
               "stream_step: the token shift needs its state and the batch layout");
  HFEE_REQUIRE(rows == nullptr || x_out == nullptr, "stream_step: chosen rows do not go on");
  HFEE_REQUIRE(ld_h >= width && token_stride >= 0 && stream_stride >= 0, "stream_step: bad strides");
  const int sms = hfee_sm_count();
  HFEE_REQUIRE(sms > 0, "stream_step: cannot ask the device for its number of SMs");
  int run = 1;
  if (shift_w != nullptr) {                            // a longer run computes fewer rows twice; one wave of three blocks an SM
    run = (n + 3 * sms - 1) / (3 * sms);
    run = run < 1 ? 1 : (run > 8 ? 8 : run);
  }
  const StreamArgs p{x, token_stride, stream_stride, y, ld_y, mix, out_w, x_out, in_w, norm_w, eps, groups, shift_w, shift_state,
                     write_state, slot_of_token, cu_tokens, requests, rows, ld_h, n, width, streams, run};
  auto aligned = [](const void* q, int bytes) { return (uintptr_t)q % bytes == 0; };
  const bool vec = (width / groups) % 4 == 0 && token_stride % 4 == 0 && stream_stride % 4 == 0 && ld_y % 4 == 0 && ld_h % 4 == 0 &&
                   aligned(x, 16) && aligned(y, 16) && aligned(x_out, 16) && aligned(norm_w, 16) && aligned(shift_w, 16) &&
                   aligned(shift_state, 16) && aligned(h_out, dtype == HFEE_F32 ? 16 : 8);
  if (dtype == HFEE_F32) return launch_stream_step_t<float>(p, vec, h_out, stream);
  if (dtype == HFEE_BF16) return launch_stream_step_t<__nv_bfloat16>(p, vec, h_out, stream);
  return hfee_fail(HFEE_ERR_ARG, "stream_step: unknown dtype %d", dtype);
}
