// A gated recurrence per channel whose gates read the current row only (minGRU):
//
//   z = sigmoid(zl + bz),  u = ul + bx,  c = u + 1/2 for u >= 0 and sigmoid(u) below,
//   S_t = (1 - z_t) S_(t-1) + z_t c_t  (float32, zero at a request's start),  y_t = S_t * silu(g_t)
//
// and, with coefficients formed elsewhere (csrc/block_gates.cu), the affine recurrence S_t = a_t S_(t-1) + b_t,
// y_t = S_t * gelu_tanh(g_t + bg).
//
// zl, ul and g (or a, b and g) are columns of float32 buffers. A block owns a request and 32 channels and walks the request's
// rows 256 at a time: a thread takes four channels of a run of four rows, forms the run's composition S -> A S + B, and after
// an exchange inside the warp and one through shared memory starts from the state behind the runs in front of it. The sums
// arrive by cp.async, two rounds deep. Only one block reads and writes a channel's state, so there is one copy of it. Requests
// with a single row take an elementwise kernel.
#include "common.cuh"

namespace {

constexpr int kChannels = 32;      // channels a block: eight threads of four
constexpr int kWarps = 16;         // a warp's 32 threads are four runs of rows
constexpr int kRows = 4;           // rows a run

// kFast: exponential and division by the special-function unit's approximations (a few units in the last place of float32),
// for models whose results are rounded to 16 bits behind it.
template <bool kFast>
__device__ __forceinline__ float exp_f(float x) { return kFast ? __expf(x) : expf(x); }
template <bool kFast>
__device__ __forceinline__ float div_f(float x, float y) { return kFast ? __fdividef(x, y) : x / y; }
template <bool kFast>
__device__ __forceinline__ float silu_f(float x) { return div_f<kFast>(x, 1.f + exp_f<kFast>(-x)); }
template <bool kFast>
__device__ __forceinline__ void keep_and_add(float zl, float u, float& a, float& b) {
  // with e = exp(-|zl|) one of z and 1 - z is 1 / (1 + e), the other e / (1 + e): no cancellation, no overflow
  const float e = exp_f<kFast>(-fabsf(zl)), big = div_f<kFast>(1.f, 1.f + e), small = e * big;
  const float z = zl >= 0.f ? big : small;
  a = zl >= 0.f ? small : big;
  const float eu = exp_f<kFast>(fminf(u, 0.f));               // sigmoid(u) = e^u / (1 + e^u) below zero
  b = z * (u >= 0.f ? u + 0.5f : div_f<kFast>(eu, 1.f + eu));
}

// four neighbouring results, at once where the rows allow it
__device__ __forceinline__ void store4(float* o, const float (&v)[4]) { *reinterpret_cast<float4*>(o) = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void store4(bf16* o, const float (&v)[4]) {
  __nv_bfloat162 x = __floats2bfloat162_rn(v[0], v[1]), y = __floats2bfloat162_rn(v[2], v[3]);
  uint2 t;
  t.x = *reinterpret_cast<unsigned*>(&x), t.y = *reinterpret_cast<unsigned*>(&y);
  *reinterpret_cast<uint2*>(o) = t;
}

// what the state is multiplied by on its way out
template <bool kFast>
__device__ __forceinline__ float gelu_tanh_f(float z) {
  const float t = 0.7978845608028654f * (z + 0.044715f * z * z * z);
  return kFast ? div_f<true>(z, 1.f + exp_f<true>(-2.f * t)) : 0.5f * z * (1.f + tanhf(t));
}

// kAffine: col 0 and col_step of `zug` hold a and b themselves, and `bias` [channels] is that of the output gate
template <typename TO, bool kFast, bool kAffine>
__global__ void __launch_bounds__(kWarps * 32)
mingru_scan_kernel(TO* __restrict__ out, long long out_stride, const float* __restrict__ zug, long long stride, int col_step,
                   const float* __restrict__ gate, long long gate_stride, const float* __restrict__ bias, float* __restrict__ state, long long state_stride, const int* __restrict__ cu_seqlens,
                   const int* __restrict__ token_req, const int* __restrict__ state_slots, int channels, int whole_fours) {
  pdl_start();
  __shared__ float4 sa[2][kWarps][8], sb[2][kWarps][8];
  extern __shared__ __align__(16) float4 stage[];  // two rounds' sums: [2][kRows * 3][threads], a thread's own by itself
  const int b = blockIdx.x;
  const int start = cu_seqlens[b], n = cu_seqlens[b + 1] - start;
  if (n <= 1 || token_req[start] < 0) return;      // (single rows: mingru_step_kernel; a padding request owns no state)
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, quad = lane & 7, run = lane >> 3;
  const int c = blockIdx.y * kChannels + quad * 4;
  const int cc = min(c, (channels - 1) & ~3);      // threads behind the last channel follow along and store nothing
  float bz[4], bx[4], S[4];
  float* st = state + (size_t)state_slots[b] * state_stride + cc;
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    const bool in = cc + k < channels;
    bz[k] = in ? bias[cc + k] : 0.f;                 // (kAffine: the output gate's)
    bx[k] = in && !kAffine ? bias[channels + cc + k] : 0.f;
    S[k] = in ? st[k] : 0.f;
  }
  constexpr int kWalk = kWarps * 4 * kRows;        // rows of a round
  const float* base = zug + (size_t)start * stride + cc;
  const float* gate_base = gate + (size_t)start * gate_stride + cc;
  TO* o_base = out + (size_t)start * out_stride + cc;
  constexpr int kThreads = kWarps * 32;
  float4* const mine_in = stage + threadIdx.x;
  auto request = [&](int t0, int turn) {           // a round's rows are on their way (cp.async) while the one before is worked on
    if (t0 < n) {
#pragma unroll
      for (int i = 0; i < kRows; ++i) {
        const int r = min(t0 + (warp * 4 + run) * kRows + i, n - 1);
        const float* p = base + (size_t)r * stride;
#pragma unroll
        for (int k = 0; k < 3; ++k) {
          const unsigned dst = (unsigned)__cvta_generic_to_shared(mine_in + (turn * kRows * 3 + i * 3 + k) * kThreads);
          asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(dst), "l"(k < 2 ? p + k * col_step : gate_base + (size_t)r * gate_stride) : "memory");
        }
      }
    }
    asm volatile("cp.async.commit_group;\n" ::: "memory");
  };
  request(0, 0);
  request(kWalk, 1);
  int turn = 0;
  for (int t0 = 0; t0 < n; t0 += kWalk, turn ^= 1) {
    const int first = t0 + (warp * 4 + run) * kRows;
    float a[kRows][4], v[kRows][4], g[kRows][4];
    float A[4] = {1.f, 1.f, 1.f, 1.f}, B[4] = {0.f, 0.f, 0.f, 0.f};
    asm volatile("cp.async.wait_group 1;\n" ::: "memory");
#pragma unroll
    for (int i = 0; i < kRows; ++i) {
      const float4 z = mine_in[(turn * kRows * 3 + i * 3) * kThreads], u = mine_in[(turn * kRows * 3 + i * 3 + 1) * kThreads],
                   gg = mine_in[(turn * kRows * 3 + i * 3 + 2) * kThreads];
      const float z4[4] = {z.x, z.y, z.z, z.w}, u4[4] = {u.x, u.y, u.z, u.w};
      g[i][0] = gg.x, g[i][1] = gg.y, g[i][2] = gg.z, g[i][3] = gg.w;
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        a[i][k] = 1.f, v[i][k] = 0.f;              // rows behind the last one leave the state as it is
        if (first + i < n) {
          if (kAffine) a[i][k] = z4[k], v[i][k] = u4[k], g[i][k] += bz[k];
          else keep_and_add<kFast>(z4[k] + bz[k], u4[k] + bx[k], a[i][k], v[i][k]);
        }
        A[k] *= a[i][k];
        B[k] = a[i][k] * B[k] + v[i][k];
      }
    }
    request(t0 + 2 * kWalk, turn);                 // into the place just read (a thread's own)
    // the warp's four runs: every lane's composition behind those of the runs in front of it, then the last one for the block
    float EA[4], EB[4];                            // of the runs in front of this lane's
#pragma unroll
    for (int k = 0; k < 4; ++k) {
#pragma unroll
      for (int d = 8; d <= 16; d *= 2) {
        const float pa = __shfl_up_sync(0xffffffffu, A[k], d), pb = __shfl_up_sync(0xffffffffu, B[k], d);
        if (lane >= d) B[k] = A[k] * pb + B[k], A[k] *= pa;
      }
      const float pa = __shfl_up_sync(0xffffffffu, A[k], 8), pb = __shfl_up_sync(0xffffffffu, B[k], 8);
      EA[k] = run ? pa : 1.f;
      EB[k] = run ? pb : 0.f;
    }
    if (run == 3) {
      sa[turn][warp][quad] = make_float4(A[0], A[1], A[2], A[3]);
      sb[turn][warp][quad] = make_float4(B[0], B[1], B[2], B[3]);
    }
    __syncthreads();
    float mine[4];
#pragma unroll
    for (int w = 0; w < kWarps; ++w) {
      const float4 fa = sa[turn][w][quad], fb = sb[turn][w][quad];
      const float wa[4] = {fa.x, fa.y, fa.z, fa.w}, wb[4] = {fb.x, fb.y, fb.z, fb.w};
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        if (w == warp) mine[k] = S[k];
        S[k] = wa[k] * S[k] + wb[k];
      }
    }
#pragma unroll
    for (int k = 0; k < 4; ++k) mine[k] = EA[k] * mine[k] + EB[k];
#pragma unroll
    for (int i = 0; i < kRows; ++i) {
      float y[4];
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        mine[k] = a[i][k] * mine[k] + v[i][k];
        y[k] = mine[k] * (kAffine ? gelu_tanh_f<kFast>(g[i][k]) : silu_f<kFast>(g[i][k]));
      }
      if (first + i < n && c < channels) {
        TO* o = o_base + (size_t)(first + i) * out_stride;
        if (whole_fours) {
          store4(o, y);
        } else {
#pragma unroll
          for (int k = 0; k < 4; ++k)
            if (c + k < channels) o[k] = from_f32<TO>(y[k]);
        }
      }
    }
  }
  if (warp == 0 && run == 0 && c < channels)
#pragma unroll
    for (int k = 0; k < 4; ++k)
      if (c + k < channels) st[k] = S[k];
}

// the requests that bring one row
template <typename TO, bool kFast>
__global__ void mingru_step_kernel(TO* __restrict__ out, long long out_stride, const float* __restrict__ zug, long long stride,
                                   int col_step, const float* __restrict__ bias, float* __restrict__ state, long long state_stride,
                                   const int* __restrict__ cu_seqlens, const int* __restrict__ token_req,
                                   const int* __restrict__ state_slots, int channels) {
  pdl_start();
  const int b = blockIdx.x, t = cu_seqlens[b];
  if (cu_seqlens[b + 1] - t != 1) return;
  const int c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= channels) return;
  TO* o = out + (size_t)t * out_stride + c;
  if (token_req[t] < 0) {
    *o = from_f32<TO>(0.f);
    return;
  }
  const float* p = zug + (size_t)t * stride + c;
  float* st = state + (size_t)state_slots[b] * state_stride + c;
  float a, v;
  keep_and_add<kFast>(p[0] + bias[c], p[col_step] + bias[channels + c], a, v);
  const float S = a * *st + v;
  *st = S;
  *o = from_f32<TO>(S * silu_f<kFast>(p[2 * col_step]));
}

}  // namespace

// zug float32 [tokens, stride]: gate logits, raw candidates and output gate at columns 0, col_step and 2 col_step; bias float32
// [2, channels]; state float32 [slots, state_stride]; out [tokens, channels]. singles / longer: some request brings
// one row / more than one.
OI_API int oi_mingru_scan(void* out, int out_dtype, long long out_stride, const float* zug, long long stride, int col_step,
                          const float* bias, float* state, long long state_stride, const int* cu_seqlens, const int* token_req,
                          const int* state_slots, int tokens, int requests, int channels, int singles, int longer, void* stream) {
  OI_REQUIRE(tokens >= 0 && requests >= 0 && channels > 0 && col_step >= channels && stride >= 2LL * col_step + channels &&
             out_stride >= channels && state_stride >= channels, "mingru_scan: bad sizes tokens=%d channels=%d", tokens, channels);
  OI_REQUIRE(zug && bias && state && cu_seqlens && token_req && state_slots && out, "mingru_scan: a buffer is missing");
  if (tokens == 0 || requests == 0) return OI_OK;
  OI_REQUIRE(stride % 4 == 0 && col_step % 4 == 0 && ((uintptr_t)zug & 15) == 0, "mingru_scan: the sums must be readable 16 bytes at a time");
  const int fours = channels % 4 == 0 && out_stride % 4 == 0 && ((uintptr_t)out & 15) == 0 ? 1 : 0;
  cudaStream_t s = (cudaStream_t)stream;
  const size_t smem = (size_t)2 * kRows * 3 * kWarps * 32 * sizeof(float4);
#define OI_GRU(TO, FAST)                                                                                                   \
  do {                                                                                                                     \
    if (longer) {                                                                                                          \
      OI_CHECK_CUDA(cudaFuncSetAttribute(mingru_scan_kernel<TO, FAST, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)); \
      oi_launch(mingru_scan_kernel<TO, FAST, false>, dim3(requests, (channels + kChannels - 1) / kChannels), kWarps * 32, smem, s, (TO*)out, \
                out_stride, zug, stride, col_step, zug + 2 * (size_t)col_step, stride, bias, state, state_stride, cu_seqlens, token_req, state_slots, channels, fours); \
      OI_CHECK_LAUNCH();                                                                                                   \
    }                                                                                                                      \
    if (singles)                                                                                                           \
      oi_launch(mingru_step_kernel<TO, FAST>, dim3(requests, (channels + 127) / 128), 128, 0, s, (TO*)out, out_stride, zug, stride, \
                col_step, bias, state, state_stride, cu_seqlens, token_req, state_slots, channels);                        \
  } while (0)
  if (out_dtype == OI_F32) OI_GRU(float, false);
  else if (out_dtype == OI_BF16) OI_GRU(bf16, true);
  else OI_REQUIRE(false, "mingru_scan: unknown dtype code %d", out_dtype);
#undef OI_GRU
  OI_CHECK_LAUNCH();
  return OI_OK;
}

// ab float32 [tokens, ab_stride]: a at column 0, b at col_step; y float32 [tokens, y_stride] and y_bias [channels]: the output gate;
// state float32 [slots, state_stride]; out [tokens, channels]. Requests that bring one row are left alone (oi_rglru_gates).
OI_API int oi_affine_scan(void* out, int out_dtype, long long out_stride, const float* ab, long long ab_stride, int col_step,
                          const float* y, long long y_stride, const float* y_bias, float* state, long long state_stride,
                          const int* cu_seqlens, const int* token_req, const int* state_slots, int tokens, int requests, int channels,
                          void* stream) {
  OI_REQUIRE(tokens >= 0 && requests >= 0 && channels > 0 && col_step >= channels && ab_stride >= (long long)col_step + channels &&
             y_stride >= channels && out_stride >= channels && state_stride >= channels, "affine_scan: bad sizes tokens=%d channels=%d", tokens, channels);
  OI_REQUIRE(ab && y && y_bias && state && cu_seqlens && token_req && state_slots && out, "affine_scan: a buffer is missing");
  if (tokens == 0 || requests == 0) return OI_OK;
  // (the last four channels are read whole: the buffers' columns are padded to fours)
  OI_REQUIRE(ab_stride % 4 == 0 && col_step % 4 == 0 && y_stride % 4 == 0 && ((uintptr_t)ab & 15) == 0 && ((uintptr_t)y & 15) == 0 &&
             ab_stride >= (long long)col_step + ((channels + 3) & ~3) && y_stride >= ((channels + 3) & ~3),
             "affine_scan: the coefficients must be readable 16 bytes at a time");
  const int fours = channels % 4 == 0 && out_stride % 4 == 0 && ((uintptr_t)out & 15) == 0 ? 1 : 0;
  cudaStream_t s = (cudaStream_t)stream;
  const size_t smem = (size_t)2 * kRows * 3 * kWarps * 32 * sizeof(float4);
  const dim3 grid(requests, (channels + kChannels - 1) / kChannels);
#define OI_AFFINE(TO, FAST)                                                                                                       \
  do {                                                                                                                            \
    OI_CHECK_CUDA(cudaFuncSetAttribute(mingru_scan_kernel<TO, FAST, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)); \
    oi_launch(mingru_scan_kernel<TO, FAST, true>, grid, kWarps * 32, smem, s, (TO*)out, out_stride, ab, ab_stride, col_step, y,    \
              y_stride, y_bias, state, state_stride, cu_seqlens, token_req, state_slots, channels, fours);                         \
  } while (0)
  if (out_dtype == OI_F32) OI_AFFINE(float, false);
  else if (out_dtype == OI_BF16) OI_AFFINE(bf16, true);
  else OI_REQUIRE(false, "affine_scan: unknown dtype code %d", out_dtype);
#undef OI_AFFINE
  OI_CHECK_LAUNCH();
  return OI_OK;
}
