// A gated recurrence per channel whose gates read the current row only (minGRU):
//
//   z = sigmoid(zl + bz),  u = ul + bx,  c = u + 1/2 for u >= 0 and sigmoid(u) below,
//   S_t = (1 - z_t) S_(t-1) + z_t c_t  (float32, zero at a request's start),  y_t = S_t * silu(g_t)
//
// zl, ul and g are columns of one fused product's float32 sums. A block owns a request and 32 channels (a lane each) and
// walks the request's rows 128 at a time: every warp takes a run of eight rows, forms the run's composition
// S -> A S + B from its own rows, and after one exchange through shared memory starts from the state behind the runs in
// front of it. Only one block reads and writes a channel's state, so there is one copy of it. A request with a single row
// takes the same kernel (or, when every request of the step has one, an elementwise one).
#include "common.cuh"

namespace {

constexpr int kChannels = 32;      // channels a block
constexpr int kRuns = 16;          // warps: runs of rows that are worked on at a time
constexpr int kRows = 8;           // rows a run

__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float silu_f(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ void keep_and_add(float zl, float u, float& a, float& b) {
  const float z = sigmoid_f(zl);
  a = 1.f / (1.f + expf(zl));       // 1 - z without the cancellation
  b = z * (u >= 0.f ? u + 0.5f : sigmoid_f(u));
}

template <typename TO>
__global__ void __launch_bounds__(kChannels * kRuns)
mingru_scan_kernel(TO* __restrict__ out, long long out_stride, const float* __restrict__ zug, long long stride, int col_step,
                   const float* __restrict__ bias, float* __restrict__ state, long long state_stride, const int* __restrict__ cu_seqlens,
                   const int* __restrict__ token_req, const int* __restrict__ state_slots, int channels) {
  pdl_start();
  __shared__ float sa[2][kRuns][kChannels], sb[2][kRuns][kChannels];
  const int b = blockIdx.x;
  const int start = cu_seqlens[b], n = cu_seqlens[b + 1] - start;
  if (n <= 0 || token_req[start] < 0) return;      // a padding request of a recorded step owns no state
  const int lane = threadIdx.x & 31, run = threadIdx.x >> 5;
  const int c = blockIdx.y * kChannels + lane;
  const bool on = c < channels;
  const int cc = on ? c : channels - 1;            // lanes behind the last channel follow along and store nothing
  const float bz = bias[cc], bx = bias[channels + cc];
  float* st = state + (size_t)state_slots[b] * state_stride + cc;
  float S = *st;
  const float* base = zug + (size_t)start * stride + cc;
  float zl[kRows], ul[kRows], gl[kRows];
  auto load = [&](int first) {
#pragma unroll
    for (int i = 0; i < kRows; ++i) {
      const int t = min(first + i, n - 1);
      const float* p = base + (size_t)t * stride;
      zl[i] = p[0];
      ul[i] = p[col_step];
      gl[i] = p[2 * col_step];
    }
  };
  load(run * kRows);
  int turn = 0;
  for (int t0 = 0; t0 < n; t0 += kRuns * kRows, turn ^= 1) {
    const int first = t0 + run * kRows;
    float a[kRows], v[kRows], g[kRows];
    float A = 1.f, B = 0.f;
#pragma unroll
    for (int i = 0; i < kRows; ++i) {
      a[i] = 1.f, v[i] = 0.f;                      // rows behind the last one leave the state as it is
      if (first + i < n) keep_and_add(zl[i] + bz, ul[i] + bx, a[i], v[i]);
      g[i] = gl[i];
      A *= a[i];
      B = a[i] * B + v[i];
    }
    if (t0 + kRuns * kRows < n) load(first + kRuns * kRows);      // the next rows are on their way meanwhile
    sa[turn][run][lane] = A;
    sb[turn][run][lane] = B;
    __syncthreads();
    float mine = S;
#pragma unroll
    for (int r = 0; r < kRuns; ++r) {
      if (r == run) mine = S;
      S = sa[turn][r][lane] * S + sb[turn][r][lane];
    }
#pragma unroll
    for (int i = 0; i < kRows; ++i) {
      mine = a[i] * mine + v[i];
      if (on && first + i < n) out[(size_t)(start + first + i) * out_stride + c] = from_f32<TO>(mine * silu_f(g[i]));
    }
  }
  if (on && run == 0) *st = S;
}

// every request of the step brings one row
template <typename TO>
__global__ void mingru_step_kernel(TO* __restrict__ out, long long out_stride, const float* __restrict__ zug, long long stride,
                                   int col_step, const float* __restrict__ bias, float* __restrict__ state, long long state_stride,
                                   const int* __restrict__ cu_seqlens, const int* __restrict__ token_req,
                                   const int* __restrict__ state_slots, int channels) {
  pdl_start();
  const int b = blockIdx.x, t = cu_seqlens[b];
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
  keep_and_add(p[0] + bias[c], p[col_step] + bias[channels + c], a, v);
  const float S = a * *st + v;
  *st = S;
  *o = from_f32<TO>(S * silu_f(p[2 * col_step]));
}

}  // namespace

// zug float32 [tokens, stride]: gate logits, raw candidates and output gate at columns 0, col_step and 2 col_step; bias float32
// [2, channels]; state float32 [slots, state_stride]; out [tokens, channels]. single_rows: every request brings one row.
OI_API int oi_mingru_scan(void* out, int out_dtype, long long out_stride, const float* zug, long long stride, int col_step,
                          const float* bias, float* state, long long state_stride, const int* cu_seqlens, const int* token_req,
                          const int* state_slots, int tokens, int requests, int channels, int single_rows, void* stream) {
  OI_REQUIRE(tokens >= 0 && requests >= 0 && channels > 0 && col_step >= channels && stride >= 2LL * col_step + channels &&
             out_stride >= channels && state_stride >= channels, "mingru_scan: bad sizes tokens=%d channels=%d", tokens, channels);
  OI_REQUIRE(zug && bias && state && cu_seqlens && token_req && state_slots && out, "mingru_scan: a buffer is missing");
  OI_REQUIRE(!single_rows || tokens == requests, "mingru_scan: %d rows of %d requests are not one each", tokens, requests);
  if (tokens == 0 || requests == 0) return OI_OK;
  cudaStream_t s = (cudaStream_t)stream;
#define OI_GRU(TO)                                                                                                         \
  do {                                                                                                                     \
    if (single_rows)                                                                                                       \
      oi_launch(mingru_step_kernel<TO>, dim3(requests, (channels + 127) / 128), 128, 0, s, (TO*)out, out_stride, zug, stride, col_step, \
                bias, state, state_stride, cu_seqlens, token_req, state_slots, channels);                                  \
    else                                                                                                                   \
      oi_launch(mingru_scan_kernel<TO>, dim3(requests, (channels + kChannels - 1) / kChannels), kChannels * kRuns, 0, s, (TO*)out, \
                out_stride, zug, stride, col_step, bias, state, state_stride, cu_seqlens, token_req, state_slots, channels); \
  } while (0)
  if (out_dtype == OI_F32) OI_GRU(float);
  else if (out_dtype == OI_BF16) OI_GRU(bf16);
  else OI_REQUIRE(false, "mingru_scan: unknown dtype code %d", out_dtype);
#undef OI_GRU
  OI_CHECK_LAUNCH();
  return OI_OK;
}
