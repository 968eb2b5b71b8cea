// The gates of a real-gated linear recurrent unit (RG-LRU), for all rows of a step at once.
//
// u [tokens, blocks * size] in equal parts; every part n has two square matrices [out, in] and two biases:
//   r = sigmoid(Wr_n u_n + br_n),  i = sigmoid(Wi_n u_n + bi_n),  log a = -r * rate  (rate = 8 softplus(lambda), a number a channel),
//   a = exp(log a),  put = sqrt(1 - a^2) i u,  the recurrence being S_t = a S_(t-1) + put.
// Rows of requests that bring several rows leave (a, put) for the scan (csrc/gated_scan.cu). A request's single row takes its
// step here: S <- a S + put, out = S gelu_tanh(y + by); nobody else touches the request's state.
//
// u arrives as float32 sums. For 16-bit matrices it is split into two bfloat16 numbers, u = hi + lo (16 bits), and both halves
// are multiplied with the same fragments of the matrices on the tensor cores (mma.sync m16n8k16, float32 accumulation): a block
// takes 64 rows and 64 channels of one part, both matrices, 64 numbers of K at a time, the matrices by cp.async in two buffers.
// float32 matrices take the ordinary pipes. Everything behind the products is float32: with the exact functions for float32
// results, with the special-function unit's exponential, division and root (a few units in the last place of float32) for
// results that are rounded to 16 bits behind it.
#include "oi_api.h"

namespace {

struct GateArgs {
  const float* u;            // [tokens, ld_u]
  const void* w;             // [2, blocks, size, size]: Wr, then Wi
  const float* bias;         // [2, blocks * size]
  const float* rate;         // [blocks * size]
  float* ab;                 // [tokens, ld_ab]: a at column 0, put at col_step
  const float* y;            // [tokens, ld_y]
  const float* y_bias;       // [blocks * size]
  void* out;                 // [tokens, ld_out]
  float* state;              // [slots, state_stride]
  const int* cu_seqlens;
  const int* token_req;
  const int* state_slots;
  long long ld_u, ld_ab, ld_y, ld_out, state_stride;
  int col_step, tokens, blocks, size, vec;
};

__device__ __forceinline__ float gelu_tanh_f(float z) {
  return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

// what a row needs to know beside its sums: the place of its state when it is its request's only row of the step (else -1);
// -2: a row of a padding request
__device__ __forceinline__ int single_slot(const GateArgs& p, int t) {
  const int req = p.token_req[t];
  if (req < 0) return -2;
  return p.cu_seqlens[req + 1] - p.cu_seqlens[req] == 1 ? p.state_slots[req] : -1;
}

// exp(-|..|)-style coefficients of one number: a = exp(la) and sqrt(1 - a^2) for la <= 0
template <bool kFast>
__device__ __forceinline__ void decay_and_root(float la, float& a, float& root) {
  if (!kFast) {
    a = expf(la);
    root = sqrtf(-expm1f(2.f * la));
    return;
  }
  a = __expf(la);
  // 1 - e^x, x = 2 la: near zero by its series (seven terms: below 2^-24 of it for |x| < 1/2), else as it stands
  const float x = 2.f * la;
  float p = 1.f + x * (1.f / 7.f);
  p = 1.f + x * (1.f / 6.f) * p;
  p = 1.f + x * (1.f / 5.f) * p;
  p = 1.f + x * (1.f / 4.f) * p;
  p = 1.f + x * (1.f / 3.f) * p;
  p = 1.f + x * (1.f / 2.f) * p;
  const float m = x > -0.5f ? -x * p : 1.f - a * a;
  asm("sqrt.approx.ftz.f32 %0, %1;\n" : "=f"(root) : "f"(m));
}
template <bool kFast>
__device__ __forceinline__ float sigmoid_f(float z) {
  return kFast ? __fdividef(1.f, 1.f + __expf(-z)) : 1.f / (1.f + expf(-z));
}

// two neighbouring numbers of a row that leaves its coefficients for the scan
__device__ __forceinline__ void finish_pair(const GateArgs& p, int t, int c, float zr0, float zi0, float zr1, float zi1) {
  const int C = p.blocks * p.size;
  const float2 br = *reinterpret_cast<const float2*>(p.bias + c), bi = *reinterpret_cast<const float2*>(p.bias + C + c);
  const float2 rate = *reinterpret_cast<const float2*>(p.rate + c), u = *reinterpret_cast<const float2*>(p.u + (size_t)t * p.ld_u + c);
  float2 a, root;
  decay_and_root<true>(-sigmoid_f<true>(zr0 + br.x) * rate.x, a.x, root.x);
  decay_and_root<true>(-sigmoid_f<true>(zr1 + br.y) * rate.y, a.y, root.y);
  float* ab = p.ab + (size_t)t * p.ld_ab + c;
  *reinterpret_cast<float2*>(ab) = a;
  *reinterpret_cast<float2*>(ab + p.col_step) = make_float2(root.x * sigmoid_f<true>(zi0 + bi.x) * u.x, root.y * sigmoid_f<true>(zi1 + bi.y) * u.y);
}

template <typename TO>
__device__ __forceinline__ void finish(const GateArgs& p, int t, int c, int slot, float zr, float zi) {
  const int C = p.blocks * p.size;
  constexpr bool kFast = sizeof(TO) == 2;
  float a, root;
  decay_and_root<kFast>(-sigmoid_f<kFast>(zr + p.bias[c]) * p.rate[c], a, root);
  const float put = root * sigmoid_f<kFast>(zi + p.bias[C + c]) * p.u[(size_t)t * p.ld_u + c];
  if (slot == -1) {
    p.ab[(size_t)t * p.ld_ab + c] = a;
    p.ab[(size_t)t * p.ld_ab + p.col_step + c] = put;
    return;
  }
  float v = 0.f;
  if (slot >= 0) {
    float* st = p.state + (size_t)slot * p.state_stride + c;
    const float S = a * *st + put;
    *st = S;
    v = S * gelu_tanh_f(p.y[(size_t)t * p.ld_y + c] + p.y_bias[c]);
  }
  reinterpret_cast<TO*>(p.out)[(size_t)t * p.ld_out + c] = from_f32<TO>(v);
}

// float32 matrices: a block of 256 threads takes 32 rows and 32 channels of one part, both matrices, 32 numbers of K at a time
constexpr int kFm = 32, kFn = 32, kFk = 32;
template <typename TO>
__global__ void __launch_bounds__(256) rglru_gates_f32_kernel(const GateArgs p) {
  pdl_start();
  __shared__ float As[kFk][kFm + 1], Ws[2][kFk][kFn + 1];
  const int per = (p.size + kFn - 1) / kFn;
  const int part = blockIdx.y / per, n0 = (blockIdx.y - part * per) * kFn, t0 = blockIdx.x * kFm;
  const float* w = reinterpret_cast<const float*>(p.w);
  const int tn = threadIdx.x % 32, tm = threadIdx.x / 32;      // channel tn, rows tm + 8 i
  float acc[2][4] = {};
  for (int k0 = 0; k0 < p.size; k0 += kFk) {
    for (int i = threadIdx.x; i < kFm * kFk; i += 256) {
      const int m = i / kFk, k = i % kFk;
      As[k][m] = (t0 + m < p.tokens && k0 + k < p.size) ? p.u[(size_t)(t0 + m) * p.ld_u + part * p.size + k0 + k] : 0.f;
    }
    for (int i = threadIdx.x; i < 2 * kFn * kFk; i += 256) {
      const int g = i / (kFn * kFk), n = (i / kFk) % kFn, k = i % kFk;
      Ws[g][k][n] = (n0 + n < p.size && k0 + k < p.size)
                        ? w[(((size_t)g * p.blocks + part) * p.size + n0 + n) * p.size + k0 + k] : 0.f;
    }
    __syncthreads();
#pragma unroll 8
    for (int k = 0; k < kFk; ++k) {
      const float wr = Ws[0][k][tn], wi = Ws[1][k][tn];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float a = As[k][tm + 8 * i];
        acc[0][i] += a * wr;
        acc[1][i] += a * wi;
      }
    }
    __syncthreads();
  }
  if (n0 + tn >= p.size) return;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int t = t0 + tm + 8 * i;
    if (t < p.tokens) finish<TO>(p, t, part * p.size + n0 + tn, single_slot(p, t), acc[0][i], acc[1][i]);
  }
}

// bfloat16 matrices and few rows (single decoded tokens): a warp takes ONE channel, its rows of both matrices in registers (asked
// for before the kernels ahead on the stream have finished), and walks the step's rows, 32 at a time, whose part of u lies in
// shared memory; lane n ends row n.
constexpr int kFewRows = 64, kFewSize = 512, kFewWarps = 8;

__global__ void __launch_bounds__(kFewWarps * 32) rglru_gates_few_kernel(const GateArgs p) {
  pdl_trigger();
  extern __shared__ __align__(16) float us[];          // [32][size]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int per = (p.size + kFewWarps - 1) / kFewWarps;
  const int part = blockIdx.x / per, n = (blockIdx.x - part * per) * kFewWarps + warp;
  const bool mine = n < p.size;
  const bf16* w = reinterpret_cast<const bf16*>(p.w);
  __nv_bfloat162 wr[kFewSize / 64], wi[kFewSize / 64];  // numbers 64 q + 2 lane, + 1 (p.vec: the size is a multiple of eight)
  const __nv_bfloat162 zero = __floats2bfloat162_rn(0.f, 0.f);
#pragma unroll
  for (int q = 0; q < kFewSize / 64; ++q) {
    const int k = 64 * q + 2 * lane;
    const bool ok = mine && k < p.size;
    const bf16* src = w + ((size_t)part * p.size + (ok ? n : 0)) * p.size + (ok ? k : 0);
    wr[q] = ok ? *reinterpret_cast<const __nv_bfloat162*>(src) : zero;
    wi[q] = ok ? *reinterpret_cast<const __nv_bfloat162*>(src + (size_t)p.blocks * p.size * p.size) : zero;
  }
  pdl_wait();
  for (int t0 = 0; t0 < p.tokens; t0 += 32) {
    const int rows = min(32, p.tokens - t0), quads = p.size / 4;
    if (t0) __syncthreads();
    for (int i = threadIdx.x; i < rows * quads; i += kFewWarps * 32) {
      const int r = i / quads, c = (i - r * quads) * 4;
      *reinterpret_cast<float4*>(us + r * p.size + c) = *reinterpret_cast<const float4*>(p.u + (size_t)(t0 + r) * p.ld_u + part * p.size + c);
    }
    const int slot = lane < rows ? single_slot(p, t0 + lane) : -3;
    __syncthreads();
    if (!mine) continue;
    float zr = 0.f, zi = 0.f;
    for (int r = 0; r < rows; ++r) {
      float a = 0.f, b = 0.f;
#pragma unroll
      for (int q = 0; q < kFewSize / 64; ++q) {
        const int k = 64 * q + 2 * lane;
        if (64 * q < p.size) {
          const float2 x = k < p.size ? *reinterpret_cast<const float2*>(us + r * p.size + k) : make_float2(0.f, 0.f);
          const float2 fr = __bfloat1622float2(wr[q]), fi = __bfloat1622float2(wi[q]);
          a += x.x * fr.x + x.y * fr.y;
          b += x.x * fi.x + x.y * fi.y;
        }
      }
      a = warp_sum(a), b = warp_sum(b);
      if (lane == r) zr = a, zi = b;
    }
    if (lane < rows) finish<bf16>(p, t0 + lane, part * p.size + n, slot, zr, zi);
  }
}

// bfloat16 matrices on the tensor cores
constexpr int kM = 64, kN = 64, kK = 64, kPad = kK + 8;
struct GateTile {
  bf16 A[2][2][kM][kPad];     // [buffer][hi | lo]
  bf16 W[2][2][kN][kPad];     // [buffer][r | i]
  int slot[kM];
};

__device__ __forceinline__ void mma_16816(float (&d)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm4(unsigned (&r)[4], const void* row) {
  const unsigned addr = (unsigned)__cvta_generic_to_shared(row);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void cp16(void* dst, const void* src, bool valid) {
  const unsigned d = (unsigned)__cvta_generic_to_shared(dst);
  const int n = valid ? 16 : 0;          // 0: the 16 bytes are filled with zeros and src is not read
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(d), "l"(src), "r"(n));
}

__global__ void __launch_bounds__(256) rglru_gates_mma_kernel(const GateArgs p) {
  pdl_trigger();
  extern __shared__ __align__(16) unsigned char raw[];
  GateTile& s = *reinterpret_cast<GateTile*>(raw);
  const int per = (p.size + kN - 1) / kN;
  const int part = blockIdx.y / per, n0 = (blockIdx.y - part * per) * kN, t0 = blockIdx.x * kM;
  const bf16* w = reinterpret_cast<const bf16*>(p.w);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, tg = lane & 3;
  const int wm = (warp & 3) * 16, wn = (warp >> 2) * 32;
  // the matrices' tile: 128 rows (r, then i) of 64 numbers, four 16-byte pieces a thread
  auto load_w = [&](int k0, int buf) {
    if (p.vec) {
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const int id = threadIdx.x + 256 * q, row = id >> 3, k = (id & 7) * 8, n = row & 63, gate = row >> 6;
        const bool ok = n0 + n < p.size && k0 + k < p.size;
        const bf16* src = w + (((size_t)gate * p.blocks + part) * p.size + (ok ? n0 + n : 0)) * p.size + (ok ? k0 + k : 0);
        cp16(&s.W[buf][gate][n][k], src, ok);
      }
    } else {
      for (int i = threadIdx.x; i < 2 * kN * kK; i += 256) {
        const int gate = i / (kN * kK), n = (i / kK) % kN, k = i % kK;
        const bool ok = n0 + n < p.size && k0 + k < p.size;
        s.W[buf][gate][n][k] = ok ? w[(((size_t)gate * p.blocks + part) * p.size + n0 + n) * p.size + k0 + k] : __float2bfloat16_rn(0.f);
      }
    }
    asm volatile("cp.async.commit_group;\n" ::: "memory");
  };
  // the rows' tile: 64 rows of 64 numbers, sixteen a thread (row id / 4, numbers 16 (id % 4) ..), asked for a step ahead
  const int ar = threadIdx.x >> 2, ak = (threadIdx.x & 3) * 16;
  float av[16];
  auto fetch_a = [&](int k0) {
    const float* src = p.u + (size_t)min(t0 + ar, p.tokens - 1) * p.ld_u + part * p.size + k0 + ak;
    const bool row_ok = t0 + ar < p.tokens;
    if (p.vec) {
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const float4 v = row_ok && k0 + ak + 4 * q < p.size ? *reinterpret_cast<const float4*>(src + 4 * q) : make_float4(0.f, 0.f, 0.f, 0.f);
        av[4 * q] = v.x, av[4 * q + 1] = v.y, av[4 * q + 2] = v.z, av[4 * q + 3] = v.w;
      }
    } else {
#pragma unroll
      for (int q = 0; q < 16; ++q) av[q] = row_ok && k0 + ak + q < p.size ? src[q] : 0.f;
    }
  };
  auto put_a = [&](int buf) {
#pragma unroll
    for (int q = 0; q < 16; q += 2) {
      const __nv_bfloat162 hi = __floats2bfloat162_rn(av[q], av[q + 1]);
      const float2 back = __bfloat1622float2(hi);
      *reinterpret_cast<__nv_bfloat162*>(&s.A[buf][0][ar][ak + q]) = hi;
      *reinterpret_cast<__nv_bfloat162*>(&s.A[buf][1][ar][ak + q]) = __floats2bfloat162_rn(av[q] - back.x, av[q + 1] - back.y);
    }
  };
  load_w(0, 0);                          // the matrices do not depend on the kernels ahead on the stream
  pdl_wait();
  if (threadIdx.x < kM) s.slot[threadIdx.x] = t0 + (int)threadIdx.x < p.tokens ? single_slot(p, t0 + threadIdx.x) : -3;
  fetch_a(0);
  float acc[2][4][4] = {};
  int buf = 0;
  const bool busy = t0 + wm < p.tokens;  // a warp whose 16 rows lie behind the last one has nothing to multiply
  for (int k0 = 0; k0 < p.size; k0 += kK, buf ^= 1) {
    put_a(buf);
    asm volatile("cp.async.wait_group 0;\n" ::: "memory");
    __syncthreads();                     // this step's tiles are complete, and everyone has left the other buffers
    if (k0 + kK < p.size) {
      load_w(k0 + kK, buf ^ 1);
      fetch_a(k0 + kK);
    }
    if (busy) {
#pragma unroll
      for (int kk = 0; kk < kK; kk += 16) {
        if (k0 + kk >= p.size) break;
        unsigned hi[4], lo[4];
        const int row = wm + (lane & 7) + ((lane >> 3) & 1) * 8, col = kk + (lane >> 4) * 8;
        ldsm4(hi, &s.A[buf][0][row][col]);
        ldsm4(lo, &s.A[buf][1][row][col]);
#pragma unroll
        for (int gate = 0; gate < 2; ++gate)
#pragma unroll
          for (int j = 0; j < 4; j += 2) {
            unsigned b[4];
            ldsm4(b, &s.W[buf][gate][wn + 8 * (j + (lane >> 4)) + (lane & 7)][kk + ((lane >> 3) & 1) * 8]);
            mma_16816(acc[gate][j], lo, b[0], b[1]);
            mma_16816(acc[gate][j + 1], lo, b[2], b[3]);
            mma_16816(acc[gate][j], hi, b[0], b[1]);
            mma_16816(acc[gate][j + 1], hi, b[2], b[3]);
          }
      }
    }
  }
  if (!busy) return;
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    const int m = wm + g + 8 * h, t = t0 + m;
    if (t >= p.tokens) continue;
    const int slot = s.slot[m];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + wn + 8 * j + 2 * tg;
      if (p.vec && slot == -1) {         // (the size is a multiple of eight: both numbers or none)
        if (n < p.size)
          finish_pair(p, t, part * p.size + n, acc[0][j][2 * h], acc[1][j][2 * h], acc[0][j][2 * h + 1], acc[1][j][2 * h + 1]);
        continue;
      }
#pragma unroll
      for (int e = 0; e < 2; ++e)
        if (n + e < p.size) finish<bf16>(p, t, part * p.size + n + e, slot, acc[0][j][2 * h + e], acc[1][j][2 * h + e]);
    }
  }
}

}  // namespace

// u float32 [tokens, blocks * size]; w [2, blocks, size, size] (float32; bfloat16 with bfloat16 results); bias float32 [2, blocks *
// size]; rate float32 [blocks * size] (what multiplies -r in log a); ab float32 [tokens, >= col_step + channels]; y float32 rows and
// y_bias [channels]: what a single row's state is multiplied by, behind gelu_tanh; state float32 [slots, state_stride].
OI_API int oi_rglru_gates(const float* u, long long ld_u, const void* w, int w_dtype, const float* bias, const float* rate, float* ab,
                          long long ld_ab, int col_step, const float* y, long long ld_y, const float* y_bias, void* out, int out_dtype,
                          long long ld_out, float* state, long long state_stride, const int* cu_seqlens, const int* token_req,
                          const int* state_slots, int tokens, int blocks, int size, void* stream) {
  const int C = blocks * size;
  OI_REQUIRE(tokens >= 0 && blocks > 0 && size > 0 && ld_u >= C && ld_ab >= (long long)col_step + C && col_step >= C && ld_y >= C &&
             ld_out >= C && state_stride >= C, "rglru_gates: bad sizes tokens=%d blocks=%d size=%d", tokens, blocks, size);
  OI_REQUIRE(u && w && bias && rate && ab && y && y_bias && out && state && cu_seqlens && token_req && state_slots, "rglru_gates: a buffer is missing");
  OI_REQUIRE((out_dtype == OI_F32 || out_dtype == OI_BF16) && (w_dtype == OI_F32 || (w_dtype == OI_BF16 && out_dtype == OI_BF16)),
             "rglru_gates: matrices and results of types %d and %d are not covered",
             w_dtype, out_dtype);
  if (tokens == 0) return OI_OK;
  GateArgs p{u, w, bias, rate, ab, y, y_bias, out, state, cu_seqlens, token_req, state_slots, ld_u, ld_ab, ld_y, ld_out, state_stride,
             col_step, tokens, blocks, size, 0};
  cudaStream_t s = (cudaStream_t)stream;
  if (w_dtype == OI_F32) {
    const dim3 grid((tokens + kFm - 1) / kFm, blocks * ((size + kFn - 1) / kFn));
    if (out_dtype == OI_F32) oi_launch(rglru_gates_f32_kernel<float>, grid, 256, 0, s, p);
    else oi_launch(rglru_gates_f32_kernel<bf16>, grid, 256, 0, s, p);
    OI_CHECK_LAUNCH();
    return OI_OK;
  }
  p.vec = size % 8 == 0 && ld_u % 4 == 0 && ld_ab % 2 == 0 && col_step % 2 == 0 && ((uintptr_t)u & 15) == 0 && ((uintptr_t)w & 15) == 0 &&
          ((uintptr_t)bias & 7) == 0 && ((uintptr_t)rate & 7) == 0 && ((uintptr_t)ab & 7) == 0;
  // (batch-invariant mode: one kernel whatever the step's size)
  if (p.vec && tokens <= kFewRows && size <= kFewSize && !oi_option(OI_OPT_BATCH_INVARIANT)) {
    const size_t smem = (size_t)(tokens < 32 ? tokens : 32) * size * sizeof(float);
    static bool few_configured = false;
    if (!few_configured) {
      OI_CHECK_CUDA(cudaFuncSetAttribute(rglru_gates_few_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 32 * kFewSize * (int)sizeof(float)));
      few_configured = true;
    }
    oi_launch(rglru_gates_few_kernel, blocks * ((size + kFewWarps - 1) / kFewWarps), kFewWarps * 32, smem, s, p);
    OI_CHECK_LAUNCH();
    return OI_OK;
  }
  const dim3 grid((tokens + kM - 1) / kM, blocks * ((size + kN - 1) / kN));
  static bool configured = false;
  if (!configured) {
    OI_CHECK_CUDA(cudaFuncSetAttribute(rglru_gates_mma_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sizeof(GateTile)));
    configured = true;
  }
  oi_launch(rglru_gates_mma_kernel, grid, 256, sizeof(GateTile), s, p);
  OI_CHECK_LAUNCH();
  return OI_OK;
}
