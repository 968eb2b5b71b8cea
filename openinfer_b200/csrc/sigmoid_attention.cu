// Attention whose weights are sigmoids, not normalised over the keys, over the paged cache; what its layer does around it.
//
//   joint_norm_rope_store_kernel  one block per row of the fused projection: q over ALL its heads divided by its root mean
//                                 square and multiplied by a weight, k likewise; the first 2 * rot_half numbers of every head
//                                 turned in neighbouring pairs (2 n, 2 n + 1) by the position's angles; q back in place, k and
//                                 v (which may be the k columns as projected) to the row's page slot.
//   sigmoid_attention_kernel      the general form: any head size that is a multiple of eight, any heads and groups, float32
//                                 or bfloat16 storage. One block per row with all its heads, because mixing makes every head's
//                                 weights depend on all heads' scores:
//                                   x_h(j) = scale * sum_g T[h, g] (q_g . k_c(g),j) + bias_h,  w = 1 / (1 + e^-x),  j <= pos,
//                                   o_h = sum_j w_h(j) v_c(h),j, times sigmoid(gate) where a gate is given.
//                                 The keys are visited 32 at a time in position order, whatever else is in the batch.
//   slice_sum_gate_kernel         adds up the partial results that key slices of a row left (csrc/sigmoid_attention_mma.cu)
//                                 and applies the gate.
//
// All arithmetic is float32 with one rounding at the output.
#include "oi_api.h"

namespace {

constexpr int kThreads = 256;

__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }

template <typename T>
__device__ __forceinline__ void load8(const T* p, float (&v)[8]);
template <>
__device__ __forceinline__ void load8<float>(const float* p, float (&v)[8]) {
  const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
  v[0] = a.x, v[1] = a.y, v[2] = a.z, v[3] = a.w, v[4] = b.x, v[5] = b.y, v[6] = b.z, v[7] = b.w;
}
template <>
__device__ __forceinline__ void load8<bf16>(const bf16* p, float (&v)[8]) {
  const uint4 t = *reinterpret_cast<const uint4*>(p);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&t);
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    const float2 f = __bfloat1622float2(h[k]);
    v[2 * k] = f.x, v[2 * k + 1] = f.y;
  }
}
__device__ __forceinline__ void store8(float* p, const float (&v)[8]) {
  reinterpret_cast<float4*>(p)[0] = make_float4(v[0], v[1], v[2], v[3]);
  reinterpret_cast<float4*>(p)[1] = make_float4(v[4], v[5], v[6], v[7]);
}
__device__ __forceinline__ void store8(bf16* p, const float (&v)[8]) {
  uint4 t;
  __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&t);
#pragma unroll
  for (int k = 0; k < 4; ++k) h[k] = __floats2bfloat162_rn(v[2 * k], v[2 * k + 1]);
  *reinterpret_cast<uint4*>(p) = t;
}

// eight neighbouring numbers of a head, starting at number d of it: scaled by inv * weight (or as they are), then turned
__device__ __forceinline__ void norm_and_turn(float (&x)[8], float inv, const float* w, int d, const float* cos_row,
                                              const float* sin_row, int rot_half) {
  if (w) {
    float wv[8];
    load8<float>(w, wv);
#pragma unroll
    for (int e = 0; e < 8; ++e) x[e] = x[e] * inv * wv[e];
  }
  const int n0 = d >> 1;
  if (n0 >= rot_half) return;
  float c[4], s[4];
  if (rot_half % 4 == 0) {                     // the angles of four pairs at a time
    const float4 c4 = *reinterpret_cast<const float4*>(cos_row + n0), s4 = *reinterpret_cast<const float4*>(sin_row + n0);
    c[0] = c4.x, c[1] = c4.y, c[2] = c4.z, c[3] = c4.w;
    s[0] = s4.x, s[1] = s4.y, s[2] = s4.z, s[3] = s4.w;
  } else {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const bool in = n0 + e < rot_half;
      c[e] = in ? cos_row[n0 + e] : 1.f;
      s[e] = in ? sin_row[n0 + e] : 0.f;
    }
  }
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const float u = x[2 * e], v = x[2 * e + 1];
    x[2 * e] = u * c[e] - v * s[e];
    x[2 * e + 1] = v * c[e] + u * s[e];
  }
}

// Two sums over the block at once. `red` holds 64 floats.
__device__ __forceinline__ void block_sum2(float& a, float& b, float* red) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = (blockDim.x + 31) >> 5;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    a += __shfl_xor_sync(0xffffffffu, a, o);
    b += __shfl_xor_sync(0xffffffffu, b, o);
  }
  if (lane == 0) red[warp] = a, red[32 + warp] = b;
  __syncthreads();
  a = b = 0.f;
  for (int w = 0; w < warps; ++w) a += red[w], b += red[32 + w];
}

// kKeep: eights of q | k a thread keeps in registers between the sum and the turn (0: they are read again)
template <typename T, int kKeep>
__global__ void __launch_bounds__(kThreads)
joint_norm_rope_store_kernel(T* __restrict__ proj, long long row_stride, int nq, int nkv, int hd, int qk_dim, int k_off, int v_off,
                             const float* __restrict__ q_w, const float* __restrict__ k_w, float eps,
                             const float* __restrict__ cos_tab, const float* __restrict__ sin_tab, int rot_half, int max_pos,
                             const int* __restrict__ positions, const int* __restrict__ slots, T* __restrict__ k_cache,
                             T* __restrict__ v_cache, long long page_stride, int page_size) {
  pdl_start();
  __shared__ float red[64];
  const int t = blockIdx.x, step = blockDim.x;
  T* row = proj + (size_t)t * row_stride;
  const int q8 = nq * hd / 8, k8 = nkv * hd / 8;
  const int slot = slots[t];
  int pos = positions[t];
  float keep[kKeep ? kKeep : 1][8];
  auto source = [&](int i) { return i < q8 ? row + (size_t)i * 8 : row + k_off + (size_t)(i - q8) * 8; };
  float q_inv = 1.f, k_inv = 1.f;
  if (q_w || kKeep) {
    float qs = 0.f, ks = 0.f;
    auto add = [&](int i, const float (&x)[8]) {
      float s = 0.f;
#pragma unroll
      for (int e = 0; e < 8; ++e) s += x[e] * x[e];
      if (i < q8) qs += s; else ks += s;
    };
    if (kKeep) {
#pragma unroll
      for (int n = 0; n < kKeep; ++n) {
        const int i = threadIdx.x + n * step;
        if (i < q8 + k8) load8<T>(source(i), keep[n]);
      }
#pragma unroll
      for (int n = 0; n < kKeep; ++n)
        if ((int)threadIdx.x + n * step < q8 + k8) add(threadIdx.x + n * step, keep[n]);
    } else {
      for (int i = threadIdx.x; i < q8 + k8; i += step) {
        float x[8];
        load8<T>(source(i), x);
        add(i, x);
      }
    }
    if (q_w) {
      block_sum2(qs, ks, red);
      q_inv = 1.f / sqrtf(qs / (float)(nq * qk_dim) + eps);
      k_inv = 1.f / sqrtf(ks / (float)(nkv * qk_dim) + eps);
    }
  }
  pos = pos < 0 ? 0 : (rot_half > 0 && pos >= max_pos ? max_pos - 1 : pos);      // admission bounds positions
  const float* cr = rot_half > 0 ? cos_tab + (size_t)pos * rot_half : nullptr;
  const float* sr = rot_half > 0 ? sin_tab + (size_t)pos * rot_half : nullptr;
  const size_t at = slot >= 0 ? (size_t)(slot / page_size) * page_stride + (size_t)(slot % page_size) * nkv * hd : 0;
  auto finish = [&](int i, float (&x)[8]) {
    if (i < q8) {
      const int c = i * 8;
      norm_and_turn(x, q_inv, q_w ? q_w + c : nullptr, c % hd, cr, sr, rot_half);
      store8(row + c, x);
      return;
    }
    if (slot < 0) return;                                       // a padding row stores nothing
    const int c = (i - q8) * 8;
    if (v_off == k_off) store8(v_cache + at + c, x);            // the value is the key as projected
    norm_and_turn(x, k_inv, k_w ? k_w + c : nullptr, c % hd, cr, sr, rot_half);
    store8(k_cache + at + c, x);
  };
  if (kKeep) {
#pragma unroll
    for (int n = 0; n < kKeep; ++n)
      if ((int)threadIdx.x + n * step < q8 + k8) finish(threadIdx.x + n * step, keep[n]);
  } else {
    for (int i = threadIdx.x; i < q8 + k8; i += step) {
      float x[8];
      load8<T>(source(i), x);
      finish(i, x);
    }
  }
  if (v_off != k_off && slot >= 0)
    for (int i = threadIdx.x; i < k8; i += step) {
      float x[8];
      load8<T>(row + v_off + (size_t)i * 8, x);
      store8(v_cache + at + (size_t)i * 8, x);
    }
}

constexpr int kChunk = 32;     // keys at a time

template <typename T>
__global__ void __launch_bounds__(kThreads)
sigmoid_attention_kernel(const T* __restrict__ q, long long q_stride, T* __restrict__ out, long long out_stride,
                         const T* __restrict__ gate, long long gate_stride, const T* __restrict__ k_cache,
                         const T* __restrict__ v_cache, long long page_stride, int page_size, const int* __restrict__ block_table,
                         int bt_stride, const int* __restrict__ token_req, const int* __restrict__ positions, int nq, int nkv, int hd,
                         float scale, const float* __restrict__ mix, const float* __restrict__ bias) {
  pdl_start();
  extern __shared__ float sh[];
  const int token = blockIdx.x;
  const int req = token_req[token];
  if (req < 0) return;                        // a padding row
  float* qs = sh;                             // [nq * hd]
  float* acc = qs + nq * hd;                  // [nq * hd]
  float* raw = acc + nq * hd;                 // [nq][kChunk + 1] dot products
  float* w = raw + nq * (kChunk + 1);         // [nq][kChunk + 1] weights
  __shared__ long long where[kChunk];         // offset of a key's row in the layer's pages
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, warps = blockDim.x >> 5;
  const int group = nq / nkv, pos = positions[token];
  const int* bt = block_table + (size_t)req * bt_stride;
  for (int i = tid; i < nq * hd; i += blockDim.x) {
    qs[i] = to_f32(q[(size_t)token * q_stride + i]);
    acc[i] = 0.f;
  }
  for (int base = 0; base <= pos; base += kChunk) {
    const int n = min(kChunk, pos + 1 - base);
    if (tid < n) where[tid] = (long long)bt[(base + tid) / page_size] * page_stride + (long long)((base + tid) % page_size) * nkv * hd;
    __syncthreads();                          // also: q and the last chunk's weights are done with
    for (int h = warp; h < nq; h += warps) {
      float dot = 0.f;
      if (lane < n) {
        const T* kp = k_cache + where[lane] + (size_t)(h / group) * hd;
        const float* qh = qs + h * hd;
        for (int d = 0; d < hd; d += 8) {
          float kv[8];
          load8<T>(kp + d, kv);
#pragma unroll
          for (int e = 0; e < 8; ++e) dot += qh[d + e] * kv[e];
        }
      }
      raw[h * (kChunk + 1) + lane] = dot;
    }
    __syncthreads();
    for (int i = tid; i < nq * kChunk; i += blockDim.x) {
      const int h = i / kChunk, j = i % kChunk;
      float x = 0.f;
      for (int g = 0; g < nq; ++g) x += mix[h * nq + g] * (raw[g * (kChunk + 1) + j] * scale);
      w[h * (kChunk + 1) + j] = j < n ? sigmoid_f(x + bias[h]) : 0.f;
    }
    __syncthreads();
    for (int i = tid; i < nq * hd; i += blockDim.x) {
      const int h = i / hd, d = i - h * hd;
      const T* vp = v_cache + (size_t)(h / group) * hd + d;
      const float* wh = w + h * (kChunk + 1);
      float a = 0.f;
      for (int j = 0; j < n; ++j) a += wh[j] * to_f32(vp[where[j]]);
      acc[i] += a;
    }
    __syncthreads();
  }
  for (int i = tid; i < nq * hd; i += blockDim.x) {
    float o = acc[i];
    if (gate) o *= sigmoid_f(to_f32(gate[(size_t)token * gate_stride + i]));
    out[(size_t)token * out_stride + i] = from_f32<T>(o);
  }
}

// out[t] = sigmoid(gate[t]) * sum_s part[row_base[t] + s], for the rows whose keys were cut into more than one slice. kWays
// neighbouring warps share 128 columns, each adding up every kWays-th slice.
template <typename T, int kWays>
__global__ void __launch_bounds__(kThreads)
slice_sum_gate_kernel(const float* __restrict__ part, const int* __restrict__ row_splits, const int* __restrict__ row_base,
                      T* __restrict__ out, long long out_stride, const T* __restrict__ gate, long long gate_stride, int cols) {
  pdl_start();
  __shared__ float4 sums[kWays > 1 ? kThreads : 1];
  const int t = blockIdx.x, n = row_splits[t];
  if (n <= 1) return;
  const int lane = threadIdx.x & 31, way = (threadIdx.x >> 5) % kWays;
  const int c = ((blockIdx.y * (blockDim.x / (32 * kWays)) + (threadIdx.x >> 5) / kWays) * 32 + lane) * 4;
  const float* p = part + (size_t)row_base[t] * cols;
  float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
  if (c < cols) {
#pragma unroll 4
    for (int s = way; s < n; s += kWays) {
      const float4 v = *reinterpret_cast<const float4*>(p + (size_t)s * cols + c);
      a.x += v.x, a.y += v.y, a.z += v.z, a.w += v.w;
    }
  }
  if (kWays > 1) {
    sums[threadIdx.x] = a;
    __syncthreads();
    if (way != 0) return;
#pragma unroll
    for (int w = 1; w < kWays; ++w) {
      const float4 v = sums[threadIdx.x + w * 32];
      a.x += v.x, a.y += v.y, a.z += v.z, a.w += v.w;
    }
  }
  if (c >= cols) return;
  float o[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    if (gate) o[e] *= sigmoid_f(to_f32(gate[(size_t)t * gate_stride + c + e]));
    out[(size_t)t * out_stride + c + e] = from_f32<T>(o[e]);
  }
}

bool aligned16(const void* p) { return ((uintptr_t)p & 15) == 0; }

}  // namespace

OI_API int oi_joint_norm_rope_store(void* proj, int dtype, long long row_stride, int tokens, int nq, int nkv, int hd, int qk_dim,
                                    int k_off, int v_off, const float* q_w, const float* k_w, float eps, const float* cos_tab,
                                    const float* sin_tab, int rot_half, int max_pos, const int* positions, const int* slots,
                                    void* k_cache, void* v_cache, long long page_stride, int page_size, void* stream) {
  OI_REQUIRE(tokens >= 0 && nq > 0 && nkv > 0 && hd > 0 && hd % 8 == 0 && qk_dim > 0 && qk_dim <= hd && k_off % 8 == 0 && v_off % 8 == 0,
             "joint_norm_rope_store: bad sizes nq=%d nkv=%d hd=%d qk_dim=%d", nq, nkv, hd, qk_dim);
  OI_REQUIRE((q_w == nullptr) == (k_w == nullptr), "joint_norm_rope_store: the two norms come together or not at all");
  OI_REQUIRE(rot_half >= 0 && 2 * rot_half <= hd && (rot_half == 0 || (cos_tab && sin_tab && max_pos > 0)),
             "joint_norm_rope_store: %d rotated pairs in a head of %d numbers, or no tables", rot_half, hd);
  OI_REQUIRE(positions && slots && k_cache && v_cache && page_size > 0, "joint_norm_rope_store: positions, slots and pages are needed");
  OI_REQUIRE(row_stride % 8 == 0 && page_stride % 8 == 0 && aligned16(proj) && aligned16(k_cache) && aligned16(v_cache) &&
             aligned16(q_w) && aligned16(k_w) && aligned16(cos_tab) && aligned16(sin_tab), "joint_norm_rope_store: rows and pages must be readable 16 bytes at a time");
  if (tokens == 0) return OI_OK;
  cudaStream_t s = (cudaStream_t)stream;
  // a row's eights over the threads as evenly as whole warps allow, one or two a thread where that suffices
  const int work = (nq + nkv) * hd / 8, keep = work <= kThreads ? 1 : (work <= 2 * kThreads ? 2 : (work <= 4 * kThreads ? 4 : 0));
  const int threads = keep ? ((work + keep - 1) / keep + 31) / 32 * 32 : kThreads;
#define OI_JNRS(T)                                                                                                         \
  do {                                                                                                                     \
    if (keep == 1) OI_JNRS_K(T, 1); else if (keep == 2) OI_JNRS_K(T, 2); else if (keep == 4) OI_JNRS_K(T, 4); else OI_JNRS_K(T, 0); \
  } while (0)
#define OI_JNRS_K(T, KEEP)                                                                                                 \
  oi_launch(joint_norm_rope_store_kernel<T, KEEP>, tokens, threads, 0, s, (T*)proj, row_stride, nq, nkv, hd, qk_dim, k_off, v_off, q_w, \
            k_w, eps, cos_tab, sin_tab, rot_half, max_pos, positions, slots, (T*)k_cache, (T*)v_cache, page_stride, page_size)
  if (dtype == OI_F32) OI_JNRS(float);
  else if (dtype == OI_BF16) OI_JNRS(bf16);
  else OI_REQUIRE(false, "joint_norm_rope_store: unknown dtype code %d", dtype);
#undef OI_JNRS
#undef OI_JNRS_K
  OI_CHECK_LAUNCH();
  return OI_OK;
}

OI_API int oi_sigmoid_attention(const void* q, long long q_stride, void* out, long long out_stride, const void* gate,
                                long long gate_stride, int dtype, const void* k_cache, const void* v_cache, long long page_stride,
                                int page_size, const int* block_table, int bt_stride, const int* token_req, const int* positions,
                                int tokens, int nq, int nkv, int hd, float scale, const float* mix, const float* bias, void* stream) {
  OI_REQUIRE(tokens >= 0 && nq > 0 && nkv > 0 && nq % nkv == 0 && hd > 0 && hd % 8 == 0, "sigmoid_attention: bad sizes nq=%d nkv=%d hd=%d",
             nq, nkv, hd);
  OI_REQUIRE(mix && bias && page_size > 0 && page_stride % 8 == 0 && aligned16(k_cache) && aligned16(v_cache),
             "sigmoid_attention: the head mix, the biases and aligned pages are needed");
  const size_t smem = ((size_t)2 * nq * hd + (size_t)2 * nq * (kChunk + 1)) * sizeof(float);
  OI_REQUIRE(smem <= 200 * 1024, "sigmoid_attention: %d heads of %d numbers do not fit a block", nq, hd);
  if (tokens == 0) return OI_OK;
  cudaStream_t s = (cudaStream_t)stream;
#define OI_SIG(T)                                                                                                            \
  do {                                                                                                                       \
    if (smem > 40 * 1024)                                                                                                    \
      OI_CHECK_CUDA(cudaFuncSetAttribute(sigmoid_attention_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024)); \
    oi_launch(sigmoid_attention_kernel<T>, tokens, kThreads, smem, s, (const T*)q, q_stride, (T*)out, out_stride, (const T*)gate, \
              gate_stride, (const T*)k_cache, (const T*)v_cache, page_stride, page_size, block_table, bt_stride, token_req, positions, \
              nq, nkv, hd, scale, mix, bias);                                                                                \
  } while (0)
  if (dtype == OI_F32) OI_SIG(float);
  else if (dtype == OI_BF16) OI_SIG(bf16);
  else OI_REQUIRE(false, "sigmoid_attention: unknown dtype code %d", dtype);
#undef OI_SIG
  OI_CHECK_LAUNCH();
  return OI_OK;
}

OI_API int oi_slice_sum_gate(const float* part, const int* row_splits, const int* row_base, void* out, int dtype, long long out_stride,
                             const void* gate, long long gate_stride, int tokens, int cols, void* stream) {
  OI_REQUIRE(tokens >= 0 && cols > 0 && cols % 4 == 0 && aligned16(part) && row_splits && row_base, "slice_sum_gate: bad arguments");
  if (tokens == 0) return OI_OK;
  // few rows (of many slices, in a step of single tokens): several warps a column; many rows: one
  const int ways = tokens <= 256 ? 8 : 1, per_block = kThreads / 32 / ways * 128;
  const dim3 grid(tokens, (cols + per_block - 1) / per_block);
  cudaStream_t s = (cudaStream_t)stream;
#define OI_SSG(T)                                                                                                            \
  do {                                                                                                                       \
    if (ways == 8)                                                                                                           \
      oi_launch(slice_sum_gate_kernel<T, 8>, grid, kThreads, 0, s, part, row_splits, row_base, (T*)out, out_stride, (const T*)gate, \
                gate_stride, cols);                                                                                          \
    else                                                                                                                     \
      oi_launch(slice_sum_gate_kernel<T, 1>, grid, kThreads, 0, s, part, row_splits, row_base, (T*)out, out_stride, (const T*)gate, \
                gate_stride, cols);                                                                                          \
  } while (0)
  if (dtype == OI_F32) OI_SSG(float);
  else if (dtype == OI_BF16) OI_SSG(bf16);
  else OI_REQUIRE(false, "slice_sum_gate: unknown dtype code %d", dtype);
#undef OI_SSG
  OI_CHECK_LAUNCH();
  return OI_OK;
}
