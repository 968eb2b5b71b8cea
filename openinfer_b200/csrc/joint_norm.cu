// The step between the fused q | k | v projection of an attention and its scores, for layers that norm q, and k, over ALL
// their heads together and turn the pairs (d, d + rot_half):
//
//   x <- x + bias;  q, k: x / sqrt(mean over all heads of x^2 + eps) * w, then every head's first 2 * rot_half numbers turned by
//   the position's angles; q back in place, k and v to the row's page slot.
//
// One block a row. A thread takes V neighbouring numbers of a head together with the V numbers they are turned with (behind the
// turned part: V numbers of its first half with V of its second), so that a row is read and written without an exchange
// between threads; up to kKeep such pairs a thread stay in registers between the two sums of squares and the turn. Heads are hd
// numbers apart of which the first qk_dim count; the others are zero in the projection, the bias and the weights.
#include "oi_api.h"

namespace {

template <int V, typename T>
__device__ __forceinline__ void load_v(const T* p, float (&v)[V]) {
  if (V == 8 && sizeof(T) == 2) {
    const uint4 t = *reinterpret_cast<const uint4*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&t);
#pragma unroll
    for (int k = 0; k < V / 2; ++k) {
      const float2 f = __bfloat1622float2(h[k]);
      v[2 * k] = f.x, v[2 * k + 1] = f.y;
    }
  } else if (V == 4 && sizeof(T) == 2) {
    const uint2 t = *reinterpret_cast<const uint2*>(p);
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&t);
#pragma unroll
    for (int k = 0; k < V / 2; ++k) {
      const float2 f = __bfloat1622float2(h[k]);
      v[2 * k] = f.x, v[2 * k + 1] = f.y;
    }
  } else if (V % 4 == 0 && sizeof(T) == 4) {
#pragma unroll
    for (int k = 0; k < V / 4; ++k) {
      const float4 t = reinterpret_cast<const float4*>(p)[k];
      v[4 * k] = t.x, v[4 * k + 1] = t.y, v[4 * k + 2] = t.z, v[4 * k + 3] = t.w;
    }
  } else {
#pragma unroll
    for (int k = 0; k < V; ++k) v[k] = to_f32(p[k]);
  }
}
template <int V, typename T>
__device__ __forceinline__ void store_v(T* p, const float (&v)[V]) {
  if (V % 4 == 0 && sizeof(T) == 2) {
    unsigned t[V / 2 > 0 ? V / 2 : 1];
#pragma unroll
    for (int k = 0; k < V / 2; ++k) {
      const __nv_bfloat162 h = __floats2bfloat162_rn(v[2 * k], v[2 * k + 1]);
      t[k] = *reinterpret_cast<const unsigned*>(&h);
    }
    if (V == 8) *reinterpret_cast<uint4*>(p) = make_uint4(t[0], t[1], t[V > 4 ? 2 : 0], t[V > 4 ? 3 : 0]);
    else *reinterpret_cast<uint2*>(p) = make_uint2(t[0], t[V >= 4 ? 1 : 0]);
  } else if (V % 4 == 0 && sizeof(T) == 4) {
#pragma unroll
    for (int k = 0; k < V / 4; ++k) reinterpret_cast<float4*>(p)[k] = make_float4(v[4 * k], v[4 * k + 1], v[4 * k + 2], v[4 * k + 3]);
  } else {
#pragma unroll
    for (int k = 0; k < V; ++k) p[k] = from_f32<T>(v[k]);
  }
}

// two sums over the block at once; `red` holds 64 floats
__device__ __forceinline__ void block_sum2(float& a, float& b, float* red) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = (blockDim.x + 31) >> 5;
  a = warp_sum(a), b = warp_sum(b);
  if (lane == 0) red[warp] = a, red[32 + warp] = b;
  __syncthreads();
  a = b = 0.f;
  for (int w = 0; w < warps; ++w) a += red[w], b += red[32 + w];
}

struct JointArgs {
  long long row_stride, page_stride;
  const float* bias;      // [(nq + 2 nkv) * hd] or null
  const float* q_w;       // [nq * hd]
  const float* k_w;       // [nkv * hd]
  const float* cos_tab;
  const float* sin_tab;
  const int* positions;
  const int* slots;
  int nq, nkv, hd, qk_dim, rot_half, max_pos, page_size;
  float eps;
};

template <typename T, int V, int kKeep>
__global__ void __launch_bounds__(256) joint_norm_half_store_kernel(T* __restrict__ qkv, T* __restrict__ k_cache, T* __restrict__ v_cache,
                                                                    const JointArgs p) {
  pdl_start();
  __shared__ float red[64];
  const int t = blockIdx.x, step = blockDim.x, hd = p.hd;
  T* row = qkv + (size_t)t * p.row_stride;
  const int per = hd / (2 * V), turned = p.rot_half / V;      // pairs of a head, and how many of them are turned
  const int q_items = p.nq * per, items = q_items + p.nkv * per;
  const int rest_half = (hd - 2 * p.rot_half) / 2;
  const int slot = p.slots[t];
  int pos = p.positions[t];
  pos = pos < 0 ? 0 : (p.rot_half > 0 && pos >= p.max_pos ? p.max_pos - 1 : pos);      // admission bounds positions
  // the columns of item i: c and c + gap of the row (k heads lie behind the q heads)
  auto column = [&](int i, int& gap) {
    const int head = i / per, n = i - head * per;
    gap = n < turned ? p.rot_half : rest_half;
    return head * hd + (n < turned ? n * V : 2 * p.rot_half + (n - turned) * V);
  };
  auto load = [&](int i, float (&x)[V], float (&y)[V]) {
    int gap;
    const int c = column(i, gap);
    load_v<V>(row + c, x);
    load_v<V>(row + c + gap, y);
    if (p.bias) {
      float b[V];
      load_v<V>(p.bias + c, b);
#pragma unroll
      for (int e = 0; e < V; ++e) x[e] += b[e];
      load_v<V>(p.bias + c + gap, b);
#pragma unroll
      for (int e = 0; e < V; ++e) y[e] += b[e];
    }
  };
  float X[kKeep > 0 ? kKeep : 1][V], Y[kKeep > 0 ? kKeep : 1][V];
  float qs = 0.f, ks = 0.f;
  auto add = [&](int i, const float (&x)[V], const float (&y)[V]) {
    float s = 0.f;
#pragma unroll
    for (int e = 0; e < V; ++e) s += x[e] * x[e] + y[e] * y[e];
    if (i < q_items) qs += s; else ks += s;
  };
  if (kKeep > 0) {
#pragma unroll
    for (int n = 0; n < kKeep; ++n)
      if ((int)threadIdx.x + n * step < items) load(threadIdx.x + n * step, X[n], Y[n]);
#pragma unroll
    for (int n = 0; n < kKeep; ++n)
      if ((int)threadIdx.x + n * step < items) add(threadIdx.x + n * step, X[n], Y[n]);
  } else {
    for (int i = threadIdx.x; i < items; i += step) {
      load(i, X[0], Y[0]);
      add(i, X[0], Y[0]);
    }
  }
  block_sum2(qs, ks, red);
  const float q_inv = 1.f / sqrtf(qs / (float)(p.nq * p.qk_dim) + p.eps), k_inv = 1.f / sqrtf(ks / (float)(p.nkv * p.qk_dim) + p.eps);
  const float* cr = p.rot_half > 0 ? p.cos_tab + (size_t)pos * p.rot_half : nullptr;
  const float* sr = p.rot_half > 0 ? p.sin_tab + (size_t)pos * p.rot_half : nullptr;
  const size_t at = slot >= 0 ? (size_t)(slot / p.page_size) * p.page_stride + (size_t)(slot % p.page_size) * p.nkv * hd : 0;
  auto finish = [&](int i, float (&x)[V], float (&y)[V]) {
    const bool is_q = i < q_items;
    if (!is_q && slot < 0) return;                            // a padding row stores nothing
    int gap;
    const int c = column(i, gap), own = is_q ? c : c - p.nq * hd;
    const float* w = is_q ? p.q_w + own : p.k_w + own;
    const float inv = is_q ? q_inv : k_inv;
    float a[V], b[V];
    load_v<V>(w, a);
    load_v<V>(w + gap, b);
#pragma unroll
    for (int e = 0; e < V; ++e) x[e] *= inv * a[e], y[e] *= inv * b[e];
    const int n = i % per;
    if (n < turned) {
      load_v<V>(cr + n * V, a);
      load_v<V>(sr + n * V, b);
#pragma unroll
      for (int e = 0; e < V; ++e) {
        const float u = x[e], v = y[e];
        x[e] = u * a[e] - v * b[e];
        y[e] = v * a[e] + u * b[e];
      }
    }
    T* dst = is_q ? row + own : k_cache + at + own;
    store_v<V>(dst, x);
    store_v<V>(dst + gap, y);
  };
  if (kKeep > 0) {
#pragma unroll
    for (int n = 0; n < kKeep; ++n)
      if ((int)threadIdx.x + n * step < items) finish(threadIdx.x + n * step, X[n], Y[n]);
  } else {
    for (int i = threadIdx.x; i < items; i += step) {
      load(i, X[0], Y[0]);
      finish(i, X[0], Y[0]);
    }
  }
  if (slot < 0) return;
  const int v0 = (p.nq + p.nkv) * hd;
  for (int i = threadIdx.x; i < p.nkv * hd / V; i += step) {
    float x[V], b[V];
    load_v<V>(row + v0 + (size_t)i * V, x);
    if (p.bias) {
      load_v<V>(p.bias + v0 + (size_t)i * V, b);
#pragma unroll
      for (int e = 0; e < V; ++e) x[e] += b[e];
    }
    store_v<V>(v_cache + at + (size_t)i * V, x);
  }
}

}  // namespace

// qkv [tokens, row_stride]: heads of hd numbers, nq query heads, nkv key heads, nkv value heads; bias float32 [(nq + 2 nkv) * hd]
// or null; q_w [nq * hd], k_w [nkv * hd] float32; cos / sin float32 [max_pos, rot_half] or null (rot_half 0).
OI_API int oi_joint_norm_half_store(void* qkv, int dtype, long long row_stride, int tokens, int nq, int nkv, int hd, int qk_dim,
                                    const float* bias, const float* q_w, const float* k_w, float eps, const float* cos_tab,
                                    const float* sin_tab, int rot_half, int max_pos, const int* positions, const int* slots,
                                    void* k_cache, void* v_cache, long long page_stride, int page_size, void* stream) {
  OI_REQUIRE(tokens >= 0 && nq > 0 && nkv > 0 && hd > 0 && hd % 8 == 0 && qk_dim > 0 && qk_dim <= hd && row_stride >= (long long)(nq + 2 * nkv) * hd,
             "joint_norm_half_store: bad sizes nq=%d nkv=%d hd=%d qk_dim=%d", nq, nkv, hd, qk_dim);
  OI_REQUIRE(rot_half >= 0 && 2 * rot_half <= hd && (rot_half == 0 || (cos_tab && sin_tab && max_pos > 0)),
             "joint_norm_half_store: %d turned pairs in a head of %d numbers, or no tables", rot_half, hd);
  OI_REQUIRE(q_w && k_w && positions && slots && k_cache && v_cache && page_size > 0, "joint_norm_half_store: a tensor is missing");
  if (tokens == 0) return OI_OK;
  const JointArgs a{row_stride, page_stride, bias, q_w, k_w, cos_tab, sin_tab, positions, slots, nq, nkv, hd, qk_dim, rot_half, max_pos,
                    page_size, eps};
  cudaStream_t s = (cudaStream_t)stream;
  auto al = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
  const int elem = dtype == OI_F32 ? 4 : 2;
  const bool ok = al(qkv) && al(k_cache) && al(v_cache) && al(bias) && al(q_w) && al(k_w) && al(cos_tab) && al(sin_tab) &&
                  (row_stride * elem) % 16 == 0 && (page_stride * elem) % 16 == 0;
  const int rest = hd - 2 * rot_half;
  const int V = ok && rot_half % 8 == 0 && rest % 16 == 0 ? 8 : (ok && rot_half % 4 == 0 && rest % 8 == 0 ? 4 : 1);
  const int items = (nq + nkv) * hd / (2 * V);
  const int threads = items >= 256 ? 256 : ((items + 31) / 32) * 32;
  const int keep = items <= threads ? 1 : (items <= 2 * threads ? 2 : 0);
#define OI_JOINT(T, VV)                                                                                                       \
  do {                                                                                                                        \
    if (keep == 1) oi_launch(joint_norm_half_store_kernel<T, VV, 1>, tokens, threads, 0, s, (T*)qkv, (T*)k_cache, (T*)v_cache, a); \
    else if (keep == 2) oi_launch(joint_norm_half_store_kernel<T, VV, 2>, tokens, threads, 0, s, (T*)qkv, (T*)k_cache, (T*)v_cache, a); \
    else oi_launch(joint_norm_half_store_kernel<T, VV, 0>, tokens, threads, 0, s, (T*)qkv, (T*)k_cache, (T*)v_cache, a);       \
  } while (0)
#define OI_JOINT_T(T)                                                          \
  do {                                                                         \
    if (V == 8) OI_JOINT(T, 8); else if (V == 4) OI_JOINT(T, 4); else OI_JOINT(T, 1); \
  } while (0)
  if (dtype == OI_F32) OI_JOINT_T(float);
  else if (dtype == OI_BF16) OI_JOINT_T(bf16);
  else OI_REQUIRE(false, "joint_norm_half_store: unknown dtype code %d", dtype);
#undef OI_JOINT_T
#undef OI_JOINT
  OI_CHECK_LAUNCH();
  return OI_OK;
}
