// Attention with sigmoid weights (see sigmoid_attention.cu) on tensor cores, for bfloat16, heads of 32, 64 or 128 numbers and
// up to 32 heads: prompt portions and split decode.
//
// Mixing the heads' scores makes every weight depend on all heads' scores for the same query and key, so a warp holds ALL
// heads of its queries. Everything is laid out so that the three products chain in registers:
//
//   S^T = K Q^T      mma m16n8k16: 16 keys x 8 columns. A column is a (head, token): four heads x two neighbouring tokens in
//                    prompt tiles (column 2 * head + token), eight heads of the one token in decode.
//   X^T = S^T T^T    mma m16n8k8 (tf32): the accumulators of S^T are its left operand as they lie, a thread's four numbers of
//                    a pair of tiles being (key, key + 8) x (head t, head t + 4) once the sum over heads is taken in a suited
//                    order. S is split into two tf32 numbers (T, with its 8 bits of mantissa, is one as it is), so that
//                    the mix is as exact as float32.
//   w = sigmoid      float32: 1 / (1 + 2^-(...)), scale and bias in one multiply-add; masked keys weigh zero.
//   O^T += V^T w     mma m16n8k16: V^T by transposing ldmatrix, w^T rounded to bfloat16 and transposed by movmatrix.
//
// When the query heads of a kv head do not fill whole column tiles, a tile is multiplied once per kv head with the other
// heads' columns set to zero. The sums have neither a maximum nor a denominator: the results of key slices are simply added
// up (slice_sum_gate_kernel), and an item that is the only slice of its rows applies the gate and writes them itself.
//
// Tile kernel: a warp's columns are four heads x four tokens; the warps that share the tokens exchange their raw scores. A CTA
// of 16 warps owns 32, 16 or 8 tokens of a request; K and V of 32 keys (all kv heads) are staged in turns by cp.async,
// swizzled, several stages deep.
// Decode kernel: a CTA owns a slice of the keys of one token, its warps take 16 keys in turn, each through a private ring of
// cp.async stages of one kv head's 16 rows, and add their sums up in shared memory at the end.
#include "oi_api.h"

namespace {

constexpr int kTile = 16;              // keys of a step
constexpr float kLog2eF = 1.4426950408889634f;

struct SigParams {
  const bf16* q; long long q_stride;
  bf16* out; long long out_stride;
  const bf16* gate; long long gate_stride;       // or null
  const bf16* k_cache; const bf16* v_cache; long long page_stride; int page_size;     // page_size a multiple of 16
  const int* block_table; int bt_stride;
  const int* cu_seqlens; const int* kv_lens;
  const int4* items;                   // (request, first token of the tile, slice, slices)
  const int* row_base;                 // [tokens] where a row's partial results begin in part
  float* part;                         // [*, nq * HD]
  int nq, nkv, group;
  float neg_scale_log2;                // -scale * log2(e)
  const float* mix;                    // [nq, nq], exact in tf32
  const float* bias;                   // [nq]
};

__device__ __forceinline__ unsigned smem_u32(const void* p) { return (unsigned)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void cp_async16(unsigned dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(dst), "l"(src));
}
__device__ __forceinline__ void cp_async16_or_zero(unsigned dst, const void* src, bool valid) {
  const int n = valid ? 16 : 0;        // source size 0: the 16 bytes are zero-filled
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(dst), "l"(src), "r"(n));
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;\n" ::); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N)); }
__device__ __forceinline__ void ldmatrix_x4(unsigned (&r)[4], unsigned addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x4_trans(unsigned (&r)[4], unsigned addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ unsigned movmatrix_trans(unsigned a) {
  unsigned d;
  asm volatile("movmatrix.sync.aligned.m8n8.trans.b16 %0, %1;\n" : "=r"(d) : "r"(a));
  return d;
}
__device__ __forceinline__ void mma_bf16(float (&c)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void mma_tf32(float (&c)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
  asm volatile("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ float fast_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float fast_rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ unsigned pack_bf16(float lo, float hi) {
  __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<unsigned*>(&v);
}

// Element offset of 16-byte chunk `chunk` of row `row` (a head's HD numbers at `head_off` of a row of `row_elems`): the chunks
// of a head are XORed with the row so that the rows an ldmatrix reads fall into different banks.
template <int HD>
__device__ __forceinline__ int swz(int row, int row_elems, int head_off, int chunk) {
  return row * row_elems + head_off + ((chunk ^ (row & 7 & (HD / 8 - 1))) * 8);
}

// Decode, column tiles of eight heads. S^T[tile] += K_c (16 keys x HD at `k`) times the columns of kv head c; a tile may hold
// query heads of other kv heads too, whose columns are then taken as zero.
template <int HD, int NT>
__device__ __forceinline__ void scores(float (&S)[NT][4], const bf16* k, const bf16* q, int c, int group, int lane) {
  const int lo = c * group / 8, hi = ((c + 1) * group - 1) / 8, mat = lane >> 3, rin = lane & 7;
  const unsigned kb = smem_u32(k), qb = smem_u32(q);
  const int k_row = (mat & 1) * 8 + rin;
  unsigned a[HD / 16][4];
#pragma unroll
  for (int ks = 0; ks < HD / 16; ++ks) ldmatrix_x4(a[ks], kb + swz<HD>(k_row, HD, 0, 2 * ks + (mat >> 1)) * 2);
#pragma unroll
  for (int i = 0; i < NT; ++i) {
    if (i < lo || i > hi) continue;
    const int h = 8 * i + (lane >> 2);
    const bool mine = h >= c * group && h < (c + 1) * group;
    float even[4] = {0.f, 0.f, 0.f, 0.f}, odd[4] = {0.f, 0.f, 0.f, 0.f};     // two chains of products in flight
#pragma unroll
    for (int k2 = 0; k2 < HD / 32; ++k2) {
      unsigned b[4];
      ldmatrix_x4(b, qb + swz<HD>(i * 8 + rin, HD, 0, 4 * k2 + mat) * 2);
#pragma unroll
      for (int r = 0; r < 4; ++r) b[r] = mine ? b[r] : 0u;
      mma_bf16(even, a[2 * k2], b[0], b[1]);
      mma_bf16(odd, a[2 * k2 + 1], b[2], b[3]);
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) S[i][e] += even[e] + odd[e];
  }
}

// O^T[tile] += V_c^T times the weights of kv head c's columns (w0: keys 0-7, w1: keys 8-15)
template <int HD, int NT>
__device__ __forceinline__ void values(float (&O)[NT][HD / 16][4], const bf16* v, const unsigned (&w0)[NT], const unsigned (&w1)[NT], int c,
                                       int group, int lane) {
  const int lo = c * group / 8, hi = ((c + 1) * group - 1) / 8, mat = lane >> 3, rin = lane & 7;
  const unsigned vb = smem_u32(v);
  const int v_row = (mat >> 1) * 8 + rin;
  unsigned a[HD / 16][4];
#pragma unroll
  for (int m = 0; m < HD / 16; ++m) ldmatrix_x4_trans(a[m], vb + swz<HD>(v_row, HD, 0, 2 * m + (mat & 1)) * 2);
#pragma unroll
  for (int i = 0; i < NT; ++i) {
    if (i < lo || i > hi) continue;
    const int h = 8 * i + (lane >> 2);
    const bool mine = h >= c * group && h < (c + 1) * group;
    const unsigned b0 = mine ? w0[i] : 0u, b1 = mine ? w1[i] : 0u;
#pragma unroll
    for (int m = 0; m < HD / 16; ++m) mma_bf16(O[i][m], a[m], b0, b1);
  }
}

__device__ __forceinline__ void split_tf32(float x, unsigned& hi, unsigned& lo) {
  hi = __float_as_uint(x) & 0xffffe000u;
  lo = __float_as_uint(x - __uint_as_float(hi));
}

// The mix's right operand as this thread of the decode kernel holds it: step s of the sum over heads, output tile j.
// k < 4 stands for head 8 s + 2 k, k >= 4 for head 8 s + 2 (k - 4) + 1 (the order in which a thread holds a tile's columns);
// output column n is head 8 j + n.
__device__ __forceinline__ float mix_at(const SigParams& p, int s, int k, int j, int n) {
  const int h = 8 * j + n;
  const int g = 8 * s + (k < 4 ? 2 * k : 2 * (k - 4) + 1);
  return h < p.nq && g < p.nq ? p.mix[h * p.nq + g] : 0.f;
}

__device__ __forceinline__ float weight(float x, float neg_scale_log2, float neg_bias_log2) {
  return fast_rcp(1.f + fast_exp2(fmaf(x, neg_scale_log2, neg_bias_log2)));
}

__device__ __forceinline__ float sigmoid_gate(float g) { return __fdividef(1.f, 1.f + __expf(-g)); }

// ---------------------------------------------------------------------------------------------
// Prompt tiles. NQ: quads of heads. NQ warps share four neighbouring tokens: a warp owns one quad of heads, its columns are
// two tiles of 4 heads x 2 tokens, so a fragment of K or V read from shared memory feeds two products. A step is KT x 16 keys.
// The mix needs all heads of a (16 keys, two tokens) at once, so it is shared out the other way round: the warps leave their
// raw scores in shared memory (lane to lane: the fragments lie alike in all of them), each takes KT of the KT * NQ (16 keys,
// two tokens, eight output heads), forms their weights and leaves them for the warps that own the heads.
// ALIGNED: a quad's query heads share one kv head.
// ---------------------------------------------------------------------------------------------
constexpr int kTileWarps = 16;

template <int HD, int NQ, int KT, bool ALIGNED>
__global__ void __launch_bounds__(kTileWarps * 32, 1) sigmoid_tile_kernel(const SigParams p, int stages) {
  pdl_start();
  extern __shared__ __align__(128) unsigned char smem_raw[];
  constexpr int kGroups = kTileWarps / NQ, head_chunks = HD / 8, kStep = KT * kTile, kSwz = head_chunks - 1 < 7 ? head_chunks - 1 : 7;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, group4 = warp / NQ, quad = warp % NQ;
  const int row_elems = p.nkv * HD, unit = kStep * row_elems;
  bf16* const q_all = reinterpret_cast<bf16*>(smem_raw);
  bf16* const q_sm = q_all + (size_t)warp * 16 * HD;               // this warp's columns: row 8 pair + 2 head + token
  float4* const mail_all = reinterpret_cast<float4*>(q_all + (size_t)kTileWarps * 16 * HD);
  float4* const mail = mail_all + (size_t)group4 * KT * 2 * NQ * 32 + lane;          // [key tile][pair][quad][32 lanes]
  uint2* const wmail_all = reinterpret_cast<uint2*>(mail_all + (size_t)kTileWarps * KT * 2 * 32);
  uint2* const wmail = wmail_all + (size_t)group4 * KT * 2 * NQ * 32 + lane;         // the weights, in the same order
  bf16* const ring = reinterpret_cast<bf16*>(wmail_all + (size_t)kTileWarps * KT * 2 * 32);
  const int4 item = p.items[blockIdx.x];
  const int req = item.x, tok0 = item.y, slice = item.z, slices = item.w;
  const int q_start = p.cu_seqlens[req], q_len = p.cu_seqlens[req + 1] - q_start;
  const int* bt = p.block_table + (size_t)req * p.bt_stride;
  const int tile_toks = min(4 * kGroups, q_len - tok0);
  const int pos0 = p.kv_lens[req] - q_len + tok0;
  const int key_end = pos0 + tile_toks;
  const int span = (key_end + kStep - 1) / kStep;
  const int per = (span + slices - 1) / slices;
  const int t_begin = slice * per, t_end = min(span, t_begin + per);

  // stage u of the ring: K of step t_begin + u / 2 (u even) or its V (u odd); a thread copies chunks of one key's row
  const int units = 2 * max(0, t_end - t_begin);
  constexpr int per_row = kTileWarps * 32 / kStep;
  const int my_row = threadIdx.x / per_row, my_chunk = threadIdx.x % per_row, row_chunks = row_elems / 8;
  const unsigned my_dst = smem_u32(ring) + 2 * swz<HD>(my_row, row_elems, (my_chunk / head_chunks) * HD, my_chunk % head_chunks);
  int requested = 0, rq_slot = 0, rq_key = t_begin * kStep + my_row;
  // the element where this thread's chunks of a step begin, in K's pages as in V's; the page of the step behind it is looked up
  // two stages before its use
  int next_page = units > 0 && rq_key < key_end ? bt[rq_key / p.page_size] : 0;
  size_t at = 0;
  auto request = [&]() {
    if (requested < units) {
      const bool is_v = requested & 1, valid = rq_key < key_end;
      if (!is_v) {
        at = (size_t)next_page * p.page_stride + (size_t)(rq_key % p.page_size) * row_elems + my_chunk * 8;
        next_page = rq_key + kStep < key_end ? bt[(rq_key + kStep) / p.page_size] : 0;
      }
      const bf16* src = (is_v ? p.v_cache : p.k_cache) + at;
      const unsigned dst = my_dst + (unsigned)(rq_slot * unit * 2);
      for (int i = 0; i * per_row + my_chunk < row_chunks; ++i) cp_async16_or_zero(dst + i * per_row * 16, src + i * per_row * 8, valid);
      if (is_v) rq_key += kStep;
    }
    ++requested;
    rq_slot = rq_slot + 1 == stages ? 0 : rq_slot + 1;
    cp_async_commit();
  };
  for (int u = 0; u < stages; ++u) request();

  for (int i = lane; i < 16 * head_chunks; i += 32) {
    const int r = i / head_chunks, ch = i % head_chunks;
    const int h = 4 * quad + ((r & 7) >> 1), tok = 4 * group4 + 2 * (r >> 3) + (r & 1);
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (h < p.nq && tok < tile_toks) v = *reinterpret_cast<const uint4*>(p.q + (size_t)(q_start + tok0 + tok) * p.q_stride + (size_t)h * HD + ch * 8);
    *reinterpret_cast<uint4*>(q_sm + swz<HD>(r, HD, 0, ch)) = v;
  }
  // This warp's share of the mix: item i is output tile it % (NQ / 2) (heads 8 tile ...) of combination it / (NQ / 2) (16 keys
  // and two tokens: key tile * 2 + pair), it = KT quad + i. The right operand: step s of the sum takes heads 8 s + k in
  // order; output column n stands for head 8 tile + 4 (n & 1) + (n >> 1), so that a thread's two columns are head t of the
  // tile's first quad and head t of its second.
  constexpr int kTiles = NQ / 2;
  unsigned T0[KT][kTiles], T1[KT][kTiles];
  float nb[KT][2];
#pragma unroll
  for (int i = 0; i < KT; ++i) {
    const int tile = (KT * quad + i) % kTiles, n = lane >> 2, h = 8 * tile + 4 * (n & 1) + (n >> 1);
#pragma unroll
    for (int s = 0; s < kTiles; ++s) {
      const int g = 8 * s + (lane & 3);
      T0[i][s] = __float_as_uint(h < p.nq && g < p.nq ? p.mix[h * p.nq + g] : 0.f);
      T1[i][s] = __float_as_uint(h < p.nq && g + 4 < p.nq ? p.mix[h * p.nq + g + 4] : 0.f);
    }
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int hh = 8 * tile + 4 * u + (lane & 3);
      nb[i][u] = hh < p.nq ? -p.bias[hh] * kLog2eF : 0.f;
    }
  }
  const int my_head = 4 * quad + (lane & 3);
  const int first_pos = pos0 + 4 * group4, toks = min(4, tile_toks - 4 * group4), last_pos = toks > 0 ? first_pos + toks - 1 : -1;
  float O[2][HD / 16][4];
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int m = 0; m < HD / 16; ++m)
#pragma unroll
      for (int e = 0; e < 4; ++e) O[i][m][e] = 0.f;
  __syncwarp();                        // (a warp reads its own columns only)

  // where this lane's fragments begin, in bytes: chunk 2 j + (...) of a head, j = 0..3; further chunks follow 128 bytes on
  const int mat = lane >> 3, rin = lane & 7;
  constexpr int kJ = HD / 16 < 4 ? HD / 16 : 4;
  const int c_first = min(quad * 4 / p.group, p.nkv), c_last = min(p.nkv - 1, (quad * 4 + 3) / p.group);
  const int kv_off = min(c_first, p.nkv - 1) * HD * 2;
  int k_at[kJ], v_at[kJ], q_at[2];
#pragma unroll
  for (int j = 0; j < kJ; ++j) {
    k_at[j] = ((mat & 1) * 8 + rin) * row_elems * 2 + (((2 * j) ^ ((mat >> 1) ^ (rin & kSwz))) * 16);
    v_at[j] = ((mat >> 1) * 8 + rin) * row_elems * 2 + (((2 * j) ^ ((mat & 1) ^ (rin & kSwz))) * 16);
  }
#pragma unroll
  for (int j = 0; j < 2; ++j) q_at[j] = (int)smem_u32(q_sm) + rin * HD * 2 + (((4 * j) ^ mat ^ (rin & kSwz)) * 16);
  const unsigned ring_at = smem_u32(ring);
  const int tile_bytes = kTile * row_elems * 2;

  // The raw scores of a step out of its K, left for the warps that mix them.
  auto form_scores = [&](int slot) {
    float S[KT][2][4];
#pragma unroll
    for (int kt = 0; kt < KT; ++kt)
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[kt][i][e] = 0.f;
    const unsigned base = ring_at + (unsigned)(slot * unit * 2);
    for (int c = c_first; c <= (ALIGNED ? c_first : c_last); ++c) {
      const unsigned head = base + (ALIGNED ? kv_off : c * HD * 2);
      bool mine = true;
      if constexpr (!ALIGNED) {
        const int h = 4 * quad + (lane >> 3);
        mine = h >= c * p.group && h < (c + 1) * p.group;
      }
#pragma unroll
      for (int k2 = 0; k2 < HD / 32; ++k2) {
        unsigned b[2][4], a[KT][2][4];
#pragma unroll
        for (int kt = 0; kt < KT; ++kt)
#pragma unroll
          for (int x = 0; x < 2; ++x)
            ldmatrix_x4(a[kt][x], head + kt * tile_bytes + k_at[(2 * k2 + x) % kJ] + ((2 * k2 + x) / 4) * 128);
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          ldmatrix_x4(b[i], q_at[k2 & 1] + i * 8 * HD * 2 + (k2 >> 1) * 128);
          if constexpr (!ALIGNED) {
#pragma unroll
            for (int r = 0; r < 4; ++r) b[i][r] = mine ? b[i][r] : 0u;
          }
        }
#pragma unroll
        for (int x = 0; x < 2; ++x)
#pragma unroll
          for (int kt = 0; kt < KT; ++kt)
#pragma unroll
            for (int i = 0; i < 2; ++i) mma_bf16(S[kt][i], a[kt][x], b[i][2 * x], b[i][2 * x + 1]);
      }
    }
#pragma unroll
    for (int kt = 0; kt < KT; ++kt)
#pragma unroll
      for (int i = 0; i < 2; ++i) mail[((kt * 2 + i) * NQ + quad) * 32] = make_float4(S[kt][i][0], S[kt][i][1], S[kt][i][2], S[kt][i][3]);
  };
  // This warp's share of a step's mix and weights, left for the warps that own the heads.
  auto form_weights = [&](int key0) {
    const bool full = key0 + kStep - 1 <= first_pos && toks == 4;
    constexpr int kShare = KT > 1 && kTiles > 1 ? KT : 1;          // items of a warp that are of one combination
#pragma unroll
    for (int i0 = 0; i0 < KT; i0 += kShare) {
      const int combo = (KT * quad + i0) / kTiles;
      float X[kShare][2][4];
#pragma unroll
      for (int i = 0; i < kShare; ++i)
#pragma unroll
        for (int e = 0; e < 2; ++e)
#pragma unroll
          for (int r = 0; r < 4; ++r) X[i][e][r] = 0.f;
#pragma unroll
      for (int s = 0; s < kTiles; ++s) {
        const float4 fa = mail[(combo * NQ + 2 * s) * 32], fb = mail[(combo * NQ + 2 * s + 1) * 32];
        unsigned hi[2][4], lo[2][4];
        split_tf32(fa.x, hi[0][0], lo[0][0]);
        split_tf32(fa.z, hi[0][1], lo[0][1]);
        split_tf32(fb.x, hi[0][2], lo[0][2]);
        split_tf32(fb.z, hi[0][3], lo[0][3]);
        split_tf32(fa.y, hi[1][0], lo[1][0]);
        split_tf32(fa.w, hi[1][1], lo[1][1]);
        split_tf32(fb.y, hi[1][2], lo[1][2]);
        split_tf32(fb.w, hi[1][3], lo[1][3]);
#pragma unroll
        for (int i = 0; i < kShare; ++i)
#pragma unroll
          for (int e = 0; e < 2; ++e) mma_tf32(X[i][e], hi[e], T0[i0 + i][s], T1[i0 + i][s]);
#pragma unroll
        for (int i = 0; i < kShare; ++i)
#pragma unroll
          for (int e = 0; e < 2; ++e) mma_tf32(X[i][e], lo[e], T0[i0 + i][s], T1[i0 + i][s]);
      }
      const int pair = combo & 1, key = key0 + (combo >> 1) * kTile + (lane >> 2);
#pragma unroll
      for (int i = 0; i < kShare; ++i) {
#pragma unroll
        for (int e = 0; e < 2; ++e)
#pragma unroll
          for (int r = 0; r < 4; ++r) {
            float w = weight(X[i][e][r], p.neg_scale_log2, nb[i0 + i][r & 1]);
            if (!full && (key + 8 * (r >> 1) > first_pos + 2 * pair + e || 2 * pair + e >= toks)) w = 0.f;
            X[i][e][r] = w;
          }
        const int tile = (KT * quad + i0 + i) % kTiles;
#pragma unroll
        for (int u = 0; u < 2; ++u)
          wmail[(combo * NQ + 2 * tile + u) * 32] = make_uint2(movmatrix_trans(pack_bf16(X[i][0][u], X[i][1][u])),
                                                               movmatrix_trans(pack_bf16(X[i][0][2 + u], X[i][1][2 + u])));
      }
    }
  };
  // The step's weights (this warp's heads) times its V.
  auto add_values = [&](int slot) {
    unsigned w0[KT][2], w1[KT][2];
#pragma unroll
    for (int kt = 0; kt < KT; ++kt)
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const uint2 w = wmail[((kt * 2 + i) * NQ + quad) * 32];
        w0[kt][i] = w.x, w1[kt][i] = w.y;
      }
    const unsigned base = ring_at + (unsigned)(slot * unit * 2);
    for (int c = c_first; c <= (ALIGNED ? c_first : c_last); ++c) {
      const unsigned head = base + (ALIGNED ? kv_off : c * HD * 2);
      bool mine = true;
      if constexpr (!ALIGNED) {
        const int h = 4 * quad + (lane >> 3);
        mine = h >= c * p.group && h < (c + 1) * p.group;
      }
#pragma unroll
      for (int kt = 0; kt < KT; ++kt)
#pragma unroll
        for (int m2 = 0; m2 < HD / 16; m2 += 2) {
          unsigned a[2][4];
#pragma unroll
          for (int x = 0; x < 2; ++x) ldmatrix_x4_trans(a[x], head + kt * tile_bytes + v_at[(m2 + x) % kJ] + ((m2 + x) / 4) * 128);
#pragma unroll
          for (int x = 0; x < 2; ++x)
#pragma unroll
            for (int i = 0; i < 2; ++i) mma_bf16(O[i][m2 + x], a[x], mine ? w0[kt][i] : 0u, mine ? w1[kt][i] : 0u);
        }
    }
  };
  // Two meetings of the block a step. Between the first and the second: the values of a step and the raw scores of the next
  // one, which do not wait for one another; between the second and the next first: that step's mix. So scores are read, and
  // weights written, while nobody writes scores or reads weights.
  const int steps = units / 2;
  auto seen = [&](int n) { return n < steps && (t_begin + n) * kStep <= last_pos; };      // the same for all warps of four tokens
  auto next_slot = [&](int slot) { return slot + 1 == stages ? 0 : slot + 1; };
  if (steps > 0) {
    if (stages == 4) cp_async_wait<3>(); else if (stages == 3) cp_async_wait<2>(); else cp_async_wait<1>();
    __syncthreads();
    if (seen(0)) form_scores(0);
    __syncthreads();
    request();
    if (seen(0)) form_weights(t_begin * kStep);
  }
  int slot = 1;
  for (int n = 0; n < steps; ++n) {
    if (stages == 4) cp_async_wait<2>(); else if (stages == 3) cp_async_wait<1>(); else cp_async_wait<0>();
    __syncthreads();
    const int k_slot = next_slot(slot);
    if (seen(n)) add_values(slot);
    if (seen(n + 1)) form_scores(k_slot);
    __syncthreads();
    request();
    request();
    if (seen(n + 1)) form_weights((t_begin + n + 1) * kStep);
    slot = next_slot(k_slot);
  }
  cp_async_wait<0>();

  // ---- a thread holds, of pair i, head t of the quad: numbers 16 m + lane / 4 (+ 8) of the pair's token 0 (registers 0, 2)
  // and token 1 (1, 3)
  const int t4 = lane & 3, g8 = lane >> 2;
  if (toks <= 0) return;
  if (slices > 1) {
    if (my_head >= p.nq) return;
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        if (2 * i + e >= toks) continue;
        float* o = p.part + (size_t)(p.row_base[q_start + tok0 + 4 * group4 + 2 * i + e] + slice) * p.nq * HD + (size_t)my_head * HD + g8;
#pragma unroll
        for (int m = 0; m < HD / 16; ++m) {
          o[16 * m] = O[i][m][e];
          o[16 * m + 8] = O[i][m][2 + e];
        }
      }
    return;
  }
  // the place of the warp's queries takes the gate, then the gated result, then leaves in whole rows
  auto for_rows = [&](auto&& fn) {
    for (int i = lane; i < 16 * head_chunks; i += 32) {
      const int r = i / head_chunks, ch = i % head_chunks;
      const int h = 4 * quad + ((r & 7) >> 1), tok = 2 * (r >> 3) + (r & 1);
      if (h < p.nq && tok < toks)
        fn(q_start + tok0 + 4 * group4 + tok, h * HD + ch * 8, reinterpret_cast<uint4*>(q_sm + swz<HD>(r, HD, 0, ch)));
    }
  };
  __syncwarp();
  if (p.gate) for_rows([&](int row, int col, uint4* s) { *s = *reinterpret_cast<const uint4*>(p.gate + (size_t)row * p.gate_stride + col); });
  __syncwarp();
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int m = 0; m < HD / 16; ++m)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int r = 8 * i + 2 * t4 + (e & 1), ch = 2 * m + (e >> 1);
        bf16* s = q_sm + swz<HD>(r, HD, 0, ch) + g8;
        float o = O[i][m][e];
        if (p.gate) o *= sigmoid_gate(__bfloat162float(*s));
        *s = __float2bfloat16_rn(o);
      }
  __syncwarp();
  for_rows([&](int row, int col, uint4* s) { *reinterpret_cast<uint4*>(p.out + (size_t)row * p.out_stride + col) = *s; });
}

// ---------------------------------------------------------------------------------------------
// Single tokens. NT: tiles of eight heads.
// ---------------------------------------------------------------------------------------------
constexpr int kDecodeWarps = 4;
constexpr int kRing = 6;

template <int HD, int NT>
__global__ void __launch_bounds__(kDecodeWarps * 32) sigmoid_decode_kernel(const SigParams p) {
  pdl_start();
  extern __shared__ __align__(128) unsigned char smem_raw[];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  constexpr int unit = kTile * HD, head_chunks = HD / 8;
  bf16* const q_sm = reinterpret_cast<bf16*>(smem_raw);
  bf16* const rings = q_sm + NT * 8 * HD;
  bf16* const ring = rings + (size_t)warp * kRing * unit;
  const int4 item = p.items[blockIdx.x];
  const int req = item.x, slice = item.z, slices = item.w;
  const int row = p.cu_seqlens[req];
  const int kv_len = p.kv_lens[req], pos = kv_len - 1;
  const int* bt = p.block_table + (size_t)req * p.bt_stride;
  const int row_elems = p.nkv * HD;
  const int span = (kv_len + kTile - 1) / kTile;
  const int per = (span + slices - 1) / slices;
  const int t_begin = slice * per, t_end = min(span, t_begin + per);
  // this warp's tiles: t_begin + warp, + kDecodeWarps, ...; stages in order K of every kv head, V of every kv head
  const int mine = max(0, (t_end - t_begin - warp + kDecodeWarps - 1) / kDecodeWarps);
  const int units = mine * 2 * p.nkv;
  int rq = 0, rq_tile = t_begin + warp, rq_unit = 0;        // the next stage to request
  const bf16* rq_k = nullptr;
  const bf16* rq_v = nullptr;
  auto request = [&]() {
    if (rq < units) {
      if (rq_unit == 0) {
        const int key0 = rq_tile * kTile;
        const size_t at = (size_t)bt[key0 / p.page_size] * p.page_stride + (size_t)(key0 % p.page_size) * row_elems;
        rq_k = p.k_cache + at;
        rq_v = p.v_cache + at;
      }
      const bf16* src = rq_unit < p.nkv ? rq_k + rq_unit * HD : rq_v + (rq_unit - p.nkv) * HD;
      const unsigned dst = smem_u32(ring + (size_t)(rq % kRing) * unit);
#pragma unroll
      for (int i = 0; i < kTile * head_chunks / 32; ++i) {
        const int r = (i * 32 + lane) / head_chunks, ch = (i * 32 + lane) % head_chunks;
        cp_async16(dst + swz<HD>(r, HD, 0, ch) * 2, src + (size_t)r * row_elems + ch * 8);
      }
      ++rq;
      if (++rq_unit == 2 * p.nkv) rq_unit = 0, rq_tile += kDecodeWarps;
    }
    cp_async_commit();
  };
#pragma unroll
  for (int u = 0; u < kRing - 1; ++u) request();
  for (int i = threadIdx.x; i < NT * 8 * head_chunks; i += blockDim.x) {
    const int r = i / head_chunks, ch = i - r * head_chunks;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (r < p.nq) v = *reinterpret_cast<const uint4*>(p.q + (size_t)row * p.q_stride + (size_t)r * HD + ch * 8);
    *reinterpret_cast<uint4*>(q_sm + swz<HD>(r, HD, 0, ch)) = v;
  }
  unsigned T0[NT][NT], T1[NT][NT];
#pragma unroll
  for (int s = 0; s < NT; ++s)
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      T0[s][j] = __float_as_uint(mix_at(p, s, lane & 3, j, lane >> 2));
      T1[s][j] = __float_as_uint(mix_at(p, s, (lane & 3) + 4, j, lane >> 2));
    }
  float nb[NT][2];
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int h = 8 * i + 2 * (lane & 3) + e;
      nb[i][e] = h < p.nq ? -p.bias[h] * kLog2eF : 0.f;
    }
  float O[NT][HD / 16][4];
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int m = 0; m < HD / 16; ++m)
#pragma unroll
      for (int e = 0; e < 4; ++e) O[i][m][e] = 0.f;
  __syncthreads();

  int u = 0;
  for (int tile = t_begin + warp; tile < t_end; tile += kDecodeWarps) {
    float S[NT][4];
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) S[i][e] = 0.f;
    for (int c = 0; c < p.nkv; ++c, ++u) {
      cp_async_wait<kRing - 2>();
      __syncwarp();
      request();
      scores<HD, NT>(S, ring + (size_t)(u % kRing) * unit, q_sm, c, p.group, lane);
    }
    float X[NT][4];
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
      for (int r = 0; r < 4; ++r) X[j][r] = 0.f;
#pragma unroll
    for (int s = 0; s < NT; ++s) {
      unsigned hi[4], lo[4];
      split_tf32(S[s][0], hi[0], lo[0]);
      split_tf32(S[s][2], hi[1], lo[1]);
      split_tf32(S[s][1], hi[2], lo[2]);
      split_tf32(S[s][3], hi[3], lo[3]);
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        mma_tf32(X[j], hi, T0[s][j], T1[s][j]);
        mma_tf32(X[j], lo, T0[s][j], T1[s][j]);
      }
    }
    unsigned w0[NT], w1[NT];
    const int key = tile * kTile + (lane >> 2);
#pragma unroll
    for (int j = 0; j < NT; ++j) {
#pragma unroll
      for (int r = 0; r < 4; ++r) {
        const float w = weight(X[j][r], p.neg_scale_log2, nb[j][r & 1]);
        X[j][r] = key + 8 * (r >> 1) <= pos ? w : 0.f;
      }
      w0[j] = movmatrix_trans(pack_bf16(X[j][0], X[j][1]));
      w1[j] = movmatrix_trans(pack_bf16(X[j][2], X[j][3]));
    }
    for (int c = 0; c < p.nkv; ++c, ++u) {
      cp_async_wait<kRing - 2>();
      __syncwarp();
      request();
      values<HD, NT>(O, ring + (size_t)(u % kRing) * unit, w0, w1, c, p.group, lane);
    }
  }
  cp_async_wait<0>();
  __syncthreads();                     // every warp is done with its ring: their place takes the warps' sums
  // a thread holds, of tile i, heads 8 i + 2 t and + 1 (registers 0, 2 and 1, 3): numbers 16 m + lane / 4 (+ 8)
  float* sums = reinterpret_cast<float*>(rings);        // [warps][nq * HD], rows of HD + 4 apart
  constexpr int kRowF = HD + 4;
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int h = 8 * i + 2 * (lane & 3) + (e & 1);
      if (h >= p.nq) continue;
      float* s = sums + ((size_t)warp * p.nq + h) * kRowF + (lane >> 2) + 8 * (e >> 1);
#pragma unroll
      for (int m = 0; m < HD / 16; ++m) s[16 * m] = O[i][m][e];
    }
  __syncthreads();
  for (int i = threadIdx.x; i < p.nq * HD / 2; i += blockDim.x) {
    const int h = i / (HD / 2), d = (i - h * (HD / 2)) * 2;
    float2 a = make_float2(0.f, 0.f);
#pragma unroll
    for (int w = 0; w < kDecodeWarps; ++w) {
      const float2 v = *reinterpret_cast<const float2*>(sums + ((size_t)w * p.nq + h) * kRowF + d);
      a.x += v.x, a.y += v.y;
    }
    const size_t col = (size_t)h * HD + d;
    if (slices > 1) {
      *reinterpret_cast<float2*>(p.part + (size_t)(p.row_base[row] + slice) * p.nq * HD + col) = a;
    } else {
      if (p.gate) {
        const float2 g = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p.gate + (size_t)row * p.gate_stride + col));
        a.x *= sigmoid_gate(g.x), a.y *= sigmoid_gate(g.y);
      }
      *reinterpret_cast<__nv_bfloat162*>(p.out + (size_t)row * p.out_stride + col) = __floats2bfloat162_rn(a.x, a.y);
    }
  }
}

constexpr size_t kMaxSmem = 227 * 1024;

int quads_for(int nq) { return nq <= 8 ? 2 : (nq <= 16 ? 4 : 8); }

size_t tile_smem(int nkv, int hd, int kt, int stages) {
  return (size_t)kTileWarps * 16 * hd * 2 + (size_t)kTileWarps * kt * 2 * 32 * 24 + (size_t)stages * kt * kTile * nkv * hd * 2;
}
// key tiles of a step of the tile kernel and stages of its ring for a geometry: the most that fit (0: not two stages)
int tile_stages(int nkv, int hd, int& kt) {
  for (kt = 2; kt >= 1; --kt)
    for (int stages = 4; stages >= 2; --stages)
      if (tile_smem(nkv, hd, kt, stages) <= kMaxSmem) return stages;
  return 0;
}

size_t decode_smem(int nq, int hd) {
  const int nt = quads_for(nq) / 2;
  const size_t ring = (size_t)kDecodeWarps * kRing * kTile * hd * 2, sums = (size_t)kDecodeWarps * nq * (hd + 4) * 4;
  return (size_t)nt * 8 * hd * 2 + (ring > sums ? ring : sums);
}

template <int HD, int NQ>
int launch_tiles(const SigParams& p, int items, cudaStream_t s) {
  int kt;
  const int stages = tile_stages(p.nkv, HD, kt);
  const size_t smem = tile_smem(p.nkv, HD, kt, stages);
#define OI_SIG_TILE(KT, ALIGNED)                                                                                              \
  do {                                                                                                                        \
    OI_CHECK_CUDA(cudaFuncSetAttribute(sigmoid_tile_kernel<HD, NQ, KT, ALIGNED>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kMaxSmem)); \
    oi_launch(sigmoid_tile_kernel<HD, NQ, KT, ALIGNED>, items, kTileWarps * 32, smem, s, p, stages);                          \
  } while (0)
  if (p.group % 4 == 0 && kt == 2) OI_SIG_TILE(2, true);
  else if (p.group % 4 == 0) OI_SIG_TILE(1, true);
  else if (kt == 2) OI_SIG_TILE(2, false);
  else OI_SIG_TILE(1, false);
#undef OI_SIG_TILE
  OI_CHECK_LAUNCH();
  return OI_OK;
}

template <int HD, int NT>
int launch_decode(const SigParams& p, int items, cudaStream_t s) {
  const size_t smem = decode_smem(p.nq, HD);
  OI_CHECK_CUDA(cudaFuncSetAttribute(sigmoid_decode_kernel<HD, NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kMaxSmem));
  oi_launch(sigmoid_decode_kernel<HD, NT>, items, kDecodeWarps * 32, smem, s, p);
  OI_CHECK_LAUNCH();
  return OI_OK;
}

template <int HD>
int launch_all(SigParams p, const int* tile_items, int n_tiles, const int* decode_items, int n_decode, cudaStream_t s) {
  const int quads = quads_for(p.nq);
  if (n_tiles > 0) {
    p.items = reinterpret_cast<const int4*>(tile_items);
    const int rc = quads == 2 ? launch_tiles<HD, 2>(p, n_tiles, s) : (quads == 4 ? launch_tiles<HD, 4>(p, n_tiles, s) : launch_tiles<HD, 8>(p, n_tiles, s));
    if (rc != OI_OK) return rc;
  }
  if (n_decode > 0) {
    p.items = reinterpret_cast<const int4*>(decode_items);
    const int rc = quads == 2 ? launch_decode<HD, 1>(p, n_decode, s) : (quads == 4 ? launch_decode<HD, 2>(p, n_decode, s) : launch_decode<HD, 4>(p, n_decode, s));
    if (rc != OI_OK) return rc;
  }
  return OI_OK;
}

bool aligned16(const void* p) { return ((uintptr_t)p & 15) == 0; }

}  // namespace

// Tokens a prompt tile holds for a geometry (0: the tensor-core kernels do not take it).
OI_API int oi_sigmoid_attention_tile_tokens(int nq, int nkv, int hd) {
  if ((hd != 32 && hd != 64 && hd != 128) || nq <= 0 || nkv <= 0 || nq % nkv || nq > 32) return 0;
  int kt;
  return tile_stages(nkv, hd, kt) > 0 && decode_smem(nq, hd) <= kMaxSmem ? 4 * (kTileWarps / quads_for(nq)) : 0;
}

// bfloat16. Items: int32 [n, 4] (request, first token of the tile, slice, slices); a tile item covers
// oi_sigmoid_attention_tile_tokens tokens of its request, a decode item the request's one token. Rows of more than one slice
// leave float32 results in part[row_base[row] + slice]; slice_sum_gate_kernel then has to add them up (the caller's next call).
OI_API int oi_sigmoid_attention_mma(const void* q, long long q_stride, void* out, long long out_stride, const void* gate,
                                    long long gate_stride, const void* k_cache, const void* v_cache, long long page_stride,
                                    int page_size, const int* block_table, int bt_stride, const int* cu_seqlens, const int* kv_lens,
                                    const int* tile_items, int n_tiles, const int* decode_items, int n_decode, const int* row_base,
                                    float* part, int nq, int nkv, int hd, float scale, const float* mix, const float* bias, void* stream) {
  OI_REQUIRE(oi_sigmoid_attention_tile_tokens(nq, nkv, hd) > 0, "sigmoid_attention_mma: nq=%d nkv=%d hd=%d is not taken", nq, nkv, hd);
  OI_REQUIRE(page_size > 0 && page_size % kTile == 0, "sigmoid_attention_mma: pages of %d keys are no multiple of %d", page_size, kTile);
  OI_REQUIRE(q_stride % 8 == 0 && out_stride % 8 == 0 && gate_stride % 8 == 0 && page_stride % 8 == 0 && aligned16(q) && aligned16(out) &&
             aligned16(gate) && aligned16(k_cache) && aligned16(v_cache), "sigmoid_attention_mma: rows and pages must be readable 16 bytes at a time");
  OI_REQUIRE(n_tiles >= 0 && n_decode >= 0 && row_base && mix && bias, "sigmoid_attention_mma: a buffer is missing");
  SigParams p = {};
  p.q = (const bf16*)q, p.q_stride = q_stride, p.out = (bf16*)out, p.out_stride = out_stride;
  p.gate = (const bf16*)gate, p.gate_stride = gate_stride;
  p.k_cache = (const bf16*)k_cache, p.v_cache = (const bf16*)v_cache, p.page_stride = page_stride, p.page_size = page_size;
  p.block_table = block_table, p.bt_stride = bt_stride, p.cu_seqlens = cu_seqlens, p.kv_lens = kv_lens;
  p.row_base = row_base, p.part = part, p.nq = nq, p.nkv = nkv, p.group = nq / nkv;
  p.neg_scale_log2 = -scale * kLog2eF, p.mix = mix, p.bias = bias;
  cudaStream_t s = (cudaStream_t)stream;
  if (hd == 32) return launch_all<32>(p, tile_items, n_tiles, decode_items, n_decode, s);
  if (hd == 64) return launch_all<64>(p, tile_items, n_tiles, decode_items, n_decode, s);
  return launch_all<128>(p, tile_items, n_tiles, decode_items, n_decode, s);
}
