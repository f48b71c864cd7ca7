// Causal grouped-query attention whose heads' softmax weights are mixed before they meet the values:
//
//   s_g(i, j) = cap * tanh((q_i,g . k_j,kv(g)) * scale / cap)                      (cap 0: no cap)
//   p_g(i, j) = exp(s_g(i, j)) / (exp(sink_g) + sum_j' exp(s_g(i, j')))            (the sink has no key and no value)
//   w_h(i, j) = sum_g talk[h, g] p_g(i, j),      out_i,h = sum_j w_h(i, j) v_j,kv(h)
//
// with kv(h) = h / (H / G).  A token's cache row holds the keys of all key/value heads, then their values: [G * n | G * dv].
//
// Mixing needs every head's normalised weight of the same query and key, so a kernel here owns all heads of its queries.
//
// qv_talking_attention_generic   one CTA per token, float32 throughout: a pass over the keys for every head's maximum and sum, then
//                                a pass that forms the weights of 32 keys, mixes them and adds the values.  Keys in blocks of 32
//                                aligned to absolute positions: the order of every sum depends on the token's position alone.
// qv_talking_attention_mma       bfloat16 on the tensor cores (mma.sync m16n8k16, float32 sums; the mixed weights enter the product
//                                with the values as three bfloat16 terms that together hold their 24 bits):
//   portions       a cluster of CTAs owns 16 consecutive tokens and all heads (a warp a head); its CTAs share out the blocks of 32
//                  keys.  Pass 1: every head's maximum and sum, joined over the cluster through distributed shared memory.  Pass 2:
//                  the normalised weights of a block go to shared memory and are mixed in place (up to eight heads: a thread mixes all
//                  heads of one (query, key); more: products of the matrix with the weights of eight pairs on the tensor cores, the
//                  weights as three bfloat16 terms), and a warp multiplies its head's mixed weights with the values; at the end the cluster's partial outputs are added in rank order.
//   single tokens  a CTA owns one token and a slice of its keys, with the heads as the tile's rows.  Since mixing is linear,
//                      out_h = sum_g talk[h, g] / L_g * (sum_j exp(s_g(j)) v_j,kv(h)),
//                  a slice multiplies every head's unnormalised weights with the values of ALL key/value heads (read once), and
//                  talking_merge_kernel joins the slices, divides and mixes.
#include "common.cuh"
#include <cooperative_groups.h>
#include <type_traits>
namespace cg = cooperative_groups;

#define TA_KEYS 32
#define TA_MAX_H 16                // heads of the tensor-core kernels
#define TA_PS 36                   // row and head strides of the weights in shared memory (floats)
#define TA_HS (16 * TA_PS + 4)
#define TA_LOG2E 1.4426950408889634f

// ---------------------------------------------------------------- float32 and other sizes
template <typename T>
__global__ void __launch_bounds__(256) talking_attention_generic_kernel(
    T* __restrict__ out, int ld_out, const T* __restrict__ q, int ld_q, const T* __restrict__ cache, const int* __restrict__ tok_pos,
    const int* __restrict__ tok_seg, const int* __restrict__ block_table, int max_blocks, int H, int G, int n, int dv, int page,
    float scale, float cap, const float* __restrict__ sink, const float* __restrict__ talk) {
  extern __shared__ float tg_smem[];
  float* qs = tg_smem;                     // [H][n]
  float* os = qs + (size_t)H * n;          // [H][dv]
  float* ps = os + (size_t)H * dv;         // [H][32] a block's weights
  float* ws = ps + (size_t)H * 32;         // [H][32] ... mixed
  float* ms = ws + (size_t)H * 32;         // [H] maximum
  float* il = ms + H;                      // [H] 1 / sum
  float* ts = il + H;                      // [H][H]
  pdl_wait();
  pdl_launch_dependents();
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int i = threadIdx.x; i < H * n; i += 256) qs[i] = to_f(q[(size_t)t * ld_q + i]);
  for (int i = threadIdx.x; i < H * dv; i += 256) os[i] = 0.f;
  for (int i = threadIdx.x; i < H * H; i += 256) ts[i] = talk[i];
  __syncthreads();
  const int pos = tok_pos[t];
  const int* bt = block_table + (size_t)tok_seg[t] * max_blocks;
  const size_t width = (size_t)G * (n + dv);
  const int gs = H / G;
  auto score = [&](int h, size_t base) {
    const T* kp = cache + base + (size_t)(h / gs) * n;
    const float* qh = qs + (size_t)h * n;
    float d = 0.f;
    for (int i = 0; i < n; ++i) d = fmaf(qh[i], to_f(kp[i]), d);
    d *= scale;
    return cap > 0.f ? cap * tanhf(d / cap) : d;
  };
  for (int h = warp; h < H; h += 8) {
    float m = sink[h], l = 1.f;                                // the sink's own share
    for (int kb = 0; kb <= pos; kb += 32) {
      const int tk = kb + lane;
      float s = -INFINITY;
      if (tk <= pos) s = score(h, ((size_t)bt[tk / page] * page + (size_t)(tk % page)) * width);
      const float mn = fmaxf(m, warp_max(s));
      l = l * expf(m - mn) + warp_sum(tk <= pos ? expf(s - mn) : 0.f);
      m = mn;
    }
    if (lane == 0) { ms[h] = m; il[h] = 1.0f / l; }
  }
  __syncthreads();
  for (int kb = 0; kb <= pos; kb += 32) {
    const int tk = kb + lane;
    size_t base = 0;
    if (tk <= pos) base = ((size_t)bt[tk / page] * page + (size_t)(tk % page)) * width;
    for (int h = warp; h < H; h += 8) ps[h * 32 + lane] = tk <= pos ? expf(score(h, base) - ms[h]) * il[h] : 0.f;
    __syncthreads();
    for (int i = threadIdx.x; i < H * 32; i += 256) {
      const float* tr = ts + (size_t)(i >> 5) * H;
      float w = 0.f;
      for (int g = 0; g < H; ++g) w = fmaf(tr[g], ps[g * 32 + (i & 31)], w);
      ws[i] = w;
    }
    __syncthreads();
    const int nkeys = pos - kb + 1 < 32 ? pos - kb + 1 : 32;
    for (int i = threadIdx.x; i < H * dv; i += 256) {
      const int h = i / dv, c = i - h * dv;
      float o = os[i];
      for (int j = 0; j < nkeys; ++j) {
        const int kj = kb + j;
        const T* vp = cache + ((size_t)bt[kj / page] * page + (size_t)(kj % page)) * width + (size_t)G * n + (size_t)(h / gs) * dv;
        o = fmaf(ws[h * 32 + j], to_f(vp[c]), o);
      }
      os[i] = o;
    }
    __syncthreads();
  }
  for (int i = threadIdx.x; i < H * dv; i += 256) out[(size_t)t * ld_out + i] = from_f<T>(os[i]);
}

extern "C" int qv_talking_attention_generic(void* out, int ld_out, const void* q, int ld_q, const void* cache, const int* tok_pos,
                                            const int* tok_seg, const int* block_table, int max_blocks, int T, int H, int G, int n,
                                            int dv, int page, float scale, float cap, const float* sink, const float* talk, int dt,
                                            void* stream) {
  if (T <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || n <= 0 || dv <= 0) return QV_ERR_UNSUPPORTED;
  const size_t smem = ((size_t)H * (n + dv) + (size_t)H * 64 + 2 * H + (size_t)H * H) * sizeof(float);
  if (smem > 200 * 1024) return QV_ERR_TOO_LARGE;
  cudaStream_t st = (cudaStream_t)stream;
  QV_DISPATCH_DT(dt, TT, {
    if (smem > 48 * 1024)
      cudaFuncSetAttribute(talking_attention_generic_kernel<TT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    return qv_launch(talking_attention_generic_kernel<TT>, dim3(T), dim3(256), smem, st, (TT*)out, ld_out, (const TT*)q, ld_q,
                     (const TT*)cache, tok_pos, tok_seg, block_table, max_blocks, H, G, n, dv, page, scale, cap, sink, talk);
  });
  return QV_ERR_UNSUPPORTED;
}

// ---------------------------------------------------------------- tensor cores (bfloat16)
struct TalkArgs {
  bf16* out; int ld_out;
  const bf16* q; int ld_q;
  const bf16* cache;
  const int* seg_q_start; const int* seg_pos0; const int* block_table; int max_blocks;
  int H, G, n, dv, page;
  float pre, post;                                 // score in base 2 = post * f(pre * dot): capped f = tanh, else the identity
  int capped;
  const float* sink;
  const float* talk; int talk_terms;               // [H, H]; terms 1: every entry is a bfloat16 number, else 3
  float* partial; int slices; int slice_keys;      // single tokens: [S, slices, H, 2 + G * dv] (m, l, o)
};
// for few heads the mixing matrix rides in the kernel's parameters: its entries are then operands of the multiply-adds (no loads)
template <int HP> struct TalkMatrix { float t[HP * HP]; };

__device__ __forceinline__ void ta_ldsm4(uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3, const void* p) {
  const unsigned a = (unsigned)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(a));
}
__device__ __forceinline__ void ta_ldsm4_trans(uint32_t& r0, uint32_t& r1, uint32_t& r2, uint32_t& r3, const void* p) {
  const unsigned a = (unsigned)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(a));
}
__device__ __forceinline__ void ta_ldsm2_trans(uint32_t& r0, uint32_t& r1, const void* p) {
  const unsigned a = (unsigned)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(a));
}
__device__ __forceinline__ void ta_mma(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// 16 bytes, or 16 zero bytes where `valid` is false (src must still be an address that may be formed)
__device__ __forceinline__ void ta_cp16(void* dst, const void* src, bool valid) {
  const int bytes = valid ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void ta_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void ta_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ uint32_t ta_pack(float lo, float hi) {
  __nv_bfloat162 h = __floats2bfloat162_rn(lo, hi);
  return *(uint32_t*)&h;
}
// the three bfloat16 terms of two float32 weights: rounded, what is left rounded, and again
__device__ __forceinline__ void ta_split3(float x, float y, uint32_t& t0, uint32_t& t1, uint32_t& t2) {
  t0 = ta_pack(x, y);
  const float xr = x - __uint_as_float(t0 << 16), yr = y - __uint_as_float(t0 & 0xffff0000u);
  t1 = ta_pack(xr, yr);
  t2 = ta_pack(xr - __uint_as_float(t1 << 16), yr - __uint_as_float(t1 & 0xffff0000u));
}
// 2^x and 1 / x as the special-function unit gives them (two float32 ulp, one ulp; results below the smallest normal number are zero)
__device__ __forceinline__ float ta_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float ta_rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// post * tanh(x) through one exponential: tanh(x) = 1 - 2 / (1 + e^(2x)); the error is an ulp of the cap
__device__ __forceinline__ float ta_score(float dot, const TalkArgs& a) {
  const float x = dot * a.pre;
  if (!a.capped) return x;
  return fmaf(-2.0f * a.post, ta_rcp(1.0f + ta_exp2(x)), a.post);    // pre carries 2 log2 e here
}

// ---- portions: 16 tokens, all heads
// shared memory: sQ [H][16][KS], two buffers of [G][32][max(KS, VS)], sP [H][TA_HS] float, stats [2][H][16] float; the
// cluster's partial outputs [H][16][dv + 4] float lie over the front at the end
static inline size_t ta_buf_bytes(int G, int NP, int DP) { return (size_t)G * TA_KEYS * ((NP > DP ? NP : DP) + 8) * sizeof(bf16); }
static inline size_t ta_tile_smem(int H, int G, int NP, int DP, int dv) {
  const size_t front = (size_t)H * 16 * (NP + 8) * sizeof(bf16) + 2 * ta_buf_bytes(G, NP, DP);
  const size_t body = front + (size_t)H * TA_HS * sizeof(float);
  const size_t outs = (size_t)H * 16 * (dv + 4) * sizeof(float);
  return (body > outs ? body : outs) + (size_t)2 * H * 16 * sizeof(float);
}

template <int NP, int DP, int HP>
__global__ void __launch_bounds__(HP * 32) talking_tile_kernel(TalkArgs a, const __grid_constant__ TalkMatrix<HP < 16 ? HP : 1> mix, int cs, size_t stat_off) {
  extern __shared__ __align__(16) unsigned char ta_smem[];
  constexpr int KS = NP + 8, VS = DP + 8;                 // row strides: an odd number of 16-byte units
  constexpr int KC = NP / 8, VC = DP / 8, BS = (NP > DP ? KS : VS);
  constexpr int PS = TA_PS, HS = TA_HS;
  const int H = a.H, G = a.G, n = a.n, dv = a.dv, page = a.page, gs = H / G, NT = 32 * H;
  bf16* sQ = (bf16*)ta_smem;
  bf16* buf0 = sQ + H * 16 * KS;
  bf16* buf1 = buf0 + G * TA_KEYS * BS;
  float* sP = (float*)(buf1 + G * TA_KEYS * BS);
  float* stat = (float*)(ta_smem + stat_off);
  pdl_wait();
  const int tid = threadIdx.x, lane = tid & 31, h = tid >> 5, g8 = lane >> 2, tg = lane & 3, kvh = h / gs;
  const int s = blockIdx.z, rank = blockIdx.x % cs;
  const int q0 = a.seg_q_start[s], len = a.seg_q_start[s + 1] - q0, pos0 = a.seg_pos0[s];
  const int rb = (int)(gridDim.x / cs) - 1 - (int)(blockIdx.x / cs);       // the longest tiles first
  if (rb * 16 >= len) return;                             // the whole cluster leaves
  const int* bt = a.block_table + (size_t)s * a.max_blocks;
  const int i0 = pos0 + rb * 16, rows_valid = min(16, len - rb * 16), k_hi = i0 + rows_valid;
  const size_t width = (size_t)G * (n + dv);

  for (int idx = tid; idx < H * 16 * KC; idx += NT) {
    const int hr = idx / KC, c = idx - hr * KC, hh = hr >> 4, r = hr & 15;
    const bool valid = r < rows_valid && c * 8 < n;
    const bf16* src = valid ? a.q + (size_t)(q0 + rb * 16 + r) * a.ld_q + (size_t)hh * n + c * 8 : a.q;
    ta_cp16(sQ + hr * KS + c * 8, src, valid);
  }
  // a block of keys (or values) of all key/value heads: a warp copies whole rows; lane r works out where key j0 + r lies
  auto load = [&](bf16* dst, int j0, auto values) {
    constexpr bool V = decltype(values)::value;
    constexpr int C = V ? VC : KC, stride = V ? VS : KS;
    const int jr = j0 + lane, size = V ? dv : n;
    unsigned long long row_at = 0;
    if (jr < k_hi) row_at = ((unsigned long long)bt[jr / page] * page + (unsigned long long)(jr % page)) * width + (V ? G * n : 0);
    for (int r = h; r < TA_KEYS; r += H) {
      const bf16* row = a.cache + __shfl_sync(0xffffffffu, row_at, r);
      const bool in = j0 + r < k_hi;
      for (int gc = lane; gc < G * C; gc += 32) {
        const int g = gc / C, c = gc % C;
        const bool valid = in && c * 8 < size;
        ta_cp16(dst + (g * TA_KEYS + r) * stride + c * 8, valid ? row + g * size + c * 8 : a.cache, valid);
      }
    }
    ta_commit();
  };
  constexpr std::false_type KEYS{};
  constexpr std::true_type VALUES{};
  const int pos_lo = min(i0 + g8, k_hi - 1), pos_hi = min(i0 + g8 + 8, k_hi - 1);
  const int mat = lane >> 3, r8 = lane & 7;
  // this head's scores of a block (base 2, capped, keys behind a row's position -inf)
  auto scores = [&](const bf16* kbuf, int j0, float (&sc)[4][4]) {
    const bf16* tK = kbuf + kvh * TA_KEYS * KS;
    const bf16* tQ = sQ + h * 16 * KS;
#pragma unroll
    for (int i = 0; i < 4; ++i) sc[i][0] = sc[i][1] = sc[i][2] = sc[i][3] = 0.f;
#pragma unroll
    for (int kk = 0; kk < NP / 16; ++kk) {
      uint32_t qf[4];
      ta_ldsm4(qf[0], qf[1], qf[2], qf[3], tQ + ((mat & 1) * 8 + r8) * KS + kk * 16 + (mat >> 1) * 8);
#pragma unroll
      for (int nb = 0; nb < 2; ++nb) {
        uint32_t b0, b1, b2, b3;
        ta_ldsm4(b0, b1, b2, b3, tK + (nb * 16 + (mat >> 1) * 8 + r8) * KS + kk * 16 + (mat & 1) * 8);
        ta_mma(sc[2 * nb], qf, b0, b1);
        ta_mma(sc[2 * nb + 1], qf, b2, b3);
      }
    }
    const bool edge = j0 + TA_KEYS - 1 > i0;              // some row does not see all of the block
#pragma unroll
    for (int nt = 0; nt < 4; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        float v = ta_score(sc[nt][e], a);
        if (edge && j0 + nt * 8 + 2 * tg + (e & 1) > (e >= 2 ? pos_hi : pos_lo)) v = -INFINITY;
        sc[nt][e] = v;
      }
  };

  const int nkb = (k_hi + TA_KEYS - 1) / TA_KEYS;
  const float snk = a.sink[h] * TA_LOG2E;
  float m_lo = snk, m_hi = snk, l_lo = 0.f, l_hi = 0.f;   // finite from the start: a row may see nothing of a block
  // pass 1: maximum and sum (the sink's share is added once, below)
  if (rank < nkb) load(buf0, rank * TA_KEYS, KEYS);
  for (int kb = rank, it = 0; kb < nkb; kb += cs, ++it) {
    if (kb + cs < nkb) {
      load((it & 1) ? buf0 : buf1, (kb + cs) * TA_KEYS, KEYS);
      ta_wait<1>();
    } else {
      ta_wait<0>();
    }
    __syncthreads();
    float sc[4][4];
    scores((it & 1) ? buf1 : buf0, kb * TA_KEYS, sc);
    float mx_lo = m_lo, mx_hi = m_hi;
#pragma unroll
    for (int nt = 0; nt < 4; ++nt) {
      mx_lo = fmaxf(mx_lo, fmaxf(sc[nt][0], sc[nt][1]));
      mx_hi = fmaxf(mx_hi, fmaxf(sc[nt][2], sc[nt][3]));
    }
    mx_lo = fmaxf(mx_lo, __shfl_xor_sync(0xffffffffu, mx_lo, 1));
    mx_lo = fmaxf(mx_lo, __shfl_xor_sync(0xffffffffu, mx_lo, 2));
    mx_hi = fmaxf(mx_hi, __shfl_xor_sync(0xffffffffu, mx_hi, 1));
    mx_hi = fmaxf(mx_hi, __shfl_xor_sync(0xffffffffu, mx_hi, 2));
    float s_lo = 0.f, s_hi = 0.f;
#pragma unroll
    for (int nt = 0; nt < 4; ++nt) {
      s_lo += ta_exp2(sc[nt][0] - mx_lo) + ta_exp2(sc[nt][1] - mx_lo);
      s_hi += ta_exp2(sc[nt][2] - mx_hi) + ta_exp2(sc[nt][3] - mx_hi);
    }
    l_lo = l_lo * ta_exp2(m_lo - mx_lo) + s_lo;
    l_hi = l_hi * ta_exp2(m_hi - mx_hi) + s_hi;
    m_lo = mx_lo; m_hi = mx_hi;
    __syncthreads();
  }
  if (rank < nkb) load(buf0, rank * TA_KEYS, KEYS);      // pass 2's first keys; flies while the sums are joined
  l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 1); l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 2);
  l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 1); l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 2);
  if (cs > 1) {
    cg::cluster_group cl = cg::this_cluster();
    if (tg == 0) {
      stat[h * 16 + g8] = m_lo; stat[h * 16 + g8 + 8] = m_hi;
      stat[(H + h) * 16 + g8] = l_lo; stat[(H + h) * 16 + g8 + 8] = l_hi;
    }
    cl.sync();
    float M_lo = snk, M_hi = snk;
    for (int r = 0; r < cs; ++r) {
      const float* o = cl.map_shared_rank(stat, r);
      M_lo = fmaxf(M_lo, o[h * 16 + g8]); M_hi = fmaxf(M_hi, o[h * 16 + g8 + 8]);
    }
    float L_lo = 0.f, L_hi = 0.f;
    for (int r = 0; r < cs; ++r) {
      const float* o = cl.map_shared_rank(stat, r);
      L_lo += o[(H + h) * 16 + g8] * ta_exp2(o[h * 16 + g8] - M_lo);
      L_hi += o[(H + h) * 16 + g8 + 8] * ta_exp2(o[h * 16 + g8 + 8] - M_hi);
    }
    m_lo = M_lo; m_hi = M_hi; l_lo = L_lo; l_hi = L_hi;
  }
  const float inv_lo = 1.0f / (l_lo + ta_exp2(snk - m_lo)), inv_hi = 1.0f / (l_hi + ta_exp2(snk - m_hi));

  // pass 2
  // the mixing matrix as a product's first operand: its bfloat16 term `term` (0: rounded, 1: what is left rounded, 2: and again)
  auto talk_operand = [&](int term, uint32_t (&tf)[4]) {
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      const int row = g8 + (x & 1) * 8, col = 2 * tg + (x >> 1) * 8;
      const float t0 = row < H && col < H ? a.talk[row * H + col] : 0.f, t1 = row < H && col + 1 < H ? a.talk[row * H + col + 1] : 0.f;
      uint32_t y[3];
      ta_split3(t0, t1, y[0], y[1], y[2]);
      tf[x] = term == 0 ? y[0] : term == 1 ? y[1] : y[2];
    }
  };
  uint32_t tf[4];
  if constexpr (HP == 16) talk_operand(0, tf);
  float o[DP / 8][4];
#pragma unroll
  for (int i = 0; i < DP / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  for (int kb = rank; kb < nkb; kb += cs) {
    const int j0 = kb * TA_KEYS;
    ta_wait<0>();
    __syncthreads();                                      // the keys are there; values and weights of the last block are used up
    load(buf1, j0, VALUES);
    {
      float sc[4][4];
      scores(buf0, j0, sc);
      float* pw = sP + h * HS;
#pragma unroll
      for (int nt = 0; nt < 4; ++nt) {
        *(float2*)(pw + g8 * PS + nt * 8 + 2 * tg) = make_float2(ta_exp2(sc[nt][0] - m_lo) * inv_lo, ta_exp2(sc[nt][1] - m_lo) * inv_lo);
        *(float2*)(pw + (g8 + 8) * PS + nt * 8 + 2 * tg) = make_float2(ta_exp2(sc[nt][2] - m_hi) * inv_hi, ta_exp2(sc[nt][3] - m_hi) * inv_hi);
      }
    }
    __syncthreads();                                      // all heads' weights are there; the keys are used up
    if (kb + cs < nkb) load(buf0, (kb + cs) * TA_KEYS, KEYS);
    else ta_commit();                                     // an empty group, so that the counts below hold
    if constexpr (HP == 16) {
      // eight (query, key) pairs of one query a product: talk [16 x 16] times the heads' weights of the pairs (as three bfloat16
      // terms), in place: the tile of pairs belongs to this warp
      for (int tile = h; tile < 16 * TA_KEYS / 8; tile += H) {
        float* pp = sP + (tile >> 2) * PS + (tile & 3) * 8;
        uint32_t b[3][2];
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          const int g = 2 * tg + 8 * x;
          const float w0 = g < H ? pp[g * HS + g8] : 0.f, w1 = g + 1 < H ? pp[(g + 1) * HS + g8] : 0.f;
          ta_split3(w0, w1, b[0][x], b[1][x], b[2][x]);
        }
        float c[4] = {0.f, 0.f, 0.f, 0.f};
        if (a.talk_terms > 1) {                           // a matrix that bfloat16 does not hold exactly
          uint32_t t1[4], t2[4];
          talk_operand(1, t1);
          talk_operand(2, t2);
          ta_mma(c, t2, b[0][0], b[0][1]);
          ta_mma(c, t1, b[1][0], b[1][1]);
          ta_mma(c, t1, b[0][0], b[0][1]);
        }
#pragma unroll
        for (int term = 2; term >= 0; --term) ta_mma(c, tf, b[term][0], b[term][1]);
        __syncwarp();
        if (g8 < H) *(float2*)(pp + g8 * HS + 2 * tg) = make_float2(c[0], c[1]);
        if (g8 + 8 < H) *(float2*)(pp + (g8 + 8) * HS + 2 * tg) = make_float2(c[2], c[3]);
      }
    } else
    for (int pr = tid; pr < 16 * TA_KEYS; pr += NT) {     // one (query, key) a thread: all heads mixed in place
      float* pp = sP + (pr >> 5) * PS + (pr & 31);
      float p[HP];
#pragma unroll
      for (int g = 0; g < HP; ++g) p[g] = g < H ? pp[g * HS] : 0.f;
#pragma unroll
      for (int hh = 0; hh < HP; ++hh) {
        float w = 0.f;
#pragma unroll
        for (int g = 0; g < HP; ++g) w = fmaf(mix.t[HP < 16 ? hh * HP + g : 0], p[g], w);
        if (hh < H) pp[hh * HS] = w;
      }
    }
    ta_wait<1>();
    __syncthreads();                                      // the values and the mixed weights are there
    const bf16* tV = buf1 + kvh * TA_KEYS * VS;
    const float* pw = sP + h * HS;
#pragma unroll
    for (int kk = 0; kk < 2; ++kk) {
      uint32_t t[3][4];
#pragma unroll
      for (int q4 = 0; q4 < 4; ++q4) {                    // the operand's pieces: rows g8, g8 + 8 at keys 2 tg, then at keys 8 + 2 tg
        const float2 w = *(const float2*)(pw + (g8 + (q4 & 1) * 8) * PS + kk * 16 + (q4 >> 1) * 8 + 2 * tg);
        ta_split3(w.x, w.y, t[0][q4], t[1][q4], t[2][q4]);
      }
#pragma unroll
      for (int np = 0; np < DP / 16; np += 2) {           // four accumulators in turn
        uint32_t b[8];
        ta_ldsm4_trans(b[0], b[1], b[2], b[3], tV + (kk * 16 + (mat & 1) * 8 + r8) * VS + (np * 2 + (mat >> 1)) * 8);
        ta_ldsm4_trans(b[4], b[5], b[6], b[7], tV + (kk * 16 + (mat & 1) * 8 + r8) * VS + (np * 2 + 2 + (mat >> 1)) * 8);
#pragma unroll
        for (int term = 2; term >= 0; --term) {           // the small terms first
          ta_mma(o[2 * np], t[term], b[0], b[1]);
          ta_mma(o[2 * np + 1], t[term], b[2], b[3]);
          ta_mma(o[2 * np + 2], t[term], b[4], b[5]);
          ta_mma(o[2 * np + 3], t[term], b[6], b[7]);
        }
      }
    }
  }
  pdl_launch_dependents();
  const size_t t0 = (size_t)(q0 + rb * 16);
  if (cs == 1) {
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int r = g8 + half * 8;
      if (r >= rows_valid) continue;
      bf16* orow = a.out + (t0 + r) * a.ld_out + (size_t)h * dv;
#pragma unroll
      for (int i = 0; i < DP / 8; ++i) {
        const int col = i * 8 + 2 * tg;
        if (col < dv) *(uint32_t*)(orow + col) = ta_pack(o[i][2 * half], o[i][2 * half + 1]);
      }
    }
    return;
  }
  // the cluster's partial outputs: each CTA leaves its own in shared memory, then finishes every cs-th head
  cg::cluster_group cl = cg::this_cluster();
  ta_wait<0>();
  __syncthreads();
  const int OS = dv + 4;
  float* so = (float*)ta_smem;
#pragma unroll
  for (int i = 0; i < DP / 8; ++i) {
    const int col = i * 8 + 2 * tg;
    if (col < dv) {
      *(float2*)(so + (h * 16 + g8) * OS + col) = make_float2(o[i][0], o[i][1]);
      *(float2*)(so + (h * 16 + g8 + 8) * OS + col) = make_float2(o[i][2], o[i][3]);
    }
  }
  cl.sync();
  const int half_dv = dv >> 1;
  for (int hh = rank; hh < H; hh += cs) {
    for (int idx = tid; idx < rows_valid * half_dv; idx += NT) {
      const int r = idx / half_dv, col = (idx - r * half_dv) * 2;
      float2 acc = make_float2(0.f, 0.f);
      for (int k = 0; k < cs; ++k) {
        const float2 v = *(const float2*)(cl.map_shared_rank(so, k) + (hh * 16 + r) * OS + col);
        acc.x += v.x; acc.y += v.y;
      }
      *(uint32_t*)(a.out + (t0 + r) * a.ld_out + (size_t)hh * dv + col) = ta_pack(acc.x, acc.y);
    }
  }
  cl.sync();                                              // nobody leaves while its shared memory is read
}

// ---- single tokens: one token, a slice of its keys, the heads as rows
// shared memory: sQ [16][QS], `stages` x ([KB][KR] keys, [KB][VR] values), sS [16][KB + 4] float, corr [16] float
struct TalkSliceLayout { int QS, KR, VR; };
static inline TalkSliceLayout ta_slice_layout(int G, int n, int dv) {
  TalkSliceLayout L;
  L.QS = (n + 15) / 16 * 16 + 8;
  L.KR = G * n + ((G * n / 8) % 2 ? 16 : 8);              // an odd number of 16-byte units, and room behind the last head's keys
  L.VR = G * dv + ((G * dv / 8) % 2 ? 16 : 8);
  return L;
}
static inline size_t ta_slice_smem(const TalkSliceLayout& L, int KB, int stages) {
  return (size_t)16 * L.QS * sizeof(bf16) + (size_t)stages * KB * (L.KR + L.VR) * sizeof(bf16) + (size_t)16 * (KB + 4) * sizeof(float) + 16 * sizeof(float);
}

template <int KB, int CT>                                 // keys a block; tiles of 8 value columns a warp
__global__ void __launch_bounds__(256) talking_slice_kernel(TalkArgs a, TalkSliceLayout L, int stages) {
  extern __shared__ __align__(16) unsigned char ta_smem[];
  constexpr int SS = KB + 4;
  const int H = a.H, G = a.G, n = a.n, dv = a.dv, page = a.page, gs = H / G;
  bf16* sQ = (bf16*)ta_smem;
  bf16* ring = sQ + 16 * L.QS;
  const int stage_elems = KB * (L.KR + L.VR);
  float* sS = (float*)(ring + stages * stage_elems);
  float* corr = sS + 16 * SS;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g8 = lane >> 2, tg = lane & 3, mat = lane >> 3, r8 = lane & 7;
  // what a product may read beyond the rows and columns that exist must be finite: the queries' other rows and the rows' padding
  for (int i = tid; i < 16 * L.QS / 8; i += 256) ((uint4*)sQ)[i] = make_uint4(0u, 0u, 0u, 0u);
  const int kp = (L.KR - G * n) / 8, vp_ = (L.VR - G * dv) / 8;
  for (int i = tid; i < stages * KB * (kp + vp_); i += 256) {
    const int row = i / (kp + vp_), c = i % (kp + vp_);
    bf16* base = ring + (row / KB) * stage_elems;
    bf16* dst = c < kp ? base + (row % KB) * L.KR + G * n + c * 8 : base + KB * L.KR + (row % KB) * L.VR + G * dv + (c - kp) * 8;
    *(uint4*)dst = make_uint4(0u, 0u, 0u, 0u);
  }
  for (int i = tid; i < 16 * SS + 16; i += 256) sS[i] = 0.f;
  __syncthreads();
  pdl_wait();
  pdl_launch_dependents();
  const int s = blockIdx.y;
  const int q0 = a.seg_q_start[s], pos = a.seg_pos0[s];
  const int k_lo = blockIdx.x * a.slice_keys, k_hi = min(k_lo + a.slice_keys, pos + 1);
  if (k_lo >= k_hi) return;                               // a slice past the token: the merge does not read it
  const int* bt = a.block_table + (size_t)s * a.max_blocks;
  const int nk8 = n / 8, kc = G * nk8, vc = G * (dv / 8), per = kc + vc;
  const size_t width = (size_t)per * 8;
  for (int idx = tid; idx < H * nk8; idx += 256) {
    const int h = idx / nk8, c = idx - h * nk8;
    ta_cp16(sQ + h * L.QS + c * 8, a.q + (size_t)q0 * a.ld_q + (size_t)h * n + c * 8, true);
  }
  auto load = [&](int st, int j0) {                       // whole cache rows: keys, then values
    bf16* dK = ring + st * stage_elems;
    bf16* dV = dK + KB * L.KR;
    const int jr = j0 + (lane & (KB - 1));
    unsigned long long row_at = 0;
    if (jr < k_hi) row_at = ((unsigned long long)bt[jr / page] * page + (unsigned long long)(jr % page)) * width;
    for (int r = warp; r < KB; r += 8) {
      const bf16* row = a.cache + __shfl_sync(0xffffffffu, row_at, r);
      const bool valid = j0 + r < k_hi;
      if (!valid) row = a.cache;
      for (int c = lane; c < per; c += 32)
        ta_cp16(c < kc ? dK + r * L.KR + c * 8 : dV + r * L.VR + (c - kc) * 8, row + (valid ? c * 8 : 0), valid);
    }
    ta_commit();
  };
  float o[CT][4];
#pragma unroll
  for (int i = 0; i < CT; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  constexpr int RW = KB == 16 ? 1 : 2;
  float m_[2] = {-INFINITY, -INFINITY}, l_[2] = {0.f, 0.f};
  const int nt_all = vc, nt0 = warp * CT;
  const int nkb = (k_hi - k_lo + KB - 1) / KB, n16 = (n + 15) / 16;
  load(0, k_lo);
  for (int kb = 0; kb < nkb; ++kb) {
    const int j0 = k_lo + kb * KB, st = stages > 1 ? kb & 1 : 0;
    ta_wait<0>();
    __syncthreads();                                      // the block is there, and nobody reads the other stage any more
    if (stages > 1 && kb + 1 < nkb) load(st ^ 1, j0 + KB);
    const bf16* tK = ring + st * stage_elems;
    const bf16* tV = tK + KB * L.KR;
    // scores: a unit is 16 keys of one key/value head; the rows of other heads are dropped
    for (int u = warp; u < G * (KB / 16); u += 8) {
      const int c = u / (KB / 16), kb16 = u % (KB / 16);
      float sc[2][4];
#pragma unroll
      for (int i = 0; i < 2; ++i) sc[i][0] = sc[i][1] = sc[i][2] = sc[i][3] = 0.f;
#pragma unroll 4
      for (int kk = 0; kk < n16; ++kk) {
        uint32_t qf[4], b0, b1, b2, b3;
        ta_ldsm4(qf[0], qf[1], qf[2], qf[3], sQ + ((mat & 1) * 8 + r8) * L.QS + kk * 16 + (mat >> 1) * 8);
        ta_ldsm4(b0, b1, b2, b3, tK + (kb16 * 16 + (mat >> 1) * 8 + r8) * L.KR + c * n + kk * 16 + (mat & 1) * 8);
        ta_mma(sc[0], qf, b0, b1);
        ta_mma(sc[1], qf, b2, b3);
      }
#pragma unroll
      for (int nt = 0; nt < 2; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int row = g8 + (e >> 1) * 8, col = kb16 * 16 + nt * 8 + 2 * tg + (e & 1);
          if (row < H && row / gs == c) sS[row * SS + col] = j0 + col < k_hi ? ta_score(sc[nt][e], a) : -INFINITY;
        }
    }
    __syncthreads();
    // a lane keeps its share of a row's sum; blocks of 16 keys: a row each half of the warp, else the warp's two rows one by one
#pragma unroll
    for (int x = 0; x < RW; ++x) {
      const int row = KB == 16 ? 2 * warp + (lane >> 4) : warp + x * 8, key = lane & (KB - 1);
      const float v = row < H ? sS[row * SS + key] : 0.f;
      float mn = v;
#pragma unroll
      for (int o2 = KB / 2; o2 > 0; o2 >>= 1) mn = fmaxf(mn, __shfl_xor_sync(0xffffffffu, mn, o2));
      mn = fmaxf(mn, m_[x]);                              // finite: a block holds a key
      const float p = ta_exp2(v - mn), cf = ta_exp2(m_[x] - mn);
      l_[x] = l_[x] * cf + p;
      m_[x] = mn;
      if (row < H) {
        sS[row * SS + key] = p;
        if (key == 0) corr[row] = cf;
      }
    }
    __syncthreads();
    const float c_lo = corr[g8], c_hi = corr[g8 + 8];
#pragma unroll
    for (int i = 0; i < CT; ++i) { o[i][0] *= c_lo; o[i][1] *= c_lo; o[i][2] *= c_hi; o[i][3] *= c_hi; }
#pragma unroll
    for (int kk = 0; kk < KB / 16; ++kk) {
      uint32_t t[3][4];
#pragma unroll
      for (int q4 = 0; q4 < 4; ++q4) {
        const float2 w = *(const float2*)(sS + (g8 + (q4 & 1) * 8) * SS + kk * 16 + (q4 >> 1) * 8 + 2 * tg);
        ta_split3(w.x, w.y, t[0][q4], t[1][q4], t[2][q4]);
      }
#pragma unroll
      for (int i = 0; i < CT; i += 2) {
        if (nt0 + i >= nt_all) break;
        uint32_t b[4];
        const bf16* vp = tV + (kk * 16 + (mat & 1) * 8 + r8) * L.VR + (nt0 + i + (mat >> 1)) * 8;    // one tile further may lie in the row's padding
        ta_ldsm4_trans(b[0], b[1], b[2], b[3], vp);
#pragma unroll
        for (int term = 2; term >= 0; --term) {
          ta_mma(o[i], t[term], b[0], b[1]);
          ta_mma(o[i + 1], t[term], b[2], b[3]);
        }
      }
    }
    if (stages == 1 && kb + 1 < nkb) {
      __syncthreads();
      load(0, j0 + KB);
    }
  }
  const int stride = 2 + G * dv;
  float* part = a.partial + ((size_t)s * a.slices + blockIdx.x) * H * stride;
#pragma unroll
  for (int x = 0; x < RW; ++x) {
    const int row = KB == 16 ? 2 * warp + (lane >> 4) : warp + x * 8;
#pragma unroll
    for (int o2 = KB / 2; o2 > 0; o2 >>= 1) l_[x] += __shfl_xor_sync(0xffffffffu, l_[x], o2);
    if (row < H && (lane & (KB - 1)) == 0) { part[(size_t)row * stride] = m_[x]; part[(size_t)row * stride + 1] = l_[x]; }
  }
#pragma unroll
  for (int i = 0; i < CT; ++i) {
    if (nt0 + i >= nt_all) break;
    const int col = (nt0 + i) * 8 + 2 * tg;
    if (g8 < H) *(float2*)(part + (size_t)g8 * stride + 2 + col) = make_float2(o[i][0], o[i][1]);
    if (g8 + 8 < H) *(float2*)(part + (size_t)(g8 + 8) * stride + 2 + col) = make_float2(o[i][2], o[i][3]);
  }
}

// joins a token's slices (ascending), divides by the sums (with the sink's share) and mixes.  A CTA takes 32 of the G * dv value
// columns' worth of one key/value head; a warp joins the slices of a head, then the head's outputs are mixed.
__global__ void __launch_bounds__(512) talking_merge_kernel(bf16* __restrict__ out, int ld_out, const float* __restrict__ partial,
                                                           const int* __restrict__ seg_q_start, const int* __restrict__ seg_pos0, int H,
                                                           int G, int dv, int all_slices, int slice_keys, const float* __restrict__ sink,
                                                           const float* __restrict__ talk) {
  __shared__ float R[TA_MAX_H][33];
  pdl_wait();
  pdl_launch_dependents();
  const int s = blockIdx.x, chunks = (dv + 31) / 32, c = blockIdx.y / chunks, col = (blockIdx.y % chunks) * 32 + (threadIdx.x & 31);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gs = H / G;
  const int stride = 2 + G * dv;
  const size_t step = (size_t)H * stride;
  const float* p = partial + (size_t)s * all_slices * step;
  const int slices = min(all_slices, seg_pos0[s] / slice_keys + 1);       // the slices that hold keys of this token
  for (int g = warp; g < H; g += 16) {
    const float* pg = p + (size_t)g * stride;
    const float snk = sink[g] * TA_LOG2E;
    float M = snk, L = 0.f, acc = 0.f;
    for (int i = lane; i < slices; i += 32) M = fmaxf(M, pg[(size_t)i * step]);
    M = warp_max(M);
    for (int base = 0; base < slices; base += 32) {
      const bool in = base + lane < slices;
      const float wi = in ? exp2f(pg[(size_t)(base + lane) * step] - M) : 0.f;
      L += in ? pg[(size_t)(base + lane) * step + 1] * wi : 0.f;
      const int cnt = min(32, slices - base);
#pragma unroll 16
      for (int j = 0; j < cnt; ++j) {
        const float wj = __shfl_sync(0xffffffffu, wi, j);
        if (col < dv) acc = fmaf(pg[(size_t)(base + j) * step + 2 + (size_t)c * dv + col], wj, acc);
      }
    }
    L = warp_sum(L) + exp2f(snk - M);
    R[g][lane] = acc / L;
  }
  __syncthreads();
  bf16* orow = out + (size_t)seg_q_start[s] * ld_out;
  if (col < dv)
    for (int hh = warp; hh < gs; hh += 16) {
      const int h = c * gs + hh;
      float w = 0.f;
      for (int g = 0; g < H; ++g) w = fmaf(talk[(size_t)h * H + g], R[g][lane], w);
      orow[(size_t)h * dv + col] = __float2bfloat16_rn(w);
    }
}

// S segments starting at rows seg_q_start[s] and positions seg_pos0[s].  max_q_len == 1: single tokens, their keys in `slices`
// slices of slice_keys (a multiple of 32) with `partial` [S, slices, H, 2 + G * dv] floats.  talk_host: [H, H] in host memory (it
// travels as a kernel parameter), talk: the same on the device.  cs: CTAs a tile's keys are shared out to (1, 2, 4 or 8).
// QV_ERR_UNSUPPORTED for sizes it does not take.
extern "C" int qv_talking_attention_mma(void* out, int ld_out, const void* q, int ld_q, const void* cache, const int* seg_q_start,
                                        const int* seg_pos0, const int* block_table, int max_blocks, int S, int max_q_len, int H, int G,
                                        int n, int dv, int page, float scale, float cap, const float* sink, const float* talk,
                                        const float* talk_host, float* partial, int slices, int slice_keys, int cs, void* stream) {
  if (S <= 0) return 0;
  if (n <= 0 || dv <= 0 || n % 8 || dv % 8 || n > 128 || dv > 128 || G <= 0 || H % G || H > TA_MAX_H || ld_q % 8 || ld_out % 2)
    return QV_ERR_UNSUPPORTED;
  if (S > 65535) return QV_ERR_TOO_LARGE;
  constexpr size_t LIMIT = 227 * 1024;
  TalkArgs a;
  a.out = (bf16*)out; a.ld_out = ld_out; a.q = (const bf16*)q; a.ld_q = ld_q; a.cache = (const bf16*)cache; a.seg_q_start = seg_q_start;
  a.seg_pos0 = seg_pos0; a.block_table = block_table; a.max_blocks = max_blocks; a.H = H; a.G = G; a.n = n; a.dv = dv; a.page = page;
  a.capped = cap > 0.f;
  a.pre = a.capped ? 2.0f * TA_LOG2E * scale / cap : TA_LOG2E * scale;
  a.post = a.capped ? cap * TA_LOG2E : 1.0f;
  a.sink = sink; a.talk = talk; a.talk_terms = 1; a.partial = partial;
  for (int i = 0; i < H * H; ++i) {
    uint32_t bits;
    memcpy(&bits, talk_host + i, 4);
    if (bits & 0xffffu) a.talk_terms = 3;
  } a.slices = slices < 1 ? 1 : slices; a.slice_keys = slice_keys;
  cudaStream_t st = (cudaStream_t)stream;
  int rc = QV_ERR_UNSUPPORTED;
  if (max_q_len == 1) {
    if (partial == nullptr || slice_keys <= 0 || slice_keys % TA_KEYS || G * dv > 2048) return QV_ERR_UNSUPPORTED;
    const TalkSliceLayout L = ta_slice_layout(G, n, dv);
    // blocks of 16 keys where two or three CTAs then share an SM (their loads overlap one another's products), else of 32
    int kb = ta_slice_smem(L, 32, 2) > 56 * 1024 ? 16 : 32, stages = 2;
    if (ta_slice_smem(L, kb, 2) > LIMIT) stages = 1;
    const size_t smem = ta_slice_smem(L, kb, stages);
    if (smem > LIMIT) return QV_ERR_UNSUPPORTED;
    const int per_warp = (G * (dv / 8) + 7) / 8;
#define TA_SLICE(KB_, CT_)                                                                                               \
  do {                                                                                                                   \
    cudaFuncSetAttribute(talking_slice_kernel<KB_, CT_>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);        \
    rc = qv_launch(talking_slice_kernel<KB_, CT_>, dim3(a.slices, S), dim3(256), smem, st, a, L, stages);                \
  } while (0)
    if (kb == 32) {
      if (per_warp <= 2) TA_SLICE(32, 2);
      else if (per_warp <= 8) TA_SLICE(32, 8);
      else return QV_ERR_UNSUPPORTED;                      // (56 KB do not hold so many value columns)
    } else {
      if (per_warp <= 8) TA_SLICE(16, 8);
      else if (per_warp <= 16) TA_SLICE(16, 16);
      else TA_SLICE(16, 32);
    }
#undef TA_SLICE
    if (rc) return rc;
    return qv_launch(talking_merge_kernel, dim3(S, G * ((dv + 31) / 32)), dim3(512), 0, st, (bf16*)out, ld_out, (const float*)partial,
                     seg_q_start, seg_pos0, H, G, dv, a.slices, slice_keys, sink, talk);
  }
  if (cs != 1 && cs != 2 && cs != 4 && cs != 8) return QV_ERR_UNSUPPORTED;
  const int NP = n <= 64 ? 64 : 128, DP = dv <= 64 ? 64 : 128;
  const size_t smem = ta_tile_smem(H, G, NP, DP, dv);
  if (smem > LIMIT) return QV_ERR_UNSUPPORTED;
  const size_t stat_off = smem - (size_t)2 * H * 16 * sizeof(float);
#define TA_TILE(NP_, DP_, HP_)                                                                                                       \
  do {                                                                                                                               \
    TalkMatrix<(HP_ < 16 ? HP_ : 1)> mix;                                                                                                             \
    if (HP_ < 16)                                                                                                                    \
      for (int h = 0; h < HP_; ++h)                                                                                                  \
        for (int g = 0; g < HP_; ++g) mix.t[HP_ < 16 ? h * HP_ + g : 0] = h < H && g < H ? talk_host[h * H + g] : 0.f;                              \
    cudaFuncSetAttribute(talking_tile_kernel<NP_, DP_, HP_>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);                \
    rc = qv_launch_cluster(talking_tile_kernel<NP_, DP_, HP_>, dim3((max_q_len + 15) / 16 * cs, 1, S), dim3(32 * H), smem, st,       \
                           dim3(cs, 1, 1), a, mix, cs, stat_off);                                                                    \
  } while (0)
#define TA_TILES(HP_)                                  \
  do {                                                 \
    if (NP == 64 && DP == 64) TA_TILE(64, 64, HP_);    \
    else if (NP == 64) TA_TILE(64, 128, HP_);          \
    else if (DP == 64) TA_TILE(128, 64, HP_);          \
    else TA_TILE(128, 128, HP_);                       \
  } while (0)
  if (H <= 4) TA_TILES(4);
  else if (H <= 8) TA_TILES(8);
  else TA_TILES(16);
#undef TA_TILES
#undef TA_TILE
  return rc;
}
