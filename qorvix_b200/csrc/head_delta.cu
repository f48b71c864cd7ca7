// Delta rule whose state decays by one number per head and token:
//
//   S <- g_t S;   u_t = beta_t (v_t - S^T k_t);   S <- S + k_t u_t^T;   o_t = S^T q_t
//
// per request and value head, S [dk x dv] float32 in the request's state slot, q and k unit vectors shared by the H / G value
// heads of a query/key head.  Since the decay is a number, B tokens in a row can be worked through together from the state S0
// ahead of them: with G_t = g_1 .. g_t, D(t, i) = g_(i+1) .. g_t and p_t = S0^T k_t, r_t = S0^T q_t,
//
//   u_t = beta_t v_t - (beta_t G_t) p_t - sum_(i < t) (beta_t D(t, i) k_t.k_i) u_i
//   o_t = G_t r_t + sum_(i <= t) (D(t, i) q_t.k_i) u_i
//   S   = G_B S0 + sum_i D(B, i) k_i u_i^T
//
// which is the same recurrence with other sums: the 2 B dot products with S0 do not wait for one another, so a chain of B
// tokens costs about what one token does.  There are only products of decays (each at most one), no quotients.
//
// qv_head_delta_operands  unit vectors of q and k (q times q_scale), decays g = exp(-rate softplus(a + dt_bias)), beta = sigmoid(b)
//                         and the factors above, 12 numbers per token and head (HD_COEF), for blocks of `block` tokens counted
//                         from the start of the request's portion.
// qv_head_delta_scan      the recurrence.  A column of S belongs to a few lanes that hold 16 rows each in registers; the tokens'
//                         vectors and factors arrive in shared memory by cp.async, a chunk of tokens ahead.
//
// Everything is float32.  With block = 1 (what the 32-bit path uses, and what single tokens amount to in any case) the order of
// every sum depends on the sizes alone; with block = 4 it also depends on where a portion starts, that is, cuts agree to rounding.
#include "common.cuh"
#include <type_traits>

// factors per token and head: beta, beta G, G, g, then beta D(t, i) k_t.k_i for i < 3, then D(t, i) q_t.k_i for i < 4
#define HD_COEF 12
#define HD_BLOCK 4
#define HD_WARPS 4
#define HD_ROWS 16
#define HD_PAD 20           // floats a lane's rows take in a stage: 16 and 4 of padding, so that 16-byte reads of the LPC lanes miss one another's banks

// q, k [T, G * n] float32 (row strides), a, b [T, H] -> qn, kn [T, G * n] dense, coef [T, H, HD_COEF].  One warp per (token, query/key head).
__global__ void __launch_bounds__(128) head_delta_operands_kernel(float* __restrict__ qn, float* __restrict__ kn, float* __restrict__ coef,
                                                                 const float* __restrict__ q, int ld_q, const float* __restrict__ k, int ld_k,
                                                                 const float* __restrict__ a, int ld_a, const float* __restrict__ b, int ld_b,
                                                                 const float* __restrict__ rate, const float* __restrict__ dt_bias,
                                                                 const int* __restrict__ tok_seg, const int* __restrict__ seg_q_start, int H,
                                                                 int G, int n, float eps, float q_scale, int block) {
  pdl_wait();
  pdl_launch_dependents();
  const int t = blockIdx.x, c = blockIdx.y * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (c >= G) return;
  const int tau = (t - seg_q_start[tok_seg[t]]) % block;           // the token's place in its block
  const float* qr = q + (size_t)t * ld_q + (size_t)c * n;
  const float* kr = k + (size_t)t * ld_k + (size_t)c * n;
  float qq = 0.f, qk[HD_BLOCK] = {}, kk[HD_BLOCK] = {}, k2[HD_BLOCK] = {};      // index d: the token d places back in the block
  for (int i = lane; i < n; i += 32) {
    const float qv = qr[i], kv = kr[i];
    qq = fmaf(qv, qv, qq);
    qk[0] = fmaf(qv, kv, qk[0]);
    k2[0] = fmaf(kv, kv, k2[0]);
#pragma unroll
    for (int d = 1; d < HD_BLOCK; ++d) {
      if (d <= tau) {
        const float o = kr[i - (long long)d * ld_k];
        qk[d] = fmaf(qv, o, qk[d]);
        kk[d] = fmaf(kv, o, kk[d]);
        k2[d] = fmaf(o, o, k2[d]);
      }
    }
  }
  qq = warp_sum(qq);
  qk[0] = warp_sum(qk[0]);
  k2[0] = warp_sum(k2[0]);
#pragma unroll
  for (int d = 1; d < HD_BLOCK; ++d)
    if (d <= tau) { qk[d] = warp_sum(qk[d]); kk[d] = warp_sum(kk[d]); k2[d] = warp_sum(k2[d]); }
  const float iq = q_scale / sqrtf(qq + eps);
  float ik[HD_BLOCK];
#pragma unroll
  for (int d = 0; d < HD_BLOCK; ++d) ik[d] = 1.0f / sqrtf(k2[d] + eps);
  const size_t o = ((size_t)t * G + c) * n;
  for (int i = lane; i < n; i += 32) {
    qn[o + i] = qr[i] * iq;
    kn[o + i] = kr[i] * ik[0];
  }
  const int gs = H / G;
  for (int hh = lane; hh < gs; hh += 32) {
    const int h = c * gs + hh;
    const float rt = rate[h], db = dt_bias[h];
    const float beta = 1.0f / (1.0f + expf(-b[(size_t)t * ld_b + h]));
    float out[HD_COEF];
#pragma unroll
    for (int i = 0; i < HD_COEF; ++i) out[i] = 0.f;
    float D = 1.0f;                                                // D(t, t - d)
#pragma unroll
    for (int d = 0; d < HD_BLOCK; ++d) {
      if (d <= tau) {
        const int i = tau - d;                                     // the place of that token in the block
#pragma unroll
        for (int x = 0; x < HD_BLOCK; ++x)
          if (x == i) {
            out[7 + x] = D * (qk[d] * iq * ik[d]);
            if (d > 0 && x < 3) out[4 + x] = beta * D * (kk[d] * ik[0] * ik[d]);
          }
        const float z = a[(size_t)(t - d) * ld_a + h] + db;
        const float g = expf(-rt * (fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)))));
        if (d == 0) out[3] = g;
        D *= g;
      }
    }
    out[0] = beta; out[1] = beta * D; out[2] = D;
    float4* dst = (float4*)(coef + ((size_t)t * H + h) * HD_COEF);
    dst[0] = make_float4(out[0], out[1], out[2], out[3]);
    dst[1] = make_float4(out[4], out[5], out[6], out[7]);
    dst[2] = make_float4(out[8], out[9], out[10], out[11]);
  }
}

extern "C" int qv_head_delta_coef() { return HD_COEF; }
extern "C" int qv_head_delta_block() { return HD_BLOCK; }

extern "C" int qv_head_delta_operands(float* qn, float* kn, float* coef, const float* q, int ld_q, const float* k, int ld_k, const float* a,
                                      int ld_a, const float* b, int ld_b, const float* rate, const float* dt_bias, const int* tok_seg,
                                      const int* seg_q_start, int T, int H, int G, int n, float eps, float q_scale, int block, void* stream) {
  if (T <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || n <= 0 || (block != 1 && block != HD_BLOCK)) return QV_ERR_UNSUPPORTED;
  return qv_launch(head_delta_operands_kernel, dim3(T, (G + 3) / 4), dim3(128), 0, (cudaStream_t)stream, qn, kn, coef, q, ld_q, k, ld_k, a,
                   ld_a, b, ld_b, rate, dt_bias, tok_seg, seg_q_start, H, G, n, eps, q_scale, block);
}

// ---------------------------------------------------------------- the scan
struct HeadDeltaArgs {
  float* out; int ld_out;                 // [T, H * dv]
  const float* qn; const float* kn;       // [T, G * dk] dense
  const float* v; int ld_v;               // [T, H * dv]
  const float* coef;                      // [T, H, HD_COEF]
  float* state; long long slot_stride;    // per slot: [H][tiles][HD_ROWS][32]
  const int* seg_q_start; const int* seg_slot;
  int H, G, dk, dv;
};

// 4 or 16 bytes, or as many zero bytes where `valid` is false
__device__ __forceinline__ void hd_cp4(float* dst, const float* src, bool valid) {
  const int bytes = valid ? 4 : 0;
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void hd_cp16(float* dst, const float* src, bool valid) {
  const int bytes = valid ? 16 : 0;
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src), "r"(bytes) : "memory");
}

// sum over the lane's rows of x * S (four partial sums, a fixed order)
__device__ __forceinline__ float hd_dot(const float4* x, const float (&S)[HD_ROWS]) {
  float p0 = 0.f, p1 = 0.f, p2 = 0.f, p3 = 0.f;
#pragma unroll
  for (int i = 0; i < HD_ROWS / 4; ++i) {
    const float4 x4 = x[i];
    p0 = fmaf(x4.x, S[4 * i], p0); p1 = fmaf(x4.y, S[4 * i + 1], p1);
    p2 = fmaf(x4.z, S[4 * i + 2], p2); p3 = fmaf(x4.w, S[4 * i + 3], p3);
  }
  return (p0 + p1) + (p2 + p3);
}

// LPC lanes own a column (key sizes up to 16 LPC), a warp 32 / LPC columns, a CTA four times that.  B tokens at a time; `chunk` (a
// multiple of B) tokens a stage, two stages.  vec4: dk is a multiple of 4 (16-byte copies).
template <int LPC, int B>
__global__ void __launch_bounds__(32 * HD_WARPS) head_delta_scan_kernel(HeadDeltaArgs a, int chunk, int vec4) {
  extern __shared__ __align__(16) float hd_ring[];
  constexpr int CPW = 32 / LPC, CTA_COLS = HD_WARPS * CPW, NTH = 32 * HD_WARPS;
  constexpr int VEC = HD_PAD * LPC;                       // floats a vector takes in a stage
  constexpr int ROW = 2 * VEC + HD_COEF + CTA_COLS;       // floats a token takes: k, q, factors, values
  pdl_wait();
  const int s = blockIdx.x, h = blockIdx.y;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int lic = lane % LPC, cw = lane / LPC;
  const int dk = a.dk, dv = a.dv, H = a.H;
  const int cta_col0 = blockIdx.z * CTA_COLS;
  const int col = cta_col0 + warp * CPW + cw;
  const int tiles = (dv + CPW - 1) / CPW;
  const int q0 = a.seg_q_start[s], len = a.seg_q_start[s + 1] - q0;
  const int tile = blockIdx.z * HD_WARPS + warp;
  const bool active = tile < tiles;
  float* st = a.state + (size_t)a.seg_slot[s] * a.slot_stride + ((size_t)h * tiles + tile) * (HD_ROWS * 32) + lane;
  float S[HD_ROWS];
#pragma unroll
  for (int i = 0; i < HD_ROWS; ++i) S[i] = active ? st[i * 32] : 0.f;
  const int c = h / (H / a.G), ldk = a.G * dk;
  const size_t ck = (size_t)c * dk, hv = (size_t)h * dv;
  const float* srcs[2] = {a.kn + ck, a.qn + ck};
  auto issue = [&](int ch) {
    float* base = hd_ring + (size_t)(ch & 1) * chunk * ROW;
    const int j0 = ch * chunk, nt = min(chunk, len - j0);
#pragma unroll
    for (int v = 0; v < 2; ++v) {
      if (vec4) {
        constexpr int PER = HD_ROWS * LPC / 4;            // 16-byte pieces a vector (padding rows included)
        for (int i = tid; i < nt * PER; i += NTH) {
          const int j = i / PER, r = (i % PER) * 4;
          hd_cp16(base + j * ROW + v * VEC + r + (r / HD_ROWS) * (HD_PAD - HD_ROWS), srcs[v] + (size_t)(q0 + j0 + j) * ldk + (r < dk ? r : 0), r < dk);
        }
      } else {
        constexpr int PER = HD_ROWS * LPC;
        for (int i = tid; i < nt * PER; i += NTH) {
          const int j = i / PER, r = i % PER;
          hd_cp4(base + j * ROW + v * VEC + r + (r / HD_ROWS) * (HD_PAD - HD_ROWS), srcs[v] + (size_t)(q0 + j0 + j) * ldk + (r < dk ? r : 0), r < dk);
        }
      }
    }
    for (int i = tid; i < nt * (HD_COEF / 4); i += NTH) {
      const int j = i / (HD_COEF / 4), r = (i % (HD_COEF / 4)) * 4;
      hd_cp16(base + j * ROW + 2 * VEC + r, a.coef + ((size_t)(q0 + j0 + j) * H + h) * HD_COEF + r, true);
    }
    for (int i = tid; i < nt * CTA_COLS; i += NTH) {
      const int j = i / CTA_COLS, cc = i % CTA_COLS;
      const bool in = cta_col0 + cc < dv;
      hd_cp4(base + j * ROW + 2 * VEC + HD_COEF + cc, a.v + (size_t)(q0 + j0 + j) * a.ld_v + hv + (in ? cta_col0 + cc : 0), in);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  // up to B tokens at a time (FULL: all B, without a branch, so that their reads and sums interleave)
  auto tokens = [&](const float* d, int j, int nb, auto full) {
    constexpr bool FULL = decltype(full)::value;
    float p[B], r[B], u[B], e[B];
#pragma unroll
    for (int t = 0; t < B; ++t) {
      p[t] = r[t] = 0.f;
      if (FULL || t < nb) {
        p[t] = hd_dot((const float4*)(d + t * ROW + lic * HD_PAD), S);
        r[t] = hd_dot((const float4*)(d + t * ROW + VEC + lic * HD_PAD), S);
      }
    }
#pragma unroll
    for (int o = LPC / 2; o > 0; o >>= 1)
#pragma unroll
      for (int t = 0; t < B; ++t) {
        p[t] += __shfl_xor_sync(0xffffffffu, p[t], o);
        r[t] += __shfl_xor_sync(0xffffffffu, r[t], o);
      }
    float Gall = 1.0f;
#pragma unroll
    for (int t = 0; t < B; ++t) {
      u[t] = 0.f;
      e[t] = 1.f;
      if (FULL || t < nb) {
        const float* f = d + t * ROW + 2 * VEC;
        const float4 f0 = *(const float4*)f, f1 = *(const float4*)(f + 4), f2 = *(const float4*)(f + 8);
        const float kkc[3] = {f1.x, f1.y, f1.z}, qkc[4] = {f1.w, f2.x, f2.y, f2.z};
        float uu = fmaf(f0.x, f[HD_COEF + warp * CPW + cw], -f0.y * p[t]);
#pragma unroll
        for (int i = 0; i < t; ++i) uu = fmaf(-kkc[i], u[i], uu);
        u[t] = uu;
        float y = f0.z * r[t];
#pragma unroll
        for (int i = 0; i <= t; ++i) y = fmaf(qkc[i], u[i], y);
        if (lic == 0 && col < dv) a.out[(size_t)(q0 + j + t) * a.ld_out + hv + col] = y;
        Gall = f0.z;
#pragma unroll
        for (int i = 0; i < t; ++i) e[i] *= f0.w;
      }
    }
#pragma unroll
    for (int i = 0; i < HD_ROWS; ++i) S[i] *= Gall;
#pragma unroll
    for (int t = 0; t < B; ++t) {
      if (FULL || t < nb) {
        const float ue = u[t] * e[t];
        const float4* pk = (const float4*)(d + t * ROW + lic * HD_PAD);
#pragma unroll
        for (int i = 0; i < HD_ROWS / 4; ++i) {
          const float4 k4 = pk[i];
          S[4 * i] = fmaf(k4.x, ue, S[4 * i]); S[4 * i + 1] = fmaf(k4.y, ue, S[4 * i + 1]);
          S[4 * i + 2] = fmaf(k4.z, ue, S[4 * i + 2]); S[4 * i + 3] = fmaf(k4.w, ue, S[4 * i + 3]);
        }
      }
    }
  };
  const int nchunks = (len + chunk - 1) / chunk;
  if (nchunks > 0) issue(0);
  for (int ch = 0; ch < nchunks; ++ch) {
    if (ch + 1 < nchunks) {
      issue(ch + 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const int j0 = ch * chunk, nt = min(chunk, len - j0);
    if (active) {
      const float* d = hd_ring + (size_t)(ch & 1) * chunk * ROW;
      int jb = 0;
      for (; jb + B <= nt; jb += B) tokens(d + jb * ROW, j0 + jb, B, std::true_type{});
      if (jb < nt) tokens(d + jb * ROW, j0 + jb, nt - jb, std::false_type{});
    }
    __syncthreads();
  }
  pdl_launch_dependents();
  if (!active) return;
#pragma unroll
  for (int i = 0; i < HD_ROWS; ++i) st[i * 32] = S[i];
}

// A launch that starts only when the kernel before it has ended: a scan over portions is a long kernel of few CTAs that wants an
// SM each; launched ahead its CTAs are placed while the kernel before it still fills the SMs, several on one SM.
template <typename... KArgs, typename... Args>
static inline int hd_launch_after(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t st, Args&&... args) {
  cudaLaunchConfig_t cfg;
  memset(&cfg, 0, sizeof(cfg));
  cfg.gridDim = grid;
  cfg.blockDim = block;
  cfg.dynamicSmemBytes = smem;
  cfg.stream = st;
  return (int)cudaLaunchKernelEx(&cfg, kernel, std::forward<Args>(args)...);
}

static inline int hd_lanes_per_column(int dk) { return dk <= 16 ? 1 : dk <= 32 ? 2 : dk <= 64 ? 4 : dk <= 128 ? 8 : 16; }

extern "C" long long qv_head_delta_state_floats(int H, int dk, int dv) {
  const int cpw = 32 / hd_lanes_per_column(dk);
  return (long long)H * ((dv + cpw - 1) / cpw) * HD_ROWS * 32;
}

// block: as for qv_head_delta_operands.  max_q_len: the longest segment of the step.
extern "C" int qv_head_delta_scan(float* out, int ld_out, const float* qn, const float* kn, const float* v, int ld_v, const float* coef,
                                  float* state, long long slot_stride, const int* seg_q_start, const int* seg_slot, int S, int max_q_len,
                                  int H, int G, int dk, int dv, int block, void* stream) {
  if (S <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || dk <= 0 || dv <= 0 || H > 65535 || (block != 1 && block != HD_BLOCK)) return QV_ERR_UNSUPPORTED;
  if (dk > 256) return QV_ERR_TOO_LARGE;
  HeadDeltaArgs a;
  a.out = out; a.ld_out = ld_out; a.qn = qn; a.kn = kn; a.v = v; a.ld_v = ld_v; a.coef = coef; a.state = state; a.slot_stride = slot_stride;
  a.seg_q_start = seg_q_start; a.seg_slot = seg_slot; a.H = H; a.G = G; a.dk = dk; a.dv = dv;
  const int lpc = hd_lanes_per_column(dk);
  const int cta_cols = HD_WARPS * 32 / lpc;
  const int ctas = (dv + cta_cols - 1) / cta_cols;
  if (ctas > 65535) return QV_ERR_TOO_LARGE;
  dim3 grid(S, H, ctas), blk(32 * HD_WARPS);
  cudaStream_t st = (cudaStream_t)stream;
  const int row = 2 * HD_PAD * lpc + HD_COEF + cta_cols;
  int chunk = max_q_len <= 1 ? 1 : (max_q_len > 32 ? 32 : (max_q_len + 3) / 4 * 4);
  while (chunk > HD_BLOCK && (size_t)2 * chunk * row * sizeof(float) > 96 * 1024) chunk -= HD_BLOCK;
  if (block > 1 && max_q_len > 1 && chunk < HD_BLOCK) chunk = HD_BLOCK;
  const size_t smem = (size_t)2 * chunk * row * sizeof(float);
  const int vec4 = dk % 4 == 0 && (((uintptr_t)qn | (uintptr_t)kn) & 15) == 0;
  if (((uintptr_t)coef) & 15) return QV_ERR_UNSUPPORTED;
#define HD_LAUNCH(LPC_, B_)                                                                                                  \
  do {                                                                                                                       \
    cudaFuncSetAttribute(head_delta_scan_kernel<LPC_, B_>, cudaFuncAttributeMaxDynamicSharedMemorySize, 96 * 1024);          \
    if (max_q_len >= 16) return hd_launch_after(head_delta_scan_kernel<LPC_, B_>, grid, blk, smem, st, a, chunk, vec4);      \
    return qv_launch(head_delta_scan_kernel<LPC_, B_>, grid, blk, smem, st, a, chunk, vec4);                                 \
  } while (0)
#define HD_BLOCKS(LPC_)                                   \
  do {                                                    \
    if (block == 1 || max_q_len <= 1) HD_LAUNCH(LPC_, 1); \
    HD_LAUNCH(LPC_, HD_BLOCK);                            \
  } while (0)
  if (lpc == 1) HD_BLOCKS(1);
  if (lpc == 2) HD_BLOCKS(2);
  if (lpc == 4) HD_BLOCKS(4);
  if (lpc == 8) HD_BLOCKS(8);
  HD_BLOCKS(16);
#undef HD_BLOCKS
#undef HD_LAUNCH
}
