// The state-space layer (Mamba-2's form): a linear attention whose state decays by one number per head and token, with keys B and
// queries C shared by groups of heads and values x per head,
//
//   S_t = a_t S_(t-1) + dt_t B_t x_t^T,   y_t = S_t^T C_t + D x_t        per head; S is [N, vdim], 32-bit, one record per sequence
//   a_t = exp(-exp(A_log) dt_t),          dt_t = softplus(raw_t + dt_bias)
//
//   ssm_gates            dt and log a = -exp(A_log) dt per token and head, 32-bit, from the projection in the run's element type
//   (token by token)     `gated_attn` of gated_recurrent.cu with q = C, k = B, v = x, b = dt: decode steps, short portions, 32-bit runs
//   scalar_decay chunked the same recurrence for the prompts of bfloat16 runs, chunks of 64 tokens on the tensor cores (below)
//   ssm_gate_norm        y + D x, times silu(z), each of several equal parts of the row divided by its root mean square, times a weight:
//                        the gate comes before the norm
#include "common.cuh"

RL_DEFINE_ERROR_TEXT()

template <typename T>
__device__ __forceinline__ float ss_load(const T* p) { return to_f32(__ldcg(p)); }

// ---------------------------------------------------------------- step size and decay
template <typename T>
__global__ void ssm_gates_kernel(const T* __restrict__ raw, int raw_stride, const float* __restrict__ a_log, const float* __restrict__ dt_bias,
                                 float* __restrict__ log_a, float* __restrict__ dt_out, int n_tokens, int H) {
  pdl_trigger();
  pdl_wait();
  const int idx = blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= n_tokens * H) return;
  const int t = idx / H, h = idx - t * H;
  const float z = ss_load(raw + (size_t)t * raw_stride + h) + dt_bias[h];
  const float dt = fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)));
  dt_out[idx] = dt;
  log_a[idx] = -expf(a_log[h]) * dt;
}

RL_API int rl_ssm_gates(const void* raw, int dtype, int raw_stride, const float* a_log, const float* dt_bias, float* log_a, float* dt,
                        int n_tokens, int H, cudaStream_t stream) {
  if (n_tokens <= 0 || H <= 0 || raw_stride < H) RL_REFUSE(1, "ssm_gates: T=%d H=%d row stride %d", n_tokens, H, raw_stride);
  if ((long long)n_tokens * H > 0x7fffff00LL) RL_REFUSE(2, "ssm_gates: %d tokens of %d heads are too many", n_tokens, H);
  const int blocks = (n_tokens * H + 127) / 128;
  if (dtype == RL_BF16)
    RL_LAUNCH_CHECK(rl_launch(ssm_gates_kernel<bf16>, blocks, 128, 0, stream, (const bf16*)raw, raw_stride, a_log, dt_bias, log_a, dt, n_tokens, H));
  else if (dtype == RL_F32)
    RL_LAUNCH_CHECK(rl_launch(ssm_gates_kernel<float>, blocks, 128, 0, stream, (const float*)raw, raw_stride, a_log, dt_bias, log_a, dt, n_tokens, H));
  else
    RL_REFUSE(3, "ssm_gates: unknown dtype %d", dtype);
  return 0;
}

// ---------------------------------------------------------------- skip, gate, norm in parts
// Row t: v = (y + D[head] x) * silu(z); the row of n numbers cut into `groups` equal parts, out = v / sqrt(mean(v^2 over its part) + eps) * w.
// One block per row; a unit is U neighbouring numbers (four where the sizes allow), kept in registers; every unit leaves its sum of
// squares in shared memory and a warp per part adds them up, so a row's bits depend on the sizes alone.
template <typename T, int U, int UNITS>
__global__ void __launch_bounds__(UNITS == 1 ? 1024 : 512)
ssm_gate_norm_kernel(const float* __restrict__ y, int y_stride, const T* __restrict__ x, int x_stride, const float* __restrict__ D, int vdim,
                     const T* __restrict__ z, int z_stride, const float* __restrict__ w, float eps, int groups, T* __restrict__ out,
                     int out_stride, int n, float out_scale) {
  extern __shared__ __align__(16) float unit_ss[];  // [n / U], then 1 / rms of the parts
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x;
  const int n_units = n / U, per_group = n_units / groups;
  float* inv_rms = unit_ss + n_units;
  float v[UNITS][U];
#pragma unroll
  for (int c = 0; c < UNITS; ++c) {
    const int u = threadIdx.x + c * blockDim.x, i = u * U;
    if (u >= n_units) continue;
    float yv[U], xv[U], zv[U];
    if (U == 4) {
      load4_g<float>(y + (size_t)t * y_stride + i, yv);
      load4_g<T>(x + (size_t)t * x_stride + i, xv);
      load4_g<T>(z + (size_t)t * z_stride + i, zv);
    } else {
      yv[0] = __ldcg(y + (size_t)t * y_stride + i);
      xv[0] = ss_load(x + (size_t)t * x_stride + i);
      zv[0] = ss_load(z + (size_t)t * z_stride + i);
    }
    const float d = D[i / vdim];
    float ss = 0.f;
#pragma unroll
    for (int e = 0; e < U; ++e) {
      v[c][e] = (yv[e] + d * xv[e]) * (zv[e] / (1.0f + expf(-zv[e])));
      ss += v[c][e] * v[c][e];
    }
    unit_ss[u] = ss;
  }
  __syncthreads();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
  for (int g = warp; g < groups; g += nwarps) {
    float ss = 0.f;
    for (int u = lane; u < per_group; u += 32) ss += unit_ss[g * per_group + u];
    ss = warp_sum(ss);
    if (lane == 0) inv_rms[g] = out_scale / sqrtf(ss / (float)(per_group * U) + eps);
  }
  __syncthreads();
#pragma unroll
  for (int c = 0; c < UNITS; ++c) {
    const int u = threadIdx.x + c * blockDim.x, i = u * U;
    if (u >= n_units) continue;
    const float inv = inv_rms[u / per_group];
    float o[U];
#pragma unroll
    for (int e = 0; e < U; ++e) o[e] = v[c][e] * inv * w[i + e];
    if (U == 4) store4<T>(out + (size_t)t * out_stride + i, o);
    else out[(size_t)t * out_stride + i] = from_f32<T>(o[0]);
  }
}

template <typename T>
static int launch_gate_norm(const float* y, int y_stride, const void* x, int x_stride, const float* D, int vdim, const void* z, int z_stride,
                            const float* w, float eps, int groups, void* out, int out_stride, int n_rows, int n, float out_scale,
                            cudaStream_t stream) {
  const bool vec = (n / groups) % 4 == 0 && vdim % 4 == 0 && ((y_stride | x_stride | z_stride | out_stride) & 3) == 0 &&
                   ((((uintptr_t)y | (uintptr_t)w) & 15) == 0) && ((((uintptr_t)x | (uintptr_t)z | (uintptr_t)out) & (4 * sizeof(T) - 1)) == 0);
  const int n_units = vec ? n / 4 : n;
  const size_t smem = (size_t)(n_units + groups) * sizeof(float);
  if (n_units > 8 * 1024 || smem > 48 * 1024) RL_REFUSE(4, "ssm_gate_norm: a row of %d numbers (%d parts) is too long", n, groups);
  const int full = n_units >= 1024 ? 1024 : ((n_units + 31) / 32) * 32;
#define RL_SGN(U, UNITS, TH)                                                                                                         \
  do {                                                                                                                               \
    RL_LAUNCH_CHECK(rl_launch(ssm_gate_norm_kernel<T, U, UNITS>, n_rows, TH, smem, stream, y, y_stride, (const T*)x, x_stride, D, vdim, \
                              (const T*)z, z_stride, w, eps, groups, (T*)out, out_stride, n, out_scale));                            \
    return 0;                                                                                                                        \
  } while (0)
  if (vec) {
    if (n_units <= 1024 && (n_rows < 64 || n_units <= 256)) RL_SGN(4, 1, full);
    if (n_units <= 1024) RL_SGN(4, 4, 256);
    if (n_units <= 2048) RL_SGN(4, 4, 512);
    RL_SGN(4, 16, 512);
  }
  if (n_units <= 1024) RL_SGN(1, 1, full);
  RL_SGN(1, 16, 512);
#undef RL_SGN
}

RL_API int rl_ssm_gate_norm(const float* y, int y_stride, const void* x, int x_stride, const float* D, int vdim, const void* z, int z_stride,
                            const float* w, float eps, int groups, void* out, int out_stride, int act_dtype, int n_rows, int n, float out_scale,
                            cudaStream_t stream) {
  if (n_rows <= 0 || n <= 0 || vdim <= 0 || n % vdim || groups <= 0 || n % groups)
    RL_REFUSE(1, "ssm_gate_norm: rows=%d n=%d head=%d parts=%d", n_rows, n, vdim, groups);
  if (!y || !x || !D || !z || !w || !out) RL_REFUSE(2, "ssm_gate_norm: an operand is missing");
  if (act_dtype == RL_BF16)
    return launch_gate_norm<bf16>(y, y_stride, x, x_stride, D, vdim, z, z_stride, w, eps, groups, out, out_stride, n_rows, n, out_scale, stream);
  if (act_dtype == RL_F32)
    return launch_gate_norm<float>(y, y_stride, x, x_stride, D, vdim, z, z_stride, w, eps, groups, out, out_stride, n_rows, n, out_scale, stream);
  RL_REFUSE(3, "ssm_gate_norm: unknown dtype %d", act_dtype);
}

// ---------------------------------------------------------------- the recurrence, chunk by chunk, on the tensor cores
// Chunks of SC tokens; with n tokens in a chunk, S the state before it, A_i = sum_{l <= i} log a_l inside the chunk:
//   U      = sum_j exp(A_(n-1) - A_j) b_j k_j v_j^T                                            (1) what the chunk adds, every chunk at once
//   S_next = exp(A_(n-1)) S + U                                                                 (2) the states before every chunk, in order
//   o_i    = exp(A_i) S^T q_i + sum_{j <= i} (q_i . k_j) exp(A_i - A_j) b_j v_j                 (3) the outputs, every chunk at once
// Only exponents <= 0 occur.  q, k, v are bfloat16 (activations); every 32-bit operand of a product (the weighted values of (1), the
// decayed scores and the state of (3)) goes to the tensor cores as two bfloat16 numbers, the value rounded and what the rounding
// left, so the products see 16 digits of it; all sums, decays and the states are 32-bit.
#define SC 64  // tokens per chunk

__device__ __forceinline__ void sc_ldmatrix_x4(uint32_t (&r)[4], const void* smem) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(smem);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void sc_ldmatrix_x4_trans(uint32_t (&r)[4], const void* smem) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(smem);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void sc_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void sc_split(float v, bf16& hi, bf16& lo) {
  hi = __float2bfloat16_rn(v);
  lo = __float2bfloat16_rn(v - __bfloat162float(hi));
}
__device__ __forceinline__ uint32_t sc_pack(bf16 a, bf16 b) {
  __nv_bfloat162 v(a, b);
  return *reinterpret_cast<uint32_t*>(&v);
}
__device__ __forceinline__ void sc_cp_async_16(void* smem, const void* gmem) {
  const uint32_t s = (uint32_t)__cvta_generic_to_shared(smem);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(s), "l"(gmem));
}
__device__ __forceinline__ void sc_cp_async_wait_all() {
  asm volatile("cp.async.commit_group;\ncp.async.wait_group 0;\n" ::: "memory");
}

// rows [SC][width] of bfloat16 (row stride `stride` in global memory, rows from n on and columns from width on zero) into dst [SC][HD + 8]
template <int HD>
__device__ __forceinline__ void sc_load_tile(bf16* dst, const bf16* src, int stride, int n, int width, bool vec8) {
  constexpr int STRIDE = HD + 8;
  for (int idx = threadIdx.x; idx < SC * (HD / 8); idx += 128) {
    const int i = idx / (HD / 8), r = 8 * (idx - i * (HD / 8));
    bf16* d = dst + i * STRIDE + r;
    if (i < n && vec8 && r < width) {
      sc_cp_async_16(d, src + (size_t)i * stride + r);
    } else {
#pragma unroll
      for (int e = 0; e < 8; ++e) d[e] = (i < n && r + e < width) ? __ldcg(src + (size_t)i * stride + r + e) : __float2bfloat16_rn(0.f);
    }
  }
}

// A_i of the chunk's tokens (tokens past the end repeat the last sum) and b_j, by the first two warps; a barrier must follow
__device__ __forceinline__ void sc_load_decays(float* A_s, float* b_s, const float* log_decay, const float* in_scale, size_t t0, int n, int H, int h) {
  if (threadIdx.x < 32) {
    const int lane = threadIdx.x;
    float a0 = 2 * lane < n ? __ldcg(log_decay + (t0 + 2 * lane) * H + h) : 0.f;
    float a1 = 2 * lane + 1 < n ? __ldcg(log_decay + (t0 + 2 * lane + 1) * H + h) : 0.f;
    float run = a0 + a1;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float up = __shfl_up_sync(0xffffffffu, run, o);
      if (lane >= o) run += up;
    }
    A_s[2 * lane + 1] = run;
    A_s[2 * lane] = run - a1;
  } else if (threadIdx.x < 32 + SC) {
    const int j = threadIdx.x - 32;
    b_s[j] = j < n ? (in_scale ? __ldcg(in_scale + (t0 + j) * H + h) : 1.f) : 0.f;
  }
}

// (1): a block of four warps per (sequence, head, chunk); warp w owns rows HDK/4 w .. of U.  The keys lie in shared memory as
// [token][dim], the transpose of the product's first operand: `ldmatrix.trans` turns each 8 x 8 piece as it loads it.
template <int HDK, int HDV>
__global__ void __launch_bounds__(128)
scalar_chunk_state_kernel(const bf16* __restrict__ k, const bf16* __restrict__ v, int in_stride, const float* __restrict__ log_decay,
                          const float* __restrict__ in_scale, const int* __restrict__ seq_start, float* __restrict__ scratch,
                          float* __restrict__ chunk_decay, int max_chunks, int H, int QH, int dim, int vdim) {
  constexpr int KS = HDK + 8, VS = HDV + 8;
  constexpr int MT = HDK / 64;  // 16-row tiles per warp
  extern __shared__ __align__(16) unsigned char sc_smem[];
  bf16* k_s = reinterpret_cast<bf16*>(sc_smem);  // [SC][KS]
  bf16* vh_s = k_s + SC * KS;                    // [SC][VS] the weighted values, rounded
  bf16* vl_s = vh_s + SC * VS;                   // [SC][VS] what the rounding left
  __shared__ float A_s[SC], b_s[SC];
  pdl_trigger();
  pdl_wait();
  const int s = blockIdx.x / H, h = blockIdx.x % H, c = blockIdx.y, qh = h / (H / QH);
  const int t0 = __ldcg(seq_start + s) + c * SC;
  const int n = min(SC, __ldcg(seq_start + s + 1) - t0);
  if (n <= 0) return;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int g = lane >> 2, t4 = lane & 3;
  const bool vec8 = ((dim | vdim | in_stride) & 7) == 0 && ((((uintptr_t)k) | ((uintptr_t)v)) & 15) == 0;
  sc_load_tile<HDK>(k_s, k + (size_t)t0 * in_stride + (size_t)qh * dim, in_stride, n, dim, vec8);
  sc_load_decays(A_s, b_s, log_decay, in_scale, (size_t)t0, n, H, h);
  __syncthreads();
  const float A_end = A_s[n - 1];
  if (tid == 0) chunk_decay[(size_t)blockIdx.x * max_chunks + c] = expf(A_end);
  for (int idx = tid; idx < SC * (HDV / 8); idx += 128) {
    const int i = idx / (HDV / 8), r = 8 * (idx - i * (HDV / 8));
    float f[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) f[e] = 0.f;
    if (i < n) {
      const bf16* src = v + (size_t)(t0 + i) * in_stride + (size_t)h * vdim + r;
      if (vec8) {
        if (r < vdim) bf16x8_to_f32(__ldcg(reinterpret_cast<const uint4*>(src)), f);
      } else {
#pragma unroll
        for (int e = 0; e < 8; ++e)
          if (r + e < vdim) f[e] = __bfloat162float(__ldcg(src + e));
      }
    }
    const float wgt = i < n ? expf(A_end - A_s[i]) * b_s[i] : 0.f;
    bf16 hi[8], lo[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) sc_split(f[e] * wgt, hi[e], lo[e]);
    uint4 ho, lw;
    ho.x = sc_pack(hi[0], hi[1]); ho.y = sc_pack(hi[2], hi[3]); ho.z = sc_pack(hi[4], hi[5]); ho.w = sc_pack(hi[6], hi[7]);
    lw.x = sc_pack(lo[0], lo[1]); lw.y = sc_pack(lo[2], lo[3]); lw.z = sc_pack(lo[4], lo[5]); lw.w = sc_pack(lo[6], lo[7]);
    *reinterpret_cast<uint4*>(vh_s + i * VS + r) = ho;
    *reinterpret_cast<uint4*>(vl_s + i * VS + r) = lw;
  }
  sc_cp_async_wait_all();
  __syncthreads();
  float acc[MT][HDV / 8][4];
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int i = 0; i < HDV / 8; ++i) acc[mt][i][0] = acc[mt][i][1] = acc[mt][i][2] = acc[mt][i][3] = 0.f;
#pragma unroll
  for (int kk = 0; kk < SC / 16; ++kk) {
    uint32_t a[MT][4];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
      sc_ldmatrix_x4_trans(a[mt], k_s + (size_t)(kk * 16 + 8 * (lane >> 4) + (lane & 7)) * KS + warp * (HDK / 4) + mt * 16 + 8 * ((lane >> 3) & 1));
#pragma unroll
    for (int dp = 0; dp < HDV / 16; ++dp) {
      const size_t at = (size_t)(kk * 16 + (lane & 7) + 8 * ((lane >> 3) & 1)) * VS + dp * 16 + 8 * (lane >> 4);
      uint32_t bh[4], bl[4];
      sc_ldmatrix_x4_trans(bh, vh_s + at);
      sc_ldmatrix_x4_trans(bl, vl_s + at);
#pragma unroll
      for (int mt = 0; mt < MT; ++mt) {
        sc_mma(acc[mt][2 * dp], a[mt], bh[0], bh[1]);
        sc_mma(acc[mt][2 * dp + 1], a[mt], bh[2], bh[3]);
        sc_mma(acc[mt][2 * dp], a[mt], bl[0], bl[1]);
        sc_mma(acc[mt][2 * dp + 1], a[mt], bl[2], bl[3]);
      }
    }
  }
  float* u = scratch + ((size_t)blockIdx.x * max_chunks + c) * dim * vdim;
#pragma unroll
  for (int mt = 0; mt < MT; ++mt) {
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int r = warp * (HDK / 4) + mt * 16 + g + 8 * half;
      if (r < dim) {
#pragma unroll
        for (int nn = 0; nn < HDV / 8; ++nn) {
          const int col = nn * 8 + 2 * t4;
          if ((vdim & 1) == 0) {
            if (col < vdim) *reinterpret_cast<float2*>(u + (size_t)r * vdim + col) = make_float2(acc[mt][nn][2 * half], acc[mt][nn][2 * half + 1]);
          } else {
            if (col < vdim) u[(size_t)r * vdim + col] = acc[mt][nn][2 * half];
            if (col + 1 < vdim) u[(size_t)r * vdim + col + 1] = acc[mt][nn][2 * half + 1];
          }
        }
      }
    }
  }
}

// (2): V numbers of a (sequence, head)'s state per thread; leaves in every chunk's place the state BEFORE that chunk.
template <int V>
__global__ void scalar_chunk_scan_kernel(float* __restrict__ state, const int* __restrict__ slot_ids, const int* __restrict__ seq_start,
                                         float* __restrict__ scratch, const float* __restrict__ chunk_decay, int max_chunks, int H, int elems) {
  pdl_trigger();
  pdl_wait();
  const int s = blockIdx.x / H, h = blockIdx.x % H;
  const int e = (blockIdx.y * blockDim.x + threadIdx.x) * V;
  if (e >= elems) return;
  const int len = __ldcg(seq_start + s + 1) - __ldcg(seq_start + s);
  float* st = state + ((size_t)__ldcg(slot_ids + s) * H + h) * elems + e;
  float* u = scratch + (size_t)blockIdx.x * max_chunks * elems + e;
  const float* dec = chunk_decay + (size_t)blockIdx.x * max_chunks;
  const int n_chunks = (len + SC - 1) / SC;
  float S[V];
  if (V == 4) load4_g<float>(st, S);
  else S[0] = __ldcg(st);
  for (int c0 = 0; c0 < n_chunks; c0 += 8) {  // eight chunks' additions are asked for at once, then taken in order
    float add[8][V], d[8];
#pragma unroll
    for (int j = 0; j < 8; ++j)
      if (c0 + j < n_chunks) {
        if (V == 4) load4_g<float>(u + (size_t)(c0 + j) * elems, add[j]);
        else add[j][0] = __ldcg(u + (size_t)(c0 + j) * elems);
        d[j] = __ldcg(dec + c0 + j);
      }
#pragma unroll
    for (int j = 0; j < 8; ++j)
      if (c0 + j < n_chunks) {
        if (V == 4) store4<float>(u + (size_t)(c0 + j) * elems, S);
        else u[(size_t)(c0 + j) * elems] = S[0];
#pragma unroll
        for (int v = 0; v < V; ++v) S[v] = d[j] * S[v] + add[j][v];
      }
  }
  if (V == 4) store4<float>(st, S);
  else st[0] = S[0];
}

// (3): a block of four warps per (sequence, head, chunk), a warp per 16 tokens.  The state before the chunk takes the place of the
// chunk's keys and values in shared memory, one bfloat16 half of it after the other.
template <int HDK, int HDV>
__global__ void __launch_bounds__(128)
scalar_chunk_out_kernel(const bf16* __restrict__ q, const bf16* __restrict__ k, const bf16* __restrict__ v, int in_stride,
                        const float* __restrict__ log_decay, const float* __restrict__ in_scale, const int* __restrict__ seq_start,
                        const float* __restrict__ scratch, int max_chunks, float* __restrict__ out, int out_stride, int H, int QH, int dim,
                        int vdim) {
  constexpr int KS = HDK + 8, VS = HDV + 8;
  static_assert(HDK * VS <= SC * (KS + VS), "a half of the state must fit the keys' and values' place");
  extern __shared__ __align__(16) unsigned char sc_smem[];
  bf16* q_s = reinterpret_cast<bf16*>(sc_smem);  // [SC][KS]
  bf16* k_s = q_s + SC * KS;                     // [SC][KS]
  bf16* v_s = k_s + SC * KS;                     // [SC][VS]
  __shared__ float A_s[SC], b_s[SC];
  pdl_trigger();
  pdl_wait();
  const int s = blockIdx.x / H, h = blockIdx.x % H, c = blockIdx.y, qh = h / (H / QH);
  const int t0 = __ldcg(seq_start + s) + c * SC;
  const int n = min(SC, __ldcg(seq_start + s + 1) - t0);
  if (n <= 0) return;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int g = lane >> 2, t4 = lane & 3;
  const bool vec8 = ((dim | vdim | in_stride) & 7) == 0 && ((((uintptr_t)q) | ((uintptr_t)k) | ((uintptr_t)v)) & 15) == 0;
  sc_load_tile<HDK>(q_s, q + (size_t)t0 * in_stride + (size_t)qh * dim, in_stride, n, dim, vec8);
  sc_load_tile<HDK>(k_s, k + (size_t)t0 * in_stride + (size_t)qh * dim, in_stride, n, dim, vec8);
  sc_load_tile<HDV>(v_s, v + (size_t)t0 * in_stride + (size_t)h * vdim, in_stride, n, vdim, vec8);
  sc_load_decays(A_s, b_s, log_decay, in_scale, (size_t)t0, n, H, h);
  sc_cp_async_wait_all();
  __syncthreads();

  // ---- the chunk's scores for this warp's 16 tokens against its 64 tokens
  float s_acc[SC / 8][4];
#pragma unroll
  for (int i = 0; i < SC / 8; ++i) s_acc[i][0] = s_acc[i][1] = s_acc[i][2] = s_acc[i][3] = 0.f;
  const bf16* qa = q_s + (size_t)(warp * 16 + (lane & 7) + 8 * ((lane >> 3) & 1)) * KS + 8 * (lane >> 4);
#pragma unroll
  for (int kk = 0; kk < HDK / 16; ++kk) {
    uint32_t a[4];
    sc_ldmatrix_x4(a, qa + kk * 16);
#pragma unroll
    for (int np = 0; np < SC / 16; ++np) {
      if (np <= warp) {  // (later tokens are masked anyway)
        uint32_t b[4];
        sc_ldmatrix_x4(b, k_s + (size_t)(np * 16 + (lane & 7) + 8 * (lane >> 4)) * KS + kk * 16 + 8 * ((lane >> 3) & 1));
        sc_mma(s_acc[2 * np], a, b[0], b[1]);
        sc_mma(s_acc[2 * np + 1], a, b[2], b[3]);
      }
    }
  }
  // ---- decay, input strength and mask in 32-bit; each score as two bfloat16 numbers, laid out as the next product's A operand
  float intra[HDV / 8][4];
#pragma unroll
  for (int i = 0; i < HDV / 8; ++i) intra[i][0] = intra[i][1] = intra[i][2] = intra[i][3] = 0.f;
  const int row[2] = {warp * 16 + g, warp * 16 + g + 8};
  const float A_row[2] = {A_s[row[0]], A_s[row[1]]};
#pragma unroll
  for (int kk = 0; kk < SC / 16; ++kk) {
    if (kk > warp) continue;
    uint32_t p_hi[4], p_lo[4];
#pragma unroll
    for (int half = 0; half < 2; ++half) {
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        bf16 hi[2], lo[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int j = kk * 16 + half * 8 + 2 * t4 + e;
          const float p = j <= row[r] ? s_acc[2 * kk + half][2 * r + e] * expf(A_row[r] - A_s[j]) * b_s[j] : 0.f;
          sc_split(p, hi[e], lo[e]);
        }
        p_hi[2 * half + r] = sc_pack(hi[0], hi[1]);
        p_lo[2 * half + r] = sc_pack(lo[0], lo[1]);
      }
    }
#pragma unroll
    for (int dp = 0; dp < HDV / 16; ++dp) {
      uint32_t b[4];
      sc_ldmatrix_x4_trans(b, v_s + (size_t)(kk * 16 + (lane & 7) + 8 * ((lane >> 3) & 1)) * VS + dp * 16 + 8 * (lane >> 4));
      sc_mma(intra[2 * dp], p_hi, b[0], b[1]);
      sc_mma(intra[2 * dp + 1], p_hi, b[2], b[3]);
      sc_mma(intra[2 * dp], p_lo, b[0], b[1]);
      sc_mma(intra[2 * dp + 1], p_lo, b[2], b[3]);
    }
  }
  // ---- the queries against the state before the chunk
  float inter[HDV / 8][4];
#pragma unroll
  for (int i = 0; i < HDV / 8; ++i) inter[i][0] = inter[i][1] = inter[i][2] = inter[i][3] = 0.f;
  const float* sp = scratch + ((size_t)blockIdx.x * max_chunks + c) * dim * vdim;
  bf16* st_s = k_s;  // [HDK][VS]
  for (int pass = 0; pass < 2; ++pass) {
    __syncthreads();  // the keys and values (or the first half) are no longer read
    if ((vdim & 3) == 0) {  // four numbers a load, four loads in flight
#pragma unroll 4
      for (int idx = tid; idx < HDK * (HDV / 4); idx += 128) {
        const int r = idx / (HDV / 4), cc = 4 * (idx - r * (HDV / 4));
        float4 t = make_float4(0.f, 0.f, 0.f, 0.f);
        if (r < dim && cc < vdim) t = __ldcg(reinterpret_cast<const float4*>(sp + (size_t)r * vdim + cc));
        const float f[4] = {t.x, t.y, t.z, t.w};
        bf16 o[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          bf16 hi, lo;
          sc_split(f[e], hi, lo);
          o[e] = pass == 0 ? hi : lo;
        }
        uint2 raw;
        raw.x = sc_pack(o[0], o[1]);
        raw.y = sc_pack(o[2], o[3]);
        *reinterpret_cast<uint2*>(st_s + r * VS + cc) = raw;
      }
    } else {
      for (int idx = tid; idx < HDK * HDV; idx += 128) {
        const int r = idx / HDV, cc = idx - r * HDV;
        bf16 hi = __float2bfloat16_rn(0.f), lo = hi;
        if (r < dim && cc < vdim) sc_split(__ldcg(sp + (size_t)r * vdim + cc), hi, lo);
        st_s[r * VS + cc] = pass == 0 ? hi : lo;
      }
    }
    __syncthreads();
#pragma unroll
    for (int kk = 0; kk < HDK / 16; ++kk) {
      uint32_t a[4];
      sc_ldmatrix_x4(a, qa + kk * 16);
#pragma unroll
      for (int dp = 0; dp < HDV / 16; ++dp) {
        uint32_t b[4];
        sc_ldmatrix_x4_trans(b, st_s + (size_t)(kk * 16 + (lane & 7) + 8 * ((lane >> 3) & 1)) * VS + dp * 16 + 8 * (lane >> 4));
        sc_mma(inter[2 * dp], a, b[0], b[1]);
        sc_mma(inter[2 * dp + 1], a, b[2], b[3]);
      }
    }
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int i = row[r];
    if (i < n) {
      const float w = expf(A_row[r]);
      float* o = out + (size_t)(t0 + i) * out_stride + (size_t)h * vdim;
#pragma unroll
      for (int nn = 0; nn < HDV / 8; ++nn) {
        const int d = nn * 8 + 2 * t4;
        const float o0 = intra[nn][2 * r] + w * inter[nn][2 * r], o1 = intra[nn][2 * r + 1] + w * inter[nn][2 * r + 1];
        if ((vdim & 1) == 0 && (out_stride & 1) == 0) {
          if (d < vdim) *reinterpret_cast<float2*>(o + d) = make_float2(o0, o1);
        } else {
          if (d < vdim) o[d] = o0;
          if (d + 1 < vdim) o[d + 1] = o1;
        }
      }
    }
  }
}

RL_API int rl_scalar_decay_chunked_takes(int dim, int vdim) { return dim > 0 && vdim > 0 && dim <= 128 && vdim <= 128; }

RL_API long long rl_scalar_decay_chunked_scratch_floats(int n_seqs, int max_q_len, int H, int dim, int vdim) {
  return (long long)n_seqs * H * ((max_q_len + SC - 1) / SC) * ((long long)dim * vdim + 1);
}

template <int HDK, int HDV>
static int launch_scalar_chunked(const bf16* q, const bf16* k, const bf16* v, int in_stride, const float* log_decay, const float* in_scale,
                                 float* state, const int* slot_ids, const int* seq_start, float* scratch, float* chunk_decay, float* out,
                                 int out_stride, int n_seqs, int max_chunks, int H, int QH, int dim, int vdim, cudaStream_t stream) {
  const size_t smem1 = (size_t)SC * ((HDK + 8) + 2 * (HDV + 8)) * sizeof(bf16), smem3 = (size_t)SC * (2 * (HDK + 8) + (HDV + 8)) * sizeof(bf16);
  if ((smem1 > 48 * 1024 && cudaFuncSetAttribute(scalar_chunk_state_kernel<HDK, HDV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem1) != cudaSuccess) ||
      (smem3 > 48 * 1024 && cudaFuncSetAttribute(scalar_chunk_out_kernel<HDK, HDV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem3) != cudaSuccess))
    RL_REFUSE(5, "scalar_decay_chunked: %zu bytes of shared memory refused", smem3);
  const int elems = dim * vdim;
  dim3 grid(n_seqs * H, max_chunks);
  RL_LAUNCH_CHECK(rl_launch(scalar_chunk_state_kernel<HDK, HDV>, grid, 128, smem1, stream, k, v, in_stride, log_decay, in_scale, seq_start, scratch,
                            chunk_decay, max_chunks, H, QH, dim, vdim));
  if (elems % 4 == 0) {
    dim3 grid2(n_seqs * H, (elems / 4 + 127) / 128);
    RL_LAUNCH_CHECK(rl_launch(scalar_chunk_scan_kernel<4>, grid2, 128, 0, stream, state, slot_ids, seq_start, scratch, (const float*)chunk_decay,
                              max_chunks, H, elems));
  } else {
    dim3 grid2(n_seqs * H, (elems + 127) / 128);
    RL_LAUNCH_CHECK(rl_launch(scalar_chunk_scan_kernel<1>, grid2, 128, 0, stream, state, slot_ids, seq_start, scratch, (const float*)chunk_decay,
                              max_chunks, H, elems));
  }
  RL_LAUNCH_CHECK(rl_launch(scalar_chunk_out_kernel<HDK, HDV>, grid, 128, smem3, stream, q, k, v, in_stride, log_decay, in_scale, seq_start,
                            (const float*)scratch, max_chunks, out, out_stride, H, QH, dim, vdim));
  return 0;
}

// q, k: [T, >= QH dim] rows, v: [T, >= H vdim] rows of one stride (bfloat16); log_decay: float32 [T, H]; in_scale: float32 [T, H] or null;
// state: float32 [slots, H, dim, vdim]; scratch: rl_scalar_decay_chunked_scratch_floats(...) floats, 16-byte aligned; out: float32 [T, H vdim].
RL_API int rl_scalar_decay_chunked(const void* q, const void* k, const void* v, int in_stride, const float* log_decay, const float* in_scale,
                                   float* state, const int* slot_ids, const int* seq_start, float* scratch, float* out, int out_stride,
                                   int n_seqs, int max_q_len, int H, int QH, int dim, int vdim, cudaStream_t stream) {
  if (n_seqs <= 0 || max_q_len <= 0 || H <= 0 || QH <= 0 || H % QH || !scratch || !log_decay)
    RL_REFUSE(1, "scalar_decay_chunked: S=%d max_q=%d H=%d on %d", n_seqs, max_q_len, H, QH);
  if (!rl_scalar_decay_chunked_takes(dim, vdim)) RL_REFUSE(2, "scalar_decay_chunked: sizes %d x %d exceed 128", dim, vdim);
  const int max_chunks = (max_q_len + SC - 1) / SC;
  if (max_chunks > 65535 || (long long)n_seqs * H > 0x7fffffffLL) RL_REFUSE(3, "scalar_decay_chunked: %d chunks exceed the grid", max_chunks);
  if (((uintptr_t)scratch | (uintptr_t)state) & 15) RL_REFUSE(4, "scalar_decay_chunked: scratch and state must be 16-byte aligned");
  float* chunk_decay = scratch + (long long)n_seqs * H * max_chunks * dim * vdim;
#define RL_SDC(K, V)                                                                                                                      \
  return launch_scalar_chunked<K, V>((const bf16*)q, (const bf16*)k, (const bf16*)v, in_stride, log_decay, in_scale, state, slot_ids, seq_start, \
                                     scratch, chunk_decay, out, out_stride, n_seqs, max_chunks, H, QH, dim, vdim, stream)
  if (dim <= 64 && vdim <= 64) RL_SDC(64, 64);
  if (dim <= 64) RL_SDC(64, 128);
  if (vdim <= 64) RL_SDC(128, 64);
  RL_SDC(128, 128);
#undef RL_SDC
}
