// Grouped-query softmax attention with the options that a plain causal attention lacks, over the paged cache:
//
//   - keys of `kdim` and values of `vdim` numbers per head (the two may differ),
//   - biases on the projected q, k and v,
//   - an RMS norm of every q head and every k head over the head's numbers (one weight row for all q heads, one for all k
//     heads), after the biases and before the rotation; or one norm over all q heads together and one over all k heads together
//     (`norm_whole`), with a weight for every column,
//   - a temperature of the queries that grows with the position: q at position p is multiplied by
//     1 + temp_coef ln(floor((p + 1) / temp_every) + 1), after the norm,
//   - values that are the keys as projected, before their norm (`v_from_k`; the rows then hold no values),
//   - a learned bias on every score by head and distance (`rl_distance_bias`), added after scale, mixing and cap,
//   - a rotation of the first `rot` dimensions of q and k in either pair layout, cosines and sines
//     multiplied by a constant `magnitude`,
//   - a score scale given by the caller,
//   - a mixing of the heads' scaled scores before the softmax, s_h <- sum_g mix[h][g] s_g,
//   - a window (query at position p sees keys j with 0 <= p - j < window),
//   - chunks (query at position p sees keys j <= p of its own chunk only, floor(j / chunk) = floor(p / chunk), positions
//     counted from the start of the sequence),
//   - a cap on the scores, s <- cap tanh(s / cap), after the scale (and the mixing),
//   - a sink per head: exp(sink_h) joins the softmax's denominator and nothing else,
//   - a gate on the result, out *= sigmoid(gate), and a constant factor `out_scale`,
//   - two maps per head (`maps` 2): query heads 2h and 2h + 1 are the two halves of head h's query row of `kdim` numbers and meet
//     the same halves of the keys, kdim / 2 numbers each; `map_combine` makes o_h = a_2h - lambda a_(2h+1) of their results,
//     divided by its root mean square over the head's values, times a constant.
//
// Two kernels.  `qkv_prep` adds the biases, rotates q in place and writes the rotated k and v to the token's
// place in its sequence's pages; with `v_src` the value that is stored is (1 - lambda) v + lambda v_src[t] (values that an
// earlier layer projected for the same token; lambda a learned number on the device), computed in 32-bit.  `attn_ext` is the attention itself, for prompts and for decoding, in both
// element types: one warp per (token, head), the keys taken 32 at a time counted from the first key the
// query may see, online softmax, every sum in 32-bit and in a fixed order, so a result's bits depend neither
// on how its sequence was cut into steps nor on what else is in the batch.  With a mixing matrix the warps
// of all heads of a token share a block and exchange their scores of a group of keys through shared memory.
//
// Cache layout of one layer: k_pages[page][kv head][slot in page][kdim], v_pages[...][vdim]; the page of
// position p of batch sequence s is block_table[s][p / page_size].
#include "common.cuh"

RL_DEFINE_ERROR_TEXT()

// ---------------------------------------------------------------- biases, norms, rotation, cache write
__device__ __forceinline__ float qp_temperature(int pos, float coef, int every) {
  return 1.0f + coef * logf((float)((pos + 1) / every) + 1.0f);
}

// One block per token.  row = qkv[t]: H query heads of kdim, then K key heads of kdim, then K value heads of vdim.
template <typename T>
__global__ void qkv_prep_kernel(T* __restrict__ qkv, int row_stride, const float* __restrict__ bias,
                                const int* __restrict__ tok_pos, const int* __restrict__ tok_seq,
                                const int* __restrict__ block_table, int table_width, T* __restrict__ k_pages,
                                T* __restrict__ v_pages, const float* __restrict__ inv_freq, float magnitude,
                                const float* __restrict__ q_norm, const float* __restrict__ k_norm, float norm_eps, int H, int K,
                                int kdim, int vdim, int rot, int interleaved, int page_size, const T* __restrict__ v_src,
                                int v_src_stride, const float* __restrict__ v_lambda, int norm_whole, int v_from_k, float temp_coef,
                                int temp_every) {
  extern __shared__ float trig[];  // cos[rot/2], sin[rot/2], both times the magnitude; then 1 / rms of every q and k head
  const int t = blockIdx.x;
  const int pos = tok_pos[t];
  const int half = rot >> 1;
  float* cs = trig;
  float* sn = trig + half;
  for (int j = threadIdx.x; j < half; j += blockDim.x) {
    const float a = (float)pos * inv_freq[j];
    float s, c;
    sincosf(a, &s, &c);
    cs[j] = c * magnitude;
    sn[j] = s * magnitude;
  }
  T* row = qkv + (size_t)t * row_stride;
  float* inv_rms = trig + rot;
  if (q_norm != nullptr || k_norm != nullptr) {  // a warp per head, the sums in lane order and then by the warp's tree
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
    for (int h = warp; h < H + K; h += nwarps) {
      const T* head = row + (size_t)h * kdim;
      const float* b = bias ? bias + (size_t)h * kdim : nullptr;
      float ss = 0.f;
      for (int i = lane; i < kdim; i += 32) {
        const float x = to_f32(head[i]) + (b ? b[i] : 0.f);
        ss += x * x;
      }
      ss = warp_sum(ss);
      if (lane == 0) inv_rms[h] = norm_whole ? ss : ((h < H ? q_norm : k_norm) != nullptr) ? 1.0f / sqrtf(ss / (float)kdim + norm_eps) : 1.f;
    }
    if (norm_whole) {  // one thread adds the q heads' sums in their order, another the k heads'
      __syncthreads();
      if (threadIdx.x < 2) {
        const int lo = threadIdx.x == 0 ? 0 : H, hi = threadIdx.x == 0 ? H : H + K;
        float ss = 0.f;
        for (int h = lo; h < hi; ++h) ss += inv_rms[h];
        const float inv = ((threadIdx.x == 0 ? q_norm : k_norm) != nullptr) ? 1.0f / sqrtf(ss / (float)((hi - lo) * kdim) + norm_eps) : 1.f;
        for (int h = lo; h < hi; ++h) inv_rms[h] = inv;
      }
    }
  }
  __syncthreads();
  const float temp = temp_every > 0 ? qp_temperature(pos, temp_coef, temp_every) : 1.f;
  const int page = K > 0 ? block_table[(size_t)tok_seq[t] * table_width + pos / page_size] : 0;
  const int in_page = pos % page_size;
  // q and k heads: one thread per rotated pair or per unrotated value
  const int per_head = half + (kdim - rot);
  for (int idx = threadIdx.x; idx < (H + K) * per_head; idx += blockDim.x) {
    const int h = idx / per_head, e = idx - h * per_head;
    T* head = row + (size_t)h * kdim;
    const float* b = bias ? bias + (size_t)h * kdim : nullptr;
    const float* nw = h < H ? q_norm : k_norm;
    if (nw && norm_whole) nw += (size_t)(h < H ? h : h - H) * kdim;
    const float inv = nw ? inv_rms[h] : 1.f;
    const float by = h < H ? temp : 1.f;
    T* dst = h < H ? head : k_pages + (((size_t)page * K + (h - H)) * page_size + in_page) * kdim;
    if (e < half) {
      const int i0 = interleaved ? 2 * e : e;
      const int i1 = interleaved ? 2 * e + 1 : e + half;
      float x0 = to_f32(head[i0]) + (b ? b[i0] : 0.f);
      float x1 = to_f32(head[i1]) + (b ? b[i1] : 0.f);
      if (nw) {
        x0 = x0 * inv * nw[i0];
        x1 = x1 * inv * nw[i1];
      }
      x0 *= by;
      x1 *= by;
      dst[i0] = from_f32<T>(x0 * cs[e] - x1 * sn[e]);
      dst[i1] = from_f32<T>(x1 * cs[e] + x0 * sn[e]);
    } else {
      const int i = rot + (e - half);
      float x = to_f32(head[i]) + (b ? b[i] : 0.f);
      if (nw) x = x * inv * nw[i];
      dst[i] = from_f32<T>(x * by);
    }
  }
  const T* vrow = row + (size_t)(v_from_k ? H : H + K) * kdim;
  const float* vb = bias ? bias + (size_t)(H + K) * kdim : nullptr;
  const float lam = v_src ? v_lambda[0] : 0.f;
  const T* vs = v_src ? v_src + (size_t)t * v_src_stride : nullptr;
  for (int idx = threadIdx.x; idx < K * vdim; idx += blockDim.x) {
    const int h = idx / vdim, i = idx - h * vdim;
    float v = to_f32(vrow[idx]) + (vb ? vb[idx] : 0.f);
    if (vs) v = (1.0f - lam) * v + lam * to_f32(vs[idx]);
    v_pages[(((size_t)page * K + h) * page_size + in_page) * vdim + i] = from_f32<T>(v);
  }
}

// The same for bfloat16 rows whose sizes are multiples of 8 and whose pairs are neighbours (or that are not rotated at all): a
// thread takes 8 numbers of a head with one 16-byte load, the kdim / 8 threads of a head (in a run of a power of two of lanes, the
// rest of which idle) add their squares up by shuffles, a norm over all heads by a pass over the row before that, and the four pairs a thread holds are rotated in its registers; q goes back and k, v go to their pages with 16-byte stores.
__device__ __forceinline__ void qp_unpack8(const uint4& raw, float* x) {
  const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const float2 f = __bfloat1622float2(p[j]);
    x[2 * j] = f.x;
    x[2 * j + 1] = f.y;
  }
}

__device__ __forceinline__ uint4 qp_pack8(const float* x) {
  uint4 raw;
  __nv_bfloat162* p = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
  for (int j = 0; j < 4; ++j) p[j] = __floats2bfloat162_rn(x[2 * j], x[2 * j + 1]);
  return raw;
}

__device__ __forceinline__ void qp_add8(float* x, const float* b) {
  const float4 b0 = *reinterpret_cast<const float4*>(b), b1 = *reinterpret_cast<const float4*>(b + 4);
  x[0] += b0.x; x[1] += b0.y; x[2] += b0.z; x[3] += b0.w;
  x[4] += b1.x; x[5] += b1.y; x[6] += b1.z; x[7] += b1.w;
}

__global__ void __launch_bounds__(256)
qkv_prep_rows8_kernel(bf16* __restrict__ qkv, int row_stride, const float* __restrict__ bias, const int* __restrict__ tok_pos,
                      const int* __restrict__ tok_seq, const int* __restrict__ block_table, int table_width,
                      bf16* __restrict__ k_pages, bf16* __restrict__ v_pages, const float* __restrict__ inv_freq, float magnitude,
                      const float* __restrict__ q_norm, const float* __restrict__ k_norm, float norm_eps, int H, int K, int kdim,
                      int vdim, int rot, int page_size, const bf16* __restrict__ v_src, int v_src_stride,
                      const float* __restrict__ v_lambda, int g, int norm_whole, int v_from_k, float temp_coef, int temp_every) {
  __shared__ float red[32];
  extern __shared__ float trig[];  // cos[rot/2], sin[rot/2], both times the magnitude
  const int t = blockIdx.x;
  const int pos = tok_pos[t];
  const int half = rot >> 1;
  float* cs = trig;
  float* sn = trig + half;
  for (int j = threadIdx.x; j < half; j += blockDim.x) {
    const float a = (float)pos * inv_freq[j];
    float s, c;
    sincosf(a, &s, &c);
    cs[j] = c * magnitude;
    sn[j] = s * magnitude;
  }
  __syncthreads();
  bf16* row = qkv + (size_t)t * row_stride;
  const int page = K > 0 ? block_table[(size_t)tok_seq[t] * table_width + pos / page_size] : 0;
  const int in_page = pos % page_size;
  const int total = (H + K) * g;  // g: lanes to a head, the power of two from kdim / 8 on, up to 32
  const bool normed = (q_norm != nullptr || k_norm != nullptr) && !norm_whole;
  const float temp = temp_every > 0 ? qp_temperature(pos, temp_coef, temp_every) : 1.f;
  float whole_q = 1.f, whole_k = 1.f;  // 1 / rms of all q heads, of all k heads
  if (norm_whole) {
    float own_q = 0.f, own_k = 0.f;
    const int nq = (H * kdim) >> 3, n8 = ((H + K) * kdim) >> 3;
    for (int c = threadIdx.x; c < n8; c += blockDim.x) {
      float x[8], sum = 0.f;
      qp_unpack8(*reinterpret_cast<const uint4*>(row + (size_t)c * 8), x);
      if (bias) qp_add8(x, bias + (size_t)c * 8);
#pragma unroll
      for (int j = 0; j < 8; ++j) sum += x[j] * x[j];
      if (c < nq) own_q += sum;
      else own_k += sum;
    }
    const float sq = block_sum(own_q, red), sk = block_sum(own_k, red);
    if (q_norm) whole_q = 1.0f / sqrtf(sq / (float)(H * kdim) + norm_eps);
    if (k_norm && K > 0) whole_k = 1.0f / sqrtf(sk / (float)(K * kdim) + norm_eps);
  }
  for (int base = 0; base < total; base += blockDim.x) {
    const int idx = base + threadIdx.x;
    const bool valid = idx < total && (idx & (g - 1)) * 8 < kdim;  // (every lane takes part in the shuffles)
    const int h = valid ? idx / g : 0, i0 = valid ? (idx & (g - 1)) * 8 : 0;
    float x[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    if (valid) {
      qp_unpack8(*reinterpret_cast<const uint4*>(row + (size_t)h * kdim + i0), x);
      if (bias) qp_add8(x, bias + (size_t)h * kdim + i0);
    }
    if (normed) {
      float ss = 0.f;
#pragma unroll
      for (int j = 0; j < 8; ++j) ss += x[j] * x[j];
      for (int o = g >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      const float* nw = h < H ? q_norm : k_norm;
      if (valid && nw) {
        const float inv = 1.0f / sqrtf(ss / (float)kdim + norm_eps);
        const float4 w0 = *reinterpret_cast<const float4*>(nw + i0), w1 = *reinterpret_cast<const float4*>(nw + i0 + 4);
        x[0] = x[0] * inv * w0.x; x[1] = x[1] * inv * w0.y; x[2] = x[2] * inv * w0.z; x[3] = x[3] * inv * w0.w;
        x[4] = x[4] * inv * w1.x; x[5] = x[5] * inv * w1.y; x[6] = x[6] * inv * w1.z; x[7] = x[7] * inv * w1.w;
      }
    }
    if (norm_whole && valid) {
      const float* nw = h < H ? (q_norm ? q_norm + (size_t)h * kdim + i0 : nullptr) : (k_norm ? k_norm + (size_t)(h - H) * kdim + i0 : nullptr);
      if (nw) {
        const float inv = h < H ? whole_q : whole_k;
        const float4 w0 = *reinterpret_cast<const float4*>(nw), w1 = *reinterpret_cast<const float4*>(nw + 4);
        x[0] = x[0] * inv * w0.x; x[1] = x[1] * inv * w0.y; x[2] = x[2] * inv * w0.z; x[3] = x[3] * inv * w0.w;
        x[4] = x[4] * inv * w1.x; x[5] = x[5] * inv * w1.y; x[6] = x[6] * inv * w1.z; x[7] = x[7] * inv * w1.w;
      }
    }
    if (temp_every > 0 && h < H) {
#pragma unroll
      for (int j = 0; j < 8; ++j) x[j] *= temp;
    }
    if (valid) {
      if (i0 < rot) {
#pragma unroll
        for (int p = 0; p < 4; ++p) {
          const float c = cs[(i0 >> 1) + p], sv = sn[(i0 >> 1) + p];
          const float a = x[2 * p], b = x[2 * p + 1];
          x[2 * p] = a * c - b * sv;
          x[2 * p + 1] = b * c + a * sv;
        }
      }
      bf16* dst = h < H ? row + (size_t)h * kdim + i0 : k_pages + (((size_t)page * K + (h - H)) * page_size + in_page) * kdim + i0;
      *reinterpret_cast<uint4*>(dst) = qp_pack8(x);
    }
  }
  const bf16* vrow = row + (size_t)(v_from_k ? H : H + K) * kdim;
  const float* vb = bias ? bias + (size_t)(H + K) * kdim : nullptr;
  const int gv = vdim >> 3;
  for (int idx = threadIdx.x; idx < K * gv; idx += blockDim.x) {
    const int h = idx / gv, i = (idx - h * gv) * 8;
    uint4 raw = *reinterpret_cast<const uint4*>(vrow + (size_t)h * vdim + i);
    if (vb || v_src) {
      float x[8];
      qp_unpack8(raw, x);
      if (vb) qp_add8(x, vb + (size_t)h * vdim + i);
      if (v_src) {
        const float lam = v_lambda[0];
        float y[8];
        qp_unpack8(*reinterpret_cast<const uint4*>(v_src + (size_t)t * v_src_stride + (size_t)h * vdim + i), y);
#pragma unroll
        for (int j = 0; j < 8; ++j) x[j] = (1.0f - lam) * x[j] + lam * y[j];
      }
      raw = qp_pack8(x);
    }
    *reinterpret_cast<uint4*>(v_pages + (((size_t)page * K + h) * page_size + in_page) * vdim + i) = raw;
  }
}

RL_API int rl_qkv_prep(void* qkv, int dtype, int row_stride, const float* bias, const int* tok_pos, const int* tok_seq,
                       const int* block_table, int table_width, void* k_pages, void* v_pages, const float* inv_freq,
                       float magnitude, const float* q_norm, const float* k_norm, float norm_eps, int n_tokens, int H, int K, int kdim,
                       int vdim, int rot, int interleaved, int page_size, const void* v_src, int v_src_stride, const float* v_lambda,
                       int norm_whole, int v_from_k, float temp_coef, int temp_every, cudaStream_t stream) {
  if (v_from_k && (vdim != kdim || v_src != nullptr || bias != nullptr)) RL_REFUSE(9, "qkv_prep: values that are the keys are as long (%d, %d), with no bias and no mixing", kdim, vdim);
  if (temp_every < 0) RL_REFUSE(10, "qkv_prep: temperature steps of %d positions", temp_every);
  if (v_src != nullptr && (v_lambda == nullptr || v_src_stride < K * vdim)) RL_REFUSE(8, "qkv_prep: values to mix in need a factor and rows of %d numbers", K * vdim);
  if (n_tokens <= 0 || H < 0 || K < 0 || H + K <= 0 || kdim <= 0 || vdim <= 0 || page_size <= 0 || table_width <= 0)  // (H 0: rows of keys and values only; K 0: of queries)
    RL_REFUSE(1, "qkv_prep: T=%d H=%d K=%d kdim=%d vdim=%d page=%d", n_tokens, H, K, kdim, vdim, page_size);
  if (rot < 0 || rot > kdim || (rot & 1)) RL_REFUSE(2, "qkv_prep: %d rotated dimensions do not fit a head of %d", rot, kdim);
  if (row_stride < (H + K) * kdim + (v_from_k ? 0 : K * vdim)) RL_REFUSE(3, "qkv_prep: row stride %d too small", row_stride);
  if (rot > 0 && inv_freq == nullptr) RL_REFUSE(4, "qkv_prep: no frequency table");
  if (!tok_pos || !tok_seq || (K > 0 && (!block_table || !k_pages || !v_pages))) RL_REFUSE(5, "qkv_prep: pages, page table and positions are needed");
  const size_t smem = ((size_t)rot + H + K) * sizeof(float);
  if (smem > 48 * 1024) RL_REFUSE(6, "qkv_prep: rotary size %d or %d heads too large", rot, H + K);
  const int threads = 256;
  int g = 1;
  while (g * 8 < kdim) g *= 2;
  const uintptr_t bits = (uintptr_t)qkv | (uintptr_t)k_pages | (uintptr_t)v_pages | (uintptr_t)bias | (uintptr_t)q_norm | (uintptr_t)k_norm |
                         (uintptr_t)v_src;
  if (dtype == RL_BF16 && (interleaved || rot == 0) && kdim % 8 == 0 && vdim % 8 == 0 && rot % 8 == 0 && row_stride % 8 == 0 &&
      v_src_stride % 8 == 0 && g <= 32 && (bits & 15) == 0)
    qkv_prep_rows8_kernel<<<n_tokens, threads, (size_t)rot * sizeof(float), stream>>>(
        (bf16*)qkv, row_stride, bias, tok_pos, tok_seq, block_table, table_width, (bf16*)k_pages, (bf16*)v_pages, inv_freq, magnitude,
        q_norm, k_norm, norm_eps, H, K, kdim, vdim, rot, page_size, (const bf16*)v_src, v_src_stride, v_lambda,
        g, norm_whole, v_from_k, temp_coef, temp_every);
  else if (dtype == RL_BF16)
    qkv_prep_kernel<bf16><<<n_tokens, threads, smem, stream>>>((bf16*)qkv, row_stride, bias, tok_pos, tok_seq, block_table, table_width,
                                                               (bf16*)k_pages, (bf16*)v_pages, inv_freq, magnitude, q_norm, k_norm, norm_eps, H, K,
                                                               kdim, vdim, rot, interleaved, page_size, (const bf16*)v_src, v_src_stride, v_lambda,
                                                               norm_whole, v_from_k, temp_coef, temp_every);
  else if (dtype == RL_F32)
    qkv_prep_kernel<float><<<n_tokens, threads, smem, stream>>>((float*)qkv, row_stride, bias, tok_pos, tok_seq, block_table, table_width,
                                                                (float*)k_pages, (float*)v_pages, inv_freq, magnitude, q_norm, k_norm, norm_eps, H, K,
                                                                kdim, vdim, rot, interleaved, page_size, (const float*)v_src, v_src_stride, v_lambda,
                                                                norm_whole, v_from_k, temp_coef, temp_every);
  else
    RL_REFUSE(7, "qkv_prep: unknown dtype %d", dtype);
  RL_LAUNCH_RESULT();
}

// ---------------------------------------------------------------- the attention
#define EXT_MAX_V_PER_LANE 8  // value sizes up to 256

// blockDim = (32, HB): HB = 1 and grid (T, H) without a mixing matrix; HB = H and grid (T, 1) with one.
template <typename T>
__global__ void attn_ext_kernel(const T* __restrict__ q, int q_stride, const T* __restrict__ k_pages, const T* __restrict__ v_pages,
                                const int* __restrict__ block_table, int table_width, const int* __restrict__ tok_seq,
                                const int* __restrict__ tok_pos, const float* __restrict__ sink, const float* __restrict__ mix,
                                const T* __restrict__ gate, int gate_stride, float out_scale, T* __restrict__ out, int out_stride,
                                int H, int K, int kdim, int vdim, int page_size, int window, float scale, int chunk, float softcap, int maps,
                                const float* __restrict__ bias, int bias_len) {
  extern __shared__ float smem[];  // q of the block's heads [HB][kdim], then (with mix) scores [HB][32]
  const int lane = threadIdx.x;
  const int hb = threadIdx.y, HB = blockDim.y;
  const int t = blockIdx.x, h = blockIdx.y * HB + hb;
  const int kh = h / (H / K);
  const int pos = tok_pos[t];
  const int* table = block_table + (size_t)tok_seq[t] * table_width;
  float* q_s = smem + (size_t)hb * kdim;
  float* sc = smem + (size_t)HB * kdim;
  const T* qh = q + (size_t)t * q_stride + (size_t)(h / maps) * kdim;
  const int i_lo = (h % maps) * (kdim / maps), i_hi = i_lo + kdim / maps;  // the numbers of query and key that make this head's score
  for (int i = i_lo + lane; i < i_hi; i += 32) q_s[i] = to_f32(qh[i]);
  __syncwarp();

  int first = (window != 0 && pos + 1 > window) ? pos + 1 - window : 0;
  if (chunk != 0) first = max(first, pos - pos % chunk);
  float m = -INFINITY, l = 0.f;
  if (sink != nullptr) {  // the sink is a key without a value whose score is sink[h]
    m = sink[h];
    l = 1.f;
  }
  float acc[EXT_MAX_V_PER_LANE];
#pragma unroll
  for (int i = 0; i < EXT_MAX_V_PER_LANE; ++i) acc[i] = 0.f;

  for (int base = first; base <= pos; base += 32) {
    const int key = base + lane;
    const bool valid = key <= pos;
    float s = 0.f;
    if (valid) {
      const int page = table[key / page_size];
      const T* kr = k_pages + (((size_t)page * K + kh) * page_size + key % page_size) * kdim;
      float dot = 0.f;
      for (int i = i_lo; i < i_hi; ++i) dot += q_s[i] * to_f32(kr[i]);
      s = dot * scale;
    }
    if (mix != nullptr) {
      __syncthreads();  // the scores of the group before have been read
      sc[hb * 32 + lane] = s;
      __syncthreads();
      float mixed = 0.f;
      for (int g = 0; g < HB; ++g) mixed += mix[h * HB + g] * sc[g * 32 + lane];
      s = mixed;
    }
    if (softcap > 0.f) s = softcap * tanhf(s / softcap);
    if (bias != nullptr) s += rl_distance_bias(bias + (size_t)h * bias_len, bias_len, pos - key);
    if (!valid) s = -INFINITY;
    const float m_new = fmaxf(m, warp_max(s));  // finite: the group holds at least key `base`
    const float alpha = expf(m - m_new);        // 0 for the first group without a sink, where m is -inf
    const float p = valid ? expf(s - m_new) : 0.f;
    l = l * alpha + warp_sum(p);
#pragma unroll
    for (int i = 0; i < EXT_MAX_V_PER_LANE; ++i) acc[i] *= alpha;
    const int count = min(32, pos - base + 1);
    for (int j = 0; j < count; ++j) {
      const float pj = __shfl_sync(0xffffffffu, p, j);
      const int kj = base + j;
      const int page = table[kj / page_size];
      const T* vr = v_pages + (((size_t)page * K + kh) * page_size + kj % page_size) * vdim;
#pragma unroll
      for (int i = 0; i < EXT_MAX_V_PER_LANE; ++i) {
        const int dim = lane + 32 * i;
        if (dim < vdim) acc[i] += pj * to_f32(vr[dim]);
      }
    }
    m = m_new;
  }
  const float inv = 1.0f / l;
  T* o = out + (size_t)t * out_stride + (size_t)h * vdim;
  const T* g = gate ? gate + (size_t)t * gate_stride + (size_t)h * vdim : nullptr;
#pragma unroll
  for (int i = 0; i < EXT_MAX_V_PER_LANE; ++i) {
    const int dim = lane + 32 * i;
    if (dim < vdim) {
      float r = acc[i] * inv;
      if (g) r *= 1.0f / (1.0f + expf(-to_f32(g[dim])));
      o[dim] = from_f32<T>(r * out_scale);
    }
  }
}

RL_API int rl_attn_ext(const void* q, int dtype, int q_stride, const void* k_pages, const void* v_pages, const int* block_table,
                       int table_width, const int* tok_seq, const int* tok_pos, const float* sink, const float* mix,
                       const void* gate, int gate_stride, float out_scale, void* out, int out_stride, int n_tokens, int H, int K,
                       int kdim, int vdim, int page_size, int window, float scale, int chunk, float softcap, int maps,
                       const float* bias, int bias_len, cudaStream_t stream) {
  if (bias != nullptr && bias_len <= 0) RL_REFUSE(10, "attn_ext: a bias by distance of %d numbers a head", bias_len);
  if (maps < 1 || maps > 2 || H % maps || kdim % maps || (maps > 1 && mix != nullptr)) RL_REFUSE(9, "attn_ext: %d maps in %d heads of %d numbers%s", maps, H, kdim, mix ? " whose scores are mixed" : "");
  if (n_tokens <= 0 || H <= 0 || K <= 0 || kdim <= 0 || vdim <= 0 || page_size <= 0)
    RL_REFUSE(1, "attn_ext: T=%d H=%d K=%d kdim=%d vdim=%d page=%d", n_tokens, H, K, kdim, vdim, page_size);
  if (H % K) RL_REFUSE(2, "attn_ext: %d query heads are not a multiple of %d kv heads", H, K);
  if (vdim > 32 * EXT_MAX_V_PER_LANE) RL_REFUSE(3, "attn_ext: value size %d exceeds %d", vdim, 32 * EXT_MAX_V_PER_LANE);
  if (H > 65535) RL_REFUSE(4, "attn_ext: %d heads exceed 65535", H);
  if (window < 0 || chunk < 0) RL_REFUSE(5, "attn_ext: negative window or chunk");
  if (mix != nullptr && H > 32) RL_REFUSE(6, "attn_ext: scores of %d heads cannot be mixed (at most 32)", H);
  const int HB = mix != nullptr ? H : 1;
  dim3 grid(n_tokens, H / HB), block(32, HB);
  const size_t smem = ((size_t)HB * kdim + (mix != nullptr ? (size_t)HB * 32 : 0)) * sizeof(float);
  if (smem > 48 * 1024) RL_REFUSE(7, "attn_ext: %d heads of %d numbers do not fit shared memory", HB, kdim);
  if (dtype == RL_BF16)
    attn_ext_kernel<bf16><<<grid, block, smem, stream>>>((const bf16*)q, q_stride, (const bf16*)k_pages, (const bf16*)v_pages,
                                                         block_table, table_width, tok_seq, tok_pos, sink, mix, (const bf16*)gate,
                                                         gate_stride, out_scale, (bf16*)out, out_stride, H, K, kdim, vdim, page_size,
                                                         window, scale, chunk, softcap, maps, bias, bias_len);
  else if (dtype == RL_F32)
    attn_ext_kernel<float><<<grid, block, smem, stream>>>((const float*)q, q_stride, (const float*)k_pages, (const float*)v_pages,
                                                          block_table, table_width, tok_seq, tok_pos, sink, mix, (const float*)gate,
                                                          gate_stride, out_scale, (float*)out, out_stride, H, K, kdim, vdim, page_size,
                                                          window, scale, chunk, softcap, maps, bias, bias_len);
  else
    RL_REFUSE(8, "attn_ext: unknown dtype %d", dtype);
  RL_LAUNCH_RESULT();
}

// ---------------------------------------------------------------- two maps into one head
// One warp per (token, head): a1 = a[t][2h], a2 = a[t][2h + 1] (vdim numbers each), o = a1 - lambda a2, out[t][h] = o / sqrt(mean(o^2) + eps) * factor.
// All of it 32-bit.  U: neighbouring numbers a lane takes at a time.
template <typename T, int U>
__global__ void map_combine_kernel(const T* __restrict__ a, int a_stride, float lambda, float eps, float factor, T* __restrict__ out, int out_stride,
                                   int n_rows, int H, int vdim) {
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const int pair = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (pair >= n_rows * H) return;
  const int t = pair / H, h = pair - t * H;
  const T* a1 = a + (size_t)t * a_stride + (size_t)(2 * h) * vdim;
  const T* a2 = a1 + vdim;
  constexpr int N = 256 / (32 * U);  // value sizes up to 256
  float v[N][U];
  float ss = 0.f;
#pragma unroll
  for (int c = 0; c < N; ++c) {
    const int i = (lane + 32 * c) * U;
    if (i < vdim) {
      float x[U], y[U];
      if (U == 4) {
        load4_g<T>(a1 + i, x);
        load4_g<T>(a2 + i, y);
      } else {
        x[0] = to_f32(__ldcg(a1 + i));
        y[0] = to_f32(__ldcg(a2 + i));
      }
#pragma unroll
      for (int e = 0; e < U; ++e) {
        v[c][e] = x[e] - lambda * y[e];
        ss += v[c][e] * v[c][e];
      }
    }
  }
  const float inv = factor / sqrtf(warp_sum(ss) / (float)vdim + eps);
  T* o = out + (size_t)t * out_stride + (size_t)h * vdim;
#pragma unroll
  for (int c = 0; c < N; ++c) {
    const int i = (lane + 32 * c) * U;
    if (i < vdim) {
#pragma unroll
      for (int e = 0; e < U; ++e) v[c][e] *= inv;
      if (U == 4) store4<T>(o + i, v[c]);
      else o[i] = from_f32<T>(v[c][0]);
    }
  }
}

RL_API int rl_map_combine(const void* a, int dtype, int a_stride, float lambda, float eps, float factor, void* out, int out_stride, int n_rows,
                          int H, int vdim, cudaStream_t stream) {
  if (n_rows <= 0 || H <= 0 || vdim <= 0 || vdim > 256) RL_REFUSE(1, "map_combine: rows=%d H=%d values=%d (at most 256)", n_rows, H, vdim);
  if (a_stride < 2 * H * vdim || out_stride < H * vdim) RL_REFUSE(2, "map_combine: rows too short");
  if ((long long)n_rows * H > 0x7ffffff0LL) RL_REFUSE(3, "map_combine: %d rows of %d heads are too many", n_rows, H);
  const int blocks = (int)(((long long)n_rows * H + 3) / 4);
  const size_t bytes = dtype == RL_BF16 ? 8 : 16;
  const bool vec = vdim % 4 == 0 && a_stride % 4 == 0 && out_stride % 4 == 0 && (((uintptr_t)a | (uintptr_t)out) % bytes) == 0;
#define RL_MC(T, U) \
  RL_LAUNCH_CHECK(rl_launch(map_combine_kernel<T, U>, blocks, 128, 0, stream, (const T*)a, a_stride, lambda, eps, factor, (T*)out, out_stride, n_rows, H, vdim))
  if (dtype == RL_BF16 && vec) RL_MC(bf16, 4);
  else if (dtype == RL_BF16) RL_MC(bf16, 1);
  else if (dtype == RL_F32 && vec) RL_MC(float, 4);
  else if (dtype == RL_F32) RL_MC(float, 1);
  else RL_REFUSE(4, "map_combine: unknown dtype %d", dtype);
#undef RL_MC
  return 0;
}
