// What stands around attention with normed queries and keys: the norm over whole projections,
// rotations of keys, queries and values, the stores into the paged cache, the pooled blocks'
// means, and the turn back of a head's result.  Float32 arithmetic; T is the storage type.
//
//   x     = x / sqrt(mean_row x^2 + eps) * w                 over all heads of q (of k) at once
//   (a, b)= (a cos - b sin, b cos + a sin)                   pair (i, i + n/2), angle = pos * freq[i]
//   q    *= head_scale[head]
// A page of the cache holds all its key rows [kv head, entry, head_dim], then all its value
// rows [kv head, entry, value_dim].
#include "common.cuh"

// ---------------------------------------------------------------------------
// One block per token.  qkv row: q (H d) | k (G d) | v (G dv); G = 0: a layer without keys and
// values of its own.  rot_freq [rot_dims / 2] (null: no rotation), value_freq [dv / 2] (null:
// values are stored as they are).
// ---------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256)
qk_norm_rotate_store_kernel(const T* __restrict__ qkv, int row_width, const float* __restrict__ q_norm,
                            const float* __restrict__ k_norm, float eps, const float* __restrict__ head_scale,
                            const float* __restrict__ rot_freq, int rot_dims, const float* __restrict__ value_freq,
                            T* __restrict__ q_out, T* __restrict__ cache, const int* __restrict__ block_table,
                            int max_pages, const int* __restrict__ token_seq, const int* __restrict__ positions,
                            int H, int G, int d, int dv, int page_size, int num_pages, int write_cache, int* err) {
  pdl_wait_block();
  pdl_launch_dependents();
  extern __shared__ float row[];  // (H + G) d floats, 33 scratch, cos and sin of rot_dims / 2 and of dv / 2 angles
  const int nq = H * d, nk = G * d;
  float* scratch = row + nq + nk;
  const int half = rot_dims / 2, vhalf = dv / 2;
  float* cs_qk = scratch + 33;    // [half] cos, [half] sin
  float* cs_v = cs_qk + 2 * half;  // [vhalf] cos, [vhalf] sin
  const int t = blockIdx.x;
  const T* x = qkv + (size_t)t * row_width;
  const float pos = (float)positions[t];
  // A token's angles are the same for all its heads: once per block.
  if (rot_freq != nullptr)
    for (int i = threadIdx.x; i < half; i += blockDim.x) sincosf(pos * rot_freq[i], cs_qk + half + i, cs_qk + i);
  if (value_freq != nullptr && write_cache && nk > 0)
    for (int i = threadIdx.x; i < vhalf; i += blockDim.x) sincosf(pos * value_freq[i], cs_v + vhalf + i, cs_v + i);

  constexpr int N = Vec<T>::N;
  const bool vec = d % N == 0 && row_width % N == 0;  // whole 16-byte groups inside a head
  float ssq = 0.f, ssk = 0.f;
  if (vec) {
    for (int i = threadIdx.x * N; i < nq + nk; i += blockDim.x * N) {
      float v[N];
      Vec<T>::load(x + i, v);
      float ss = 0.f;
#pragma unroll
      for (int e = 0; e < N; ++e) {
        row[i + e] = v[e];
        ss = fmaf(v[e], v[e], ss);
      }
      if (i < nq) ssq += ss; else ssk += ss;
    }
  } else {
    for (int i = threadIdx.x; i < nq + nk; i += blockDim.x) {
      const float v = to_f32<T>(x[i]);
      row[i] = v;
      if (i < nq) ssq = fmaf(v, v, ssq); else ssk = fmaf(v, v, ssk);
    }
  }
  ssq = block_sum(ssq, scratch);
  const float rq = 1.0f / sqrtf(ssq / (float)nq + eps);
  float rk = 0.f;
  if (nk > 0) {
    ssk = block_sum(ssk, scratch);
    rk = 1.0f / sqrtf(ssk / (float)nk + eps);
  }
  for (int i = threadIdx.x; i < nq + nk; i += blockDim.x)
    row[i] = i < nq ? row[i] * rq * q_norm[i] : row[i] * rk * k_norm[i - nq];
  __syncthreads();

  long long page = -1;
  int off = 0;
  if (write_cache && nk > 0) {
    const int p = positions[t];
    page = block_table[(size_t)token_seq[t] * max_pages + p / page_size];
    off = p % page_size;
    if (page < 0 || page >= num_pages) {
      if (threadIdx.x == 0) atomicOr(err, SB_ERR_BAD_PAGE);
      page = -1;
    }
  }
  const size_t page_stride = (size_t)G * page_size * (d + dv);
  if (vec) {
    for (int i0 = threadIdx.x * N; i0 < nq + nk; i0 += blockDim.x * N) {
      const int head = i0 / d, c0 = i0 - head * d;
      const float scale = i0 < nq ? head_scale[head] : 1.f;
      float o[N];
#pragma unroll
      for (int e = 0; e < N; ++e) {
        const int c = c0 + e;
        float v = row[i0 + e];
        if (rot_freq != nullptr && c < rot_dims) {
          const int pair = c < half ? c : c - half;
          const float cs = cs_qk[pair], sn = cs_qk[half + pair];
          const float a = row[i0 - c0 + pair], b = row[i0 - c0 + pair + half];
          v = c < half ? a * cs - b * sn : b * cs + a * sn;
        }
        o[e] = v * scale;
      }
      if (i0 < nq)
        Vec<T>::store(q_out + (size_t)t * nq + i0, o);
      else if (page >= 0)
        Vec<T>::store(cache + page * page_stride + ((size_t)(head - H) * page_size + off) * d + c0, o);
    }
  }
  for (int i = threadIdx.x; i < (vec ? 0 : nq + nk); i += blockDim.x) {
    const int head = i / d, c = i % d;
    float v = row[i];
    if (rot_freq != nullptr && c < rot_dims) {
      const int pair = c < half ? c : c - half;
      const float cs = cs_qk[pair], sn = cs_qk[half + pair];
      const float a = row[i - c + pair], b = row[i - c + pair + half];
      v = c < half ? a * cs - b * sn : b * cs + a * sn;
    }
    if (i < nq) {
      q_out[(size_t)t * nq + i] = from_f32<T>(v * head_scale[head]);
    } else if (page >= 0) {
      const int m = head - H;
      cache[page * page_stride + ((size_t)m * page_size + off) * d + c] = from_f32<T>(v);
    }
  }
  if (page >= 0) {
    const T* vx = x + nq + nk;
    T* dst = cache + page * page_stride + (size_t)G * page_size * d;
    const bool vec_v = vec && dv % N == 0 && (value_freq == nullptr || vhalf % N == 0) && (nq + nk) % N == 0;
    if (vec_v) {
      for (int i0 = threadIdx.x * N; i0 < G * dv; i0 += blockDim.x * N) {
        const int m = i0 / dv, c0 = i0 - m * dv;
        float own[N], other[N], o[N];
        Vec<T>::load(vx + i0, own);
        if (value_freq != nullptr) {
          Vec<T>::load(vx + (c0 < vhalf ? i0 + vhalf : i0 - vhalf), other);
#pragma unroll
          for (int e = 0; e < N; ++e) {
            const int pair = c0 < vhalf ? c0 + e : c0 + e - vhalf;
            const float cs = cs_v[pair], sn = cs_v[vhalf + pair];
            o[e] = c0 < vhalf ? own[e] * cs - other[e] * sn : own[e] * cs + other[e] * sn;
          }
        } else {
#pragma unroll
          for (int e = 0; e < N; ++e) o[e] = own[e];
        }
        Vec<T>::store(dst + ((size_t)m * page_size + off) * dv + c0, o);
      }
    }
    for (int i = threadIdx.x; i < (vec_v ? 0 : G * dv); i += blockDim.x) {
      const int m = i / dv, c = i % dv;
      float v = to_f32<T>(vx[i]);
      if (value_freq != nullptr) {
        const int pair = c < vhalf ? c : c - vhalf;
        const float cs = cs_v[pair], sn = cs_v[vhalf + pair];
        const float a = to_f32<T>(vx[i - c + pair]), b = to_f32<T>(vx[i - c + pair + vhalf]);
        v = c < vhalf ? a * cs - b * sn : b * cs + a * sn;
      }
      dst[((size_t)m * page_size + off) * dv + c] = from_f32<T>(v);
    }
  }
}

extern "C" int sb_qk_norm_rotate_store(const void* qkv, int row_width, int dtype, const float* q_norm,
                                       const float* k_norm, float eps, const float* head_scale,
                                       const float* rot_freq, int rot_dims, const float* value_freq, void* q_out,
                                       void* cache, const int* block_table, int max_pages, const int* token_seq,
                                       const int* positions, int num_tokens, int H, int G, int d, int dv,
                                       int page_size, int num_pages, int write_cache, int* err,
                                       cudaStream_t stream) {
  if (num_tokens == 0) return 0;
  const size_t smem = ((size_t)(H + G) * d + 33 + rot_dims + dv) * sizeof(float);
  if (smem > 200 * 1024) return -2;
  if (rot_dims % 2 || rot_dims > d || (value_freq != nullptr && dv % 2)) return -4;
  if (dtype == SB_DTYPE_F32) {
    if (smem > 48 * 1024) cudaFuncSetAttribute(qk_norm_rotate_store_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    sb_launch(qk_norm_rotate_store_kernel<float>, num_tokens, 256, smem, stream, (const float*)qkv, row_width,
              q_norm, k_norm, eps, head_scale, rot_freq, rot_dims, value_freq, (float*)q_out, (float*)cache,
              block_table, max_pages, token_seq, positions, H, G, d, dv, page_size, num_pages, write_cache, err);
  } else {
    if (smem > 48 * 1024) cudaFuncSetAttribute(qk_norm_rotate_store_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    sb_launch(qk_norm_rotate_store_kernel<bf16>, num_tokens, 256, smem, stream, (const bf16*)qkv, row_width,
              q_norm, k_norm, eps, head_scale, rot_freq, rot_dims, value_freq, (bf16*)q_out, (bf16*)cache,
              block_table, max_pages, token_seq, positions, H, G, d, dv, page_size, num_pages, write_cache, err);
  }
  SB_LAUNCH_CHECK();
  return 0;
}

// ---------------------------------------------------------------------------
// Pooled blocks: for every block of P tokens whose last token arrived in this step, the mean of
// its keys and of its values as the cache holds them, summed in float32 in the tokens' order,
// into the storage of block entries.  Grid (block within the step, sequence, kv head).
// ---------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(1024)
pool_blocks_kernel(const T* __restrict__ cache, const int* __restrict__ block_table, int max_pages, int num_pages,
                   T* __restrict__ pool, const int* __restrict__ pool_table, int pool_max_pages,
                   int pool_pages, const int* __restrict__ cu_q, const int* __restrict__ q_start, int G, int d,
                   int dv, int page_size, int P, int* err) {
  pdl_wait_block();
  pdl_launch_dependents();
  const int b = blockIdx.y, m = blockIdx.z;
  const int start = q_start[b], end = start + cu_q[b + 1] - cu_q[b];
  const int c = start / P + blockIdx.x;
  if (c >= end / P) return;
  const int first = c * P;
  const int entries = (page_size + P - 1) / P;
  const long long to = pool_table[(size_t)b * pool_max_pages + first / page_size];
  if (to < 0 || to >= pool_pages) {
    if (threadIdx.x == 0) atomicOr(err, SB_ERR_BAD_PAGE);
    return;
  }
  const size_t page_stride = (size_t)G * page_size * (d + dv);
  const size_t pool_stride = (size_t)G * entries * (d + dv);
  const size_t entry = (size_t)m * entries + (first % page_size) / P;
  // Where the block's tokens live: worked out once per 64 tokens, by the first threads.
  __shared__ long long where[64];  // the token's page times the page's size; -1: not held
  __shared__ int row_in_page[64];
  float sums[4] = {0.f, 0.f, 0.f, 0.f};  // this thread's channels: threadIdx.x, + 128, ...
  bool ok = true;
  for (int j0 = 0; j0 < P; j0 += 64) {
    const int count = min(64, P - j0);
    __syncthreads();
    if ((int)threadIdx.x < count) {
      const int p = first + j0 + threadIdx.x;
      const long long page = block_table[(size_t)b * max_pages + p / page_size];
      where[threadIdx.x] = (page < 0 || page >= num_pages) ? -1 : page * (long long)page_stride;
      row_in_page[threadIdx.x] = p % page_size;
    }
    __syncthreads();
#pragma unroll
    for (int turn = 0; turn < 4; ++turn) {
      const int ch = turn * blockDim.x + threadIdx.x;
      if (ch >= d + dv) break;
      const bool is_key = ch < d;
      const int cc = is_key ? ch : ch - d, width = is_key ? d : dv;
      const size_t base = (is_key ? 0 : (size_t)G * page_size * d) + (size_t)m * page_size * width + cc;
      float sum = sums[turn];
      for (int j = 0; j < count; j += 8) {  // eight tokens' loads together, added in the tokens' order
        float x[8];
#pragma unroll
        for (int u = 0; u < 8; ++u) {
          x[u] = 0.f;
          if (j + u < count) {
            const long long at = where[j + u];
            if (at < 0) ok = false;
            else x[u] = to_f32<T>(cache[at + base + (size_t)row_in_page[j + u] * width]);
          }
        }
#pragma unroll
        for (int u = 0; u < 8; ++u)
          if (j + u < count) sum += x[u];
      }
      sums[turn] = sum;
    }
  }
  if (!ok) atomicOr(err, SB_ERR_BAD_PAGE);
#pragma unroll
  for (int turn = 0; turn < 4; ++turn) {
    const int ch = turn * blockDim.x + threadIdx.x;
    if (ch >= d + dv || !ok) break;
    const bool is_key = ch < d;
    const int cc = is_key ? ch : ch - d, width = is_key ? d : dv;
    T* dst = pool + to * pool_stride + (is_key ? 0 : (size_t)G * entries * d) + entry * width + cc;
    *dst = from_f32<T>(sums[turn] / (float)P);
  }
}

extern "C" int sb_pool_blocks(const void* cache, int dtype, const int* block_table, int max_pages, int num_pages,
                              void* pool, const int* pool_table, int pool_max_pages, int pool_pages,
                              const int* cu_q, const int* q_start, int num_seqs, int max_blocks, int G, int d,
                              int dv, int page_size, int P, int* err, cudaStream_t stream) {
  if (num_seqs == 0 || max_blocks <= 0) return 0;
  if (P <= 0) return -13;
  const dim3 grid(max_blocks, num_seqs, G);
  // a thread keeps up to four channels' sums: wider heads get wider blocks
  int threads = 128;
  while (threads * 4 < d + dv && threads < 1024) threads *= 2;
  if (threads * 4 < d + dv) return -13;
  if (dtype == SB_DTYPE_F32)
    sb_launch(pool_blocks_kernel<float>, grid, threads, 0, stream, (const float*)cache, block_table, max_pages,
              num_pages, (float*)pool, pool_table, pool_max_pages, pool_pages, cu_q, q_start, G, d, dv, page_size, P, err);
  else
    sb_launch(pool_blocks_kernel<bf16>, grid, threads, 0, stream, (const bf16*)cache, block_table, max_pages,
              num_pages, (bf16*)pool, pool_table, pool_max_pages, pool_pages, cu_q, q_start, G, d, dv, page_size, P, err);
  SB_LAUNCH_CHECK();
  return 0;
}

// ---------------------------------------------------------------------------
// Turns every head of x [T, H, n] by its token's position: pair (i, i + n/2) by
// sign * pos * freq[i].  One block per token.
// ---------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256)
rotate_heads_kernel(const T* __restrict__ x, const int* __restrict__ positions, const float* __restrict__ freq,
                    float sign, int H, int n, T* __restrict__ out) {
  pdl_wait_block();
  pdl_launch_dependents();
  extern __shared__ float cs[];  // [n / 2] cos, [n / 2] sin: a token's angles are the same for all its heads
  const int t = blockIdx.x, half = n / 2;
  const float pos = sign * (float)positions[t];
  for (int i = threadIdx.x; i < half; i += blockDim.x) sincosf(pos * freq[i], cs + half + i, cs + i);
  __syncthreads();
  constexpr int N = Vec<T>::N;
  if (half % N == 0) {
    for (int i0 = threadIdx.x * N; i0 < H * half; i0 += blockDim.x * N) {
      const int h = i0 / half, pair = i0 - h * half;
      const size_t at = ((size_t)t * H + h) * n + pair;
      float a[N], b[N], lo[N], hi[N];
      Vec<T>::load(x + at, a);
      Vec<T>::load(x + at + half, b);
#pragma unroll
      for (int e = 0; e < N; ++e) {
        const float c = cs[pair + e], s = cs[half + pair + e];
        lo[e] = a[e] * c - b[e] * s;
        hi[e] = b[e] * c + a[e] * s;
      }
      Vec<T>::store(out + at, lo);
      Vec<T>::store(out + at + half, hi);
    }
    return;
  }
  for (int i = threadIdx.x; i < H * half; i += blockDim.x) {
    const int h = i / half, pair = i % half;
    const size_t at = ((size_t)t * H + h) * n + pair;
    const float c = cs[pair], s = cs[half + pair];
    const float a = to_f32<T>(x[at]), b = to_f32<T>(x[at + half]);
    out[at] = from_f32<T>(a * c - b * s);
    out[at + half] = from_f32<T>(b * c + a * s);
  }
}

extern "C" int sb_rotate_heads(const void* x, int dtype, const int* positions, const float* freq, float sign,
                               int num_tokens, int H, int n, void* out, cudaStream_t stream) {
  if (num_tokens == 0) return 0;
  if (n % 2) return -4;
  if (dtype == SB_DTYPE_F32)
    sb_launch(rotate_heads_kernel<float>, num_tokens, 256, (size_t)n * sizeof(float), stream, (const float*)x, positions, freq, sign, H, n,
              (float*)out);
  else
    sb_launch(rotate_heads_kernel<bf16>, num_tokens, 256, (size_t)n * sizeof(float), stream, (const bf16*)x, positions, freq, sign, H, n,
              (bf16*)out);
  SB_LAUNCH_CHECK();
  return 0;
}

// ---------------------------------------------------------------------------
// Attention whose heads are normed one by one after rotation.  One block per token, a warp per
// head.  Row of `proj`: q (H d) | k (G d) | [v (G dv)] | whatever follows (a gate, which this
// kernel does not read).
//   (a, b) = (a cos - b sin, b cos + a sin)     neighbours (2i, 2i + 1) for `interleaved`, else
//                                               (i, i + rot_dims/2); angle = pos * rot_freq[i]
//   x      = x / sqrt(mean_head x^2 + eps)      (no scale; `head_norm` = 0 skips it)
//   q     *= q_scale
// Keys go to the cache rotated and normed.  Values: with `tie_values` a key head as the projection
// left it (before rotation and norm) is also the value head; otherwise the v columns as they are.
// ---------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256)
rotate_headnorm_store_kernel(const T* __restrict__ proj, int row_width, const float* __restrict__ bias, float eps, float q_scale,
                             const float* __restrict__ rot_freq, int rot_dims, int interleaved, int head_norm,
                             int tie_values, T* __restrict__ q_out, T* __restrict__ cache,
                             const int* __restrict__ block_table, int max_pages, const int* __restrict__ token_seq,
                             const int* __restrict__ positions, int H, int G, int d, int dv, int page_size,
                             int num_pages, int write_cache, int* err) {
  pdl_wait_block();
  pdl_launch_dependents();
  extern __shared__ float row[];  // (H + G) d floats, then cos and sin of rot_dims / 2 angles
  const int nq = H * d, nk = G * d, half = rot_dims / 2;
  float* cs = row + nq + nk;
  const int t = blockIdx.x;
  const T* x = proj + (size_t)t * row_width;
  const float pos = (float)positions[t];
  for (int i = threadIdx.x; i < half; i += blockDim.x) sincosf(pos * rot_freq[i], cs + half + i, cs + i);
  // `bias`: a learned offset on q, k and (untied) v, added in float32 before anything else
  for (int i = threadIdx.x; i < nq + nk; i += blockDim.x) row[i] = to_f32<T>(x[i]) + (bias != nullptr ? bias[i] : 0.f);
  __syncthreads();

  long long page = -1;
  int off = 0;
  if (write_cache && nk > 0) {
    const int p = positions[t];
    page = block_table[(size_t)token_seq[t] * max_pages + p / page_size];
    off = p % page_size;
    if (page < 0 || page >= num_pages) {
      if (threadIdx.x == 0) atomicOr(err, SB_ERR_BAD_PAGE);
      page = -1;
    }
  }
  const size_t page_stride = (size_t)G * page_size * (d + dv);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
  for (int head = warp; head < H + G; head += nwarps) {
    float* v = row + (size_t)head * d;
    const bool is_q = head < H;
    T* value_dst = nullptr;
    T* key_dst = nullptr;
    if (!is_q && page >= 0) {
      key_dst = cache + page * page_stride + ((size_t)(head - H) * page_size + off) * d;
      value_dst = cache + page * page_stride + (size_t)G * page_size * d + ((size_t)(head - H) * page_size + off) * dv;
      if (tie_values)  // the head as projected, before this warp turns it
        for (int c = lane; c < d; c += 32) value_dst[c] = from_f32<T>(v[c]);
    }
    __syncwarp();
    for (int i = lane; i < half; i += 32) {
      const int ia = interleaved ? 2 * i : i, ib = interleaved ? 2 * i + 1 : i + half;
      const float a = v[ia], b = v[ib], c = cs[i], sn = cs[half + i];
      v[ia] = a * c - b * sn;
      v[ib] = b * c + a * sn;
    }
    __syncwarp();
    float scale = is_q ? q_scale : 1.0f;
    if (head_norm) {
      float ss = 0.f;
      for (int c = lane; c < d; c += 32) ss = fmaf(v[c], v[c], ss);
      ss = warp_sum(ss);
      scale *= 1.0f / sqrtf(ss / (float)d + eps);
    }
    if (is_q) {
      T* dst = q_out + (size_t)t * nq + (size_t)head * d;
      for (int c = lane; c < d; c += 32) dst[c] = from_f32<T>(v[c] * scale);
    } else if (key_dst != nullptr) {
      for (int c = lane; c < d; c += 32) key_dst[c] = from_f32<T>(v[c] * scale);
    }
  }
  if (!tie_values && page >= 0) {
    const T* vx = x + nq + nk;
    T* dst = cache + page * page_stride + (size_t)G * page_size * d;
    for (int i = threadIdx.x; i < G * dv; i += blockDim.x) {
      const int m = i / dv, c = i - m * dv;
      dst[((size_t)m * page_size + off) * dv + c] =
          bias != nullptr ? from_f32<T>(to_f32<T>(vx[i]) + bias[nq + nk + i]) : vx[i];
    }
  }
}

extern "C" int sb_rotate_headnorm_store(const void* proj, int row_width, int dtype, const float* bias, float eps, float q_scale,
                                        const float* rot_freq, int rot_dims, int interleaved, int head_norm,
                                        int tie_values, void* q_out, void* cache, const int* block_table,
                                        int max_pages, const int* token_seq, const int* positions, int num_tokens,
                                        int H, int G, int d, int dv, int page_size, int num_pages, int write_cache,
                                        int* err, cudaStream_t stream) {
  if (num_tokens == 0) return 0;
  if (rot_freq == nullptr) rot_dims = 0;
  const size_t smem = ((size_t)(H + G) * d + rot_dims) * sizeof(float);
  if (smem > 200 * 1024) return -2;
  if (rot_dims % 2 || rot_dims > d || (tie_values && dv != d)) return -4;
  if (dtype == SB_DTYPE_F32) {
    if (smem > 48 * 1024) cudaFuncSetAttribute(rotate_headnorm_store_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    sb_launch(rotate_headnorm_store_kernel<float>, num_tokens, 256, smem, stream, (const float*)proj, row_width, bias, eps,
              q_scale, rot_freq, rot_dims, interleaved, head_norm, tie_values, (float*)q_out, (float*)cache,
              block_table, max_pages, token_seq, positions, H, G, d, dv, page_size, num_pages, write_cache, err);
  } else {
    if (smem > 48 * 1024) cudaFuncSetAttribute(rotate_headnorm_store_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    sb_launch(rotate_headnorm_store_kernel<bf16>, num_tokens, 256, smem, stream, (const bf16*)proj, row_width, bias, eps,
              q_scale, rot_freq, rot_dims, interleaved, head_norm, tie_values, (bf16*)q_out, (bf16*)cache,
              block_table, max_pages, token_seq, positions, H, G, d, dv, page_size, num_pages, write_cache, err);
  }
  SB_LAUNCH_CHECK();
  return 0;
}

// ---------------------------------------------------------------------------
// Attention whose q, k and v pass a short causal convolution, then (q and k) a norm per head with a
// scale per channel, then the rotation.  Row of `proj`: q (H d) | k (G d) | v (G dv) | whatever follows.
//   u_t  = sum_j w[j, c] p_(t - taps + 1 + j, c)    p: the sequence's projected rows; before the step's
//                                                  first token the state's, zeros before the sequence
//   x    = u / sqrt(mean_head u^2 + eps) * scale   q and k heads
//   pair (i, i + rot/2), or neighbours, turned by position * rot_freq[i]; q times q_scale
// A warp takes one head of a few tokens in a row: what the taps read again is in L1.
// With `alone` every sequence brings one token, and the warp that has read a channel's state moves it
// on (of rows that share a slot the first serves all); else a kernel of its own does, after this one.
// ---------------------------------------------------------------------------
#define SB_ERR_BAD_SLOT 16
constexpr int PREP_WARPS = 8;

template <typename T, int TAPS>  // TAPS: 0 none, 2 .. 4, -1 any number
__global__ void __launch_bounds__(PREP_WARPS * 32)
conv_headnorm_store_kernel(const T* __restrict__ proj, int row_width, const float* __restrict__ conv_w, int taps_rt,
                           float* __restrict__ state, const int* __restrict__ slots, int num_slots, int num_seqs, int alone,
                           const float* __restrict__ q_norm, const float* __restrict__ k_norm, float eps, float q_scale,
                           const float* __restrict__ rot_freq, int rot_dims, int interleaved, T* __restrict__ q_out,
                           T* __restrict__ cache, const int* __restrict__ block_table, int max_pages,
                           const int* __restrict__ token_seq, const int* __restrict__ cu_q,
                           const int* __restrict__ positions, int num_tokens, int rows_per_block, int H, int G, int d, int dv,
                           int page_size, int num_pages, int write_cache, int* err) {
  pdl_wait_block();
  pdl_launch_dependents();
  extern __shared__ float prep_smem[];  // cos and sin of the block's tokens, then a head's row per warp
  const int half = rot_dims / 2, hd = max(d, dv);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int t0 = blockIdx.x * rows_per_block, rows = min(rows_per_block, num_tokens - t0);
  for (int i = threadIdx.x; i < rows * half; i += blockDim.x) {
    const int r = i / half, a = i - r * half;
    sincosf((float)positions[t0 + r] * rot_freq[a], prep_smem + (2 * r + 1) * half + a, prep_smem + 2 * r * half + a);
  }
  __syncthreads();
  const int head = blockIdx.y * PREP_WARPS + warp;
  if (head >= H + 2 * G) return;
  float* buf = prep_smem + 2 * rows_per_block * half + (size_t)warp * hd;
  const int taps = TAPS >= 0 ? TAPS : taps_rt;
  const bool is_q = head < H, is_v = head >= H + G;
  const int n = is_v ? dv : d;                                            // channels of this head
  const int c0 = is_v ? (H + G) * d + (head - H - G) * dv : head * d;     // its first channel
  const int channels = (H + G) * d + G * dv;
  const float* scale_w = is_q ? q_norm : k_norm;
  const size_t page_stride = (size_t)G * page_size * (d + dv);

  for (int r = 0; r < rows; ++r) {
    const int t = t0 + r, b = token_seq[t];
    const int i = t - cu_q[b];  // the token's place among the step's tokens of its sequence
    int copies = 1;
    float* st = nullptr;
    if (taps > 1) {
      const int slot = slots[b];
      if (slot < 0 || slot >= num_slots) {
        if (lane == 0) atomicOr(err, SB_ERR_BAD_SLOT);
        continue;
      }
      st = state + (size_t)slot * (taps - 1) * channels + c0;
      if (alone) {
        copies = rows_sharing_slot(slots, b, num_seqs);
        if (copies == 0) continue;  // an earlier row's warp serves this one
      }
    }
    const T* x = proj + (size_t)t * row_width + c0;
    float ss = 0.f;
    for (int c = lane; c < n; c += 32) {
      const float own = to_f32<T>(x[c]);
      float u = own;
      if (taps > 0) {
        const float* w = conv_w + c0 + c;  // [taps][channels]
        if (alone) {
          u = 0.f;
#pragma unroll
          for (int j = 0; j + 1 < taps; ++j) {
            const float s = st[(size_t)j * channels + c];
            u = fmaf(w[(size_t)j * channels], s, u);
            if (j > 0) st[(size_t)(j - 1) * channels + c] = s;
          }
          u = fmaf(w[(size_t)(taps - 1) * channels], own, u);
          if (taps > 1) st[(size_t)(taps - 2) * channels + c] = own;
        } else {
          u = 0.f;
#pragma unroll
          for (int j = 0; j < taps; ++j) {
            const int at = i - (taps - 1) + j;
            const float p = j == taps - 1 ? own
                            : at >= 0     ? to_f32<T>(x[c - (long long)(taps - 1 - j) * row_width])
                                          : st[(size_t)(taps - 1 + at) * channels + c];
            u = fmaf(w[(size_t)j * channels], p, u);
          }
        }
      }
      buf[c] = u;
      ss = fmaf(u, u, ss);
    }
    __syncwarp();
    T* dst = nullptr;
    if (is_q) {
      dst = q_out + ((size_t)t * H + head) * d;
    } else if (write_cache) {
      const int p = positions[t];
      const long long page = block_table[(size_t)b * max_pages + p / page_size];
      if (page < 0 || page >= num_pages) {
        if (lane == 0) atomicOr(err, SB_ERR_BAD_PAGE);
      } else if (is_v) {
        dst = cache + page * page_stride + (size_t)G * page_size * d + ((size_t)(head - H - G) * page_size + p % page_size) * dv;
      } else {
        dst = cache + page * page_stride + ((size_t)(head - H) * page_size + p % page_size) * d;
      }
    }
    if (is_v) {
      if (dst != nullptr)
        for (int c = lane; c < n; c += 32) dst[c] = from_f32<T>(buf[c]);
    } else {
      const float inv = (is_q ? q_scale : 1.0f) / sqrtf(warp_sum(ss) / (float)d + eps);
      const float* cs = prep_smem + 2 * r * half;
      if (dst != nullptr) {
        for (int c = lane; c < n; c += 32) {
          float v = buf[c] * scale_w[c];
          if (c < rot_dims) {
            const int a = interleaved ? c >> 1 : (c < half ? c : c - half);
            const bool low = interleaved ? (c & 1) == 0 : c < half;
            const int other = interleaved ? c ^ 1 : (low ? c + half : c - half);
            const float o = buf[other] * scale_w[other];
            v = low ? v * cs[a] - o * cs[half + a] : v * cs[a] + o * cs[half + a];
          }
          v *= inv;
          for (int k = 0; k < copies; ++k) dst[(is_q ? (size_t)k * H * d : 0) + c] = from_f32<T>(v);
        }
      }
    }
    __syncwarp();
  }
}

// The same for steps with prompt portions, two neighbouring channels per lane: the taps' weights of a warp's
// head and all rows of a block stay in registers.  Heads of up to 64 * NCH channels, whole
// pairs of channels everywhere (d, dv, the row width and half the turned dims are even).
template <typename T> struct Pair;
template <> struct Pair<float> {
  __device__ static float2 load(const float* p) { return *reinterpret_cast<const float2*>(p); }
  __device__ static void store(float* p, float2 v) { *reinterpret_cast<float2*>(p) = v; }
};
template <> struct Pair<bf16> {
  __device__ static float2 load(const bf16* p) {
    const uint32_t v = *reinterpret_cast<const uint32_t*>(p);
    return make_float2(__uint_as_float(v << 16), __uint_as_float(v & 0xffff0000u));
  }
  __device__ static void store(bf16* p, float2 v) { *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v.x, v.y); }
};

template <typename T, int TAPS, int NCH, int ROWS>
__global__ void __launch_bounds__(PREP_WARPS * 32)
conv_headnorm_store_pairs_kernel(const T* __restrict__ proj, int row_width, const float* __restrict__ conv_w,
                                 const float* __restrict__ state, const int* __restrict__ slots, int num_slots,
                                 const float* __restrict__ q_norm, const float* __restrict__ k_norm, float eps, float q_scale,
                                 const float* __restrict__ rot_freq, int rot_dims, int interleaved, T* __restrict__ q_out,
                                 T* __restrict__ cache, const int* __restrict__ block_table, int max_pages,
                                 const int* __restrict__ token_seq, const int* __restrict__ cu_q,
                                 const int* __restrict__ positions, int num_tokens, int H, int G, int d, int dv,
                                 int page_size, int num_pages, int write_cache, int* err) {
  extern __shared__ float prep_smem[];
  // per token of the block: its place in its sequence's part of the step, its state slot, its page and place there
  __shared__ int s_place[ROWS], s_slot[ROWS], s_page[ROWS], s_off[ROWS];
  const int half = rot_dims / 2, hd = max(d, dv);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int t0 = blockIdx.x * ROWS, rows = min(ROWS, num_tokens - t0);
  const int head = blockIdx.y * PREP_WARPS + warp;
  const bool on = head < H + 2 * G, is_q = head < H, is_v = head >= H + G;
  const int n = is_v ? dv : d;
  const int c0 = is_v ? (H + G) * d + (head - H - G) * dv : head * d;
  const int channels = (H + G) * d + G * dv;
  constexpr int W = TAPS > 0 ? TAPS : 1, BACK = W - 1;  // rows before a token that it reads
  float2 w[W][NCH], scale[NCH];
  if (on) {  // (weights: before the wait)
    const float* scale_w = is_q ? q_norm : k_norm;
#pragma unroll
    for (int k = 0; k < NCH; ++k) {
      const int c = 2 * lane + 64 * k;
      scale[k] = c < n && !is_v ? Pair<float>::load(scale_w + c) : make_float2(0.f, 0.f);
#pragma unroll
      for (int j = 0; j < TAPS; ++j)
        w[j][k] = c < n ? Pair<float>::load(conv_w + (size_t)j * channels + c0 + c) : make_float2(0.f, 0.f);
    }
  }
  pdl_wait_block();
  pdl_launch_dependents();
  for (int r = threadIdx.x; r < rows; r += blockDim.x) {
    const int t = t0 + r, b = token_seq[t], p = positions[t];
    s_place[r] = t - cu_q[b];
    const int slot = TAPS > 1 ? slots[b] : 0;
    const bool bad_slot = TAPS > 1 && (slot < 0 || slot >= num_slots);
    s_slot[r] = bad_slot ? -1 : slot;
    int page = write_cache ? block_table[(size_t)b * max_pages + p / page_size] : 0;
    if (page < 0 || page >= num_pages) {
      if (write_cache && blockIdx.y == 0) atomicOr(err, SB_ERR_BAD_PAGE);
      page = -1;
    }
    if (bad_slot && blockIdx.y == 0) atomicOr(err, SB_ERR_BAD_SLOT);
    s_page[r] = page;
    s_off[r] = p % page_size;
  }
  for (int i = threadIdx.x; i < rows * half; i += blockDim.x) {
    const int r = i / half, a = i - r * half;
    sincosf((float)positions[t0 + r] * rot_freq[a], prep_smem + (2 * r + 1) * half + a, prep_smem + 2 * r * half + a);
  }
  __syncthreads();
  if (!on) return;
  float* buf = prep_smem + 2 * ROWS * half + (size_t)warp * hd;
  const size_t page_stride = (size_t)G * page_size * (d + dv);
  // The block's rows and the BACK rows ahead of them, all under way at once (those of another sequence are not used).
  float2 row[BACK + ROWS][NCH];
#pragma unroll
  for (int a = 0; a < BACK + ROWS; ++a) {
    const int t = t0 - BACK + a;
#pragma unroll
    for (int k = 0; k < NCH; ++k) {
      const int c = 2 * lane + 64 * k;
      row[a][k] = c < n && t >= 0 && t < num_tokens ? Pair<T>::load(proj + (size_t)t * row_width + c0 + c) : make_float2(0.f, 0.f);
    }
  }

#pragma unroll
  for (int r = 0; r < ROWS; ++r) {
    if (r >= rows) break;
    const int t = t0 + r, i = s_place[r], slot = s_slot[r];
    float2 u[NCH];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < NCH; ++k) {
      const int c = 2 * lane + 64 * k;
      u[k] = TAPS > 0 ? make_float2(0.f, 0.f) : row[BACK + r][k];
#pragma unroll
      for (int j = 0; j < TAPS; ++j) {
        float2 v = row[r + j][k];
        if (i < BACK - j)  // before the step's first token of the sequence
          v = c < n && slot >= 0 ? Pair<float>::load(state + ((size_t)slot * BACK + i + j) * channels + c0 + c) : make_float2(0.f, 0.f);
        u[k].x = fmaf(w[j][k].x, v.x, u[k].x);
        u[k].y = fmaf(w[j][k].y, v.y, u[k].y);
      }
      ss = fmaf(u[k].x, u[k].x, fmaf(u[k].y, u[k].y, ss));
    }
    T* dst = nullptr;
    if (is_q) {
      dst = q_out + ((size_t)t * H + head) * d;
    } else if (write_cache && s_page[r] >= 0) {
      T* page = cache + s_page[r] * page_stride;
      dst = is_v ? page + (size_t)G * page_size * d + ((size_t)(head - H - G) * page_size + s_off[r]) * dv
                 : page + ((size_t)(head - H) * page_size + s_off[r]) * d;
    }
    if (is_v) {
#pragma unroll
      for (int k = 0; k < NCH; ++k) {
        const int c = 2 * lane + 64 * k;
        if (c < n && dst != nullptr) Pair<T>::store(dst + c, u[k]);
      }
      continue;
    }
    const float inv = (is_q ? q_scale : 1.0f) / sqrtf(warp_sum(ss) / (float)d + eps);
    const float* cs = prep_smem + 2 * r * half;
#pragma unroll
    for (int k = 0; k < NCH; ++k) {
      u[k].x *= inv * scale[k].x;
      u[k].y *= inv * scale[k].y;
      const int c = 2 * lane + 64 * k;
      if (!interleaved && c < rot_dims) Pair<float>::store(buf + c, u[k]);
    }
    __syncwarp();
#pragma unroll
    for (int k = 0; k < NCH; ++k) {
      const int c = 2 * lane + 64 * k;
      if (c >= n) continue;
      float2 v = u[k];
      if (c < rot_dims) {
        if (interleaved) {
          const float cc = cs[c >> 1], sn = cs[half + (c >> 1)];
          v = make_float2(u[k].x * cc - u[k].y * sn, u[k].y * cc + u[k].x * sn);
        } else {
          const bool low = c < half;
          const int a = low ? c : c - half;
          const float2 o = Pair<float>::load(buf + (low ? c + half : a));
          const float2 cc = Pair<float>::load(cs + a), sn = Pair<float>::load(cs + half + a);
          v = low ? make_float2(v.x * cc.x - o.x * sn.x, v.y * cc.y - o.y * sn.y)
                  : make_float2(v.x * cc.x + o.x * sn.x, v.y * cc.y + o.y * sn.y);
        }
      }
      if (dst != nullptr) Pair<T>::store(dst + c, v);
    }
    __syncwarp();  // the row in shared memory is read before the next token's
  }
}

extern "C" int sb_conv_headnorm_store(const void* proj, int row_width, int dtype, const float* conv_w, int taps, float* state,
                                      const int* slots, int num_slots, int num_seqs, int alone, const float* q_norm,
                                      const float* k_norm, float eps, float q_scale, const float* rot_freq, int rot_dims,
                                      int interleaved, void* q_out, void* cache, const int* block_table, int max_pages,
                                      const int* token_seq, const int* cu_q, const int* positions, int num_tokens, int H,
                                      int G, int d, int dv, int page_size, int num_pages, int write_cache, int* err,
                                      cudaStream_t stream) {
  if (num_tokens == 0) return 0;
  if (rot_freq == nullptr) rot_dims = 0;
  if (rot_dims % 2 || rot_dims > d) return -4;
  if (taps < 0 || (taps > 1 && state == nullptr) || G <= 0 || H % G) return -13;
  const int rows = num_tokens >= 1024 ? 4 : 1;
  const dim3 grid((unsigned)((num_tokens + rows - 1) / rows), (unsigned)((H + 2 * G + PREP_WARPS - 1) / PREP_WARPS));
  const size_t smem = ((size_t)rows * rot_dims + (size_t)PREP_WARPS * (d > dv ? d : dv)) * sizeof(float);
  if (smem > 200 * 1024 || grid.y > 65535) return -2;
  // (in the activation dtype's pairs: rows, heads and the turned halves start on whole pairs)
  const bool pairs = !alone && taps != 1 && taps <= 4 && d % 2 == 0 && dv % 2 == 0 && row_width % 2 == 0 &&
                     (interleaved || rot_dims % 4 == 0) && d <= 256 && dv <= 256;
  const int widest = d > dv ? d : dv;
#define SB_PAIRS(T_, TAPS_, NCH_)                                                                                      \
  do {                                                                                                                 \
    if (rows == 4) SB_PAIRS_ROWS(T_, TAPS_, NCH_, 4); else SB_PAIRS_ROWS(T_, TAPS_, NCH_, 1);                          \
  } while (0)
#define SB_PAIRS_ROWS(T_, TAPS_, NCH_, ROWS_)                                                                                      \
  do {                                                                                                                 \
    auto k = conv_headnorm_store_pairs_kernel<T_, TAPS_, NCH_, ROWS_>;                                                        \
    sb_launch(k, grid, PREP_WARPS * 32, smem, stream, (const T_*)proj, row_width, conv_w, (const float*)state, slots,  \
              num_slots, q_norm, k_norm, eps, q_scale, rot_freq, rot_dims, interleaved, (T_*)q_out, (T_*)cache,        \
              block_table, max_pages, token_seq, cu_q, positions, num_tokens, H, G, d, dv, page_size, num_pages,       \
              write_cache, err);                                                                                       \
  } while (0)
#define SB_PAIRS_OF(T_, TAPS_)                          \
  do {                                                  \
    if (widest <= 64) SB_PAIRS(T_, TAPS_, 1);           \
    else if (widest <= 128) SB_PAIRS(T_, TAPS_, 2);     \
    else SB_PAIRS(T_, TAPS_, 4);                        \
  } while (0)
#define SB_PAIRS_ANY(T_)                          \
  switch (taps) {                                 \
    case 0: SB_PAIRS_OF(T_, 0); break;            \
    case 2: SB_PAIRS_OF(T_, 2); break;            \
    case 3: SB_PAIRS_OF(T_, 3); break;            \
    default: SB_PAIRS_OF(T_, 4);                  \
  }
  if (pairs && smem <= 48 * 1024) {
    if (dtype == SB_DTYPE_F32) {
      SB_PAIRS_ANY(float)
    } else {
      SB_PAIRS_ANY(bf16)
    }
    SB_LAUNCH_CHECK();
    return 0;
  }
#undef SB_PAIRS_ANY
#undef SB_PAIRS_OF
#undef SB_PAIRS
#undef SB_PAIRS_ROWS
#define SB_PREP2(T_, TAPS_)                                                                                          \
  do {                                                                                                               \
    auto k = conv_headnorm_store_kernel<T_, TAPS_>;                                                                  \
    if (smem > 48 * 1024) cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);           \
    sb_launch(k, grid, PREP_WARPS * 32, smem, stream, (const T_*)proj, row_width, conv_w, taps, state, slots,        \
              num_slots, num_seqs, alone, q_norm, k_norm, eps, q_scale, rot_freq, rot_dims, interleaved, (T_*)q_out, \
              (T_*)cache, block_table, max_pages, token_seq, cu_q, positions, num_tokens, rows, H, G, d, dv,         \
              page_size, num_pages, write_cache, err);                                                               \
  } while (0)
#define SB_PREP(T_)                  \
  switch (taps) {                    \
    case 0: SB_PREP2(T_, 0); break;  \
    case 2: SB_PREP2(T_, 2); break;  \
    case 3: SB_PREP2(T_, 3); break;  \
    case 4: SB_PREP2(T_, 4); break;  \
    default: SB_PREP2(T_, -1);       \
  }
  if (dtype == SB_DTYPE_F32) {
    SB_PREP(float)
  } else {
    SB_PREP(bf16)
  }
#undef SB_PREP
#undef SB_PREP2
  SB_LAUNCH_CHECK();
  return 0;
}

// ---------------------------------------------------------------------------
// Output gate: x[t, c] *= sigmoid(gate[t, c]), the gate read from a wider row (a column range of
// the fused projection).
// ---------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256)
sigmoid_gate_kernel(T* __restrict__ x, const T* __restrict__ gate, int gate_width, int width, int per) {
  pdl_wait_block();
  pdl_launch_dependents();
  const int t = blockIdx.y;
  for (int c = blockIdx.x * blockDim.x + threadIdx.x; c < width; c += gridDim.x * blockDim.x) {
    const float g = to_f32<T>(gate[(size_t)t * gate_width + c / per]);  // one gate per `per` neighbours
    const size_t at = (size_t)t * width + c;
    x[at] = from_f32<T>(to_f32<T>(x[at]) / (1.0f + expf(-g)));
  }
}

extern "C" int sb_sigmoid_gate(void* x, const void* gate, int gate_width, int dtype, int num_tokens, int width,
                               int per, cudaStream_t stream) {
  if (num_tokens == 0 || width == 0) return 0;
  if (per < 1) return -13;
  for (int t0 = 0; t0 < num_tokens; t0 += 65535) {
    const dim3 grid((unsigned)min((width + 255) / 256, 64), (unsigned)min(65535, num_tokens - t0));
    if (dtype == SB_DTYPE_F32)
      sb_launch(sigmoid_gate_kernel<float>, grid, 256, 0, stream, (float*)x + (size_t)t0 * width,
                (const float*)gate + (size_t)t0 * gate_width, gate_width, width, per);
    else
      sb_launch(sigmoid_gate_kernel<bf16>, grid, 256, 0, stream, (bf16*)x + (size_t)t0 * width,
                (const bf16*)gate + (size_t)t0 * gate_width, gate_width, width, per);
  }
  SB_LAUNCH_CHECK();
  return 0;
}
