// Pending branches onto the residual stream, two RMS norms of the sum, and a shift towards the previous
// token, in one kernel.
//
//   x_t  = h_t + branch_t + branch2_t                        -> h_out (float32), where there is a branch
//   n_t  = x_t / sqrt(mean(x_t^2) + eps)
//   y_t  = n_t * (w1 [+ 1]),   y2_t = n_t' * (w2 [+ 1])      (n' with eps2)
//   out  = y_t + (y_(t-1) - y_t) * shift                     -> stored as T; y2_t likewise
//
// y_(t-1) of a request's first token of the step comes from `state` [slots, width] (float32), into which
// the y of its last token goes.  The stream is written to a buffer of its own, so that a block may read the
// row before its first one (whose y it computes once more) whatever other blocks have done; and the
// block that reads a request's old state also writes the new one (it computes the y of the request's
// last token for this), so no other kernel has to follow.  One block per ROWS tokens.
#include "common.cuh"

#define SB_ERR_BAD_SLOT 16

struct TwoNorms {
  const float* h;
  float* h_out;  // null: there is no branch
  const void* branch;
  const void* branch2;
  const void* w1;
  const void* w2;  // null: one norm
  int w1_f32, w2_f32;
  float eps1, eps2, one1, one2;
  const float* shift;  // null: no shift
  float* state;
  int num_slots, num_seqs, num_tokens, width;
  const int *token_seq, *cu_q, *slots;
  void* y;
  void* y2;
  int* err;
};

// Sums of M values over the block, in the same order whatever M is; `scratch`: M * 32 floats.
template <int M>
__device__ __forceinline__ void block_sums(float (&v)[M], float* scratch) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
#pragma unroll
  for (int m = 0; m < M; ++m) v[m] = warp_sum(v[m]);
  __syncthreads();
  if (lane == 0) {
#pragma unroll
    for (int m = 0; m < M; ++m) scratch[m * 32 + warp] = v[m];
  }
  __syncthreads();
#pragma unroll
  for (int m = 0; m < M; ++m) {
    float s = 0.f;
    for (int w = 0; w < nwarps; ++w) s += scratch[m * 32 + w];
    v[m] = s;
  }
}

// Rows of one 16-byte vector per thread: everything a block needs is loaded before its first sum.  ROWS 1 is
// the kernel of short steps: there the weights, the request's place and its old row are fetched ahead as
// well.  Larger ROWS keep the registers low, so that one block's sums and stores overlap another's loads.
template <typename T, int ROWS, int MAX_THREADS>
__global__ void __launch_bounds__(MAX_THREADS, ROWS == 1 ? 1 : 2) two_norms_kernel(const TwoNorms p) {
  constexpr int N = Vec<T>::N;
  constexpr bool AHEAD = ROWS == 1;
  __shared__ float scratch[(ROWS + 1) * 32];
  const int i = threadIdx.x * N;
  const bool on = i < p.width;
  float w1[N], w2[N], sh[N];
  auto load_weights = [&]() {
#pragma unroll
    for (int k = 0; k < N; ++k) w1[k] = w2[k] = sh[k] = 0.f;
    if (on) {
      load_scalars<N>(p.w1, p.w1_f32, i, w1);
      if (p.w2 != nullptr) load_scalars<N>(p.w2, p.w2_f32, i, w2);
      if (p.shift != nullptr) load_scalars<N>(p.shift, 1, i, sh);
    }
#pragma unroll
    for (int k = 0; k < N; ++k) {
      w1[k] += p.one1;
      w2[k] += p.one2;
    }
  };
  if constexpr (AHEAD) load_weights();  // (no kernel writes them: before the wait)
  pdl_wait_block();
  pdl_launch_dependents();
  const float inv_width = 1.0f / (float)p.width;
  auto load_row = [&](int t, float (&v)[N]) {
#pragma unroll
    for (int k = 0; k < N; ++k) v[k] = 0.f;
    if (!on || t < 0 || t >= p.num_tokens) return;
    const size_t at = (size_t)t * p.width + i;
#pragma unroll
    for (int k = 0; k < N; k += 4) Vec<float>::load(p.h + at + k, v + k);
    float b[N];
    if (p.branch != nullptr) {
      Vec<T>::load(reinterpret_cast<const T*>(p.branch) + at, b);
#pragma unroll
      for (int k = 0; k < N; ++k) v[k] += b[k];
    }
    if (p.branch2 != nullptr) {
      Vec<T>::load(reinterpret_cast<const T*>(p.branch2) + at, b);
#pragma unroll
      for (int k = 0; k < N; ++k) v[k] += b[k];
    }
  };
  const int t0 = blockIdx.x * ROWS;
  // Row m is token t0 - 1 + m.  (Without a shift row 0 is not needed.)
  float x[ROWS + 1][N], sums[ROWS + 1];
#pragma unroll
  for (int m = 0; m <= ROWS; ++m) load_row(p.shift != nullptr || m > 0 ? t0 - 1 + m : -1, x[m]);
  // The request of every row, and for a request's first token the row's part of the state.
  int first[ROWS], last[ROWS], slot[ROWS], copies[ROWS];
  float old[AHEAD ? N : 1];
#pragma unroll
  for (int m = 0; m < ROWS; ++m) {
    const int t = t0 + m;
    first[m] = -1;
    last[m] = t;
    slot[m] = 0;
    copies[m] = 1;
    if (p.shift != nullptr && t < p.num_tokens) {
      const int b = p.token_seq[t];
      first[m] = p.cu_q[b];
      if (first[m] == t) {
        last[m] = p.cu_q[b + 1] - 1;
        slot[m] = p.slots[b];
        if (slot[m] < 0 || slot[m] >= p.num_slots) {
          if (threadIdx.x == 0) atomicOr(p.err, SB_ERR_BAD_SLOT);
          copies[m] = 0;
        } else {
          copies[m] = rows_sharing_slot(p.slots, b, p.num_seqs);  // 0: an earlier row of the slot writes this one's results
        }
        if constexpr (AHEAD) {
#pragma unroll
          for (int k = 0; k < N; ++k) old[k] = 0.f;
          if (on && copies[m] > 0) {
#pragma unroll
            for (int k = 0; k < N; k += 4) Vec<float>::load(p.state + (size_t)slot[m] * p.width + i + k, old + k);
          }
        }
      }
    }
  }
#pragma unroll
  for (int m = 0; m <= ROWS; ++m) {
    sums[m] = 0.f;
#pragma unroll
    for (int k = 0; k < N; ++k) sums[m] = fmaf(x[m][k], x[m][k], sums[m]);
  }
  block_sums<ROWS + 1>(sums, scratch);
  if constexpr (!AHEAD) load_weights();
#pragma unroll
  for (int m = 1; m <= ROWS; ++m) {
    const int t = t0 - 1 + m;
    if (t >= p.num_tokens) break;
    if (copies[m - 1] == 0) continue;
    const float mean = sums[m] * inv_width;
    const float r1 = 1.0f / sqrtf(mean + p.eps1);
    const bool starts = first[m - 1] == t;  // (the same for the whole block)
    float out[N];
    if (starts) {
      float* st = p.state + (size_t)slot[m - 1] * p.width + i;
#pragma unroll
      for (int k = 0; k < N; ++k) out[k] = 0.f;
      if constexpr (AHEAD) {
#pragma unroll
        for (int k = 0; k < N; ++k) out[k] = old[k];
      } else if (on) {
#pragma unroll
        for (int k = 0; k < N; k += 4) Vec<float>::load(st + k, out + k);
      }
      float z[N], rl = r1;
#pragma unroll
      for (int k = 0; k < N; ++k) z[k] = x[m][k];
      if (last[m - 1] != t) {
        float s[1] = {0.f};
        load_row(last[m - 1], z);
#pragma unroll
        for (int k = 0; k < N; ++k) s[0] = fmaf(z[k], z[k], s[0]);
        block_sums<1>(s, scratch);
        rl = 1.0f / sqrtf(s[0] * inv_width + p.eps1);
      }
#pragma unroll
      for (int k = 0; k < N; ++k) z[k] *= rl * w1[k];
      if (on) {
#pragma unroll
        for (int k = 0; k < N; k += 4) Vec<float>::store(st + k, z + k);
      }
    } else {
      const float rp = 1.0f / sqrtf(sums[m - 1] * inv_width + p.eps1);
#pragma unroll
      for (int k = 0; k < N; ++k) out[k] = x[m - 1][k] * rp * w1[k];
    }
    if (!on) continue;
#pragma unroll
    for (int k = 0; k < N; ++k) {
      const float y = x[m][k] * r1 * w1[k];
      out[k] = fmaf(out[k] - y, sh[k], y);  // (without a shift its factors are zero)
    }
    const float r2 = p.eps2 == p.eps1 ? r1 : 1.0f / sqrtf(mean + p.eps2);
    for (int c = 0; c < copies[m - 1]; ++c) {  // (rows that repeat a request follow it)
      const size_t at = (size_t)(t + c) * p.width + i;
      if (p.h_out != nullptr) {
#pragma unroll
        for (int k = 0; k < N; k += 4) Vec<float>::store(p.h_out + at + k, x[m] + k);
      }
      Vec<T>::store(reinterpret_cast<T*>(p.y) + at, out);
      if (p.w2 != nullptr) {
        float y2[N];
#pragma unroll
        for (int k = 0; k < N; ++k) y2[k] = x[m][k] * r2 * w2[k];
        Vec<T>::store(reinterpret_cast<T*>(p.y2) + at, y2);
      }
    }
  }
}

// Any width: one block per token, channels in turn, the stream's row read once per use.
template <typename T>
__global__ void __launch_bounds__(256) two_norms_wide_kernel(const TwoNorms p) {
  __shared__ float scratch[32];
  pdl_wait_block();
  pdl_launch_dependents();
  auto value = [&](int t, int c) {
    const size_t at = (size_t)t * p.width + c;
    float v = p.h[at];
    if (p.branch != nullptr) v += to_f32<T>(reinterpret_cast<const T*>(p.branch)[at]);
    if (p.branch2 != nullptr) v += to_f32<T>(reinterpret_cast<const T*>(p.branch2)[at]);
    return v;
  };
  auto mean_square = [&](int t) {
    float s[1] = {0.f};
    for (int c = threadIdx.x; c < p.width; c += blockDim.x) {
      const float v = value(t, c);
      s[0] = fmaf(v, v, s[0]);
    }
    block_sums<1>(s, scratch);
    return s[0] / (float)p.width;
  };
  const int t = blockIdx.x;
  const float mean = mean_square(t);
  const float r1 = 1.0f / sqrtf(mean + p.eps1), r2 = 1.0f / sqrtf(mean + p.eps2);
  int copies = 1, last = t;
  float rp = 0.f, rl = 0.f;
  float* st = nullptr;
  bool from_state = false;
  if (p.shift != nullptr) {
    const int b = p.token_seq[t], first = p.cu_q[b];
    last = p.cu_q[b + 1] - 1;
    if (t > first) {
      rp = 1.0f / sqrtf(mean_square(t - 1) + p.eps1);
    } else {
      from_state = true;
      const int slot = p.slots[b];
      if (slot < 0 || slot >= p.num_slots) {
        if (threadIdx.x == 0) atomicOr(p.err, SB_ERR_BAD_SLOT);
        return;
      }
      copies = rows_sharing_slot(p.slots, b, p.num_seqs);
      if (copies == 0) return;
      st = p.state + (size_t)slot * p.width;
      rl = last == t ? r1 : 1.0f / sqrtf(mean_square(last) + p.eps1);
    }
  }
  for (int c = threadIdx.x; c < p.width; c += blockDim.x) {
    const float x = value(t, c), w1 = load_scalar(p.w1, p.w1_f32, c) + p.one1;
    float out = x * r1 * w1;
    if (p.shift != nullptr) {
      float before;
      if (from_state) {
        before = st[c];
        st[c] = value(last, c) * rl * w1;
      } else {
        before = value(t - 1, c) * rp * w1;
      }
      out = fmaf(before - out, p.shift[c], out);
    }
    const float y2 = p.w2 != nullptr ? x * r2 * (load_scalar(p.w2, p.w2_f32, c) + p.one2) : 0.f;
    for (int k = 0; k < copies; ++k) {
      const size_t at = (size_t)(t + k) * p.width + c;
      if (p.h_out != nullptr) p.h_out[at] = x;
      reinterpret_cast<T*>(p.y)[at] = from_f32<T>(out);
      if (p.w2 != nullptr) reinterpret_cast<T*>(p.y2)[at] = from_f32<T>(y2);
    }
  }
}

extern "C" int sb_residual_two_norms(const float* h, float* h_out, const void* branch, const void* branch2, int dtype,
                                     const void* w1, int w1_f32, float eps1, int one1, const void* w2, int w2_f32,
                                     float eps2, int one2, const float* shift, float* state, int num_slots,
                                     const int* token_seq, const int* cu_q, const int* slots, int num_seqs,
                                     int num_tokens, int width, void* y, void* y2, int rows_per_block, int* err,
                                     cudaStream_t stream) {
  if (num_tokens == 0) return 0;
  if ((branch2 != nullptr && branch == nullptr) || (branch != nullptr) != (h_out != nullptr)) return -3;
  if (shift != nullptr && state == nullptr) return -13;
  TwoNorms p{h, h_out, branch, branch2, w1, w2, w1_f32, w2_f32, eps1, eps2, one1 ? 1.f : 0.f, one2 ? 1.f : 0.f, shift,
             state, num_slots, num_seqs, num_tokens, width, token_seq, cu_q, slots, y, y2, err};
  const int vec = dtype == SB_DTYPE_F32 ? 4 : 8;
  if (width % vec == 0 && width / vec <= 1024) {
    const int threads = ((width / vec + 31) / 32) * 32;
    // Many tokens: several per block, so that fewer rows are read once more for the token after them.
    // (Blocks of more than 512 threads keep to one row: their registers would not hold more.)
    int rows = rows_per_block > 0 ? rows_per_block : (num_tokens >= 512 && shift != nullptr ? 2 : 1);
    if (threads > 512) rows = 1;
#define SB_TWO_NORMS_OF(T_, R_, M_) \
  sb_launch(two_norms_kernel<T_, R_, M_>, (unsigned)((num_tokens + R_ - 1) / R_), threads, 0, stream, p)
#define SB_TWO_NORMS(T_, R_)                            \
  do {                                                  \
    if (threads > 512) SB_TWO_NORMS_OF(T_, 1, 1024);    \
    else SB_TWO_NORMS_OF(T_, R_, 512);                  \
  } while (0)
    if (dtype == SB_DTYPE_F32) {
      if (rows >= 3) SB_TWO_NORMS(float, 3); else if (rows == 2) SB_TWO_NORMS(float, 2); else SB_TWO_NORMS(float, 1);
    } else {
      if (rows >= 3) SB_TWO_NORMS(bf16, 3); else if (rows == 2) SB_TWO_NORMS(bf16, 2); else SB_TWO_NORMS(bf16, 1);
    }
#undef SB_TWO_NORMS
#undef SB_TWO_NORMS_OF
  } else if (dtype == SB_DTYPE_F32) {
    sb_launch(two_norms_wide_kernel<float>, num_tokens, 256, 0, stream, p);
  } else {
    sb_launch(two_norms_wide_kernel<bf16>, num_tokens, 256, 0, stream, p);
  }
  SB_LAUNCH_CHECK();
  return 0;
}
