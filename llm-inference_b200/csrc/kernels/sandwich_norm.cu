// Row kernels of layers with a norm on either side of each sublayer: x <- x + mult * norm_b(branch(norm_a(x))).
//
// `sandwich_norm`, one block per row, everything in 32-bit. What stands between two sublayers is one kernel: the finished
// branch d (one output, or a weighted pair a_scale * a + b_scale * b plus a constant per column) is divided by its root mean
// square, weighted and added to the stream, x <- x + mult * w_b * d / rms(d); the new row is divided by its own root mean
// square and weighted, h = w_a * x / rms(x), which is the next sublayer's input (or, for gathered rows, the output head's).
// The root mean square is sqrt(mean(v^2) + eps). Either half may be absent (no branch yet: the first layer).
//
// A layer may blend what its mixer reads with the previous token's row, h_t <- h_t + (h_(t-1) - h_t) * shift per column, the
// h on the right being the unblended ones; a request's last h lives in its state slot (32-bit, zeros after admission).
// SHIFT_SINGLE is for steps in which every request feeds one token: the blend reads the slot and writes the new h to it, in
// the same kernel. In other steps a token's neighbour is another block's row: SHIFT_DEFER stops after the stream, leaves
// 1 / rms(x) per row and copies the slots of the step's requests aside, and `shift_norm` forms h_t and h_(t-1) from the
// stream's rows, blends them and moves the slots on. Both ways round the blend once, at the end.
#include "common.cuh"
#include "packs.cuh"

namespace {

enum : int { SHIFT_NONE = 0, SHIFT_SINGLE = 1, SHIFT_DEFER = 2 };

struct SandwichParams {
  float* x;                // [tokens][hidden]; rows[r] (or r) is the row read, written back unless `rows` is given
  const void* a;           // branch output, or null
  const void* b;           // second output of a pair, or null
  float a_scale, b_scale;
  const float* constant;   // [hidden] added to the combined output, or null
  const float* branch_weight;  // [hidden]
  float mult, branch_eps;
  const float* weight;     // [hidden] of the norm whose output is `out`
  float eps;
  const int* rows;
  int hidden;
  void* out;               // [rows][hidden]
  const float* shift;      // [hidden]
  float* slots;            // [slots][hidden]
  const int* token_seq;
  const int* seq_q_start;
  const int* seq_slot;
  float* rstd_out;         // [tokens], SHIFT_DEFER
  float* previous;         // [requests][hidden], SHIFT_DEFER: the slots as they were before the step
};

// PER packs of W numbers a thread, in registers; PER = 0: any row length, the row in shared memory.
template <typename T, int W, int PER, int SHIFT>
__global__ void sandwich_norm_kernel(const SandwichParams p) {
  using P = Pack<W>;
  using V = typename P::type;
  constexpr bool kInSmem = PER == 0;
  extern __shared__ __align__(16) unsigned char row_smem[];
  V* row = reinterpret_cast<V*>(row_smem);
  __shared__ float scratch[32];
  let_successor_start();
  const int r = blockIdx.x, tid = threadIdx.x, stride = blockDim.x;
  const int packs = p.hidden / W;
  V held[kInSmem ? 1 : PER];
  auto each = [&](auto&& body) {  // body(slot, pack index): this thread's packs
    if constexpr (kInSmem) {
      for (int i = tid; i < packs; i += stride) body(row[i], i);
    } else {
#pragma unroll
      for (int j = 0; j < PER; ++j) {
        const int i = tid + j * stride;
        if (i < packs) body(held[j], i);
      }
    }
  };
  const int src = p.rows ? p.rows[r] : r;  // step metadata: on the device before the step began
  wait_for_predecessor();
  float* x = p.x + static_cast<int64_t>(src) * p.hidden;
  const float inv_width = 1.f / static_cast<float>(p.hidden);
  float ss = 0.f;
  if (p.a != nullptr) {
    const T* a = static_cast<const T*>(p.a) + static_cast<int64_t>(src) * p.hidden;
    const T* b = p.b ? static_cast<const T*>(p.b) + static_cast<int64_t>(src) * p.hidden : nullptr;
    float ds = 0.f;
    each([&](V& v, int i) {
      V d = P::load(a + i * W);
      if (b) {
        d = scale_each(d, p.a_scale);
        d = add_each(d, scale_each(P::load(b + i * W), p.b_scale));
      }
      if (p.constant) d = add_each(d, P::load(p.constant + i * W));
      v = d;
      ds = square_sum(d, ds);
    });
    ds = block_sum(ds, scratch);
    const float factor = p.mult / sqrtf(ds * inv_width + p.branch_eps);
    each([&](V& v, int i) {
      const V sum = fma_each(scale_each(v, factor), P::load(p.branch_weight + i * W), P::load(x + i * W));
      if (!p.rows) P::store(x + i * W, sum);
      v = sum;
      ss = square_sum(sum, ss);
    });
  } else {
    each([&](V& v, int i) {
      v = P::load(x + i * W);
      ss = square_sum(v, ss);
    });
  }
  ss = block_sum(ss, scratch);
  const float rstd = 1.f / sqrtf(ss * inv_width + p.eps);
  if constexpr (SHIFT == SHIFT_DEFER) {
    if (tid == 0) p.rstd_out[r] = rstd;
    const int seq = p.token_seq[r];
    if (p.seq_q_start[seq] == r) {
      const float* slot = p.slots + static_cast<int64_t>(p.seq_slot[seq]) * p.hidden;
      float* aside = p.previous + static_cast<int64_t>(seq) * p.hidden;
      for (int i = tid; i < packs; i += stride) P::store(aside + i * W, P::load(slot + i * W));
    }
    return;
  }
  T* out = static_cast<T*>(p.out) + static_cast<int64_t>(r) * p.hidden;
  float* slot = SHIFT == SHIFT_SINGLE ? p.slots + static_cast<int64_t>(p.seq_slot[p.token_seq[r]]) * p.hidden : nullptr;
  each([&](V& v, int i) {
    V h = mul_each(scale_each(v, rstd), P::load(p.weight + i * W));
    if constexpr (SHIFT == SHIFT_SINGLE) {
      const V before = P::load(slot + i * W);
      P::store(slot + i * W, h);
      h = fma_each(sub_each(before, h), P::load(p.shift + i * W), h);
    }
    P::store(out + i * W, h);
  });
}

// out[t] = h_t + (h_(t-1) - h_t) * blend with h = weight * x * rstd; a request's first token of the step takes `previous`
// for h_(t-1), its last one leaves h_t in the slot.
template <typename T, int W>
__global__ void shift_norm_kernel(const float* x, const float* rstd, const float* __restrict__ weight, const float* __restrict__ blend,
                                  const float* previous, float* slots, const int* __restrict__ token_seq, const int* __restrict__ seq_q_start,
                                  const int* __restrict__ seq_q_len, const int* __restrict__ seq_slot, int hidden, T* out) {
  using P = Pack<W>;
  using V = typename P::type;
  let_successor_start();
  const int t = blockIdx.x;
  const int seq = token_seq[t];
  const int start = seq_q_start[seq];
  const bool first = t == start, last = t == start + seq_q_len[seq] - 1;
  float* slot = slots + static_cast<int64_t>(seq_slot[seq]) * hidden;
  const float* cur = x + static_cast<int64_t>(t) * hidden;
  const float* aside = previous + static_cast<int64_t>(seq) * hidden;
  wait_for_predecessor();
  const float rs = rstd[t], rs_before = first ? 0.f : rstd[t - 1];
  for (int i = threadIdx.x; i < hidden / W; i += blockDim.x) {
    const V w = P::load(weight + i * W);
    const V h = mul_each(scale_each(P::load(cur + i * W), rs), w);
    const V before = first ? P::load(aside + i * W) : mul_each(scale_each(P::load(cur - hidden + i * W), rs_before), w);
    P::store(out + static_cast<int64_t>(t) * hidden + i * W, fma_each(sub_each(before, h), P::load(blend + i * W), h));
    if (last) P::store(slot + i * W, h);
  }
}

template <typename T, int W, int PER, int SHIFT>
void launch_sandwich(const SandwichParams& p, int count, int threads, cudaStream_t stream) {
  const size_t smem = PER == 0 ? sizeof(float) * p.hidden : 0;
  if (smem > 48 * 1024)
    cudaFuncSetAttribute(sandwich_norm_kernel<T, W, PER, SHIFT>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  launch_kernel(sandwich_norm_kernel<T, W, PER, SHIFT>, dim3(count), dim3(threads), smem, stream, p);
}

template <typename T, int SHIFT>
void sandwich_by_width(const SandwichParams& p, int count, bool wide, cudaStream_t stream) {
  // Whole warps, at most `per` packs of four a thread.
  auto threads_for = [&](int per) { return ((p.hidden / 4 + per - 1) / per + 31) / 32 * 32; };
  if (wide && p.hidden <= 1024) {
    launch_sandwich<T, 4, 1, SHIFT>(p, count, threads_for(1), stream);
  } else if (wide && p.hidden <= 4096) {
    launch_sandwich<T, 4, 2, SHIFT>(p, count, threads_for(2), stream);
  } else if (wide && p.hidden <= 8192) {
    launch_sandwich<T, 4, 4, SHIFT>(p, count, threads_for(4), stream);
  } else if (wide) {
    launch_sandwich<T, 4, 0, SHIFT>(p, count, 512, stream);
  } else {
    launch_sandwich<T, 1, 0, SHIFT>(p, count, p.hidden >= 1024 ? 256 : 128, stream);
  }
}

template <typename T>
void sandwich_by_mode(const SandwichParams& p, int count, bool wide, int mode, cudaStream_t stream) {
  if (mode == SHIFT_SINGLE) sandwich_by_width<T, SHIFT_SINGLE>(p, count, wide, stream);
  else if (mode == SHIFT_DEFER) sandwich_by_width<T, SHIFT_DEFER>(p, count, wide, stream);
  else sandwich_by_width<T, SHIFT_NONE>(p, count, wide, stream);
}

}  // namespace

// mode: SHIFT_NONE, SHIFT_SINGLE (slots: [slots][hidden], one token per request) or SHIFT_DEFER (`previous`
// [requests][hidden] and `rstd_out` [tokens] are written for `shift_norm`; `out` is not).
B200_API int b200_sandwich_norm(float* x, const void* a, const void* b, float a_scale, float b_scale, const float* constant,
                                const float* branch_weight, float mult, float branch_eps, const float* weight, float eps, const int* rows,
                                int count, int hidden, void* out, int mode, const float* shift, float* slots, const int* token_seq,
                                const int* seq_q_start, const int* seq_slot, float* rstd_out, float* previous, int dtype,
                                cudaStream_t stream) {
  if (count == 0) return 0;
  B200_REQUIRE(count > 0 && hidden > 0 && x != nullptr && weight != nullptr, "sandwich_norm: bad sizes");
  B200_REQUIRE(hidden * sizeof(float) <= 200 * 1024, "sandwich_norm: rows of %d numbers do not fit one block", hidden);
  B200_REQUIRE(a == nullptr || branch_weight != nullptr, "sandwich_norm: a branch comes with its norm's weight");
  B200_REQUIRE(mode == SHIFT_NONE || (rows == nullptr && slots != nullptr && token_seq != nullptr && seq_slot != nullptr),
               "sandwich_norm: a blend with the previous token wants state slots and the whole step");
  B200_REQUIRE(mode != SHIFT_SINGLE || shift != nullptr, "sandwich_norm: no blend factors");
  B200_REQUIRE(mode != SHIFT_DEFER || (rstd_out != nullptr && previous != nullptr && seq_q_start != nullptr), "sandwich_norm: nowhere to leave the row's statistics");
  B200_REQUIRE(mode == SHIFT_DEFER || out != nullptr, "sandwich_norm: no output");
  SandwichParams p{x, a, b, a_scale, b_scale, constant, branch_weight, mult, branch_eps, weight, eps, rows, hidden, out,
                   shift, slots, token_seq, seq_q_start, seq_slot, rstd_out, previous};
  const bool wide = packs_of_four(hidden, x, a, b, constant, branch_weight, weight, out, shift, slots, previous);
  if (dtype == DTYPE_F32) sandwich_by_mode<float>(p, count, wide, mode, stream);
  else if (dtype == DTYPE_BF16) sandwich_by_mode<__nv_bfloat16>(p, count, wide, mode, stream);
  else return b200_fail("sandwich_norm: unknown dtype %d", dtype);
  return b200_check_launch("sandwich_norm");
}

B200_API int b200_shift_norm(const float* x, const float* rstd, const float* weight, const float* shift, const float* previous, float* slots,
                             const int* token_seq, const int* seq_q_start, const int* seq_q_len, const int* seq_slot, int tokens, int hidden,
                             void* out, int dtype, cudaStream_t stream) {
  if (tokens == 0) return 0;
  B200_REQUIRE(tokens > 0 && hidden > 0, "shift_norm: bad sizes");
  const bool wide = packs_of_four(hidden, x, weight, shift, previous, slots, out);
  auto launch = [&](auto kernel, auto* typed) {
    const int packs = wide ? hidden / 4 : hidden;
    const int threads = packs >= 256 ? 256 : (packs + 31) / 32 * 32;
    launch_kernel(kernel, dim3(tokens), dim3(threads), 0, stream, x, rstd, weight, shift, previous, slots, token_seq, seq_q_start, seq_q_len,
                  seq_slot, hidden, typed);
  };
  if (dtype == DTYPE_F32) {
    if (wide) launch(shift_norm_kernel<float, 4>, static_cast<float*>(out));
    else launch(shift_norm_kernel<float, 1>, static_cast<float*>(out));
  } else if (dtype == DTYPE_BF16) {
    if (wide) launch(shift_norm_kernel<__nv_bfloat16, 4>, static_cast<__nv_bfloat16*>(out));
    else launch(shift_norm_kernel<__nv_bfloat16, 1>, static_cast<__nv_bfloat16*>(out));
  } else {
    return b200_fail("shift_norm: unknown dtype %d", dtype);
  }
  return b200_check_launch("shift_norm");
}
