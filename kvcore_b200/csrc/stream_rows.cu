// Kernels of a model that keeps a 32-bit residual stream and leaves a sub-layer's output to the norm behind it.
//
//   stream_add_rows: X = x + a per token, where a is a sub-layer's output row, the weighted sum of the rows that a
//   token's chosen experts left (ascending slot), one row for all tokens, or nothing.  From X, as asked: X itself (the new stream), its RMS norm
//   y = X * rsqrt(mean(X^2) + eps) * w in the activation type, and the row [X | x0] in the activation type (the
//   input of a product that reads the stream together with what it was at the start).  With a list of token rows
//   only those are worked on and the outputs are compact.  With a norm behind the sub-layer (`after`) it is
//   X = x + a * rsqrt(mean(a^2) + eps) * w_after (+ one row for all tokens, `step`); experts without tensors then add
//   their weight times the token's own input row.
//
//   embed_pairs: the first value of the stream, table[id] + pairs[row], with an RMS norm over the sum: row =
//   (id in front * mul_prev + id * mul_cur) mod buckets, or `buckets` (the row behind the last bucket) for a
//   request's first token.  The id in front of a portion is the request's state (one 32-bit word), which the block
//   of the portion's first token reads and brings up to date.
//
//   softcap: cap * tanh(logit * scale / cap), in place.
//
// One block per row; sums over a row follow its width only, so a row does not depend on the batch.
#include "common.cuh"

#define SR_THREADS 256
#define SR_PIECES 4            // pieces of N entries a thread keeps between the sum and the store

template <typename T, int N>
struct __align__(N * sizeof(T)) RowPiece { T v[N]; };

struct AddRowsParams {
  const float* x;                                    // [tokens, width]
  const void* rows; int top;                         // row of pair (token, slot): row_of_pair[pair], or pair itself
  const int* row_of_pair; const float* pair_weight;  // weights 1 without a list
  int one_row;                                       // every token's row is row 0
  // experts without tensors: a pair whose id is `identity_from` or more adds all_weight[pair] * input[token]
  const int* ids; int identity_from; const float* all_weight; const void* input;
  const void* after; float after_eps;                // AFTER: the weight of the norm that the sum of the rows gets
  const void* step;                                  // [width] or null: one row for all tokens, added behind that
  const int* token_rows;                             // tokens to work on, or null: all
  float* stream;                                     // [tokens, width] or null
  void* normed; const void* weight; float eps;       // [count, width] or null
  void* packed; const float* origin;                 // [count, 2 * width] or null
  int width;
};

// With a norm behind the sub-layer (AFTER) a row has two sums in a chain, which more threads with fewer pieces each
// shorten where there are few rows; many rows run better in blocks of 256.  So that a row's bits are the same either way,
// its sums are taken as if 1,024 threads had a piece each: one butterfly for every 32 of those, then one over the 32.
#define SR_VIRTUAL 1024
template <int THREADS, int PIECES>
__device__ __forceinline__ float virtual_sum(const float (&part)[PIECES], float* scratch) {
  static_assert(THREADS * PIECES == SR_VIRTUAL, "a thread stands for PIECES virtual ones");
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  float sums[PIECES];
#pragma unroll
  for (int s = 0; s < PIECES; ++s) sums[s] = warp_sum(part[s]);
  __syncthreads();
  if (lane == 0)
#pragma unroll
    for (int s = 0; s < PIECES; ++s) scratch[s * (THREADS / 32) + warp] = sums[s];
  __syncthreads();
  return warp_sum(scratch[lane]);
}

template <typename T, typename OUT, typename W, int N, bool AFTER, int THREADS>
__global__ void __launch_bounds__(THREADS, AFTER && THREADS == 256 ? 3 : 1)
stream_add_rows_kernel(const AddRowsParams p) {
  KVB_KERNEL_PROLOGUE(KVB_TAG_ADD_ROWS);
  constexpr int PIECES = AFTER ? SR_VIRTUAL / THREADS : SR_PIECES;
  __shared__ float scratch[32];
  const int n = blockIdx.x, t = p.token_rows != nullptr ? p.token_rows[n] : n;
  const int width = p.width;
  const float* x = p.x + (size_t)t * width;
  // the row and the weight of a slot of this token (null: none)
  auto slot_row = [&](int slot, float& w) -> const T* {
    const long long pair = (long long)t * p.top + slot;
    if (AFTER && p.ids != nullptr && p.ids[pair] >= p.identity_from) {
      w = p.all_weight[pair];
      return (const T*)p.input + (size_t)t * width;
    }
    w = p.pair_weight != nullptr ? p.pair_weight[pair] : 1.0f;
    const long long row = p.row_of_pair != nullptr ? (long long)p.row_of_pair[pair] : p.one_row ? 0ll : pair;
    return row < 0 ? nullptr : (const T*)p.rows + (size_t)row * width;
  };
  auto added = [&](int i, float (&a)[N]) {           // one piece of what is added: what the registers do not hold
#pragma unroll
    for (int j = 0; j < N; ++j) a[j] = 0.0f;
    for (int slot = 0; slot < p.top; ++slot) {
      float w;
      const T* row = slot_row(slot, w);
      if (row == nullptr) continue;
      const RowPiece<T, N> r = *reinterpret_cast<const RowPiece<T, N>*>(row + i);
#pragma unroll
      for (int j = 0; j < N; ++j) a[j] = fmaf(w, to_float(r.v[j]), a[j]);
    }
  };
  float kept[PIECES][N];
  float ss = 0.0f, inv_a = 1.0f;
  float parts[PIECES];                               // AFTER: the squares' sums of the virtual threads
#pragma unroll
  for (int s = 0; s < PIECES; ++s) parts[s] = 0.0f;
  // the new stream from what is added
  auto join = [&](int i, const RowPiece<float, N>& s, const RowPiece<W, N>& g, float (&v)[N]) {
    if (AFTER) {
#pragma unroll
      for (int j = 0; j < N; ++j) v[j] = s.v[j] + v[j] * inv_a * to_float(g.v[j]);
      if (p.step != nullptr) {
        const RowPiece<T, N> r = *reinterpret_cast<const RowPiece<T, N>*>((const T*)p.step + i);
#pragma unroll
        for (int j = 0; j < N; ++j) v[j] += to_float(r.v[j]);
      }
    } else {
#pragma unroll
      for (int j = 0; j < N; ++j) v[j] = s.v[j] + v[j];
    }
  };
  auto summed = [&](int i, float (&v)[N]) {          // one piece of the new stream, from the beginning
    added(i, v);
    RowPiece<W, N> g;
    if (AFTER) g = *reinterpret_cast<const RowPiece<W, N>*>((const W*)p.after + i);
    join(i, *reinterpret_cast<const RowPiece<float, N>*>(x + i), g, v);
  };
  auto first_pass = [&](int i, const float (&v)[N]) {
    if (p.stream != nullptr) {
      RowPiece<float, N> s;
#pragma unroll
      for (int j = 0; j < N; ++j) s.v[j] = v[j];
      *reinterpret_cast<RowPiece<float, N>*>(p.stream + (size_t)t * width + i) = s;
    }
    if (p.packed != nullptr) {
      RowPiece<OUT, N> now, start;
      const RowPiece<float, N> x0 = *reinterpret_cast<const RowPiece<float, N>*>(p.origin + (size_t)t * width + i);
#pragma unroll
      for (int j = 0; j < N; ++j) { now.v[j] = from_float<OUT>(v[j]); start.v[j] = from_float<OUT>(x0.v[j]); }
      OUT* dst = (OUT*)p.packed + (size_t)n * 2 * width + i;
      *reinterpret_cast<RowPiece<OUT, N>*>(dst) = now;
      *reinterpret_cast<RowPiece<OUT, N>*>(dst + width) = start;
    }
  };
  auto squares = [&](const float (&v)[N], float& sum) {
#pragma unroll
    for (int j = 0; j < N; ++j) sum = fmaf(v[j], v[j], sum);
  };
  // the kept pieces: the stream's, the weights' and a slot's loads are each in flight together
  RowPiece<float, N> xs[PIECES];
  RowPiece<W, N> ws[PIECES], gs[AFTER ? PIECES : 1];
#pragma unroll
  for (int s = 0; s < PIECES; ++s) {
    const int i = (threadIdx.x + s * THREADS) * N;
#pragma unroll
    for (int j = 0; j < N; ++j) kept[s][j] = 0.0f;
    if (i < width) {
      xs[s] = *reinterpret_cast<const RowPiece<float, N>*>(x + i);
      if (p.normed != nullptr) ws[s] = *reinterpret_cast<const RowPiece<W, N>*>((const W*)p.weight + i);
      if (AFTER) gs[s] = *reinterpret_cast<const RowPiece<W, N>*>((const W*)p.after + i);
    }
  }
#pragma unroll 2
  for (int slot = 0; slot < p.top; ++slot) {
    float w;
    const T* row = slot_row(slot, w);
    if (row == nullptr) continue;
    RowPiece<T, N> r[PIECES];
#pragma unroll
    for (int s = 0; s < PIECES; ++s) {
      const int i = (threadIdx.x + s * THREADS) * N;
      if (i < width) r[s] = *reinterpret_cast<const RowPiece<T, N>*>(row + i);
    }
#pragma unroll
    for (int s = 0; s < PIECES; ++s) {
      const int i = (threadIdx.x + s * THREADS) * N;
      if (i < width) {
#pragma unroll
        for (int j = 0; j < N; ++j) kept[s][j] = fmaf(w, to_float(r[s].v[j]), kept[s][j]);
      }
    }
  }
  const int rest = (threadIdx.x + PIECES * THREADS) * N;
  if constexpr (AFTER) {                             // the root mean square of what is added
    float sa[PIECES];
#pragma unroll
    for (int s = 0; s < PIECES; ++s) {               // (pieces beyond the width are zeros)
      sa[s] = 0.0f;
      squares(kept[s], sa[s]);
    }
    for (int i = rest, s = 0; i < width; i += THREADS * N, s = s + 1 < PIECES ? s + 1 : 0) {
      float a[N];
      added(i, a);
#pragma unroll
      for (int k = 0; k < PIECES; ++k)               // (an array indexed by a variable would leave the registers)
        if (k == s) squares(a, sa[k]);
    }
    inv_a = 1.0f / sqrtf(virtual_sum<THREADS, PIECES>(sa, scratch) / (float)width + p.after_eps);
  }
#pragma unroll
  for (int s = 0; s < PIECES; ++s) {
    const int i = (threadIdx.x + s * THREADS) * N;
    if (i < width) {
      join(i, xs[s], gs[AFTER ? s : 0], kept[s]);
      first_pass(i, kept[s]);
      squares(kept[s], AFTER ? parts[s] : ss);
    }
  }
  // rows wider than the registers hold: the sum goes through `stream`, which the same thread reads again
  for (int i = rest, s = 0; i < width; i += THREADS * N, s = s + 1 < PIECES ? s + 1 : 0) {
    float v[N];
    summed(i, v);
    first_pass(i, v);
    if (AFTER) {
#pragma unroll
      for (int k = 0; k < PIECES; ++k)
        if (k == s) squares(v, parts[k]);
    } else {
      squares(v, ss);
    }
  }
  if (p.normed == nullptr) return;
  float total;
  if constexpr (AFTER) total = virtual_sum<THREADS, PIECES>(parts, scratch);
  else total = block_sum(ss, scratch);
  const float inv = 1.0f / sqrtf(total / (float)width + p.eps);
  const W* weight = (const W*)p.weight;
  OUT* dst = (OUT*)p.normed + (size_t)n * width;
  auto put = [&](int i, const float (&v)[N], const RowPiece<W, N>& w) {
    RowPiece<OUT, N> r;
#pragma unroll
    for (int j = 0; j < N; ++j) r.v[j] = from_float<OUT>(v[j] * inv * to_float(w.v[j]));
    *reinterpret_cast<RowPiece<OUT, N>*>(dst + i) = r;
  };
#pragma unroll
  for (int s = 0; s < PIECES; ++s) {
    const int i = (threadIdx.x + s * THREADS) * N;
    if (i < width) put(i, kept[s], ws[s]);
  }
  for (int i = rest; i < width; i += THREADS * N) {
    float v[N];
    if (p.stream != nullptr) {
      const RowPiece<float, N> s = *reinterpret_cast<const RowPiece<float, N>*>(p.stream + (size_t)t * width + i);
#pragma unroll
      for (int j = 0; j < N; ++j) v[j] = s.v[j];
    } else {
      summed(i, v);
    }
    put(i, v, *reinterpret_cast<const RowPiece<W, N>*>(weight + i));
  }
}

// The sum goes into `stream` (which may be x itself) when given; `token_rows` (count entries) only without `stream`.
extern "C" int kvb_stream_add_rows(const float* x, const void* rows, int top, const int* row_of_pair,
                                   const float* pair_weight, int one_row, const int* token_rows, int count, float* stream,
                                   void* normed, const void* weight, float eps, void* packed, const float* origin,
                                   const void* after, float after_eps, const void* step, const int* ids,
                                   int identity_from, const float* all_weight, const void* input, int width, int dtype, int out_dtype, int weight_dtype, cudaStream_t cuda_stream) {
  if (count == 0) return 0;
  KVB_REQUIRE(width > 0 && top >= 0 && x != nullptr && (rows != nullptr || top == 0), "stream_add_rows: empty rows");
  KVB_REQUIRE(normed == nullptr || weight != nullptr, "stream_add_rows: the norm needs its weight");
  KVB_REQUIRE(packed == nullptr || origin != nullptr, "stream_add_rows: the packed rows need what the stream started as");
  KVB_REQUIRE(token_rows == nullptr || stream == nullptr, "stream_add_rows: a list of tokens leaves the stream alone");
  KVB_REQUIRE(after != nullptr || (step == nullptr && ids == nullptr),
              "stream_add_rows: a step row and identity experts come with the norm behind the sub-layer");
  KVB_REQUIRE(ids == nullptr || (all_weight != nullptr && input != nullptr),
              "stream_add_rows: identity experts need the weights and the input rows");
  AddRowsParams p;
  p.after = after; p.after_eps = after_eps; p.step = step; p.ids = ids; p.identity_from = identity_from;
  p.all_weight = all_weight; p.input = input;
  p.x = x; p.rows = rows; p.top = top; p.row_of_pair = row_of_pair; p.pair_weight = pair_weight;
  p.one_row = one_row; p.token_rows = token_rows; p.stream = stream; p.normed = normed; p.weight = weight; p.eps = eps; p.packed = packed;
  p.origin = origin; p.width = width;
  const bool quads = width % 4 == 0 && aligned16(x) && aligned16(rows) && (stream == nullptr || aligned16(stream)) &&
                     (normed == nullptr || (aligned16(normed) && aligned16(weight))) &&
                     (packed == nullptr || (aligned16(packed) && aligned16(origin))) && aligned16(after) &&
                     aligned16(step) && aligned16(input);
  cudaError_t err;
#define KVB_AR_SHAPE(T, OUT, W, N, A, TH) \
  kvb_launch((stream_add_rows_kernel<T, OUT, W, N, A, TH>), dim3(count), dim3(TH), 0, cuda_stream, true, p)
  // few rows: as many threads as a row has pieces (the bits of a row are the same for each number of them)
  const int few = kvb_sm_count() > 0 ? 2 * kvb_sm_count() : 256;
  const int threads = !quads || count > few || width <= 1024 ? 256 : width <= 2048 ? 512 : 1024;
#define KVB_AR(T, OUT, W)                                                                                        \
  err = after == nullptr ? (quads ? KVB_AR_SHAPE(T, OUT, W, 4, false, 256) : KVB_AR_SHAPE(T, OUT, W, 1, false, 256)) \
        : !quads         ? KVB_AR_SHAPE(T, OUT, W, 1, true, 256)                                                  \
        : threads == 256 ? KVB_AR_SHAPE(T, OUT, W, 4, true, 256)                                                  \
        : threads == 512 ? KVB_AR_SHAPE(T, OUT, W, 4, true, 512)                                                  \
                         : KVB_AR_SHAPE(T, OUT, W, 4, true, 1024)
  const int code = (dtype == KVB_BF16 ? 4 : 0) | (out_dtype == KVB_BF16 ? 2 : 0) | (weight_dtype == KVB_BF16 ? 1 : 0);
  switch (code) {
    case 0: KVB_AR(float, float, float); break;
    case 1: KVB_AR(float, float, bf16); break;
    case 2: KVB_AR(float, bf16, float); break;
    case 3: KVB_AR(float, bf16, bf16); break;
    case 4: KVB_AR(bf16, float, float); break;
    case 5: KVB_AR(bf16, float, bf16); break;
    case 6: KVB_AR(bf16, bf16, float); break;
    default: KVB_AR(bf16, bf16, bf16); break;
  }
#undef KVB_AR
#undef KVB_AR_SHAPE
  KVB_CHECK_CUDA(err);
  KVB_CHECK_LAUNCH();
  return 0;
}

// N entries a piece; rows up to SR_THREADS * SR_PIECES * N entries are kept between the passes, wider ones read again.
template <typename T, int N>
__global__ void __launch_bounds__(SR_THREADS)
embed_pairs_kernel(float* __restrict__ out, const T* __restrict__ table, const T* __restrict__ pairs,
                   const float* __restrict__ weight, const int* __restrict__ ids, const int* __restrict__ positions,
                   const int* __restrict__ req_index, const int* __restrict__ query_start,
                   const int* __restrict__ state_slots, int* state, int vocab, int width, long long buckets,
                   long long mul_prev, long long mul_cur, float eps, int* status) {
  KVB_KERNEL_PROLOGUE(KVB_TAG_EMBED_PAIRS);
  __shared__ float scratch[32];
  const int t = blockIdx.x;
  auto checked = [&](int id) {
    if (id >= 0 && id < vocab) return id;
    if (threadIdx.x == 0) atomicOr(status, KVB_STATUS_BAD_TOKEN);
    return 0;
  };
  const int id = checked(ids[t]);
  const T* src = table + (size_t)id * width;
  const T* pair = nullptr;
  int slot = -1, last = 0;
  if (pairs != nullptr) {
    const int req = req_index[t], first = query_start[req];
    long long row = buckets;
    if (positions[t] > 0) {
      const int before = checked(t > first ? ids[t - 1] : state[state_slots[req]]);
      row = (before * mul_prev + id * mul_cur) % buckets;
      if (row < 0) row += buckets;
    }
    pair = pairs + (size_t)row * width;
    if (t == first) { slot = state_slots[req]; last = ids[query_start[req + 1] - 1]; }
  }
  auto value = [&](int i, float (&v)[N]) {
    const RowPiece<T, N> a = *reinterpret_cast<const RowPiece<T, N>*>(src + i);
#pragma unroll
    for (int j = 0; j < N; ++j) v[j] = to_float(a.v[j]);
    if (pair != nullptr) {
      const RowPiece<T, N> b = *reinterpret_cast<const RowPiece<T, N>*>(pair + i);
#pragma unroll
      for (int j = 0; j < N; ++j) v[j] += to_float(b.v[j]);
    }
  };
  float kept[SR_PIECES][N];
  float ss = 0.0f;
#pragma unroll
  for (int s = 0; s < SR_PIECES; ++s) {
    const int i = (threadIdx.x + s * SR_THREADS) * N;
    if (i < width) {
      value(i, kept[s]);
#pragma unroll
      for (int j = 0; j < N; ++j) ss = fmaf(kept[s][j], kept[s][j], ss);
    }
  }
  const int rest = (threadIdx.x + SR_PIECES * SR_THREADS) * N;
  for (int i = rest; i < width; i += SR_THREADS * N) {
    float v[N];
    value(i, v);
#pragma unroll
    for (int j = 0; j < N; ++j) ss = fmaf(v[j], v[j], ss);
  }
  // (the barriers of this sum stand between every thread's read of the state and the write below)
  const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)width + eps);
  float* dst = out + (size_t)t * width;
  auto put = [&](int i, const float (&v)[N]) {
    RowPiece<float, N> r;
#pragma unroll
    for (int j = 0; j < N; ++j) r.v[j] = weight != nullptr ? v[j] * inv * weight[i + j] : v[j];
    *reinterpret_cast<RowPiece<float, N>*>(dst + i) = r;
  };
#pragma unroll
  for (int s = 0; s < SR_PIECES; ++s) {
    const int i = (threadIdx.x + s * SR_THREADS) * N;
    if (i < width) put(i, kept[s]);
  }
  for (int i = rest; i < width; i += SR_THREADS * N) {
    float v[N];
    value(i, v);
    put(i, v);
  }
  if (slot >= 0 && threadIdx.x == 0) state[slot] = last;
}

// pairs null: no second table; weight null: no norm.
extern "C" int kvb_embed_pairs(float* out, const void* table, const void* pairs, const float* weight, const int* ids,
                               const int* positions, const int* req_index, const int* query_start,
                               const int* state_slots, int* state, int tokens, int vocab, int width, long long buckets,
                               long long mul_prev, long long mul_cur, float eps, int dtype, cudaStream_t stream) {
  if (tokens == 0) return 0;
  KVB_REQUIRE(vocab > 0 && width > 0, "embed_pairs: bad sizes");
  KVB_REQUIRE(pairs == nullptr || (buckets > 0 && state != nullptr && positions != nullptr && req_index != nullptr &&
                                   query_start != nullptr && state_slots != nullptr),
              "embed_pairs: the pair table needs its buckets, the state and the batch's request arrays");
  int* status = kvb_status_word();
  KVB_REQUIRE(status != nullptr, "embed_pairs: no status word");
  const size_t esize = dtype == KVB_F32 ? 4 : 2;
  const bool quads = width % 4 == 0 && aligned16(out) && (uintptr_t)table % (4 * esize) == 0 && (uintptr_t)pairs % (4 * esize) == 0;
#define KVB_EP(T, N)                                                                                                 \
  KVB_CHECK_CUDA(kvb_launch((embed_pairs_kernel<T, N>), dim3(tokens), dim3(SR_THREADS), 0, stream, true, out,        \
      (const T*)table, (const T*)pairs, weight, ids, positions, req_index, query_start, state_slots, state, vocab,   \
      width, buckets, mul_prev, mul_cur, eps, status))
  if (dtype == KVB_F32) { if (quads) KVB_EP(float, 4); else KVB_EP(float, 1); }
  else { if (quads) KVB_EP(bf16, 4); else KVB_EP(bf16, 1); }
#undef KVB_EP
  KVB_CHECK_LAUNCH();
  return 0;
}

__global__ void __launch_bounds__(SR_THREADS)
softcap_kernel(float* __restrict__ logits, long long count, float scale, float cap) {
  KVB_KERNEL_PROLOGUE(KVB_TAG_SOFTCAP);
  const long long step = (long long)gridDim.x * SR_THREADS;
  for (long long i = (long long)blockIdx.x * SR_THREADS + threadIdx.x; i < count; i += step)
    logits[i] = cap * tanhf(logits[i] * scale / cap);
}

extern "C" int kvb_softcap(float* logits, long long count, float scale, float cap, cudaStream_t stream) {
  if (count == 0) return 0;
  KVB_REQUIRE(cap > 0.0f, "softcap: the cap must be positive");
  const long long wanted = (count + SR_THREADS - 1) / SR_THREADS;
  const long long resident = (long long)(kvb_sm_count() > 0 ? kvb_sm_count() : 1) * 8;
  KVB_CHECK_CUDA(kvb_launch((softcap_kernel), dim3((unsigned)(wanted < resident ? wanted : resident)), dim3(SR_THREADS),
                            0, stream, true, logits, count, scale, cap));
  KVB_CHECK_LAUNCH();
  return 0;
}

KVB_TRACE_TU(stream_rows)
