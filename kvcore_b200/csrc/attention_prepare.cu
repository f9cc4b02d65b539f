// Between the projections and the attention of a mixer that caches one row [k of all heads | v of all heads] a token.
//
//   attention_prepare: q [H, D], k [G, D] and v of a token's projected row, in this order, each step where asked for:
//     a causal convolution over time per channel of q, k and v (taps [K, channels], the last tap on the current token,
//       no bias; the K - 1 inputs in front of a portion come from the request's state row, [K - 1, channels] 32-bit,
//       oldest first);
//     one RMS norm over all of q and one over all of k, with weights;
//     a turn of the first `rot` entries of every q and k head in halves: entry i and entry i + rot / 2 form the pair
//       (u, w) -> (u c - w s, w c + u s) with the token's (c, s) of frequency i.
//   q goes to rows of its own (or back in place where nothing is convolved: the tokens behind a convolved one still need
//   its projections), k and v into the token's place of the cache.
//
// A thread takes N neighbouring entries of a head's first half together with their partners, or N entries that do not
// turn, so a pair never leaves the thread.  With a norm a block owns a whole token and keeps up to AP_KEEP such units a
// thread in registers between the sum and the store; without one the units of a token may be spread over blocks.
// Everything is 32-bit up to the store; sums depend on the sizes only, not on the batch or the cut.  In a step of single
// tokens the thread that has read a channel's inputs also moves the kept ones on; otherwise a second kernel does
// (keep_inputs), because several tokens of a portion may read what the state held.
#include "common.cuh"

#define AP_THREADS 256
#define AP_KEEP 3

extern "C" int kvb_keep_inputs(float* state, long long state_stride, long long state_offset, const void* rows,
                               long long row_stride, int channels, int keep, const int* query_start,
                               const int* state_slots, int num_reqs, int dtype, cudaStream_t stream);

template <typename T, int N>
struct __align__(N * sizeof(T) > 16 ? 16 : N * sizeof(T)) ApPiece { T v[N]; };

struct AttentionPrepareParams {
  const void* rows; long long row_stride;
  void* q_out; long long q_stride;
  const float2* cos_sin; int rot;                    // [T, rot / 2]
  const int* positions; const int* req_index; const int* query_start; const int* state_slots;
  const int* table; int table_stride;
  void* cache; int page_size, num_pages, write;
  int tokens, H, G, D, v_width;
  const void* taps; int num_taps;                    // 0: no convolution
  float* state; long long state_stride, state_offset;
  int single;                                        // one token a request: the kept inputs are moved on here
  const void* q_weight; const void* k_weight; float eps;
  int run;                                           // tokens a block walks
  int units_per_block;
  int* status;
};

template <typename T, int N, bool NORM>
__global__ void __launch_bounds__(AP_THREADS)
attention_prepare_kernel(const AttentionPrepareParams p) {
  KVB_KERNEL_PROLOGUE(KVB_TAG_ATTN_PREPARE);
  __shared__ float scratch[32];
  const int half = p.rot >> 1, turned = half / N, per_head = turned + (p.D - p.rot) / N;
  const int q_len = p.H * p.D, k_len = p.G * p.D, channels = q_len + k_len + p.v_width, keep = p.num_taps - 1;
  const int heads = p.write ? p.H + p.G : p.H;
  const int qk_units = heads * per_head, units = qk_units + (p.write ? p.v_width / N : 0);
  const int u_begin = blockIdx.y * p.units_per_block, u_end = min(units, u_begin + p.units_per_block);
  const int t_end = min(p.tokens, (int)(blockIdx.x + 1) * p.run);
  for (int t = blockIdx.x * p.run; t < t_end; ++t) {
    const T* row = (const T*)p.rows + (size_t)t * p.row_stride;
    const int pos = p.positions[t], req = p.req_index[t];
    T* dst = nullptr;
    if (p.write) {
      const int page = p.table[(size_t)req * p.table_stride + pos / p.page_size];
      if (page <= 0 || page >= p.num_pages) {
        if (threadIdx.x == 0 && blockIdx.y == 0) atomicOr(p.status, KVB_STATUS_BAD_PAGE);
      } else {
        dst = (T*)p.cache + ((size_t)page * p.page_size + pos % p.page_size) * ((size_t)k_len + p.v_width);
      }
    }
    int back = 0;
    float* held = nullptr;
    if (keep > 0) {
      back = t - p.query_start[req];
      held = p.state + (size_t)p.state_slots[req] * p.state_stride + p.state_offset;
    }
    // N channels of this token from channel c on; `last`: nobody reads the state of these channels again
    auto fetch = [&](int c, float (&x)[N], bool last) {
      const ApPiece<T, N> now = *reinterpret_cast<const ApPiece<T, N>*>(row + c);
      if (p.num_taps == 0) {
#pragma unroll
        for (int j = 0; j < N; ++j) x[j] = to_float(now.v[j]);
        return;
      }
#pragma unroll
      for (int j = 0; j < N; ++j) x[j] = 0.0f;
      const T* taps = (const T*)p.taps + c;
      const bool move = p.single && last;
      for (int tap = 0; tap < keep; ++tap) {
        const int ago = keep - tap;                  // this tap reads the input `ago` tokens back
        float was[N];
        if (ago <= back) {
          const ApPiece<T, N> in = *reinterpret_cast<const ApPiece<T, N>*>(row - (size_t)ago * p.row_stride + c);
#pragma unroll
          for (int j = 0; j < N; ++j) was[j] = to_float(in.v[j]);
        } else {
          const float* from = held + (size_t)(keep - (ago - back)) * channels + c;
#pragma unroll
          for (int j = 0; j < N; ++j) was[j] = from[j];
        }
        const ApPiece<T, N> w = *reinterpret_cast<const ApPiece<T, N>*>(taps + (size_t)tap * channels);
#pragma unroll
        for (int j = 0; j < N; ++j) x[j] = fmaf(to_float(w.v[j]), was[j], x[j]);
        if (move && tap > 0) {
#pragma unroll
          for (int j = 0; j < N; ++j) held[(size_t)(tap - 1) * channels + c + j] = was[j];
        }
      }
      const ApPiece<T, N> w = *reinterpret_cast<const ApPiece<T, N>*>(taps + (size_t)keep * channels);
#pragma unroll
      for (int j = 0; j < N; ++j) x[j] = fmaf(to_float(w.v[j]), to_float(now.v[j]), x[j]);
      if (move && keep > 0) {
#pragma unroll
        for (int j = 0; j < N; ++j) held[(size_t)(keep - 1) * channels + c + j] = to_float(now.v[j]);
      }
    };
    auto store = [&](T* at, const float (&x)[N]) {
      ApPiece<T, N> r;
#pragma unroll
      for (int j = 0; j < N; ++j) r.v[j] = from_float<T>(x[j]);
      *reinterpret_cast<ApPiece<T, N>*>(at) = r;
    };
    // where unit u lies: its head, its first entry, whether it has a partner
    auto locate = [&](int u, int& head, int& i, bool& pair) {
      head = u / per_head;
      const int piece = u - head * per_head;
      pair = piece < turned;
      i = pair ? piece * N : p.rot + (piece - turned) * N;
    };
    auto load_unit = [&](int u, float (&a)[N], float (&b)[N], bool last) {
      int head, i;
      bool pair;
      locate(u, head, i, pair);
      fetch(head * p.D + i, a, last);
      if (pair) {
        fetch(head * p.D + i + half, b, last);
      } else {
#pragma unroll
        for (int j = 0; j < N; ++j) b[j] = 0.0f;
      }
    };
    auto put_unit = [&](int u, float (&a)[N], float (&b)[N], float q_inv, float k_inv) {
      int head, i;
      bool pair;
      locate(u, head, i, pair);
      const bool is_q = head < p.H;
      const int at = (is_q ? head : head - p.H) * p.D + i;
      if (NORM) {
        const T* weight = (const T*)(is_q ? p.q_weight : p.k_weight) + at;
        const float inv = is_q ? q_inv : k_inv;
        const ApPiece<T, N> w = *reinterpret_cast<const ApPiece<T, N>*>(weight);
#pragma unroll
        for (int j = 0; j < N; ++j) a[j] *= inv * to_float(w.v[j]);
        if (pair) {
          const ApPiece<T, N> w2 = *reinterpret_cast<const ApPiece<T, N>*>(weight + half);
#pragma unroll
          for (int j = 0; j < N; ++j) b[j] *= inv * to_float(w2.v[j]);
        }
      }
      if (pair) {
        const ApPiece<float2, N> cs = *reinterpret_cast<const ApPiece<float2, N>*>(p.cos_sin + (size_t)t * half + i);
#pragma unroll
        for (int j = 0; j < N; ++j) {
          const float u0 = a[j], w0 = b[j];
          a[j] = u0 * cs.v[j].x - w0 * cs.v[j].y;
          b[j] = w0 * cs.v[j].x + u0 * cs.v[j].y;
        }
      }
      T* to = is_q ? (T*)p.q_out + (size_t)t * p.q_stride + at : dst == nullptr ? nullptr : dst + at;
      if (to == nullptr) return;
      store(to, a);
      if (pair) store(to + half, b);
    };
    float q_inv = 1.0f, k_inv = 1.0f;
    if (NORM) {                                      // (the block owns every unit of the token)
      float a[AP_KEEP][N], b[AP_KEEP][N];
      float q_sum = 0.0f, k_sum = 0.0f;
      auto count = [&](int u, const float (&av)[N], const float (&bv)[N]) {
        float sq = 0.0f;
#pragma unroll
        for (int j = 0; j < N; ++j) sq = fmaf(bv[j], bv[j], fmaf(av[j], av[j], sq));
        if (u < p.H * per_head) q_sum += sq; else k_sum += sq;
      };
#pragma unroll
      for (int s = 0; s < AP_KEEP; ++s) {
        const int u = threadIdx.x + s * AP_THREADS;
        if (u < qk_units) load_unit(u, a[s], b[s], true);
      }
#pragma unroll
      for (int s = 0; s < AP_KEEP; ++s) {
        const int u = threadIdx.x + s * AP_THREADS;
        if (u < qk_units) count(u, a[s], b[s]);
      }
      for (int u = threadIdx.x + AP_KEEP * AP_THREADS; u < qk_units; u += AP_THREADS) {
        float av[N], bv[N];
        load_unit(u, av, bv, false);
        count(u, av, bv);
      }
      q_inv = 1.0f / sqrtf(block_sum(q_sum, scratch) / (float)q_len + p.eps);
      k_inv = 1.0f / sqrtf(block_sum(k_sum, scratch) / (float)k_len + p.eps);
#pragma unroll
      for (int s = 0; s < AP_KEEP; ++s) {
        const int u = threadIdx.x + s * AP_THREADS;
        if (u < qk_units) put_unit(u, a[s], b[s], q_inv, k_inv);
      }
    }
    for (int u = u_begin + threadIdx.x + (NORM ? AP_KEEP * AP_THREADS : 0); u < min(u_end, qk_units); u += AP_THREADS) {
      float av[N], bv[N];
      load_unit(u, av, bv, true);
      put_unit(u, av, bv, q_inv, k_inv);
    }
    for (int u = max(u_begin, qk_units) + threadIdx.x; u < u_end; u += AP_THREADS) {
      const int i = (u - qk_units) * N;
      float av[N];
      fetch(q_len + k_len + i, av, true);
      if (dst != nullptr) store(dst + k_len + i, av);
    }
  }
}

template <typename T, int N>
static cudaError_t launch_attention_prepare(AttentionPrepareParams& p, bool norm, cudaStream_t stream) {
  const int per_head = p.rot / 2 / N + (p.D - p.rot) / N;
  const int units = (p.write ? p.H + p.G : p.H) * per_head + (p.write ? p.v_width / N : 0);
  // without a norm: a few tokens spread their units over blocks; many tokens go a block each
  p.units_per_block = norm || p.tokens >= 512 ? units : AP_THREADS;
  const dim3 grid((p.tokens + p.run - 1) / p.run, (units + p.units_per_block - 1) / p.units_per_block);
  if (norm) return kvb_launch((attention_prepare_kernel<T, N, true>), grid, dim3(AP_THREADS), 0, stream, true, p);
  return kvb_launch((attention_prepare_kernel<T, N, false>), grid, dim3(AP_THREADS), 0, stream, true, p);
}

// rows: [q | k | v] of every token (row stride `row_stride`); q_out: rows of q (may be `rows` itself without taps);
// cos_sin null: nothing turns; taps null: no convolution; q_weight null: no norm.
extern "C" int kvb_attention_prepare(const void* rows, long long row_stride, void* q_out, long long q_stride,
                                     const float* cos_sin, int rot, const int* positions, const int* req_index,
                                     const int* query_start, const int* state_slots, const int* table, int table_stride,
                                     void* cache, int page_size, int num_pages, int write, int tokens, int num_reqs,
                                     int H, int G, int D, int v_width, const void* taps, int num_taps, float* state,
                                     long long state_stride, long long state_offset, const void* q_weight,
                                     const void* k_weight, float eps, int dtype, cudaStream_t stream) {
  if (tokens == 0) return 0;
  if (cos_sin == nullptr) rot = 0;
  if (taps == nullptr) num_taps = 0;
  KVB_REQUIRE(H > 0 && G > 0 && D > 0 && v_width > 0, "attention_prepare: bad sizes");
  KVB_REQUIRE(rot >= 0 && rot % 2 == 0 && rot <= D, "attention_prepare: the turned entries are an even number within the head");
  KVB_REQUIRE(taps == nullptr || (num_taps >= 1 && q_out != rows), "attention_prepare: convolved queries need rows of their own");
  KVB_REQUIRE(num_taps < 2 || (state != nullptr && query_start != nullptr && state_slots != nullptr),
              "attention_prepare: a convolution needs the state rows and the batch's request arrays");
  KVB_REQUIRE((q_weight == nullptr) == (k_weight == nullptr), "attention_prepare: give both norm weights or none");
  AttentionPrepareParams p;
  p.rows = rows; p.row_stride = row_stride; p.q_out = q_out; p.q_stride = q_stride;
  p.cos_sin = (const float2*)cos_sin; p.rot = rot; p.positions = positions; p.req_index = req_index;
  p.query_start = query_start; p.state_slots = state_slots; p.table = table; p.table_stride = table_stride;
  p.cache = cache; p.page_size = page_size; p.num_pages = num_pages; p.write = write; p.tokens = tokens;
  p.H = H; p.G = G; p.D = D; p.v_width = v_width; p.taps = taps; p.num_taps = num_taps; p.state = state;
  p.state_stride = state_stride; p.state_offset = state_offset; p.single = tokens == num_reqs;
  p.q_weight = q_weight; p.k_weight = k_weight; p.eps = eps; p.run = 1;
  p.status = kvb_status_word();
  KVB_REQUIRE(p.status != nullptr, "attention_prepare: no status word");
  const int n = dtype == KVB_F32 ? 4 : 8;
  const bool vec = (rot / 2) % n == 0 && D % n == 0 && v_width % n == 0 && row_stride % n == 0 && q_stride % n == 0 &&
                   aligned16(rows) && aligned16(q_out) && aligned16(cos_sin) && aligned16(cache) && aligned16(taps) &&
                   aligned16(q_weight) && aligned16(k_weight);
  cudaError_t err;
  const bool norm = q_weight != nullptr;
  if (dtype == KVB_F32) err = vec ? launch_attention_prepare<float, 4>(p, norm, stream) : launch_attention_prepare<float, 1>(p, norm, stream);
  else err = vec ? launch_attention_prepare<bf16, 8>(p, norm, stream) : launch_attention_prepare<bf16, 1>(p, norm, stream);
  KVB_CHECK_CUDA(err);
  KVB_CHECK_LAUNCH();
  if (num_taps > 1 && !p.single)
    return kvb_keep_inputs(state, state_stride, state_offset, rows, row_stride, H * D + G * D + v_width, num_taps - 1,
                           query_start, state_slots, num_reqs, dtype, stream);
  return 0;
}

KVB_TRACE_TU(attention_prepare)
