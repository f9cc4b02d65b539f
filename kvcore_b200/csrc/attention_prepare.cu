// Between the projections and the attention of a mixer that caches keys and values, addressed by strides: side by side in
// one row a token, or in two tensors [pages, heads, page, width].
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
// A thread takes a unit: N neighbouring entries of a head's turned first half together with their partners (a pair never
// leaves the thread), or two pieces of N entries that do not turn (one, where their number is odd).  Two kernels: with a norm a block owns a whole token, with a thread a
// unit where a block has that many, so that everything a token needs is on its way at once; without one a thread owns a
// unit for a run of tokens, its taps stay in registers and its window slides over the run, so a row is read once, and the
// run's cos/sin and cache places wait in shared memory (attention_prepare_runs).
// Everything is 32-bit up to the store; sums depend on the sizes only, not on the batch or the cut.  In a step of single
// tokens the thread that has read a channel's inputs also moves the kept ones on; otherwise a second kernel does
// (keep_inputs), because several tokens of a portion may read what the state held.
#include "common.cuh"

#define AP_MAX_THREADS 1024
#define AP_RUN_THREADS 128
#define AP_RUN 16              // tokens a thread of the run kernel walks, at most
#define AP_MAX_TAPS 9          // more taps take the other kernel

extern "C" int kvb_keep_inputs(float* state, long long state_stride, long long state_offset, const void* rows,
                               long long row_stride, int channels, int keep, const int* query_start,
                               const int* state_slots, int num_reqs, int dtype, cudaStream_t stream);

template <typename T, int N>
struct __align__(N * sizeof(T) > 16 ? 16 : N * sizeof(T)) ApPiece { T v[N]; };

// How a token's [q | k | v] falls into units for pieces of N entries: a head's turned pairs, its entries that do not turn,
// then the values.
template <int N>
struct ApUnits {
  int D, half, turned, rest, rest_mate, per_head, qk_units, v_mate, units;
  __device__ __forceinline__ ApUnits(int D_, int rot, int heads, int v_width, int write) : D(D_) {
    half = rot >> 1;
    turned = half / N;
    rest = rot;
    rest_mate = (D - rot) % (2 * N) == 0 ? (D - rot) / 2 : 0;
    per_head = turned + (rest_mate ? rest_mate / N : (D - rot) / N);
    qk_units = heads * per_head;
    v_mate = v_width % (2 * N) == 0 ? v_width / 2 : 0;
    units = qk_units + (write ? (v_mate ? v_mate : v_width) / N : 0);
  }
  // a unit's head (of q, then of k), its first entry there, how far its second piece lies behind (0: none), whether it turns
  __device__ __forceinline__ void locate(int u, int& head, int& i, int& mate, bool& turns) const {
    head = u / per_head;
    const int piece = u - head * per_head;
    turns = piece < turned;
    i = turns ? piece * N : rest + (piece - turned) * N;
    mate = turns ? half : rest_mate;
  }
};

struct AttentionPrepareParams {
  const void* rows; long long row_stride;
  void* q_out; long long q_stride;
  const float2* cos_sin; int rot;                    // [T, rot / 2]
  const int* positions; const int* req_index; const int* query_start; const int* state_slots;
  const int* table; int table_stride;
  // where head g of the token in slot s of page n keeps its key: k_cache + n * k_page + g * k_head + s * k_row; values alike
  void* k_cache; long long k_page, k_head, k_row;
  void* v_cache; long long v_page, v_head, v_row;
  int page_size, num_pages, write;
  int tokens, H, G, D, V, v_width;                   // v_width = G * V
  const void* taps; int num_taps;                    // 0: no convolution
  float* state; long long state_stride, state_offset;
  int single;                                        // one token a request: the kept inputs are moved on here
  const void* q_weight; const void* k_weight; float eps;
  int run;                                           // tokens a thread of the run kernel walks
  int* status;
};

template <typename T, int N, bool NORM, bool CONV>
__global__ void __launch_bounds__(AP_MAX_THREADS)
attention_prepare_kernel(const AttentionPrepareParams p) {
  KVB_KERNEL_PROLOGUE(KVB_TAG_ATTN_PREPARE);
  __shared__ float scratch[2][32];
  const int q_len = p.H * p.D, k_len = p.G * p.D, channels = q_len + k_len + p.v_width, keep = p.num_taps - 1;
  const ApUnits<N> cut(p.D, p.rot, p.write ? p.H + p.G : p.H, p.v_width, p.write);
  const int half = cut.half, qk_units = cut.qk_units, units = cut.units;
  {
    const int t = blockIdx.x;
    const T* row = (const T*)p.rows + (size_t)t * p.row_stride;
    const int pos = p.positions[t], req = p.req_index[t];
    T* k_dst = nullptr;                              // the token's place among the keys and among the values
    T* v_dst = nullptr;
    if (p.write) {
      const int page = p.table[(size_t)req * p.table_stride + pos / p.page_size];
      if (page <= 0 || page >= p.num_pages) {
        if (threadIdx.x == 0) atomicOr(p.status, KVB_STATUS_BAD_PAGE);
      } else {
        k_dst = (T*)p.k_cache + (size_t)page * p.k_page + (size_t)(pos % p.page_size) * p.k_row;
        v_dst = (T*)p.v_cache + (size_t)page * p.v_page + (size_t)(pos % p.page_size) * p.v_row;
      }
    }
    int back = 0;
    float* held = nullptr;
    if (CONV && keep > 0) {
      back = t - p.query_start[req];
      held = p.state + (size_t)p.state_slots[req] * p.state_stride + p.state_offset;
    }
    // N channels of this token from channel c on; `last`: nobody reads the state of these channels again
    auto fetch = [&](int c, float (&x)[N], bool last) {
      const ApPiece<T, N> now = *reinterpret_cast<const ApPiece<T, N>*>(row + c);
      if constexpr (!CONV) {
#pragma unroll
        for (int j = 0; j < N; ++j) x[j] = to_float(now.v[j]);
      } else {
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
      }
    };
    auto store = [&](T* at, const float (&x)[N]) {
      ApPiece<T, N> r;
#pragma unroll
      for (int j = 0; j < N; ++j) r.v[j] = from_float<T>(x[j]);
      *reinterpret_cast<ApPiece<T, N>*>(at) = r;
    };
    auto load_unit = [&](int u, float (&a)[N], float (&b)[N], bool last) {
      int head, i, mate;
      bool turns;
      cut.locate(u, head, i, mate, turns);
      fetch(head * p.D + i, a, last);
      if (mate) {
        fetch(head * p.D + i + mate, b, last);
      } else {
#pragma unroll
        for (int j = 0; j < N; ++j) b[j] = 0.0f;
      }
    };
    auto weights_of = [&](int u, ApPiece<T, N>& w, ApPiece<T, N>& w2) {
      int head, i, mate;
      bool turns;
      cut.locate(u, head, i, mate, turns);
      const T* weight = head < p.H ? (const T*)p.q_weight + head * p.D + i : (const T*)p.k_weight + (head - p.H) * p.D + i;
      w = *reinterpret_cast<const ApPiece<T, N>*>(weight);
      if (mate) w2 = *reinterpret_cast<const ApPiece<T, N>*>(weight + mate);
    };
    auto put_unit = [&](int u, float (&a)[N], float (&b)[N], const ApPiece<T, N>& w, const ApPiece<T, N>& w2, float q_inv,
                        float k_inv) {
      int head, i, mate;
      bool turns;
      cut.locate(u, head, i, mate, turns);
      const bool is_q = head < p.H;
      const int at = (is_q ? head : head - p.H) * p.D + i;
      if (NORM) {
        const float inv = is_q ? q_inv : k_inv;
#pragma unroll
        for (int j = 0; j < N; ++j) {
          a[j] *= inv * to_float(w.v[j]);
          if (mate) b[j] *= inv * to_float(w2.v[j]);
        }
      }
      if (turns) {
        const ApPiece<float2, N> cs = *reinterpret_cast<const ApPiece<float2, N>*>(p.cos_sin + (size_t)t * half + i);
#pragma unroll
        for (int j = 0; j < N; ++j) {
          const float u0 = a[j], w0 = b[j];
          a[j] = u0 * cs.v[j].x - w0 * cs.v[j].y;
          b[j] = w0 * cs.v[j].x + u0 * cs.v[j].y;
        }
      }
      T* to = is_q ? (T*)p.q_out + (size_t)t * p.q_stride + at
                   : k_dst == nullptr ? nullptr : k_dst + (size_t)(head - p.H) * p.k_head + i;
      if (to == nullptr) return;
      store(to, a);
      if (mate) store(to + mate, b);
    };
    float q_inv = 1.0f, k_inv = 1.0f;
    const int threads = blockDim.x;
    // the values' units lie behind the heads' units, so the thread of a value's unit has no other where the block is wide
    // enough
    auto put_value = [&](int u) {
      const int i = (u - qk_units) * N;
      float av[N], bv[N];
      fetch(q_len + k_len + i, av, true);
      if (cut.v_mate) fetch(q_len + k_len + i + cut.v_mate, bv, true);
      if (v_dst == nullptr) return;
      auto at = [&](int e) { return v_dst + (size_t)(e / p.V) * p.v_head + e % p.V; };
      store(at(i), av);
      if (cut.v_mate) store(at(i + cut.v_mate), bv);
    };
    float a[N], b[N];                                // this thread's first unit stays in registers
    ApPiece<T, N> w, w2;                             // (its weights are on their way before anybody waits for a sum)
    if (NORM) {
      float q_sum = 0.0f, k_sum = 0.0f;
      auto count = [&](int u, const float (&av)[N], const float (&bv)[N]) {
        float sq = 0.0f;
#pragma unroll
        for (int j = 0; j < N; ++j) sq = fmaf(bv[j], bv[j], fmaf(av[j], av[j], sq));
        if (u < p.H * cut.per_head) q_sum += sq; else k_sum += sq;
      };
      if ((int)threadIdx.x < qk_units) {
        load_unit(threadIdx.x, a, b, true);
        weights_of(threadIdx.x, w, w2);
        count(threadIdx.x, a, b);
      } else if ((int)threadIdx.x < units) {
        put_value(threadIdx.x);
      }
      for (int u = threadIdx.x + threads; u < qk_units; u += threads) {
        float av[N], bv[N];
        load_unit(u, av, bv, false);
        count(u, av, bv);
      }
      // both sums behind one barrier: a butterfly a warp, then the warps' sums in a butterfly of their own
      q_sum = warp_sum(q_sum);
      k_sum = warp_sum(k_sum);
      const int lane = threadIdx.x & 31, warps = threads >> 5;
      if (lane == 0) { scratch[0][threadIdx.x >> 5] = q_sum; scratch[1][threadIdx.x >> 5] = k_sum; }
      __syncthreads();
      q_sum = warp_sum(lane < warps ? scratch[0][lane] : 0.0f);
      k_sum = warp_sum(lane < warps ? scratch[1][lane] : 0.0f);
      q_inv = 1.0f / sqrtf(q_sum / (float)q_len + p.eps);
      k_inv = 1.0f / sqrtf(k_sum / (float)k_len + p.eps);
      if ((int)threadIdx.x < qk_units) put_unit(threadIdx.x, a, b, w, w2, q_inv, k_inv);
    }
    for (int u = threadIdx.x + (NORM ? threads : 0); u < units; u += threads) {
      if (u >= qk_units) {
        put_value(u);
        continue;
      }
      load_unit(u, a, b, true);
      if (NORM) weights_of(u, w, w2);
      put_unit(u, a, b, w, w2, q_inv, k_inv);
    }
  }
}

__device__ __forceinline__ int ap_kind(int u, int qk_units, int q_units) { return u < q_units ? 0 : u < qk_units ? 1 : 2; }

// Without a norm.  A thread owns a unit for `run` tokens; K: taps the window is made for (the model's taps, right-aligned;
// the places in front are zero), 1 also where nothing is convolved.
template <typename T, int N, int K>
__global__ void __launch_bounds__(AP_RUN_THREADS, K <= 4 ? 4 : 2)
attention_prepare_runs_kernel(const AttentionPrepareParams p) {
  KVB_KERNEL_PROLOGUE(KVB_TAG_ATTN_PREPARE);
  extern __shared__ __align__(16) float2 run_cs[];   // [run][rot / 2]
  __shared__ long long place_of[2][AP_RUN];          // where a token's key and its value begin, or -1
  const int q_len = p.H * p.D, k_len = p.G * p.D, channels = q_len + k_len + p.v_width, keep = p.num_taps - 1;
  const ApUnits<N> cut(p.D, p.rot, p.write ? p.H + p.G : p.H, p.v_width, p.write);
  const int half = cut.half;
  const int t_begin = blockIdx.y * p.run, t_end = min(p.tokens, t_begin + p.run);
  for (int e = threadIdx.x; e < (t_end - t_begin) * half; e += AP_RUN_THREADS)
    run_cs[e] = p.cos_sin[(size_t)t_begin * half + e];
  if (p.write && (int)threadIdx.x < t_end - t_begin) {
    const int t = t_begin + threadIdx.x, pos = p.positions[t];
    const int page = p.table[(size_t)p.req_index[t] * p.table_stride + pos / p.page_size];
    const bool fine = page > 0 && page < p.num_pages;
    if (!fine && blockIdx.x == 0) atomicOr(p.status, KVB_STATUS_BAD_PAGE);
    place_of[0][threadIdx.x] = fine ? page * p.k_page + pos % p.page_size * p.k_row : -1;
    place_of[1][threadIdx.x] = fine ? page * p.v_page + pos % p.page_size * p.v_row : -1;
  }
  __syncthreads();
  const int u = blockIdx.x * AP_RUN_THREADS + threadIdx.x;
  if (u >= cut.units) return;
  int c, i = 0, mate;                                // first channel, its place in its head, where its second piece lies
  bool turns = false;
  const int kind = ap_kind(u, cut.qk_units, p.H * cut.per_head);      // 0 a query, 1 a key, 2 values
  long long inside[2] = {0, 0};                      // a key's or value's pieces behind the token's place
  if (kind < 2) {
    int head;
    cut.locate(u, head, i, mate, turns);
    c = head * p.D + i;
    if (kind == 1) {
      inside[0] = (head - p.H) * p.k_head + i;
      inside[1] = inside[0] + mate;
    }
  } else {
    const int e = (u - cut.qk_units) * N;
    c = q_len + k_len + e;
    mate = cut.v_mate;
    inside[0] = e / p.V * p.v_head + e % p.V;
    inside[1] = (e + mate) / p.V * p.v_head + (e + mate) % p.V;
  }
  ApPiece<T, N> taps[2][K];
  if (p.num_taps > 0) {
#pragma unroll
    for (int j = 0; j < K; ++j) {
      const int tap = j - (K - p.num_taps);
#pragma unroll
      for (int side = 0; side < 2; ++side)
        if (tap >= 0 && (side == 0 || mate))
          taps[side][j] = *reinterpret_cast<const ApPiece<T, N>*>((const T*)p.taps + (size_t)tap * channels + c + side * mate);
        else
#pragma unroll
          for (int n = 0; n < N; ++n) taps[side][j].v[n] = from_float<T>(0.0f);
    }
  }
  constexpr int W = K > 1 ? K - 1 : 1, AHEAD = K > 1 ? 2 : 4;      // tokens whose loads are in flight together
  float window[2][W][N];
  const T* src = (const T*)p.rows + c;
  int end = t_begin;                                 // where the request of the token in hand ends
  float* held = nullptr;
  for (int t0 = t_begin; t0 < t_end; t0 += AHEAD) {
    ApPiece<T, N> in[AHEAD][2];                   // a few tokens' loads in flight together
#pragma unroll
    for (int d = 0; d < AHEAD; ++d)
      if (t0 + d < t_end) {
        in[d][0] = *reinterpret_cast<const ApPiece<T, N>*>(src + (size_t)(t0 + d) * p.row_stride);
        if (mate) in[d][1] = *reinterpret_cast<const ApPiece<T, N>*>(src + (size_t)(t0 + d) * p.row_stride + mate);
      }
#pragma unroll
    for (int d = 0; d < AHEAD; ++d) {
      const int t = t0 + d;
      if (t >= t_end) break;
      if (t == end) {                                // the run's first token, or a portion's
        const int req = p.req_index[t];
        end = p.query_start[req + 1];
        if (K > 1 && keep > 0) {
          const int back = t - p.query_start[req];
          held = p.state + (size_t)p.state_slots[req] * p.state_stride + p.state_offset + c;
#pragma unroll
          for (int j = 0; j < K - 1; ++j) {
            const int ago = K - 1 - j;               // window[j] is the input `ago` tokens back
#pragma unroll
            for (int side = 0; side < 2; ++side) {
              if (ago > keep || (side == 1 && !mate)) {
#pragma unroll
                for (int n = 0; n < N; ++n) window[side][j][n] = 0.0f;
              } else if (ago <= back) {
                const ApPiece<T, N> was = *reinterpret_cast<const ApPiece<T, N>*>(src + (size_t)(t - ago) * p.row_stride + side * mate);
#pragma unroll
                for (int n = 0; n < N; ++n) window[side][j][n] = to_float(was.v[n]);
              } else {
                const float* from = held + (size_t)(keep - (ago - back)) * channels + side * mate;
#pragma unroll
                for (int n = 0; n < N; ++n) window[side][j][n] = from[n];
              }
            }
          }
        }
      }
      float y[2][N];
#pragma unroll
      for (int side = 0; side < 2; ++side) {
        if (side == 1 && !mate) break;
#pragma unroll
        for (int n = 0; n < N; ++n) {
          const float x = to_float(in[d][side].v[n]);
          if (p.num_taps == 0) { y[side][n] = x; continue; }
          float acc = 0.0f;
          if (K > 1) {
#pragma unroll
            for (int j = 0; j < K - 1; ++j) acc = fmaf(to_float(taps[side][j].v[n]), window[side][j][n], acc);
          }
          y[side][n] = fmaf(to_float(taps[side][K - 1].v[n]), x, acc);
          if (K > 1) {
#pragma unroll
            for (int j = 0; j + 1 < K - 1; ++j) window[side][j][n] = window[side][j + 1][n];
            window[side][W - 1][n] = x;
          }
        }
        if (K > 1 && p.single && keep > 0) {         // one token a request: nobody else reads what was held
#pragma unroll
          for (int j = 0; j < K - 1; ++j) {
            const int place = j - (K - p.num_taps);
            if (place >= 0) {
#pragma unroll
              for (int n = 0; n < N; ++n) held[(size_t)place * channels + side * mate + n] = window[side][j][n];
            }
          }
        }
      }
      if (turns) {
        const ApPiece<float2, N> cs = *reinterpret_cast<const ApPiece<float2, N>*>(run_cs + (t - t_begin) * half + i);
#pragma unroll
        for (int n = 0; n < N; ++n) {
          const float u0 = y[0][n], w0 = y[1][n];
          y[0][n] = u0 * cs.v[n].x - w0 * cs.v[n].y;
          y[1][n] = w0 * cs.v[n].x + u0 * cs.v[n].y;
        }
      }
      T* to[2];
      if (kind == 0) {
        to[0] = (T*)p.q_out + (size_t)t * p.q_stride + c;
        to[1] = to[0] + mate;
      } else {
        const long long place = place_of[kind - 1][t - t_begin];
        if (place < 0) continue;
        T* at = (T*)(kind == 1 ? p.k_cache : p.v_cache) + place;
        to[0] = at + inside[0];
        to[1] = at + inside[1];
      }
#pragma unroll
      for (int side = 0; side < 2; ++side) {
        if (side == 1 && !mate) break;
        ApPiece<T, N> r;
#pragma unroll
        for (int n = 0; n < N; ++n) r.v[n] = from_float<T>(y[side][n]);
        *reinterpret_cast<ApPiece<T, N>*>(to[side]) = r;
      }
    }
  }
}

template <typename T, int N>
static cudaError_t launch_attention_prepare(AttentionPrepareParams& p, bool norm, cudaStream_t stream) {
  const int rest = p.D - p.rot, in_rest = rest % (2 * N) == 0 ? rest / 2 / N : rest / N;
  const int in_values = p.v_width % (2 * N) == 0 ? p.v_width / 2 / N : p.v_width / N;
  const int units = (p.write ? p.H + p.G : p.H) * (p.rot / 2 / N + in_rest) + (p.write ? in_values : 0);
  const int wanted = (units + 31) / 32 * 32, threads = wanted < AP_MAX_THREADS ? wanted : AP_MAX_THREADS;
  if (norm && p.num_taps == 0)
    return kvb_launch((attention_prepare_kernel<T, N, true, false>), dim3(p.tokens), dim3(threads), 0, stream, true, p);
  if constexpr (N <= 4) {
    if (norm)
      return kvb_launch((attention_prepare_kernel<T, N, true, true>), dim3(p.tokens), dim3(threads), 0, stream, true, p);
    if (p.num_taps > AP_MAX_TAPS)
      return kvb_launch((attention_prepare_kernel<T, N, false, true>), dim3(p.tokens), dim3(threads), 0, stream, true, p);
  } else {
    return cudaErrorInvalidValue;                    // (pieces this wide are for the case above)
  }
  if constexpr (N <= 4) {
    // short runs while there are few tokens (a result does not depend on the run)
    p.run = p.single ? 1 : p.tokens >= 1024 ? AP_RUN : p.tokens >= 128 ? 8 : 4;
    const size_t turn_bytes = (size_t)p.rot / 2 * sizeof(float2);
    while (p.run > 1 && p.run * turn_bytes > 32 * 1024) p.run /= 2;
    const dim3 grid((units + AP_RUN_THREADS - 1) / AP_RUN_THREADS, (p.tokens + p.run - 1) / p.run);
#define KVB_AP_RUNS(K_) kvb_launch((attention_prepare_runs_kernel<T, N, K_>), grid, dim3(AP_RUN_THREADS), p.run * turn_bytes, stream, true, p)
    return p.num_taps <= 1 ? KVB_AP_RUNS(1) : p.num_taps <= 4 ? KVB_AP_RUNS(4) : KVB_AP_RUNS(AP_MAX_TAPS);
#undef KVB_AP_RUNS
  }
}

// rows: [q | k | v] of every token (row stride `row_stride`); q_out: rows of q (may be `rows` itself without taps);
// cos_sin null: nothing turns; taps null: no convolution; q_weight null: no norm.
extern "C" int kvb_attention_prepare(const void* rows, long long row_stride, void* q_out, long long q_stride,
                                     const float* cos_sin, int rot, const int* positions, const int* req_index,
                                     const int* query_start, const int* state_slots, const int* table, int table_stride,
                                     void* k_cache, long long k_page, long long k_head, long long k_row, void* v_cache,
                                     long long v_page, long long v_head, long long v_row, int page_size, int num_pages,
                                     int write, int tokens, int num_reqs, int H, int G, int D, int V, const void* taps, int num_taps, float* state,
                                     long long state_stride, long long state_offset, const void* q_weight,
                                     const void* k_weight, float eps, int dtype, cudaStream_t stream) {
  if (tokens == 0) return 0;
  if (cos_sin == nullptr) rot = 0;
  if (taps == nullptr) num_taps = 0;
  KVB_REQUIRE(H > 0 && G > 0 && D > 0 && V > 0, "attention_prepare: bad sizes");
  const int v_width = G * V;
  KVB_REQUIRE(rot >= 0 && rot % 2 == 0 && rot <= D, "attention_prepare: the turned entries are an even number within the head");
  KVB_REQUIRE((tokens + 3) / 4 <= 65535 || tokens == num_reqs, "attention_prepare: too many tokens for one launch");
  KVB_REQUIRE((long long)rot / 2 * 8 <= 40 * 1024, "attention_prepare: too many turned entries");
  KVB_REQUIRE(taps == nullptr || (num_taps >= 1 && q_out != rows), "attention_prepare: convolved queries need rows of their own");
  KVB_REQUIRE(num_taps < 2 || (state != nullptr && query_start != nullptr && state_slots != nullptr),
              "attention_prepare: a convolution needs the state rows and the batch's request arrays");
  KVB_REQUIRE((q_weight == nullptr) == (k_weight == nullptr), "attention_prepare: give both norm weights or none");
  AttentionPrepareParams p;
  p.rows = rows; p.row_stride = row_stride; p.q_out = q_out; p.q_stride = q_stride;
  p.cos_sin = (const float2*)cos_sin; p.rot = rot; p.positions = positions; p.req_index = req_index;
  p.query_start = query_start; p.state_slots = state_slots; p.table = table; p.table_stride = table_stride;
  p.k_cache = k_cache; p.k_page = k_page; p.k_head = k_head; p.k_row = k_row;
  p.v_cache = v_cache; p.v_page = v_page; p.v_head = v_head; p.v_row = v_row; p.V = V;
  p.page_size = page_size; p.num_pages = num_pages; p.write = write; p.tokens = tokens;
  p.H = H; p.G = G; p.D = D; p.v_width = v_width; p.taps = taps; p.num_taps = num_taps; p.state = state;
  p.state_stride = state_stride; p.state_offset = state_offset; p.single = tokens == num_reqs;
  p.q_weight = q_weight; p.k_weight = k_weight; p.eps = eps; p.run = 1;
  p.status = kvb_status_word();
  KVB_REQUIRE(p.status != nullptr, "attention_prepare: no status word");
  // entries a piece: 16 bytes where a block owns a token and nothing is convolved, else 4 entries
  const int n = q_weight != nullptr && num_taps == 0 && dtype != KVB_F32 ? 8 : 4;
  const bool vec = (rot / 2) % n == 0 && D % n == 0 && v_width % n == 0 && row_stride % n == 0 && q_stride % n == 0 &&
                   (v_head == V || V % n == 0) && (k_page | k_head | k_row | v_page | v_head | v_row) % n == 0 &&
                   aligned16(rows) && aligned16(q_out) && aligned16(cos_sin) && aligned16(k_cache) &&
                   (uintptr_t)v_cache % (n * (dtype == KVB_F32 ? 4 : 2)) == 0 && aligned16(taps) &&
                   aligned16(q_weight) && aligned16(k_weight);
  cudaError_t err;
  const bool norm = q_weight != nullptr;
  if (dtype == KVB_F32) err = vec ? launch_attention_prepare<float, 4>(p, norm, stream) : launch_attention_prepare<float, 1>(p, norm, stream);
  else if (vec && n == 8) err = launch_attention_prepare<bf16, 8>(p, norm, stream);
  else err = vec ? launch_attention_prepare<bf16, 4>(p, norm, stream) : launch_attention_prepare<bf16, 1>(p, norm, stream);
  KVB_CHECK_CUDA(err);
  KVB_CHECK_LAUNCH();
  if (num_taps > 1 && !p.single)
    return kvb_keep_inputs(state, state_stride, state_offset, rows, row_stride, H * D + G * D + v_width, num_taps - 1,
                           query_start, state_slots, num_reqs, dtype, stream);
  return 0;
}

KVB_TRACE_TU(attention_prepare)
