// A selective state-space mixer between its projections: the scan (a mode of state_scan.cuh) and what stands around it.
// Everything is 32-bit inside; the projections come in the activation type.
//
//   ssm_prepare: the convolved channels [x: H V | B: G N | C: G N] of the projected rows pass a causal convolution
//   over time per channel (taps [channels, K] with a bias, the last tap on the current token; the K - 1 inputs in
//   front of a portion come from the request's state row) and SiLU; dt = softplus(dt + dt_bias) and
//   decay = exp(-exp(A_log) dt) per head.  Written as rows [B | C | x | dt | decay].  A thread owns one channel (or
//   four neighbouring ones) for a run of tokens and slides its window over them, so a row is read once.
//   The state row keeps the last K - 1 inputs as [K - 1, channels], oldest first.  In a step of single tokens the
//   thread that has read a channel's inputs also writes the moved ones back; otherwise a second kernel does that,
//   because several runs of a portion may read what the state held.
//
//   gated_group_norm: v = o * silu(z) over the whole read-out of a token, cut into equal parts, each divided by its
//   own root mean square, times a weight over the whole read-out (the gate comes before the norm).  A warp a part
//   for short parts, a block a part for long ones, by the part's width alone: a row's bits do not depend on the batch.
#include "state_scan.cuh"

#define SSM_THREADS 128
#define SSM_RUN 16             // tokens a thread walks
#define SSM_AHEAD 4            // of which it loads this many at once
#define SSM_MAX_TAPS 9

template <typename T, int N>
struct __align__(N * sizeof(T)) SsmPiece { T v[N]; };

// (where exp(-x) runs out of range, x below -88, the quotient is a zero: what is lost is smaller than 1e-36)
__device__ __forceinline__ float ssm_silu(float x) { return __fdividef(x, 1.0f + expf(-x)); }

// N channels a thread; K: taps the window is made for (the model's taps, right-aligned; the places in front are zero).
template <typename T, int N, int K>
__global__ void __launch_bounds__(SSM_THREADS)
ssm_prepare_kernel(float* __restrict__ out, long long out_stride, const T* __restrict__ rows, long long row_stride,
                   const float* __restrict__ taps, int num_taps, const float* __restrict__ bias, float* state,
                   long long state_stride, long long state_offset, const int* __restrict__ req_index,
                   const int* __restrict__ query_start, const int* __restrict__ state_slots,
                   const float* __restrict__ a_log, const float* __restrict__ dt_bias, int tokens, int heads,
                   int x_channels, int channels, int run, int single) {
  KVB_KERNEL_PROLOGUE(KVB_TAG_SSM_PREPARE);
  const int t_begin = blockIdx.y * run, t_end = min(tokens, t_begin + run);
  const int keep = num_taps - 1, bc = channels - x_channels;
  if (blockIdx.x == 0) {                             // step sizes and decays of this run's tokens
    for (int e = threadIdx.x; e < (t_end - t_begin) * heads; e += SSM_THREADS) {
      const int t = t_begin + e / heads, h = e % heads;
      const float a = to_float(rows[(size_t)t * row_stride + channels + h]) + dt_bias[h];
      const float dt = fmaxf(a, 0.0f) + log1pf(expf(-fabsf(a)));
      float* o = out + (size_t)t * out_stride + channels;
      o[h] = dt;
      o[heads + h] = expf(-expf(a_log[h]) * dt);
    }
  }
  const int c = (blockIdx.x * SSM_THREADS + threadIdx.x) * N;
  if (c >= channels) return;
  float w[K][N], b[N], window[K - 1][N];
#pragma unroll
  for (int i = 0; i < N; ++i) {
    b[i] = bias[c + i];
#pragma unroll
    for (int j = 0; j < K; ++j) {
      const int tap = j - (K - num_taps);
      w[j][i] = tap >= 0 ? taps[(size_t)(c + i) * num_taps + tap] : 0.0f;
    }
  }
  // x goes behind B and C
  float* o = out + (c < x_channels ? bc + c : c - x_channels);
  const T* src = rows + c;
  int end = t_begin;                                 // where the request of the token in hand ends
  float* held = nullptr;
  for (int t0 = t_begin; t0 < t_end; t0 += SSM_AHEAD) {
    SsmPiece<T, N> in[SSM_AHEAD];                    // a few tokens' loads in flight together
#pragma unroll
    for (int u = 0; u < SSM_AHEAD; ++u)
      if (t0 + u < t_end) in[u] = *reinterpret_cast<const SsmPiece<T, N>*>(src + (size_t)(t0 + u) * row_stride);
#pragma unroll
    for (int u = 0; u < SSM_AHEAD; ++u) {
      const int t = t0 + u;
      if (t >= t_end) break;
      if (t == end) {                                // the run's first token, or a portion's
        const int req = req_index[t], back = t - query_start[req];
        end = query_start[req + 1];
        held = state + (size_t)state_slots[req] * state_stride + state_offset + c;
#pragma unroll
        for (int j = 0; j < K - 1; ++j) {
          const int ago = K - 1 - j;                 // window[j] is the input `ago` tokens back
          if (ago > keep) {
#pragma unroll
            for (int i = 0; i < N; ++i) window[j][i] = 0.0f;
          } else if (ago <= back) {
            const SsmPiece<T, N> was = *reinterpret_cast<const SsmPiece<T, N>*>(src + (size_t)(t - ago) * row_stride);
#pragma unroll
            for (int i = 0; i < N; ++i) window[j][i] = to_float(was.v[i]);
          } else {
            const SsmPiece<float, N> was = *reinterpret_cast<const SsmPiece<float, N>*>(held + (size_t)(keep - (ago - back)) * channels);
#pragma unroll
            for (int i = 0; i < N; ++i) window[j][i] = was.v[i];
          }
        }
      }
      SsmPiece<float, N> y;
#pragma unroll
      for (int i = 0; i < N; ++i) {
        float acc = b[i];
#pragma unroll
        for (int j = 0; j < K - 1; ++j) acc = fmaf(w[j][i], window[j][i], acc);
        const float x = to_float(in[u].v[i]);
        acc = fmaf(w[K - 1][i], x, acc);
        y.v[i] = ssm_silu(acc);
#pragma unroll
        for (int j = 0; j + 1 < K - 1; ++j) window[j][i] = window[j + 1][i];
        window[K - 2][i] = x;
      }
      *reinterpret_cast<SsmPiece<float, N>*>(o + (size_t)t * out_stride) = y;
      if (single) {                                  // one token a request: nobody else reads what was held
#pragma unroll
        for (int j = 0; j < K - 1; ++j) {
          const int place = j - (K - num_taps);
          if (place >= 0) {
            SsmPiece<float, N> moved;
#pragma unroll
            for (int i = 0; i < N; ++i) moved.v[i] = window[j][i];
            *reinterpret_cast<SsmPiece<float, N>*>(held + (size_t)place * channels) = moved;
          }
        }
      }
    }
  }
}

// The last `keep` inputs of each request, counted over what it held and what this step brought.
template <typename T>
__global__ void __launch_bounds__(SSM_THREADS)
ssm_keep_inputs_kernel(float* state, long long state_stride, long long state_offset, const T* __restrict__ rows,
                       long long row_stride, int channels, int keep, const int* __restrict__ query_start,
                       const int* __restrict__ state_slots) {
  KVB_KERNEL_PROLOGUE(KVB_TAG_SSM_PREPARE);
  const int req = blockIdx.y, c = blockIdx.x * SSM_THREADS + threadIdx.x;
  if (c >= channels) return;
  const int begin = query_start[req], n = query_start[req + 1] - begin;
  float* held = state + (size_t)state_slots[req] * state_stride + state_offset + c;
  for (int j = 0; j < keep; ++j) {                   // ascending: entry j + n is read before it is written
    const int ago = keep - 1 - j;
    held[(size_t)j * channels] = ago < n ? to_float(rows[(size_t)(begin + n - 1 - ago) * row_stride + c])
                                         : held[(size_t)(j + n) * channels];
  }
}

// The same for any mixer whose state holds the last `keep` inputs of a convolution as [keep, channels].
extern "C" int kvb_keep_inputs(float* state, long long state_stride, long long state_offset, const void* rows,
                               long long row_stride, int channels, int keep, const int* query_start,
                               const int* state_slots, int num_reqs, int dtype, cudaStream_t stream) {
  if (num_reqs == 0 || keep == 0) return 0;
  KVB_REQUIRE(num_reqs <= 65535, "keep_inputs: too many requests for one launch");
  const dim3 grid((channels + SSM_THREADS - 1) / SSM_THREADS, num_reqs);
  if (dtype == KVB_F32)
    KVB_CHECK_CUDA(kvb_launch((ssm_keep_inputs_kernel<float>), grid, dim3(SSM_THREADS), 0, stream, true, state, state_stride,
        state_offset, (const float*)rows, row_stride, channels, keep, query_start, state_slots));
  else
    KVB_CHECK_CUDA(kvb_launch((ssm_keep_inputs_kernel<bf16>), grid, dim3(SSM_THREADS), 0, stream, true, state, state_stride,
        state_offset, (const bf16*)rows, row_stride, channels, keep, query_start, state_slots));
  KVB_CHECK_LAUNCH();
  return 0;
}

template <typename T>
static int launch_ssm_prepare(float* out, long long out_stride, const T* rows, long long row_stride, const float* taps,
                              int num_taps, const float* bias, float* state, long long state_stride,
                              long long state_offset, const int* req_index, const int* query_start,
                              const int* state_slots, const float* a_log, const float* dt_bias, int tokens,
                              int num_reqs, int heads, int x_channels, int channels, cudaStream_t stream) {
  const bool quads = x_channels % 4 == 0 && channels % 4 == 0 && row_stride % 4 == 0 && out_stride % 4 == 0 &&
                     state_stride % 4 == 0 && state_offset % 4 == 0 && (uintptr_t)rows % (4 * sizeof(T)) == 0 &&
                     aligned16(out) && aligned16(state);
  const int single = tokens == num_reqs ? 1 : 0;
  const int run = single ? 1 : SSM_RUN;
  const int n = quads ? 4 : 1;
  const dim3 grid((channels / n + SSM_THREADS - 1) / SSM_THREADS, (tokens + run - 1) / run);
  KVB_REQUIRE(grid.y <= 65535 && num_reqs <= 65535, "ssm_prepare: too many tokens for one launch");
#define KVB_SSM_CASE(N_, K_)                                                                                     \
  KVB_CHECK_CUDA(kvb_launch((ssm_prepare_kernel<T, N_, K_>), grid, dim3(SSM_THREADS), 0, stream, true, out, out_stride, \
      rows, row_stride, taps, num_taps, bias, state, state_stride, state_offset, req_index, query_start, state_slots, \
      a_log, dt_bias, tokens, heads, x_channels, channels, run, single))
  if (num_taps <= 4) { if (quads) KVB_SSM_CASE(4, 4); else KVB_SSM_CASE(1, 4); }
  else { if (quads) KVB_SSM_CASE(4, SSM_MAX_TAPS); else KVB_SSM_CASE(1, SSM_MAX_TAPS); }
#undef KVB_SSM_CASE
  if (!single && num_taps > 1)
    KVB_CHECK_CUDA(kvb_launch((ssm_keep_inputs_kernel<T>), dim3((channels + SSM_THREADS - 1) / SSM_THREADS, num_reqs),
        dim3(SSM_THREADS), 0, stream, true, state, state_stride, state_offset, rows, row_stride, channels, num_taps - 1,
        query_start, state_slots));
  KVB_CHECK_LAUNCH();
  return 0;
}

// rows: the first convolved channel of the first token; a head's step size stands behind the channels.
extern "C" int kvb_ssm_prepare(float* out, long long out_stride, const void* rows, long long row_stride,
                               const float* taps, int num_taps, const float* bias, float* state, long long state_stride,
                               long long state_offset, const int* req_index, const int* query_start,
                               const int* state_slots, const float* a_log, const float* dt_bias, int tokens,
                               int num_reqs, int heads, int x_channels, int channels, int dtype, cudaStream_t stream) {
  if (tokens == 0) return 0;
  KVB_REQUIRE(num_taps >= 1 && num_taps <= SSM_MAX_TAPS, "ssm_prepare: 1 to 9 taps");
  KVB_REQUIRE(heads > 0 && x_channels > 0 && channels > x_channels, "ssm_prepare: bad sizes");
  KVB_REQUIRE(out_stride >= channels + 2LL * heads, "ssm_prepare: the output rows are too short");
  if (dtype == KVB_F32)
    return launch_ssm_prepare<float>(out, out_stride, (const float*)rows, row_stride, taps, num_taps, bias, state,
        state_stride, state_offset, req_index, query_start, state_slots, a_log, dt_bias, tokens, num_reqs, heads,
        x_channels, channels, stream);
  return launch_ssm_prepare<bf16>(out, out_stride, (const bf16*)rows, row_stride, taps, num_taps, bias, state,
      state_stride, state_offset, req_index, query_start, state_slots, a_log, dt_bias, tokens, num_reqs, heads,
      x_channels, channels, stream);
}

// ---- the scan ----------------------------------------------------------------------------------------------------------
// Selective state space.  prepared [T, out_stride] 32-bit as ssm_prepare leaves it: B and C (G groups of D entries
// each), x (H heads of V), dt [H], decay [H]; skip [H] 32-bit: the factor of a token's own values in its read-out.
extern "C" int kvb_ssm_scan(float* out, const float* prepared, long long row_stride, const float* skip, float* state,
                            long long state_stride, long long state_offset, const int* query_start,
                            const int* state_slots, int tokens, int num_reqs, int heads, int groups, int D, int V,
                            cudaStream_t stream) {
  if (num_reqs == 0 || tokens == 0) return 0;
  KVB_REQUIRE(heads > 0 && groups > 0 && heads % groups == 0 && D > 0 && V > 0 && skip != nullptr, "ssm_scan: bad sizes");
  KVB_REQUIRE(heads <= 65535, "ssm_scan: too many heads");
  const long long gn = (long long)groups * D;
  KVB_REQUIRE(row_stride >= 2 * gn + (long long)heads * V + 2LL * heads, "ssm_scan: the prepared rows are too short");
  ScanParams p = {};
  p.k = prepared; p.q = prepared + gn; p.a = prepared; p.vec_token = row_stride;
  p.v = prepared + 2 * gn; p.v_token = row_stride;
  p.out = out; p.state = state; p.state_stride = state_stride; p.state_offset = state_offset;
  p.query_start = query_start; p.state_slots = state_slots;
  p.heads = heads; p.kv_share = heads / groups; p.D = D; p.V = V;
  p.beta = prepared + 2 * gn + (long long)heads * V;
  p.gate = p.beta + heads;
  p.bg_stride = row_stride;
  p.skip = skip;
  return launch_state_scan<float, 3>(p, num_reqs, tokens, stream);
}

// ---- the gate and the norm of parts behind the read-out --------------------------------------------------------------
#define GN_WARPS 4
#define GN_PIECES 4            // pieces of N entries a thread keeps between the sum and the store
#define GN_WARP_WIDTH 512      // parts up to this width: a warp each

// WARP: a warp a part (GN_WARPS parts a block); else a block a part.
template <typename T, int N, bool WARP>
__global__ void __launch_bounds__(WARP ? GN_WARPS * 32 : 1024)
gated_group_norm_kernel(T* __restrict__ out, long long out_stride, const float* __restrict__ o,
                        const T* __restrict__ gate, long long gate_stride, const float* __restrict__ weight,
                        long long parts, int groups, int width, float eps) {
  KVB_KERNEL_PROLOGUE(KVB_TAG_GROUP_NORM);
  __shared__ float scratch[32];
  const long long part = WARP ? (long long)blockIdx.x * GN_WARPS + (threadIdx.x >> 5) : (long long)blockIdx.x;
  if (part >= parts) return;                         // a whole warp (or block) leaves
  const int lane = WARP ? threadIdx.x & 31 : threadIdx.x, lanes = WARP ? 32 : blockDim.x;
  const long long t = part / groups;
  const int col = (int)(part % groups) * width;
  const float* src = o + part * width;
  const T* g = gate + t * gate_stride + col;
  T* dst = out + t * out_stride + col;
  const float* wt = weight + col;
  auto gated = [&](int i, float (&v)[N]) {
    const SsmPiece<float, N> a = *reinterpret_cast<const SsmPiece<float, N>*>(src + i);
    const SsmPiece<T, N> z = *reinterpret_cast<const SsmPiece<T, N>*>(g + i);
#pragma unroll
    for (int j = 0; j < N; ++j) v[j] = a.v[j] * ssm_silu(to_float(z.v[j]));
  };
  float kept[GN_PIECES][N];
  SsmPiece<float, N> as[GN_PIECES], ws[GN_PIECES];
  SsmPiece<T, N> zs[GN_PIECES];
  float ss = 0.0f;
#pragma unroll
  for (int s = 0; s < GN_PIECES; ++s) {              // every load of the kept pieces in flight together
    const int i = (lane + s * lanes) * N;
    if (i < width) {
      as[s] = *reinterpret_cast<const SsmPiece<float, N>*>(src + i);
      zs[s] = *reinterpret_cast<const SsmPiece<T, N>*>(g + i);
      ws[s] = *reinterpret_cast<const SsmPiece<float, N>*>(wt + i);
    }
  }
#pragma unroll
  for (int s = 0; s < GN_PIECES; ++s) {
    const int i = (lane + s * lanes) * N;
    if (i < width) {
#pragma unroll
      for (int j = 0; j < N; ++j) kept[s][j] = as[s].v[j] * ssm_silu(to_float(zs[s].v[j]));
#pragma unroll
      for (int j = 0; j < N; ++j) ss = fmaf(kept[s][j], kept[s][j], ss);
    }
  }
  for (int i = (lane + GN_PIECES * lanes) * N; i < width; i += lanes * N) {   // what the registers do not hold
    float v[N];
    gated(i, v);
#pragma unroll
    for (int j = 0; j < N; ++j) ss = fmaf(v[j], v[j], ss);
  }
  const float inv = 1.0f / sqrtf((WARP ? warp_sum(ss) : block_sum(ss, scratch)) / (float)width + eps);
  auto put = [&](int i, const float (&v)[N], const SsmPiece<float, N>& w) {
    SsmPiece<T, N> r;
#pragma unroll
    for (int j = 0; j < N; ++j) r.v[j] = from_float<T>(v[j] * inv * w.v[j]);
    *reinterpret_cast<SsmPiece<T, N>*>(dst + i) = r;
  };
#pragma unroll
  for (int s = 0; s < GN_PIECES; ++s) {
    const int i = (lane + s * lanes) * N;
    if (i < width) put(i, kept[s], ws[s]);
  }
  for (int i = (lane + GN_PIECES * lanes) * N; i < width; i += lanes * N) {
    float v[N];
    gated(i, v);
    put(i, v, *reinterpret_cast<const SsmPiece<float, N>*>(wt + i));
  }
}

template <typename T>
static int launch_gated_group_norm(T* out, long long out_stride, const float* o, const T* gate, long long gate_stride,
                                   const float* weight, int tokens, int groups, int width, float eps,
                                   cudaStream_t stream) {
  const long long parts = (long long)tokens * groups;
  const bool quads = width % 4 == 0 && out_stride % 4 == 0 && gate_stride % 4 == 0 && aligned16(o) && aligned16(weight) &&
                     (uintptr_t)out % (4 * sizeof(T)) == 0 && (uintptr_t)gate % (4 * sizeof(T)) == 0;
  KVB_REQUIRE(parts <= 0x7fffffffLL, "gated_group_norm: too many parts for one launch");
  const bool warp = width <= GN_WARP_WIDTH;
  const dim3 grid((unsigned)(warp ? (parts + GN_WARPS - 1) / GN_WARPS : parts));
  const int threads = warp ? GN_WARPS * 32 : width <= 1024 ? 128 : width <= 4096 ? 256 : width <= 8192 ? 512 : 1024;
#define KVB_GN_CASE(N_, W_)                                                                                       \
  KVB_CHECK_CUDA(kvb_launch((gated_group_norm_kernel<T, N_, W_>), grid, dim3(threads), 0, stream, true, out, out_stride, \
                            o, gate, gate_stride, weight, parts, groups, width, eps))
  if (warp) { if (quads) KVB_GN_CASE(4, true); else KVB_GN_CASE(1, true); }
  else { if (quads) KVB_GN_CASE(4, false); else KVB_GN_CASE(1, false); }
#undef KVB_GN_CASE
  KVB_CHECK_LAUNCH();
  return 0;
}

extern "C" int kvb_gated_group_norm(void* out, long long out_stride, const float* o, const void* gate,
                                    long long gate_stride, const float* weight, int tokens, int groups, int width,
                                    float eps, int dtype, cudaStream_t stream) {
  if (tokens == 0) return 0;
  KVB_REQUIRE(groups > 0 && width > 0, "gated_group_norm: bad sizes");
  if (dtype == KVB_F32)
    return launch_gated_group_norm<float>((float*)out, out_stride, o, (const float*)gate, gate_stride, weight, tokens,
                                          groups, width, eps, stream);
  return launch_gated_group_norm<bf16>((bf16*)out, out_stride, o, (const bf16*)gate, gate_stride, weight, tokens, groups,
                                       width, eps, stream);
}

KVB_TRACE_TU(state_space)
