// Linear attention with one fixed decay a head (a mode of state_scan.cuh) and what stands in front of the scan:
//   lightning_prepare: silu of q, k and v, q times a factor, 32-bit;
//   retention_prepare: q and k turned by the token's position, k times a factor, 32-bit (the scan reads v where the
//   projection left it).
#include "state_scan.cuh"

// What the fixed-decay scan reads, 32-bit [T, 2 * H * D + H * V]: silu(q) times q_scale, silu(k), silu(v).
// QUADS: four neighbouring entries a thread, loaded and stored as one piece (widths that are multiples of four,
// rows and pointers on the boundaries of such pieces).
template <typename T>
struct __align__(4 * sizeof(T)) ScanQuad { T v[4]; };

__device__ __forceinline__ float scan_silu(float x) { return __fdividef(x, 1.0f + expf(-x)); }

template <typename T, bool QUADS>
__global__ void __launch_bounds__(256)
lightning_prepare_kernel(float* __restrict__ out, const T* __restrict__ q, const T* __restrict__ k,
                         const T* __restrict__ v, long long row_stride, long long tokens, int width, int vwidth,
                         float q_scale) {
  KVB_KERNEL_PROLOGUE(KVB_TAG_LIGHTNING_PREPARE);
  constexpr int N = QUADS ? 4 : 1;
  const int per_token = (2 * width + vwidth) / N;
  const long long total = tokens * per_token;
  for (long long e = (long long)blockIdx.x * blockDim.x + threadIdx.x; e < total; e += (long long)gridDim.x * blockDim.x) {
    const long long t = e / per_token;
    const int i = (int)(e - t * per_token) * N;
    const T* src = (i < width ? q + i : i < 2 * width ? k + (i - width) : v + (i - 2 * width)) + t * row_stride;
    const float factor = i < width ? q_scale : 1.0f;
    if (QUADS) {
      const ScanQuad<T> in = *reinterpret_cast<const ScanQuad<T>*>(src);
      ScanQuad<float> y;
#pragma unroll
      for (int j = 0; j < 4; ++j) y.v[j] = scan_silu(to_float(in.v[j])) * factor;
      *reinterpret_cast<ScanQuad<float>*>(out + e * 4) = y;
    } else {
      out[e] = scan_silu(to_float(src[0])) * factor;
    }
  }
}

// One fixed decay a head.  q, k, v: columns of the projected rows (row stride `row_stride`, heads side by side),
// all three passed through SiLU; decay [H] 32-bit; prepared: scratch, 32-bit [T, 2 * H * D + H * V].
extern "C" int kvb_lightning_scan(float* out, float* prepared, const void* q, const void* k, const void* v,
                                  long long row_stride, const float* decay, float* state, long long state_stride,
                                  long long state_offset, const int* query_start, const int* state_slots, int tokens,
                                  int num_reqs, int heads, int D, int V, float q_scale, int dtype,
                                  cudaStream_t stream) {
  if (num_reqs == 0 || tokens == 0) return 0;
  KVB_REQUIRE(heads > 0 && D > 0 && V > 0 && decay != nullptr, "lightning_scan: bad sizes");
  KVB_REQUIRE(heads <= 65535, "lightning_scan: too many heads");
  const int width = heads * D, vwidth = heads * V;
  const long long per_token = 2LL * width + vwidth;
  const size_t piece = 4 * (dtype == KVB_F32 ? sizeof(float) : sizeof(bf16));
  const bool quads = width % 4 == 0 && vwidth % 4 == 0 && row_stride % 4 == 0 && aligned16(prepared) &&
                     ((uintptr_t)q | (uintptr_t)k | (uintptr_t)v) % piece == 0;
  const long long wanted = ((long long)tokens * per_token / (quads ? 4 : 1) + 255) / 256;
  const long long resident = (long long)(kvb_sm_count() > 0 ? kvb_sm_count() : 1) * 16;
  const dim3 grid((unsigned)(wanted < resident ? wanted : resident));
#define KVB_LP_LAUNCH(T_, Q_)                                                                                  \
  KVB_CHECK_CUDA(kvb_launch((lightning_prepare_kernel<T_, Q_>), grid, dim3(256), 0, stream, true, prepared,    \
      (const T_*)q, (const T_*)k, (const T_*)v, row_stride, (long long)tokens, width, vwidth, q_scale))
  if (dtype == KVB_F32) { if (quads) KVB_LP_LAUNCH(float, true); else KVB_LP_LAUNCH(float, false); }
  else { if (quads) KVB_LP_LAUNCH(bf16, true); else KVB_LP_LAUNCH(bf16, false); }
#undef KVB_LP_LAUNCH
  ScanParams p = {};
  p.q = prepared; p.k = prepared + width; p.a = decay; p.vec_token = per_token;
  p.v = prepared + 2 * width; p.v_token = per_token;
  p.out = out; p.state = state; p.state_stride = state_stride; p.state_offset = state_offset;
  p.query_start = query_start; p.state_slots = state_slots;
  p.heads = heads; p.kv_share = 1; p.D = D; p.V = V;
  return launch_state_scan<float, 2>(p, num_reqs, tokens, stream);
}

// What the scan of turned q and k reads, 32-bit [T, 2 * H * D]: the first `rot` entries of every head turn in halves
// (entry i and entry i + rot / 2 form the pair (u, w) -> (u c - w s, w c + u s) with the token's (c, s) of frequency i),
// the rest pass unchanged; k is multiplied by k_scale after the turn.  A thread takes N neighbouring entries of the
// first half together with their partners, or N entries that do not turn.
template <typename T, int N>
__global__ void __launch_bounds__(256)
retention_prepare_kernel(float* __restrict__ out, const T* __restrict__ q, const T* __restrict__ k, long long row_stride,
                         const float2* __restrict__ cos_sin, int rot, long long tokens, int heads, int D, float k_scale) {
  KVB_KERNEL_PROLOGUE(KVB_TAG_RETENTION_PREPARE);
  struct __align__(N * sizeof(T)) In { T v[N]; };
  struct __align__(N * sizeof(float)) Out { float v[N]; };
  struct __align__(N >= 2 ? 16 : 8) Turn { float2 v[N]; };
  const int half = rot >> 1, turned = half / N, per_head = turned + (D - rot) / N, per_token = 2 * heads * per_head;
  const long long total = tokens * per_token;
  for (long long e = (long long)blockIdx.x * blockDim.x + threadIdx.x; e < total; e += (long long)gridDim.x * blockDim.x) {
    const long long t = e / per_token;
    const int r = (int)(e - t * per_token), n = r / per_head, piece = r - n * per_head;    // n: head of q, then of k
    const bool is_q = n < heads;
    const T* src = (is_q ? q + (long long)n * D : k + (long long)(n - heads) * D) + t * row_stride;
    float* dst = out + (t * 2 * heads + n) * D;
    const float factor = is_q ? 1.0f : k_scale;
    Out y;
    if (piece < turned) {
      const int i = piece * N;
      const In u = *reinterpret_cast<const In*>(src + i), w = *reinterpret_cast<const In*>(src + i + half);
      const Turn cs = *reinterpret_cast<const Turn*>(cos_sin + t * half + i);
      Out z;
#pragma unroll
      for (int j = 0; j < N; ++j) {
        const float a = to_float(u.v[j]), b = to_float(w.v[j]);
        y.v[j] = (a * cs.v[j].x - b * cs.v[j].y) * factor;
        z.v[j] = (b * cs.v[j].x + a * cs.v[j].y) * factor;
      }
      *reinterpret_cast<Out*>(dst + i) = y;
      *reinterpret_cast<Out*>(dst + i + half) = z;
    } else {
      const int i = rot + (piece - turned) * N;
      const In u = *reinterpret_cast<const In*>(src + i);
#pragma unroll
      for (int j = 0; j < N; ++j) y.v[j] = to_float(u.v[j]) * factor;
      *reinterpret_cast<Out*>(dst + i) = y;
    }
  }
}

// q, k, v: columns of the projected rows (row stride `row_stride`, heads side by side); cos_sin [T, rot / 2] pairs or
// null (nothing turns); decay [H] 32-bit; prepared: scratch, 32-bit [T, 2 * H * D].
extern "C" int kvb_retention_scan(float* out, float* prepared, const void* q, const void* k, const void* v,
                                  long long row_stride, const float* cos_sin, int rot, const float* decay, float* state,
                                  long long state_stride, long long state_offset, const int* query_start,
                                  const int* state_slots, int tokens, int num_reqs, int heads, int D, int V, float k_scale,
                                  int dtype, cudaStream_t stream) {
  if (num_reqs == 0 || tokens == 0) return 0;
  KVB_REQUIRE(heads > 0 && D > 0 && V > 0 && decay != nullptr, "retention_scan: bad sizes");
  KVB_REQUIRE(heads <= 65535, "retention_scan: too many heads");
  if (cos_sin == nullptr) rot = 0;
  KVB_REQUIRE(rot >= 0 && rot % 2 == 0 && rot <= D, "retention_scan: the turned entries are an even number within the head");
  const size_t piece = 4 * (dtype == KVB_F32 ? sizeof(float) : sizeof(bf16));
  const bool quads = D % 4 == 0 && rot % 8 == 0 && row_stride % 4 == 0 && aligned16(prepared) && aligned16(cos_sin) &&
                     ((uintptr_t)q | (uintptr_t)k) % piece == 0;
  const long long pieces = (long long)tokens * 2 * heads * (D - rot / 2) / (quads ? 4 : 1);
  const long long wanted = (pieces + 255) / 256;
  const long long resident = (long long)(kvb_sm_count() > 0 ? kvb_sm_count() : 1) * 16;
  const dim3 grid((unsigned)(wanted < resident ? wanted : resident));
#define KVB_RP_LAUNCH(T_, N_)                                                                                      \
  KVB_CHECK_CUDA(kvb_launch((retention_prepare_kernel<T_, N_>), grid, dim3(256), 0, stream, true, prepared, (const T_*)q, \
      (const T_*)k, row_stride, (const float2*)cos_sin, rot, (long long)tokens, heads, D, k_scale))
  if (dtype == KVB_F32) { if (quads) KVB_RP_LAUNCH(float, 4); else KVB_RP_LAUNCH(float, 1); }
  else { if (quads) KVB_RP_LAUNCH(bf16, 4); else KVB_RP_LAUNCH(bf16, 1); }
#undef KVB_RP_LAUNCH
  ScanParams p = {};
  p.q = prepared; p.k = prepared + (size_t)heads * D; p.a = decay; p.vec_token = 2LL * heads * D;
  p.v = v; p.v_token = row_stride;
  p.out = out; p.state = state; p.state_stride = state_stride; p.state_offset = state_offset;
  p.query_start = query_start; p.state_slots = state_slots;
  p.heads = heads; p.kv_share = 1; p.D = D; p.V = V;
  return dtype == KVB_F32 ? launch_state_scan<float, 2>(p, num_reqs, tokens, stream)
                          : launch_state_scan<bf16, 2>(p, num_reqs, tokens, stream);
}

KVB_TRACE_TU(fixed_decay)
