// Mixers that carry a matrix-valued state per request and head instead of cached keys and values.
// Everything between the projections and the output projection is 32-bit: decays, step sizes, unit
// norms, the state, the read-out and the norm behind it.
//
//   state_scan (state_scan.cuh): the state of a (request, head) runs over the request's tokens of this step in order.
//   gla_prepare writes the vectors of the decay-per-channel form (q times its scale, k, a = sigmoid(z)^(1/tau))
//   once a token, so the blocks that share a head do not each take the exponentials.
//
//   conv_prepare (delta rule): a short causal convolution over time per channel on the q, k and v
//   projections (taps [channels, C], the last tap on the current token; the C - 1 inputs in front of a
//   portion come from the request's state row), SiLU, q and k made unit vectors per head (q also times
//   `q_scale`), beta = sigmoid(b), g = exp(-exp(A_log) softplus(a + dt_bias)).  conv_state_update then
//   moves the last C - 1 inputs of every request into its state row.
//
//   gated_rms_norm: out[t, h, :] = o[t, h, :] / rms(o[t, h, :]) * weight * silu(gate[t, h, :]) * scale
//   (or sigmoid(gate) in place of silu(gate); without a weight where none is given).
#include "state_scan.cuh"

// What the decay-per-channel scan reads, 32-bit [T, 3 * H * D]: q times q_scale, k, and the decays
// a = sigmoid(z)^(1/tau) = exp(log_sigmoid(z) / tau) with log_sigmoid(z) = min(z, 0) - log1p(exp(-|z|)).
template <typename T>
__global__ void __launch_bounds__(256)
gla_prepare_kernel(float* __restrict__ out, const T* __restrict__ q, const T* __restrict__ k, long long row_stride,
                   const T* __restrict__ z, long long z_stride, long long tokens, int width, float q_scale,
                   float inv_tau) {
  KVB_KERNEL_PROLOGUE(KVB_TAG_GLA_PREPARE);
  const long long total = tokens * width;
  for (long long e = (long long)blockIdx.x * blockDim.x + threadIdx.x; e < total; e += (long long)gridDim.x * blockDim.x) {
    const long long t = e / width;
    const int i = (int)(e - t * width);
    float* row = out + t * 3 * width;
    const float zv = to_float(z[t * z_stride + i]);
    row[i] = to_float(q[t * row_stride + i]) * q_scale;
    row[width + i] = to_float(k[t * row_stride + i]);
    row[2 * width + i] = expf((fminf(zv, 0.0f) - log1pf(expf(-fabsf(zv)))) * inv_tau);
  }
}

// Decay per key channel.  q, k, v: columns of the projected rows (row stride `row_stride`, heads side by side);
// z [T, H * D] (row stride z_stride): the decay's logits; prepared: scratch, 32-bit [T, 3 * H * D].
extern "C" int kvb_gla_scan(float* out, float* prepared, const void* q, const void* k, const void* v,
                            long long row_stride, const void* z, long long z_stride, float* state,
                            long long state_stride, long long state_offset, const int* query_start,
                            const int* state_slots, int tokens, int num_reqs, int heads, int D, int V, float q_scale,
                            float tau, int dtype, cudaStream_t stream) {
  if (num_reqs == 0 || tokens == 0) return 0;
  KVB_REQUIRE(heads > 0 && D > 0 && V > 0 && tau > 0.0f, "gla_scan: bad sizes");
  KVB_REQUIRE(heads <= 65535, "gla_scan: too many heads");
  const int width = heads * D;
  const long long wanted = ((long long)tokens * width + 255) / 256;
  const long long resident = (long long)(kvb_sm_count() > 0 ? kvb_sm_count() : 1) * 16;
  const dim3 grid((unsigned)(wanted < resident ? wanted : resident));
  if (dtype == KVB_F32)
    KVB_CHECK_CUDA(kvb_launch((gla_prepare_kernel<float>), grid, dim3(256), 0, stream, true, prepared, (const float*)q,
        (const float*)k, row_stride, (const float*)z, z_stride, (long long)tokens, width, q_scale, 1.0f / tau));
  else
    KVB_CHECK_CUDA(kvb_launch((gla_prepare_kernel<bf16>), grid, dim3(256), 0, stream, true, prepared, (const bf16*)q,
        (const bf16*)k, row_stride, (const bf16*)z, z_stride, (long long)tokens, width, q_scale, 1.0f / tau));
  ScanParams p = {};
  p.q = prepared; p.k = prepared + width; p.a = prepared + 2 * width; p.vec_token = 3LL * width;
  p.v = v; p.v_token = row_stride;
  p.out = out; p.state = state; p.state_stride = state_stride; p.state_offset = state_offset;
  p.query_start = query_start; p.state_slots = state_slots;
  p.heads = heads; p.kv_share = 1; p.D = D; p.V = V;
  return dtype == KVB_F32 ? launch_state_scan<float, 0>(p, num_reqs, tokens, stream)
                          : launch_state_scan<bf16, 0>(p, num_reqs, tokens, stream);
}

// Delta rule.  prepared [T, 2 * G * D + H * V + 2 * H] 32-bit as conv_prepare leaves it: q, k (G heads), v, beta, gate.
extern "C" int kvb_delta_scan(float* out, const float* prepared, float* state, long long state_stride,
                              long long state_offset, const int* query_start, const int* state_slots, int tokens,
                              int num_reqs, int heads, int kv_heads, int D, int V, cudaStream_t stream) {
  if (num_reqs == 0) return 0;
  KVB_REQUIRE(heads > 0 && kv_heads > 0 && heads % kv_heads == 0 && D > 0 && V > 0, "delta_scan: bad sizes");
  KVB_REQUIRE(heads <= 65535, "delta_scan: too many heads");
  const long long width = 2LL * kv_heads * D + (long long)heads * V + 2LL * heads;
  ScanParams p = {};
  p.q = prepared; p.k = prepared + (size_t)kv_heads * D; p.a = prepared; p.vec_token = width;
  p.v = prepared + 2 * (size_t)kv_heads * D; p.v_token = width;
  p.out = out; p.state = state; p.state_stride = state_stride; p.state_offset = state_offset;
  p.query_start = query_start; p.state_slots = state_slots;
  p.heads = heads; p.kv_share = heads / kv_heads; p.D = D; p.V = V;
  p.beta = prepared + 2 * (size_t)kv_heads * D + (size_t)heads * V;
  p.gate = p.beta + heads;
  p.bg_stride = width;
  return launch_state_scan<float, 1>(p, num_reqs, tokens, stream);
}

// ---- short convolution, activations, unit vectors, step sizes --------------------------------------------------
#define CP_THREADS 128
#define CP_MAX_TAPS 8

template <typename T>
__global__ void __launch_bounds__(CP_THREADS)
conv_prepare_kernel(float* __restrict__ out, long long out_stride, const T* __restrict__ rows, long long row_stride,
                    const T* __restrict__ taps, int num_taps, const float* __restrict__ state, long long state_stride,
                    long long state_offset, const int* __restrict__ req_index, const int* __restrict__ query_start,
                    const int* __restrict__ state_slots, const T* __restrict__ a_log, const T* __restrict__ dt_bias,
                    int heads, int kv_heads, int D, int V, int b_col, int a_col, float q_scale, float unit_eps) {
  KVB_KERNEL_PROLOGUE(KVB_TAG_CONV_PREPARE);
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int req = req_index[t];
  const int first = query_start[req];                 // the portion's first token row
  const int back = t - first;                         // tokens of the portion in front of this one
  const float* held = state + (size_t)state_slots[req] * state_stride + state_offset;   // [channels, taps - 1]
  const int vectors = 2 * kv_heads + heads;
  const T* row = rows + (size_t)t * row_stride;
  float* orow = out + (size_t)t * out_stride;
  for (int n = blockIdx.y * (CP_THREADS / 32) + warp; n < vectors; n += gridDim.y * (CP_THREADS / 32)) {
    const bool unit = n < 2 * kv_heads;
    const int len = unit ? D : V;
    const int c0 = unit ? n * D : 2 * kv_heads * D + (n - 2 * kv_heads) * V;     // first channel of the vector
    float ss = 0.0f;
    for (int i = lane; i < len; i += 32) {
      const int c = c0 + i;
      float acc = 0.0f;
      for (int j = 0; j < num_taps; ++j) {
        const int ago = num_taps - 1 - j;             // tap j reads the input `ago` tokens back
        float x;
        if (ago <= back) x = to_float(rows[(size_t)(t - ago) * row_stride + c]);
        else x = held[(size_t)c * (num_taps - 1) + (num_taps - 1) - (ago - back)];
        acc = fmaf(to_float(taps[(size_t)c * num_taps + j]), x, acc);
      }
      const float y = acc / (1.0f + expf(-acc));
      orow[c] = y;                                    // unit vectors are scaled below
      ss = fmaf(y, y, ss);
    }
    if (unit) {
      const float inv = (n < kv_heads ? q_scale : 1.0f) / sqrtf(warp_sum(ss) + unit_eps);
      __syncwarp();
      for (int i = lane; i < len; i += 32) orow[c0 + i] *= inv;
    }
  }
  if (blockIdx.y == 0) {
    float* extra = orow + 2 * (size_t)kv_heads * D + (size_t)heads * V;
    for (int h = threadIdx.x; h < heads; h += CP_THREADS) {
      const float b = to_float(row[b_col + h]);
      const float a = to_float(row[a_col + h]) + to_float(dt_bias[h]);
      const float softplus = fmaxf(a, 0.0f) + log1pf(expf(-fabsf(a)));
      extra[h] = 1.0f / (1.0f + expf(-b));
      extra[heads + h] = expf(-expf(to_float(a_log[h])) * softplus);
    }
  }
}

// The last taps - 1 inputs of each request, counted over what it held and what this step brought.
template <typename T>
__global__ void conv_state_update_kernel(float* __restrict__ state, long long state_stride, long long state_offset,
                                         const T* __restrict__ rows, long long row_stride, int channels, int keep,
                                         const int* __restrict__ query_start, const int* __restrict__ state_slots) {
  KVB_KERNEL_PROLOGUE(KVB_TAG_CONV_PREPARE);
  const int req = blockIdx.x;
  const int begin = query_start[req], n = query_start[req + 1] - begin;
  float* held = state + (size_t)state_slots[req] * state_stride + state_offset;
  for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < channels; c += gridDim.y * blockDim.x) {
    float fresh[CP_MAX_TAPS];
#pragma unroll
    for (int j = 0; j < CP_MAX_TAPS; ++j) {
      if (j < keep) {
        const int ago = keep - 1 - j;                 // new entry j is the input `ago` tokens before the portion's end
        fresh[j] = ago < n ? to_float(rows[(size_t)(begin + n - 1 - ago) * row_stride + c])
                           : held[(size_t)c * keep + (j + n)];
      }
    }
#pragma unroll
    for (int j = 0; j < CP_MAX_TAPS; ++j)
      if (j < keep) held[(size_t)c * keep + j] = fresh[j];
  }
}

extern "C" int kvb_conv_prepare(float* out, const void* rows, long long row_stride, const void* taps, int num_taps,
                                float* state, long long state_stride, long long state_offset, const int* req_index,
                                const int* query_start, const int* state_slots, const void* a_log, const void* dt_bias,
                                int tokens, int num_reqs, int heads, int kv_heads, int D, int V, int b_col, int a_col,
                                float q_scale, float unit_eps, int dtype, cudaStream_t stream) {
  if (tokens == 0) return 0;
  KVB_REQUIRE(num_taps >= 1 && num_taps <= CP_MAX_TAPS + 1, "conv_prepare: 1 to 9 taps");
  KVB_REQUIRE(heads > 0 && kv_heads > 0 && D > 0 && V > 0, "conv_prepare: bad sizes");
  const int vectors = 2 * kv_heads + heads;
  const long long out_stride = 2LL * kv_heads * D + (long long)heads * V + 2LL * heads;
  int groups = (vectors + CP_THREADS / 32 - 1) / (CP_THREADS / 32);
  if (tokens >= 512 || groups > 65535) groups = 1;     // many tokens: a block a token walks its vectors
  const int channels = 2 * kv_heads * D + heads * V;
  const int update_blocks = (channels + 255) / 256 > 65535 ? 65535 : (channels + 255) / 256;
  if (dtype == KVB_F32) {
    KVB_CHECK_CUDA(kvb_launch((conv_prepare_kernel<float>), dim3(tokens, groups), dim3(CP_THREADS), 0, stream, true,
        out, out_stride, (const float*)rows, row_stride, (const float*)taps, num_taps, (const float*)state, state_stride,
        state_offset, req_index, query_start, state_slots, (const float*)a_log, (const float*)dt_bias, heads, kv_heads,
        D, V, b_col, a_col, q_scale, unit_eps));
    if (num_taps > 1)
      KVB_CHECK_CUDA(kvb_launch((conv_state_update_kernel<float>), dim3(num_reqs, update_blocks), dim3(256), 0, stream,
          true, state, state_stride, state_offset, (const float*)rows, row_stride, channels, num_taps - 1, query_start,
          state_slots));
  } else {
    KVB_CHECK_CUDA(kvb_launch((conv_prepare_kernel<bf16>), dim3(tokens, groups), dim3(CP_THREADS), 0, stream, true,
        out, out_stride, (const bf16*)rows, row_stride, (const bf16*)taps, num_taps, (const float*)state, state_stride,
        state_offset, req_index, query_start, state_slots, (const bf16*)a_log, (const bf16*)dt_bias, heads, kv_heads,
        D, V, b_col, a_col, q_scale, unit_eps));
    if (num_taps > 1)
      KVB_CHECK_CUDA(kvb_launch((conv_state_update_kernel<bf16>), dim3(num_reqs, update_blocks), dim3(256), 0, stream,
          true, state, state_stride, state_offset, (const bf16*)rows, row_stride, channels, num_taps - 1, query_start,
          state_slots));
  }
  KVB_CHECK_LAUNCH();
  return 0;
}

// ---- the norm and the gate behind the read-out -------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(CP_THREADS)
gated_rms_norm_kernel(T* __restrict__ out, long long out_stride, const float* __restrict__ o,
                      const T* __restrict__ gate, long long gate_stride, const T* __restrict__ weight, long long vectors,
                      int heads, int V, float eps, float scale, int sigmoid_gate) {
  KVB_KERNEL_PROLOGUE(KVB_TAG_GATED_NORM);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (long long n = (long long)blockIdx.x * (CP_THREADS / 32) + warp; n < vectors;
       n += (long long)gridDim.x * (CP_THREADS / 32)) {
    const long long t = n / heads;
    const int h = (int)(n % heads);
    const float* src = o + n * V;
    const T* g = gate + t * gate_stride + (long long)h * V;
    T* dst = out + t * out_stride + (long long)h * V;
    float ss = 0.0f;
    for (int i = lane; i < V; i += 32) { const float v = src[i]; ss = fmaf(v, v, ss); }
    const float inv = scale / sqrtf(warp_sum(ss) / (float)V + eps);
    for (int i = lane; i < V; i += 32) {
      const float gv = to_float(g[i]);
      const float sig = 1.0f / (1.0f + expf(-gv));
      dst[i] = from_float<T>(src[i] * inv * (weight != nullptr ? to_float(weight[i]) : 1.0f) * (sigmoid_gate ? sig : gv * sig));
    }
  }
}

// The same for vectors of more than a thousand entries (one norm over all heads of a token): a block a vector.
template <typename T>
__global__ void __launch_bounds__(1024)
gated_rms_norm_wide_kernel(T* __restrict__ out, long long out_stride, const float* __restrict__ o,
                           const T* __restrict__ gate, long long gate_stride, const T* __restrict__ weight, int heads,
                           int V, float eps, float scale, int sigmoid_gate) {
  KVB_KERNEL_PROLOGUE(KVB_TAG_GATED_NORM);
  __shared__ float scratch[32];
  const long long n = blockIdx.x;
  const long long t = n / heads;
  const int h = (int)(n % heads);
  const float* src = o + n * V;
  const T* g = gate + t * gate_stride + (long long)h * V;
  T* dst = out + t * out_stride + (long long)h * V;
  float ss = 0.0f;
  for (int i = threadIdx.x; i < V; i += blockDim.x) { const float v = src[i]; ss = fmaf(v, v, ss); }
  const float inv = scale / sqrtf(block_sum(ss, scratch) / (float)V + eps);
  for (int i = threadIdx.x; i < V; i += blockDim.x) {
    const float gv = to_float(g[i]);
    const float sig = 1.0f / (1.0f + expf(-gv));
    dst[i] = from_float<T>(src[i] * inv * (weight != nullptr ? to_float(weight[i]) : 1.0f) * (sigmoid_gate ? sig : gv * sig));
  }
}

extern "C" int kvb_gated_rms_norm(void* out, long long out_stride, const float* o, const void* gate,
                                  long long gate_stride, const void* weight, int tokens, int heads, int V, float eps,
                                  float scale, int sigmoid_gate, int dtype, cudaStream_t stream) {
  const long long vectors = (long long)tokens * heads;
  if (vectors == 0) return 0;
  KVB_REQUIRE(V > 0, "gated_rms_norm: bad width");
  if (V > 1024 && vectors <= 0x7fffffffLL) {
    // the threads of a block follow the width alone, so a vector's sum does not depend on the batch
    const int wide_threads = V >= 4096 ? 1024 : V >= 2048 ? 512 : 256;
    if (dtype == KVB_F32)
      KVB_CHECK_CUDA(kvb_launch((gated_rms_norm_wide_kernel<float>), dim3((unsigned)vectors), dim3(wide_threads), 0, stream, true,
          (float*)out, out_stride, o, (const float*)gate, gate_stride, (const float*)weight, heads, V, eps, scale,
          sigmoid_gate));
    else
      KVB_CHECK_CUDA(kvb_launch((gated_rms_norm_wide_kernel<bf16>), dim3((unsigned)vectors), dim3(wide_threads), 0, stream, true,
          (bf16*)out, out_stride, o, (const bf16*)gate, gate_stride, (const bf16*)weight, heads, V, eps, scale,
          sigmoid_gate));
    KVB_CHECK_LAUNCH();
    return 0;
  }
  const long long wanted = (vectors + CP_THREADS / 32 - 1) / (CP_THREADS / 32);
  const long long resident = (long long)(kvb_sm_count() > 0 ? kvb_sm_count() : 1) * 16;
  const int blocks = (int)(wanted < resident ? wanted : resident);
  if (dtype == KVB_F32)
    KVB_CHECK_CUDA(kvb_launch((gated_rms_norm_kernel<float>), dim3(blocks), dim3(CP_THREADS), 0, stream, true,
        (float*)out, out_stride, o, (const float*)gate, gate_stride, (const float*)weight, vectors, heads, V, eps, scale, sigmoid_gate));
  else
    KVB_CHECK_CUDA(kvb_launch((gated_rms_norm_kernel<bf16>), dim3(blocks), dim3(CP_THREADS), 0, stream, true,
        (bf16*)out, out_stride, o, (const bf16*)gate, gate_stride, (const bf16*)weight, vectors, heads, V, eps, scale, sigmoid_gate));
  KVB_CHECK_LAUNCH();
  return 0;
}

KVB_TRACE_TU(recurrence)
