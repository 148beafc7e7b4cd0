// Operations on the residual stream between a layer's sublayers and the next layer.
//
//   sum_updates      hidden += a + b (+ a rounded copy of the result): the updates of two sublayers that read the same norm
//   side_gate        gelu(g) * e, e a token's row of a table with one piece per layer: the per-layer token input
//   depth_mix        x = hidden + norm(update);  history[last] = x;  hidden = sum_j a_j history[j];  out = norm(hidden):
//                    the average over the results of all layers so far, between the norms on either side of it
//
// The stream, the history and all sums are float; T is the element type of updates and normed rows.
#include "common.cuh"

using namespace erb;

ERB_DEFINE_LAST_ERROR(erb_last_error)

#define ERB_OUT_CAST 0
#define ERB_OUT_LAYERNORM 1
#define ERB_OUT_RMSNORM 2

namespace {

// An update of the stream: rows of T, or (n_parts > 0) float partial sums [n_parts][rows][width] added in their order.
struct Update {
  const void* data;
  int n_parts;
  size_t part_stride;
};

// Four (VEC) or one neighbouring entries of an update's row at element offset `at`.
template <typename T, int N>
__device__ __forceinline__ void load_update(const Update& u, size_t at, float* v) {
  if (u.n_parts > 0) {
    const float* p = static_cast<const float*>(u.data) + at;
    if constexpr (N == 4) load4(p, v); else v[0] = *p;
#pragma unroll 4
    for (int s = 1; s < u.n_parts; ++s) {
      float m[N];
      if constexpr (N == 4) load4(p + s * u.part_stride, m); else m[0] = p[s * u.part_stride];
#pragma unroll
      for (int i = 0; i < N; ++i) v[i] += m[i];
    }
  } else {
    const T* p = static_cast<const T*>(u.data) + at;
    if constexpr (N == 4) Pack4<T>::load(p, v); else v[0] = Elem<T>::load(p);
  }
}
template <int N> __device__ __forceinline__ void load_f(const float* p, float* v) {
  if constexpr (N == 4) load4(p, v); else v[0] = *p;
}
template <int N> __device__ __forceinline__ void store_f(float* p, const float* v) {
  if constexpr (N == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); else *p = v[0];
}
template <typename T, int N> __device__ __forceinline__ void store_t(T* p, const float* v) {
  if constexpr (N == 4) Pack4<T>::store(p, v); else Elem<T>::store(p, v[0]);
}

template <typename T, int N>
__global__ void __launch_bounds__(256)
sum_updates_kernel(float* __restrict__ hidden, Update a, Update b, T* __restrict__ out, size_t total) {
  chain_wait();
  for (size_t i = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * N; i < total; i += (size_t)gridDim.x * blockDim.x * N) {
    float h[N], x[N];
    load_f<N>(hidden + i, h);
    load_update<T, N>(a, i, x);
    if (b.data) {
      float z[N];
      load_update<T, N>(b, i, z);
#pragma unroll
      for (int k = 0; k < N; ++k) x[k] += z[k];
    }
#pragma unroll
    for (int k = 0; k < N; ++k) h[k] += x[k];
    store_f<N>(hidden + i, h);
    if (out) store_t<T, N>(out + i, h);
  }
}

// out[t][i] = gelu(g[t][i]) * table[ids[t]][offset + i] for i < dim, zeros from there to the end of the row; a token id outside the table reads as zeros (the embedding's
// kernel has flagged it).
template <typename T>
__global__ void side_gate_kernel(const T* __restrict__ g, int ld_g, const T* __restrict__ table, int table_ld, int vocab,
                                 const int* __restrict__ ids, int offset, int dim, T* __restrict__ out, int ld_out) {
  chain_wait();
  const int t = blockIdx.x, id = ids[t];
  const T* e = table + (size_t)(id >= 0 && id < vocab ? id : 0) * table_ld + offset;
  const bool real = id >= 0 && id < vocab;
  for (int i = blockIdx.y * blockDim.x + threadIdx.x; i < ld_out; i += gridDim.y * blockDim.x)
    Elem<T>::store(out + (size_t)t * ld_out + i,
                   real && i < dim ? gelu_tanh_mul(Elem<T>::load(g + (size_t)t * ld_g + i), Elem<T>::load(e + i)) : 0.f);
}

// One block per row; the row is parked in shared memory between the passes.  A thread owns the groups of N neighbouring
// entries threadIdx.x, threadIdx.x + blockDim.x, ... of the row.
template <typename T, int N>
__global__ void __launch_bounds__(512)
depth_mix_kernel(float* __restrict__ hidden, Update delta, const float* __restrict__ post_w, float post_eps,
                 float* __restrict__ history, size_t layer_stride, int n_history, const float* __restrict__ mix, int out_kind,
                 const float* __restrict__ w, const float* __restrict__ b, float eps, T* __restrict__ out, int out_ld,
                 const int* __restrict__ rows, int width, int write_back) {
  chain_wait();
  extern __shared__ __align__(16) float row_s[];          // width floats, then 32 of scratch
  float* scratch = row_s + ((width + 3) & ~3);
  const int o = blockIdx.x, r = rows ? rows[o] : o;
  const size_t at = (size_t)r * width;
  const float inv_w = 1.f / (float)width;
  const int step = blockDim.x * N;
  float rs = 1.f;
  if (delta.data) {
    float ss = 0.f;
    for (int i = threadIdx.x * N; i < width; i += step) {
      float v[N];
      load_update<T, N>(delta, at + i, v);
      store_f<N>(row_s + i, v);
#pragma unroll
      for (int k = 0; k < N; ++k) ss = fmaf(v[k], v[k], ss);
    }
    if (post_w) rs = rsqrtf(block_sum(ss, scratch) * inv_w + post_eps);
  }
  const float own = mix[n_history];
  float sum = 0.f;
  for (int i = threadIdx.x * N; i < width; i += step) {
    float x[N], acc[N];
    load_f<N>(hidden + at + i, x);
    if (delta.data) {
      float v[N], pw[N];
      load_f<N>(row_s + i, v);                              // (written by this thread)
      if (post_w) {
        load_f<N>(post_w + i, pw);
#pragma unroll
        for (int k = 0; k < N; ++k) v[k] *= rs * pw[k];
      }
#pragma unroll
      for (int k = 0; k < N; ++k) x[k] += v[k];
    }
#pragma unroll
    for (int k = 0; k < N; ++k) acc[k] = 0.f;
    const float* past = history + at + i;
#pragma unroll 8
    for (int j = 0; j < n_history; ++j) {
      float v[N];
      load_f<N>(past + j * layer_stride, v);
      const float a = mix[j];
#pragma unroll
      for (int k = 0; k < N; ++k) acc[k] = fmaf(a, v[k], acc[k]);
    }
#pragma unroll
    for (int k = 0; k < N; ++k) acc[k] = fmaf(own, x[k], acc[k]);
    if (write_back) {
      store_f<N>(history + (size_t)n_history * layer_stride + at + i, x);
      store_f<N>(hidden + at + i, acc);
    }
    store_f<N>(row_s + i, acc);
#pragma unroll
    for (int k = 0; k < N; ++k) sum += out_kind == ERB_OUT_RMSNORM ? acc[k] * acc[k] : acc[k];
  }
  if (!out) return;
  T* y = out + (size_t)o * out_ld;
  float mean = 0.f, scale = 1.f;
  if (out_kind == ERB_OUT_RMSNORM) {
    scale = rsqrtf(block_sum(sum, scratch) * inv_w + eps);
  } else if (out_kind == ERB_OUT_LAYERNORM) {
    mean = block_sum(sum, scratch) * inv_w;
    float sq = 0.f;
    for (int i = threadIdx.x * N; i < width; i += step) {
      float v[N];
      load_f<N>(row_s + i, v);
#pragma unroll
      for (int k = 0; k < N; ++k) sq = fmaf(v[k] - mean, v[k] - mean, sq);
    }
    scale = rsqrtf(block_sum(sq, scratch) * inv_w + eps);
  }
  for (int i = threadIdx.x * N; i < width; i += step) {
    float v[N];
    load_f<N>(row_s + i, v);
    if (out_kind != ERB_OUT_CAST) {
      float ww[N], wb[N];
      load_f<N>(w + i, ww);
#pragma unroll
      for (int k = 0; k < N; ++k) wb[k] = 0.f;
      if (b) load_f<N>(b + i, wb);
#pragma unroll
      for (int k = 0; k < N; ++k) v[k] = (v[k] - mean) * scale * ww[k] + wb[k];
    }
    store_t<T, N>(y + i, v);
  }
}

// The same for rows of up to 2,048 V entries of whole 16-byte pieces: a thread owns the groups of four entries threadIdx.x +
// v * blockDim.x, which stay in registers, and everything it reads (the update, the stream, the history) is asked for before
// the first sum over the block.
template <typename T, int V>
__global__ void __launch_bounds__(512)
depth_mix_reg_kernel(float* __restrict__ hidden, Update delta, const float* __restrict__ post_w, float post_eps,
                     float* __restrict__ history, size_t layer_stride, int n_history, const float* __restrict__ mix, int out_kind,
                     const float* __restrict__ w, const float* __restrict__ b, float eps, T* __restrict__ out, int out_ld,
                     const int* __restrict__ rows, int width, int write_back) {
  __shared__ float scratch[32];
  const int groups = width >> 2;
  chain_wait();
  const int o = blockIdx.x, r = rows ? rows[o] : o;
  const size_t at = (size_t)r * width;
  const float inv_w = 1.f / (float)width;
  float d[V][4], x[V][4], acc[V][4];
  float ss = 0.f;
#pragma unroll
  for (int v = 0; v < V; ++v) {
    const int g = threadIdx.x + v * blockDim.x;
#pragma unroll
    for (int k = 0; k < 4; ++k) d[v][k] = x[v][k] = acc[v][k] = 0.f;
    if (g >= groups) continue;
    load4(hidden + at + 4 * g, x[v]);
    if (delta.data) load_update<T, 4>(delta, at + 4 * g, d[v]);
    const float* past = history + at + 4 * g;
    int j = 0;
    for (; j + 4 <= n_history; j += 4) {
      float h[4][4];
#pragma unroll
      for (int i = 0; i < 4; ++i) load4(past + (size_t)(j + i) * layer_stride, h[i]);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float a = mix[j + i];
#pragma unroll
        for (int k = 0; k < 4; ++k) acc[v][k] = fmaf(a, h[i][k], acc[v][k]);
      }
    }
    for (; j < n_history; ++j) {
      float h[4];
      load4(past + (size_t)j * layer_stride, h);
      const float a = mix[j];
#pragma unroll
      for (int k = 0; k < 4; ++k) acc[v][k] = fmaf(a, h[k], acc[v][k]);
    }
#pragma unroll
    for (int k = 0; k < 4; ++k) ss = fmaf(d[v][k], d[v][k], ss);
  }
  const float own = mix[n_history];
  const float rs = post_w ? rsqrtf(block_sum(ss, scratch) * inv_w + post_eps) : 1.f;
  float sum = 0.f;
#pragma unroll
  for (int v = 0; v < V; ++v) {
    const int g = threadIdx.x + v * blockDim.x;
    if (g >= groups) continue;
    if (post_w) {
      float pw[4];
      load4(post_w + 4 * g, pw);
#pragma unroll
      for (int k = 0; k < 4; ++k) d[v][k] *= rs * pw[k];
    }
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      x[v][k] += d[v][k];
      acc[v][k] = fmaf(own, x[v][k], acc[v][k]);
      sum += out_kind == ERB_OUT_RMSNORM ? acc[v][k] * acc[v][k] : acc[v][k];
    }
    if (write_back) {
      store_f<4>(history + (size_t)n_history * layer_stride + at + 4 * g, x[v]);
      store_f<4>(hidden + at + 4 * g, acc[v]);
    }
  }
  if (!out) return;
  float mean = 0.f, scale = 1.f;
  if (out_kind == ERB_OUT_RMSNORM) {
    scale = rsqrtf(block_sum(sum, scratch) * inv_w + eps);
  } else if (out_kind == ERB_OUT_LAYERNORM) {
    mean = block_sum(sum, scratch) * inv_w;
    float sq = 0.f;
#pragma unroll
    for (int v = 0; v < V; ++v) {
      if ((int)(threadIdx.x + v * blockDim.x) >= groups) continue;
#pragma unroll
      for (int k = 0; k < 4; ++k) sq = fmaf(acc[v][k] - mean, acc[v][k] - mean, sq);
    }
    scale = rsqrtf(block_sum(sq, scratch) * inv_w + eps);
  }
  T* y = out + (size_t)o * out_ld;
#pragma unroll
  for (int v = 0; v < V; ++v) {
    const int g = threadIdx.x + v * blockDim.x;
    if (g >= groups) continue;
    float res[4];
    if (out_kind == ERB_OUT_CAST) {
#pragma unroll
      for (int k = 0; k < 4; ++k) res[k] = acc[v][k];
    } else {
      float ww[4], wb[4] = {0.f, 0.f, 0.f, 0.f};
      load4(w + 4 * g, ww);
      if (b) load4(b + 4 * g, wb);
#pragma unroll
      for (int k = 0; k < 4; ++k) res[k] = (acc[v][k] - mean) * scale * ww[k] + wb[k];
    }
    Pack4<T>::store(y + 4 * g, res);
  }
}

bool aligned16(const void* p) { return ((uintptr_t)p & 15) == 0; }

}  // namespace

// hidden += a (+ b); out (may be null) = the result in the element type.  a, b: rows of the element type, or (parts > 0)
// float partial sums whose parts lie `stride` floats apart.  total = rows * width.
ERB_EXPORT int erb_sum_updates(float* hidden, const void* a, int a_parts, long long a_stride, const void* b, int b_parts,
                               long long b_stride, void* out, long long total, void* stream) {
  if (total <= 0) return ERB_OK;
  if (!a || !hidden) return fail(ERB_ERR_ARG, "sum_updates: an update is missing");
  const Update ua{a, a_parts, (size_t)a_stride}, ub{b, b_parts, (size_t)b_stride};
  const bool vec = total % 4 == 0 && aligned16(hidden) && aligned16(a) && aligned16(b) && aligned16(out) && a_stride % 4 == 0 && b_stride % 4 == 0;
  const long long groups = vec ? total / 4 : total;
  const unsigned blocks = (unsigned)((groups + 255) / 256 < 148 * 16 ? (groups + 255) / 256 : 148 * 16);
  if (vec)
    launch_chained(sum_updates_kernel<elem_t, 4>, dim3(blocks), dim3(256), 0, (cudaStream_t)stream, hidden, ua, ub, (elem_t*)out, (size_t)total);
  else
    launch_chained(sum_updates_kernel<elem_t, 1>, dim3(blocks), dim3(256), 0, (cudaStream_t)stream, hidden, ua, ub, (elem_t*)out, (size_t)total);
  return check_launch("sum_updates");
}

ERB_EXPORT int erb_side_gate(const void* g, int ld_g, const void* table, int table_ld, int vocab, const int* ids, int offset, int dim,
                             void* out, int ld_out, int n_tokens, void* stream) {
  if (n_tokens <= 0) return ERB_OK;
  if (dim <= 0 || ld_g < dim || ld_out < dim || offset < 0 || offset + dim > table_ld || vocab <= 0) return fail(ERB_ERR_ARG, "side_gate: bad sizes");
  launch_chained(side_gate_kernel<elem_t>, dim3(n_tokens, (ld_out + 127) / 128), dim3(128), 0, (cudaStream_t)stream, (const elem_t*)g, ld_g,
                 (const elem_t*)table, table_ld, vocab, ids, offset, dim, (elem_t*)out, ld_out);
  return check_launch("side_gate");
}

// n_history: how many layers' results precede this one in `history` (float, `layer_stride` floats apart, rows of `width`);
// mix: float [n_history + 1].  delta (may be null) as in erb_sum_updates; post_w: unit RMS times a weight acts on it first.
// out (may be null): out_kind 0 a rounded copy, 1 layer norm (b may be null), 2 RMS norm.  `rows` selects the rows that
// `out` gets; nothing is then written to hidden and history.
ERB_EXPORT int erb_depth_mix(float* hidden, const void* delta, int n_parts, long long part_stride, const float* post_w, float post_eps,
                             float* history, long long layer_stride, int n_history, const float* mix, int out_kind, const float* w,
                             const float* b, float eps, void* out, int out_ld, const int* rows, int n_rows, int width,
                             int write_back, void* stream) {
  if (n_rows <= 0) return ERB_OK;
  if (width <= 0 || n_history < 0 || !mix || !history || (out && out_ld < width) || (post_w && !delta) || out_kind < 0 || out_kind > 2 ||
      (out && out_kind != ERB_OUT_CAST && !w) || (rows && write_back))
    return fail(ERB_ERR_ARG, "depth_mix: bad sizes or missing tensors");
  const size_t smem = sizeof(float) * ((size_t)((width + 3) & ~3) + 32);
  if (smem > 200 * 1024) return fail(ERB_ERR_UNSUPPORTED, "depth_mix: width %d does not fit shared memory", width);
  const Update u{delta, n_parts, (size_t)part_stride};
  const bool vec = width % 4 == 0 && layer_stride % 4 == 0 && part_stride % 4 == 0 && out_ld % 4 == 0 && aligned16(hidden) &&
                   aligned16(delta) && aligned16(post_w) && aligned16(history) && aligned16(w) && aligned16(b) && aligned16(out);
  const int groups = vec ? width / 4 : width;
  const int threads = groups >= 512 ? 512 : (groups + 31) / 32 * 32;
  if (vec && groups <= 4 * 512) {
    auto reg = groups <= 512 ? depth_mix_reg_kernel<elem_t, 1> : groups <= 1024 ? depth_mix_reg_kernel<elem_t, 2> : depth_mix_reg_kernel<elem_t, 4>;
    launch_chained(reg, dim3(n_rows), dim3(threads), 0, (cudaStream_t)stream, hidden, u, post_w, post_eps, history, (size_t)layer_stride,
                   n_history, mix, out_kind, w, b, eps, (elem_t*)out, out_ld, rows, width, write_back);
    return check_launch("depth_mix");
  }
  auto kern = vec ? depth_mix_kernel<elem_t, 4> : depth_mix_kernel<elem_t, 1>;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return fail(ERB_ERR_CUDA, "depth_mix: %s", cudaGetErrorString(e));
  }
  launch_chained(kern, dim3(n_rows), dim3(threads), smem, (cudaStream_t)stream, hidden, u, post_w, post_eps, history, (size_t)layer_stride,
                 n_history, mix, out_kind, w, b, eps, (elem_t*)out, out_ld, rows, width, write_back);
  return check_launch("depth_mix");
}
