// Layers whose input is a learned average over everything before them, and a norm without statistics.
//
//   dynamic_tanh   y = tanh(alpha x) w + b, element by element (alpha one number, w and b vectors), for one or
//                  two readers of the same row; an output that is still to be added to the row may come along
//   depth_join     what stands between two layers in one pass over the row.  With x the layer's input, a and f its
//                  two sublayers' results, za and zf the products their gates are made of:
//                      r     = x + mult (sigmoid(za + ba) a + sigmoid(zf + bf) f)
//                      X_n   = r                                  (kept: later layers read it)
//                      x'    = sum_(j < n) depth[j] X_j + depth[n] r
//                      y1,y2 = dynamic_tanh(x')                   (what the next layer's sublayers read)
//                  a may be a pair of results side by side, weight (a / rms(a) gain_a + b / rms(b) gain_b); that norm
//                  is the only sum over the row, everything else is element by element, so a block takes a row
//                  or a part of one.
// Streams, averages and norms are 32-bit; a, f, za, zf, y1 and y2 have the activation type.
#include <initializer_list>

#include "common.cuh"

namespace ek {

constexpr int kDepthThreads = 256;

template <typename T> __device__ __forceinline__ float tanh_of(float x) { return tanhf(x); }
template <> __device__ __forceinline__ float tanh_of<bf16>(float x) { return tanh_by_exp(x); }
template <typename T> __device__ __forceinline__ float sigmoid_of(float x) { return 1.f / (1.f + expf(-x)); }
template <> __device__ __forceinline__ float sigmoid_of<bf16>(float x) { return __fdividef(1.f, 1.f + __expf(-x)); }

// V neighbouring values as floats: V = 4 is one wide access, V = 1 any alignment.
template <typename T, int V> struct Row;
template <typename T> struct Row<T, 4> {
  static __device__ __forceinline__ void load(float* d, const T* p) {
    const float4 v = Vec4<T>::load(p);
    d[0] = v.x; d[1] = v.y; d[2] = v.z; d[3] = v.w;
  }
  static __device__ __forceinline__ void store(T* p, const float* d) {
    Vec4<T>::store(p, make_float4(d[0], d[1], d[2], d[3]));
  }
};
template <typename T> struct Row<T, 1> {
  static __device__ __forceinline__ void load(float* d, const T* p) { d[0] = to_f<T>(*p); }
  static __device__ __forceinline__ void store(T* p, const float* d) { *p = from_f<T>(d[0]); }
};

// tanh(alpha x) w + b; y null: no such reader
struct TanhNorm {
  void* y;
  const float* alpha;
  const float* w;
  const float* b;
};

template <typename T, int V>
__device__ __forceinline__ void write_tanh_norm(const TanhNorm& n, size_t at, int c, const float* x) {
  if (n.y == nullptr) return;
  const float alpha = *n.alpha;
  float w[V], b[V], y[V];
  Row<float, V>::load(w, n.w + c);
  Row<float, V>::load(b, n.b + c);
#pragma unroll
  for (int i = 0; i < V; ++i) y[i] = fmaf(tanh_of<T>(alpha * x[i]), w[i], b[i]);
  Row<T, V>::store((T*)n.y + at, y);
}

// grid (rows, column tiles).  y rows are packed; `rows` (optional) picks stream rows, and the same rows of `add`.
template <typename T, int V>
__global__ void __launch_bounds__(kDepthThreads)
dynamic_tanh_kernel(TanhNorm n1, TanhNorm n2, float* stream, const T* __restrict__ add, const int* __restrict__ rows,
                    int hidden, int write_back) {
  pdl_launch_dependents();
  pdl_wait();
  const int c = (blockIdx.y * kDepthThreads + threadIdx.x) * V;
  if (c >= hidden) return;
  const size_t src = (size_t)(rows ? rows[blockIdx.x] : (int)blockIdx.x) * hidden + c;
  const size_t dst = (size_t)blockIdx.x * hidden + c;
  float x[V];
  Row<float, V>::load(x, stream + src);
  if (add != nullptr) {
    float a[V];
    Row<T, V>::load(a, add + src);
#pragma unroll
    for (int i = 0; i < V; ++i) x[i] += a[i];
    if (write_back) Row<float, V>::store(stream + src, x);
  }
  write_tanh_norm<T, V>(n1, dst, c, x);
  write_tanh_norm<T, V>(n2, dst, c, x);
}

struct DepthJoin {
  const float* x;           // the layer's input [rows, hidden]
  float* x_next;            // may be x itself
  const float* first;       // X_0
  float* kept;              // X_1, X_2, ... `kept_stride` values apart
  long long kept_stride;
  const float* depth;       // n + 1 weights
  int n;                    // results before this one: X_0 .. X_(n-1)
  int keep;                 // this result is read again later: store it as X_n
  float mult;
  const void* a;            // first sublayer's result
  const float* bias_a;      // added to it (null: none; not with a pair)
  const void* b;            // its partner in a pair, or null
  const float* gain_a;      // gains of the pair's two norms
  const float* gain_b;
  float pair_eps, pair_weight;
  const void* za;           // products of the gates, and their biases
  const float* ba;
  const void* f;            // second sublayer's result, or null
  const void* zf;
  const float* bf;
  TanhNorm n1, n2;
  int hidden;
};

template <typename T, int V>
__global__ void __launch_bounds__(kDepthThreads)
depth_join_kernel(const __grid_constant__ DepthJoin p, int cols_per_block) {
  __shared__ float scratch[33];
  pdl_launch_dependents();
  pdl_wait();
  const size_t row = (size_t)blockIdx.x * p.hidden;
  float ra = 1.f, rb = 1.f;
  if (p.b != nullptr) {                          // (every block of a row sums the whole row)
    float sa = 0.f, sb = 0.f;
    for (int c = threadIdx.x * V; c < p.hidden; c += kDepthThreads * V) {
      float a[V], b[V];
      Row<T, V>::load(a, (const T*)p.a + row + c);
      Row<T, V>::load(b, (const T*)p.b + row + c);
#pragma unroll
      for (int i = 0; i < V; ++i) { sa += a[i] * a[i]; sb += b[i] * b[i]; }
    }
    ra = p.pair_weight * rsqrtf(block_sum(sa, scratch) / (float)p.hidden + p.pair_eps);
    rb = p.pair_weight * rsqrtf(block_sum(sb, scratch) / (float)p.hidden + p.pair_eps);
  }
  const int c_end = min(p.hidden, (int)(blockIdx.y + 1) * cols_per_block);
  for (int c = blockIdx.y * cols_per_block + threadIdx.x * V; c < c_end; c += kDepthThreads * V) {
    const size_t at = row + c;
    float sum[V], t[V], r[V];
#pragma unroll
    for (int i = 0; i < V; ++i) sum[i] = 0.f;
    {
      const float w0 = p.depth[0];
      Row<float, V>::load(t, p.first + at);
#pragma unroll
      for (int i = 0; i < V; ++i) sum[i] = w0 * t[i];
    }
#pragma unroll 4
    for (int j = 1; j < p.n; ++j) {
      float k[V];
      Row<float, V>::load(k, p.kept + (size_t)(j - 1) * p.kept_stride + at);
      const float w = p.depth[j];
#pragma unroll
      for (int i = 0; i < V; ++i) sum[i] = fmaf(w, k[i], sum[i]);
    }
    float m[V], z[V];
    Row<T, V>::load(m, (const T*)p.a + at);
    if (p.b != nullptr) {
      float b[V], ga[V], gb[V];
      Row<T, V>::load(b, (const T*)p.b + at);
      Row<float, V>::load(ga, p.gain_a + c);
      Row<float, V>::load(gb, p.gain_b + c);
#pragma unroll
      for (int i = 0; i < V; ++i) m[i] = m[i] * ra * ga[i] + b[i] * rb * gb[i];
    } else if (p.bias_a != nullptr) {
      float b[V];
      Row<float, V>::load(b, p.bias_a + c);
#pragma unroll
      for (int i = 0; i < V; ++i) m[i] += b[i];
    }
    Row<T, V>::load(z, (const T*)p.za + at);
    Row<float, V>::load(t, p.ba + c);
#pragma unroll
    for (int i = 0; i < V; ++i) m[i] *= sigmoid_of<T>(z[i] + t[i]);
    if (p.f != nullptr) {
      float f[V];
      Row<T, V>::load(f, (const T*)p.f + at);
      Row<T, V>::load(z, (const T*)p.zf + at);
      Row<float, V>::load(t, p.bf + c);
#pragma unroll
      for (int i = 0; i < V; ++i) m[i] = fmaf(sigmoid_of<T>(z[i] + t[i]), f[i], m[i]);
    }
    Row<float, V>::load(r, p.x + at);
#pragma unroll
    for (int i = 0; i < V; ++i) r[i] = fmaf(p.mult, m[i], r[i]);
    if (p.keep) Row<float, V>::store(p.kept + (size_t)(p.n - 1) * p.kept_stride + at, r);
    const float wn = p.depth[p.n];
#pragma unroll
    for (int i = 0; i < V; ++i) sum[i] = fmaf(wn, r[i], sum[i]);
    Row<float, V>::store(p.x_next + at, sum);
    write_tanh_norm<T, V>(p.n1, at, c, sum);
    write_tanh_norm<T, V>(p.n2, at, c, sum);
  }
}

// Column tiles a row is cut into: one where the rows alone fill the machine.
static int column_tiles(int rows, int hidden, int v) {
  const int whole = (hidden + kDepthThreads * v - 1) / (kDepthThreads * v);
  const int want = (2 * sm_count() + rows - 1) / rows;
  return want < 1 ? 1 : (want < whole ? want : whole);
}

template <typename T>
static bool four_at_a_time(int hidden, std::initializer_list<const void*> wide, std::initializer_list<const void*> narrow) {
  if (hidden % 4) return false;
  for (const void* q : wide) if ((uintptr_t)q & 15) return false;
  for (const void* q : narrow) if ((uintptr_t)q % (4 * sizeof(T))) return false;
  return true;
}

template <typename T>
static int launch_tanh(void* y1, const float* alpha1, const float* w1, const float* b1, void* y2, const float* alpha2,
                       const float* w2, const float* b2, float* stream, const void* add, const int* rows, int n_rows,
                       int hidden, int write_back, cudaStream_t cuda_stream) {
  if (n_rows <= 0) return 0;
  if (hidden <= 0 || !y1 || !alpha1 || !w1 || !b1 || (y2 && (!alpha2 || !w2 || !b2))) return EK_ERR_ARG;
  const TanhNorm n1{y1, alpha1, w1, b1}, n2{y2, alpha2, w2, b2};
  if (four_at_a_time<T>(hidden, {w1, b1, w2, b2, stream}, {y1, y2, add})) {
    const int tiles = (hidden + kDepthThreads * 4 - 1) / (kDepthThreads * 4);
    return (int)launch_pdl(dynamic_tanh_kernel<T, 4>, dim3(n_rows, tiles), dim3(kDepthThreads), 0, cuda_stream, n1, n2,
                           stream, (const T*)add, rows, hidden, write_back);
  }
  const int tiles = (hidden + kDepthThreads - 1) / kDepthThreads;
  if (tiles > 65535) return EK_ERR_ARG;
  return (int)launch_pdl(dynamic_tanh_kernel<T, 1>, dim3(n_rows, tiles), dim3(kDepthThreads), 0, cuda_stream, n1, n2,
                         stream, (const T*)add, rows, hidden, write_back);
}

template <typename T>
static int launch_join(const DepthJoin& p, int n_rows, cudaStream_t stream) {
  if (n_rows <= 0) return 0;
  if (p.hidden <= 0 || p.n < 1 || !p.x || !p.x_next || !p.first || !p.depth || !p.a || !p.za || !p.ba ||
      ((p.n > 1 || p.keep) && !p.kept) || (p.b && (!p.gain_a || !p.gain_b || p.bias_a)) || (p.f && (!p.zf || !p.bf)) ||
      (p.n1.y && (!p.n1.alpha || !p.n1.w || !p.n1.b)) || (p.n2.y && (!p.n2.alpha || !p.n2.w || !p.n2.b)))
    return EK_ERR_ARG;
  const bool vec = p.kept_stride % 4 == 0 &&
      four_at_a_time<T>(p.hidden, {p.x, p.x_next, p.first, p.kept, p.bias_a, p.gain_a, p.gain_b, p.ba, p.bf, p.n1.w,
                                   p.n1.b, p.n2.w, p.n2.b},
                        {p.a, p.b, p.za, p.f, p.zf, p.n1.y, p.n2.y});
  const int v = vec ? 4 : 1;
  const int tiles = column_tiles(n_rows, p.hidden, v);
  const int unit = kDepthThreads * v;
  const int cols = ((p.hidden + tiles - 1) / tiles + unit - 1) / unit * unit;
  const dim3 grid(n_rows, (p.hidden + cols - 1) / cols);
  return (int)launch_pdl(vec ? depth_join_kernel<T, 4> : depth_join_kernel<T, 1>, grid, dim3(kDepthThreads), 0, stream, p,
                         cols);
}

}  // namespace ek

#define EK_INSTANTIATE(SUFFIX, T)                                                                                \
  EK_EXPORT int ek_dynamic_tanh_##SUFFIX(void* y1, const float* alpha1, const float* w1, const float* b1, void* y2, \
                                         const float* alpha2, const float* w2, const float* b2, float* stream,   \
                                         const void* add, const int* rows, int n_rows, int hidden,               \
                                         int write_back, cudaStream_t cuda_stream) {                             \
    return ek::launch_tanh<T>(y1, alpha1, w1, b1, y2, alpha2, w2, b2, stream, add, rows, n_rows, hidden,         \
                              write_back, cuda_stream);                                                          \
  }                                                                                                              \
  EK_EXPORT int ek_depth_join_##SUFFIX(                                                                          \
      const float* x, float* x_next, const float* first, float* kept, long long kept_stride, const float* depth, \
      int n, int keep, float mult, const void* a, const float* bias_a, const void* b, const float* gain_a,       \
      const float* gain_b, float pair_eps, float pair_weight, const void* za, const float* ba, const void* f,    \
      const void* zf, const float* bf, void* y1, const float* alpha1, const float* w1, const float* b1,          \
      void* y2, const float* alpha2, const float* w2, const float* b2, int n_rows, int hidden,                   \
      cudaStream_t stream) {                                                                                     \
    const ek::DepthJoin p{x, x_next, first, kept, kept_stride, depth, n, keep, mult, a, bias_a, b, gain_a,       \
                          gain_b, pair_eps, pair_weight, za, ba, f, zf, bf, {y1, alpha1, w1, b1},                \
                          {y2, alpha2, w2, b2}, hidden};                                                         \
    return ek::launch_join<T>(p, n_rows, stream);                                                                \
  }

EK_INSTANTIATE(f32, float)
EK_INSTANTIATE(bf16, ek::bf16)
