// Layer norm and dynamic tanh of the residual stream, and the kernel that hands the stream to a matrix product.
//
//   ms_add_layernorm      pending outputs (or a vector) are added to the float32 stream, and the sum is layer-normed for the
//                         sublayers that read it next: one output, or two with weights and biases of their own that share the
//                         row's mean and deviation (a block whose mixer and feed-forward each have a norm of the same stream)
//   ms_add_dynamic_tanh   pending outputs are added to the float32 stream, and the sum passes weight * tanh(alpha x) + bias entry by
//                         entry: a norm without statistics, so nothing ties the entries of a row together
//   ms_stream_to_columns  the stream with its pending outputs, rounded once to the compute type, as some columns of a wider
//                         matrix (the input of a product over the stream and something beside it)
//
// All arithmetic is float32; the mean is taken off before the deviations are squared.
#include "common.cuh"
#include "elementwise_vec.cuh"

namespace ms {

// For output row k (source row r = rows ? rows[k] : k):
//   x = residual[r] + (delta[r] + delta2[r]) + vector      (what is null is left out; written back to residual unless rows
//                                                           are gathered or nothing was added)
//   y = (x - mean(x)) / sqrt(mean((x - mean(x))^2) + eps)
//   out[k] = weight * y + bias,   out2[k] = weight2 * y + bias2 (if out2 is given), each rounded once to T
template <typename T>
__global__ void add_layernorm_kernel(float* __restrict__ residual, const T* __restrict__ delta, const T* __restrict__ delta2,
                                     const float* __restrict__ vector, const void* __restrict__ weight, const void* __restrict__ bias,
                                     const void* __restrict__ weight2, const void* __restrict__ bias2, int weight_dtype, float eps,
                                     const int* __restrict__ rows, T* __restrict__ out, T* __restrict__ out2, int hidden) {
  grid_dependency_wait();
  grid_dependency_launch();
  __shared__ float scratch[32];
  const size_t k = blockIdx.x;
  const size_t r = rows ? (size_t)rows[k] : k;
  float* res = residual + r * hidden;
  const bool write_back = rows == nullptr && (delta != nullptr || vector != nullptr);
  auto summed = [&](int c) {
    float x = res[c];
    if (delta) x += delta2 ? to_float(delta[r * hidden + c]) + to_float(delta2[r * hidden + c]) : to_float(delta[r * hidden + c]);
    if (vector) x += vector[c];
    return x;
  };
  float sum = 0.f;
  for (int c = threadIdx.x; c < hidden; c += blockDim.x) {
    const float x = summed(c);
    if (write_back) res[c] = x;                              // (read again below by the thread that wrote it)
    sum += x;
  }
  const float mean = block_sum(sum, scratch) / (float)hidden;
  sum = 0.f;
  for (int c = threadIdx.x; c < hidden; c += blockDim.x) {
    const float x = (write_back ? res[c] : summed(c)) - mean;
    sum += x * x;
  }
  const float inv = 1.0f / sqrtf(block_sum(sum, scratch) / (float)hidden + eps);
  for (int c = threadIdx.x; c < hidden; c += blockDim.x) {
    const float y = ((write_back ? res[c] : summed(c)) - mean) * inv;
    out[k * hidden + c] = from_float<T>(load_as_float(weight, weight_dtype, c) * y + load_as_float(bias, weight_dtype, c));
    if (out2) out2[k * hidden + c] = from_float<T>(load_as_float(weight2, weight_dtype, c) * y + load_as_float(bias2, weight_dtype, c));
  }
}

// The same with sixteen-byte loads and stores: each thread keeps up to CHUNKS groups of eight elements in registers, so every
// row is read once.  Requires hidden % 8 == 0 and hidden <= 8 * blockDim.x * CHUNKS.  EARLY (one group a thread, launches of few
// rows): weights and biases, which are no kernel's output, are fetched while the kernel before ends; in launches of many rows
// the registers that hold them cost more than their wait.
template <typename T, int CHUNKS, bool EARLY>
__global__ void add_layernorm_vec_kernel(float* __restrict__ residual, const T* __restrict__ delta, const T* __restrict__ delta2,
                                         const float* __restrict__ vector, const void* __restrict__ weight,
                                         const void* __restrict__ bias, const void* __restrict__ weight2,
                                         const void* __restrict__ bias2, int weight_dtype, float eps, const int* __restrict__ rows,
                                         T* __restrict__ out, T* __restrict__ out2, int hidden) {
  static_assert(!EARLY || CHUNKS == 1, "one group a thread");
  Vec8 w, b, w2, b2;
  if (EARLY && (int)threadIdx.x * 8 < hidden) {
    w = load8_any(weight, weight_dtype, threadIdx.x * 8);
    b = load8_any(bias, weight_dtype, threadIdx.x * 8);
    if (out2) {
      w2 = load8_any(weight2, weight_dtype, threadIdx.x * 8);
      b2 = load8_any(bias2, weight_dtype, threadIdx.x * 8);
    }
  }
  grid_dependency_wait();
  grid_dependency_launch();
  __shared__ float scratch[32];
  const size_t k = blockIdx.x;
  const size_t r = rows ? (size_t)rows[k] : k;
  float* res = residual + r * hidden;
  const T* del = delta ? delta + r * hidden : nullptr;
  const T* del2 = delta2 ? delta2 + r * hidden : nullptr;      // (only with delta: the stream gets delta + delta2)
  const bool write_back = rows == nullptr && (delta != nullptr || vector != nullptr);
  Vec8 x[CHUNKS];
  float sum = 0.f;
#pragma unroll
  for (int i = 0; i < CHUNKS; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * 8;
    if (c < hidden) {
      x[i] = load8(res + c);
      if (del) {
        Vec8 d = load8(del + c);
        if (del2) {
          const Vec8 d2 = load8(del2 + c);
#pragma unroll
          for (int e = 0; e < 8; ++e) d.v[e] += d2.v[e];
        }
#pragma unroll
        for (int e = 0; e < 8; ++e) x[i].v[e] += d.v[e];
      }
      if (vector) {
        const Vec8 d = load8(vector + c);
#pragma unroll
        for (int e = 0; e < 8; ++e) x[i].v[e] += d.v[e];
      }
      if (write_back) store8(res + c, x[i]);
#pragma unroll
      for (int e = 0; e < 8; ++e) sum += x[i].v[e];
    }
  }
  const float mean = block_sum(sum, scratch) / (float)hidden;
  sum = 0.f;
#pragma unroll
  for (int i = 0; i < CHUNKS; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * 8;
    if (c < hidden) {
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        x[i].v[e] -= mean;
        sum += x[i].v[e] * x[i].v[e];
      }
    }
  }
  const float inv = 1.0f / sqrtf(block_sum(sum, scratch) / (float)hidden + eps);
#pragma unroll
  for (int i = 0; i < CHUNKS; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * 8;
    if (c < hidden) {
      if (!EARLY) {
        w = load8_any(weight, weight_dtype, c);
        b = load8_any(bias, weight_dtype, c);
      }
      Vec8 y;
#pragma unroll
      for (int e = 0; e < 8; ++e) y.v[e] = w.v[e] * (x[i].v[e] * inv) + b.v[e];
      store8(out + k * hidden + c, y);
      if (out2) {
        if (!EARLY) {
          w2 = load8_any(weight2, weight_dtype, c);
          b2 = load8_any(bias2, weight_dtype, c);
        }
#pragma unroll
        for (int e = 0; e < 8; ++e) y.v[e] = w2.v[e] * (x[i].v[e] * inv) + b2.v[e];
        store8(out2 + k * hidden + c, y);
      }
    }
  }
}

// For output row k (source row r = rows ? rows[k] : k), entry by entry:
//   x = residual[r] + (delta[r] + delta2[r])      (written back unless rows are gathered or nothing was added)
//   out[k] = weight * tanh(alpha x) + bias, rounded once to T
// PER entries a thread (8: sixteen-byte accesses, hidden % 8 == 0; 1 otherwise).  A thread keeps its columns
// from row to row: grid.x blocks cover the columns, grid.y strides over the rows, so weights and biases are fetched once, while
// the kernel before ends.
template <typename T, int PER>
__global__ void __launch_bounds__(128)
add_dynamic_tanh_kernel(float* __restrict__ residual, const T* __restrict__ delta, const T* __restrict__ delta2, float alpha,
                        const float* __restrict__ weight, const float* __restrict__ bias, const int* __restrict__ rows,
                        T* __restrict__ out, int n_out, int hidden) {
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * PER;
  Vec8 w, b;
  if (c < hidden) {
    if (PER == 8) {
      w = load8(weight + c), b = load8(bias + c);
    } else {
      w.v[0] = weight[c], b.v[0] = bias[c];
    }
  }
  grid_dependency_wait();
  grid_dependency_launch();
  if (c >= hidden) return;
  for (int k = blockIdx.y; k < n_out; k += gridDim.y) {
    const size_t at = (size_t)(rows ? rows[k] : k) * hidden + c;
    Vec8 x, y;
    if (PER == 8) {
      x = load8(residual + at);
      if (delta) {
        Vec8 d = load8(delta + at);
        if (delta2) {
          const Vec8 d2 = load8(delta2 + at);
#pragma unroll
          for (int e = 0; e < 8; ++e) d.v[e] += d2.v[e];
        }
#pragma unroll
        for (int e = 0; e < 8; ++e) x.v[e] += d.v[e];
        if (rows == nullptr) store8(residual + at, x);
      }
#pragma unroll
      for (int e = 0; e < 8; ++e) y.v[e] = w.v[e] * tanhf(alpha * x.v[e]) + b.v[e];
      store8(out + (size_t)k * hidden + c, y);
    } else {
      float v = residual[at];
      if (delta) {
        v += delta2 ? to_float(delta[at]) + to_float(delta2[at]) : to_float(delta[at]);
        if (rows == nullptr) residual[at] = v;
      }
      out[(size_t)k * hidden + c] = from_float<T>(w.v[0] * tanhf(alpha * v) + b.v[0]);
    }
  }
}

// out[n, col + c] = residual[n, c] + (delta[n, c] + delta2[n, c]), rounded once to T; `pieces`: groups of eight a row (0: one
// number a thread).
template <typename T>
__global__ void stream_to_columns_kernel(const float* __restrict__ residual, const T* __restrict__ delta, const T* __restrict__ delta2,
                                         T* __restrict__ out, int ld, int col, int hidden, size_t total, int pieces) {
  grid_dependency_wait();
  grid_dependency_launch();
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= total) return;
  if (pieces) {
    const size_t n = i / pieces, at = i * 8;
    Vec8 x = load8(residual + at);
    if (delta) {
      Vec8 d = load8(delta + at);
      if (delta2) {
        const Vec8 d2 = load8(delta2 + at);
#pragma unroll
        for (int e = 0; e < 8; ++e) d.v[e] += d2.v[e];
      }
#pragma unroll
      for (int e = 0; e < 8; ++e) x.v[e] += d.v[e];
    }
    store8(out + n * ld + col + (i - n * pieces) * 8, x);
    return;
  }
  const size_t n = i / hidden;
  float x = residual[i];
  if (delta) x += delta2 ? to_float(delta[i]) + to_float(delta2[i]) : to_float(delta[i]);
  out[n * ld + col + (i - n * hidden)] = from_float<T>(x);
}

}  // namespace ms

using namespace ms;

#define MS_LN_DISPATCH(dtype, ...)                               \
  if ((dtype) == MS_F32) { using T = float; __VA_ARGS__; }       \
  else if ((dtype) == MS_BF16) { using T = __nv_bfloat16; __VA_ARGS__; } \
  else MS_FAIL("unknown element type code %d", (dtype));

// residual float32 [rows, hidden]; delta, delta2 (delta2 only with delta) [rows, hidden] and out, out2 [n_out, hidden] of type
// `dtype`; vector float32 [hidden]; weights and biases [hidden] of type weight_dtype (the second pair with out2); rows int32
// [n_out] or null (then n_out rows in place, and the residual receives the sum).
MS_EXPORT int ms_add_layernorm(float* residual, const void* delta, const void* delta2, int dtype, const float* vector,
                               const void* weight, const void* bias, const void* weight2, const void* bias2, int weight_dtype,
                               float eps, const int* rows, void* out, void* out2, int n_out, int hidden, cudaStream_t stream) {
  if (n_out == 0) return 0;
  MS_REQUIRE(hidden > 0, "add_layernorm: width %d", hidden);
  MS_REQUIRE(delta2 == nullptr || delta != nullptr, "add_layernorm: a second output without a first");
  MS_REQUIRE(out2 == nullptr || (weight2 && bias2), "add_layernorm: a second output of the norm needs its weight and bias");
  if (hidden % 8 == 0 && hidden <= 8192) {
    const int groups = hidden / 8;
    const int threads = groups >= 256 ? 256 : ((groups + 31) / 32) * 32;
    const int chunks = (groups + threads - 1) / threads;
#define MS_LN_VEC(C, E)                                                                                                             \
  MS_LN_DISPATCH(dtype, (ms::launch(add_layernorm_vec_kernel<T, C, E>, n_out, threads, 0, stream, residual, (const T*)delta,        \
                                    (const T*)delta2, vector, weight, bias, weight2, bias2, weight_dtype, eps, rows, (T*)out,    \
                                    (T*)out2, hidden)))
    if (chunks == 1 && n_out <= 256) { MS_LN_VEC(1, true); } else if (chunks == 1) { MS_LN_VEC(1, false); }
    else if (chunks == 2) { MS_LN_VEC(2, false); } else { MS_LN_VEC(4, false); }
#undef MS_LN_VEC
    MS_CHECK_LAUNCH("add_layernorm");
    return 0;
  }
  const int threads = hidden >= 1024 ? 256 : 128;
  MS_LN_DISPATCH(dtype, (ms::launch(add_layernorm_kernel<T>, n_out, threads, 0, stream, residual, (const T*)delta, (const T*)delta2,
                                    vector, weight, bias, weight2, bias2, weight_dtype, eps, rows, (T*)out, (T*)out2, hidden)));
  MS_CHECK_LAUNCH("add_layernorm");
  return 0;
}

// residual float32 [rows, hidden]; delta, delta2 (delta2 only with delta) [rows, hidden] and out [n_out, hidden] of type `dtype`;
// weight, bias float32 [hidden]; rows int32 [n_out] or null (then n_out rows in place, and the residual receives the sum).
MS_EXPORT int ms_add_dynamic_tanh(float* residual, const void* delta, const void* delta2, int dtype, float alpha, const float* weight,
                                  const float* bias, const int* rows, void* out, int n_out, int hidden, cudaStream_t stream) {
  if (n_out == 0) return 0;
  MS_REQUIRE(hidden > 0, "add_dynamic_tanh: width %d", hidden);
  MS_REQUIRE(delta2 == nullptr || delta != nullptr, "add_dynamic_tanh: a second output without a first");
  auto aligned = [](const void* p) { return reinterpret_cast<size_t>(p) % 16 == 0; };
  const bool wide = hidden % 8 == 0 && aligned(residual) && aligned(delta) && aligned(delta2) && aligned(weight) && aligned(bias) && aligned(out);
  const int items = wide ? hidden / 8 : hidden;
  int threads = items >= 128 ? 128 : ((items + 31) / 32) * 32;
  const int column_blocks = (items + threads - 1) / threads;
  // about sixteen blocks of 128 threads a multiprocessor stride over the rows
  long long row_blocks = 148LL * 16 / column_blocks;
  if (row_blocks < 1) row_blocks = 1;
  if (row_blocks > n_out) row_blocks = n_out;
  dim3 grid(column_blocks, (unsigned)row_blocks);
#define MS_DYNAMIC_TANH(PER)                                                                                                   \
  MS_LN_DISPATCH(dtype, (ms::launch(add_dynamic_tanh_kernel<T, PER>, grid, threads, 0, stream, residual, (const T*)delta,     \
                                    (const T*)delta2, alpha, weight, bias, rows, (T*)out, n_out, hidden)))
  if (wide) { MS_DYNAMIC_TANH(8); } else { MS_DYNAMIC_TANH(1); }
#undef MS_DYNAMIC_TANH
  MS_CHECK_LAUNCH("add_dynamic_tanh");
  return 0;
}

// residual float32 [rows, hidden]; delta, delta2 (null: none) [rows, hidden] and out [rows, ld] of type `dtype`.
MS_EXPORT int ms_stream_to_columns(const float* residual, const void* delta, const void* delta2, int dtype, void* out, int ld,
                                   int col, int n_tokens, int hidden, cudaStream_t stream) {
  const long long total = (long long)n_tokens * hidden;
  if (total == 0) return 0;
  MS_REQUIRE(col >= 0 && col + hidden <= ld, "stream_to_columns: columns %d .. %d of rows of %d", col, col + hidden, ld);
  MS_REQUIRE(delta2 == nullptr || delta != nullptr, "stream_to_columns: a second output without a first");
  const bool wide = hidden % 8 == 0 && ld % 8 == 0 && col % 8 == 0 && reinterpret_cast<size_t>(out) % 16 == 0 &&
                    reinterpret_cast<size_t>(delta) % 16 == 0 && reinterpret_cast<size_t>(delta2) % 16 == 0;
  const long long items = wide ? total / 8 : total, blocks = (items + 127) / 128;
  MS_REQUIRE(blocks < 2147483647LL, "stream_to_columns: %lld elements in one launch is too many", total);
  MS_LN_DISPATCH(dtype, (ms::launch(stream_to_columns_kernel<T>, (unsigned)blocks, 128, 0, stream, residual, (const T*)delta,
                                    (const T*)delta2, (T*)out, ld, col, hidden, (size_t)items, wide ? hidden / 8 : 0)));
  MS_CHECK_LAUNCH("stream_to_columns");
  return 0;
}
