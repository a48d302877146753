// The matrix recurrence with a decay per token, head and key channel, S_t = diag(a_t) S_(t-1) + k_t v_t^T, y_t = S_t^T q_t, for long
// portions: what ms_matrix_scan does token after token (its mode 4), in chunks of tokens that do not wait for one another.
//
// The recurrence is linear in S, so a portion is cut into chunks and takes three launches:
//   1. every chunk but the portion's last is walked from a matrix of zeros: its own matrix and the product of its decays;
//   2. a portion's chunks are joined, S <- diag(product) S + matrix, which leaves the S that each chunk starts from;
//   3. every chunk is walked from there and writes its tokens' rows; the last one leaves the request's state.
// A portion of one chunk is walked from and into its state in the third launch alone.
//
// The walk: 256 threads own 4 * 256 / LPC columns of one head's matrix.  Keys, queries and decays of a token come from shared
// memory, and reading them would bound a walk (each column needs the whole key, query and decays): a lane therefore holds
// kEntries entries of kColumns neighbouring columns, so that what it reads serves four columns, and the LPC lanes of those
// columns divide the key channels.  Reading out, the lanes' four sums are exchanged by halves (two exchanges leave every lane
// with one column), then added up.  Entries lie in registers in pairs (two multiply-adds an instruction); tokens go by fours
// without a branch between them.  They are staged kTokens at a time, the next stage on its way (16-byte asynchronous copies
// where rows lie so) while one is walked.
//
// All arithmetic is float32; decays, states and products are float32 in memory, projections in the model's compute type.
#include "common.cuh"
#include "mma_common.cuh"

#include <type_traits>

namespace ms {
namespace channel_scan {

constexpr int kThreads = 256, kColumns = 4, kEntries = 8, kPairs = kEntries / 2, kTokens = 16, kTogether = 4, kMaxShift = 5;

struct Chunks {
  int length;                // tokens of a chunk
  int most;                  // chunks of the longest portion: blockIdx.z = request * most + chunk
  float* states;             // [places][heads][vdim][dim]
  float* decays;             // [places][heads][dim]
};
// Chunk c of a request's portion lies at this place.  Places of different requests do not meet: a portion of n tokens has at most
// one chunk more than it holds borders of `length` tokens counted from the step's first token.
__device__ __forceinline__ size_t place_of(const Chunks& chunks, int first_token, int request, int c) {
  return (size_t)(first_token / chunks.length + request + c);
}

// Where entry i of a row of LANES * kEntries numbers lies in shared memory: the 16-byte pieces that neighbouring lanes read at the same
// time are neighbours.
template <typename T, int LANES>
__device__ __forceinline__ int entry_at(int i) {
  constexpr int E = 16 / sizeof(T), PIECES = kEntries / E;
  return (i / E % PIECES) * LANES * E + i / kEntries * E + i % E;
}

template <typename T, int LANES>
__device__ __forceinline__ void load_pairs(const T* row, int sub, unsigned long long (&out)[kPairs]) {
  constexpr int E = 16 / sizeof(T), PIECES = kEntries / E;
#pragma unroll
  for (int p = 0; p < PIECES; ++p) {
    const uint4 raw = *reinterpret_cast<const uint4*>(row + (p * LANES + sub) * E);
    const T* v = reinterpret_cast<const T*>(&raw);
#pragma unroll
    for (int e = 0; e < E; e += 2) out[(p * E + e) / 2] = pack2(to_float(v[e]), to_float(v[e + 1]));
  }
}

template <typename T> struct alignas(sizeof(T) * kColumns) Values { T v[kColumns]; };

// 2^SHIFT lanes (LPC above) cover the key channels.  LOCAL: the first launch (nothing is read out).  `wide`: rows of keys, queries,
// values and decays lie on 16-byte boundaries and hold whole 16-byte pieces.
template <typename T, int SHIFT, bool LOCAL>
__global__ void __launch_bounds__(kThreads, 2)
walk_kernel(const T* __restrict__ q, int q_ld, int q_col, const T* __restrict__ k, int k_ld, int k_col, const T* __restrict__ v, int v_ld,
            int v_col, float q_scale, const float* __restrict__ decay, float* __restrict__ states, long long state_stride,
            int state_offset, const int* __restrict__ state_slots, const int* __restrict__ query_start, int heads, int kv_heads,
            int dim, int vdim, int wide, float* __restrict__ y, const Chunks chunks) {
  grid_dependency_wait();
  grid_dependency_launch();
  const int request = blockIdx.z / chunks.most, c = blockIdx.z % chunks.most, head = blockIdx.y;
  const int first_token = query_start[request], q_len = query_start[request + 1] - first_token;
  const int t_first = first_token + c * chunks.length, left = q_len - c * chunks.length;
  if (left <= 0 || (LOCAL && left <= chunks.length)) return;              // (the whole block)
  const int len = min(left, chunks.length);
  const bool last = left <= chunks.length, several = q_len > chunks.length;

  constexpr int lanes = 1 << SHIFT, row = lanes * kEntries, block_columns = (kThreads >> SHIFT) * kColumns;
  const int tid = threadIdx.x, group = tid >> SHIFT, sub = tid & (lanes - 1);
  const int column0 = blockIdx.x * block_columns + group * kColumns;
  const int kv_head = head / (heads / kv_heads);
  extern __shared__ __align__(16) unsigned char scan_smem[];
  // two stages of [kTokens][row] decays, keys and queries and [kTokens][block_columns] values
  float* ds = reinterpret_cast<float*>(scan_smem);
  T* ks = reinterpret_cast<T*>(ds + 2 * kTokens * row);
  T* qs = ks + 2 * kTokens * row;
  T* vs = qs + (LOCAL ? 0 : 2 * kTokens * row);

  const size_t place = several ? place_of(chunks, first_token, request, c) : 0;
  float* chunk_state = chunks.states + (place * heads + head) * (size_t)vdim * dim;
  float* kept = states + (long long)state_slots[request] * state_stride + state_offset + (size_t)head * vdim * dim;
  const float* from = several ? chunk_state : kept;
  unsigned long long s[kColumns][kPairs], product[LOCAL ? kPairs : 1];       // pairs of neighbouring entries
#pragma unroll
  for (int j = 0; j < kColumns; ++j)
#pragma unroll
    for (int e = 0; e < kPairs; ++e) {
      const int i = sub * kEntries + 2 * e;
      const float* at = from + (size_t)(column0 + j) * dim + i;
      const bool real = !LOCAL && column0 + j < vdim;
      s[j][e] = pack2(real && i < dim ? at[0] : 0.f, real && i + 1 < dim ? at[1] : 0.f);
    }
  if (LOCAL)
#pragma unroll
    for (int e = 0; e < kPairs; ++e) product[LOCAL ? e : 0] = pack2(1.f, 1.f);

  const T* k_head = k + k_col + (size_t)kv_head * dim;
  const T* q_head = q + q_col + (size_t)kv_head * dim;
  const T* v_head = v + v_col + (size_t)head * vdim + (size_t)blockIdx.x * block_columns;
  const float* d_head = decay + (size_t)head * dim;
  const int d_ld = heads * dim, columns_here = min(block_columns, vdim - (int)blockIdx.x * block_columns);
  auto stage_rows = [&](auto* to, const auto* rows, int ld, int t0, int count, int width, auto size, auto apart) {
    // `count` tokens' rows of `width` numbers, zeros behind them up to `padded` numbers
    constexpr int padded = decltype(size)::value;
    constexpr bool pieces_apart = decltype(apart)::value;
    using E_T = typename std::remove_const<typename std::remove_reference<decltype(*rows)>::type>::type;
    constexpr int E = 16 / sizeof(E_T);
    if (wide) {
      constexpr int per_row = padded / E;
      for (int i = tid; i < count * per_row; i += kThreads) {
        const int t = i / per_row, at = (i % per_row) * E;
        const bool real = at < width;
        cp_async_16(to + t * padded + (pieces_apart ? entry_at<E_T, lanes>(at) : at), rows + (real ? (size_t)(t0 + t) * ld + at : 0), real);
      }
    } else {
      for (int i = tid; i < count * padded; i += kThreads) {
        const int t = i / padded, at = i % padded;
        to[t * padded + (pieces_apart ? entry_at<E_T, lanes>(at) : at)] =
            at < width ? rows[(size_t)(t0 + t) * ld + at] : from_float<E_T>(0.f);
      }
    }
  };
  auto fetch = [&](int stage, int t0) {
    const int count = min(kTokens, len - t0);
    const std::integral_constant<int, row> row_size;
    const std::integral_constant<int, block_columns> columns_size;
    stage_rows(ds + stage * kTokens * row, d_head, d_ld, t_first + t0, count, dim, row_size, std::true_type());
    stage_rows(ks + stage * kTokens * row, k_head, k_ld, t_first + t0, count, dim, row_size, std::true_type());
    if (!LOCAL) stage_rows(qs + stage * kTokens * row, q_head, q_ld, t_first + t0, count, dim, row_size, std::true_type());
    stage_rows(vs + stage * kTokens * block_columns, v_head, v_ld, t_first + t0, count, columns_here, columns_size, std::false_type());
  };
  // the column whose sum this lane ends up with, and whether it writes it
  constexpr int half_1 = lanes >> 1, half_2 = lanes >> 2;
  const int mine = ((sub & half_1) ? 2 : 0) + ((sub & half_2) ? 1 : 0);
  float* out_at = (!LOCAL && (sub & (half_2 - 1)) == 0 && column0 + mine < vdim)
                      ? y + ((size_t)t_first * heads + head) * vdim + column0 + mine : nullptr;
  const size_t out_step = (size_t)heads * vdim;
  const bool high_1 = (sub & half_1) != 0, high_2 = (sub & half_2) != 0;

  fetch(0, 0);
  cp_async_commit();
  for (int t0 = 0, stage = 0; t0 < len; t0 += kTokens, stage ^= 1) {
    if (t0 + kTokens < len) fetch(stage ^ 1, t0 + kTokens);
    cp_async_commit();
    cp_async_wait<1>();
    __syncthreads();
    const int count = min(kTokens, len - t0);
    const float* d_row = ds + stage * kTokens * row;
    const T* k_row = ks + stage * kTokens * row;
    const T* q_row = qs + stage * kTokens * row;
    const T* v_row = vs + stage * kTokens * block_columns + group * kColumns;
    auto walk = [&](int t) {                                  // one token; the column sum that this lane ends up with
      unsigned long long kv[kPairs], dv[kPairs], value[kColumns];
      load_pairs<T, lanes>(k_row + t * row, sub, kv);
      load_pairs<float, lanes>(d_row + t * row, sub, dv);
      const Values<T> four = *reinterpret_cast<const Values<T>*>(v_row + t * block_columns);
#pragma unroll
      for (int j = 0; j < kColumns; ++j) value[j] = pack2(to_float(four.v[j]), to_float(four.v[j]));
#pragma unroll
      for (int j = 0; j < kColumns; ++j)
#pragma unroll
        for (int e = 0; e < kPairs; ++e) s[j][e] = fma2(value[j], kv[e], mul2(dv[e], s[j][e]));
      if (LOCAL) {
#pragma unroll
        for (int e = 0; e < kPairs; ++e) product[LOCAL ? e : 0] = mul2(product[LOCAL ? e : 0], dv[e]);
        return 0.f;
      }
      unsigned long long qv[kPairs];
      float sum[kColumns];
      load_pairs<T, lanes>(q_row + t * row, sub, qv);
#pragma unroll
      for (int j = 0; j < kColumns; ++j) {
        unsigned long long two = mul2(s[j][0], qv[0]);
#pragma unroll
        for (int e = 1; e < kPairs; ++e) two = fma2(s[j][e], qv[e], two);
        float even, odd;
        unpack2(two, even, odd);
        sum[j] = even + odd;
      }
      // two exchanges of halves: columns 2, 3 against 0, 1, then the odd against the even of those
      const float a = (high_1 ? sum[2] : sum[0]) + __shfl_xor_sync(0xffffffffu, high_1 ? sum[0] : sum[2], half_1);
      const float b = (high_1 ? sum[3] : sum[1]) + __shfl_xor_sync(0xffffffffu, high_1 ? sum[1] : sum[3], half_1);
      float total = (high_2 ? b : a) + __shfl_xor_sync(0xffffffffu, high_2 ? a : b, half_2);
#pragma unroll
      for (int o = half_2 >> 1; o > 0; o >>= 1) total += __shfl_xor_sync(0xffffffffu, total, o);
      return q_scale * total;
    };
    // (tokens by fours without a branch between them, so that their shuffles and loads overlap)
    int t = 0;
    for (; t + kTogether <= count; t += kTogether) {
      float total[kTogether];
#pragma unroll
      for (int u = 0; u < kTogether; ++u) total[u] = walk(t + u);
      if (out_at != nullptr) {
#pragma unroll
        for (int u = 0; u < kTogether; ++u, out_at += out_step) *out_at = total[u];
      }
    }
    for (; t < count; ++t) {
      const float total = walk(t);
      if (out_at != nullptr) {
        *out_at = total;
        out_at += out_step;
      }
    }
    __syncthreads();                                          // this stage has been read before it is filled again
  }
  cp_async_wait<0>();
  if (!LOCAL && !last) return;                                // (the chunk behind it starts from what was joined)
  float* to = LOCAL ? chunk_state : kept;
  auto store_pair = [&](float* at, int i, unsigned long long two) {
    float even, odd;
    unpack2(two, even, odd);
    if (i < dim) at[i] = even;
    if (i + 1 < dim) at[i + 1] = odd;
  };
#pragma unroll
  for (int j = 0; j < kColumns; ++j)
#pragma unroll
    for (int e = 0; e < kPairs; ++e)
      if (column0 + j < vdim) store_pair(to + (size_t)(column0 + j) * dim, sub * kEntries + 2 * e, s[j][e]);
  if (LOCAL && blockIdx.x == 0 && group == 0) {
#pragma unroll
    for (int e = 0; e < kPairs; ++e)
      store_pair(chunks.decays + (place * heads + head) * dim, sub * kEntries + 2 * e, product[LOCAL ? e : 0]);
  }
}

// The second launch: grid (pieces of the heads' matrices, requests), PER numbers of the matrices a thread, from the request's state
// through its portion's chunks.
template <int PER> struct alignas(4 * PER) Piece { float v[PER]; };

template <int PER>
__global__ void __launch_bounds__(256)
join_kernel(const float* __restrict__ states, long long state_stride, int state_offset, const int* __restrict__ state_slots,
            const int* __restrict__ query_start, int heads, int dim, int vdim, const Chunks chunks) {
  grid_dependency_wait();
  grid_dependency_launch();
  const int request = blockIdx.y, first_token = query_start[request];
  const int count = (query_start[request + 1] - first_token + chunks.length - 1) / chunks.length;
  const size_t all = (size_t)heads * vdim * dim, at = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * PER;
  if (count <= 1 || at >= all) return;
  const size_t channel = at / ((size_t)vdim * dim) * dim + at % dim, first = place_of(chunks, first_token, request, 0);
  const float* kept = states + (long long)state_slots[request] * state_stride + state_offset;
  Piece<PER> s;
#pragma unroll
  for (int e = 0; e < PER; ++e) s.v[e] = kept[at + e];
  // chunks by fours: their matrices are requested together (a portion's last chunk left none)
  for (int c0 = 0; c0 < count; c0 += 4) {
    Piece<PER> wrote[4], decay[4];
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      if (c0 + u + 1 >= count) continue;
      wrote[u] = *reinterpret_cast<const Piece<PER>*>(chunks.states + (first + c0 + u) * all + at);
      decay[u] = *reinterpret_cast<const Piece<PER>*>(chunks.decays + (first + c0 + u) * heads * dim + channel);
    }
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      if (c0 + u >= count) break;
      *reinterpret_cast<Piece<PER>*>(chunks.states + (first + c0 + u) * all + at) = s;
#pragma unroll
      for (int e = 0; e < PER; ++e) s.v[e] = c0 + u + 1 < count ? decay[u].v[e] * s.v[e] + wrote[u].v[e] : 0.f;
    }
  }
}

static int lanes_shift(int dim) {
  int shift = 2;                                              // (four columns are exchanged between four lanes or more)
  while ((kEntries << shift) < dim) ++shift;
  return shift;
}

}  // namespace channel_scan
}  // namespace ms

using namespace ms;
using namespace ms::channel_scan;

#define MS_CS_DISPATCH(dtype, ...)                               \
  if ((dtype) == MS_F32) { using T = float; __VA_ARGS__; }       \
  else if ((dtype) == MS_BF16) { using T = __nv_bfloat16; __VA_ARGS__; } \
  else MS_FAIL("unknown element type code %d", (dtype));

// The chunk length (tokens) in which n_requests portions, the longest of max_query_len tokens, should be scanned, 0 where the walk of
// ms_matrix_scan, token after token, is the better one: few tokens, keys of more than 256 entries, or so many portions that
// those walks fill the GPU.  The chunks' matrices are walked nearly twice, at two blocks a multiprocessor in one round.
MS_EXPORT int ms_channel_scan_chunk(int n_requests, int max_query_len, int heads, int dim, int vdim) {
  if (n_requests <= 0 || heads <= 0 || dim <= 0 || dim > (kEntries << kMaxShift) || max_query_len < 128) return 0;
  int device = 0, sms = 148;
  if (cudaGetDevice(&device) == cudaSuccess) cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, device);
  const int columns = (kThreads >> lanes_shift(dim)) * kColumns;
  const long long blocks = (long long)heads * ((vdim + columns - 1) / columns) * n_requests;
  long long most = 2LL * sms / blocks;
  if (most > max_query_len / 32) most = max_query_len / 32;
  if (most < 2 || most * n_requests > 65535) return 0;
  const long long length = ((max_query_len + most - 1) / most + kTokens - 1) / kTokens * kTokens;
  return (int)length;
}

// Arguments as ms_matrix_scan's mode 4 (channel_decay float32 [n_tokens, heads, dim]; state [heads, vdim, dim] at state_offset of a
// slot's row), and `chunk` tokens a chunk with scratch chunk_states float32 [places, heads, vdim, dim] and chunk_decays float32
// [places, heads, dim], places = n_tokens / chunk + n_requests.
MS_EXPORT int ms_channel_scan(const void* q, int q_ld, int q_col, const void* k, int k_ld, int k_col, const void* v, int v_ld, int v_col,
                              int dtype, float q_scale, const float* channel_decay, float* states, long long state_stride,
                              int state_offset, const int* state_slots, const int* query_start, int n_requests, int max_query_len,
                              int heads, int kv_heads, int dim, int vdim, float* y, int chunk, float* chunk_states,
                              float* chunk_decays, cudaStream_t stream) {
  if (n_requests == 0 || max_query_len <= 0 || heads == 0) return 0;
  MS_REQUIRE(kv_heads > 0 && heads % kv_heads == 0 && dim >= 1 && dim <= (kEntries << kMaxShift) && vdim >= 1,
             "channel_scan: %d/%d heads of %d/%d", heads, kv_heads, dim, vdim);
  MS_REQUIRE(chunk >= 1 && channel_decay && chunk_states && chunk_decays, "channel_scan: chunks of %d tokens need decays and scratch", chunk);
  const Chunks chunks{chunk, (max_query_len + chunk - 1) / chunk, chunk_states, chunk_decays};
  MS_REQUIRE(heads <= 65535 && (long long)n_requests * chunks.most <= 65535, "channel_scan: %d heads, %d requests of %d chunks exceed the launch limits",
             heads, n_requests, chunks.most);
  const int shift = lanes_shift(dim), row = kEntries << shift, columns = (kThreads >> shift) * kColumns;
  const size_t element = dtype == MS_F32 ? 4 : 2;
  const int per = (int)(16 / element);
  auto aligned = [](const void* p) { return reinterpret_cast<size_t>(p) % 16 == 0; };
  const int wide = aligned(q) && aligned(k) && aligned(v) && aligned(channel_decay) && q_ld % per == 0 && k_ld % per == 0 && v_ld % per == 0 &&
                   q_col % per == 0 && k_col % per == 0 && v_col % per == 0 && dim % per == 0 && dim % 4 == 0 && vdim % per == 0;
  dim3 grid((vdim + columns - 1) / columns, heads, n_requests * chunks.most);
  auto bytes = [&](bool local) { return (size_t)2 * kTokens * (row * (sizeof(float) + (local ? 1 : 2) * element) + columns * element); };
#define MS_CHANNEL_WALK_AT(SHIFT, LOCAL)                                                                                                    \
  MS_CS_DISPATCH(dtype, {                                                                                                         \
    auto kernel = walk_kernel<T, SHIFT, LOCAL>;                                                                                   \
    static bool known = false;                                                                                                    \
    if (!known) {                                                                                                                 \
      cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 112 * 1024);                      \
      if (e != cudaSuccess) MS_FAIL("channel_scan: shared memory refused: %s", cudaGetErrorString(e));                            \
      known = true;                                                                                                               \
    }                                                                                                                             \
    ms::launch(kernel, grid, kThreads, bytes(LOCAL), stream, (const T*)q, q_ld, q_col, (const T*)k, k_ld, k_col, (const T*)v, v_ld, \
               v_col, q_scale, channel_decay, states, state_stride, state_offset, state_slots, query_start, heads, kv_heads, dim,  \
               vdim, wide, y, chunks);                                                                                     \
  })
#define MS_CHANNEL_WALK(LOCAL)                                                                                                    \
  if (shift == 2) { MS_CHANNEL_WALK_AT(2, LOCAL); } else if (shift == 3) { MS_CHANNEL_WALK_AT(3, LOCAL); }                          \
  else if (shift == 4) { MS_CHANNEL_WALK_AT(4, LOCAL); } else { MS_CHANNEL_WALK_AT(5, LOCAL); }
  if (chunks.most > 1) {
    MS_CHANNEL_WALK(true);
    MS_CHECK_LAUNCH("channel_scan: chunks alone");
    const bool four = dim % 4 == 0;
    const size_t threads = (size_t)heads * vdim * dim / (four ? 4 : 1);
    ms::launch(four ? join_kernel<4> : join_kernel<1>, dim3((unsigned)((threads + 255) / 256), n_requests), 256, 0, stream, states,
               state_stride, state_offset, state_slots, query_start, heads, dim, vdim, chunks);
    MS_CHECK_LAUNCH("channel_scan: chunks joined");
  }
  MS_CHANNEL_WALK(false);
#undef MS_CHANNEL_WALK
#undef MS_CHANNEL_WALK_AT
  MS_CHECK_LAUNCH("channel_scan");
  return 0;
}
