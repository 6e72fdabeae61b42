// Rotary position encoding of q and k, and the write of k and v into the paged cache.
//
// Rotation (NeoX pairing): for each head and i < d/2, with (s, c) the sine and cosine of
// position * base^(-2i/d): out[i] = a*c - b*s, out[i + d/2] = a*s + b*c where a = in[i],
// b = in[i + d/2] (crates/vipera-backend-cpu/src/model.rs:4226-4251; the reference's device
// kernel computes powf and sincosf per element, crates/vipera-backend-gpu/src/layer.cu:61-84;
// here the angles come from a 32-bit table built once on the host).
// Cache write: position p of a request goes to page block_table[p / page], slot p % page
// (model.rs:1507-1542); the reference's device port does this with two device copies per
// layer and token (crates/vipera-backend-gpu/src/device.rs:299-320).
#include "common.cuh"

enum RopeStyle { ROPE_NONE = 0, ROPE_NEOX = 1, ROPE_INTERLEAVED = 2 };

// One block per token; its threads walk the pairs of all heads, two pairs (four values) at
// a time where the head size allows, so that loads and stores are 8 and 16 bytes wide.
// Input: the 32-bit result of the q/k/v product with bias, [tokens, (heads + 2*kv_heads) * d].
// Output: rotated q in the activation type, [tokens, heads * d]; rotated k and plain v in
// the cache's type, written to their page (when write_cache is set).
template <typename T>
__device__ __forceinline__ void store_pair(T* dst, float a, float b);
template <>
__device__ __forceinline__ void store_pair<float>(float* dst, float a, float b) {
  *reinterpret_cast<float2*>(dst) = make_float2(a, b);
}
template <>
__device__ __forceinline__ void store_pair<__nv_bfloat16>(__nv_bfloat16* dst, float a, float b) {
  *reinterpret_cast<__nv_bfloat162*>(dst) = __floats2bfloat162_rn(a, b);
}

template <typename T>
__global__ void __launch_bounds__(256)
rope_cache_kernel(const float* __restrict__ qkv, T* __restrict__ q_out, int num_heads, int num_kv_heads,
                  int head_dim, const int* __restrict__ positions, const float* __restrict__ cos_table,
                  const float* __restrict__ sin_table, int style, T* __restrict__ k_pool, T* __restrict__ v_pool,
                  const int* __restrict__ token_seq, const int* __restrict__ block_table, int table_width,
                  int page_size, int write_cache) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  const int half = head_dim >> 1;
  const int all_heads = num_heads + 2 * num_kv_heads;
  const float* row = qkv + static_cast<size_t>(t) * all_heads * head_dim;
  const int position = positions[t];
  T* k_row = nullptr;
  T* v_row = nullptr;
  if (write_cache) {
    const int page = block_table[static_cast<size_t>(token_seq[t]) * table_width + position / page_size];
    if (page >= 0) {
      const size_t at = (static_cast<size_t>(page) * page_size + position % page_size) * num_kv_heads * head_dim;
      k_row = k_pool + at;
      v_row = v_pool + at;
    }
  }
  const float* cos_row = cos_table ? cos_table + static_cast<size_t>(position) * half : nullptr;
  const float* sin_row = sin_table ? sin_table + static_cast<size_t>(position) * half : nullptr;
  // work item: (head, pair of neighbouring pair indices i, i + 1); head sizes are even, and a
  // head size that is a multiple of 4 keeps every access 8 bytes aligned
  const int pairs = half >> 1;  // items per head when two pairs go together
  const bool two = (half & 1) == 0;
  const int per_head = two ? pairs : half;
  for (int item = threadIdx.x; item < all_heads * per_head; item += blockDim.x) {
    const int h = item / per_head;
    const int i = (item % per_head) * (two ? 2 : 1);
    const bool is_q = h < num_heads;
    const bool is_v = h >= num_heads + num_kv_heads;
    const float* head = row + static_cast<size_t>(h) * head_dim;
    T* dst;
    if (is_q) dst = q_out + (static_cast<size_t>(t) * num_heads + h) * head_dim;
    else if (is_v) dst = v_row ? v_row + static_cast<size_t>(h - num_heads - num_kv_heads) * head_dim : nullptr;
    else dst = k_row ? k_row + static_cast<size_t>(h - num_heads) * head_dim : nullptr;
    if (!dst) continue;
    const int count = two ? 2 : 1;
    float lo[2], hi[2];
    int at_lo[2], at_hi[2];
    for (int e = 0; e < count; ++e) {
      at_lo[e] = style == ROPE_INTERLEAVED ? 2 * (i + e) : i + e;
      at_hi[e] = style == ROPE_INTERLEAVED ? 2 * (i + e) + 1 : i + e + half;
      const float a = head[at_lo[e]], b = head[at_hi[e]];
      if (is_v || style == ROPE_NONE) {
        lo[e] = a;
        hi[e] = b;
      } else {
        const float c = cos_row[i + e], s = sin_row[i + e];
        lo[e] = a * c - b * s;
        hi[e] = a * s + b * c;
      }
    }
    if (two && style != ROPE_INTERLEAVED) {
      store_pair<T>(dst + at_lo[0], lo[0], lo[1]);  // i and i + 1 are neighbours in both halves
      store_pair<T>(dst + at_hi[0], hi[0], hi[1]);
    } else {
      for (int e = 0; e < count; ++e) {
        dst[at_lo[e]] = from_float<T>(lo[e]);
        dst[at_hi[e]] = from_float<T>(hi[e]);
      }
    }
  }
}

// The general form: only the first `rot_dims` values of a q or k head turn (value i with value
// i + rot_dims/2 in the NeoX pairing, 2i with 2i + 1 in the interleaved one; the tables are
// [positions, rot_dims/2]), the rest pass unchanged, and a value row has `value_dim` values.
// Input [tokens, heads*d + kv_heads*d + kv_heads*value_dim].  One block per token, a thread per value.
template <typename T>
__global__ void __launch_bounds__(256)
rope_cache_partial_kernel(const float* __restrict__ qkv, T* __restrict__ q_out, int num_heads, int num_kv_heads,
                          int head_dim, int value_dim, int rot_dims, const int* __restrict__ positions,
                          const float* __restrict__ cos_table, const float* __restrict__ sin_table, int style,
                          T* __restrict__ k_pool, T* __restrict__ v_pool, const int* __restrict__ token_seq,
                          const int* __restrict__ block_table, int table_width, int page_size, int write_cache,
                          long long row_stride, float* __restrict__ v_publish, const float* __restrict__ v_blend,
                          const float* __restrict__ blend) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  const int qk_width = (num_heads + num_kv_heads) * head_dim;
  const int v_width = num_kv_heads * value_dim;
  const float* row = qkv + static_cast<size_t>(t) * row_stride;
  const int position = positions[t];
  T* k_row = nullptr;
  T* v_row = nullptr;
  if (write_cache) {
    const int page = block_table[static_cast<size_t>(token_seq[t]) * table_width + position / page_size];
    if (page >= 0) {
      const size_t at = static_cast<size_t>(page) * page_size + position % page_size;
      k_row = k_pool + at * num_kv_heads * head_dim;
      v_row = v_pool + at * num_kv_heads * value_dim;
    }
  }
  const int half = rot_dims >> 1;
  const float* cos_row = cos_table ? cos_table + static_cast<size_t>(position) * half : nullptr;
  const float* sin_row = sin_table ? sin_table + static_cast<size_t>(position) * half : nullptr;
  for (int item = threadIdx.x; item < qk_width; item += blockDim.x) {
    const int h = item / head_dim, e = item % head_dim;
    const float* head = row + static_cast<size_t>(h) * head_dim;
    float value = head[e];
    if (style != ROPE_NONE && e < rot_dims) {
      if (style == ROPE_INTERLEAVED) {
        const int i = e >> 1;
        const float a = head[2 * i], b = head[2 * i + 1], c = cos_row[i], s = sin_row[i];
        value = (e & 1) ? a * s + b * c : a * c - b * s;
      } else {
        const int i = e < half ? e : e - half;
        const float a = head[i], b = head[i + half], c = cos_row[i], s = sin_row[i];
        value = e < half ? a * c - b * s : a * s + b * c;
      }
    }
    if (h < num_heads) q_out[(static_cast<size_t>(t) * num_heads + h) * head_dim + e] = from_float<T>(value);
    else if (k_row) k_row[static_cast<size_t>(h - num_heads) * head_dim + e] = from_float<T>(value);
  }
  // Values: as projected, or blended with the values another layer published for the same tokens,
  // v = (1 - b) v + b v_other with b = blend[0], in 32-bit; `v_publish` receives this layer's values
  // as projected (32-bit), for the layers behind it.
  if (v_publish)
    for (int item = threadIdx.x; item < v_width; item += blockDim.x)
      v_publish[static_cast<size_t>(t) * v_width + item] = row[qk_width + item];
  if (v_row) {
    const float b = v_blend ? blend[0] : 0.0f;
    for (int item = threadIdx.x; item < v_width; item += blockDim.x) {
      float value = row[qk_width + item];
      if (v_blend) value = (1.0f - b) * value + b * v_blend[static_cast<size_t>(t) * v_width + item];
      v_row[item] = from_float<T>(value);
    }
  }
}

// The general form with the input's rows `row_stride` floats apart (q, k, v first; what follows them
// is not read) and values that are published or blended: `v_publish` (null: not) receives the values
// as projected, 32-bit [tokens, kv_heads * value_dim]; with `v_blend` (null: not) the cached values
// are (1 - blend[0]) v + blend[0] v_blend, `blend` a 32-bit number on the device.
VIPERA_API int vipera_rope_cache_blend(const float* qkv, long long row_stride, void* q_out, int dtype, int num_tokens,
                                       int num_heads, int num_kv_heads, int head_dim, int value_dim, int rot_dims,
                                       const int* positions, const float* cos_table, const float* sin_table, int style,
                                       void* k_pool, void* v_pool, const int* token_seq, const int* block_table,
                                       int table_width, int page_size, int write_cache, float* v_publish,
                                       const float* v_blend, const float* blend, void* stream) {
  if (num_tokens <= 0) return VIPERA_OK;
  if (head_dim <= 0 || value_dim <= 0 || num_heads <= 0 || num_kv_heads <= 0) return VIPERA_BAD_SHAPE;
  if (rot_dims < 0 || (rot_dims & 1) || rot_dims > head_dim) return VIPERA_BAD_SHAPE;
  if (row_stride < static_cast<long long>(num_heads + num_kv_heads) * head_dim + num_kv_heads * value_dim) return VIPERA_BAD_SHAPE;
  if (style != ROPE_NONE && rot_dims > 0 && (!cos_table || !sin_table)) return VIPERA_BAD_ARGUMENT;
  if (write_cache && (!k_pool || !v_pool || !token_seq || !block_table || page_size <= 0)) return VIPERA_BAD_ARGUMENT;
  if (v_blend && !blend) return VIPERA_BAD_ARGUMENT;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  dim3 grid(num_tokens);
  const int work = (num_heads + num_kv_heads) * head_dim;
  const int threads = work >= 256 ? 256 : (work >= 128 ? 128 : 64);
  if (dtype == VIPERA_F32)
    return vipera_launch(rope_cache_partial_kernel<float>, grid, threads, 0, s, qkv, static_cast<float*>(q_out), num_heads,
        num_kv_heads, head_dim, value_dim, rot_dims, positions, cos_table, sin_table, style, static_cast<float*>(k_pool),
        static_cast<float*>(v_pool), token_seq, block_table, table_width, page_size, write_cache, row_stride, v_publish,
        v_blend, blend);
  if (dtype == VIPERA_BF16)
    return vipera_launch(rope_cache_partial_kernel<__nv_bfloat16>, grid, threads, 0, s, qkv, static_cast<__nv_bfloat16*>(q_out),
        num_heads, num_kv_heads, head_dim, value_dim, rot_dims, positions, cos_table, sin_table, style,
        static_cast<__nv_bfloat16*>(k_pool), static_cast<__nv_bfloat16*>(v_pool), token_seq, block_table, table_width,
        page_size, write_cache, row_stride, v_publish, v_blend, blend);
  return VIPERA_BAD_DTYPE;
}

VIPERA_API int vipera_rope_cache_partial(const float* qkv, void* q_out, int dtype, int num_tokens, int num_heads,
                                         int num_kv_heads, int head_dim, int value_dim, int rot_dims,
                                         const int* positions, const float* cos_table, const float* sin_table,
                                         int style, void* k_pool, void* v_pool, const int* token_seq,
                                         const int* block_table, int table_width, int page_size, int write_cache,
                                         void* stream) {
  if (num_tokens <= 0) return VIPERA_OK;
  if (head_dim <= 0 || value_dim <= 0 || num_heads <= 0 || num_kv_heads <= 0) return VIPERA_BAD_SHAPE;
  if (rot_dims < 0 || (rot_dims & 1) || rot_dims > head_dim) return VIPERA_BAD_SHAPE;
  if (style != ROPE_NONE && rot_dims > 0 && (!cos_table || !sin_table)) return VIPERA_BAD_ARGUMENT;
  if (write_cache && (!k_pool || !v_pool || !token_seq || !block_table || page_size <= 0)) return VIPERA_BAD_ARGUMENT;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  dim3 grid(num_tokens);
  const long long stride = static_cast<long long>(num_heads + num_kv_heads) * head_dim + static_cast<long long>(num_kv_heads) * value_dim;
  const int work = (num_heads + num_kv_heads) * head_dim;
  const int threads = work >= 256 ? 256 : (work >= 128 ? 128 : 64);
  if (dtype == VIPERA_F32)
    return vipera_launch(rope_cache_partial_kernel<float>, grid, threads, 0, s, qkv, static_cast<float*>(q_out), num_heads,
        num_kv_heads, head_dim, value_dim, rot_dims, positions, cos_table, sin_table, style, static_cast<float*>(k_pool),
        static_cast<float*>(v_pool), token_seq, block_table, table_width, page_size, write_cache, stride, nullptr, nullptr,
        nullptr);
  if (dtype == VIPERA_BF16)
    return vipera_launch(rope_cache_partial_kernel<__nv_bfloat16>, grid, threads, 0, s, qkv, static_cast<__nv_bfloat16*>(q_out),
        num_heads, num_kv_heads, head_dim, value_dim, rot_dims, positions, cos_table, sin_table, style,
        static_cast<__nv_bfloat16*>(k_pool), static_cast<__nv_bfloat16*>(v_pool), token_seq, block_table, table_width,
        page_size, write_cache, stride, nullptr, nullptr, nullptr);
  return VIPERA_BAD_DTYPE;
}

// The form with a norm over whole rows in front: the q row (all heads together) and the k row are
// each divided by their root mean square, sqrt(mean(x^2) + eps), and multiplied by a weight per
// value (`q_norm`, `k_norm`; null: that row is left as it is) before the first `rot_dims` values of
// each head turn.  `v_from_k` != 0: there is no value projection, the values are the keys as
// projected (before norm and rotation), and the input row is [heads*d + kv_heads*d].  One block
// per token; sums in 32-bit in a fixed order.
template <typename T>
__global__ void __launch_bounds__(256)
qk_prepare_kernel(const float* __restrict__ qkv, T* __restrict__ q_out, int num_heads, int num_kv_heads,
                  int head_dim, int value_dim, int rot_dims, const float* __restrict__ q_norm,
                  const float* __restrict__ k_norm, float eps, int v_from_k, const int* __restrict__ positions,
                  const float* __restrict__ cos_table, const float* __restrict__ sin_table, int style,
                  T* __restrict__ k_pool, T* __restrict__ v_pool, const int* __restrict__ token_seq,
                  const int* __restrict__ block_table, int table_width, int page_size, int write_cache) {
  __shared__ float scratch[32];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  const int q_width = num_heads * head_dim, k_width = num_kv_heads * head_dim;
  const int qk_width = q_width + k_width;
  const int v_width = num_kv_heads * value_dim;
  const float* row = qkv + static_cast<size_t>(t) * (qk_width + (v_from_k ? 0 : v_width));
  float q_inverse = 1.0f, k_inverse = 1.0f;
  if (q_norm) {
    float sum = 0.0f;
    for (int i = threadIdx.x; i < q_width; i += blockDim.x) sum = fmaf(row[i], row[i], sum);
    q_inverse = 1.0f / sqrtf(block_sum(sum, scratch) / static_cast<float>(q_width) + eps);
  }
  if (k_norm) {
    float sum = 0.0f;
    for (int i = threadIdx.x; i < k_width; i += blockDim.x) sum = fmaf(row[q_width + i], row[q_width + i], sum);
    k_inverse = 1.0f / sqrtf(block_sum(sum, scratch) / static_cast<float>(k_width) + eps);
  }
  const int position = positions[t];
  T* k_row = nullptr;
  T* v_row = nullptr;
  if (write_cache) {
    const int page = block_table[static_cast<size_t>(token_seq[t]) * table_width + position / page_size];
    if (page >= 0) {
      const size_t at = static_cast<size_t>(page) * page_size + position % page_size;
      k_row = k_pool + at * num_kv_heads * head_dim;
      v_row = v_pool + at * num_kv_heads * value_dim;
    }
  }
  const int half = rot_dims >> 1;
  const float* cos_row = cos_table ? cos_table + static_cast<size_t>(position) * half : nullptr;
  const float* sin_row = sin_table ? sin_table + static_cast<size_t>(position) * half : nullptr;
  for (int item = threadIdx.x; item < qk_width; item += blockDim.x) {
    const int h = item / head_dim, e = item % head_dim;
    const bool is_q = h < num_heads;
    const float inverse = is_q ? q_inverse : k_inverse;
    const float* gain = is_q ? q_norm : k_norm;
    const int base = h * head_dim - (is_q ? 0 : q_width);   // index of the head's first value within its own row
    const float* head = row + static_cast<size_t>(h) * head_dim;
    auto normed = [&](int i) { return gain ? head[i] * inverse * gain[base + i] : head[i]; };
    float value = normed(e);
    if (style != ROPE_NONE && e < rot_dims) {
      if (style == ROPE_INTERLEAVED) {
        const int i = e >> 1;
        const float a = normed(2 * i), b = normed(2 * i + 1), c = cos_row[i], s = sin_row[i];
        value = (e & 1) ? a * s + b * c : a * c - b * s;
      } else {
        const int i = e < half ? e : e - half;
        const float a = normed(i), b = normed(i + half), c = cos_row[i], s = sin_row[i];
        value = e < half ? a * c - b * s : a * s + b * c;
      }
    }
    if (is_q) q_out[(static_cast<size_t>(t) * num_heads + h) * head_dim + e] = from_float<T>(value);
    else if (k_row) k_row[static_cast<size_t>(h - num_heads) * head_dim + e] = from_float<T>(value);
  }
  if (v_row) {
    const float* values = row + (v_from_k ? q_width : qk_width);
    for (int item = threadIdx.x; item < v_width; item += blockDim.x) v_row[item] = from_float<T>(values[item]);
  }
}

VIPERA_API int vipera_qk_prepare(const float* qkv, void* q_out, int dtype, int num_tokens, int num_heads,
                                 int num_kv_heads, int head_dim, int value_dim, int rot_dims, const float* q_norm,
                                 const float* k_norm, float eps, int v_from_k, const int* positions,
                                 const float* cos_table, const float* sin_table, int style, void* k_pool, void* v_pool,
                                 const int* token_seq, const int* block_table, int table_width, int page_size,
                                 int write_cache, void* stream) {
  if (num_tokens <= 0) return VIPERA_OK;
  if (head_dim <= 0 || value_dim <= 0 || num_heads <= 0 || num_kv_heads <= 0) return VIPERA_BAD_SHAPE;
  if (rot_dims < 0 || (rot_dims & 1) || rot_dims > head_dim) return VIPERA_BAD_SHAPE;
  if (v_from_k && value_dim != head_dim) return VIPERA_BAD_SHAPE;
  if (style != ROPE_NONE && rot_dims > 0 && (!cos_table || !sin_table)) return VIPERA_BAD_ARGUMENT;
  if (write_cache && (!k_pool || !v_pool || !token_seq || !block_table || page_size <= 0)) return VIPERA_BAD_ARGUMENT;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  dim3 grid(num_tokens);
  if (dtype == VIPERA_F32)
    return vipera_launch(qk_prepare_kernel<float>, grid, 256, 0, s, qkv, static_cast<float*>(q_out), num_heads,
        num_kv_heads, head_dim, value_dim, rot_dims, q_norm, k_norm, eps, v_from_k, positions, cos_table, sin_table, style,
        static_cast<float*>(k_pool), static_cast<float*>(v_pool), token_seq, block_table, table_width, page_size, write_cache);
  if (dtype == VIPERA_BF16)
    return vipera_launch(qk_prepare_kernel<__nv_bfloat16>, grid, 256, 0, s, qkv, static_cast<__nv_bfloat16*>(q_out),
        num_heads, num_kv_heads, head_dim, value_dim, rot_dims, q_norm, k_norm, eps, v_from_k, positions, cos_table, sin_table,
        style, static_cast<__nv_bfloat16*>(k_pool), static_cast<__nv_bfloat16*>(v_pool), token_seq, block_table,
        table_width, page_size, write_cache);
  return VIPERA_BAD_DTYPE;
}

// ---------------------------------------------------------------------------------------
// The form with options per head.  Each query and key head is divided by its own root mean square,
// sqrt(mean(x^2) + eps), and multiplied by a weight per value that all heads share (`q_norm`, `k_norm`
// [head_dim]; null: left as it is); then its first `rot_dims` values turn; then a query is multiplied by a
// number of its position (`q_factor` [positions], null: 1).  A warp per head of a token, eight to a block;
// the head waits in shared memory, since a value's partner of the rotation belongs to another lane.
// Rows of the input may hold more than q, k and v (`row_stride` values apart).
// ---------------------------------------------------------------------------------------
constexpr int kHeadWarps = 8;
constexpr int kHeadMost = 256;   // values of a head

struct HeadRowsParams {
  const float* qkv;         // [tokens, row_stride]: q heads, k heads, v heads, and what else the product holds
  long long row_stride;
  void* q_out;              // [tokens, heads, head_dim]
  int num_tokens, num_heads, num_kv_heads, head_dim, value_dim, rot_dims, style;
  int norm_size;            // values a norm's mean is over (the rest of a head is zeros)
  const float* q_norm;
  const float* k_norm;
  float eps;
  const float* q_factor;
  const int* positions;
  const float* cos_table;   // [positions, rot_dims / 2]
  const float* sin_table;
  void* k_pool;
  void* v_pool;
  const int* token_entry;
  const int* block_table;
  int table_width, page_size, write_cache;
};

template <typename T>
__global__ void __launch_bounds__(kHeadWarps * 32)
head_rows_kernel(const HeadRowsParams p) {
  __shared__ float rows[kHeadWarps][kHeadMost];
  constexpr int kPerLane = kHeadMost / 32;
  pdl_launch_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x;
  const int job = blockIdx.y * kHeadWarps + warp;   // query heads, key heads, value heads
  if (job >= p.num_heads + 2 * p.num_kv_heads) return;
  const bool is_q = job < p.num_heads, is_v = job >= p.num_heads + p.num_kv_heads;
  const int size = is_v ? p.value_dim : p.head_dim;
  const int kv = is_v ? job - p.num_heads - p.num_kv_heads : job - p.num_heads;
  // the step's description, the tables and the weights were there before the kernel ahead
  const int position = p.positions[t];
  const float* gain = is_v ? nullptr : (is_q ? p.q_norm : p.k_norm);
  const float factor = is_q && p.q_factor ? p.q_factor[position] : 1.0f;
  T* dst = nullptr;
  if (is_q) {
    dst = static_cast<T*>(p.q_out) + (static_cast<size_t>(t) * p.num_heads + job) * p.head_dim;
  } else if (p.write_cache) {
    const int page = p.block_table[static_cast<size_t>(p.token_entry[t]) * p.table_width + position / p.page_size];
    if (page >= 0) {
      const size_t at = static_cast<size_t>(page) * p.page_size + position % p.page_size;
      dst = static_cast<T*>(is_v ? p.v_pool : p.k_pool) + (at * p.num_kv_heads + kv) * size;
    }
  }
  const long long start = is_v ? static_cast<long long>(p.num_heads + p.num_kv_heads) * p.head_dim + static_cast<long long>(kv) * p.value_dim
                               : static_cast<long long>(job) * p.head_dim;
  const float* src = p.qkv + static_cast<long long>(t) * p.row_stride + start;
  pdl_wait();
  if (!dst) return;
  float x[kPerLane];
  float sum = 0.0f;
#pragma unroll
  for (int j = 0; j < kPerLane; ++j) {
    const int e = lane + 32 * j;
    x[j] = e < size ? src[e] : 0.0f;
    sum = fmaf(x[j], x[j], sum);
  }
  if (gain) {
    const float inverse = 1.0f / sqrtf(warp_sum(sum) / static_cast<float>(p.norm_size) + p.eps);
#pragma unroll
    for (int j = 0; j < kPerLane; ++j) {
      const int e = lane + 32 * j;
      if (e < size) x[j] = x[j] * inverse * gain[e];
    }
  }
  if (!is_v && p.style != ROPE_NONE && p.rot_dims > 0) {
    const int half = p.rot_dims >> 1;
    const float* cos_row = p.cos_table + static_cast<size_t>(position) * half;
    const float* sin_row = p.sin_table + static_cast<size_t>(position) * half;
    float* row = rows[warp];
#pragma unroll
    for (int j = 0; j < kPerLane; ++j)
      if (lane + 32 * j < p.rot_dims) row[lane + 32 * j] = x[j];
    __syncwarp();
#pragma unroll
    for (int j = 0; j < kPerLane; ++j) {
      const int e = lane + 32 * j;
      if (e < p.rot_dims) {
        const bool second = p.style == ROPE_INTERLEAVED ? (e & 1) : e >= half;
        const int i = p.style == ROPE_INTERLEAVED ? e >> 1 : (second ? e - half : e);
        const float partner = row[p.style == ROPE_INTERLEAVED ? (e ^ 1) : (second ? e - half : e + half)];
        const float c = cos_row[i], s = sin_row[i];
        x[j] = second ? fmaf(partner, s, x[j] * c) : fmaf(-partner, s, x[j] * c);
      }
    }
  }
#pragma unroll
  for (int j = 0; j < kPerLane; ++j) {
    const int e = lane + 32 * j;
    if (e < size) dst[e] = from_float<T>(x[j] * factor);
  }
}

// The same where everything is whole vectors of four (heads of up to 128 * PIECES values): a lane holds
// values 4 (lane + 32 j) .. + 3 of each of its warp's kHeadJobs heads, whose loads are in flight together.
constexpr int kHeadJobs = 2;

template <typename T, int PIECES>
__global__ void __launch_bounds__(kHeadWarps * 32)
head_rows_vector_kernel(const HeadRowsParams p) {
  __shared__ __align__(16) float rows[kHeadWarps][128 * PIECES];
  pdl_launch_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x;
  const int position = p.positions[t];
  const int jobs = p.num_heads + 2 * p.num_kv_heads;
  const int job0 = (blockIdx.y * kHeadWarps + warp) * kHeadJobs;
  if (job0 >= jobs) return;
  size_t place = 0;
  bool stored = false;
  if (p.write_cache) {
    const int page = p.block_table[static_cast<size_t>(p.token_entry[t]) * p.table_width + position / p.page_size];
    stored = page >= 0;
    place = static_cast<size_t>(max(page, 0)) * p.page_size + position % p.page_size;
  }
  const float factor = p.q_factor ? p.q_factor[position] : 1.0f;
  const int half = p.rot_dims >> 1;
  const bool turns = p.style != ROPE_NONE && p.rot_dims > 0;
  pdl_wait();
  const float* row = p.qkv + static_cast<long long>(t) * p.row_stride;
  float4 x[kHeadJobs][PIECES];
#pragma unroll
  for (int n = 0; n < kHeadJobs; ++n) {
    const int job = job0 + n;
    const bool is_v = job >= p.num_heads + p.num_kv_heads;
    const int size = job >= jobs ? 0 : (is_v ? p.value_dim : p.head_dim);
    const float* src = row + (is_v ? (p.num_heads + p.num_kv_heads) * p.head_dim + (job - p.num_heads - p.num_kv_heads) * p.value_dim
                                   : job * p.head_dim);
#pragma unroll
    for (int j = 0; j < PIECES; ++j) {
      const int e = 4 * (lane + 32 * j);
      x[n][j] = e < size ? *reinterpret_cast<const float4*>(src + e) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    }
  }
#pragma unroll
  for (int n = 0; n < kHeadJobs; ++n) {
    const int job = job0 + n;
    if (job >= jobs) break;
    const bool is_q = job < p.num_heads, is_v = job >= p.num_heads + p.num_kv_heads;
    const int size = is_v ? p.value_dim : p.head_dim;
    const float* gain = is_v ? nullptr : (is_q ? p.q_norm : p.k_norm);
    if (gain) {
      float sum = 0.0f;
#pragma unroll
      for (int j = 0; j < PIECES; ++j)
        sum += x[n][j].x * x[n][j].x + x[n][j].y * x[n][j].y + x[n][j].z * x[n][j].z + x[n][j].w * x[n][j].w;
      const float inverse = 1.0f / sqrtf(warp_sum(sum) / static_cast<float>(p.norm_size) + p.eps);
#pragma unroll
      for (int j = 0; j < PIECES; ++j) {
        const int e = 4 * (lane + 32 * j);
        if (e < size) {
          const float4 g = *reinterpret_cast<const float4*>(gain + e);
          x[n][j] = make_float4(x[n][j].x * inverse * g.x, x[n][j].y * inverse * g.y, x[n][j].z * inverse * g.z, x[n][j].w * inverse * g.w);
        }
      }
    }
    if (turns && !is_v) {
      const float* cos_row = p.cos_table + static_cast<size_t>(position) * half;
      const float* sin_row = p.sin_table + static_cast<size_t>(position) * half;
      if (p.style == ROPE_INTERLEAVED) {
#pragma unroll
        for (int j = 0; j < PIECES; ++j) {
          const int e = 4 * (lane + 32 * j);
          if (e < p.rot_dims) {
            const float2 c = *reinterpret_cast<const float2*>(cos_row + e / 2), s = *reinterpret_cast<const float2*>(sin_row + e / 2);
            const float4 v = x[n][j];
            x[n][j] = make_float4(v.x * c.x - v.y * s.x, v.y * c.x + v.x * s.x, v.z * c.y - v.w * s.y, v.w * c.y + v.z * s.y);
          }
        }
      } else {
        // a value's partner belongs to another lane
        __syncwarp();
#pragma unroll
        for (int j = 0; j < PIECES; ++j)
          if (4 * (lane + 32 * j) < p.rot_dims) *reinterpret_cast<float4*>(&rows[warp][4 * (lane + 32 * j)]) = x[n][j];
        __syncwarp();
#pragma unroll
        for (int j = 0; j < PIECES; ++j) {
          const int e = 4 * (lane + 32 * j);
          if (e < p.rot_dims) {
            const bool second = e >= half;
            const int i = second ? e - half : e;
            const float4 o = *reinterpret_cast<const float4*>(&rows[warp][second ? e - half : e + half]);
            const float4 c = *reinterpret_cast<const float4*>(cos_row + i);
            float4 s = *reinterpret_cast<const float4*>(sin_row + i);
            if (!second) s = make_float4(-s.x, -s.y, -s.z, -s.w);
            const float4 v = x[n][j];
            x[n][j] = make_float4(v.x * c.x + o.x * s.x, v.y * c.y + o.y * s.y, v.z * c.z + o.z * s.z, v.w * c.w + o.w * s.w);
          }
        }
      }
    }
    T* dst;
    if (is_q) dst = static_cast<T*>(p.q_out) + (static_cast<size_t>(t) * p.num_heads + job) * p.head_dim;
    else if (!stored) continue;
    else if (is_v) dst = static_cast<T*>(p.v_pool) + (place * p.num_kv_heads + (job - p.num_heads - p.num_kv_heads)) * p.value_dim;
    else dst = static_cast<T*>(p.k_pool) + (place * p.num_kv_heads + (job - p.num_heads)) * p.head_dim;
    const float f = is_q ? factor : 1.0f;
#pragma unroll
    for (int j = 0; j < PIECES; ++j) {
      const int e = 4 * (lane + 32 * j);
      if (e >= size) continue;
      const float4 v = x[n][j];
      store_pair(dst + e, v.x * f, v.y * f);
      store_pair(dst + e + 2, v.z * f, v.w * f);
    }
  }
}

template <typename T>
static int launch_head_rows(const HeadRowsParams& p, cudaStream_t s) {
  const int jobs = p.num_heads + 2 * p.num_kv_heads;
  const bool turns = p.style != ROPE_NONE && p.rot_dims > 0;
  const uintptr_t bases = reinterpret_cast<uintptr_t>(p.qkv) | reinterpret_cast<uintptr_t>(p.q_out) | reinterpret_cast<uintptr_t>(p.q_norm) |
                          reinterpret_cast<uintptr_t>(p.k_norm) | reinterpret_cast<uintptr_t>(p.k_pool) | reinterpret_cast<uintptr_t>(p.v_pool) |
                          (turns ? reinterpret_cast<uintptr_t>(p.cos_table) | reinterpret_cast<uintptr_t>(p.sin_table) : 0);
  const bool vectors = p.head_dim % 4 == 0 && p.value_dim % 4 == 0 && p.row_stride % 4 == 0 && (bases & 15) == 0 &&
                       (!turns || (p.style == ROPE_INTERLEAVED ? p.rot_dims % 4 == 0 : p.rot_dims % 8 == 0));
  if (vectors) {
    const dim3 grid(p.num_tokens, (jobs + kHeadWarps * kHeadJobs - 1) / (kHeadWarps * kHeadJobs));
    if (p.head_dim <= 128 && p.value_dim <= 128) return vipera_launch(head_rows_vector_kernel<T, 1>, grid, kHeadWarps * 32, 0, s, p);
    return vipera_launch(head_rows_vector_kernel<T, 2>, grid, kHeadWarps * 32, 0, s, p);
  }
  return vipera_launch(head_rows_kernel<T>, dim3(p.num_tokens, (jobs + kHeadWarps - 1) / kHeadWarps), kHeadWarps * 32, 0, s, p);
}

// dtype: the type of q_out and of the pools.
VIPERA_API int vipera_head_rows(const HeadRowsParams* params, int dtype, void* stream) {
  const HeadRowsParams& p = *params;
  if (p.num_tokens <= 0) return VIPERA_OK;
  if (p.head_dim <= 0 || p.head_dim > kHeadMost || p.value_dim <= 0 || p.value_dim > kHeadMost || p.num_heads <= 0 ||
      p.num_kv_heads <= 0 || p.rot_dims < 0 || (p.rot_dims & 1) || p.rot_dims > p.head_dim || p.norm_size <= 0)
    return VIPERA_BAD_SHAPE;
  if (!p.qkv || !p.q_out || !p.positions) return VIPERA_BAD_ARGUMENT;
  if (p.style != ROPE_NONE && p.rot_dims > 0 && (!p.cos_table || !p.sin_table)) return VIPERA_BAD_ARGUMENT;
  if (p.write_cache && (!p.k_pool || !p.v_pool || !p.token_entry || !p.block_table || p.page_size <= 0)) return VIPERA_BAD_ARGUMENT;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == VIPERA_F32) return launch_head_rows<float>(p, s);
  if (dtype == VIPERA_BF16) return launch_head_rows<__nv_bfloat16>(p, s);
  return VIPERA_BAD_DTYPE;
}

VIPERA_API int vipera_head_rows_params_size() { return static_cast<int>(sizeof(HeadRowsParams)); }

VIPERA_API int vipera_rope_cache(const float* qkv, void* q_out, int dtype, int num_tokens, int num_heads,
                                 int num_kv_heads, int head_dim, const int* positions,
                                 const float* cos_table, const float* sin_table, int style, void* k_pool,
                                 void* v_pool, const int* token_seq, const int* block_table,
                                 int table_width, int page_size, int write_cache, void* stream) {
  if (num_tokens <= 0) return VIPERA_OK;
  if (head_dim <= 0 || (head_dim & 1) || num_heads <= 0 || num_kv_heads <= 0) return VIPERA_BAD_SHAPE;
  if (style != ROPE_NONE && (!cos_table || !sin_table)) return VIPERA_BAD_ARGUMENT;
  if (write_cache && (!k_pool || !v_pool || !token_seq || !block_table || page_size <= 0)) return VIPERA_BAD_ARGUMENT;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  dim3 grid(num_tokens);
  const int work = (num_heads + 2 * num_kv_heads) * (head_dim / 4);
  const int threads = work >= 256 ? 256 : (work >= 128 ? 128 : 64);
  if (dtype == VIPERA_F32)
    return vipera_launch(rope_cache_kernel<float>, grid, threads, 0, s, qkv, static_cast<float*>(q_out), num_heads, num_kv_heads, head_dim,
        positions, cos_table, sin_table, style, static_cast<float*>(k_pool), static_cast<float*>(v_pool),
        token_seq, block_table, table_width, page_size, write_cache);
  if (dtype == VIPERA_BF16)
    return vipera_launch(rope_cache_kernel<__nv_bfloat16>, grid, threads, 0, s, qkv, static_cast<__nv_bfloat16*>(q_out), num_heads, num_kv_heads, head_dim,
        positions, cos_table, sin_table, style, static_cast<__nv_bfloat16*>(k_pool), static_cast<__nv_bfloat16*>(v_pool),
        token_seq, block_table, table_width, page_size, write_cache);
  return VIPERA_BAD_DTYPE;
}

VIPERA_API const char* vipera_rope_cache_status_text(int status) { return vipera_status_text(status); }
