// Attention over a cached low-rank latent.
//
// A token leaves in the cache a latent c [rank] (RMS-normed) and one rotated key part kr [rot]
// that all heads share.  Head h's unrotated key is U_h c and its value V_h c, with U_h [d, rank]
// and V_h [dv, rank].  Since q . (U_h c) = (U_h^T q) . c and sum_j p_j V_h c_j = V_h sum_j p_j c_j, the
// heads attend to the latents themselves:
//
//   qa_h = [U_h^T q_h | rotated q_h] * scale        (latent_absorb_kernel)
//   s_j  = qa_h . [c_j | kr_j],  p = softmax over the visible j,  l_h = sum_j p_j c_j
//                                                    (latent_attention_kernel, latent_fold_kernel)
//   out_h = (V_h l_h) * sigmoid(gate_h)              (latent_expand_kernel)
//
// so the keys and values of earlier tokens are never expanded.  Scores, softmax, the sums over
// keys, the latent's norm and the rotation are 32-bit.  Rotation: values (2i, 2i + 1) of the
// rotated part (`pairing` 0) or values (i, i + rot/2) (`pairing` 1) turn by the angle whose cosine
// and sine the tables hold at [position, i].  With a window w > 0 the query at position p sees keys
// p - w + 1 .. p only; earlier keys' pages may have been given back and are never read.  With a
// sink per head the softmax's denominator also holds exp(sink_h): a term without a key or a value,
// which the scale does not touch.
#include "attention_mma.cuh"

constexpr int kMaxRank = 512;   // latent size
constexpr int kMaxRot = 128;    // rotated part
constexpr int kWarps = 4;

// The two values of the rotated part that turn together as pair i.
__device__ __forceinline__ void rot_pair(int pairing, int rot, int i, int& a, int& b) {
  if (pairing) { a = i; b = i + rot / 2; } else { a = 2 * i; b = 2 * i + 1; }
}

// ---------------------------------------------------------------------------------------
// The step's latents and rotated key parts into their pages.  `proj` [tokens, proj_width] holds
// the down projection at column kv_off: rank latent values, then rot key values.  One block per
// token.  k_pool rows are latents [rank], v_pool rows the rotated key parts [rot].  Where the queries
// come through a latent of their own (q_rank > 0), its pre-norm values are at column cq_off and the
// block leaves them normed in `cq` [tokens, q_rank], the operand of the product that makes the
// queries.  kv_off < 0: the layer keeps nothing of its own, only the query latent is normed.
// ---------------------------------------------------------------------------------------
// blockIdx.y 0: the cache write, 1: the query latent; each block reads its row once.
constexpr int kStoreThreads = 128;
constexpr int kStoreKept = 8;   // values a thread keeps between its two passes: latents up to 1024

template <typename T>
__device__ __forceinline__ void norm_latent(const float* __restrict__ row, int n, const float* __restrict__ weight, float eps,
                                            T* __restrict__ dst, float* scratch) {
  float kept[kStoreKept], gain[kStoreKept], sum = 0.0f;
#pragma unroll
  for (int j = 0; j < kStoreKept; ++j) {
    const int i = threadIdx.x + j * kStoreThreads;
    kept[j] = i < n ? row[i] : 0.0f;
    gain[j] = i < n ? weight[i] : 0.0f;
  }
#pragma unroll
  for (int j = 0; j < kStoreKept; ++j) sum += kept[j] * kept[j];
  for (int i = threadIdx.x + kStoreKept * kStoreThreads; i < n; i += kStoreThreads) sum += row[i] * row[i];
  const float inverse = 1.0f / sqrtf(block_sum(sum, scratch) / static_cast<float>(n) + eps);
#pragma unroll
  for (int j = 0; j < kStoreKept; ++j) {
    const int i = threadIdx.x + j * kStoreThreads;
    if (i < n) dst[i] = from_float<T>(kept[j] * inverse * gain[j]);
  }
  for (int i = threadIdx.x + kStoreKept * kStoreThreads; i < n; i += kStoreThreads) dst[i] = from_float<T>(row[i] * inverse * weight[i]);
}

template <typename T>
__global__ void __launch_bounds__(kStoreThreads)
latent_store_kernel(const float* __restrict__ proj, long long proj_width, int kv_off, const float* __restrict__ norm_weight,
                    float eps, const int* __restrict__ positions, const float* __restrict__ cos_table,
                    const float* __restrict__ sin_table, T* __restrict__ k_pool, T* __restrict__ v_pool,
                    const int* __restrict__ token_entry, const int* __restrict__ block_table, int table_width,
                    int page_size, int rank, int rot, int pairing, int cq_off, int q_rank,
                    const float* __restrict__ cq_norm_weight, T* __restrict__ cq) {
  __shared__ float scratch[32];
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  const float* row = proj + static_cast<size_t>(t) * proj_width;
  if (blockIdx.y == 1 || kv_off < 0) {
    if (q_rank > 0 && (blockIdx.y == 1 || gridDim.y == 1))
      norm_latent<T>(row + cq_off, q_rank, cq_norm_weight, eps, cq + static_cast<size_t>(t) * q_rank, scratch);
    return;
  }
  row += kv_off;
  const int position = positions[t];
  const int page = block_table[static_cast<size_t>(token_entry[t]) * table_width + position / page_size];
  const size_t slot = static_cast<size_t>(page) * page_size + position % page_size;
  T* r_row = v_pool + slot * rot;
  const float* cs = cos_table + static_cast<size_t>(position) * (rot / 2);
  const float* sn = sin_table + static_cast<size_t>(position) * (rot / 2);
  for (int i = threadIdx.x; i < rot / 2; i += blockDim.x) {
    int ia, ib;
    rot_pair(pairing, rot, i, ia, ib);
    const float u = row[rank + ia], v = row[rank + ib];
    r_row[ia] = from_float<T>(u * cs[i] - v * sn[i]);
    r_row[ib] = from_float<T>(v * cs[i] + u * sn[i]);
  }
  norm_latent<T>(row, rank, norm_weight, eps, k_pool + slot * rank, scratch);
}

// ---------------------------------------------------------------------------------------
// qa[t, h, :rank] = scale * sum_d q[t, h, d] U[h, d, :],  qa[t, h, rank:] = scale * rotated q.
// q sits in `proj` at column q_off, head by head as [d unrotated | rot rotated].  U is stored
// [heads * d, rank].  A block serves kTile tokens of one head and 64 columns, so U is read once per tile.
// ---------------------------------------------------------------------------------------
constexpr int kTile = 8;

// acc = A B for up to kTile rows A [kTile][K] (shared memory, transposed: a_t[k * kTile + row]) and COLS
// columns of B [K, n] (rows of n values, COLS neighbouring ones from `b` on).  A block of eight warps:
// a lane takes four neighbouring columns, COLS / 4 lanes a row of B, so a warp reads 128 / COLS rows at
// a time and the eight warps share K between them, all their reads of B in flight together.  The
// warps' sums are added in their order: on return thread i holds element (i / COLS, i % COLS) of the
// tile for i < kTile * COLS (and i + 256 where there are more) through `put`.  n and b's column are
// multiples of 4; columns from `valid` on are not read and come out as 0.
constexpr int kUpThreads = 256;

template <typename TW>
__device__ __forceinline__ float4 load_four(const TW* src);
template <>
__device__ __forceinline__ float4 load_four<float>(const float* src) { return *reinterpret_cast<const float4*>(src); }
template <>
__device__ __forceinline__ float4 load_four<__nv_bfloat16>(const __nv_bfloat16* src) {
  const uint2 raw = *reinterpret_cast<const uint2*>(src);
  const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
  const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
  return make_float4(lo.x, lo.y, hi.x, hi.y);
}

template <typename TW, int COLS, typename Put>
__device__ __forceinline__ void tile_product(const float* a_t, const TW* __restrict__ b, int k_count, int n, int valid,
                                             float* partial /* [8][kTile][COLS] */, Put put) {
  constexpr int kLanes = COLS / 4, kRowsWarp = 32 / kLanes, kStep = 8 * kRowsWarp;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int c4 = (lane % kLanes) * 4, k0 = warp * kRowsWarp + lane / kLanes;
  float acc[kTile][4];
#pragma unroll
  for (int t = 0; t < kTile; ++t)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[t][e] = 0.0f;
  if (c4 < valid) {
#pragma unroll 8
    for (int k = k0; k < k_count; k += kStep) {
      const float4 w = load_four<TW>(b + static_cast<size_t>(k) * n + c4);
      const float4 lo = *reinterpret_cast<const float4*>(a_t + k * kTile), hi = *reinterpret_cast<const float4*>(a_t + k * kTile + 4);
      const float a[kTile] = {lo.x, lo.y, lo.z, lo.w, hi.x, hi.y, hi.z, hi.w};
#pragma unroll
      for (int t = 0; t < kTile; ++t) {
        acc[t][0] = fmaf(a[t], w.x, acc[t][0]);
        acc[t][1] = fmaf(a[t], w.y, acc[t][1]);
        acc[t][2] = fmaf(a[t], w.z, acc[t][2]);
        acc[t][3] = fmaf(a[t], w.w, acc[t][3]);
      }
    }
  }
#pragma unroll
  for (int offset = kLanes; offset < 32; offset <<= 1)
#pragma unroll
    for (int t = 0; t < kTile; ++t)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[t][e] += __shfl_xor_sync(0xffffffffu, acc[t][e], offset);
  if (lane < kLanes) {
#pragma unroll
    for (int t = 0; t < kTile; ++t)
      *reinterpret_cast<float4*>(partial + (warp * kTile + t) * COLS + c4) = make_float4(acc[t][0], acc[t][1], acc[t][2], acc[t][3]);
  }
  __syncthreads();
  for (int i = threadIdx.x; i < kTile * COLS; i += kUpThreads) {
    float sum = partial[i];
#pragma unroll
    for (int w = 1; w < 8; ++w) sum += partial[w * kTile * COLS + i];
    put(i / COLS, i % COLS, sum);
  }
}

// A tile's rows into shared memory, transposed: warp w reads row w.
template <typename Row>
__device__ __forceinline__ void load_tile_rows(float* a_t, int k_count, int count, Row row) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const float* src = row(min(warp, count - 1));
#pragma unroll 8
  for (int k = lane; k < k_count; k += 32) a_t[k * kTile + warp] = warp < count ? src[k] : 0.0f;
}

constexpr int kAbsorbCols = 64;   // columns of the latent a block takes

template <typename TW>
__global__ void __launch_bounds__(kUpThreads)
latent_absorb_kernel(const float* __restrict__ proj, long long proj_width, int q_off, const TW* __restrict__ up_k,
                     const int* __restrict__ positions, const float* __restrict__ cos_table,
                     const float* __restrict__ sin_table, float* __restrict__ qa, int num_tokens, int heads, int d,
                     int rank, int rot, float scale, int pairing) {
  extern __shared__ __align__(16) float up_shared[];
  float* a_t = up_shared;                     // [d][kTile]
  float* partial = up_shared + d * kTile;     // [8][kTile][kAbsorbCols]
  pdl_launch_dependents();
  pdl_wait();
  const int t0 = blockIdx.x * kTile, h = blockIdx.y;
  const int count = min(kTile, num_tokens - t0);
  const int head_width = d + rot;
  load_tile_rows(a_t, d, count, [&](int tt) { return proj + static_cast<size_t>(t0 + tt) * proj_width + q_off + h * head_width; });
  if (blockIdx.z == 0) {
    for (int i = threadIdx.x; i < count * (rot / 2); i += blockDim.x) {
      const int tt = i / (rot / 2), pair = i % (rot / 2);
      const int t = t0 + tt;
      const float* q_rot = proj + static_cast<size_t>(t) * proj_width + q_off + h * head_width + d;
      const int position = positions[t];
      const float c = cos_table[static_cast<size_t>(position) * (rot / 2) + pair];
      const float s = sin_table[static_cast<size_t>(position) * (rot / 2) + pair];
      int ia, ib;
      rot_pair(pairing, rot, pair, ia, ib);
      const float a = q_rot[ia], b = q_rot[ib];
      float* dst = qa + (static_cast<size_t>(t) * heads + h) * (rank + rot) + rank;
      dst[ia] = (a * c - b * s) * scale;
      dst[ib] = (b * c + a * s) * scale;
    }
  }
  __syncthreads();
  const TW* u = up_k + static_cast<size_t>(h) * d * rank;
  const int r0 = blockIdx.z * kAbsorbCols;
  if (rank % 4 == 0) {
    tile_product<TW, kAbsorbCols>(a_t, u + r0, d, rank, rank - r0, partial, [&](int tt, int c, float sum) {
      if (tt < count && r0 + c < rank) qa[(static_cast<size_t>(t0 + tt) * heads + h) * (rank + rot) + r0 + c] = sum * scale;
    });
    return;
  }
  for (int i = threadIdx.x; i < kTile * kAbsorbCols; i += blockDim.x) {   // ranks that are no whole vectors
    const int tt = i / kAbsorbCols, r = r0 + i % kAbsorbCols;
    if (tt >= count || r >= rank) continue;
    float sum = 0.0f;
#pragma unroll 8
    for (int e = 0; e < d; ++e) sum = fmaf(a_t[e * kTile + tt], to_float<TW>(u[static_cast<size_t>(e) * rank + r]), sum);
    qa[(static_cast<size_t>(t0 + tt) * heads + h) * (rank + rot) + r] = sum * scale;
  }
}

// ---------------------------------------------------------------------------------------
// One warp per (token, head) folds the visible keys 32 at a time with a running (max, sum, l):
// a lane scores one key (its whole row), then the 32 latents are added with their weights, a lane
// owning every 32nd latent value.  Causal: the query at position p sees keys 0 .. p.
// ---------------------------------------------------------------------------------------
template <typename T>
__device__ __forceinline__ float dot_span(const float* __restrict__ q, const T* __restrict__ row, int n) {
  float sum = 0.0f;
  for (int i = 0; i < n; ++i) sum = fmaf(q[i], to_float<T>(row[i]), sum);
  return sum;
}
template <>
__device__ __forceinline__ float dot_span<float>(const float* __restrict__ q, const float* __restrict__ row, int n) {
  float sum = 0.0f;
  if (n & 3) {
    for (int i = 0; i < n; ++i) sum = fmaf(q[i], row[i], sum);
    return sum;
  }
  const float4* r4 = reinterpret_cast<const float4*>(row);
  for (int i = 0; i < n / 4; ++i) {
    const float4 v = r4[i];
    sum = fmaf(q[4 * i], v.x, sum);
    sum = fmaf(q[4 * i + 1], v.y, sum);
    sum = fmaf(q[4 * i + 2], v.z, sum);
    sum = fmaf(q[4 * i + 3], v.w, sum);
  }
  return sum;
}
template <>
__device__ __forceinline__ float dot_span<__nv_bfloat16>(const float* __restrict__ q, const __nv_bfloat16* __restrict__ row, int n) {
  float sum = 0.0f;
  if (n & 7) {
    for (int i = 0; i < n; ++i) sum = fmaf(q[i], __bfloat162float(row[i]), sum);
    return sum;
  }
  const uint4* r8 = reinterpret_cast<const uint4*>(row);
  for (int i = 0; i < n / 8; ++i) {
    const uint4 raw = r8[i];
    const __nv_bfloat162* pairs = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float2 f = __bfloat1622float2(pairs[e]);
      sum = fmaf(q[8 * i + 2 * e], f.x, sum);
      sum = fmaf(q[8 * i + 2 * e + 1], f.y, sum);
    }
  }
  return sum;
}

template <typename T>
__global__ void __launch_bounds__(kWarps * 32)
latent_attention_kernel(const float* __restrict__ qa, float* __restrict__ mixed, const T* __restrict__ k_pool,
                        const T* __restrict__ v_pool, const int* __restrict__ token_entry,
                        const int* __restrict__ positions, const int* __restrict__ block_table, int table_width,
                        int page_size, int heads, int rank, int rot, int window, const float* __restrict__ sink) {
  extern __shared__ float q_shared[];   // [kWarps][rank + rot]
  pdl_launch_dependents();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x;
  const int h = blockIdx.y * kWarps + warp;
  if (h >= heads) return;
  const int width = rank + rot;
  const int position = positions[t];
  const int* table = block_table + static_cast<size_t>(token_entry[t]) * table_width;
  float* qs = q_shared + warp * width;
  const float* q_row = qa + (static_cast<size_t>(t) * heads + h) * width;
  for (int i = lane; i < width; i += 32) qs[i] = q_row[i];
  __syncwarp();

  float acc[kMaxRank / 32];
#pragma unroll
  for (int i = 0; i < kMaxRank / 32; ++i) acc[i] = 0.0f;
  float running_max = -INFINITY, running_sum = 0.0f;
  for (int base = window > 0 ? max(0, position - window + 1) : 0; base <= position; base += 32) {
    const int j = base + lane;
    const bool valid = j <= position;
    float score = -INFINITY;
    if (valid) {
      const size_t slot = static_cast<size_t>(table[j / page_size]) * page_size + j % page_size;
      score = dot_span<T>(qs, k_pool + slot * rank, rank) + dot_span<T>(qs + rank, v_pool + slot * rot, rot);
    }
    const float new_max = fmaxf(running_max, warp_max(score));
    const float alpha = expf(running_max - new_max);   // 0 on the first tile
    const float weight = valid ? expf(score - new_max) : 0.0f;
    running_sum = running_sum * alpha + warp_sum(weight);
    running_max = new_max;
#pragma unroll
    for (int i = 0; i < kMaxRank / 32; ++i) acc[i] *= alpha;
    const int count = min(32, position - base + 1);
    for (int jj = 0; jj < count; ++jj) {
      const float w = __shfl_sync(0xffffffffu, weight, jj);
      const int key = base + jj;
      const T* c_row = k_pool + (static_cast<size_t>(table[key / page_size]) * page_size + key % page_size) * rank;
#pragma unroll
      for (int i = 0; i < kMaxRank / 32; ++i) {
        const int e = lane + 32 * i;
        if (e < rank) acc[i] = fmaf(w, to_float<T>(c_row[e]), acc[i]);
      }
    }
  }
  if (sink) {
    // where the sink is far above every score the quotient is 0, as it should be
    running_sum += expf(sink[h] - running_max);
  }
  const float inverse = 1.0f / running_sum;
  float* out_row = mixed + (static_cast<size_t>(t) * heads + h) * rank;
#pragma unroll
  for (int i = 0; i < kMaxRank / 32; ++i) {
    const int e = lane + 32 * i;
    if (e < rank) out_row[e] = acc[i] * inverse;
  }
}

// ---------------------------------------------------------------------------------------
// The same fold on the tensor cores (bfloat16 caches; mma.sync m16n8k16, 32-bit accumulation).
// A block owns 16 (or 32) query rows, a row being a (token, head) and the rows of a step numbered token
// by token: `tile_rows` neighbouring rows (whole tokens where the heads allow and rows are few, so that
// a step of single tokens folds each request's keys once; else as many as the block holds).  A tile
// that spans several requests is folded once per request, the other requests' rows masked.  Keys come 64 at a time as rows [c | kr] of shared
// memory, the next tile on its way (cp.async) while this one is used.  Per tile the eight warps
//   1. each score 8 keys against all 16 rows: S = Q K^T over rank + rot values;
//   2. each take two rows: running maximum, weights p = exp(s - m) rounded to bfloat16, their sum;
//   3. each add P C into their 1/8 of the latent's columns.
// With `num_splits` > 1 a block folds `split_keys` keys only and leaves (m, sum, unnormalised
// columns); latent_combine_kernel joins the splits.  The splits are counted from key 0 or, with a
// window, from the tile of 64 keys that holds the first key the pass's rows see (so a long history
// costs a windowed step no more than the window).  NR: the columns the block's
// accumulators cover (128, 256 or 512, at least the rank rounded up to 16).
// ---------------------------------------------------------------------------------------
constexpr int kFoldRows = 16;
constexpr int kFoldKeys = 64;
constexpr int kFoldThreads = 256;
constexpr int kScoreStride = kFoldKeys + 4;   // floats
constexpr int kWeightStride = kFoldKeys + 8;  // bf16

struct LatentFoldParams {
  const float* qa;                 // [tokens, heads, rank + rot]
  const __nv_bfloat16* k_pool;     // latents
  const __nv_bfloat16* v_pool;     // rotated key parts
  const int* token_entry;
  const int* positions;
  const int* block_table;
  float* out;                      // [tokens * heads, rank]
  float* part;                     // splits: [num_splits][tokens * heads][rank + 2]: columns, then m and sum
  int num_tokens, heads, rank, rot, table_width, page_size;
  int tile_rows, split_keys, num_splits;
  int window;                      // > 0: a row at position p sees keys p - window + 1 .. p
  const float* sink;               // [heads] or null: exp(sink_h) joins the softmax's denominator
  // Head-major form (the products on both sides of the fold run as grouped tensor-core products, a
  // head a group): the unrotated part of qa comes unscaled from qa_heads [heads, padded_tokens, rank]
  // and the rotated, scaled part from q_rot [tokens, heads, rot]; the folded latents leave as
  // bfloat16 rows of l_heads [heads, padded_tokens, rank].  Null: qa and out as above.
  const float* qa_heads;
  const float* q_rot;
  __nv_bfloat16* l_heads;
  int padded_tokens;
  float scale;
};

__host__ __device__ __forceinline__ int round_up(int v, int to) { return (v + to - 1) / to * to; }

template <int NR, int MT>
__global__ void __launch_bounds__(kFoldThreads)
latent_fold_kernel(LatentFoldParams p) {
  extern __shared__ __align__(16) unsigned char fold_shared[];
  const int rank_pad = round_up(p.rank, 16);
  const int width_pad = round_up(rank_pad + round_up(p.rot, 16), 32);
  const int stride = width_pad + 8;   // bf16 per row: rows 16 bytes apart modulo 128, so ldmatrix meets no bank twice
  __nv_bfloat16* q_s = reinterpret_cast<__nv_bfloat16*>(fold_shared);
  constexpr int kRows = kFoldRows * MT;   // MT groups of sixteen rows share every tile of keys
  __nv_bfloat16* k_s = q_s + kRows * stride;                       // two tiles of kFoldKeys rows
  float* s_s = reinterpret_cast<float*>(k_s + 2 * kFoldKeys * stride);
  __nv_bfloat16* p_s = reinterpret_cast<__nv_bfloat16*>(s_s + kRows * kScoreStride);
  float* m_s = reinterpret_cast<float*>(p_s + kRows * kWeightStride);
  float* l_s = m_s + kRows;
  float* alpha_s = l_s + kRows;
  int* limit_s = reinterpret_cast<int*>(alpha_s + kRows);
  int* row_s = limit_s + kRows;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  {
    // what the copies never write (the columns that pad rank and rot) must read as zero
    const int pad_a = (rank_pad - p.rank) / 8, pads = pad_a + (width_pad - rank_pad - p.rot) / 8;
    for (int i = threadIdx.x; i < (kRows + 2 * kFoldKeys) * pads; i += kFoldThreads) {
      const int row = i / pads, c = i % pads;   // (q_s and k_s follow one another)
      const int column = c < pad_a ? p.rank + c * 8 : rank_pad + p.rot + (c - pad_a) * 8;
      *reinterpret_cast<uint4*>(q_s + row * stride + column) = make_uint4(0u, 0u, 0u, 0u);
    }
  }
  pdl_launch_dependents();
  pdl_wait();
  const int total_rows = p.num_tokens * p.heads;
  const int row0 = (gridDim.x - 1 - blockIdx.x) * p.tile_rows;   // the longest histories of a prompt first
  const int rows_here = min(p.tile_rows, total_rows - row0);
  const int t0 = row0 / p.heads, tokens_here = (row0 + rows_here - 1) / p.heads - t0 + 1;   // at most kRows
  const int split = blockIdx.y;
  const int width = p.rank + p.rot;
  const int rank_chunks = p.rank / 8, row_chunks = rank_chunks + p.rot / 8;
  unsigned done = 0;
  for (;;) {
    int lead = -1;
    for (int tq = 0; tq < tokens_here; ++tq)
      if (!((done >> tq) & 1u)) { lead = tq; break; }
    if (lead < 0) break;
    const int entry = p.token_entry[t0 + lead];
    int last_key = -1, first_key = 0x7fffffff;
    unsigned taken = 0;
    for (int tq = lead; tq < tokens_here; ++tq)
      if (!((done >> tq) & 1u) && p.token_entry[t0 + tq] == entry) {
        taken |= 1u << tq;
        last_key = max(last_key, p.positions[t0 + tq]);
        first_key = min(first_key, p.positions[t0 + tq]);
      }
    // the first key any of the pass's rows sees: nothing before it is read (its page may be gone)
    first_key = p.window > 0 ? max(0, first_key - p.window + 1) : 0;
    __syncthreads();   // the pass before is done with the rows' tables
    if (threadIdx.x < kRows) {
      const int r = threadIdx.x, tq = min((row0 + r) / p.heads - t0, 31);
      const bool valid = r < rows_here && ((taken >> tq) & 1u);
      limit_s[r] = valid ? p.positions[t0 + tq] : -1;
      row_s[r] = valid ? row0 + r : -1;
      m_s[r] = -INFINITY;
      l_s[r] = 0.0f;
    }
    done |= taken;
    __syncthreads();
    // first_key is 0 without a window; tiles start at multiples of kFoldKeys either way
    const int begin = first_key / kFoldKeys * kFoldKeys + split * p.split_keys;
    const int end = p.num_splits > 1 ? min(last_key + 1, begin + p.split_keys) : last_key + 1;
    const int num_tiles = end > begin ? (end - begin + kFoldKeys - 1) / kFoldKeys : 0;
    if (num_tiles == 0) {   // a split that sees no key says so (and leaves no columns); only splits can be such
      if (threadIdx.x < kRows && row_s[threadIdx.x] >= 0 && p.num_splits > 1) {
        float* part = p.part + (static_cast<size_t>(split) * total_rows + row_s[threadIdx.x]) * (p.rank + 2);
        part[p.rank] = -INFINITY;
        part[p.rank + 1] = 0.0f;
      }
      continue;
    }
    const int* table = p.block_table + static_cast<size_t>(entry) * p.table_width;

    // A warp copies 8 keys of a tile.  Their places in the pools are looked up a tile ahead, a lane a
    // key, so that the copies need not wait for the page table; then each row's 16-byte pieces, a lane
    // taking every 32nd.
    auto look_up = [&](int tile) {
      const int key = max(min(begin + tile * kFoldKeys + warp * 8 + (lane & 7), end - 1), first_key);
      return static_cast<unsigned>(table[key / p.page_size]) * static_cast<unsigned>(p.page_size) + key % p.page_size;
    };
    auto copy_tile = [&](int tile, unsigned place) {
      __nv_bfloat16* dst_tile = k_s + (tile & 1) * kFoldKeys * stride;
      const int key0 = begin + tile * kFoldKeys + warp * 8;
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const bool valid = key0 + i < end && key0 + i >= first_key;
        const size_t slot = __shfl_sync(0xffffffffu, place, i);
        const __nv_bfloat16* c_row = p.k_pool + slot * p.rank;
        const __nv_bfloat16* r_row = p.v_pool + slot * p.rot;
        __nv_bfloat16* dst = dst_tile + (warp * 8 + i) * stride;
        for (int chunk = lane; chunk < row_chunks; chunk += 32) {
          const bool latent = chunk < rank_chunks;
          cp_async_16(smem_addr(dst + (latent ? chunk * 8 : rank_pad + (chunk - rank_chunks) * 8)),
                      latent ? c_row + chunk * 8 : r_row + (chunk - rank_chunks) * 8, valid);
        }
      }
      cp_async_commit();
    };

    constexpr int kPairs = NR / 8 / 16;   // pairs of 8-column tiles a warp accumulates
    float acc[MT][2 * kPairs][4];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int j = 0; j < 2 * kPairs; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[mt][j][e] = 0.0f;
    const int column0 = warp * (NR / 8);
    const int g = lane >> 2, pair = (lane & 3) * 2;
    copy_tile(0, look_up(0));
    unsigned ahead = num_tiles > 1 ? look_up(1) : 0u;
    // The queries while the first keys are on their way: 8 values at a time, four reads in flight a thread.
    constexpr int kAtOnce = 4;
    for (int i0 = threadIdx.x; i0 < kRows * row_chunks; i0 += kAtOnce * kFoldThreads) {
      float4 lo[kAtOnce], hi[kAtOnce];
#pragma unroll
      for (int j = 0; j < kAtOnce; ++j) {
        const int i = i0 + j * kFoldThreads;
        const int r = i / row_chunks, c = (i - r * row_chunks) * 8;
        const int source_row = r < kRows ? row_s[r] : -1;
        lo[j] = hi[j] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        if (source_row >= 0) {
          const float* src;
          if (p.qa_heads == nullptr) src = p.qa + static_cast<size_t>(source_row) * width + c;
          else if (c < p.rank)
            src = p.qa_heads + (static_cast<size_t>(source_row % p.heads) * p.padded_tokens + source_row / p.heads) * p.rank + c;
          else src = p.q_rot + static_cast<size_t>(source_row) * p.rot + c - p.rank;
          lo[j] = *reinterpret_cast<const float4*>(src);
          hi[j] = *reinterpret_cast<const float4*>(src + 4);
        }
      }
#pragma unroll
      for (int j = 0; j < kAtOnce; ++j) {
        const int i = i0 + j * kFoldThreads;
        const int r = i / row_chunks, c = (i - r * row_chunks) * 8;
        if (r >= kRows) continue;
        const float f = p.qa_heads != nullptr && c < p.rank ? p.scale : 1.0f;
        *reinterpret_cast<uint4*>(q_s + r * stride + (c < p.rank ? c : rank_pad + c - p.rank)) =
            make_uint4(pack_bf16(lo[j].x * f, lo[j].y * f), pack_bf16(lo[j].z * f, lo[j].w * f),
                       pack_bf16(hi[j].x * f, hi[j].y * f), pack_bf16(hi[j].z * f, hi[j].w * f));
      }
    }
    for (int tile = 0; tile < num_tiles; ++tile) {
      cp_async_wait<0>();
      __syncthreads();   // this tile has landed (and the queries, before the first); the tile before is read out
      if (tile + 1 < num_tiles) {
        copy_tile(tile + 1, ahead);
        if (tile + 2 < num_tiles) ahead = look_up(tile + 2);
      }
      const __nv_bfloat16* keys = k_s + (tile & 1) * kFoldKeys * stride;
      const int key0 = begin + tile * kFoldKeys;
      {
        float c[MT][4], c_odd[MT][4];   // two chains of products per group of rows
#pragma unroll
        for (int mt = 0; mt < MT; ++mt)
#pragma unroll
          for (int e = 0; e < 4; ++e) c[mt][e] = c_odd[mt][e] = 0.0f;
        const uint32_t k_addr = smem_addr(keys + (warp * 8 + (lane & 7)) * stride + (lane >> 3) * 8);
        const uint32_t q_addr = smem_addr(q_s + ((lane & 7) + ((lane >> 3) & 1) * 8) * stride + (lane >> 4) * 8);
#pragma unroll 3
        for (int k0 = 0; k0 < width_pad; k0 += 32) {
          uint32_t b[4];
          ldmatrix_x4(b, k_addr + k0 * 2);
#pragma unroll
          for (int mt = 0; mt < MT; ++mt) {
            uint32_t a[4], a_odd[4];
            ldmatrix_x4(a, q_addr + (mt * kFoldRows * stride + k0) * 2);
            ldmatrix_x4(a_odd, q_addr + (mt * kFoldRows * stride + k0 + 16) * 2);
            mma_16816(c[mt], a, b[0], b[1]);
            mma_16816(c_odd[mt], a_odd, b[2], b[3]);
          }
        }
#pragma unroll
        for (int mt = 0; mt < MT; ++mt)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int row = mt * kFoldRows + g + (e >> 1) * 8, col = warp * 8 + pair + (e & 1);
            const int key = key0 + col;
            const bool seen = key <= limit_s[row] && key < end && (p.window <= 0 || key > limit_s[row] - p.window);
            s_s[row * kScoreStride + col] = seen ? c[mt][e] + c_odd[mt][e] : -INFINITY;
          }
      }
      __syncthreads();
      {
        // a warp's rows side by side, so that their reductions fill one another's waits; a lane takes
        // two neighbouring keys
        constexpr int kOwn = 2 * MT;
        const int own0 = warp * kOwn;
        float2 v[kOwn];
        float before[kOwn], top[kOwn], sum[kOwn];
#pragma unroll
        for (int i = 0; i < kOwn; ++i) {
          v[i] = *reinterpret_cast<const float2*>(s_s + (own0 + i) * kScoreStride + 2 * lane);
          before[i] = m_s[own0 + i];
          top[i] = fmaxf(v[i].x, v[i].y);
        }
#pragma unroll
        for (int offset = 16; offset > 0; offset >>= 1)
#pragma unroll
          for (int i = 0; i < kOwn; ++i) top[i] = fmaxf(top[i], __shfl_xor_sync(0xffffffffu, top[i], offset));
#pragma unroll
        for (int i = 0; i < kOwn; ++i) {
          top[i] = fmaxf(top[i], before[i]);
          const float shift = top[i] > -INFINITY ? top[i] : 0.0f;   // (a row that has seen nothing: e^(-inf) = 0)
          const __nv_bfloat162 w = __floats2bfloat162_rn(expf(v[i].x - shift), expf(v[i].y - shift));
          *reinterpret_cast<__nv_bfloat162*>(p_s + (own0 + i) * kWeightStride + 2 * lane) = w;
          const float2 rounded = __bfloat1622float2(w);
          sum[i] = rounded.x + rounded.y;
        }
#pragma unroll
        for (int offset = 16; offset > 0; offset >>= 1)
#pragma unroll
          for (int i = 0; i < kOwn; ++i) sum[i] += __shfl_xor_sync(0xffffffffu, sum[i], offset);
#pragma unroll
        for (int i = 0; i < kOwn; ++i) {
          if (lane == i) {
            const float alpha = top[i] > -INFINITY ? expf(before[i] - top[i]) : 1.0f;   // 0 while nothing was seen
            m_s[own0 + i] = top[i];
            l_s[own0 + i] = l_s[own0 + i] * alpha + sum[i];
            alpha_s[own0 + i] = alpha;
          }
        }
      }
      __syncthreads();
      {
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) {
          const float alpha0 = alpha_s[mt * kFoldRows + g], alpha1 = alpha_s[mt * kFoldRows + g + 8];
#pragma unroll
          for (int j = 0; j < 2 * kPairs; ++j) {
            acc[mt][j][0] *= alpha0, acc[mt][j][1] *= alpha0;
            acc[mt][j][2] *= alpha1, acc[mt][j][3] *= alpha1;
          }
        }
        const uint32_t p_addr = smem_addr(p_s + ((lane & 7) + ((lane >> 3) & 1) * 8) * kWeightStride + (lane >> 4) * 8);
        const uint32_t c_addr = smem_addr(keys + ((lane & 7) + ((lane >> 3) & 1) * 8) * stride + column0 + (lane >> 4) * 8);
#pragma unroll
        for (int kk = 0; kk < kFoldKeys / 16; ++kk) {
          uint32_t a[MT][4];
#pragma unroll
          for (int mt = 0; mt < MT; ++mt) ldmatrix_x4(a[mt], p_addr + (mt * kFoldRows * kWeightStride + kk * 16) * 2);
#pragma unroll
          for (int j = 0; j < kPairs; ++j) {
            if (column0 + 16 * j < rank_pad) {
              uint32_t b[4];
              ldmatrix_x4_trans(b, c_addr + (kk * 16 * stride + 16 * j) * 2);
#pragma unroll
              for (int mt = 0; mt < MT; ++mt) {
                mma_16816(acc[mt][2 * j], a[mt], b[0], b[1]);
                mma_16816(acc[mt][2 * j + 1], a[mt], b[2], b[3]);
              }
            }
          }
        }
      }
    }
    __syncthreads();   // the last sums are written
#pragma unroll
    for (int part_row = 0; part_row < 2 * MT; ++part_row) {
      const int mt = part_row >> 1, half = part_row & 1;
      const int row = mt * kFoldRows + g + half * 8;
      const int out_row = row_s[row];
      if (out_row < 0) continue;
      float total = l_s[row];
      if (p.sink && p.num_splits == 1) total += expf(p.sink[out_row % p.heads] - m_s[row]);
      if (p.num_splits == 1 && p.l_heads != nullptr) {
        const float inverse = 1.0f / total;
        __nv_bfloat16* l_row = p.l_heads + (static_cast<size_t>(out_row % p.heads) * p.padded_tokens + out_row / p.heads) * p.rank;
#pragma unroll
        for (int j = 0; j < 2 * kPairs; ++j) {
          const int col = column0 + 8 * j + pair;   // (even, and the rank is a multiple of 8)
          if (col < p.rank)
            *reinterpret_cast<uint32_t*>(l_row + col) = pack_bf16(acc[mt][j][2 * half] * inverse, acc[mt][j][2 * half + 1] * inverse);
        }
      } else if (p.num_splits == 1) {
        const float inverse = 1.0f / total;
#pragma unroll
        for (int j = 0; j < 2 * kPairs; ++j) {
          const int col = column0 + 8 * j + pair;
          if (col < p.rank) p.out[static_cast<size_t>(out_row) * p.rank + col] = acc[mt][j][2 * half] * inverse;
          if (col + 1 < p.rank) p.out[static_cast<size_t>(out_row) * p.rank + col + 1] = acc[mt][j][2 * half + 1] * inverse;
        }
      } else {
        float* part = p.part + (static_cast<size_t>(split) * total_rows + out_row) * (p.rank + 2);
#pragma unroll
        for (int j = 0; j < 2 * kPairs; ++j) {
          const int col = column0 + 8 * j + pair;
          if (col < p.rank) part[col] = acc[mt][j][2 * half];
          if (col + 1 < p.rank) part[col + 1] = acc[mt][j][2 * half + 1];
        }
        if (warp == 0 && pair == 0) {
          part[p.rank] = m_s[row];
          part[p.rank + 1] = total;
        }
      }
    }
  }
}

// out[row, :] = sum_s e^(m_s - m) columns_s / sum_s e^(m_s - m) sum_s over the splits that saw a key
// (the others left no columns).  The first warp reads the splits' maxima and sums side by side and lists
// the splits that count with their weights e^(m_s - m) / total; a column's terms are asked for eight
// splits at a time and added in the splits' order.
constexpr int kMostSplits = 64;

__global__ void __launch_bounds__(128)
latent_combine_kernel(LatentFoldParams p) {
  __shared__ float weight_s[kMostSplits];
  __shared__ int split_s[kMostSplits];
  __shared__ int counted;
  pdl_launch_dependents();
  pdl_wait();
  const int row = blockIdx.x;
  const size_t rows = static_cast<size_t>(p.num_tokens) * p.heads, each = p.rank + 2;
  const float* first = p.part + static_cast<size_t>(row) * each;
  if (threadIdx.x < 32) {
    const int lane = threadIdx.x;
    float top[2], sum[2];
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int split = lane + 32 * j;
      const float* part = first + static_cast<size_t>(min(split, p.num_splits - 1)) * rows * each;
      sum[j] = split < p.num_splits ? part[p.rank + 1] : 0.0f;
      top[j] = sum[j] > 0.0f ? part[p.rank] : -INFINITY;
    }
    const float most = warp_max(fmaxf(top[0], top[1]));
    float weight[2];
#pragma unroll
    for (int j = 0; j < 2; ++j) weight[j] = sum[j] > 0.0f ? expf(top[j] - most) : 0.0f;
    float total = warp_sum(sum[0] * weight[0] + sum[1] * weight[1]);
    if (p.sink) total += expf(p.sink[row % p.heads] - most);
    const float inverse = 1.0f / total;
    int base = 0;
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const unsigned live = __ballot_sync(0xffffffffu, sum[j] > 0.0f);
      if (sum[j] > 0.0f) {
        const int at = base + __popc(live & ((1u << lane) - 1u));
        split_s[at] = lane + 32 * j;
        weight_s[at] = weight[j] * inverse;
      }
      base += __popc(live);
    }
    if (lane == 0) counted = base;
  }
  __syncthreads();
  const int splits = counted;
  // two neighbouring columns to a thread where rows are whole pairs (`each` is even with the rank)
  const bool pairs = (p.rank & 1) == 0;
  for (int c = threadIdx.x * 2; c < p.rank; c += 2 * blockDim.x) {
    float sum0 = 0.0f, sum1 = 0.0f;
    for (int s0 = 0; s0 < splits; s0 += 8) {
      float2 v[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const float* part = first + static_cast<size_t>(split_s[min(s0 + i, splits - 1)]) * rows * each + c;
        if (pairs) v[i] = *reinterpret_cast<const float2*>(part);
        else v[i] = make_float2(part[0], c + 1 < p.rank ? part[1] : 0.0f);
      }
#pragma unroll
      for (int i = 0; i < 8; ++i)
        if (s0 + i < splits) {
          sum0 = fmaf(v[i].x, weight_s[s0 + i], sum0);
          sum1 = fmaf(v[i].y, weight_s[s0 + i], sum1);
        }
    }
    if (p.l_heads != nullptr) {
      __nv_bfloat16* dst = p.l_heads + (static_cast<size_t>(row % p.heads) * p.padded_tokens + row / p.heads) * p.rank + c;
      dst[0] = __float2bfloat16(sum0);
      if (c + 1 < p.rank) dst[1] = __float2bfloat16(sum1);
    } else {
      float* dst = p.out + static_cast<size_t>(row) * p.rank + c;
      dst[0] = sum0;
      if (c + 1 < p.rank) dst[1] = sum1;
    }
  }
}

// ---------------------------------------------------------------------------------------
// Head-major form, in front of the fold: a block per token puts each head's unrotated q values
// (bfloat16) at row [head, token] of a_heads [heads, padded_tokens, d], the operand of the grouped
// product with U_h^T, and the rotated, scaled rest at q_rot [token, head, rot].  The first block
// also fills the table that gives every tile of 128 rows its head.
// ---------------------------------------------------------------------------------------
__global__ void __launch_bounds__(128)
latent_prep_kernel(const float* __restrict__ proj, long long proj_width, int q_off, const int* __restrict__ positions,
                   const float* __restrict__ cos_table, const float* __restrict__ sin_table,
                   __nv_bfloat16* __restrict__ a_heads, float* __restrict__ q_rot, int* __restrict__ tile_group,
                   int heads, int d, int rot, int padded_tokens, float scale, int pairing) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  if (t == 0)
    for (int i = threadIdx.x; i < heads * (padded_tokens / 128); i += blockDim.x) tile_group[i] = i / (padded_tokens / 128);
  const float* row = proj + static_cast<size_t>(t) * proj_width + q_off;
  for (int i = threadIdx.x; i < heads * d; i += blockDim.x) {
    const int h = i / d, e = i % d;
    a_heads[(static_cast<size_t>(h) * padded_tokens + t) * d + e] = __float2bfloat16(row[h * (d + rot) + e]);
  }
  const int position = positions[t];
  const float* cs = cos_table + static_cast<size_t>(position) * (rot / 2);
  const float* sn = sin_table + static_cast<size_t>(position) * (rot / 2);
  for (int i = threadIdx.x; i < heads * (rot / 2); i += blockDim.x) {
    const int h = i / (rot / 2), pair = i % (rot / 2);
    int ia, ib;
    rot_pair(pairing, rot, pair, ia, ib);
    const float a = row[h * (d + rot) + d + ia], b = row[h * (d + rot) + d + ib];
    float* dst = q_rot + (static_cast<size_t>(t) * heads + h) * rot;
    dst[ia] = (a * cs[pair] - b * sn[pair]) * scale;
    dst[ib] = (b * cs[pair] + a * sn[pair]) * scale;
  }
}

// Head-major form, behind the second product: out[t, h * dv + v] = o_heads[h, t, v] * sigmoid(gate).
template <typename TO>
__global__ void __launch_bounds__(256)
latent_gate_kernel(const float* __restrict__ o_heads, const float* __restrict__ proj, long long proj_width, int g_off,
                   TO* __restrict__ out, int num_tokens, int heads, int dv, int padded_tokens) {
  pdl_launch_dependents();
  pdl_wait();
  const long long i = static_cast<long long>(blockIdx.x) * blockDim.x + threadIdx.x;
  if (i >= static_cast<long long>(num_tokens) * heads * dv) return;
  const long long t = i / (heads * dv);
  const int c = static_cast<int>(i % (heads * dv)), h = c / dv, v = c % dv;
  float y = o_heads[(static_cast<size_t>(h) * padded_tokens + t) * dv + v];
  if (g_off >= 0) y *= 1.0f / (1.0f + expf(-proj[t * proj_width + g_off + c]));
  out[i] = from_float<TO>(y);
}

// ---------------------------------------------------------------------------------------
// out[t, h * dv + v] = (sum_r l[t, h, r] V[h, r, v]) * sigmoid(gate[t, h * dv + v]); a block: kTile tokens of
// one head, 32 values.  V is stored
// transposed per head, [heads, rank, dv], so that neighbouring threads read neighbouring values.
// `gate` is the pre-activation in `proj` at column g_off (g_off < 0: no gate).
// ---------------------------------------------------------------------------------------
constexpr int kExpandCols = 32;   // values of a head a block takes

template <typename TW, typename TO>
__global__ void __launch_bounds__(kUpThreads)
latent_expand_kernel(const float* __restrict__ latent_out, const TW* __restrict__ up_v, const float* __restrict__ proj,
                     long long proj_width, int g_off, TO* __restrict__ out, int num_tokens, int heads, int dv,
                     int rank) {
  extern __shared__ __align__(16) float up_shared[];
  float* a_t = up_shared;                       // [rank][kTile]
  float* partial = up_shared + rank * kTile;    // [8][kTile][kExpandCols]
  pdl_launch_dependents();
  pdl_wait();
  const int t0 = blockIdx.x * kTile, h = blockIdx.y;
  const int count = min(kTile, num_tokens - t0);
  load_tile_rows(a_t, rank, count, [&](int tt) { return latent_out + (static_cast<size_t>(t0 + tt) * heads + h) * rank; });
  __syncthreads();
  const TW* w = up_v + static_cast<size_t>(h) * rank * dv;
  const int v0 = blockIdx.z * kExpandCols;
  auto put = [&](int tt, int c, float y) {
    if (tt >= count || v0 + c >= dv) return;
    const size_t t = t0 + tt;
    if (g_off >= 0) y *= 1.0f / (1.0f + expf(-proj[t * proj_width + g_off + h * dv + v0 + c]));
    out[(t * heads + h) * dv + v0 + c] = from_float<TO>(y);
  };
  if (dv % 4 == 0) {
    tile_product<TW, kExpandCols>(a_t, w + v0, rank, dv, dv - v0, partial, put);
    return;
  }
  for (int i = threadIdx.x; i < kTile * kExpandCols; i += blockDim.x) {
    const int tt = i / kExpandCols, c = i % kExpandCols;
    if (tt >= count || v0 + c >= dv) continue;
    float sum = 0.0f;
#pragma unroll 8
    for (int r = 0; r < rank; ++r) sum = fmaf(a_t[r * kTile + tt], to_float<TW>(w[static_cast<size_t>(r) * dv + v0 + c]), sum);
    put(tt, c, sum);
  }
}

struct LatentParams {
  const float* proj;       // [tokens, proj_width] 32-bit: q, the gate's pre-activation, the down projection
  long long proj_width;
  int q_off, g_off, kv_off;  // columns; g_off < 0: no gate; kv_off < 0: the layer reads a cache it does not write
  const void* up_k;        // [heads * d, rank]
  const void* up_v;        // [heads, rank, dv]
  const float* norm_weight;  // [rank]
  const int* positions;
  const int* token_entry;
  const int* block_table;
  const float* cos_table;
  const float* sin_table;
  void* k_pool;            // latents [pages, page_size, 1, rank]
  void* v_pool;            // rotated key parts [pages, page_size, 1, rot]
  float* qa;               // scratch [tokens, heads, rank + rot]
  float* latent_out;       // scratch [tokens, heads, rank]
  void* out;               // [tokens, heads * dv]
  int num_tokens, heads, d, rot, dv, rank, table_width, page_size;
  float scale, eps;
  float* part;             // scratch of the tensor-core fold's splits: [num_splits][tokens * heads][rank + 2], or null
  int split_keys, num_splits;   // as vipera_latent_plan gives them (1 split: the whole history in one block)
  // Head-major form (bfloat16): the caller runs the grouped products between the stages.
  //   stage 1: cache write, a_heads, q_rot, tile_group;  [qa_heads = a_heads x U_h^T]
  //   stage 2: the fold, leaving l_heads;                [o_heads = l_heads x V_h^T]
  //   stage 3: the gate and the output.    stage 0: everything in one call, without these buffers.
  int stage, padded_tokens;
  void* a_heads;           // [heads, padded_tokens, d]
  float* qa_heads;         // [heads, padded_tokens, rank]
  float* q_rot;            // [tokens, heads, rot]
  void* l_heads;           // [heads, padded_tokens, rank]
  float* o_heads;          // [heads, padded_tokens, dv]
  int* tile_group;         // [heads * padded_tokens / 128]
  int window;              // > 0: a query at position p sees keys p - window + 1 .. p
  int pairing;             // of the rotated part: 0 values (2i, 2i + 1), 1 values (i, i + rot/2)
  const float* sink;       // [heads] or null
  // Queries that are no columns of `proj`: [tokens, q_width], at column q_off (null: in `proj`).
  const float* q;
  long long q_width;
  // stage 4 (ahead of the product that makes such queries): the cache write as above and, with
  // q_rank > 0, the normed query latent.
  int cq_off, q_rank;
  const float* cq_norm_weight;   // [q_rank]
  void* cq;                      // [tokens, q_rank], the run's type
  int single;              // 1: every request of the step brings one token
};

// How the tensor-core fold cuts a step.  Rows are tokens x heads.  Many rows: two groups of sixteen to a
// block.  Few rows (decode) are cut along the keys besides, in whole tiles of 64; whole tokens to a
// block then, one at a time where every request brings one token (`single`), so that no block folds
// the keys of two requests one behind the other.
struct FoldPlan { int groups, tile_rows, tiles, split_keys, num_splits; };

static size_t fold_shared_bytes(int rank, int rot, int groups) {
  const int rank_pad = round_up(rank, 16), rows = kFoldRows * groups;
  const int stride = round_up(rank_pad + round_up(rot, 16), 32) + 8;
  return static_cast<size_t>(rows + 2 * kFoldKeys) * stride * 2 + rows * kScoreStride * 4 + rows * kWeightStride * 2 + rows * 5 * 4;
}

static FoldPlan latent_plan(int tokens, int heads, int rank, int rot, int max_keys, int window, int single, int sms) {
  FoldPlan plan{};
  const long rows = static_cast<long>(tokens) * heads;
  const bool many = rows >= 2L * sms * kFoldRows && !single;
  plan.groups = many || (heads > kFoldRows && single) ? 2 : 1;
  const int most = kFoldRows * plan.groups;
  plan.tile_rows = most;
  if (!many && heads <= most) plan.tile_rows = single ? heads : most / heads * heads;
  plan.tiles = static_cast<int>((rows + plan.tile_rows - 1) / plan.tile_rows);
  // histories grow from step to step: the cut changes with powers of two only.  With a window a tile's
  // rows together see fewer than window + 32 keys, counted from the start of a tile of keys.
  int bound = kFoldKeys;
  while (bound < max_keys) bound *= 2;
  if (window > 0) bound = std::min(bound, round_up(window + 32 + kFoldKeys, kFoldKeys));
  const int key_tiles = bound / kFoldKeys;
  const int per_sm = static_cast<int>(std::min<size_t>(2, 227 * 1024 / (fold_shared_bytes(rank, rot, plan.groups) + 1024)));
  const long at_once = static_cast<long>(sms) * std::max(per_sm, 1);
  plan.num_splits = 1, plan.split_keys = bound;
  // (waves of blocks) x (tiles of keys in a row + what a block costs besides), the smallest
  double best = 0.0;
  for (int splits = 1; splits <= std::min(key_tiles, 64); ++splits) {
    const int each = (key_tiles + splits - 1) / splits;
    if (splits > 1 && (key_tiles + each - 1) / each != splits) continue;
    // (the splits' partial sums stay within 1,300 groups of sixteen rows, which memory is planned for)
    if (splits > 1 && static_cast<long>(plan.tiles) * splits * plan.groups > 1300) break;
    const double waves = static_cast<double>((plan.tiles * static_cast<long>(splits) + at_once - 1) / at_once);
    const double cost = waves * (each + 2.0) + (splits > 1 ? 1.0 + 0.1 * splits : 0.0);
    if (splits == 1 || cost < best) best = cost, plan.num_splits = splits, plan.split_keys = each * kFoldKeys;
  }
  return plan;
}

// {rows of a tile, groups of sixteen rows, keys per split, splits}
VIPERA_API int vipera_latent_plan(int tokens, int heads, int rank, int rot, int max_keys, int window, int single, int sms, int* plan) {
  if (tokens <= 0 || heads <= 0 || sms <= 0 || window < 0 || rank <= 0 || rot <= 0) return VIPERA_BAD_ARGUMENT;
  const FoldPlan f = latent_plan(tokens, heads, rank, rot, max_keys < 1 ? 1 : max_keys, window, single, sms);
  plan[0] = f.tile_rows;
  plan[1] = f.groups;
  plan[2] = f.split_keys;
  plan[3] = f.num_splits;
  return VIPERA_OK;
}

template <int NR, int MT>
static int launch_fold(const LatentFoldParams& f, dim3 grid, size_t shared, cudaStream_t s) {
  static bool configured = false;
  if (!configured) {
    if (cudaFuncSetAttribute(latent_fold_kernel<NR, MT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 225 * 1024) != cudaSuccess)
      return VIPERA_BAD_ARGUMENT;
    configured = true;
  }
  return vipera_launch(latent_fold_kernel<NR, MT>, grid, kFoldThreads, shared, s, f);
}

static int launch_fold_any(const LatentParams& p, cudaStream_t s) {
  LatentFoldParams f{};
  f.qa = p.qa;
  f.k_pool = static_cast<const __nv_bfloat16*>(p.k_pool);
  f.v_pool = static_cast<const __nv_bfloat16*>(p.v_pool);
  f.token_entry = p.token_entry;
  f.positions = p.positions;
  f.block_table = p.block_table;
  f.out = p.latent_out;
  f.part = p.part;
  f.num_tokens = p.num_tokens, f.heads = p.heads, f.rank = p.rank, f.rot = p.rot;
  f.table_width = p.table_width, f.page_size = p.page_size;
  f.window = p.window;
  f.sink = p.sink;
  if (p.stage == 2) {
    f.qa_heads = p.qa_heads, f.q_rot = p.q_rot, f.l_heads = static_cast<__nv_bfloat16*>(p.l_heads);
    f.padded_tokens = p.padded_tokens, f.scale = p.scale;
  }
  int device = 0, sms = 0;
  cudaGetDevice(&device);
  cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, device);
  const FoldPlan plan = latent_plan(p.num_tokens, p.heads, p.rank, p.rot, 1, p.window, p.single, sms > 0 ? sms : 148);
  const int groups = plan.groups;   // (rows and tiles do not depend on the keys)
  f.tile_rows = plan.tile_rows;
  f.num_splits = p.num_splits > 1 && p.part ? p.num_splits : 1;
  f.split_keys = f.num_splits > 1 ? p.split_keys : 0x3fffffff;
  if (f.num_splits > kMostSplits) return VIPERA_BAD_ARGUMENT;
  const int rank_pad = round_up(p.rank, 16);
  const size_t shared = fold_shared_bytes(p.rank, p.rot, groups);
  const dim3 grid(plan.tiles, f.num_splits);
  int status;
  if (groups == 2)
    status = rank_pad <= 128 ? launch_fold<128, 2>(f, grid, shared, s)
           : rank_pad <= 256 ? launch_fold<256, 2>(f, grid, shared, s) : launch_fold<512, 2>(f, grid, shared, s);
  else
    status = rank_pad <= 128 ? launch_fold<128, 1>(f, grid, shared, s)
           : rank_pad <= 256 ? launch_fold<256, 1>(f, grid, shared, s) : launch_fold<512, 1>(f, grid, shared, s);
  if (status || f.num_splits == 1) return status;
  return vipera_launch(latent_combine_kernel, p.num_tokens * p.heads, 128, 0, s, f);
}

template <typename T>
static int launch_latent(const LatentParams& p, cudaStream_t s) {
  int status = VIPERA_OK;
  if (p.stage == 2) return launch_fold_any(p, s);
  if (p.stage == 3) {
    const long long values = static_cast<long long>(p.num_tokens) * p.heads * p.dv;
    return vipera_launch(latent_gate_kernel<T>, static_cast<unsigned>((values + 255) / 256), 256, 0, s, p.o_heads, p.proj,
                         p.proj_width, p.g_off, static_cast<T*>(p.out), p.num_tokens, p.heads, p.dv, p.padded_tokens);
  }
  if (p.kv_off >= 0 || p.stage == 4) {
    const int cq_rank = p.stage == 4 ? p.q_rank : 0;
    status = vipera_launch(latent_store_kernel<T>, dim3(p.num_tokens, p.kv_off >= 0 && cq_rank > 0 ? 2 : 1), kStoreThreads, 0, s, p.proj, p.proj_width, p.kv_off, p.norm_weight,
                           p.eps, p.positions, p.cos_table, p.sin_table, static_cast<T*>(p.k_pool),
                           static_cast<T*>(p.v_pool), p.token_entry, p.block_table, p.table_width, p.page_size, p.rank,
                           p.rot, p.pairing, p.cq_off, cq_rank, p.cq_norm_weight, static_cast<T*>(p.cq));
    if (status || p.stage == 4) return status;
  }
  const float* q = p.q ? p.q : p.proj;
  const long long q_width = p.q ? p.q_width : p.proj_width;
  if (p.stage == 1)
    return vipera_launch(latent_prep_kernel, p.num_tokens, 128, 0, s, q, q_width, p.q_off, p.positions, p.cos_table,
                         p.sin_table, static_cast<__nv_bfloat16*>(p.a_heads), p.q_rot, p.tile_group, p.heads, p.d, p.rot,
                         p.padded_tokens, p.scale, p.pairing);
  const dim3 tiles((p.num_tokens + kTile - 1) / kTile, p.heads);
  const dim3 absorb_grid(tiles.x, tiles.y, (p.rank + kAbsorbCols - 1) / kAbsorbCols);
  status = vipera_launch(latent_absorb_kernel<T>, absorb_grid, kUpThreads, (kTile * p.d + 8 * kTile * kAbsorbCols) * sizeof(float), s, q, q_width, p.q_off,
                         static_cast<const T*>(p.up_k), p.positions, p.cos_table, p.sin_table, p.qa, p.num_tokens,
                         p.heads, p.d, p.rank, p.rot, p.scale, p.pairing);
  if (status) return status;
  // bfloat16 caches whose rows are whole 16-byte pieces fold on the tensor cores
  if (sizeof(T) == 2 && p.rank % 8 == 0 && p.rot % 8 == 0 && p.num_tokens < (1 << 24) / p.heads &&
      (p.num_splits <= 1 || p.split_keys % kFoldKeys == 0))
    status = launch_fold_any(p, s);
  else
    status = vipera_launch(latent_attention_kernel<T>, dim3(p.num_tokens, (p.heads + kWarps - 1) / kWarps), kWarps * 32,
                           kWarps * (p.rank + p.rot) * sizeof(float), s, p.qa, p.latent_out,
                           static_cast<const T*>(p.k_pool), static_cast<const T*>(p.v_pool), p.token_entry, p.positions,
                           p.block_table, p.table_width, p.page_size, p.heads, p.rank, p.rot, p.window, p.sink);
  if (status) return status;
  const dim3 expand_grid(tiles.x, tiles.y, (p.dv + kExpandCols - 1) / kExpandCols);
  return vipera_launch(latent_expand_kernel<T, T>, expand_grid, kUpThreads, (kTile * p.rank + 8 * kTile * kExpandCols) * sizeof(float), s, p.latent_out,
                       static_cast<const T*>(p.up_v), p.proj, p.proj_width, p.g_off, static_cast<T*>(p.out),
                       p.num_tokens, p.heads, p.dv, p.rank);
}

// dtype: the type of the cache pools, the two up matrices and `out`.
VIPERA_API int vipera_latent_attention(const LatentParams* params, int dtype, void* stream) {
  const LatentParams& p = *params;
  if (p.num_tokens <= 0) return VIPERA_OK;
  if (p.rank <= 0 || p.rank > kMaxRank || p.rot <= 0 || p.rot > kMaxRot || (p.rot & 1)) return VIPERA_BAD_SHAPE;
  if (p.heads <= 0 || p.d <= 0 || p.d > 1024 || p.dv <= 0 || p.page_size <= 0 || p.table_width <= 0) return VIPERA_BAD_SHAPE;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (p.stage < 0 || p.stage > 4 || p.window < 0 || p.pairing < 0 || p.pairing > 1) return VIPERA_BAD_ARGUMENT;
  if (p.q && p.q_width < static_cast<long long>(p.q_off) + static_cast<long long>(p.heads) * (p.d + p.rot)) return VIPERA_BAD_SHAPE;
  if (p.stage == 4) {
    if (p.q_rank < 0 || (p.q_rank > 0 && (!p.cq || !p.cq_norm_weight || p.cq_off < 0 || p.cq_off + p.q_rank > p.proj_width)))
      return VIPERA_BAD_ARGUMENT;
  } else if (p.stage != 0) {
    if (dtype != VIPERA_BF16 || p.rank % 8 || p.rot % 8 || p.d % 8 || p.padded_tokens < p.num_tokens || p.padded_tokens % 128 ||
        !p.a_heads || !p.qa_heads || !p.q_rot || !p.l_heads || !p.o_heads || !p.tile_group ||
        p.num_tokens >= (1 << 24) / p.heads || (p.num_splits > 1 && p.split_keys % kFoldKeys))
      return VIPERA_BAD_ARGUMENT;
  }
  if (dtype == VIPERA_F32) return launch_latent<float>(p, s);
  if (dtype == VIPERA_BF16) return launch_latent<__nv_bfloat16>(p, s);
  return VIPERA_BAD_DTYPE;
}

VIPERA_API int vipera_latent_params_size() { return static_cast<int>(sizeof(LatentParams)); }
VIPERA_API const char* vipera_latent_status_text(int status) { return vipera_status_text(status); }
