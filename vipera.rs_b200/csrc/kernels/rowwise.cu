// Row-wise kernels: embedding lookup into the 32-bit residual stream, and RMSNorm.
//
// Embedding: a row lookup (crates/vipera-backend-cpu/src/model.rs:956-966; the reference's
// device version dequantises one row, crates/vipera-backend-gpu/src/layer.cu:545-563).  The
// reference's model does not scale the rows; `scale` is for architectures that do, and a
// scale of exactly 1 leaves the values as they are.
// RMSNorm: out = x * rsqrt(mean(x^2) + eps) * w with 32-bit statistics
// (model.rs:4282-4288; device version layer.cu:32-58, one block per row with a tree sum).
#include "common.cuh"

// ---------------------------------------------------------------------------------------
// embedding: out[t, :] = scale * table[tokens[t], :]  (32-bit out, whatever the table's type)
// ---------------------------------------------------------------------------------------
template <typename TW>
__global__ void embed_kernel(const TW* __restrict__ table, const int* __restrict__ tokens,
                             float* __restrict__ out, float* __restrict__ also, int hidden, int vocab, float scale) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x;
  int token = tokens[t];
  // The host refuses ids outside the vocabulary before the launch; the clamp only keeps
  // a stale buffer in a replayed graph from reading outside the table.
  token = min(max(token, 0), vocab - 1);
  const TW* row = table + static_cast<size_t>(token) * hidden;
  float* dst = out + static_cast<size_t>(t) * hidden;
  float* second = also ? also + static_cast<size_t>(t) * hidden : nullptr;
  for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
    const float value = scale * to_float<TW>(row[i]);
    dst[i] = value;
    if (second) second[i] = value;
  }
}

// `also` (null: none): a second buffer that receives the same rows.
VIPERA_API int vipera_embed(const void* table, int table_dtype, const int* tokens, float* out, float* also,
                            int num_tokens, int hidden, int vocab, float scale, void* stream) {
  if (num_tokens <= 0) return VIPERA_OK;
  if (hidden <= 0 || vocab <= 0) return VIPERA_BAD_SHAPE;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const int threads = hidden >= 1024 ? 256 : 128;
  if (table_dtype == VIPERA_F32)
    return vipera_launch(embed_kernel<float>, num_tokens, threads, 0, s, static_cast<const float*>(table), tokens, out, also, hidden, vocab, scale);
  if (table_dtype == VIPERA_BF16)
    return vipera_launch(embed_kernel<__nv_bfloat16>, num_tokens, threads, 0, s, static_cast<const __nv_bfloat16*>(table), tokens, out, also, hidden, vocab, scale);
  return VIPERA_BAD_DTYPE;
}

// ---------------------------------------------------------------------------------------
// RMSNorm over rows of the 32-bit residual stream.  `rows` (optional) picks which rows of
// x are normalised: out[r, :] = norm(x[rows[r], :]).  For few rows, one block per output row;
// the row stays in registers between the two passes when it is short enough, else it is read
// twice.
// ---------------------------------------------------------------------------------------
constexpr int kNormThreads = 256;
constexpr int kNormRegs = 8;  // elements per thread kept in registers: rows up to 2048 wide

template <typename TO>
__global__ void rmsnorm_kernel(const float* __restrict__ x, const float* __restrict__ weight,
                               const int* __restrict__ rows, TO* __restrict__ out, int hidden, float eps) {
  __shared__ float scratch[32];
  pdl_launch_dependents();
  const int r = blockIdx.x;
  const bool fits = hidden <= kNormThreads * kNormRegs;
  // The norm's weights depend on no kernel ahead of this one: they are in registers before the
  // wait, so that the second pass does not pay a memory round trip for them.
  float gain[kNormRegs];
  if (fits) {
#pragma unroll
    for (int j = 0; j < kNormRegs; ++j) {
      const int i = threadIdx.x + j * kNormThreads;
      gain[j] = i < hidden ? weight[i] : 0.0f;
    }
  }
  pdl_wait();
  const int src_row = rows ? rows[r] : r;
  const float* src = x + static_cast<size_t>(src_row) * hidden;
  TO* dst = out + static_cast<size_t>(r) * hidden;
  float kept[kNormRegs];
  float sum = 0.0f;
  if (fits) {
#pragma unroll
    for (int j = 0; j < kNormRegs; ++j) {
      const int i = threadIdx.x + j * kNormThreads;
      kept[j] = i < hidden ? src[i] : 0.0f;
      sum += kept[j] * kept[j];
    }
  } else {
    for (int i = threadIdx.x; i < hidden; i += kNormThreads) {
      const float v = src[i];
      sum += v * v;
    }
  }
  const float total = block_sum(sum, scratch);
  const float inverse = 1.0f / sqrtf(total / static_cast<float>(hidden) + eps);
  if (fits) {
#pragma unroll
    for (int j = 0; j < kNormRegs; ++j) {
      const int i = threadIdx.x + j * kNormThreads;
      if (i < hidden) dst[i] = from_float<TO>(kept[j] * inverse * gain[j]);
    }
  } else {
    for (int i = threadIdx.x; i < hidden; i += kNormThreads)
      dst[i] = from_float<TO>(src[i] * inverse * weight[i]);
  }
}

// The same for many rows (prompt portions): a warp per row, the row in registers as 16-byte
// vectors, the sum by shuffles; no block-wide barrier, eight rows to a block.  VECS vectors
// of four values per lane: rows up to 128 * VECS wide, a multiple of four.
constexpr int kRowsPerBlock = 8;
constexpr int kManyRows = 128;  // from this many rows on

__device__ __forceinline__ void store_four(float* dst, float a, float b, float c, float d) {
  *reinterpret_cast<float4*>(dst) = make_float4(a, b, c, d);
}
__device__ __forceinline__ void store_four(__nv_bfloat16* dst, float a, float b, float c, float d) {
  __nv_bfloat162 lo = __floats2bfloat162_rn(a, b), hi = __floats2bfloat162_rn(c, d);
  uint2 packed;
  packed.x = *reinterpret_cast<uint32_t*>(&lo);
  packed.y = *reinterpret_cast<uint32_t*>(&hi);
  *reinterpret_cast<uint2*>(dst) = packed;
}

template <typename TO, int VECS>
__global__ void __launch_bounds__(kRowsPerBlock * 32)
rmsnorm_rows_kernel(const float* __restrict__ x, const float* __restrict__ weight, const int* __restrict__ rows,
                    TO* __restrict__ out, int num_rows, int hidden, float eps) {
  pdl_launch_dependents();
  pdl_wait();
  const int r = blockIdx.x * kRowsPerBlock + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (r >= num_rows) return;
  const int src_row = rows ? rows[r] : r;
  const float4* src = reinterpret_cast<const float4*>(x + static_cast<size_t>(src_row) * hidden);
  const float4* w = reinterpret_cast<const float4*>(weight);
  TO* dst = out + static_cast<size_t>(r) * hidden;
  const int vectors = hidden >> 2;
  float4 kept[VECS];
  float sum = 0.0f;
#pragma unroll
  for (int j = 0; j < VECS; ++j) {
    const int i = lane + j * 32;
    kept[j] = i < vectors ? src[i] : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    sum += kept[j].x * kept[j].x + kept[j].y * kept[j].y + kept[j].z * kept[j].z + kept[j].w * kept[j].w;
  }
#pragma unroll
  for (int offset = 16; offset > 0; offset >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, offset);
  const float inverse = 1.0f / sqrtf(sum / static_cast<float>(hidden) + eps);
#pragma unroll
  for (int j = 0; j < VECS; ++j) {
    const int i = lane + j * 32;
    if (i < vectors) {
      const float4 g = w[i];
      store_four(dst + 4 * i, kept[j].x * inverse * g.x, kept[j].y * inverse * g.y, kept[j].z * inverse * g.z,
                 kept[j].w * inverse * g.w);
    }
  }
}

template <typename TO>
static int launch_rmsnorm_rows(const float* x, const float* weight, const int* rows, TO* out, int num_rows, int hidden,
                               float eps, cudaStream_t s) {
  const int blocks = (num_rows + kRowsPerBlock - 1) / kRowsPerBlock;
  if (hidden <= 128 * 8)
    return vipera_launch(rmsnorm_rows_kernel<TO, 8>, blocks, kRowsPerBlock * 32, 0, s, x, weight, rows, out, num_rows, hidden, eps);
  if (hidden <= 128 * 16)
    return vipera_launch(rmsnorm_rows_kernel<TO, 16>, blocks, kRowsPerBlock * 32, 0, s, x, weight, rows, out, num_rows, hidden, eps);
  return vipera_launch(rmsnorm_rows_kernel<TO, 32>, blocks, kRowsPerBlock * 32, 0, s, x, weight, rows, out, num_rows, hidden, eps);
}

VIPERA_API int vipera_rmsnorm(const float* x, const float* weight, const int* rows, void* out,
                              int out_dtype, int num_rows, int hidden, float eps, void* stream) {
  if (num_rows <= 0) return VIPERA_OK;
  if (hidden <= 0) return VIPERA_BAD_SHAPE;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const bool aligned = ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(weight) | reinterpret_cast<uintptr_t>(out)) & 15) == 0;
  if (num_rows >= kManyRows && hidden % 4 == 0 && hidden <= 128 * 32 && aligned) {
    if (out_dtype == VIPERA_F32) return launch_rmsnorm_rows(x, weight, rows, static_cast<float*>(out), num_rows, hidden, eps, s);
    if (out_dtype == VIPERA_BF16) return launch_rmsnorm_rows(x, weight, rows, static_cast<__nv_bfloat16*>(out), num_rows, hidden, eps, s);
    return VIPERA_BAD_DTYPE;
  }
  if (out_dtype == VIPERA_F32)
    return vipera_launch(rmsnorm_kernel<float>, num_rows, kNormThreads, 0, s, x, weight, rows, static_cast<float*>(out), hidden, eps);
  if (out_dtype == VIPERA_BF16)
    return vipera_launch(rmsnorm_kernel<__nv_bfloat16>, num_rows, kNormThreads, 0, s, x, weight, rows, static_cast<__nv_bfloat16*>(out), hidden, eps);
  return VIPERA_BAD_DTYPE;
}

// ---------------------------------------------------------------------------------------
// Layer norm over rows of a 32-bit stream: (x - mean) / sqrt(var + eps) * w + b, the variance
// being the mean of the squared deviations (two passes over the row, which stays in registers
// when it is short enough).  `rows` picks the rows as in RMSNorm.  ACC: the output is 32-bit
// and the result is added to what it holds (a sublayer's normalised output joining the
// residual stream).  A block per row.
// ---------------------------------------------------------------------------------------
template <typename TO, bool ACC>
__global__ void __launch_bounds__(kNormThreads)
layernorm_kernel(const float* __restrict__ x, const float* __restrict__ weight, const float* __restrict__ bias,
                 const int* __restrict__ rows, TO* __restrict__ out, int hidden, float eps) {
  __shared__ float scratch[32];
  pdl_launch_dependents();
  const int r = blockIdx.x;
  const bool fits = hidden <= kNormThreads * kNormRegs;
  float gain[kNormRegs], shift[kNormRegs];
  if (fits) {
#pragma unroll
    for (int j = 0; j < kNormRegs; ++j) {
      const int i = threadIdx.x + j * kNormThreads;
      gain[j] = i < hidden ? weight[i] : 0.0f;
      shift[j] = i < hidden ? bias[i] : 0.0f;
    }
  }
  pdl_wait();
  const int src_row = rows ? rows[r] : r;
  const float* src = x + static_cast<size_t>(src_row) * hidden;
  TO* dst = out + static_cast<size_t>(r) * hidden;
  float kept[kNormRegs];
  float sum = 0.0f;
  if (fits) {
#pragma unroll
    for (int j = 0; j < kNormRegs; ++j) {
      const int i = threadIdx.x + j * kNormThreads;
      kept[j] = i < hidden ? src[i] : 0.0f;
      sum += kept[j];
    }
  } else {
    for (int i = threadIdx.x; i < hidden; i += kNormThreads) sum += src[i];
  }
  const float mean = block_sum(sum, scratch) / static_cast<float>(hidden);
  float squares = 0.0f;
  if (fits) {
#pragma unroll
    for (int j = 0; j < kNormRegs; ++j) {
      const int i = threadIdx.x + j * kNormThreads;
      const float d = i < hidden ? kept[j] - mean : 0.0f;
      squares += d * d;
    }
  } else {
    for (int i = threadIdx.x; i < hidden; i += kNormThreads) {
      const float d = src[i] - mean;
      squares += d * d;
    }
  }
  const float inverse = 1.0f / sqrtf(block_sum(squares, scratch) / static_cast<float>(hidden) + eps);
  if (fits) {
#pragma unroll
    for (int j = 0; j < kNormRegs; ++j) {
      const int i = threadIdx.x + j * kNormThreads;
      if (i < hidden) {
        const float v = (kept[j] - mean) * inverse * gain[j] + shift[j];
        if (ACC) dst[i] = from_float<TO>(to_float<TO>(dst[i]) + v);
        else dst[i] = from_float<TO>(v);
      }
    }
  } else {
    for (int i = threadIdx.x; i < hidden; i += kNormThreads) {
      const float v = (src[i] - mean) * inverse * weight[i] + bias[i];
      if (ACC) dst[i] = from_float<TO>(to_float<TO>(dst[i]) + v);
      else dst[i] = from_float<TO>(v);
    }
  }
}

// accumulate != 0: out is 32-bit and receives out + norm(x).
VIPERA_API int vipera_layernorm(const float* x, const float* weight, const float* bias, const int* rows, void* out,
                                int out_dtype, int num_rows, int hidden, float eps, int accumulate, void* stream) {
  if (num_rows <= 0) return VIPERA_OK;
  if (hidden <= 0) return VIPERA_BAD_SHAPE;
  if (!weight || !bias) return VIPERA_BAD_ARGUMENT;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (accumulate) {
    if (out_dtype != VIPERA_F32) return VIPERA_BAD_DTYPE;
    return vipera_launch(layernorm_kernel<float, true>, num_rows, kNormThreads, 0, s, x, weight, bias, rows,
                         static_cast<float*>(out), hidden, eps);
  }
  if (out_dtype == VIPERA_F32)
    return vipera_launch(layernorm_kernel<float, false>, num_rows, kNormThreads, 0, s, x, weight, bias, rows,
                         static_cast<float*>(out), hidden, eps);
  if (out_dtype == VIPERA_BF16)
    return vipera_launch(layernorm_kernel<__nv_bfloat16, false>, num_rows, kNormThreads, 0, s, x, weight, bias, rows,
                         static_cast<__nv_bfloat16*>(out), hidden, eps);
  return VIPERA_BAD_DTYPE;
}

VIPERA_API const char* vipera_rowwise_status_text(int status) { return vipera_status_text(status); }

// ---------------------------------------------------------------------------------------
// Branches computed from one and the same stream join it, and the norms that read the result next
// follow in the same pass over the row:
//   x += scale_a * (sum of a's parts) + scale_b * (sum of b's parts)
//   out1 = norm1(x), out2 = norm2(x)                      (RMS norms, 32-bit statistics)
// A branch is [rows, parts, hidden] (its parts added in their order), its scale one number per
// channel or null; either branch and either norm may be missing.  With `rows` the kernel computes
// norms of the rows named there and leaves x as it is.  A block per row; VEC values to an access; the
// row stays in registers between its passes where it is short enough.
// A second form (join_normed_kernel) takes up to four branches, of which the first two may be divided
// by the root mean square of their own row before they join (`normed`, `eps`; the norm's weight is in
// `scale`):   x += scale_0 * b_0 / rms(b_0) + scale_1 * b_1 / rms(b_1) + scale_2 * b_2 + scale_3 * b_3
// ---------------------------------------------------------------------------------------
struct JoinBranch {
  const float* values;   // null: no such branch
  const float* scale;    // [hidden] or null: 1
  int parts;
  int normed;            // 1: the branch's row is divided by sqrt(mean of its squares + eps)
  float eps;
};
struct JoinNorm {
  const float* gain;     // null: no such norm
  void* out;             // [rows, hidden]
  float eps;
};
struct JoinParams {
  float* x;
  const int* rows;
  JoinBranch branch[4];
  JoinNorm norm[2];
  int num_rows, hidden, out_dtype;
};

template <int VEC>
struct JoinVector { float v[VEC]; };

template <int VEC>
__device__ __forceinline__ JoinVector<VEC> join_load(const float* src) {
  JoinVector<VEC> r;
  if constexpr (VEC == 4) {
    const float4 q = *reinterpret_cast<const float4*>(src);
    r.v[0] = q.x, r.v[1] = q.y, r.v[2] = q.z, r.v[3] = q.w;
  } else {
    r.v[0] = *src;
  }
  return r;
}

template <typename TO, int VEC>
__device__ __forceinline__ void join_store(TO* dst, const JoinVector<VEC>& a) {
  if constexpr (VEC == 4) store_four(dst, a.v[0], a.v[1], a.v[2], a.v[3]);
  else *dst = from_float<TO>(a.v[0]);
}

// The branch's share of values i .. i + VEC - 1 of a row, added to `to`.
template <int VEC>
__device__ __forceinline__ void join_add(JoinVector<VEC>& to, const JoinBranch& b, size_t row, int hidden, int i) {
  if (!b.values) return;
  const float* src = b.values + row * b.parts * hidden + i;
  JoinVector<VEC> sum = join_load<VEC>(src);
#pragma unroll 4
  for (int p = 1; p < b.parts; ++p) {
    const JoinVector<VEC> more = join_load<VEC>(src + static_cast<size_t>(p) * hidden);
#pragma unroll
    for (int e = 0; e < VEC; ++e) sum.v[e] += more.v[e];
  }
  if (b.scale) {
    const JoinVector<VEC> s = join_load<VEC>(b.scale + i);
#pragma unroll
    for (int e = 0; e < VEC; ++e) to.v[e] = fmaf(s.v[e], sum.v[e], to.v[e]);
  } else {
#pragma unroll
    for (int e = 0; e < VEC; ++e) to.v[e] += sum.v[e];
  }
}

template <typename TO, int VEC>
__global__ void __launch_bounds__(kNormThreads)
join_norms_kernel(const JoinParams p) {
  __shared__ float scratch[32];
  constexpr int kKept = VEC == 4 ? 4 : 8;   // vectors a thread keeps: rows up to 4096 (2048) wide
  pdl_launch_dependents();
  const int r = blockIdx.x;
  const int first = threadIdx.x * VEC, step = kNormThreads * VEC;
  const bool fits = p.hidden <= kKept * step;
  pdl_wait();
  const size_t row = p.rows ? p.rows[r] : r;
  float* x = p.x + row * p.hidden;
  JoinVector<VEC> kept[kKept];
  float squares = 0.0f;
  auto joined = [&](int i) {
    JoinVector<VEC> v = join_load<VEC>(x + i);
    join_add<VEC>(v, p.branch[0], row, p.hidden, i);
    join_add<VEC>(v, p.branch[1], row, p.hidden, i);
#pragma unroll
    for (int e = 0; e < VEC; ++e) squares = fmaf(v.v[e], v.v[e], squares);
    return v;
  };
  const bool writes = p.rows == nullptr && (p.branch[0].values || p.branch[1].values);
  if (fits) {
#pragma unroll
    for (int j = 0; j < kKept; ++j) {
      const int i = first + j * step;
      if (i < p.hidden) {
        kept[j] = joined(i);
        if (writes) join_store<float, VEC>(x + i, kept[j]);
      }
    }
  } else {
    for (int i = first; i < p.hidden; i += step) {
      const JoinVector<VEC> v = joined(i);
      if (writes) join_store<float, VEC>(x + i, v);
    }
  }
  if (!p.norm[0].gain && !p.norm[1].gain) return;
  const float mean = block_sum(squares, scratch) / static_cast<float>(p.hidden);
#pragma unroll
  for (int n = 0; n < 2; ++n) {
    const JoinNorm& norm = p.norm[n];
    if (!norm.gain) continue;
    const float inverse = 1.0f / sqrtf(mean + norm.eps);
    TO* out = static_cast<TO*>(norm.out) + static_cast<size_t>(r) * p.hidden;
    auto finish = [&](JoinVector<VEC> v, int i) {
      const JoinVector<VEC> g = join_load<VEC>(norm.gain + i);
#pragma unroll
      for (int e = 0; e < VEC; ++e) v.v[e] = v.v[e] * inverse * g.v[e];
      join_store<TO, VEC>(out + i, v);
    };
    if (fits) {
#pragma unroll
      for (int j = 0; j < kKept; ++j) {
        const int i = first + j * step;
        if (i < p.hidden) finish(kept[j], i);
      }
    } else {
      // a thread reads back what it wrote itself; with `rows` nothing was written and the sum is formed again
      for (int i = first; i < p.hidden; i += step) finish(writes || (!p.branch[0].values && !p.branch[1].values) ? join_load<VEC>(x + i) : joined(i), i);
    }
  }
}

// The sum of a branch's parts for values i .. i + VEC - 1 of a row.
template <int VEC>
__device__ __forceinline__ JoinVector<VEC> join_parts(const JoinBranch& b, size_t row, int hidden, int i) {
  JoinVector<VEC> sum;
#pragma unroll
  for (int e = 0; e < VEC; ++e) sum.v[e] = 0.0f;
  if (!b.values) return sum;
  const float* src = b.values + row * b.parts * hidden + i;
  sum = join_load<VEC>(src);
  for (int part = 1; part < b.parts; ++part) {
    const JoinVector<VEC> more = join_load<VEC>(src + static_cast<size_t>(part) * hidden);
#pragma unroll
    for (int e = 0; e < VEC; ++e) sum.v[e] += more.v[e];
  }
  return sum;
}

// Both sums over the block of kNormThreads threads, in one exchange.
__device__ __forceinline__ float2 block_sum_pair(float a, float b, float2* scratch) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  a = warp_sum(a), b = warp_sum(b);
  if (lane == 0) scratch[warp] = make_float2(a, b);
  __syncthreads();
  const float2 mine = lane < kNormThreads / 32 ? scratch[lane] : make_float2(0.0f, 0.0f);
  return make_float2(warp_sum(mine.x), warp_sum(mine.y));
}

template <typename TO, int VEC>
__global__ void __launch_bounds__(kNormThreads)
join_normed_kernel(const JoinParams p) {
  __shared__ float scratch[32];
  __shared__ float2 pairs[kNormThreads / 32];
  constexpr int kKept = VEC == 4 ? 4 : 8;
  pdl_launch_dependents();
  const int r = blockIdx.x;
  const int first = threadIdx.x * VEC, step = kNormThreads * VEC;
  const bool fits = p.hidden <= kKept * step;
  pdl_wait();
  const size_t row = p.rows ? p.rows[r] : r;
  float* x = p.x + row * p.hidden;
  const bool writes = p.rows == nullptr;
  JoinVector<VEC> kept[kKept], own0[kKept], own1[kKept];
  float squares0 = 0.0f, squares1 = 0.0f;
  auto square = [](float& sum, const JoinVector<VEC>& v) {
#pragma unroll
    for (int e = 0; e < VEC; ++e) sum = fmaf(v.v[e], v.v[e], sum);
  };
  if (fits) {
    // the row of the stream with the plain branches, and the two branches that may be normed: all asked for together
#pragma unroll
    for (int j = 0; j < kKept; ++j) {
      const int i = first + j * step;
      if (i < p.hidden) {
        own0[j] = join_parts<VEC>(p.branch[0], row, p.hidden, i);
        own1[j] = join_parts<VEC>(p.branch[1], row, p.hidden, i);
        kept[j] = join_load<VEC>(x + i);
        join_add<VEC>(kept[j], p.branch[2], row, p.hidden, i);
        join_add<VEC>(kept[j], p.branch[3], row, p.hidden, i);
        square(squares0, own0[j]);
        square(squares1, own1[j]);
      }
    }
  } else {
    for (int i = first; i < p.hidden; i += step) {
      square(squares0, join_parts<VEC>(p.branch[0], row, p.hidden, i));
      square(squares1, join_parts<VEC>(p.branch[1], row, p.hidden, i));
    }
  }
  const float2 sums = block_sum_pair(squares0, squares1, pairs);
  const float width = static_cast<float>(p.hidden);
  const float inverse0 = p.branch[0].normed ? 1.0f / sqrtf(sums.x / width + p.branch[0].eps) : 1.0f;
  const float inverse1 = p.branch[1].normed ? 1.0f / sqrtf(sums.y / width + p.branch[1].eps) : 1.0f;
  auto add_scaled = [&](JoinVector<VEC>& to, const JoinVector<VEC>& own, const JoinBranch& b, float inverse, int i) {
    if (!b.values) return;
    JoinVector<VEC> s;
#pragma unroll
    for (int e = 0; e < VEC; ++e) s.v[e] = 1.0f;
    if (b.scale) s = join_load<VEC>(b.scale + i);
#pragma unroll
    for (int e = 0; e < VEC; ++e) to.v[e] = fmaf(s.v[e], own.v[e] * inverse, to.v[e]);
  };
  float squares = 0.0f;
  auto joined = [&](int i) {   // rows too long for the registers
    JoinVector<VEC> v = join_load<VEC>(x + i);
    join_add<VEC>(v, p.branch[2], row, p.hidden, i);
    join_add<VEC>(v, p.branch[3], row, p.hidden, i);
    add_scaled(v, join_parts<VEC>(p.branch[0], row, p.hidden, i), p.branch[0], inverse0, i);
    add_scaled(v, join_parts<VEC>(p.branch[1], row, p.hidden, i), p.branch[1], inverse1, i);
    return v;
  };
  if (fits) {
#pragma unroll
    for (int j = 0; j < kKept; ++j) {
      const int i = first + j * step;
      if (i < p.hidden) {
        add_scaled(kept[j], own0[j], p.branch[0], inverse0, i);
        add_scaled(kept[j], own1[j], p.branch[1], inverse1, i);
        square(squares, kept[j]);
        if (writes) join_store<float, VEC>(x + i, kept[j]);
      }
    }
  } else {
    for (int i = first; i < p.hidden; i += step) {
      const JoinVector<VEC> v = joined(i);
      square(squares, v);
      if (writes) join_store<float, VEC>(x + i, v);
    }
  }
  if (!p.norm[0].gain && !p.norm[1].gain) return;
  const float mean = block_sum(squares, scratch) / width;
#pragma unroll
  for (int n = 0; n < 2; ++n) {
    const JoinNorm& norm = p.norm[n];
    if (!norm.gain) continue;
    const float inverse = 1.0f / sqrtf(mean + norm.eps);
    TO* out = static_cast<TO*>(norm.out) + static_cast<size_t>(r) * p.hidden;
    auto finish = [&](JoinVector<VEC> v, int i) {
      const JoinVector<VEC> g = join_load<VEC>(norm.gain + i);
#pragma unroll
      for (int e = 0; e < VEC; ++e) v.v[e] = v.v[e] * inverse * g.v[e];
      join_store<TO, VEC>(out + i, v);
    };
    if (fits) {
#pragma unroll
      for (int j = 0; j < kKept; ++j) {
        const int i = first + j * step;
        if (i < p.hidden) finish(kept[j], i);
      }
    } else {
      for (int i = first; i < p.hidden; i += step) finish(writes ? join_load<VEC>(x + i) : joined(i), i);
    }
  }
}

template <typename TO>
static int launch_join(const JoinParams& p, bool vectors, cudaStream_t s) {
  if (p.branch[2].values || p.branch[3].values || p.branch[0].normed || p.branch[1].normed) {
    if (vectors) return vipera_launch(join_normed_kernel<TO, 4>, p.num_rows, kNormThreads, 0, s, p);
    return vipera_launch(join_normed_kernel<TO, 1>, p.num_rows, kNormThreads, 0, s, p);
  }
  if (vectors) return vipera_launch(join_norms_kernel<TO, 4>, p.num_rows, kNormThreads, 0, s, p);
  return vipera_launch(join_norms_kernel<TO, 1>, p.num_rows, kNormThreads, 0, s, p);
}

// out_dtype: the type of both norms' outputs.
VIPERA_API int vipera_join_norms(const JoinParams* params, void* stream) {
  const JoinParams& p = *params;
  if (p.num_rows <= 0) return VIPERA_OK;
  if (p.hidden <= 0 || !p.x) return VIPERA_BAD_SHAPE;
  uintptr_t bases = reinterpret_cast<uintptr_t>(p.x);
  for (int i = 0; i < 4; ++i) {
    if (p.branch[i].values && p.branch[i].parts <= 0) return VIPERA_BAD_ARGUMENT;
    if (p.branch[i].normed && (i > 1 || !p.branch[i].values)) return VIPERA_BAD_ARGUMENT;
    bases |= reinterpret_cast<uintptr_t>(p.branch[i].values) | reinterpret_cast<uintptr_t>(p.branch[i].scale);
  }
  for (int i = 0; i < 2; ++i) {
    if (p.norm[i].gain && !p.norm[i].out) return VIPERA_BAD_ARGUMENT;
    bases |= reinterpret_cast<uintptr_t>(p.norm[i].gain) | reinterpret_cast<uintptr_t>(p.norm[i].out);
  }
  const bool vectors = p.hidden % 4 == 0 && (bases & 15) == 0;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (p.out_dtype == VIPERA_F32) return launch_join<float>(p, vectors, s);
  if (p.out_dtype == VIPERA_BF16) return launch_join<__nv_bfloat16>(p, vectors, s);
  return VIPERA_BAD_DTYPE;
}

VIPERA_API int vipera_join_params_size() { return static_cast<int>(sizeof(JoinParams)); }
