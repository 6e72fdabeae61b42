// Mamba-2's recurrence (state-space duality): one decay per head and token.
//
// Per head h (of group g = h / (heads / groups)) a matrix S [state, vdim] of 32-bit floats, zero at a
// request's start.  With dt_t = softplus(raw_t + bias_h) and a_h = -exp(A_log_h), for each token
//
//     S = exp(a_h dt_t) S + dt_t b_t x_t^T        y_t = S^T c_t + D_h x_t
//
// (b_t, c_t [state] of the group, x_t [vdim] of the head).  A finishing kernel multiplies the heads'
// concatenated y by silu(z), divides each of `norm_groups` equal parts by its own root mean square and
// multiplies by a weight per value.  x, b and c come from the caller's convolution in the run's type, raw
// and z from its projection in 32-bit.
//
// Two forms.
//   walk     (32-bit runs, short steps, single tokens) a block owns up to 64 value columns of a head's
//            state for one entry, a thread four columns of some rows in registers, and walks the entry's
//            tokens; 32-bit arithmetic throughout.  For single tokens it is one pass over the state.
//   chunks   (long steps in bfloat16) chunks of 128 tokens of an entry, all of a step's side by side.
//            With l_t = a_h sum_{s <= t} dt_s over the chunk's tokens (at most 0),
//
//     y_t = exp(l_t) S_0^T c_t + sum_{s <= t} exp(l_t - l_s) dt_s (c_t . b_s) x_s + D_h x_t
//     S_L = exp(l_L) S_0 + sum_s exp(l_L - l_s) dt_s b_s x_s^T
//
//            mamba2_parts_kernel leaves each chunk's own sum, mamba2_carry_kernel walks each entry's chunks
//            (leaving the state at every chunk's start and the request's new state), mamba2_outputs_kernel
//            computes y.  The products are mma.sync m16n8k16 with 32-bit accumulators.  b, c and x are
//            bfloat16 as they come; what the recurrence forms in 32-bit on the way (the weights of a chunk,
//            dt_s exp(l_L - l_s) x_s, the state read by the outputs) enters its product as two bfloat16
//            halves, value = high + low, two products instead of one, so that it keeps 16 bits of its
//            significand; decays, step sizes, accumulators and the state itself are 32-bit.
//            The scores c_t . b_s belong to a group: a block computes them once for several heads of it.
// Chunks start where an entry's tokens start in the step, so another cut of a prompt only re-associates
// sums.  Entries of one token walk, also beside chunks.
#include "common.cuh"

constexpr int kChunk = 128;          // tokens of a chunk
constexpr int kThreads = 256;
constexpr int kCols = 64;            // value columns of a block
constexpr int kRowGroups = 16;       // walk: row r of the state belongs to the threads of group r % 16
constexpr int kStage = 16;           // walk: tokens staged at a time
constexpr int kMaxState = 256;

struct Mamba2Params {
  const void* xbc;          // [tokens, xbc_width]: x heads * vdim | b groups * state | c groups * state, the run's type
  long long xbc_width;
  const float* proj;        // [tokens, proj_width] 32-bit: z at z_off, the raw step sizes at dt_off
  long long proj_width;
  int z_off, dt_off;
  const float* dt_bias;     // [heads]
  const float* a;           // [heads] -exp(A_log)
  const float* d;           // [heads]
  float* state;             // [slots, heads * state * vdim]
  const int* entry_starts;  // [entries + 1]
  const int* state_slots;   // [entries]
  const int* fresh;         // [entries]
  float* y;                 // [tokens, heads * vdim] before gate and norm
  const float* norm_weight; // [heads * vdim]
  void* out;                // [tokens, heads * vdim] the run's type
  float* chunk_state;       // [jobs, heads, state, vdim] a chunk's own sum   (chunks only)
  void* chunk_start;        // [jobs, heads, 2, state, vdim] bfloat16: high, then low halves of the state at a chunk's start
  float* chunk_decay;       // [jobs, heads] l_L / ln 2
  int heads, vdim, groups, states, norm_groups, num_entries, num_tokens, num_jobs;
  int heads_per_block;      // chunks: heads of one group a block works on
  int single_only;          // walk: entries of other than one token are left out
  float eps;
};

__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z))); }

__device__ __forceinline__ float dt_of(const Mamba2Params& p, int token, int h) {
  return softplus(p.proj[static_cast<size_t>(token) * p.proj_width + p.dt_off + h] + p.dt_bias[h]);
}

// ---------------------------------------------------------------------------------------
// walk.  grid: (column tiles, heads, entries).  Thread (rg, cg): rows rg, rg + 16, ...; columns 4 cg ..
// 4 cg + 3 of the tile (VEC) or cg, cg + 16, cg + 32, cg + 48 (a value size that is no multiple of four).
// ---------------------------------------------------------------------------------------
template <typename T, int ROWS, bool VEC>
__global__ void __launch_bounds__(kThreads)
mamba2_walk_kernel(const Mamba2Params p) {
  extern __shared__ __align__(16) float walk_shared[];
  float* b_s = walk_shared;                         // [kStage][states]
  float* c_s = b_s + kStage * p.states;             // [kStage][states]
  float* x_s = c_s + kStage * p.states;             // [kStage][kCols]
  float* part = x_s + kStage * kCols;               // [2][8 warps][kCols]
  __shared__ float dt_s[kStage], decay_s[kStage];
  pdl_launch_dependents();
  const int entry = blockIdx.z, h = blockIdx.y, col0 = blockIdx.x * kCols;
  const int begin = p.entry_starts[entry], end = p.entry_starts[entry + 1];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int cg = threadIdx.x & 15, rg = threadIdx.x >> 4;
  const float a = p.a[h], skip = p.d[h];
  const bool fresh = p.fresh[entry] != 0;
  const size_t head_size = static_cast<size_t>(p.states) * p.vdim;
  float* own = p.state + (static_cast<size_t>(p.state_slots[entry]) * p.heads + h) * head_size;
  if (!fresh) {
    // the state is on its way to L2 while the kernel ahead still runs (a hint: nothing is read yet)
    for (int i = threadIdx.x; i < p.states * 2; i += kThreads) {
      const int c = col0 + (i & 1) * 32;
      if (c < p.vdim) asm volatile("prefetch.global.L2 [%0];" ::"l"(own + static_cast<size_t>(i >> 1) * p.vdim + c));
    }
  }
  pdl_wait();
  if (end <= begin || (p.single_only && end - begin != 1)) return;
  int cols[4];
#pragma unroll
  for (int j = 0; j < 4; ++j) cols[j] = col0 + (VEC ? 4 * cg + j : cg + 16 * j);
  float s[ROWS][4];
#pragma unroll
  for (int r = 0; r < ROWS; ++r) {
    const int n = rg + kRowGroups * r;
#pragma unroll
    for (int j = 0; j < 4; ++j) s[r][j] = 0.0f;
    if (!fresh && n < p.states) {
      const float* row = own + static_cast<size_t>(n) * p.vdim;
      if (VEC) {
        if (cols[0] < p.vdim) {
          const float4 v = *reinterpret_cast<const float4*>(row + cols[0]);
          s[r][0] = v.x, s[r][1] = v.y, s[r][2] = v.z, s[r][3] = v.w;
        }
      } else {
#pragma unroll
        for (int j = 0; j < 4; ++j)
          if (cols[j] < p.vdim) s[r][j] = row[cols[j]];
      }
    }
  }
  const T* xbc = static_cast<const T*>(p.xbc);
  const int group = h / (p.heads / p.groups);
  const size_t b_off = static_cast<size_t>(p.heads) * p.vdim + static_cast<size_t>(group) * p.states;
  const size_t c_off = b_off + static_cast<size_t>(p.groups) * p.states;
  for (int base = begin; base < end; base += kStage) {
    const int count = min(kStage, end - base);
    __syncthreads();
    for (int i = threadIdx.x; i < count * p.states; i += kThreads) {
      const int tt = i / p.states, n = i % p.states;
      const T* row = xbc + static_cast<size_t>(base + tt) * p.xbc_width;
      b_s[i] = to_float<T>(row[b_off + n]);
      c_s[i] = to_float<T>(row[c_off + n]);
    }
    for (int i = threadIdx.x; i < count * kCols; i += kThreads) {
      const int tt = i / kCols, c = col0 + i % kCols;
      x_s[i] = c < p.vdim ? to_float<T>(xbc[static_cast<size_t>(base + tt) * p.xbc_width + static_cast<size_t>(h) * p.vdim + c]) : 0.0f;
    }
    if (threadIdx.x < count) {
      const float dt = dt_of(p, base + threadIdx.x, h);
      dt_s[threadIdx.x] = dt;
      decay_s[threadIdx.x] = expf(a * dt);
    }
    __syncthreads();
    for (int tt = 0; tt < count; ++tt) {
      const float decay = decay_s[tt], dt = dt_s[tt];
      float x[4], y[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        x[j] = dt * x_s[tt * kCols + (VEC ? 4 * cg + j : cg + 16 * j)];
        y[j] = 0.0f;
      }
#pragma unroll
      for (int r = 0; r < ROWS; ++r) {
        const int n = rg + kRowGroups * r;
        if (n < p.states) {
          const float b = b_s[tt * p.states + n], c = c_s[tt * p.states + n];
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            s[r][j] = fmaf(decay, s[r][j], b * x[j]);
            y[j] = fmaf(s[r][j], c, y[j]);
          }
        }
      }
      // the warp's two row groups, then the eight warps in order
      float* sums = part + (tt & 1) * 8 * kCols;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        y[j] += __shfl_xor_sync(0xffffffffu, y[j], 16);
        if (lane < 16) sums[warp * kCols + (VEC ? 4 * cg + j : cg + 16 * j)] = y[j];
      }
      __syncthreads();
      if (threadIdx.x < kCols && col0 + threadIdx.x < p.vdim) {
        float total = skip * x_s[tt * kCols + threadIdx.x];
#pragma unroll
        for (int w = 0; w < 8; ++w) total += sums[w * kCols + threadIdx.x];
        p.y[static_cast<size_t>(base + tt) * (static_cast<size_t>(p.heads) * p.vdim) + static_cast<size_t>(h) * p.vdim + col0 + threadIdx.x] = total;
      }
    }
  }
#pragma unroll
  for (int r = 0; r < ROWS; ++r) {
    const int n = rg + kRowGroups * r;
    if (n < p.states) {
      float* row = own + static_cast<size_t>(n) * p.vdim;
      if (VEC) {
        if (cols[0] < p.vdim) *reinterpret_cast<float4*>(row + cols[0]) = make_float4(s[r][0], s[r][1], s[r][2], s[r][3]);
      } else {
#pragma unroll
        for (int j = 0; j < 4; ++j)
          if (cols[j] < p.vdim) row[cols[j]] = s[r][j];
      }
    }
  }
}

// ---------------------------------------------------------------------------------------
// chunks
// ---------------------------------------------------------------------------------------
__device__ __forceinline__ int chunks_of(int count) { return count > 1 ? (count + kChunk - 1) / kChunk : 0; }

// The chunk a job index names: (entry, first token, one past the last), or entry -1 past the last chunk.
// Called by a whole warp: a lane looks at every 32nd entry.
__device__ __forceinline__ void find_chunk(const int* __restrict__ entry_starts, int num_entries, int job, int* info) {
  const int lane = threadIdx.x & 31;
  int base = 0;
  if (lane == 0) info[0] = -1;
  __syncwarp();
  for (int e0 = 0; e0 < num_entries; e0 += 32) {
    const int e = e0 + lane;
    const int start = e < num_entries ? entry_starts[e] : 0, stop = e < num_entries ? entry_starts[e + 1] : 0;
    const int own = e < num_entries ? chunks_of(stop - start) : 0;
    int upto = own;
#pragma unroll
    for (int offset = 1; offset < 32; offset <<= 1) {
      const int other = __shfl_up_sync(0xffffffffu, upto, offset);
      if (lane >= offset) upto += other;
    }
    const int before = base + upto - own;
    if (job >= before && job < before + own) {
      info[0] = e;
      info[1] = start + (job - before) * kChunk;
      info[2] = min(info[1] + kChunk, stop);
    }
    base += __shfl_sync(0xffffffffu, upto, 31);
  }
  __syncwarp();
}

// Step sizes and running sums of log decays of a chunk's tokens (a warp; four tokens a lane).
// dt[t] and l[t] = a (dt[0] + .. + dt[t]) / ln 2; tokens past the chunk's end have dt = 0.
__device__ __forceinline__ void chunk_decays(const Mamba2Params& p, int begin, int len, int h, float* dt, float* l) {
  const int lane = threadIdx.x & 31;
  float own[4], sum = 0.0f;
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const int t = 4 * lane + j;
    own[j] = t < len ? dt_of(p, begin + t, h) : 0.0f;
  }
#pragma unroll
  for (int j = 0; j < 4; ++j) sum += own[j];
  float upto = sum;
#pragma unroll
  for (int offset = 1; offset < 32; offset <<= 1) {
    const float other = __shfl_up_sync(0xffffffffu, upto, offset);
    if (lane >= offset) upto += other;
  }
  float running = upto - sum;
  const float a = p.a[h] * 1.4426950408889634f;
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    running += own[j];
    dt[4 * lane + j] = own[j];
    l[4 * lane + j] = a * running;
  }
}

__device__ __forceinline__ uint32_t shared_address(const void* at) { return static_cast<uint32_t>(__cvta_generic_to_shared(at)); }
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], const __nv_bfloat16* at) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(shared_address(at)) : "memory");
}
__device__ __forceinline__ void ldsm4_trans(uint32_t (&r)[4], const __nv_bfloat16* at) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(shared_address(at)) : "memory");
}
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// Two 32-bit values as high and low bfloat16 pairs: value = high + low to 16 bits.
__device__ __forceinline__ void split_pair(float u, float v, uint32_t& high, uint32_t& low) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(u, v);
  const float2 back = __bfloat1622float2(h);
  const __nv_bfloat162 r = __floats2bfloat162_rn(u - back.x, v - back.y);
  high = *reinterpret_cast<const uint32_t*>(&h);
  low = *reinterpret_cast<const uint32_t*>(&r);
}

// 16 bytes from global to shared memory without a register in between, or 16 zero bytes.
__device__ __forceinline__ void copy_16(void* dst, const void* src, bool live) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(shared_address(dst)), "l"(src), "r"(live ? 16 : 0) : "memory");
}
__device__ __forceinline__ void copies_wait() {
  asm volatile("cp.async.commit_group;\ncp.async.wait_group 0;" ::: "memory");
}

// Rows of bfloat16 from global memory into shared memory rows of `stride` values: `width` values of `rows`
// rows, zeros up to `padded` values and `total` rows.  `vectors`: every row starts on 16 bytes and width is
// a multiple of eight; the copies are then on their way until copies_wait().
__device__ __forceinline__ void load_rows(__nv_bfloat16* dst, int stride, const __nv_bfloat16* src, long long src_stride, int rows,
                                          int total, int width, int padded, bool vectors) {
  if (vectors) {
    const int pieces = padded / 8;
    for (int i = threadIdx.x; i < total * pieces; i += kThreads) {
      const int r = i / pieces, c = (i % pieces) * 8;
      const bool live = r < rows && c < width;
      copy_16(dst + r * stride + c, live ? src + r * src_stride + c : src, live);
    }
  } else {
    for (int i = threadIdx.x; i < total * padded; i += kThreads) {
      const int r = i / padded, c = i % padded;
      dst[r * stride + c] = (r < rows && c < width) ? src[r * src_stride + c] : __float2bfloat16_rn(0.0f);
    }
  }
}

__device__ __forceinline__ bool rows_on_16_bytes(const Mamba2Params& p, size_t offset, int width) {
  return (reinterpret_cast<uintptr_t>(p.xbc) & 15) == 0 && p.xbc_width % 8 == 0 && offset % 8 == 0 && width % 8 == 0;
}

constexpr int kXStride = kCols + 8;   // shared memory rows of value columns: no bank is met twice by eight rows

__host__ __device__ static inline int padded_states(int states) { return (states + 15) / 16 * 16; }
static inline size_t parts_shared(int states) {
  return static_cast<size_t>(kChunk) * (padded_states(states) + 8) * 2 + 2 * static_cast<size_t>(kChunk) * kXStride * 2;
}
static inline size_t outputs_shared(int states) {
  const size_t np = padded_states(states);
  const size_t b_rows = static_cast<size_t>(kChunk) * (np + 8) * 2;           // b, or the state's halves behind it
  const size_t halves = 2 * np * kXStride * 2;
  return b_rows + (b_rows > halves ? b_rows : halves) + static_cast<size_t>(kChunk) * kXStride * 2;
}

// grid: (jobs, heads / heads_per_block, column tiles).  A chunk's own sum for several heads of a group:
// E[n, c] = sum_s b_s[n] (w_s x_s[c]),  w_s = exp(l_L - l_s) dt_s.
__global__ void __launch_bounds__(kThreads)
mamba2_parts_kernel(const Mamba2Params p) {
  extern __shared__ __align__(16) unsigned char raw[];
  __shared__ int info[3];
  __shared__ float dt_s[kChunk], l_s[kChunk];
  pdl_launch_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (warp == 0) find_chunk(p.entry_starts, p.num_entries, blockIdx.x, info);
  pdl_wait();
  __syncthreads();
  if (info[0] < 0) return;
  const int begin = info[1], len = info[2] - info[1];
  const int np = padded_states(p.states), bs = np + 8;
  __nv_bfloat16* Bs = reinterpret_cast<__nv_bfloat16*>(raw);   // [kChunk][bs]
  __nv_bfloat16* Xh = Bs + kChunk * bs;                        // [kChunk][kXStride] weighted x, high halves
  __nv_bfloat16* Xl = Xh + kChunk * kXStride;                  // low halves
  const int h0 = blockIdx.y * p.heads_per_block, col0 = blockIdx.z * kCols;
  const int cols = min(kCols, p.vdim - col0);
  const int steps = (len + 15) / 16;                           // sixteens of tokens
  const int group = h0 / (p.heads / p.groups);
  const __nv_bfloat16* rows = static_cast<const __nv_bfloat16*>(p.xbc) + static_cast<size_t>(begin) * p.xbc_width;
  const size_t b_off = static_cast<size_t>(p.heads) * p.vdim + static_cast<size_t>(group) * p.states;
  load_rows(Bs, bs, rows + b_off, p.xbc_width, len, steps * 16, p.states, np, rows_on_16_bytes(p, b_off, p.states));
  const size_t job_base = static_cast<size_t>(blockIdx.x) * p.heads;
  for (int i = 0; i < p.heads_per_block; ++i) {
    const int h = h0 + i;
    __syncthreads();   // the head before is done with dt_s, l_s and x
    if (warp == 0) chunk_decays(p, begin, len, h, dt_s, l_s);
    __syncthreads();
    const float last = l_s[kChunk - 1];
    const __nv_bfloat16* x = rows + static_cast<size_t>(h) * p.vdim + col0;
    if (rows_on_16_bytes(p, static_cast<size_t>(h) * p.vdim + col0, cols)) {
      for (int item = threadIdx.x; item < steps * 16 * (kCols / 8); item += kThreads) {
        const int t = item / (kCols / 8), c = (item % (kCols / 8)) * 8;
        uint4 high = make_uint4(0u, 0u, 0u, 0u), low = high;
        if (t < len && c < cols) {
          const uint4 v = *reinterpret_cast<const uint4*>(x + t * p.xbc_width + c);
          const __nv_bfloat162* pairs = reinterpret_cast<const __nv_bfloat162*>(&v);
          const float w = exp2f(last - l_s[t]) * dt_s[t];
          uint32_t* hp = reinterpret_cast<uint32_t*>(&high);
          uint32_t* lp = reinterpret_cast<uint32_t*>(&low);
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const float2 f = __bfloat1622float2(pairs[e]);
            split_pair(w * f.x, w * f.y, hp[e], lp[e]);
          }
        }
        *reinterpret_cast<uint4*>(Xh + t * kXStride + c) = high;
        *reinterpret_cast<uint4*>(Xl + t * kXStride + c) = low;
      }
    } else {
      for (int item = threadIdx.x; item < steps * 16 * kCols; item += kThreads) {
        const int t = item / kCols, c = item % kCols;
        float v = 0.0f;
        if (t < len && c < cols) v = exp2f(last - l_s[t]) * dt_s[t] * __bfloat162float(x[t * p.xbc_width + c]);
        const __nv_bfloat16 high = __float2bfloat16_rn(v);
        Xh[t * kXStride + c] = high;
        Xl[t * kXStride + c] = __float2bfloat16_rn(v - __bfloat162float(high));
      }
    }
    if (threadIdx.x == 0 && blockIdx.z == 0) p.chunk_decay[job_base + h] = last;
    copies_wait();   // b, ahead of the first head's product
    __syncthreads();
    float* E = p.chunk_state + (job_base + h) * static_cast<size_t>(p.states) * p.vdim;
    // a warp's job: sixteen rows of the state by 32 columns
    for (int job = warp; job < np / 16 * 2; job += kThreads / 32) {
      const int n0 = (job >> 1) * 16, c0 = (job & 1) * 32;
      if (c0 >= cols) continue;
      float acc[4][4];
#pragma unroll
      for (int nt = 0; nt < 4; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[nt][e] = 0.0f;
      for (int k = 0; k < steps; ++k) {
        // A[n, s] = b_s[n]: stored token by token, so the fragment is read transposed
        uint32_t a[4];
        ldsm4_trans(a, Bs + (k * 16 + (lane & 7) + ((lane >> 4) & 1) * 8) * bs + n0 + ((lane >> 3) & 1) * 8);
#pragma unroll
        for (int pair = 0; pair < 2; ++pair) {
          const int at = (k * 16 + (lane & 15)) * kXStride + c0 + pair * 16 + (lane >> 4) * 8;
          uint32_t b[4];
          ldsm4_trans(b, Xh + at);
          mma_bf16(acc[2 * pair], a, b[0], b[1]);
          mma_bf16(acc[2 * pair + 1], a, b[2], b[3]);
          ldsm4_trans(b, Xl + at);
          mma_bf16(acc[2 * pair], a, b[0], b[1]);
          mma_bf16(acc[2 * pair + 1], a, b[2], b[3]);
        }
      }
      const bool wide = (p.vdim & 1) == 0;
#pragma unroll
      for (int nt = 0; nt < 4; ++nt)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int n = n0 + (lane >> 2) + 8 * half, c = c0 + nt * 8 + 2 * (lane & 3);
          if (n >= p.states || c >= cols) continue;
          float* at = E + static_cast<size_t>(n) * p.vdim + col0 + c;
          if (wide && c + 1 < cols) *reinterpret_cast<float2*>(at) = make_float2(acc[nt][2 * half], acc[nt][2 * half + 1]);
          else {
            at[0] = acc[nt][2 * half];
            if (c + 1 < cols) at[1] = acc[nt][2 * half + 1];
          }
        }
    }
  }
}

// grid: (pieces of a head's state, heads, entries).  A thread VEC neighbouring values, the entry's chunks
// in order, eight chunks' sums asked for together: leaves the state at each chunk's start as two halves.
template <int VEC>
__global__ void __launch_bounds__(kThreads)
mamba2_carry_kernel(const Mamba2Params p) {
  pdl_launch_dependents();
  const int entry = blockIdx.z, h = blockIdx.y;
  const int count = p.entry_starts[entry + 1] - p.entry_starts[entry];
  int job0 = 0;
  const int lane = threadIdx.x & 31;
  for (int e = lane; e < entry; e += 32) job0 += chunks_of(p.entry_starts[e + 1] - p.entry_starts[e]);
#pragma unroll
  for (int offset = 16; offset > 0; offset >>= 1) job0 += __shfl_xor_sync(0xffffffffu, job0, offset);
  const int chunks = chunks_of(count);
  const size_t head_size = static_cast<size_t>(p.states) * p.vdim;
  const size_t index = (static_cast<size_t>(blockIdx.x) * kThreads + threadIdx.x) * VEC;
  float* own = p.state + (static_cast<size_t>(p.state_slots[entry]) * p.heads + h) * head_size + index;
  const bool fresh = p.fresh[entry] != 0;
  pdl_wait();
  if (chunks == 0 || index >= head_size) return;
  auto load = [](float (&v)[VEC], const float* at) {
    if constexpr (VEC == 4) {
      const float4 q = *reinterpret_cast<const float4*>(at);
      v[0] = q.x, v[1] = q.y, v[2] = q.z, v[3] = q.w;
    } else {
      v[0] = *at;
    }
  };
  auto store_halves = [&](__nv_bfloat16* at, const float (&v)[VEC]) {
    if constexpr (VEC == 4) {
      uint2 high, low;
      split_pair(v[0], v[1], high.x, low.x);
      split_pair(v[2], v[3], high.y, low.y);
      *reinterpret_cast<uint2*>(at) = high;
      *reinterpret_cast<uint2*>(at + head_size) = low;
    } else {
      const __nv_bfloat16 high = __float2bfloat16_rn(v[0]);
      at[0] = high;
      at[head_size] = __float2bfloat16_rn(v[0] - __bfloat162float(high));
    }
  };
  float s[VEC];
#pragma unroll
  for (int e = 0; e < VEC; ++e) s[e] = 0.0f;
  if (!fresh) load(s, own);
  const size_t job_stride = static_cast<size_t>(p.heads) * head_size;
  const float* E = p.chunk_state + (static_cast<size_t>(job0) * p.heads + h) * head_size + index;
  __nv_bfloat16* starts = static_cast<__nv_bfloat16*>(p.chunk_start) + (static_cast<size_t>(job0) * p.heads + h) * 2 * head_size + index;
  const float* decay = p.chunk_decay + static_cast<size_t>(job0) * p.heads + h;
  for (int c0 = 0; c0 < chunks; c0 += 8) {
    float sums[8][VEC], l[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      if (c0 + j < chunks) {
        load(sums[j], E + (c0 + j) * job_stride);
        l[j] = decay[static_cast<size_t>(c0 + j) * p.heads];
      }
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      if (c0 + j >= chunks) break;
      store_halves(starts + (c0 + j) * 2 * job_stride, s);
      const float keep = exp2f(l[j]);
#pragma unroll
      for (int e = 0; e < VEC; ++e) s[e] = fmaf(keep, s[e], sums[j][e]);
    }
  }
  if constexpr (VEC == 4) *reinterpret_cast<float4*>(own) = make_float4(s[0], s[1], s[2], s[3]);
  else *own = s[0];
}

// grid: (jobs, heads / heads_per_block, column tiles).  A warp owns sixteen tokens of the chunk.
__global__ void __launch_bounds__(kThreads, 2)
mamba2_outputs_kernel(const Mamba2Params p) {
  extern __shared__ __align__(16) unsigned char raw[];
  __shared__ int info[3];
  __shared__ float dt_s[kChunk], l_s[kChunk];
  pdl_launch_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (warp == 0) find_chunk(p.entry_starts, p.num_entries, blockIdx.x, info);
  pdl_wait();
  __syncthreads();
  if (info[0] < 0) return;
  const int begin = info[1], len = info[2] - info[1];
  const int np = padded_states(p.states), bs = np + 8;
  __nv_bfloat16* Cs = reinterpret_cast<__nv_bfloat16*>(raw);   // [kChunk][bs]
  __nv_bfloat16* Xs = Cs + kChunk * bs;                        // [kChunk][kXStride]
  __nv_bfloat16* Bs = Xs + kChunk * kXStride;                  // [kChunk][bs]
  __nv_bfloat16* Sh = Bs;                                      // then the state: [np][kXStride] high halves
  __nv_bfloat16* Sl = Sh + np * kXStride;                      // low halves
  const int h0 = blockIdx.y * p.heads_per_block, col0 = blockIdx.z * kCols;
  const int cols = min(kCols, p.vdim - col0);
  const int steps = (len + 15) / 16;
  const int group = h0 / (p.heads / p.groups);
  const __nv_bfloat16* rows = static_cast<const __nv_bfloat16*>(p.xbc) + static_cast<size_t>(begin) * p.xbc_width;
  const size_t b_off = static_cast<size_t>(p.heads) * p.vdim + static_cast<size_t>(group) * p.states;
  const size_t c_off = b_off + static_cast<size_t>(p.groups) * p.states;
  load_rows(Bs, bs, rows + b_off, p.xbc_width, len, steps * 16, p.states, np, rows_on_16_bytes(p, b_off, p.states));
  load_rows(Cs, bs, rows + c_off, p.xbc_width, len, steps * 16, p.states, np, rows_on_16_bytes(p, c_off, p.states));
  copies_wait();
  __syncthreads();
  // the scores of the warp's tokens with every token up to them: once for all heads of the block
  const bool live = warp * 16 < len;
  const int row0 = warp * 16 + (lane >> 2);   // this thread's rows: row0 and row0 + 8
  float scores[kChunk / 8][4];
#pragma unroll
  for (int nt = 0; nt < kChunk / 8; ++nt)
#pragma unroll
    for (int e = 0; e < 4; ++e) scores[nt][e] = 0.0f;
  if (live) {
    for (int k = 0; k < np / 16; ++k) {
      uint32_t a[4];
      ldsm4(a, Cs + (warp * 16 + (lane & 15)) * bs + k * 16 + (lane >> 4) * 8);
#pragma unroll
      for (int pair = 0; pair < kChunk / 16; ++pair) {
        if (pair > warp) break;
        uint32_t b[4];   // B[n, s] = b_s[n], stored token by token: the columns' fragments as they lie
        ldsm4(b, Bs + (pair * 16 + (lane & 7) + (lane >> 4) * 8) * bs + k * 16 + ((lane >> 3) & 1) * 8);
        mma_bf16(scores[2 * pair], a, b[0], b[1]);
        mma_bf16(scores[2 * pair + 1], a, b[2], b[3]);
      }
    }
  }
  for (int i = 0; i < p.heads_per_block; ++i) {
    const int h = h0 + i;
    __syncthreads();   // all are done with b, and with the head before's x, state and decays
    if (warp == 0) chunk_decays(p, begin, len, h, dt_s, l_s);
    const size_t x_off = static_cast<size_t>(h) * p.vdim + col0;
    load_rows(Xs, kXStride, rows + x_off, p.xbc_width, len, steps * 16, cols, kCols, rows_on_16_bytes(p, x_off, cols));
    const size_t head_size = static_cast<size_t>(p.states) * p.vdim;
    const __nv_bfloat16* S0 = static_cast<const __nv_bfloat16*>(p.chunk_start) +
                              (static_cast<size_t>(blockIdx.x) * p.heads + h) * 2 * head_size + col0;
    const bool whole = p.vdim % 8 == 0 && (reinterpret_cast<uintptr_t>(p.chunk_start) & 15) == 0;
    load_rows(Sh, kXStride, S0, p.vdim, p.states, np, cols, kCols, whole);
    load_rows(Sl, kXStride, S0 + head_size, p.vdim, p.states, np, cols, kCols, whole);
    copies_wait();
    __syncthreads();
    if (!live) continue;
    float y[kCols / 8][4];
#pragma unroll
    for (int nt = 0; nt < kCols / 8; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) y[nt][e] = 0.0f;
    // what the state at the chunk's start gives
    for (int k = 0; k < np / 16; ++k) {
      uint32_t a[4];
      ldsm4(a, Cs + (warp * 16 + (lane & 15)) * bs + k * 16 + (lane >> 4) * 8);
#pragma unroll
      for (int pair = 0; pair < kCols / 16; ++pair) {
        const int at = (k * 16 + (lane & 15)) * kXStride + pair * 16 + (lane >> 4) * 8;
        uint32_t b[4];
        ldsm4_trans(b, Sh + at);
        mma_bf16(y[2 * pair], a, b[0], b[1]);
        mma_bf16(y[2 * pair + 1], a, b[2], b[3]);
        ldsm4_trans(b, Sl + at);
        mma_bf16(y[2 * pair], a, b[0], b[1]);
        mma_bf16(y[2 * pair + 1], a, b[2], b[3]);
      }
    }
    const float l_first = l_s[row0], l_second = l_s[row0 + 8];
    const float from_start[2] = {exp2f(l_first), exp2f(l_second)};
#pragma unroll
    for (int nt = 0; nt < kCols / 8; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) y[nt][e] *= from_start[e >> 1];
    // the chunk's own tokens: the weights take the scores' registers as fragments of the next product
#pragma unroll
    for (int k = 0; k < kChunk / 16; ++k) {
      if (k > warp) break;
      uint32_t high[4], low[4];
#pragma unroll
      for (int part = 0; part < 4; ++part) {
        // a[0]: rows row0, columns 0-7; a[1]: rows row0 + 8; a[2], a[3]: columns 8-15
        const int nt = 2 * k + (part >> 1), e = (part & 1) * 2;
        const int row = row0 + 8 * (part & 1);
        const float l_row = (part & 1) ? l_second : l_first;
        float w[2];
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          const int col = nt * 8 + 2 * (lane & 3) + j;
          w[j] = col <= row ? scores[nt][e + j] * (exp2f(l_row - l_s[col]) * dt_s[col]) : 0.0f;
        }
        split_pair(w[0], w[1], high[part], low[part]);
      }
#pragma unroll
      for (int pair = 0; pair < kCols / 16; ++pair) {
        uint32_t b[4];
        ldsm4_trans(b, Xs + (k * 16 + (lane & 15)) * kXStride + pair * 16 + (lane >> 4) * 8);
        mma_bf16(y[2 * pair], high, b[0], b[1]);
        mma_bf16(y[2 * pair + 1], high, b[2], b[3]);
        mma_bf16(y[2 * pair], low, b[0], b[1]);
        mma_bf16(y[2 * pair + 1], low, b[2], b[3]);
      }
    }
    const float skip = p.d[h];
    const size_t width = static_cast<size_t>(p.heads) * p.vdim;
    const bool wide = (p.vdim & 1) == 0;
#pragma unroll
    for (int nt = 0; nt < kCols / 8; ++nt)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int row = row0 + 8 * half, c = nt * 8 + 2 * (lane & 3);
        if (row >= len || c >= cols) continue;
        float* at = p.y + static_cast<size_t>(begin + row) * width + static_cast<size_t>(h) * p.vdim + col0 + c;
        const float first = fmaf(skip, __bfloat162float(Xs[row * kXStride + c]), y[nt][2 * half]);
        const float second = fmaf(skip, __bfloat162float(Xs[row * kXStride + c + 1]), y[nt][2 * half + 1]);
        if (wide && c + 1 < cols) *reinterpret_cast<float2*>(at) = make_float2(first, second);
        else {
          at[0] = first;
          if (c + 1 < cols) at[1] = second;
        }
      }
  }
}

// ---------------------------------------------------------------------------------------
// The gate, then the norm of each part.  grid: (tokens, norm groups).
// ---------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(kThreads)
mamba2_finish_kernel(const Mamba2Params p) {
  __shared__ float scratch[32];
  constexpr int kKept = 16;   // values a thread keeps between its passes: parts of up to 4096 values
  pdl_launch_dependents();
  const int width = p.heads * p.vdim, size = width / p.norm_groups;
  const int t = blockIdx.x, first = blockIdx.y * size;
  const float* weight = p.norm_weight + first;
  pdl_wait();
  const float* y = p.y + static_cast<size_t>(t) * width + first;
  const float* z = p.proj + static_cast<size_t>(t) * p.proj_width + p.z_off + first;
  T* out = static_cast<T*>(p.out) + static_cast<size_t>(t) * width + first;
  const bool fits = size <= kKept * static_cast<int>(blockDim.x);
  float kept[kKept];
  float sum = 0.0f;
  auto gated = [&](int i) {
    const float gate = z[i];
    return y[i] * (gate / (1.0f + expf(-gate)));
  };
  if (fits) {
#pragma unroll
    for (int j = 0; j < kKept; ++j) {
      const int i = threadIdx.x + j * blockDim.x;
      kept[j] = i < size ? gated(i) : 0.0f;
      sum = fmaf(kept[j], kept[j], sum);
    }
  } else {
    for (int i = threadIdx.x; i < size; i += blockDim.x) {
      const float v = gated(i);
      sum = fmaf(v, v, sum);
    }
  }
  const float inverse = 1.0f / sqrtf(block_sum(sum, scratch) / static_cast<float>(size) + p.eps);
  if (fits) {
#pragma unroll
    for (int j = 0; j < kKept; ++j) {
      const int i = threadIdx.x + j * blockDim.x;
      if (i < size) out[i] = from_float<T>(kept[j] * inverse * weight[i]);
    }
  } else {
    for (int i = threadIdx.x; i < size; i += blockDim.x) out[i] = from_float<T>(gated(i) * inverse * weight[i]);
  }
}

// The same for parts of up to 128 * PIECES values that are whole vectors: a warp a part, the part in registers
// between its passes.
template <typename T, int PIECES>
__global__ void __launch_bounds__(kThreads)
mamba2_finish_rows_kernel(const Mamba2Params p) {
  pdl_launch_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long job = static_cast<long long>(blockIdx.x) * (kThreads / 32) + warp;
  const int width = p.heads * p.vdim, size = width / p.norm_groups;
  if (job >= static_cast<long long>(p.num_tokens) * p.norm_groups) return;
  const size_t t = job / p.norm_groups;
  const int first = static_cast<int>(job % p.norm_groups) * size;
  pdl_wait();
  const float* y = p.y + t * width + first;
  const float* z = p.proj + t * p.proj_width + p.z_off + first;
  float4 kept[PIECES], gate[PIECES];
#pragma unroll
  for (int j = 0; j < PIECES; ++j) {
    const int i = 4 * (lane + 32 * j);
    kept[j] = gate[j] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    if (i < size) {
      kept[j] = *reinterpret_cast<const float4*>(y + i);
      gate[j] = *reinterpret_cast<const float4*>(z + i);
    }
  }
  auto silu = [](float v) { return v / (1.0f + expf(-v)); };
  float sum = 0.0f;
#pragma unroll
  for (int j = 0; j < PIECES; ++j) {
    kept[j].x *= silu(gate[j].x), kept[j].y *= silu(gate[j].y), kept[j].z *= silu(gate[j].z), kept[j].w *= silu(gate[j].w);
    sum = fmaf(kept[j].x, kept[j].x, sum), sum = fmaf(kept[j].y, kept[j].y, sum);
    sum = fmaf(kept[j].z, kept[j].z, sum), sum = fmaf(kept[j].w, kept[j].w, sum);
  }
  const float inverse = 1.0f / sqrtf(warp_sum(sum) / static_cast<float>(size) + p.eps);
  T* out = static_cast<T*>(p.out) + t * width + first;
#pragma unroll
  for (int j = 0; j < PIECES; ++j) {
    const int i = 4 * (lane + 32 * j);
    if (i >= size) continue;
    const float4 w = *reinterpret_cast<const float4*>(p.norm_weight + first + i);
    const float v[4] = {kept[j].x * inverse * w.x, kept[j].y * inverse * w.y, kept[j].z * inverse * w.z, kept[j].w * inverse * w.w};
    if constexpr (sizeof(T) == 4) {
      *reinterpret_cast<float4*>(out + i) = make_float4(v[0], v[1], v[2], v[3]);
    } else {
      __nv_bfloat162 pair[2] = {__floats2bfloat162_rn(v[0], v[1]), __floats2bfloat162_rn(v[2], v[3])};
      *reinterpret_cast<uint2*>(out + i) = *reinterpret_cast<const uint2*>(pair);
    }
  }
}

template <typename T>
static int launch_finish(const Mamba2Params& p, cudaStream_t s) {
  const int size = p.heads * p.vdim / p.norm_groups;
  const uintptr_t bases = reinterpret_cast<uintptr_t>(p.y) | reinterpret_cast<uintptr_t>(p.proj) | reinterpret_cast<uintptr_t>(p.out) |
                          reinterpret_cast<uintptr_t>(p.norm_weight);
  if (size % 4 == 0 && size <= 1024 && p.proj_width % 4 == 0 && p.z_off % 4 == 0 && (bases & 15) == 0) {
    const long long jobs = static_cast<long long>(p.num_tokens) * p.norm_groups;
    const unsigned grid = static_cast<unsigned>((jobs + kThreads / 32 - 1) / (kThreads / 32));
    if (size <= 256) return vipera_launch(mamba2_finish_rows_kernel<T, 2>, grid, kThreads, 0, s, p);
    if (size <= 512) return vipera_launch(mamba2_finish_rows_kernel<T, 4>, grid, kThreads, 0, s, p);
    return vipera_launch(mamba2_finish_rows_kernel<T, 8>, grid, kThreads, 0, s, p);
  }
  const int threads = size >= 256 ? 256 : (size + 31) / 32 * 32;
  return vipera_launch(mamba2_finish_kernel<T>, dim3(p.num_tokens, p.norm_groups), threads, 0, s, p);
}

// ---------------------------------------------------------------------------------------
template <typename T, int ROWS>
static int launch_walk(const Mamba2Params& p, cudaStream_t s) {
  const size_t shared = (static_cast<size_t>(2 * kStage) * p.states + kStage * kCols + 2 * 8 * kCols) * sizeof(float);
  const dim3 grid((p.vdim + kCols - 1) / kCols, p.heads, p.num_entries);
  if (p.vdim % 4 == 0 && (reinterpret_cast<uintptr_t>(p.state) & 15) == 0)
    return vipera_launch(mamba2_walk_kernel<T, ROWS, true>, grid, kThreads, shared, s, p);
  return vipera_launch(mamba2_walk_kernel<T, ROWS, false>, grid, kThreads, shared, s, p);
}

template <typename T>
static int launch_walk_rows(const Mamba2Params& p, cudaStream_t s) {
  if (p.states <= 32) return launch_walk<T, 2>(p, s);
  if (p.states <= 64) return launch_walk<T, 4>(p, s);
  if (p.states <= 128) return launch_walk<T, 8>(p, s);
  return launch_walk<T, 16>(p, s);
}

static int launch_chunks(const Mamba2Params& p, cudaStream_t s) {
  static bool configured = false;
  if (!configured) {
    if (cudaFuncSetAttribute(mamba2_parts_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(parts_shared(kMaxState))) != cudaSuccess ||
        cudaFuncSetAttribute(mamba2_outputs_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(outputs_shared(kMaxState))) != cudaSuccess)
      return VIPERA_BAD_ARGUMENT;
    configured = true;
  }
  const dim3 grid(p.num_jobs, p.heads / p.heads_per_block, (p.vdim + kCols - 1) / kCols);
  int status = vipera_launch(mamba2_parts_kernel, grid, kThreads, parts_shared(p.states), s, p);
  if (status) return status;
  const size_t head_size = static_cast<size_t>(p.states) * p.vdim;
  const bool four = head_size % 4 == 0 && ((reinterpret_cast<uintptr_t>(p.state) | reinterpret_cast<uintptr_t>(p.chunk_state) | reinterpret_cast<uintptr_t>(p.chunk_start)) & 15) == 0;
  const size_t per_block = static_cast<size_t>(kThreads) * (four ? 4 : 1);
  const dim3 carry_grid(static_cast<unsigned>((head_size + per_block - 1) / per_block), p.heads, p.num_entries);
  status = four ? vipera_launch(mamba2_carry_kernel<4>, carry_grid, kThreads, 0, s, p)
                : vipera_launch(mamba2_carry_kernel<1>, carry_grid, kThreads, 0, s, p);
  if (status) return status;
  return vipera_launch(mamba2_outputs_kernel, grid, kThreads, outputs_shared(p.states), s, p);
}

// num_jobs > 0 (bfloat16, with chunk_state and chunk_decay): entries of several tokens run as chunks
// (num_jobs at least their count), entries of one token walk where `any_single` says there are some; else
// every entry walks.  `dtype`: the type of xbc and out.
VIPERA_API int vipera_mamba2(const Mamba2Params* params, int dtype, int any_single, void* stream) {
  Mamba2Params p = *params;
  if (p.num_tokens <= 0 || p.num_entries <= 0) return VIPERA_OK;
  if (p.heads <= 0 || p.heads > 65535 || p.vdim <= 0 || p.states <= 0 || p.states > kMaxState || p.groups <= 0 ||
      p.heads % p.groups || p.norm_groups <= 0 || p.norm_groups > 65535 || (p.heads * p.vdim) % p.norm_groups || p.num_entries > 65535)
    return VIPERA_BAD_SHAPE;
  const bool chunked = p.num_jobs > 0;
  if (chunked && (dtype != VIPERA_BF16 || !p.chunk_state || !p.chunk_start || !p.chunk_decay || p.heads_per_block <= 0 ||
                  (p.heads / p.groups) % p.heads_per_block))
    return VIPERA_BAD_ARGUMENT;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  int status = VIPERA_OK;
  p.single_only = chunked ? 1 : 0;
  if (chunked) status = launch_chunks(p, s);
  if (status) return status;
  if (!chunked || any_single) {
    if (dtype == VIPERA_F32) status = launch_walk_rows<float>(p, s);
    else if (dtype == VIPERA_BF16) status = launch_walk_rows<__nv_bfloat16>(p, s);
    else return VIPERA_BAD_DTYPE;
    if (status) return status;
  }
  return dtype == VIPERA_F32 ? launch_finish<float>(p, s) : launch_finish<__nv_bfloat16>(p, s);
}

VIPERA_API int vipera_mamba2_params_size() { return static_cast<int>(sizeof(Mamba2Params)); }
VIPERA_API int vipera_mamba2_chunk() { return kChunk; }
VIPERA_API const char* vipera_mamba2_status_text(int status) { return vipera_status_text(status); }
