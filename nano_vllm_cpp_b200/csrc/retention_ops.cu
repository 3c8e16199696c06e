// Matrix memories that decay by one number per head (retention, lightning attention, the state-space dual form), and the
// causal convolution over time.
//
//   causal_conv            out = h + conv(h) or silu(conv(h) + bias), a short convolution over time on every channel, its
//                          history kept per request
//   rotary_table           cosine and sine of every row's angles, shared by the heads
//   retention_step         entries of one row: rotation, state update, output (and head norm and gate) in one launch
//   retention_scan         any sizes, row by row (the twin of the others; float32 runs)
//   retention_chunk_*      entries of many rows on the tensor cores, 64 rows at a time
//   gated_norm             a row's outputs of all heads: skip term, gate and RMS norm over equal parts of the row
//
// Per head with the decay d, keys k (turned by their positions, times a constant) and values v:
//   S_t = d S_{t-1} + k_t v_t^T,   o_t = S_t^T q_t.
// What follows is either y_t = o_t / sqrt(mean(o_t^2) + eps) * silu(gate_t) per head, in the same kernels, or o_t goes out in
// float32 (gated_norm takes it).  The decay is a constant of the head, or it follows from a step size that every row has
// per head (row decays): dt = softplus(z + bias), d = exp(-exp(a) dt), and the row's key is multiplied by dt.  Several heads
// may share their q and k.
// S lives in float32.  The chunked form writes the recurrence for the rows i = 0 .. n - 1 of a chunk that starts from S:
//   o_i = d^(i+1) S^T q_i + sum_{j <= i} d^(i-j) (q_i . k_j) v_j,   S' = d^n S + sum_j d^(n-1-j) k_j v_j^T
// (with row decays d^(i-j) is the product of the rows' decays from j + 1 to i, taken as a difference of running sums of
// their logarithms) in three launches: every chunk's own sum over j (all chunks at once), a pass over each entry's chunks that turns
// these into the states the chunks start from, and every chunk's outputs (all chunks at once).  All operands of the
// tensor-core products are float32 numbers split into two bfloat16 terms (hi, and what its rounding left), with the
// three products hi hi, hi lo and lo hi, so that a product carries sixteen bits of each operand; sums are float32.
#include "common.cuh"

#include <algorithm>

namespace {

// ------------------------------------------------------------------ causal convolution
struct ConvArgs {
  const float* h;           // [T, H], rows `ld` apart
  long long ld;
  const float* w;           // [taps, H]: row j multiplies the input taps - 1 - j positions back
  const float* bias;        // [H] or nullptr
  const int* row_entry;
  const int* cu_rows;
  const int* entry_slot;
  float* state;             // per slot [taps - 1, H]: the inputs of the request's last taps - 1 positions
  long long slot_stride;
  void* out;
  int out_dt, T, H, taps, rows, update, act;           // act 0: h + conv(h); 1: silu(conv(h) + bias)
};

template <int VEC>
struct Vals { float v[VEC]; };
template <int VEC>
__device__ __forceinline__ Vals<VEC> ldv(const float* p) {
  Vals<VEC> c;
  if (VEC == 4) {
    const float4 q = *reinterpret_cast<const float4*>(p);
    c.v[0] = q.x; c.v[VEC > 1 ? 1 : 0] = q.y; c.v[VEC > 2 ? 2 : 0] = q.z; c.v[VEC > 3 ? 3 : 0] = q.w;
  } else {
#pragma unroll
    for (int j = 0; j < VEC; ++j) c.v[j] = p[j];
  }
  return c;
}
template <int VEC>
__device__ __forceinline__ void stv(float* p, const Vals<VEC>& c) {
  if (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(c.v[0], c.v[VEC > 1 ? 1 : 0], c.v[VEC > 2 ? 2 : 0], c.v[VEC > 3 ? 3 : 0]);
  else {
#pragma unroll
    for (int j = 0; j < VEC; ++j) p[j] = c.v[j];
  }
}
template <int VEC>
__device__ __forceinline__ void st_out(void* out, int dt, size_t i, const Vals<VEC>& c) {
  if (VEC == 4 && dt == NV_DT_BF16) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(c.v[0], c.v[VEC > 1 ? 1 : 0]);
    const __nv_bfloat162 hi = __floats2bfloat162_rn(c.v[VEC > 2 ? 2 : 0], c.v[VEC > 3 ? 3 : 0]);
    uint2 pk;
    pk.x = *reinterpret_cast<const uint32_t*>(&lo);
    pk.y = *reinterpret_cast<const uint32_t*>(&hi);
    *reinterpret_cast<uint2*>((bf16*)out + i) = pk;
  } else if (VEC == 4) {
    stv<VEC>((float*)out + i, c);
  } else {
#pragma unroll
    for (int j = 0; j < VEC; ++j) st_dt(out, dt, i + j, c.v[j]);
  }
}

// A thread owns VEC channels and `rows` consecutive rows of the batch; the inputs it still needs stay in registers from
// row to row (TAPS > 0) and come from the request's state where they lie before the entry.  `update`: the state is
// brought up to date here too, which is safe where every entry has one row (nobody else reads it).
// The taps are added in ascending order of time, whatever the cut, so a row's result does not depend on it.
template <int VEC, int TAPS>
__global__ void __launch_bounds__(256) causal_conv_kernel(ConvArgs a) {
  grid_dep_wait();
  grid_dep_launch();
  const int c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c * VEC >= a.H) return;
  const size_t col = (size_t)c * VEC;
  const int t0 = blockIdx.x * a.rows, t1 = min(a.T, t0 + a.rows);
  constexpr int HN = TAPS > 1 ? TAPS - 1 : 1;
  Vals<VEC> hist[HN], w[TAPS > 0 ? TAPS : 1];          // hist[d - 1]: the input d positions back
  const int taps = TAPS > 0 ? TAPS : a.taps;
  if (TAPS > 0) {
#pragma unroll
    for (int j = 0; j < TAPS; ++j) w[j] = ldv<VEC>(a.w + (size_t)j * a.H + col);
  }
  for (int t = t0; t < t1; ++t) {
    const int e = a.row_entry[t];
    const int j = t - a.cu_rows[e];
    float* st = a.state + (size_t)a.entry_slot[e] * a.slot_stride + col;
    auto back = [&](int d) {
      return j >= d ? ldv<VEC>(a.h + (size_t)(t - d) * a.ld + col) : ldv<VEC>(st + (size_t)(taps - 1 + j - d) * a.H);
    };
    const Vals<VEC> cur = ldv<VEC>(a.h + (size_t)t * a.ld + col);
    Vals<VEC> acc;
#pragma unroll
    for (int i = 0; i < VEC; ++i) acc.v[i] = 0.f;
    auto finish = [&](const Vals<VEC>& last) {         // the current token's tap, then what the mode adds or applies
      if (a.act) {
        Vals<VEC> b = acc;
        if (a.bias) b = ldv<VEC>(a.bias + col);
#pragma unroll
        for (int i = 0; i < VEC; ++i) {
          const float z = fmaf(last.v[i], cur.v[i], acc.v[i]) + (a.bias ? b.v[i] : 0.f);
          acc.v[i] = z / (1.f + expf(-z));
        }
      } else {
#pragma unroll
        for (int i = 0; i < VEC; ++i) acc.v[i] = cur.v[i] + fmaf(last.v[i], cur.v[i], acc.v[i]);
      }
    };
    if (TAPS > 0) {
      if (t == t0 || j == 0) {
#pragma unroll
        for (int d = 1; d < TAPS; ++d) hist[d - 1] = back(d);
      }
#pragma unroll
      for (int d = TAPS - 1; d >= 1; --d)
#pragma unroll
        for (int i = 0; i < VEC; ++i) acc.v[i] = fmaf(w[TAPS - 1 - d].v[i], hist[d - 1].v[i], acc.v[i]);
      finish(w[TAPS > 0 ? TAPS - 1 : 0]);
      st_out<VEC>(a.out, a.out_dt, (size_t)t * a.H + col, acc);
#pragma unroll
      for (int d = HN - 1; d >= 1; --d) hist[d] = hist[d - 1];
      hist[0] = cur;
      if (a.update && TAPS > 1) {
#pragma unroll
        for (int s = 0; s < TAPS - 1; ++s) stv<VEC>(st + (size_t)s * a.H, hist[TAPS - 2 - s]);
      }
    } else {
      for (int d = taps - 1; d >= 1; --d) {
        const Vals<VEC> x = back(d), wd = ldv<VEC>(a.w + (size_t)(taps - 1 - d) * a.H + col);
#pragma unroll
        for (int i = 0; i < VEC; ++i) acc.v[i] = fmaf(wd.v[i], x.v[i], acc.v[i]);
      }
      const Vals<VEC> wl = ldv<VEC>(a.w + (size_t)(taps - 1) * a.H + col);
      finish(wl);
      st_out<VEC>(a.out, a.out_dt, (size_t)t * a.H + col, acc);
      if (a.update)
        for (int s = 0; s < taps - 1; ++s)
          stv<VEC>(st + (size_t)s * a.H, s + 1 < taps - 1 ? ldv<VEC>(st + (size_t)(s + 1) * a.H) : cur);
    }
  }
}

// ------------------------------------------------------------------ rotation
__global__ void rotary_table_kernel(const int* __restrict__ positions, const float* __restrict__ inv_freq, int half,
                                    float2* __restrict__ out, long long n) {
  grid_dep_wait();
  grid_dep_launch();
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n) return;
  const float ang = (float)positions[i / half] * inv_freq[i % half];
  out[i] = make_float2(cosf(ang), sinf(ang));
}

struct RetArgs {
  const float* proj;        // [T, ld]: q | k | v | gate at their columns, heads side by side
  long long ld;
  int q0, k0, v0, g0;
  const float2* table;      // [T, half]: cosine and sine (the step kernel works them out itself)
  const int* positions;
  const float* inv_freq;
  int half;                 // pairs (i, i + half) of the first 2 half elements of a q or k head are turned
  const int* row_entry;
  const int* cu_rows;
  const int* entry_slot;
  const int* rows;          // step: which batch rows (nullptr: all)
  float* S;                 // [slots][H, dk, dv]
  long long S_stride;
  const float* powers;      // [H, RC + 1]: the decay to the power 0 .. RC
  float k_scale, eps;
  void* out;                // [T, H * dv]
  float* raw;               // scan: [T, H, dv]
  uint32_t* chunks;         // chunked form: per chunk and head dk * dv words (float32 sums, then the states' two terms)
  int G;                    // heads of q and k: head h reads q/k head h / (H / G)
  int hb;                   // chunked form: heads of a block, all with the same q and k
  int raw_out;              // the outputs go to `raw` [T, H, dv] in float32, without norm and gate
  // Row decays (dsrc != nullptr): step size dt = softplus(dsrc[t, d0 + h] + dt_bias[h]), decay exp(-exp(A_log[h]) dt), and
  // the row's k times dt instead of k_scale.
  const float* dsrc;
  long long d_ld;
  int d0;
  const float* A_log;
  const float* dt_bias;
  float* chunk_decay;       // chunked form with row decays: [chunks, H], what a chunk multiplies its first state by
  // v2: the chunked form reads two neighbouring elements at a time; planes: the states' terms lie row by row (see the pass)
  int out_dt, H, dk, dv, num_entries, min_rows, slice, v2, planes;
};

constexpr int RC = 64;                 // rows of a chunk
constexpr int RT_THREADS = 256;

__device__ __forceinline__ float silu_of(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float step_size_of(const RetArgs& a, int t, int h) {
  const float z = a.dsrc[(size_t)t * a.d_ld + a.d0 + h] + a.dt_bias[h];
  return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)));
}

// ------------------------------------------------------------------ one row per entry
// grid (rows, heads).  The head's matrix streams through registers once: a thread owns VEC neighbouring columns and every
// RS-th row of it, and the threads' shares of the output are added in order through shared memory.
template <int VEC>
__global__ void __launch_bounds__(RT_THREADS) retention_step_kernel(RetArgs a) {
  extern __shared__ float sm[];        // q [dk], k [dk], shares [RS][dv]
  __shared__ float red[RT_THREADS / 32];
  const int h = blockIdx.y, tid = threadIdx.x, dk = a.dk, dv = a.dv, half = a.half;
  const int t = a.rows ? a.rows[blockIdx.x] : blockIdx.x;
  const int groups = dv / VEC, RS = RT_THREADS / groups;
  float* q = sm;
  float* k = q + dk;
  float* share = k + dk;
  float* Sg = a.S + (size_t)a.entry_slot[a.row_entry[t]] * a.S_stride + (size_t)h * dk * dv;
  const float* p = a.proj + (size_t)t * a.ld;
  const int cg = tid % groups, rs = tid / groups;
  const bool owner = rs < RS;
  constexpr int U = 8;                 // rows of the matrix in flight per thread
  // The state's first rows are asked for before the projections of this step are there.
  Vals<VEC> cur[U];
  if (owner) {
#pragma unroll
    for (int u = 0; u < U; ++u)
      if (rs + u * RS < dk) cur[u] = ldv<VEC>(Sg + (size_t)(rs + u * RS) * dv + cg * VEC);
  }
  grid_dep_wait();
  grid_dep_launch();
  const int items = half + (dk - 2 * half);
  const int gh = h / (a.H / a.G);
  float d = 0.f, ks = a.k_scale;
  if (a.dsrc) {
    ks = step_size_of(a, t, h);
    d = expf(-expf(a.A_log[h]) * ks);
  } else {
    d = a.powers[(size_t)h * (RC + 1) + 1];
  }
  for (int i = tid; i < items; i += RT_THREADS) {
    const float* pq = p + a.q0 + (size_t)gh * dk;
    const float* pk = p + a.k0 + (size_t)gh * dk;
    if (i < half) {
      const float ang = (float)a.positions[t] * a.inv_freq[i];
      const float cs = cosf(ang), sn = sinf(ang);
      q[i] = pq[i] * cs - pq[i + half] * sn;
      q[i + half] = pq[i + half] * cs + pq[i] * sn;
      k[i] = (pk[i] * cs - pk[i + half] * sn) * ks;
      k[i + half] = (pk[i + half] * cs + pk[i] * sn) * ks;
    } else {
      q[i + half] = pq[i + half];
      k[i + half] = pk[i + half] * ks;
    }
  }
  __syncthreads();
  if (owner) {
    Vals<VEC> v, o;
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      v.v[i] = p[a.v0 + (size_t)h * dv + cg * VEC + i];
      o.v[i] = 0.f;
    }
    for (int r0 = rs; r0 < dk; r0 += U * RS) {
      if (r0 != rs) {
#pragma unroll
        for (int u = 0; u < U; ++u)
          if (r0 + u * RS < dk) cur[u] = ldv<VEC>(Sg + (size_t)(r0 + u * RS) * dv + cg * VEC);
      }
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int r = r0 + u * RS;
        if (r < dk) {
          const float kr = k[r], qr = q[r];
#pragma unroll
          for (int i = 0; i < VEC; ++i) {
            cur[u].v[i] = fmaf(d, cur[u].v[i], kr * v.v[i]);
            o.v[i] = fmaf(cur[u].v[i], qr, o.v[i]);
          }
          stv<VEC>(Sg + (size_t)r * dv + cg * VEC, cur[u]);
        }
      }
    }
#pragma unroll
    for (int i = 0; i < VEC; ++i) share[(size_t)rs * dv + cg * VEC + i] = o.v[i];
  }
  __syncthreads();
  float ss = 0.f;
  for (int c = tid; c < dv; c += RT_THREADS) {
    float o = 0.f;
    for (int i = 0; i < RS; ++i) o += share[(size_t)i * dv + c];
    share[c] = o;                      // (column c's shares are read by this thread alone)
    if (a.raw_out) a.raw[((size_t)t * a.H + h) * dv + c] = o;
    ss = fmaf(o, o, ss);
  }
  if (a.raw_out) return;
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  float sum = 0.f;
#pragma unroll
  for (int i = 0; i < RT_THREADS / 32; ++i) sum += red[i];
  const float r = rsqrtf(sum / (float)dv + a.eps);
  for (int c = tid; c < dv; c += RT_THREADS)
    st_dt(a.out, a.out_dt, ((size_t)t * a.H + h) * dv + c, share[c] * r * silu_of(p[a.g0 + (size_t)h * dv + c]));
}

// ------------------------------------------------------------------ any sizes, row by row
// grid (entries, heads, slices of `slice` columns); the slice of the head's matrix lives in shared memory.
__global__ void __launch_bounds__(RT_THREADS) retention_scan_kernel(RetArgs a) {
  extern __shared__ float sm[];        // S [dk][slice], q [dk], k [dk], shares [RS][slice]
  const int e = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, dk = a.dk, dv = a.dv, half = a.half, W = a.slice;
  const int row0 = a.cu_rows[e], row1 = a.cu_rows[e + 1];
  if (row1 - row0 < a.min_rows) return;
  const int RS = RT_THREADS / W, c = tid % W, rs = tid / W, col = blockIdx.z * W + c;
  float* S = sm;
  float* q = S + (size_t)dk * W;
  float* k = q + dk;
  float* share = k + dk;
  float* Sg = a.S + (size_t)a.entry_slot[e] * a.S_stride + (size_t)h * dk * dv;
  for (int r = rs; r < dk; r += RS) S[r * W + c] = col < dv ? Sg[(size_t)r * dv + col] : 0.f;
  const int items = half + (dk - 2 * half), gh = h / (a.H / a.G);
  const float rate = a.dsrc ? expf(a.A_log[h]) : 0.f;
  float d = a.dsrc ? 0.f : a.powers[(size_t)h * (RC + 1) + 1], ks = a.k_scale;
  for (int t = row0; t < row1; ++t) {
    const float* p = a.proj + (size_t)t * a.ld;
    const float* pq = p + a.q0 + (size_t)gh * dk;
    const float* pk = p + a.k0 + (size_t)gh * dk;
    if (a.dsrc) {
      ks = step_size_of(a, t, h);
      d = expf(-rate * ks);
    }
    for (int i = tid; i < items; i += RT_THREADS) {
      if (i < half) {
        const float2 cs = a.table[(size_t)t * half + i];
        q[i] = pq[i] * cs.x - pq[i + half] * cs.y;
        q[i + half] = pq[i + half] * cs.x + pq[i] * cs.y;
        k[i] = (pk[i] * cs.x - pk[i + half] * cs.y) * ks;
        k[i + half] = (pk[i + half] * cs.x + pk[i] * cs.y) * ks;
      } else {
        q[i + half] = pq[i + half];
        k[i + half] = pk[i + half] * ks;
      }
    }
    __syncthreads();
    const float v = col < dv ? p[a.v0 + (size_t)h * dv + col] : 0.f;
    float o = 0.f;
    for (int r = rs; r < dk; r += RS) {
      const float s = fmaf(d, S[r * W + c], k[r] * v);
      S[r * W + c] = s;
      o = fmaf(s, q[r], o);
    }
    share[rs * W + c] = o;
    __syncthreads();
    if (rs == 0 && col < dv) {
      float sum = 0.f;
      for (int i = 0; i < RS; ++i) sum += share[i * W + c];
      a.raw[((size_t)t * a.H + h) * dv + col] = sum;
    }
  }
  if (col < dv)
    for (int r = rs; r < dk; r += RS) Sg[(size_t)r * dv + col] = S[r * W + c];
}

// A row and head per warp: y = o / sqrt(mean(o^2) + eps) * silu(gate), for the rows of entries with min_rows or more.
__global__ void __launch_bounds__(256) retention_finish_kernel(RetArgs a, int T) {
  const int lane = threadIdx.x & 31;
  const long long item = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (item >= (long long)T * a.H) return;
  const int t = (int)(item / a.H), h = (int)(item % a.H), dv = a.dv;
  const int e = a.row_entry[t];
  if (a.cu_rows[e + 1] - a.cu_rows[e] < a.min_rows) return;
  const float* x = a.raw + (size_t)item * dv;
  float ss = 0.f;
  for (int i = lane; i < dv; i += 32) ss = fmaf(x[i], x[i], ss);
  const float r = rsqrtf(warp_sum(ss) / (float)dv + a.eps);
  for (int i = lane; i < dv; i += 32)
    st_dt(a.out, a.out_dt, (size_t)item * dv + i, x[i] * r * silu_of(a.proj[(size_t)t * a.ld + a.g0 + (size_t)h * dv + i]));
}

// ------------------------------------------------------------------ the chunked form
constexpr int CK_THREADS = 256, CK_WARPS = CK_THREADS / 32;
constexpr int VLD = 64 + 8;            // row of a 64-column slab in shared memory (sixteen bytes of padding)
constexpr int CK_HEADS = 4;            // most heads that a block takes one after the other (they share q and k)

__device__ __forceinline__ uint32_t s_u32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(s_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void ldsm4(const bf16* p, uint32_t* r) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(s_u32(p)));
}
__device__ __forceinline__ void ldsm4_t(const bf16* p, uint32_t* r) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(s_u32(p)));
}
__device__ __forceinline__ void mma16816(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// Two floats as packed bfloat16 pairs: their roundings, and the roundings of what those left.
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const __nv_bfloat162 l = __floats2bfloat162_rn(x - __bfloat162float(h.x), y - __bfloat162float(h.y));
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}
__device__ __forceinline__ void split1(float x, bf16* hi, bf16* lo) {
  const bf16 h = __float2bfloat16_rn(x);
  *hi = h;
  *lo = __float2bfloat16_rn(x - __bfloat162float(h));
}
// c += a b for operands in two terms each (the product of the two small terms is left out)
__device__ __forceinline__ void mma_terms(float* c, const uint32_t* ah, const uint32_t* al, uint32_t bh0, uint32_t bh1,
                                          uint32_t bl0, uint32_t bl1) {
  mma16816(c, ah, bh0, bh1);
  mma16816(c, ah, bl0, bl1);
  mma16816(c, al, bh0, bh1);
}

// Which (entry, chunk of it) is chunk number `want` of the step?  Entries with fewer than min_rows rows have none.
// Called by warp 0; info: entry (-1: none), first row in the batch, rows.
__device__ __forceinline__ void find_chunk(const int* cu_rows, int S, int min_rows, int want, int* info) {
  const int lane = threadIdx.x & 31;
  int base = 0;
  for (int b = 0; b < S; b += 32) {
    const int e = b + lane;
    const int n = e < S ? cu_rows[e + 1] - cu_rows[e] : 0;
    const int mine = n >= min_rows ? (n + RC - 1) / RC : 0;
    int inc = mine;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int up = __shfl_up_sync(0xffffffffu, inc, o);
      if (lane >= o) inc += up;
    }
    const int total = __shfl_sync(0xffffffffu, inc, 31);
    if (want < base + total) {
      if (base + inc > want && base + inc - mine <= want) {
        const int at = want - (base + inc - mine);
        info[0] = e;
        info[1] = cu_rows[e] + at * RC;
        info[2] = min(RC, n - at * RC);
      }
      return;
    }
    base += total;
  }
  if (lane == 0) info[0] = -1;
}

// Row decays of a chunk, worked out by a warp: lane l has rows i = 2 l and i + 1, d[] their step sizes, c[] the base-2 logarithm
// of the product of the decays of rows 0 .. i (and i + 1).  Rows beyond n neither decay nor count.
__device__ __forceinline__ void chunk_row_decays(const RetArgs& a, int h, int row0, int n, float (&c)[2], float (&d)[2]) {
  const int lane = threadIdx.x & 31, i = 2 * lane;
  const float rate2 = expf(a.A_log[h]) * 1.4426950408889634f;
  d[0] = i < n ? step_size_of(a, row0 + i, h) : 0.f;
  d[1] = i + 1 < n ? step_size_of(a, row0 + i + 1, h) : 0.f;
  const float l0 = -rate2 * d[0], l1 = -rate2 * d[1];
  float inc = l0 + l1;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float up = __shfl_up_sync(0xffffffffu, inc, o);
    if (lane >= o) inc += up;
  }
  const float before = __shfl_up_sync(0xffffffffu, inc, 1);
  c[0] = (lane ? before : 0.f) + l0;
  c[1] = c[0] + l1;
}

// Rows row0 .. row0 + n - 1 of one q or k head, turned, as two bfloat16 terms in shared memory
// [RC][LDS]; rows beyond n and elements beyond dk are zero.
template <int DKP>
__device__ __forceinline__ void load_turned(const RetArgs& a, const float* src, int row0, int n, bf16* hi, bf16* lo) {
  constexpr int LDS = DKP + 8;
  const int half = a.half, dk = a.dk, tid = threadIdx.x;
  if (a.v2) {
    // Two neighbouring elements at a time (sizes and addresses are even): a warp takes every eighth row, its lanes the
    // row's elements side by side, and the loads of four rows are in flight before the first is used.
    const int h2 = half / 2, items = h2 + (dk - 2 * half) / 2, lane = tid & 31, warp = tid >> 5;
    constexpr int B = 4;
    for (int i = lane; i < items; i += 32) {
      const bool turned = i < h2;
      const int d = turned ? 2 * i : 2 * half + 2 * (i - h2);
      for (int r0 = warp; r0 < RC; r0 += CK_WARPS * B) {
        float2 u[B], w[B];
        float4 cs[B];
#pragma unroll
        for (int b = 0; b < B; ++b) {
          const int r = r0 + CK_WARPS * b;
          u[b] = w[b] = make_float2(0.f, 0.f);
          cs[b] = make_float4(1.f, 0.f, 1.f, 0.f);
          if (r < n) {
            const float* p = src + (size_t)(row0 + r) * a.ld + d;
            u[b] = *reinterpret_cast<const float2*>(p);
            if (turned) {
              w[b] = *reinterpret_cast<const float2*>(p + half);
              cs[b] = *reinterpret_cast<const float4*>(a.table + (size_t)(row0 + r) * half + 2 * i);
            }
          }
        }
#pragma unroll
        for (int b = 0; b < B; ++b) {
          const int r = r0 + CK_WARPS * b;
          uint32_t wh, wl;
          split2(u[b].x * cs[b].x - w[b].x * cs[b].y, u[b].y * cs[b].z - w[b].y * cs[b].w, wh, wl);
          *reinterpret_cast<uint32_t*>(hi + r * LDS + d) = wh;
          *reinterpret_cast<uint32_t*>(lo + r * LDS + d) = wl;
          if (turned) {
            split2(w[b].x * cs[b].x + u[b].x * cs[b].y, w[b].y * cs[b].z + u[b].y * cs[b].w, wh, wl);
            *reinterpret_cast<uint32_t*>(hi + r * LDS + d + half) = wh;
            *reinterpret_cast<uint32_t*>(lo + r * LDS + d + half) = wl;
          }
        }
      }
    }
  } else {
    const int items = half + (dk - 2 * half);
    for (int x = tid; x < RC * items; x += CK_THREADS) {
      const int r = x / items, i = x - r * items;
      const bool live = r < n;
      const float* p = src + (size_t)(row0 + (live ? r : 0)) * a.ld;
      if (i < half) {
        const float2 cs = a.table[(size_t)(row0 + (live ? r : 0)) * half + i];
        const float u = p[i], w = p[i + half];
        split1(live ? u * cs.x - w * cs.y : 0.f, hi + r * LDS + i, lo + r * LDS + i);
        split1(live ? w * cs.x + u * cs.y : 0.f, hi + r * LDS + i + half, lo + r * LDS + i + half);
      } else {
        split1(live ? p[i + half] : 0.f, hi + r * LDS + i + half, lo + r * LDS + i + half);
      }
    }
  }
  const int pad = DKP - dk;
  for (int x = tid; x < RC * pad; x += CK_THREADS) {
    const int i = (x / pad) * LDS + dk + x % pad;
    hi[i] = lo[i] = __float2bfloat16_rn(0.f);
  }
}

// Columns c0 .. c0 + 63 of a value head of the chunk's rows, every row times weight[row] (nullptr: as it is), as two terms
// [RC][VLD]; what does not exist is zero.  Where pairs can be read (v2) a thread fetches its values into registers first,
// which may happen while the block still works on the slab before.
constexpr int VREGS = RC / CK_WARPS;
struct ValueRegs { float2 v[VREGS]; };
__device__ __forceinline__ void fetch_values(const RetArgs& a, const float* src, int row0, int n, int c0, ValueRegs& x) {
  if (!a.v2) return;
  const int c = 2 * (threadIdx.x & 31);
  const bool col = c0 + c < a.dv;
#pragma unroll
  for (int b = 0; b < VREGS; ++b) {
    const int r = (threadIdx.x >> 5) + CK_WARPS * b;
    x.v[b] = make_float2(0.f, 0.f);
    if (r < n && col) x.v[b] = *reinterpret_cast<const float2*>(src + (size_t)(row0 + r) * a.ld + c0 + c);
  }
}
__device__ __forceinline__ void store_values(const RetArgs& a, const float* src, int row0, int n, int c0, const ValueRegs& x,
                                             const float* weight, bf16* hi, bf16* lo) {
  if (a.v2) {
    const int c = 2 * (threadIdx.x & 31);
#pragma unroll
    for (int b = 0; b < VREGS; ++b) {
      const int r = (threadIdx.x >> 5) + CK_WARPS * b;
      const float f = weight ? weight[r] : 1.f;
      uint32_t wh, wl;
      split2(x.v[b].x * f, x.v[b].y * f, wh, wl);
      *reinterpret_cast<uint32_t*>(hi + r * VLD + c) = wh;
      *reinterpret_cast<uint32_t*>(lo + r * VLD + c) = wl;
    }
  } else {
    for (int x2 = threadIdx.x; x2 < RC * 64; x2 += CK_THREADS) {
      const int r = x2 / 64, c = x2 % 64;
      const float v = r < n && c0 + c < a.dv ? src[(size_t)(row0 + r) * a.ld + c0 + c] : 0.f;
      split1(weight ? v * weight[r] : v, hi + r * VLD + c, lo + r * VLD + c);
    }
  }
}

// Every chunk's own sum: U = sum_j d^(n-1-j) k_j v_j^T, float32 [dk][dv].  grid (chunks, heads / hb): a block takes hb heads
// with the same k, whose terms are made once; what a row counts for multiplies its value.
template <int DKP, bool VAR>
__global__ void __launch_bounds__(CK_THREADS, DKP <= 128 ? 3 : 1) retention_chunk_sum_kernel(RetArgs a) {
  constexpr int LDS = DKP + 8;
  extern __shared__ __align__(16) uint8_t ck_smem[];
  bf16* kh = (bf16*)ck_smem;
  bf16* kl = kh + RC * LDS;
  bf16* vh = kl + RC * LDS;
  bf16* vl = vh + RC * VLD;
  __shared__ int info[3];
  __shared__ float counts[CK_HEADS][RC];
  const int h0 = blockIdx.y * a.hb, gh = h0 / (a.H / a.G), tid = threadIdx.x, warp = tid / 32, lane = tid % 32;
  grid_dep_wait();
  grid_dep_launch();
  if (warp == 0) find_chunk(a.cu_rows, a.num_entries, a.min_rows, blockIdx.x, info);
  __syncthreads();
  if (info[0] < 0) return;
  const int row0 = info[1], n = info[2];
  ValueRegs next;
  fetch_values(a, a.proj + a.v0 + (size_t)h0 * a.dv, row0, n, 0, next);
  if (VAR) {
    if (warp < a.hb) {
      float c[2], d[2];
      chunk_row_decays(a, h0 + warp, row0, n, c, d);
      const float total = __shfl_sync(0xffffffffu, c[1], 31);        // (rows beyond n add nothing)
      counts[warp][2 * lane] = exp2f(total - c[0]) * d[0];
      counts[warp][2 * lane + 1] = exp2f(total - c[1]) * d[1];
      if (lane == 0) a.chunk_decay[(size_t)blockIdx.x * a.H + h0 + warp] = exp2f(total);
    }
  } else {
    for (int i = tid; i < a.hb * RC; i += CK_THREADS) {
      const int r = i % RC;
      counts[i / RC][r] = r < n ? a.powers[(size_t)(h0 + i / RC) * (RC + 1) + n - 1 - r] * a.k_scale : 0.f;
    }
  }
  load_turned<DKP>(a, a.proj + a.k0 + (size_t)gh * a.dk, row0, n, kh, kl);
  __syncthreads();
  const int g = lane / 4, tq = lane % 4;
  const bool even = (a.dv & 1) == 0;
  const int slabs = (a.dv + 63) / 64;
  for (int step = 0; step < a.hb * slabs; ++step) {
    const int hh = step / slabs, c0 = (step % slabs) * 64;
    float* U = reinterpret_cast<float*>(a.chunks) + ((size_t)blockIdx.x * a.H + h0 + hh) * a.dk * a.dv;
    if (step) __syncthreads();
    store_values(a, a.proj + a.v0 + (size_t)(h0 + hh) * a.dv, row0, n, c0, next, counts[hh], vh, vl);
    __syncthreads();
    if (step + 1 < a.hb * slabs)
      fetch_values(a, a.proj + a.v0 + (size_t)(h0 + (step + 1) / slabs) * a.dv, row0, n, ((step + 1) % slabs) * 64, next);
    // an item of work is sixteen rows and 32 columns of U
    for (int item = warp; item < DKP / 8; item += CK_WARPS) {
      const int d0 = (item >> 1) * 16, n0 = (item & 1) * 32;
      if (d0 >= a.dk || c0 + n0 >= a.dv) continue;
      float c[4][4];
#pragma unroll
      for (int i = 0; i < 4; ++i) c[i][0] = c[i][1] = c[i][2] = c[i][3] = 0.f;
#pragma unroll
      for (int kb = 0; kb < RC / 16; ++kb) {
        if (kb * 16 >= n) continue;
        uint32_t ah[4], al[4];
        const int at = (kb * 16 + (lane % 8) + 8 * (lane / 16)) * LDS + d0 + 8 * ((lane / 8) % 2);
        ldsm4_t(kh + at, ah);
        ldsm4_t(kl + at, al);
#pragma unroll
        for (int np = 0; np < 2; ++np) {
          uint32_t bh[4], bl[4];
          const int bt = (kb * 16 + (lane % 8) + 8 * ((lane / 8) % 2)) * VLD + n0 + np * 16 + 8 * (lane / 16);
          ldsm4_t(vh + bt, bh);
          ldsm4_t(vl + bt, bl);
          mma_terms(c[2 * np], ah, al, bh[0], bh[1], bl[0], bl[1]);
          mma_terms(c[2 * np + 1], ah, al, bh[2], bh[3], bl[2], bl[3]);
        }
      }
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int col = c0 + n0 + i * 8 + 2 * tq;
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int d = d0 + g + 8 * half;
          if (d >= a.dk || col >= a.dv) continue;
          float* p = U + (size_t)d * a.dv + col;
          if (even) *reinterpret_cast<float2*>(p) = make_float2(c[i][2 * half], c[i][2 * half + 1]);
          else {
            p[0] = c[i][2 * half];
            if (col + 1 < a.dv) p[1] = c[i][2 * half + 1];
          }
        }
      }
    }
  }
}

// Chunks of the entries before entry e, worked out by warp 0.
__device__ __forceinline__ void count_chunks_before(const int* cu_rows, int e, int min_rows, int* first) {
  if (threadIdx.x < 32) {
    int sum = 0;
    for (int i = threadIdx.x; i < e; i += 32) {
      const int m = cu_rows[i + 1] - cu_rows[i];
      sum += m >= min_rows ? (m + RC - 1) / RC : 0;
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
    if (threadIdx.x == 0) *first = sum;
  }
  __syncthreads();
}

// Turns an entry's chunk sums into the states its chunks start from, in place, and leaves the last state in the request's
// slot.  Here every row of a state becomes the row's leading terms [dv bfloat16] and behind them its rest terms
// [dv bfloat16], which the next kernel copies as they are.  A row is LPR lanes' (four columns each, NJ times): 32, or 16
// where a row has no more than 64 columns; all of a row's sums are read before its terms are written over them.  grid
// (entries, heads, rows / (256 / LPR)).
template <int NJ, int LPR>
__global__ void __launch_bounds__(256) retention_chunk_pass_rows_kernel(RetArgs a) {
  __shared__ int first_s;
  const int e = blockIdx.x, h = blockIdx.y, lane = threadIdx.x % LPR;
  grid_dep_wait();
  grid_dep_launch();
  const int n = a.cu_rows[e + 1] - a.cu_rows[e];
  if (n < a.min_rows) return;
  count_chunks_before(a.cu_rows, e, a.min_rows, &first_s);
  const int d = blockIdx.z * (256 / LPR) + threadIdx.x / LPR;
  const unsigned lanes = __ballot_sync(0xffffffffu, d < a.dk);
  if (d >= a.dk) return;
  const int count = (n + RC - 1) / RC, dv = a.dv;
  const size_t size = (size_t)a.dk * dv, step = (size_t)a.H * size;
  uint32_t* p = a.chunks + ((size_t)first_s * a.H + h) * size + (size_t)d * dv;
  float* Sg = a.S + (size_t)a.entry_slot[e] * a.S_stride + (size_t)h * size + (size_t)d * dv;
  const bool var = a.chunk_decay != nullptr;
  const float full = var ? 0.f : a.powers[(size_t)h * (RC + 1) + RC];
  const float last = var ? 0.f : a.powers[(size_t)h * (RC + 1) + n - (count - 1) * RC];
  const float* dec = a.chunk_decay + (size_t)first_s * a.H + h;
  Vals<4> S[NJ];
#pragma unroll
  for (int j = 0; j < NJ; ++j)
    if (4 * (lane + LPR * j) < dv) S[j] = ldv<4>(Sg + 4 * (lane + LPR * j));
  constexpr int U = 8 / NJ;            // chunk sums in flight
  for (int c0 = 0; c0 < count; c0 += U) {
    Vals<4> u[U][NJ];
#pragma unroll
    for (int i = 0; i < U; ++i)
#pragma unroll
      for (int j = 0; j < NJ; ++j)
        if (c0 + i < count && 4 * (lane + LPR * j) < dv)
          u[i][j] = ldv<4>(reinterpret_cast<const float*>(p) + (size_t)(c0 + i) * step + 4 * (lane + LPR * j));
    __syncwarp(lanes);                 // the row's sums have been read by all lanes
#pragma unroll
    for (int i = 0; i < U; ++i)
      if (c0 + i < count) {
        const float f = var ? dec[(size_t)(c0 + i) * a.H] : (c0 + i + 1 < count ? full : last);
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
          const int c = 4 * (lane + LPR * j);
          if (c >= dv) continue;
          uint2 hi, lo;
          split2(S[j].v[0], S[j].v[1], hi.x, lo.x);
          split2(S[j].v[2], S[j].v[3], hi.y, lo.y);
          bf16* row = reinterpret_cast<bf16*>(p + (size_t)(c0 + i) * step);
          *reinterpret_cast<uint2*>(row + c) = hi;
          *reinterpret_cast<uint2*>(row + dv + c) = lo;
#pragma unroll
          for (int x = 0; x < 4; ++x) S[j].v[x] = fmaf(f, S[j].v[x], u[i][j].v[x]);
        }
      }
  }
#pragma unroll
  for (int j = 0; j < NJ; ++j)
    if (4 * (lane + LPR * j) < dv) stv<4>(Sg + 4 * (lane + LPR * j), S[j]);
}

// The same for other sizes: an element's two terms are packed in one word (the same thread reads and writes an element).
// grid (entries, heads, elements / 256).
__global__ void __launch_bounds__(256) retention_chunk_pass_kernel(RetArgs a) {
  __shared__ int first_s;
  const int e = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
  grid_dep_wait();
  grid_dep_launch();
  const int n = a.cu_rows[e + 1] - a.cu_rows[e];
  if (n < a.min_rows) return;
  count_chunks_before(a.cu_rows, e, a.min_rows, &first_s);
  const int i = blockIdx.z * 256 + tid, size = a.dk * a.dv;
  if (i >= size) return;
  const int count = (n + RC - 1) / RC;
  const size_t step = (size_t)a.H * size;
  uint32_t* p = a.chunks + ((size_t)first_s * a.H + h) * size + i;
  float* Sg = a.S + (size_t)a.entry_slot[e] * a.S_stride + (size_t)h * size + i;
  const bool var = a.chunk_decay != nullptr;
  const float full = var ? 0.f : a.powers[(size_t)h * (RC + 1) + RC];
  const float last = var ? 0.f : a.powers[(size_t)h * (RC + 1) + n - (count - 1) * RC];
  const float* dec = a.chunk_decay + (size_t)first_s * a.H + h;
  float S = *Sg;
  constexpr int U = 8;                 // chunk sums in flight
  for (int c0 = 0; c0 < count; c0 += U) {
    float u[U];
#pragma unroll
    for (int j = 0; j < U; ++j) u[j] = c0 + j < count ? __uint_as_float(p[(size_t)(c0 + j) * step]) : 0.f;
#pragma unroll
    for (int j = 0; j < U; ++j)
      if (c0 + j < count) {
        const bf16 hi = __float2bfloat16_rn(S);
        const __nv_bfloat162 pk = __halves2bfloat162(hi, __float2bfloat16_rn(S - __bfloat162float(hi)));
        p[(size_t)(c0 + j) * step] = *reinterpret_cast<const uint32_t*>(&pk);
        S = fmaf(var ? dec[(size_t)(c0 + j) * a.H] : (c0 + j + 1 < count ? full : last), S, u[j]);
      }
  }
  *Sg = S;
}

__device__ __forceinline__ float silu_fast(float x) { return __fdividef(x, 1.f + __expf(-x)); }

// Every chunk's outputs, its heads normed and gated (or as they are, raw_out).  grid (chunks, heads / hb): a block takes hb
// heads with the same q and k one after the other; their products q . k are made once.  Two warps share sixteen rows: each
// takes half of the keys for the weights, which both then read from shared memory, and half of every slab's columns.  NS:
// slabs of 64 value columns.
template <int DKP, int NS, bool VAR>
__global__ void __launch_bounds__(CK_THREADS, DKP <= 128 && NS <= 2 ? 2 : 1) retention_chunk_out_kernel(RetArgs a) {
  constexpr int LDS = DKP + 8;
  constexpr int KS = RC * LDS > DKP * VLD ? RC * LDS : DKP * VLD;      // the keys' place is the state's afterwards
  extern __shared__ __align__(16) uint8_t ck_smem[];
  bf16* qh = (bf16*)ck_smem;
  bf16* ql = qh + RC * LDS;
  bf16* kh = ql + RC * LDS;
  bf16* kl = kh + KS;
  bf16* vh = kl + KS;
  bf16* vl = vh + RC * VLD;
  bf16* ph = vl + RC * VLD;            // the weights, two terms [RC][VLD]
  bf16* pl = ph + RC * VLD;
  __shared__ float squares[2][RC];
  __shared__ int info[3];
  // per head: the powers of the decay; with row decays their running logarithms, and the rows' step sizes
  __shared__ float pws[CK_HEADS][RC + 1], dts[VAR ? CK_HEADS : 1][RC];
  const int h0 = blockIdx.y * a.hb, gh = h0 / (a.H / a.G), tid = threadIdx.x, warp = tid / 32, lane = tid % 32;
  grid_dep_wait();
  grid_dep_launch();
  if (warp == 0) find_chunk(a.cu_rows, a.num_entries, a.min_rows, blockIdx.x, info);
  __syncthreads();
  if (info[0] < 0) return;
  const int row0 = info[1], n = info[2];
  if (VAR) {
    if (warp < a.hb) {
      float c[2], d[2];
      chunk_row_decays(a, h0 + warp, row0, n, c, d);
      pws[warp][2 * lane] = c[0];
      pws[warp][2 * lane + 1] = c[1];
      dts[VAR ? warp : 0][2 * lane] = d[0];
      dts[VAR ? warp : 0][2 * lane + 1] = d[1];
    }
  } else {
    for (int i = tid; i < a.hb * (RC + 1); i += CK_THREADS) pws[i / (RC + 1)][i % (RC + 1)] = a.powers[(size_t)h0 * (RC + 1) + i];
  }
  load_turned<DKP>(a, a.proj + a.q0 + (size_t)gh * a.dk, row0, n, qh, ql);
  load_turned<DKP>(a, a.proj + a.k0 + (size_t)gh * a.dk, row0, n, kh, kl);
  ValueRegs next;
  fetch_values(a, a.proj + a.v0 + (size_t)h0 * a.dv, row0, n, 0, next);
  __syncthreads();
  const int g = lane / 4, tq = lane % 4;
  const int rb = warp >> 1, side = warp & 1;         // rows 16 rb .. 16 rb + 15; which half of the keys and columns
  const int r_lo = rb * 16 + g, r_hi = r_lo + 8;
  const int q_at = (rb * 16 + (lane % 8) + 8 * ((lane / 8) % 2)) * LDS + 8 * (lane / 16);
  const bool busy = rb * 16 < n;

  // q_i . k_j of these rows and this warp's 32 keys
  float s[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
  if (busy && 2 * side <= rb) {
#pragma unroll
    for (int kk = 0; kk < DKP / 16; ++kk) {
      uint32_t ah[4], al[4];
      ldsm4(qh + q_at + kk * 16, ah);
      ldsm4(ql + q_at + kk * 16, al);
#pragma unroll
      for (int np = 0; np < 2; ++np) {
        if (2 * side + np > rb) continue;          // keys after these rows
        uint32_t bh[4], bl[4];
        const int at = ((2 * side + np) * 16 + (lane % 8) + 8 * (lane / 16)) * LDS + kk * 16 + 8 * ((lane / 8) % 2);
        ldsm4(kh + at, bh);
        ldsm4(kl + at, bl);
        mma_terms(s[2 * np], ah, al, bh[0], bh[1], bl[0], bl[1]);
        mma_terms(s[2 * np + 1], ah, al, bh[2], bh[3], bl[2], bl[3]);
      }
    }
  }
  for (int hh = 0; hh < a.hb; ++hh) {
    const int h = h0 + hh;
    const float* pw = pws[hh];
    const float* dt = dts[VAR ? hh : 0];
    const uint32_t* St = a.chunks + ((size_t)blockIdx.x * a.H + h) * a.dk * a.dv;
    const float f_lo = VAR ? exp2f(pw[r_lo]) : pw[r_lo + 1], f_hi = VAR ? exp2f(pw[r_hi]) : pw[r_hi + 1];
    float o[NS][4][4];
    float ss_lo = 0.f, ss_hi = 0.f;
#pragma unroll
    for (int sl = 0; sl < NS; ++sl) {
      const int c0 = sl * 64;
      __syncthreads();                               // the keys (or the last slab, the last weights) have been read by everyone
      if (sl == 0) {                                 // the weights d^(i-j) (q_i . k_j), as two terms
        auto weight = [&](float qk, int r, int from) {
          if (from > r) return 0.f;
          return VAR ? qk * exp2f(pw[r] - pw[from]) * dt[VAR ? from : 0] : qk * pw[r - from] * a.k_scale;
        };
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int j = side * 32 + i * 8 + 2 * tq;
          uint32_t wh, wl;
          split2(weight(s[i][0], r_lo, j), weight(s[i][1], r_lo, j + 1), wh, wl);
          *reinterpret_cast<uint32_t*>(ph + r_lo * VLD + j) = wh;
          *reinterpret_cast<uint32_t*>(pl + r_lo * VLD + j) = wl;
          split2(weight(s[i][2], r_hi, j), weight(s[i][3], r_hi, j + 1), wh, wl);
          *reinterpret_cast<uint32_t*>(ph + r_hi * VLD + j) = wh;
          *reinterpret_cast<uint32_t*>(pl + r_hi * VLD + j) = wl;
        }
      }
      if (a.planes) {                                // the state's terms as they are, sixteen bytes at a time
#pragma unroll 4
        for (int x = tid; x < DKP * 16; x += CK_THREADS) {
          const int d = x >> 4, c = 8 * (x & 7), term = (x >> 3) & 1;
          bf16* dst = (term ? kl : kh) + d * VLD + c;
          if (d < a.dk && c0 + c < a.dv)
            cp_async16(dst, reinterpret_cast<const bf16*>(St + (size_t)d * a.dv) + term * a.dv + c0 + c);
          else *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
      }
      store_values(a, a.proj + a.v0 + (size_t)h * a.dv, row0, n, c0, next, nullptr, vh, vl);
      {
        const int more = hh * NS + sl + 1;           // the next slab's values are on their way while this one is worked on
        if (more < a.hb * NS) fetch_values(a, a.proj + a.v0 + (size_t)(h0 + more / NS) * a.dv, row0, n, (more % NS) * 64, next);
      }
      if (a.planes) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
      } else {
        for (int x = tid; x < DKP * 64; x += CK_THREADS) {
          const int d = x / 64, c = x % 64;
          const uint32_t w = d < a.dk && c0 + c < a.dv ? St[(size_t)d * a.dv + c0 + c] : 0u;
          const __nv_bfloat162 pk = *reinterpret_cast<const __nv_bfloat162*>(&w);
          kh[d * VLD + c] = pk.x;
          kl[d * VLD + c] = pk.y;
        }
      }
      __syncthreads();
      float (&oc)[4][4] = o[sl];
#pragma unroll
      for (int i = 0; i < 4; ++i) oc[i][0] = oc[i][1] = oc[i][2] = oc[i][3] = 0.f;
      if (!busy || c0 + side * 32 >= a.dv) continue;
#pragma unroll
      for (int kk = 0; kk < DKP / 16; ++kk) {
        if (kk * 16 >= a.dk) continue;
        uint32_t ah[4], al[4];
        ldsm4(qh + q_at + kk * 16, ah);
        ldsm4(ql + q_at + kk * 16, al);
#pragma unroll
        for (int np = 0; np < 2; ++np) {
          uint32_t bh[4], bl[4];
          const int at = (kk * 16 + (lane % 8) + 8 * ((lane / 8) % 2)) * VLD + side * 32 + np * 16 + 8 * (lane / 16);
          ldsm4_t(kh + at, bh);
          ldsm4_t(kl + at, bl);
          mma_terms(oc[2 * np], ah, al, bh[0], bh[1], bl[0], bl[1]);
          mma_terms(oc[2 * np + 1], ah, al, bh[2], bh[3], bl[2], bl[3]);
        }
      }
#pragma unroll
      for (int i = 0; i < 4; ++i) { oc[i][0] *= f_lo; oc[i][1] *= f_lo; oc[i][2] *= f_hi; oc[i][3] *= f_hi; }
#pragma unroll
      for (int kb = 0; kb < 4; ++kb) {
        if (kb > rb) continue;
        uint32_t ah[4], al[4];
        const int pat = (rb * 16 + (lane % 8) + 8 * ((lane / 8) % 2)) * VLD + kb * 16 + 8 * (lane / 16);
        ldsm4(ph + pat, ah);
        ldsm4(pl + pat, al);
#pragma unroll
        for (int np = 0; np < 2; ++np) {
          uint32_t bh[4], bl[4];
          const int at = (kb * 16 + (lane % 8) + 8 * ((lane / 8) % 2)) * VLD + side * 32 + np * 16 + 8 * (lane / 16);
          ldsm4_t(vh + at, bh);
          ldsm4_t(vl + at, bl);
          mma_terms(oc[2 * np], ah, al, bh[0], bh[1], bl[0], bl[1]);
          mma_terms(oc[2 * np + 1], ah, al, bh[2], bh[3], bl[2], bl[3]);
        }
      }
#pragma unroll
      for (int i = 0; i < 4; ++i) {                  // (columns beyond dv are zero)
        ss_lo = fmaf(oc[i][0], oc[i][0], fmaf(oc[i][1], oc[i][1], ss_lo));
        ss_hi = fmaf(oc[i][2], oc[i][2], fmaf(oc[i][3], oc[i][3], ss_hi));
      }
    }
    if (a.raw_out) {
#pragma unroll
      for (int sl = 0; sl < NS; ++sl)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int r = half ? r_hi : r_lo;
          if (r >= n) continue;
          float* to = a.raw + ((size_t)(row0 + r) * a.H + h) * a.dv;
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const int col = sl * 64 + side * 32 + i * 8 + 2 * tq;
            if (col >= a.dv) continue;
            if (a.v2) *reinterpret_cast<float2*>(to + col) = make_float2(o[sl][i][2 * half], o[sl][i][2 * half + 1]);
            else {
              to[col] = o[sl][i][2 * half];
              if (col + 1 < a.dv) to[col + 1] = o[sl][i][2 * half + 1];
            }
          }
        }
      continue;
    }
    ss_lo += __shfl_xor_sync(0xffffffffu, ss_lo, 1);
    ss_lo += __shfl_xor_sync(0xffffffffu, ss_lo, 2);
    ss_hi += __shfl_xor_sync(0xffffffffu, ss_hi, 1);
    ss_hi += __shfl_xor_sync(0xffffffffu, ss_hi, 2);
    if (tq == 0) {
      squares[side][r_lo] = ss_lo;
      squares[side][r_hi] = ss_hi;
    }
    __syncthreads();
    const float n_lo = rsqrtf((squares[0][r_lo] + squares[1][r_lo]) / (float)a.dv + a.eps);
    const float n_hi = rsqrtf((squares[0][r_hi] + squares[1][r_hi]) / (float)a.dv + a.eps);
#pragma unroll
    for (int sl = 0; sl < NS; ++sl)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int r = half ? r_hi : r_lo;
        if (r >= n) continue;
        const float rn = half ? n_hi : n_lo;
        const float* gp = a.proj + (size_t)(row0 + r) * a.ld + a.g0 + (size_t)h * a.dv;
        const size_t at = ((size_t)(row0 + r) * a.H + h) * a.dv;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int col = sl * 64 + side * 32 + i * 8 + 2 * tq;
          if (col >= a.dv) continue;
          const float x = o[sl][i][2 * half] * rn, y = o[sl][i][2 * half + 1] * rn;
          if (a.v2 && a.out_dt == NV_DT_BF16) {
            const float2 gg = *reinterpret_cast<const float2*>(gp + col);
            *reinterpret_cast<__nv_bfloat162*>((bf16*)a.out + at + col) = __floats2bfloat162_rn(x * silu_fast(gg.x), y * silu_fast(gg.y));
          } else {
            st_dt(a.out, a.out_dt, at + col, x * silu_fast(gp[col]));
            if (col + 1 < a.dv) st_dt(a.out, a.out_dt, at + col + 1, y * silu_fast(gp[col + 1]));
          }
        }
      }
  }
}

// ------------------------------------------------------------------ the row of all heads: skip, gate, norm
struct GatedNormArgs {
  const float* raw;         // [T, n]
  const float* skip;        // [H] or nullptr: y += skip[h] * x[t, c]
  const float* x;           // [T, x_ld]
  long long x_ld;
  const float* gate;        // [T, gate_ld]
  long long gate_ld;
  const float* w;           // [n]
  void* out;                // [T, n]
  int out_dt, n, dv, parts, gate_first, head_chunks;   // head_chunks: a chunk's elements are all one head's
  float eps;
};

// gate_first: the parts of (o + skip x) silu(gate), each over its root mean square, times w; else the parts of o + skip x over
// their root mean square, times w sigmoid(gate).  One block per (row, part); a thread keeps its first GN_KEEP chunks in
// registers between the two passes and works further ones out again.  Sums in a fixed order.
constexpr int GN_THREADS = 256, GN_KEEP = 4;
template <int VEC>
__global__ void __launch_bounds__(GN_THREADS) gated_norm_kernel(GatedNormArgs a) {
  __shared__ float red[GN_THREADS / 32];
  const int t = blockIdx.x, tid = threadIdx.x, nt = blockDim.x;
  const int m = a.n / a.parts, base = blockIdx.y * m, chunks = m / VEC;
  grid_dep_wait();
  grid_dep_launch();
  const bool fast = a.out_dt == NV_DT_BF16;        // (the result is rounded to bfloat16)
  const float* raw = a.raw + (size_t)t * a.n + base;
  const float* gate = a.gate + (size_t)t * a.gate_ld + base;
  const float* x = a.x + (size_t)t * a.x_ld + base;
  auto value = [&](int c) {
    Vals<VEC> v = ldv<VEC>(raw + c * VEC);
    if (a.skip) {
      const Vals<VEC> xv = ldv<VEC>(x + c * VEC);
#pragma unroll
      for (int i = 0; i < VEC; ++i) v.v[i] = fmaf(a.skip[(base + c * VEC + (a.head_chunks ? 0 : i)) / a.dv], xv.v[i], v.v[i]);
    }
    if (a.gate_first) {
      const Vals<VEC> g = ldv<VEC>(gate + c * VEC);
#pragma unroll
      for (int i = 0; i < VEC; ++i) v.v[i] *= fast ? silu_fast(g.v[i]) : silu_of(g.v[i]);
    }
    return v;
  };
  Vals<VEC> keep[GN_KEEP];
  float ss = 0.f;
#pragma unroll
  for (int u = 0; u < GN_KEEP; ++u) {
    const int c = tid + u * nt;
    if (c < chunks) {
      keep[u] = value(c);
#pragma unroll
      for (int i = 0; i < VEC; ++i) ss = fmaf(keep[u].v[i], keep[u].v[i], ss);
    }
  }
  for (int c = tid + GN_KEEP * nt; c < chunks; c += nt) {
    const Vals<VEC> v = value(c);
#pragma unroll
    for (int i = 0; i < VEC; ++i) ss = fmaf(v.v[i], v.v[i], ss);
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  float sum = 0.f;
  for (int i = 0; i < nt / 32; ++i) sum += red[i];
  const float r = rsqrtf(sum / (float)m + a.eps);
  auto emit = [&](int c, Vals<VEC> v) {
    const Vals<VEC> wv = ldv<VEC>(a.w + base + c * VEC);
#pragma unroll
    for (int i = 0; i < VEC; ++i) v.v[i] = v.v[i] * r * wv.v[i];
    if (!a.gate_first) {
      const Vals<VEC> g = ldv<VEC>(gate + c * VEC);
#pragma unroll
      for (int i = 0; i < VEC; ++i) v.v[i] *= fast ? __fdividef(1.f, 1.f + __expf(-g.v[i])) : 1.f / (1.f + expf(-g.v[i]));
    }
    st_out<VEC>(a.out, a.out_dt, (size_t)t * a.n + base + (size_t)c * VEC, v);
  };
#pragma unroll
  for (int u = 0; u < GN_KEEP; ++u)
    if (tid + u * nt < chunks) emit(tid + u * nt, keep[u]);
  for (int c = tid + GN_KEEP * nt; c < chunks; c += nt) emit(c, value(c));
}

template <typename K>
int allow(K kernel, size_t bytes) {
  if (bytes > 227 * 1024) return NV_ERR_UNSUPPORTED;
  if (bytes > 40 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
    if (e != cudaSuccess) return (int)e;
  }
  return NV_OK;
}

int step_vec(int dv) { return dv % 4 == 0 ? 4 : 1; }

template <int DKP>
size_t chunk_sum_smem() { return sizeof(bf16) * (2 * (size_t)RC * (DKP + 8) + 2 * (size_t)RC * VLD); }
template <int DKP>
size_t chunk_out_smem() {
  const size_t ks = std::max((size_t)RC * (DKP + 8), (size_t)DKP * VLD);
  return sizeof(bf16) * (2 * (size_t)RC * (DKP + 8) + 2 * ks + 4 * (size_t)RC * VLD);
}

template <int DKP, int NS, bool VAR>
int launch_chunks(const RetArgs& a, int max_chunks, cudaStream_t s) {
  int rc = allow(retention_chunk_sum_kernel<DKP, VAR>, chunk_sum_smem<DKP>());
  if (rc) return rc;
  rc = allow(retention_chunk_out_kernel<DKP, NS, VAR>, chunk_out_smem<DKP>());
  if (rc) return rc;
  const dim3 grid(max_chunks, a.H / a.hb);
  NV_RETURN_IF(launch_dep(retention_chunk_sum_kernel<DKP, VAR>, grid, dim3(CK_THREADS), chunk_sum_smem<DKP>(), s, a));
  const dim3 rows(a.num_entries, a.H, (a.dk + 7) / 8), rows2(a.num_entries, a.H, (a.dk + 15) / 16);
  if (a.planes && a.dv <= 64) NV_RETURN_IF(launch_dep(retention_chunk_pass_rows_kernel<1, 16>, rows2, dim3(256), 0, s, a));
  else if (a.planes && a.dv <= 128) NV_RETURN_IF(launch_dep(retention_chunk_pass_rows_kernel<1, 32>, rows, dim3(256), 0, s, a));
  else if (a.planes) NV_RETURN_IF(launch_dep(retention_chunk_pass_rows_kernel<2, 32>, rows, dim3(256), 0, s, a));
  else NV_RETURN_IF(launch_dep(retention_chunk_pass_kernel, dim3(a.num_entries, a.H, (a.dk * a.dv + 255) / 256), dim3(256), 0, s, a));
  NV_RETURN_IF(launch_dep(retention_chunk_out_kernel<DKP, NS, VAR>, grid, dim3(CK_THREADS), chunk_out_smem<DKP>(), s, a));
  NV_RETURN_LAST();
}

template <int DKP, bool VAR>
int launch_chunks_ns(const RetArgs& a, int max_chunks, cudaStream_t s) {
  if (a.dv <= 64) return launch_chunks<DKP, 1, VAR>(a, max_chunks, s);
  if (a.dv <= 128) return launch_chunks<DKP, 2, VAR>(a, max_chunks, s);
  return launch_chunks<DKP, 4, VAR>(a, max_chunks, s);
}
template <int DKP>
int launch_chunks_dk(const RetArgs& a, int max_chunks, cudaStream_t s) {
  return a.dsrc ? launch_chunks_ns<DKP, true>(a, max_chunks, s) : launch_chunks_ns<DKP, false>(a, max_chunks, s);
}

}  // namespace

// act 0: out = h + conv(h); act 1: out = silu(conv(h) + bias).  h: [T, H] float32, rows `ld` apart; w: [taps, H] float32;
// bias: [H] or nullptr; state: per slot [taps - 1, H] float32 (nullptr with one tap).  `update` (allowed where every entry
// of the step has one row): the state is brought up to date as well.
NV_API int nv_causal_conv(const float* h, long long ld, const float* w, const float* bias, int act, int taps,
                          const int* row_entry, const int* cu_rows, const int* entry_slot, float* state,
                          long long slot_stride, void* out, int out_dt, int T, int H, int update, cudaStream_t s) {
  if (!dt_ok(out_dt)) return NV_ERR_BAD_DTYPE;
  if (taps < 1 || H < 1 || ld < H || (taps > 1 && !state) || act < 0 || act > 1 || (bias && !act)) return NV_ERR_BAD_SIZE;
  if (T == 0) return NV_OK;
  ConvArgs a = {h, ld, w, bias, row_entry, cu_rows, entry_slot, state, slot_stride, out, out_dt, T, H, taps,
                T > 512 ? 8 : 1, update, act};
  const bool vec = H % 4 == 0 && ld % 4 == 0 && slot_stride % 4 == 0 && !((uintptr_t)bias & 15) && !((uintptr_t)h & 15) && !((uintptr_t)w & 15) && !((uintptr_t)state & 15)
                   && !((uintptr_t)out & 15);
  const int chunks = vec ? H / 4 : H;
  const int threads = chunks < 256 ? (chunks + 31) / 32 * 32 : 256;
  const dim3 grid((T + a.rows - 1) / a.rows, (chunks + threads - 1) / threads);
#define NV_CONV(VEC, TAPS) NV_RETURN_IF(launch_dep(causal_conv_kernel<VEC, TAPS>, grid, dim3(threads), 0, s, a))
#define NV_CONV_TAPS(VEC)            \
  switch (taps) {                    \
    case 2: NV_CONV(VEC, 2); break;  \
    case 3: NV_CONV(VEC, 3); break;  \
    case 4: NV_CONV(VEC, 4); break;  \
    default: NV_CONV(VEC, 0); break; \
  }
  if (vec) { NV_CONV_TAPS(4) } else { NV_CONV_TAPS(1) }
#undef NV_CONV_TAPS
#undef NV_CONV
  NV_RETURN_LAST();
}

// out: [T, half] pairs (cosine, sine) of position * inv_freq.
NV_API int nv_rotary_table(const int* positions, const float* inv_freq, int half, float* out, int T, cudaStream_t s) {
  const long long n = (long long)T * half;
  if (half < 0) return NV_ERR_BAD_SIZE;
  if (n == 0) return NV_OK;
  NV_RETURN_IF(launch_dep(rotary_table_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, s, positions, inv_freq, half,
                          (float2*)out, n));
  NV_RETURN_LAST();
}

NV_API int nv_retention_chunk_rows() { return RC; }

// what 0: the form for entries of one row; 1: the chunked form; 2: the scan.
NV_API int nv_retention_usable(int what, int dk, int dv) {
  if (dk < 1 || dv < 1) return 0;
  if (what == 0) {
    const int groups = dv / step_vec(dv);
    return groups <= RT_THREADS && sizeof(float) * (2 * (size_t)dk + (size_t)(RT_THREADS / groups) * dv) <= 200 * 1024;
  }
  if (what == 1) return dk <= 256 && dv <= 256;
  return sizeof(float) * ((size_t)dk * 32 + 2 * (size_t)dk + RT_THREADS) <= 200 * 1024;
}

// One launch (what 0), or the launches of the chunked form (what 1: `chunks` holds max_chunks * H * dk * dv words) or of
// the scan (what 2: `raw` [T, H, dv]).  Entries with fewer than `min_rows` rows are skipped by what 1 and 2; what 0 takes
// the `R` batch rows in `rows` (nullptr: rows 0 .. R - 1), each an entry of its own.  Everything is float32 but `out`.
NV_API int nv_retention(int what, const float* proj, long long ld, int q0, int k0, int v0, int g0, const float* table,
                        const int* positions, const float* inv_freq, int half, const int* row_entry, const int* cu_rows,
                        const int* entry_slot, int num_entries, const int* rows, int R, float* S, long long S_stride,
                        const float* powers, float k_scale, float eps, void* out, int out_dt, float* raw, void* chunks,
                        int max_chunks, int T, int H, int dk, int dv, int min_rows, int G, int raw_out, const float* dsrc,
                        long long d_ld, int d0, const float* A_log, const float* dt_bias, float* chunk_decay,
                        cudaStream_t s) {
  // G: heads of q and k.  raw_out: the outputs go to `raw` in float32, without norm and gate (any `what`; `out` is then not
  // written).  dsrc: row decays, from the step sizes' pre-activations [T, d_ld] at column d0 (head h's at d0 + h), with
  // A_log [H] and dt_bias [H]; `powers` may then be nullptr, and what 1 takes chunk_decay [max_chunks, H] as scratch.
  if (!dt_ok(out_dt)) return NV_ERR_BAD_DTYPE;
  if (G < 1 || H % G || (raw_out && !raw) || (!dsrc && !powers) || (dsrc && (!A_log || !dt_bias))) return NV_ERR_BAD_SIZE;
  if (H < 1 || half < 0 || 2 * half > dk || num_entries < 0) return NV_ERR_BAD_SIZE;
  if (!nv_retention_usable(what, dk, dv)) return NV_ERR_UNSUPPORTED;
  if (T == 0 || num_entries == 0) return NV_OK;
  RetArgs a = {};
  a.proj = proj; a.ld = ld; a.q0 = q0; a.k0 = k0; a.v0 = v0; a.g0 = g0; a.table = (const float2*)table;
  a.positions = positions; a.inv_freq = inv_freq; a.half = half; a.row_entry = row_entry; a.cu_rows = cu_rows;
  a.entry_slot = entry_slot; a.rows = rows; a.S = S; a.S_stride = S_stride; a.powers = powers; a.k_scale = k_scale;
  a.eps = eps; a.out = out; a.raw = raw; a.chunks = (uint32_t*)chunks; a.out_dt = out_dt; a.H = H; a.dk = dk; a.dv = dv;
  a.num_entries = num_entries; a.min_rows = min_rows;
  a.G = G; a.raw_out = raw_out; a.dsrc = dsrc; a.d_ld = d_ld; a.d0 = d0; a.A_log = A_log; a.dt_bias = dt_bias;
  a.chunk_decay = nullptr;
  if (what == 0) {
    if (R == 0) return NV_OK;
    const bool vec = step_vec(dv) == 4 && S_stride % 4 == 0 && !((uintptr_t)S & 15);
    const int groups = vec ? dv / 4 : dv;
    if (groups > RT_THREADS) return NV_ERR_UNSUPPORTED;
    const size_t smem = sizeof(float) * (2 * (size_t)dk + (size_t)(RT_THREADS / groups) * dv);
    int rc = vec ? allow(retention_step_kernel<4>, smem) : allow(retention_step_kernel<1>, smem);
    if (rc) return rc;
    if (vec) NV_RETURN_IF(launch_dep(retention_step_kernel<4>, dim3(R, H), dim3(RT_THREADS), smem, s, a));
    else NV_RETURN_IF(launch_dep(retention_step_kernel<1>, dim3(R, H), dim3(RT_THREADS), smem, s, a));
    NV_RETURN_LAST();
  }
  if (half > 0 && !table) return NV_ERR_BAD_SIZE;
  if (what == 1) {
    if (!chunks || max_chunks < 1 || (dsrc && !chunk_decay)) return NV_ERR_BAD_SIZE;
    if (dsrc) a.chunk_decay = chunk_decay;
    a.v2 = (half % 2 == 0 && dk % 2 == 0 && dv % 2 == 0 && ld % 2 == 0 && q0 % 2 == 0 && k0 % 2 == 0 && v0 % 2 == 0 &&
            g0 % 2 == 0 && !((uintptr_t)proj & 15) && !((uintptr_t)table & 15) && !((uintptr_t)chunks & 15) &&
            !((uintptr_t)out & 15) && !((uintptr_t)raw & 7)) ? 1 : 0;
    a.planes = (dv % 8 == 0 && S_stride % 4 == 0 && !((uintptr_t)S & 15) && !((uintptr_t)chunks & 15)) ? 1 : 0;
    // heads that share q and k, several to a block, as long as the step has blocks enough for the multiprocessors
    a.hb = 1;
    while (a.hb < CK_HEADS && (H / G) % (2 * a.hb) == 0 && (long long)max_chunks * (H / (2 * a.hb)) >= 288) a.hb *= 2;
    if (dk <= 64) return launch_chunks_dk<64>(a, max_chunks, s);
    if (dk <= 128) return launch_chunks_dk<128>(a, max_chunks, s);
    return launch_chunks_dk<256>(a, max_chunks, s);
  }
  if (!raw) return NV_ERR_BAD_SIZE;
  a.slice = 32;
  const size_t smem = sizeof(float) * ((size_t)dk * a.slice + 2 * (size_t)dk + RT_THREADS);
  int rc = allow(retention_scan_kernel, smem);
  if (rc) return rc;
  retention_scan_kernel<<<dim3(num_entries, H, (dv + a.slice - 1) / a.slice), RT_THREADS, smem, s>>>(a);
  cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) return (int)e;
  if (raw_out) return NV_OK;
  const long long items = (long long)T * H;
  retention_finish_kernel<<<(unsigned)((items + 7) / 8), 256, 0, s>>>(a, T);
  NV_RETURN_LAST();
}

// out[t, :] from raw [T, n] (n = H * dv), see gated_norm_kernel.  skip: [H] with x [T, x_ld], or nullptr; gate: [T, gate_ld];
// w: [n]; the norm is taken over `parts` equal parts of the row.  gate_first: silu(gate) before the norm, else sigmoid(gate)
// behind it.
NV_API int nv_gated_norm(const float* raw, const float* skip, const float* x, long long x_ld, const float* gate,
                         long long gate_ld, const float* w, void* out, int out_dt, int T, int H, int dv, int parts,
                         int gate_first, float eps, cudaStream_t s) {
  if (!dt_ok(out_dt)) return NV_ERR_BAD_DTYPE;
  if (H < 1 || dv < 1 || parts < 1 || parts > 65535 || (H * dv) % parts || (skip && !x)) return NV_ERR_BAD_SIZE;
  if (T == 0) return NV_OK;
  GatedNormArgs a = {raw, skip, x, x_ld, gate, gate_ld, w, out, out_dt, H * dv, dv, parts, gate_first, 0, eps};
  if (!x) a.x = raw;                     // (never read)
  const int m = a.n / parts;
  const bool vec = m % 4 == 0 && gate_ld % 4 == 0 && (!skip || (x_ld % 4 == 0 && !((uintptr_t)x & 15))) &&
                   !((uintptr_t)raw & 15) && !((uintptr_t)gate & 15) && !((uintptr_t)w & 15) && !((uintptr_t)out & 15);
  a.head_chunks = dv % (vec ? 4 : 1) == 0;
  const int chunks = vec ? m / 4 : m;
  const int half = (chunks + 1) / 2;     // two chunks a thread: their loads are in flight together
  const int threads = half < GN_THREADS ? (half + 31) / 32 * 32 : GN_THREADS;
  if (vec) NV_RETURN_IF(launch_dep(gated_norm_kernel<4>, dim3(T, parts), dim3(threads), 0, s, a));
  else NV_RETURN_IF(launch_dep(gated_norm_kernel<1>, dim3(T, parts), dim3(threads), 0, s, a));
  NV_RETURN_LAST();
}
