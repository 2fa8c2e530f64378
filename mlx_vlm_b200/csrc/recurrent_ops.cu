// Two recurrent mixers for decoder designs assembled on the host (models/decoder_blocks.py), over the step layout of
// mixer_ops.cu (every token of a step names its slot and position, `seqs[g] = (first row, rows)` lists the sequences):
//   * a gated linear recurrence per channel (the RG-LRU of De et al., "Griffin: Mixing Gated Linear Recurrences with Local
//     Attention for Efficient Language Models"):  log a = -c r softplus(lam),  S <- a S + sqrt(1 - a^2) i u,  out = S gelu(y)
//   * a matrix memory per head with exponential gates (the mLSTM of Beck et al., "xLSTM: Extended Long Short-Term Memory"):
//     m' = max(f + m, i);  S <- exp(f + m - m') S + exp(i - m') k v^T,  n likewise with k alone,
//     o = S^T q / (max(|n . q|, exp(-m')) + 1e-6),  RMS norm per head, weight, sigmoid gate.
// States are fp32 in the slot, zero at position 0 (so a released slot is used again as it is); all arithmetic is fp32, the
// sums of log forget gates of a chunk are double.
#include "common.cuh"

namespace b200 {
namespace {

__device__ __forceinline__ float sigmoid_f32(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float softplus_f32(float x) { return x > 20.f ? x : log1pf(expf(x)); }
// z / 2 (1 + tanh(sqrt(2 / pi) (z + 0.044715 z^3))) = z sigmoid(2 sqrt(2 / pi) (...))
__device__ __forceinline__ float gelu_tanh_f32(float z) {
  return z / (1.0f + expf(-1.5957691216057308f * (z + 0.044715f * z * z * z)));
}

// ---------------------------------------------------------------------------------------------------------
// gated linear recurrence
struct LruP {
  float* G; long ldg;              // gate logits [T][blocks][r: bs | i: bs], without their biases; a long step overwrites
  int bs;                          // them with (a, sqrt(1 - a^2) i u), made once for both passes
  const bf16 *rb, *ib, *lam;       // [n]
  float c;
  const float* u; long ldu;        // [T][n]
  const float* y; long ldy;        // [T][n]: the other branch before its gelu
  float* state; long slot_stride;  // per slot [n]
  const int *seqs, *slot, *pos;
  int n;
  float* out; long ldo;            // fp32 rows, or (outb) bf16 operand rows of ldb >= n columns, zero beyond n
  bf16* outb; long ldb;
  int part_len, n_parts;           // a long sequence in parts that are walked at the same time
  float* part;                     // [n_seq][n_parts][2][n]: product of a, state walked from zero; then [n_seq][n]: start state
  int n_seq;
};
constexpr int LRU_B = 8;
struct LruC { float rb, ib, sp; };
__device__ __forceinline__ LruC lru_consts(const LruP& p, int ch) {
  return {bf2f(p.rb[ch]), bf2f(p.ib[ch]), p.c * softplus_f32(bf2f(p.lam[ch]))};
}
__device__ __forceinline__ void lru_gates(const LruC& k, float gr, float gi, float u, float& a, float& z) {
  const float la = -sigmoid_f32(gr + k.rb) * k.sp;
  a = expf(la);
  z = sqrtf(fmaxf(-expm1f(2.0f * la), 0.f)) * sigmoid_f32(gi + k.ib) * u;     // 1 - a^2 without cancellation
}
__device__ __forceinline__ void lru_store(const LruP& p, long t, int ch, float v) {
  if (p.outb) p.outb[t * p.ldb + ch] = f2bf(v);
  else p.out[t * p.ldo + ch] = v;
}
// few rows per sequence: a thread per channel walks them
__global__ void lru_walk_kernel(LruP p) {
  const int ch = blockIdx.y * blockDim.x + threadIdx.x, start = p.seqs[2 * blockIdx.x], rows = p.seqs[2 * blockIdx.x + 1];
  if (ch >= p.n) {
    if (p.outb && ch < p.ldb)
      for (int r = 0; r < rows; ++r) p.outb[(long)(start + r) * p.ldb + ch] = f2bf(0.f);
    return;
  }
  const LruC k = lru_consts(p, ch);
  const int gc = ch / p.bs * 2 * p.bs + ch % p.bs;
  float* st = p.state + (long)p.slot[start] * p.slot_stride + ch;
  float S = p.pos[start] > 0 ? *st : 0.f;
#pragma unroll 2
  for (int r = 0; r < rows; ++r) {
    const long t = start + r;
    float a, z;
    lru_gates(k, p.G[t * p.ldg + gc], p.G[t * p.ldg + gc + p.bs], p.u[t * p.ldu + ch], a, z);
    S = fmaf(a, S, z);
    lru_store(p, t, ch, S * gelu_tanh_f32(p.y[t * p.ldy + ch]));
  }
  *st = S;
}
// pass 1 over the parts: a and the input term of every token, the part's decay product and what it adds from zero
__global__ void lru_parts_kernel(LruP p) {
  const int seq = blockIdx.x / p.n_parts, part = blockIdx.x % p.n_parts, ch = blockIdx.y * blockDim.x + threadIdx.x;
  const int first = p.seqs[2 * seq], rows = min(p.part_len, p.seqs[2 * seq + 1] - part * p.part_len);
  if (rows <= 0 || ch >= p.n) return;
  const long start = first + (long)part * p.part_len;
  const LruC k = lru_consts(p, ch);
  const int gc = ch / p.bs * 2 * p.bs + ch % p.bs;
  float S = 0.f, A = 1.f;
  for (int r0 = 0; r0 < rows; r0 += LRU_B) {       // the loads of several tokens go out together, before any store
    float gr[LRU_B], gi[LRU_B], u[LRU_B];
#pragma unroll
    for (int j = 0; j < LRU_B; ++j) {
      const long t = start + min(r0 + j, rows - 1);
      gr[j] = p.G[t * p.ldg + gc];
      gi[j] = p.G[t * p.ldg + gc + p.bs];
      u[j] = p.u[t * p.ldu + ch];
    }
#pragma unroll
    for (int j = 0; j < LRU_B; ++j)
      if (r0 + j < rows) {
        float* g = p.G + (start + r0 + j) * p.ldg + gc;
        float a, z;
        lru_gates(k, gr[j], gi[j], u[j], a, z);
        g[0] = a;
        g[p.bs] = z;
        S = fmaf(a, S, z);
        A *= a;
      }
  }
  float* d = p.part + ((long)seq * p.n_parts + part) * 2 * p.n + ch;
  d[0] = A;
  d[p.n] = S;
  if (part == 0)      // kept beside the parts: the last part of pass 2 replaces the slot's state while others start from it
    p.part[(long)p.n_seq * p.n_parts * 2 * p.n + (long)seq * p.n + ch] =
        p.pos[first] > 0 ? p.state[(long)p.slot[first] * p.slot_stride + ch] : 0.f;
}
// pass 2: the part's start state from the parts before it, then the walk with outputs
__global__ void lru_scan_kernel(LruP p) {
  const int seq = blockIdx.x / p.n_parts, part = blockIdx.x % p.n_parts, ch = blockIdx.y * blockDim.x + threadIdx.x;
  const int first = p.seqs[2 * seq], total = p.seqs[2 * seq + 1], rows = min(p.part_len, total - part * p.part_len);
  if (rows <= 0) return;
  const long start = first + (long)part * p.part_len;
  if (ch >= p.n) {
    if (p.outb && ch < p.ldb)
      for (int r = 0; r < rows; ++r) p.outb[(start + r) * p.ldb + ch] = f2bf(0.f);
    return;
  }
  const int gc = ch / p.bs * 2 * p.bs + ch % p.bs;
  float S = p.part[(long)p.n_seq * p.n_parts * 2 * p.n + (long)seq * p.n + ch];
  const float* d = p.part + (long)seq * p.n_parts * 2 * p.n + ch;
#pragma unroll 8
  for (int q = 0; q < part; ++q, d += 2 * p.n) S = fmaf(d[0], S, d[p.n]);
  for (int r0 = 0; r0 < rows; r0 += LRU_B) {
    float a[LRU_B], z[LRU_B], y[LRU_B];
#pragma unroll
    for (int j = 0; j < LRU_B; ++j) {
      const long t = start + min(r0 + j, rows - 1);
      a[j] = p.G[t * p.ldg + gc];
      z[j] = p.G[t * p.ldg + gc + p.bs];
      y[j] = p.y[t * p.ldy + ch];
    }
#pragma unroll
    for (int j = 0; j < LRU_B; ++j)
      if (r0 + j < rows) {
        S = fmaf(a[j], S, z[j]);
        lru_store(p, start + r0 + j, ch, S * gelu_tanh_f32(y[j]));
      }
  }
  if ((part + 1) * (long)p.part_len >= total) p.state[(long)p.slot[first] * p.slot_stride + ch] = S;
}

// ---------------------------------------------------------------------------------------------------------
// matrix memory.  A slot keeps, per head, S [dim][vdim], n [dim] and m: state = [H][dim vdim] | [H][dim] | [H].
struct MemP {
  const float* q; long ldq;        // [T][H dim], times q_scale here
  const float* k; long ldk;
  const float* v; long ldv;        // [T][H vdim]
  const float* gi; long ldi;       // [T][H] logits of the input gate, and of the forget gate
  const float* gf; long ldf;
  float cap, q_scale;
  const float* gate; long ldg;     // [T][H vdim]
  const bf16* w; float eps;        // [H vdim]
  float* state; long slot_stride;
  const int *seqs, *slot, *pos;
  int H, dim, vdim;
  float* out; long ldo;            // fp32 rows, or (outb) bf16 operand rows of ldb >= H vdim columns, zero beyond
  bf16* outb; long ldb;
  // a prompt step, MC tokens of a sequence at a time (below)
  float* chunk;                    // per (chunk, head): dim vdim + dim floats: S and n that the chunk adds, then its start state
  double* F;                       // [T][H] sum of the log forget gates from the chunk's first token on
  float *li, *ml;                  // [T][H] log input gate; running maximum of the chunk's own tokens alone
  double* tot;                     // per (chunk, head): F and the maximum of the whole chunk
  float* m0;                       // per (chunk, head): the running maximum before the chunk
  float* mstart;                   // [n_seq][H]: the running maximum before the step
};
constexpr float MEM_EPS = 1e-6f;
__device__ __forceinline__ float log_input_gate(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float log_forget_gate(float z, float cap) {
  const float x = cap * tanhf(z / cap);
  return fminf(x, 0.f) - log1pf(expf(-fabsf(x)));
}
__device__ __forceinline__ void mem_store(const MemP& p, long t, int c, float v) {
  if (p.outb) p.outb[t * p.ldb + c] = f2bf(v);
  else p.out[t * p.ldo + c] = v;
}

// Few rows per sequence (a decode step): a block per sequence and head walks them, the state of the head stays where it is
// (a row of S per warp at a time, V columns per lane), everything up to the gated output in the same launch.
constexpr int MW_THREADS = 512;
template <int V>
__global__ void __launch_bounds__(MW_THREADS) memory_walk_kernel(MemP p) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[MW_THREADS / 32], red2[MW_THREADS / 32];
  constexpr int NW = MW_THREADS / 32;
  const int seq = blockIdx.x, h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int d = p.dim, dv = p.vdim, start = p.seqs[2 * seq], rows = p.seqs[2 * seq + 1];
  float* ks = sm;                    // dim
  float* qs = ks + d;                // dim
  float* vs = qs + d + (4 - (2 * d) % 4) % 4;   // vdim (16-byte aligned)
  float* os = vs + (dv + 3) / 4 * 4;            // [NW][vdim rounded up to 4]
  const int ldo = (dv + 3) / 4 * 4;
  float* st = p.state + (long)p.slot[start] * p.slot_stride;
  float* S = st + (long)h * d * dv;
  float* n = st + (long)p.H * d * dv + (long)h * d;
  float* mp = st + (long)p.H * d * (dv + 1) + h;
  bool fresh = p.pos[start] == 0;
  float m = fresh ? 0.f : *mp;
  for (int r = 0; r < rows; ++r) {
    const long t = start + r;
    const float i = log_input_gate(p.gi[t * p.ldi + h], p.cap), f = log_forget_gate(p.gf[t * p.ldf + h], p.cap);
    const float mn = fmaxf(f + m, i), keep = expf(f + m - mn), put = expf(i - mn), floor_ = expf(-mn);
    __syncthreads();                 // the row before is done with the staged vectors (and every thread has read m)
    for (int e = threadIdx.x; e < d; e += MW_THREADS) {
      ks[e] = put * p.k[t * p.ldk + (long)h * d + e];
      qs[e] = p.q_scale * p.q[t * p.ldq + (long)h * d + e];
    }
    for (int e = threadIdx.x; e < dv; e += MW_THREADS) vs[e] = p.v[t * p.ldv + (long)h * dv + e];
    __syncthreads();
    float nq = 0.f;
    for (int e = threadIdx.x; e < d; e += MW_THREADS) {
      const float x = fresh ? ks[e] : fmaf(keep, n[e], ks[e]);
      n[e] = x;
      nq = fmaf(x, qs[e], nq);
    }
    nq = warp_sum(nq);
    if (lane == 0) red[warp] = nq;
    for (int c = lane * V; c < dv; c += 32 * V) {
      float acc[V], vv[V];
#pragma unroll
      for (int j = 0; j < V; ++j) { acc[j] = 0.f; vv[j] = vs[c + j]; }
#pragma unroll 8
      for (int e = warp; e < d; e += NW) {
        float* s = S + (long)e * dv + c;
        float x[V];
        if constexpr (V == 4) {
          const float4 a = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(s);
          x[0] = a.x; x[1] = a.y; x[2] = a.z; x[3] = a.w;
        } else {
          x[0] = fresh ? 0.f : *s;
        }
        const float kk = ks[e], qq = qs[e];
#pragma unroll
        for (int j = 0; j < V; ++j) { x[j] = fmaf(kk, vv[j], keep * x[j]); acc[j] = fmaf(x[j], qq, acc[j]); }
        if constexpr (V == 4) *reinterpret_cast<float4*>(s) = make_float4(x[0], x[1], x[2], x[3]);
        else *s = x[0];
      }
#pragma unroll
      for (int j = 0; j < V; ++j) os[warp * ldo + c + j] = acc[j];
    }
    __syncthreads();
    float den = 0.f, ss = 0.f;
    for (int w = 0; w < NW; ++w) den += red[w];                     // fixed order
    den = fmaxf(fabsf(den), floor_) + MEM_EPS;
    for (int c = threadIdx.x; c < dv; c += MW_THREADS) {
      float o = 0.f;
#pragma unroll
      for (int w = 0; w < NW; ++w) o += os[w * ldo + c];
      o /= den;
      os[c] = o;                                                   // read again by this thread only
      ss = fmaf(o, o, ss);
    }
    ss = warp_sum(ss);
    if (lane == 0) red2[warp] = ss;
    __syncthreads();
    float tot = 0.f;
    for (int w = 0; w < NW; ++w) tot += red2[w];
    const float inv = 1.0f / sqrtf(tot / (float)dv + p.eps);
    for (int c = threadIdx.x; c < dv; c += MW_THREADS) {
      const int col = h * dv + c;
      mem_store(p, t, col, os[c] * inv * bf2f(p.w[col]) * sigmoid_f32(p.gate[t * p.ldg + col]));
    }
    m = mn;
    fresh = false;
  }
  if (threadIdx.x == 0) *mp = m;     // every thread read it before the first barrier of the walk
  if (p.outb && h == p.H - 1)
    for (int r = 0; r < rows; ++r)
      for (long c = (long)p.H * dv + threadIdx.x; c < p.ldb; c += MW_THREADS) p.outb[(start + r) * p.ldb + c] = f2bf(0.f);
}

// A prompt: MC tokens of a sequence at a time.  With F_t the sum of the chunk's log forget gates up to t, m_t the running
// maximum and (S, m) the state before the chunk,
//   m_t = max(F_t + m, max_{s <= t} (F_t - F_s + i_s)),
//   o_t = exp(F_t + m - m_t) S^T q_t + sum_{s <= t} exp(F_t - F_s + i_s - m_t) (k_s . q_t) v_s,
// n . q_t the same with v_s = 1, and at the chunk's end  S' = exp(F + m - m') S + sum_s exp(F - F_s + i_s - m') k_s v_s^T.
// No weight exceeds one.  Three launches, each parallel over the chunks or the state: what every chunk adds (relative to
// its own maximum), the chain of start states, the outputs.
constexpr int MC = 64, MC_THREADS = 256, MC_K = 32, MC_LD = MC + 4;
__device__ __forceinline__ long mem_chunk0(const int* seqs, int g) { return seqs[2 * g] / MC + g; }   // no two sequences share one
struct MemTile { float a[MC_K][MC_LD], b[MC_K][MC_LD]; };
// acc[i][j] += sum_k A[k][4 ty + i] B[k][4 tx + j], 16 x 16 threads
__device__ __forceinline__ void tile_mma(const float (*A)[MC_LD], const float (*B)[MC_LD], int nk, float (&acc)[4][4]) {
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
#pragma unroll 8
  for (int k = 0; k < nk; ++k) {
    const float4 x = *reinterpret_cast<const float4*>(&A[k][ty * 4]), y = *reinterpret_cast<const float4*>(&B[k][tx * 4]);
    const float a[4] = {x.x, x.y, x.z, x.w}, b[4] = {y.x, y.y, y.z, y.w};
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
  }
}
// A tile's numbers travel from memory through registers: the next tile is requested while the current one is multiplied.
// Along: tile[k][r] = number k0 + k of row r (rows laid out along k), times mul scale[r]; a thread takes eight numbers of one
// row (a whole sector), neighbouring lanes neighbouring rows.  Across: tile[k][c] = number c0 + c of row k0 + k, times
// scale[k0 + k]; a thread takes four numbers of two rows.  VEC: everything starts on 16-byte boundaries, sizes are multiples of 4
constexpr int MC_REGS = 8;
static_assert(MC * MC_K == MC_THREADS * MC_REGS, "");
template <bool VEC>
struct Along {
  const float* x; long ld; int n_rows, K; const float* scale; float mul;
  __device__ __forceinline__ void request(int k0, float (&v)[MC_REGS]) const {
    const int r = threadIdx.x % MC, k = k0 + threadIdx.x / MC * MC_REGS;
#pragma unroll
    for (int j = 0; j < MC_REGS; j += 4) {
      if constexpr (VEC) {
        const float4 a = (r < n_rows && k + j < K) ? *reinterpret_cast<const float4*>(x + (long)r * ld + k + j) : make_float4(0.f, 0.f, 0.f, 0.f);
        v[j] = a.x; v[j + 1] = a.y; v[j + 2] = a.z; v[j + 3] = a.w;
      } else {
#pragma unroll
        for (int e = j; e < j + 4; ++e) v[e] = (r < n_rows && k + e < K) ? x[(long)r * ld + k + e] : 0.f;
      }
    }
  }
  __device__ __forceinline__ void store(float (*tile)[MC_LD], int, const float (&v)[MC_REGS]) const {
    const int r = threadIdx.x % MC, k = threadIdx.x / MC * MC_REGS;
    const float f = scale ? scale[r] * mul : mul;
#pragma unroll
    for (int j = 0; j < MC_REGS; ++j) tile[k + j][r] = v[j] * f;
  }
};
template <bool VEC>
struct Across {
  const float* x; long ld; int K, c0, C; const float* scale;
  __device__ __forceinline__ void request(int k0, float (&v)[MC_REGS]) const {
    const int c = c0 + threadIdx.x % (MC / 4) * 4;
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int k = k0 + h * (MC_K / 2) + threadIdx.x / (MC / 4);
      if constexpr (VEC) {
        const float4 a = (k < K && c < C) ? *reinterpret_cast<const float4*>(x + (long)k * ld + c) : make_float4(0.f, 0.f, 0.f, 0.f);
        v[4 * h] = a.x; v[4 * h + 1] = a.y; v[4 * h + 2] = a.z; v[4 * h + 3] = a.w;
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e) v[4 * h + e] = (k < K && c + e < C) ? x[(long)k * ld + c + e] : 0.f;
      }
    }
  }
  __device__ __forceinline__ void store(float (*tile)[MC_LD], int k0, const float (&v)[MC_REGS]) const {
    const int c = threadIdx.x % (MC / 4) * 4;
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int k = h * (MC_K / 2) + threadIdx.x / (MC / 4);
      const float f = scale ? (k0 + k < K ? scale[k0 + k] : 0.f) : 1.f;
      *reinterpret_cast<float4*>(&tile[k][c]) = make_float4(v[4 * h] * f, v[4 * h + 1] * f, v[4 * h + 2] * f, v[4 * h + 3] * f);
    }
  }
};
// acc += A B over K numbers (staged: A is already in shared memory, [k][MC_LD])
template <class SA, class SB>
__device__ __forceinline__ void tile_product(MemTile& tile, const SA& sa, const SB& sb, int K, float (&acc)[4][4]) {
  float va[MC_REGS], vb[MC_REGS];
  sa.request(0, va);
  sb.request(0, vb);
  for (int k0 = 0; k0 < K; k0 += MC_K) {
    __syncthreads();
    sa.store(tile.a, k0, va);
    sb.store(tile.b, k0, vb);
    __syncthreads();
    if (k0 + MC_K < K) { sa.request(k0 + MC_K, va); sb.request(k0 + MC_K, vb); }
    tile_mma(tile.a, tile.b, min(MC_K, K - k0), acc);
  }
}
template <class SB>
__device__ __forceinline__ void tile_product_staged(MemTile& tile, const float (*PA)[MC_LD], const SB& sb, int K, float (&acc)[4][4]) {
  float vb[MC_REGS];
  sb.request(0, vb);
  for (int k0 = 0; k0 < K; k0 += MC_K) {
    __syncthreads();
    sb.store(tile.b, k0, vb);
    __syncthreads();
    if (k0 + MC_K < K) sb.request(k0 + MC_K, vb);
    tile_mma(PA + k0, tile.b, min(MC_K, K - k0), acc);
  }
}

template <bool VEC>
__global__ void __launch_bounds__(MC_THREADS, 4) memory_chunk_kernel(MemP p) {
  __shared__ MemTile tile;
  __shared__ float ws[MC];
  const int seq = blockIdx.z, h = blockIdx.y, d = p.dim, dv = p.vdim;
  const int first = p.seqs[2 * seq], nc = min(MC, p.seqs[2 * seq + 1] - (int)blockIdx.x * MC);
  if (nc <= 0) return;
  const long start = first + (long)blockIdx.x * MC, ch = (mem_chunk0(p.seqs, seq) + blockIdx.x) * p.H + h;
  if (threadIdx.x < 32) {            // the gates, their running sum and running maximum: a scan of (f, m) pairs
    const int lane = threadIdx.x;
    double Fc = 0.0, Mc = -INFINITY;
    double Fl[MC / 32], il[MC / 32];
#pragma unroll
    for (int g = 0; g < MC / 32; ++g) {
      const int s = g * 32 + lane;
      const bool ok = s < nc;
      const float li = ok ? log_input_gate(p.gi[(start + s) * p.ldi + h], p.cap) : -INFINITY;
      double f = ok ? (double)log_forget_gate(p.gf[(start + s) * p.ldf + h], p.cap) : 0.0, m = li;
      const float lf_in = li;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const double fp = __shfl_up_sync(0xffffffffu, f, o), mp = __shfl_up_sync(0xffffffffu, m, o);
        if (lane >= o) { m = fmax(mp + f, m); f += fp; }
      }
      m = fmax(Mc + f, m);
      f += Fc;
      if (ok) { p.F[(start + s) * p.H + h] = f; p.li[(start + s) * p.H + h] = lf_in; p.ml[(start + s) * p.H + h] = (float)m; }
      Fl[g] = f; il[g] = lf_in;
      Fc = __shfl_sync(0xffffffffu, f, 31);
      Mc = __shfl_sync(0xffffffffu, m, 31);
    }
    // (tokens past the end of the sequence have f = 0 and i = -inf: they change neither)
#pragma unroll
    for (int g = 0; g < MC / 32; ++g) ws[g * 32 + lane] = g * 32 + lane < nc ? expf((float)(Fc - Fl[g] + il[g] - Mc)) : 0.f;
    if (lane == 0) {
      p.tot[2 * ch] = Fc;
      p.tot[2 * ch + 1] = Mc;
      if (blockIdx.x == 0)
        p.mstart[(long)seq * p.H + h] =
            p.pos[first] > 0 ? p.state[(long)p.slot[first] * p.slot_stride + (long)p.H * d * (dv + 1) + h] : 0.f;
    }
  }
  __syncthreads();
  float* S = p.chunk + ch * ((long)d * (dv + 1));
  const float* k = p.k + start * p.ldk + (long)h * d;
  const float* v = p.v + start * p.ldv + (long)h * dv;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  for (int i0 = 0; i0 < d; i0 += MC)
    for (int c0 = 0; c0 < dv; c0 += MC) {
      float acc[4][4] = {};
      tile_product(tile, Across<VEC>{k, p.ldk, nc, i0, d, ws}, Across<VEC>{v, p.ldv, nc, c0, dv, nullptr}, nc, acc);
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int r = i0 + ty * 4 + i, c = c0 + tx * 4 + j;
          if (r < d && c < dv) S[(long)r * dv + c] = acc[i][j];
        }
    }
  for (int e = threadIdx.x; e < d; e += MC_THREADS) {
    float a = 0.f;
#pragma unroll 8
    for (int s = 0; s < nc; ++s) a = fmaf(ws[s], k[(long)s * p.ldk + e], a);
    S[(long)d * dv + e] = a;
  }
}

// start states, chunk after chunk; a thread per number of the head's S and n.  The running maximum of 32 chunks at a time, and
// from it what a chunk keeps of the state and what it puts, by one warp
__global__ void memory_chain_kernel(MemP p) {
  __shared__ float keep[32], put[32];
  const int seq = blockIdx.x, h = blockIdx.y, d = p.dim, dv = p.vdim;
  const long e = (long)blockIdx.z * blockDim.x + threadIdx.x, num = (long)d * (dv + 1);
  const int first = p.seqs[2 * seq], n = (p.seqs[2 * seq + 1] + MC - 1) / MC;
  const long ch0 = mem_chunk0(p.seqs, seq);
  float* st = p.state + (long)p.slot[first] * p.slot_stride;
  float* mine = e < (long)d * dv ? st + (long)h * d * dv + e : st + (long)p.H * d * dv + (long)h * d + (e - (long)d * dv);
  const bool ok = e < num;
  float S = (ok && p.pos[first] > 0) ? *mine : 0.f;
  float m = p.mstart[(long)seq * p.H + h];
  constexpr int B = 8;                // chunks whose numbers are loaded together
  for (int g0 = 0; g0 < n; g0 += 32) {
    __syncthreads();
    if (threadIdx.x < 32) {
      const int lane = threadIdx.x, c = g0 + lane;
      const long ch = (ch0 + min(c, n - 1)) * p.H + h;
      double F = c < n ? p.tot[2 * ch] : 0.0, M = c < n ? p.tot[2 * ch + 1] : -INFINITY;
      const double F1 = F, M1 = M;    // the chunk's own
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const double fp = __shfl_up_sync(0xffffffffu, F, o), mp = __shfl_up_sync(0xffffffffu, M, o);
        if (lane >= o) { M = fmax(mp + F, M); F += fp; }
      }
      const float after = (float)fmax(F + (double)m, M);
      float before = __shfl_up_sync(0xffffffffu, after, 1);
      if (lane == 0) before = m;
      keep[lane] = expf((float)(F1 + (double)before - (double)after));
      put[lane] = expf((float)(M1 - (double)after));
      if (c < n && blockIdx.z == 0) p.m0[ch] = before;
      m = __shfl_sync(0xffffffffu, after, 31);       // (chunks past the end change nothing)
    }
    __syncthreads();
    const int g1 = min(n, g0 + 32);
    for (int c0 = g0; c0 < g1; c0 += B) {
      float add[B];
#pragma unroll
      for (int j = 0; j < B; ++j) add[j] = ok ? p.chunk[((ch0 + min(c0 + j, n - 1)) * p.H + h) * num + e] : 0.f;
#pragma unroll
      for (int j = 0; j < B; ++j)
        if (c0 + j < g1) {
          if (ok) p.chunk[((ch0 + c0 + j) * p.H + h) * num + e] = S;
          S = fmaf(keep[c0 + j - g0], S, put[c0 + j - g0] * add[j]);
        }
    }
  }
  if (ok) *mine = S;
  if (e == 0) st[(long)p.H * d * (dv + 1) + h] = m;
}

template <bool VEC>
__global__ void __launch_bounds__(MC_THREADS) memory_out_kernel(MemP p) {
  extern __shared__ __align__(16) float sm[];
  MemTile& tile = *reinterpret_cast<MemTile*>(sm);
  float (*P)[MC_LD] = reinterpret_cast<float (*)[MC_LD]>(sm + sizeof(MemTile) / 4);      // P[s][t]: weighted k_s . q_t
  float* os = sm + sizeof(MemTile) / 4 + MC * MC_LD;                                     // [MC][vdim]
  __shared__ double F[MC];
  __shared__ float li[MC], mt[MC], ws[MC], den[MC];
  const int seq = blockIdx.z, h = blockIdx.y, d = p.dim, dv = p.vdim;
  const int nc = min(MC, p.seqs[2 * seq + 1] - (int)blockIdx.x * MC);
  if (nc <= 0) return;
  const long start = p.seqs[2 * seq] + (long)blockIdx.x * MC, ch = (mem_chunk0(p.seqs, seq) + blockIdx.x) * p.H + h;
  const float* S = p.chunk + ch * ((long)d * (dv + 1));
  const float* n = S + (long)d * dv;
  const float* q = p.q + start * p.ldq + (long)h * d;
  const float* k = p.k + start * p.ldk + (long)h * d;
  const float* v = p.v + start * p.ldv + (long)h * dv;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x < MC) {
    const int t = threadIdx.x;
    const bool ok = t < nc;
    const double f = ok ? p.F[(start + t) * p.H + h] : 0.0, m0 = p.m0[ch];
    const float m = ok ? (float)fmax(f + m0, (double)p.ml[(start + t) * p.H + h]) : 0.f;
    F[t] = f; mt[t] = m;
    li[t] = ok ? p.li[(start + t) * p.H + h] : 0.f;
    ws[t] = ok ? expf((float)(f + m0 - (double)m)) : 0.f;
  }
  {
    float acc[4][4] = {};
    tile_product(tile, Along<VEC>{k, p.ldk, nc, d, nullptr, 1.f}, Along<VEC>{q, p.ldq, nc, d, nullptr, p.q_scale}, d, acc);
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int s = ty * 4 + i, t = tx * 4 + j;
        P[s][t] = (s <= t && t < nc) ? acc[i][j] * expf((float)(F[t] - F[s] + (double)li[s] - (double)mt[t])) : 0.f;
      }
  }
  __syncthreads();
  for (int t = warp; t < nc; t += MC_THREADS / 32) {         // n . q_t, a warp per token
    float a = P[lane][t] + P[lane + 32][t], b = 0.f;
    for (int e = lane; e < d; e += 32) b = fmaf(n[e], q[(long)t * p.ldq + e], b);
    a = warp_sum(fmaf(ws[t] * p.q_scale, b, a));
    if (lane == 0) den[t] = fmaxf(fabsf(a), expf(-mt[t])) + MEM_EPS;
  }
  for (int c0 = 0; c0 < dv; c0 += MC) {
    float acc[4][4] = {};
    tile_product_staged(tile, P, Across<VEC>{v, p.ldv, nc, c0, dv, nullptr}, nc, acc);
    tile_product(tile, Along<VEC>{q, p.ldq, nc, d, ws, p.q_scale}, Across<VEC>{S, dv, d, c0, dv, nullptr}, d, acc);
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (c0 + tx * 4 + j < dv) os[(ty * 4 + i) * dv + c0 + tx * 4 + j] = acc[i][j];
  }
  __syncthreads();
  for (int t = warp; t < nc; t += MC_THREADS / 32) {         // a warp per token: norm, weight, gate
    float* o = os + t * dv;
    const float dn = den[t];
    float ss = 0.f;
    for (int c = lane; c < dv; c += 32) { const float a = o[c] / dn; o[c] = a; ss = fmaf(a, a, ss); }
    const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)dv + p.eps);
    for (int c = lane; c < dv; c += 32) {
      const int col = h * dv + c;
      mem_store(p, start + t, col, o[c] * inv * bf2f(p.w[col]) * sigmoid_f32(p.gate[(start + t) * p.ldg + col]));
    }
    if (p.outb && h == p.H - 1)
      for (long c = (long)p.H * dv + lane; c < p.ldb; c += 32) p.outb[(start + t) * p.ldb + c] = f2bf(0.f);
  }
}

unsigned long long g_mem_attr = 0, g_walk_attr = 0;

}  // namespace
}  // namespace b200

using namespace b200;

extern "C" {

int b200_lm_gated_recurrence(float* G, long ldg, int bs, const void* rb, const void* ib, const void* lam, float c, const float* u,
                             long ldu, const float* y, long ldy, float* state, long slot_stride, const int* seqs, int n_seq,
                             const int* slot, const int* pos, int n, float* out, long ldo, void* out_bf16, long ldb, int part_len,
                             int n_parts, float* part, void* st) {
  B200_REQUIRE(G && rb && ib && lam && u && y && state && seqs && slot && pos && (out || out_bf16), "lm_gated_recurrence: bad argument");
  B200_REQUIRE(n > 0 && n_seq > 0 && bs > 0 && n % bs == 0 && (!out_bf16 || ldb >= n), "lm_gated_recurrence: %d channels in blocks of %d", n, bs);
  B200_REQUIRE(n_parts <= 1 || (part && part_len > 0), "lm_gated_recurrence: parts need their scratch");
  LruP p{G, ldg, bs, (const bf16*)rb, (const bf16*)ib, (const bf16*)lam, c, u, ldu, y, ldy, state, slot_stride, seqs, slot, pos, n,
         out, ldo, (bf16*)out_bf16, ldb, part_len, n_parts, part, n_seq};
  const cudaStream_t cs = (cudaStream_t)st;
  const int cols = out_bf16 ? (int)ldb : n;
  if (n_parts <= 1) {
    lru_walk_kernel<<<dim3(n_seq, cdiv(cols, 64)), 64, 0, cs>>>(p);
    B200_CHECK_LAUNCH();
    return B200_OK;
  }
  lru_parts_kernel<<<dim3(n_seq * n_parts, cdiv(n, 128)), 128, 0, cs>>>(p);
  B200_CHECK_LAUNCH();
  lru_scan_kernel<<<dim3(n_seq * n_parts, cdiv(cols, 128)), 128, 0, cs>>>(p);
  B200_CHECK_LAUNCH();
  return B200_OK;
}

long b200_lm_matrix_memory_scratch(int T, int n_seq, int H, int dim, int vdim) {
  const long chunks = (long)T / MC + n_seq + 1;
  return chunks * H * ((long)dim * (vdim + 1) * 4 + 2 * 8 + 4) + (long)T * H * (8 + 4 + 4) + (long)n_seq * H * 4 + 8 * 16;
}

int b200_lm_matrix_memory(const float* q, long ldq, const float* k, long ldk, const float* v, long ldv, const float* gi, long ldi,
                          const float* gf, long ldf, float cap, float q_scale, const float* gate, long ldg, const void* w, float eps,
                          float* state, long slot_stride, const int* seqs, int n_seq, const int* slot, const int* pos, int H,
                          int dim, int vdim, float* out, long ldo, void* out_bf16, long ldb, void* scratch, long scratch_bytes,
                          int max_rows, int T, void* st) {
  B200_REQUIRE(q && k && v && gi && gf && gate && w && state && seqs && slot && pos && (out || out_bf16), "lm_matrix_memory: bad argument");
  B200_REQUIRE(H > 0 && dim > 0 && vdim > 0 && n_seq > 0 && T > 0 && cap > 0.f && (!out_bf16 || ldb >= (long)H * vdim),
               "lm_matrix_memory: %d heads of %d x %d", H, dim, vdim);
  MemP p{q, ldq, k, ldk, v, ldv, gi, ldi, gf, ldf, cap, q_scale, gate, ldg, (const bf16*)w, eps, state, slot_stride, seqs, slot, pos,
         H, dim, vdim, out, ldo, (bf16*)out_bf16, ldb, nullptr, nullptr, nullptr, nullptr, nullptr, nullptr, nullptr};
  const cudaStream_t cs = (cudaStream_t)st;
  if (!scratch) {                    // few rows
    const size_t smem = (size_t)(2 * dim + 4 + (MW_THREADS / 32 + 1) * ((vdim + 3) / 4 * 4)) * sizeof(float);
    B200_REQUIRE(smem <= 200 * 1024, "lm_matrix_memory: heads of %d x %d do not fit shared memory", dim, vdim);
    if (first_use_on_device(&g_walk_attr)) {
      B200_CUDA(cudaFuncSetAttribute(memory_walk_kernel<4>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
      B200_CUDA(cudaFuncSetAttribute(memory_walk_kernel<1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    }
    const bool vec = vdim % 4 == 0 && slot_stride % 4 == 0 && ((uintptr_t)state & 15) == 0;
    if (vec) memory_walk_kernel<4><<<dim3(n_seq, H), MW_THREADS, smem, cs>>>(p);
    else memory_walk_kernel<1><<<dim3(n_seq, H), MW_THREADS, smem, cs>>>(p);
    B200_CHECK_LAUNCH();
    return B200_OK;
  }
  B200_REQUIRE(max_rows > 0 && max_rows <= T && n_seq <= 65535 && H <= 65535, "lm_matrix_memory: the longest sequence of the step has %d of %d rows", max_rows, T);
  B200_REQUIRE(scratch_bytes >= b200_lm_matrix_memory_scratch(T, n_seq, H, dim, vdim) && ((uintptr_t)scratch & 15) == 0,
               "lm_matrix_memory: scratch of %ld bytes", scratch_bytes);
  const long chunks = (long)T / MC + n_seq + 1;
  p.F = (double*)scratch;
  p.tot = p.F + (long)T * H;
  p.chunk = (float*)(p.F + ((long)T * H + chunks * H * 2 + 1) / 2 * 2);     // 16-byte aligned
  p.li = p.chunk + chunks * H * ((long)dim * (vdim + 1));
  p.ml = p.li + (long)T * H;
  p.m0 = p.ml + (long)T * H;
  p.mstart = p.m0 + chunks * H;
  const size_t smem = sizeof(MemTile) + (size_t)MC * MC_LD * 4 + (size_t)MC * vdim * 4;
  B200_REQUIRE(smem <= 200 * 1024, "lm_matrix_memory: values of %d numbers do not fit shared memory", vdim);
  if (first_use_on_device(&g_mem_attr)) {
    B200_CUDA(cudaFuncSetAttribute(memory_out_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    B200_CUDA(cudaFuncSetAttribute(memory_out_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
  }
  const bool vec = ((dim | vdim | ldq | ldk | ldv) & 3) == 0 && (((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)p.chunk) & 15) == 0;
  const dim3 grid(cdiv(max_rows, MC), H, n_seq);
  if (vec) memory_chunk_kernel<true><<<grid, MC_THREADS, 0, cs>>>(p);
  else memory_chunk_kernel<false><<<grid, MC_THREADS, 0, cs>>>(p);
  B200_CHECK_LAUNCH();
  memory_chain_kernel<<<dim3(n_seq, H, cdiv((long)dim * (vdim + 1), 256)), 256, 0, cs>>>(p);
  B200_CHECK_LAUNCH();
  if (vec) memory_out_kernel<true><<<grid, MC_THREADS, smem, cs>>>(p);
  else memory_out_kernel<false><<<grid, MC_THREADS, smem, cs>>>(p);
  B200_CHECK_LAUNCH();
  return B200_OK;
}

}  // extern "C"
