// The gated delta rule: linear attention whose state is corrected, not only added to.
//
//   per head, with unit vectors k, q (q also scaled), a decay g and a step size beta per token:
//   S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q            S [dk, dv], float32
//
//   delta_inputs   what enters the recurrence, from the projections of a step's tokens: the short
//                  causal convolution over time per channel (its last inputs kept per request),
//                  silu, unit norms, the query's factor, beta = sigmoid(b),
//                  g = exp(-exp(A_log) softplus(a + dt_bias)) and the product k . q
//   delta_rule     the recurrence
//
// All arithmetic is float32. A request's states live in row slots[seq] of [slots, ...] tensors; a
// sequence whose first row of this step is at position 0 starts from zeros whatever its slot holds.
#include "common.cuh"
#include "kernels.h"

namespace lse {

#define LSE_CHECK_LAUNCH() (cudaPeekAtLastError() == cudaSuccess ? LSE_OK : LSE_LAUNCH_FAILED)

// ------------------------------------------------------------------------------------ inputs
// Columns of a row of the projection, from its column 0: q (G heads of dk) | k (G of dk) | v (H of dv)
// | gate (H of dv) | b (H) | a (H). One warp per (`rows` neighbouring rows, job): G jobs that make a key
// head's q and k and the numbers of its value heads, then H jobs that make a value head's v. With
// several rows a warp finds the inputs that neighbouring rows share in its SM's cache.
//
// The convolution of row i of a portion reads rows i - taps + 1 .. i, the first taps - 1 rows also
// the inputs kept from the step before (state [slots, taps - 1, channels], oldest first). The warp
// of a portion's row 0 makes all of these first rows and then writes the new state of its
// channels, so nobody else touches them. V channels per lane and visit.
constexpr int DI_WARPS = 4, DI_MAX = 256;  // DI_MAX: largest key size

struct DeltaInputs {
  const float* proj;
  long long stride;
  const float* conv;    // [taps, C], C = 2 G dk + H dv; the last row is the current token's
  float* conv_state;    // [slots, taps - 1, C], or null when taps == 1
  const float* A_log;   // [H]
  const float* dt_bias; // [H]
  const int* token_seq;
  const int* cu_q;
  const int* ctx_lens;
  const int* slots;
  float* qkv;           // [T, C]
  float4* scal;         // [T, H]: (g, beta, k . q, 0)
  int T, H, G, dk, dv, taps;
  int rows;             // rows per warp
  float q_scale;
};

template <int V>
__device__ __forceinline__ void di_load(const float* p, float (&v)[V]) {
  if constexpr (V == 4) load4<float>(p, v);
  else v[0] = p[0];
}
template <int V>
__device__ __forceinline__ void di_store(float* p, const float (&v)[V]) {
  if constexpr (V == 4) store4<float>(p, v);
  else p[0] = v[0];
}

template <int V>
__global__ void __launch_bounds__(DI_WARPS * 32) delta_inputs_kernel(const DeltaInputs a) {
  pdl_trigger();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int job = blockIdx.y * DI_WARPS + warp;
  const int past = a.taps - 1;
  pdl_wait();
  if (job >= a.G + a.H) return;
  const int t_end = min(a.T, (int)(blockIdx.x + 1) * a.rows);
  for (int t = blockIdx.x * a.rows; t < t_end; ++t) {
    const int seq = a.token_seq[t];
    const int r0 = a.cu_q[seq], n = a.cu_q[seq + 1] - r0;
    const int i0 = t - r0;  // this row's place in its portion
    if (i0 > 0 && i0 < past) continue;  // made by the warp of row 0
    const bool first = i0 == 0;
    const bool from_zero = a.ctx_lens[seq] - n == 0;
    const int C = 2 * a.G * a.dk + a.H * a.dv;
    float* st = a.conv_state ? a.conv_state + (size_t)a.slots[seq] * past * C : nullptr;
    const float* base = a.proj + (size_t)r0 * a.stride;

    // the convolution of row i, channels ch .. ch + V - 1, then silu
    auto conv = [&](int i, int ch, float (&y)[V]) {
      float x[V], w[V];
      di_load<V>(base + (size_t)i * a.stride + ch, x);
      di_load<V>(a.conv + (size_t)past * C + ch, w);
#pragma unroll
      for (int e = 0; e < V; ++e) y[e] = w[e] * x[e];
      for (int j = 1; j <= past; ++j) {
        float xp[V];
        if (i - j >= 0) {
          di_load<V>(base + (size_t)(i - j) * a.stride + ch, xp);
        } else if (from_zero) {
          break;
        } else {
          di_load<V>(st + (size_t)(past + i - j) * C + ch, xp);
        }
        di_load<V>(a.conv + (size_t)(past - j) * C + ch, w);
#pragma unroll
        for (int e = 0; e < V; ++e) y[e] = fmaf(w[e], xp[e], y[e]);
      }
      if (n == 1 && past > 0) {  // a single row: the state moves on by one, while x is at hand
        for (int s = 0; s + 1 < past; ++s) {
          float o[V];
#pragma unroll
          for (int e = 0; e < V; ++e) o[e] = 0.f;
          if (!from_zero) di_load<V>(st + (size_t)(s + 1) * C + ch, o);
          di_store<V>(st + (size_t)s * C + ch, o);
        }
        di_store<V>(st + (size_t)(past - 1) * C + ch, x);
      }
#pragma unroll
      for (int e = 0; e < V; ++e) y[e] = y[e] / (1.f + expf(-y[e]));
    };
    // the new state of channels ch .. after a portion of several rows: its last inputs
    auto keep = [&](int ch) {
      for (int s = 0; s < past; ++s) {
        const int i = n - past + s;
        float o[V];
#pragma unroll
        for (int e = 0; e < V; ++e) o[e] = 0.f;
        if (i >= 0) di_load<V>(base + (size_t)i * a.stride + ch, o);
        else if (!from_zero) di_load<V>(st + (size_t)(past + i) * C + ch, o);  // place s + n: not written yet
        di_store<V>(st + (size_t)s * C + ch, o);
      }
    };
    const int i_end = first ? min(n, max(past, 1)) : i0 + 1;
    if (job < a.G) {
      const int kh = job, group = a.H / a.G;
      const int qc = kh * a.dk, kc = (a.G + kh) * a.dk;
      constexpr int K = DI_MAX / (32 * V);
      for (int i = i0; i < i_end; ++i) {
        float q[K][V], k[K][V];
        float sq = 0.f, sk = 0.f, qk = 0.f;
#pragma unroll
        for (int c = 0; c < K; ++c) {
          const int d = (lane + 32 * c) * V;
          if (d < a.dk) {
            conv(i, qc + d, q[c]);
            conv(i, kc + d, k[c]);
#pragma unroll
            for (int e = 0; e < V; ++e) {
              sq += q[c][e] * q[c][e];
              sk += k[c][e] * k[c][e];
              qk += q[c][e] * k[c][e];
            }
          }
        }
        sq = warp_sum(sq);
        sk = warp_sum(sk);
        qk = warp_sum(qk);
        const float iq = a.q_scale / sqrtf(sq + 1e-6f), ik = 1.f / sqrtf(sk + 1e-6f);
        float* row = a.qkv + (size_t)(r0 + i) * C;
#pragma unroll
        for (int c = 0; c < K; ++c) {
          const int d = (lane + 32 * c) * V;
          if (d < a.dk) {
#pragma unroll
            for (int e = 0; e < V; ++e) {
              q[c][e] *= iq;
              k[c][e] *= ik;
            }
            di_store<V>(row + qc + d, q[c]);
            di_store<V>(row + kc + d, k[c]);
          }
        }
        for (int h = kh * group + lane; h < (kh + 1) * group; h += 32) {
          const float* p = base + (size_t)i * a.stride + C + a.H * a.dv + h;
          const float b = p[0], x = p[a.H] + a.dt_bias[h];
          const float softplus = fmaxf(x, 0.f) + log1pf(expf(-fabsf(x)));
          a.scal[(size_t)(r0 + i) * a.H + h] =
              make_float4(expf(-expf(a.A_log[h]) * softplus), 1.f / (1.f + expf(-b)), qk * iq * ik, 0.f);
        }
      }
      if (first && n > 1 && past > 0)
        for (int d = lane * V; d < a.dk; d += 32 * V) {
          keep(qc + d);
          keep(kc + d);
        }
    } else {
      const int h = job - a.G;
      const int vc = 2 * a.G * a.dk + h * a.dv;
      for (int i = i0; i < i_end; ++i)
        for (int d = lane * V; d < a.dv; d += 32 * V) {
          float y[V];
          conv(i, vc + d, y);
          di_store<V>(a.qkv + (size_t)(r0 + i) * C + vc + d, y);
        }
      if (first && n > 1 && past > 0)
        for (int d = lane * V; d < a.dv; d += 32 * V) keep(vc + d);
    }
  }
}

// ------------------------------------------------------------------------------------ recurrence
// The columns of S are independent of one another given k, q, g and beta, so a column of dk values
// is shared by P lanes (DR_ROWS rows each, in registers) and a block of DR_THREADS threads takes
// DR_THREADS / P columns of one head through all tokens of one sequence. Lane p holds the rows
// r * 4 P + 4 p + (0..3), r = 0 .. DR_ROWS / 4 - 1: neighbouring lanes read neighbouring 16-byte
// pieces, from the state in memory and from q and k in shared memory alike.
//
// Both products with the old state are formed at once and o follows from them:
//   u = beta (v - g S^T k),   o = g S^T q + (k . q) u,   S <- g S + k u^T
// which leaves one reduction over the P lanes on a token's critical path.
// q, k, v and the three numbers of DR_TT tokens are staged per pass, the next pass on its way
// (cp.async) while this one is computed. The state is stored transposed, [slot][head][dv][dk].
constexpr int DR_ROWS = 16, DR_THREADS = 128, DR_TT = 16;

struct DeltaRule {
  const float* qkv;    // [T, C]: q (G dk) | k (G dk) | v (H dv)
  const float4* scal;  // [T, H]
  float* state;        // [slots, H, dv, dk]
  float* out;          // [T, H dv]
  const int* cu_q;
  const int* ctx_lens;
  const int* slots;
  int H, G, dk, dv;
  int longest;         // longer portions than this are not served here (0: all are)
};

__device__ __forceinline__ void dr_copy(float* smem, const float* gmem, bool wide) {
  const uint32_t addr = (uint32_t)__cvta_generic_to_shared(smem);
  if (wide) asm volatile("cp.async.ca.shared.global [%0], [%1], 16;\n" ::"r"(addr), "l"(gmem));
  else asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"(addr), "l"(gmem));
}

template <int P>
__global__ void __launch_bounds__(DR_THREADS) delta_rule_kernel(const DeltaRule a) {
  constexpr int CB = DR_THREADS / P;        // columns of this block
  constexpr int LD = P * DR_ROWS;           // a staged q or k row
  constexpr int R4 = DR_ROWS / 4;
  constexpr int PER = 2 * DR_TT * LD + DR_TT * CB + DR_TT * 4;  // floats per buffer
  extern __shared__ __align__(16) float dr_smem[];
  float* os = dr_smem + 2 * PER;            // [DR_TT][CB] outputs of a pass
  pdl_trigger();
  const int dk = a.dk, dv = a.dv, H = a.H;
  const int slices = (dv + CB - 1) / CB;
  const int h = blockIdx.x / slices, c0 = (blockIdx.x - h * slices) * CB;
  const int kh = h / (H / a.G);
  const int seq = blockIdx.y;
  const int r0 = a.cu_q[seq], n = a.cu_q[seq + 1] - r0;
  const int C = 2 * a.G * dk + H * dv;
  if (a.longest > 0 && n > a.longest) {
    pdl_wait();
    return;
  }
  const int p = threadIdx.x % P, jl = threadIdx.x / P, j = c0 + jl;
  const bool has = j < dv;
  const int cols = min(CB, dv - c0);
  const bool wide_k = dk % 4 == 0 && C % 4 == 0, wide_v = wide_k && dv % 4 == 0;
  if (dk != LD || cols != CB)  // rows beyond dk and columns beyond dv stay zero in both buffers
    for (int i = threadIdx.x; i < 2 * PER; i += DR_THREADS) dr_smem[i] = 0.f;
  __syncthreads();
  pdl_wait();
  auto issue = [&](int buf, int t0) {
    float* ks = dr_smem + buf * PER;
    float* qs = ks + DR_TT * LD;
    float* vs = qs + DR_TT * LD;
    float* ss = vs + DR_TT * CB;
    const int tn = min(DR_TT, n - t0);
    const int ku = wide_k ? dk / 4 : dk, kstep = wide_k ? 4 : 1;
    for (int idx = threadIdx.x; idx < tn * ku; idx += DR_THREADS) {
      const int tt = idx / ku, i = (idx - tt * ku) * kstep;
      const float* row = a.qkv + (size_t)(r0 + t0 + tt) * C + (size_t)kh * dk + i;
      dr_copy(qs + tt * LD + i, row, wide_k);
      dr_copy(ks + tt * LD + i, row + (size_t)a.G * dk, wide_k);
    }
    const int vstep = wide_v ? 4 : 1, vu = (cols + vstep - 1) / vstep;
    for (int idx = threadIdx.x; idx < tn * vu; idx += DR_THREADS) {
      const int tt = idx / vu, i = (idx - tt * vu) * vstep;
      dr_copy(vs + tt * CB + i, a.qkv + (size_t)(r0 + t0 + tt) * C + (size_t)2 * a.G * dk + (size_t)h * dv + c0 + i, wide_v);
    }
    for (int tt = threadIdx.x; tt < tn; tt += DR_THREADS)
      dr_copy(ss + tt * 4, reinterpret_cast<const float*>(a.scal + (size_t)(r0 + t0 + tt) * H + h), true);
    asm volatile("cp.async.commit_group;\n" ::);
  };
  issue(0, 0);
  float S[DR_ROWS];
  float* st = a.state + (((size_t)a.slots[seq] * H + h) * dv + (has ? j : 0)) * dk;
  const bool read = has && a.ctx_lens[seq] - n > 0;
#pragma unroll
  for (int r = 0; r < R4; ++r) {
    const int row = (r * P + p) * 4;
    if (dk % 4 == 0) {
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (read && row < dk) v = __ldcg(reinterpret_cast<const float4*>(st + row));
      S[4 * r] = v.x; S[4 * r + 1] = v.y; S[4 * r + 2] = v.z; S[4 * r + 3] = v.w;
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e) S[4 * r + e] = (read && row + e < dk) ? st[row + e] : 0.f;
    }
  }
  int buf = 0;
  for (int t0 = 0; t0 < n; t0 += DR_TT, buf ^= 1) {
    const int tn = min(DR_TT, n - t0);
    if (t0 + DR_TT < n) {
      issue(buf ^ 1, t0 + DR_TT);
      asm volatile("cp.async.wait_group 1;\n" ::);
    } else {
      asm volatile("cp.async.wait_group 0;\n" ::);
    }
    __syncthreads();
    const float* ks = dr_smem + buf * PER;
    const float* qs = ks + DR_TT * LD;
    const float* vs = qs + DR_TT * LD;
    const float4* ss = reinterpret_cast<const float4*>(vs + DR_TT * CB);
    const float4* k4 = reinterpret_cast<const float4*>(ks) + p;
    const float4* q4 = reinterpret_cast<const float4*>(qs) + p;
#pragma unroll 2
    for (int tt = 0; tt < tn; ++tt, k4 += LD / 4, q4 += LD / 4) {
      float kv[DR_ROWS];
      float kd0 = 0.f, kd1 = 0.f, qd0 = 0.f, qd1 = 0.f;
#pragma unroll
      for (int r = 0; r < R4; ++r) {
        const float4 k = k4[r * P], q = q4[r * P];
        kv[4 * r] = k.x; kv[4 * r + 1] = k.y; kv[4 * r + 2] = k.z; kv[4 * r + 3] = k.w;
        kd0 = fmaf(S[4 * r], k.x, kd0);
        kd1 = fmaf(S[4 * r + 1], k.y, kd1);
        kd0 = fmaf(S[4 * r + 2], k.z, kd0);
        kd1 = fmaf(S[4 * r + 3], k.w, kd1);
        qd0 = fmaf(S[4 * r], q.x, qd0);
        qd1 = fmaf(S[4 * r + 1], q.y, qd1);
        qd0 = fmaf(S[4 * r + 2], q.z, qd0);
        qd1 = fmaf(S[4 * r + 3], q.w, qd1);
      }
      float kd = kd0 + kd1, qd = qd0 + qd1;
#pragma unroll
      for (int o = P >> 1; o > 0; o >>= 1) {
        kd += __shfl_xor_sync(0xffffffffu, kd, o);
        qd += __shfl_xor_sync(0xffffffffu, qd, o);
      }
      const float4 sc = ss[tt];
      const float u = sc.y * (vs[tt * CB + jl] - sc.x * kd);
#pragma unroll
      for (int r = 0; r < DR_ROWS; ++r) S[r] = fmaf(kv[r], u, sc.x * S[r]);
      if (p == 0) os[tt * CB + jl] = fmaf(sc.z, u, sc.x * qd);
    }
    __syncthreads();  // the outputs are there, and the buffer is free for the pass after the next
    for (int idx = threadIdx.x; idx < tn * cols; idx += DR_THREADS) {
      const int tt = idx / cols, c = idx - tt * cols;
      a.out[(size_t)(r0 + t0 + tt) * ((size_t)H * dv) + (size_t)h * dv + c0 + c] = os[tt * CB + c];
    }
    // (the next pass writes `os` only behind its own barrier)
  }
  if (!has || n == 0) return;
#pragma unroll
  for (int r = 0; r < R4; ++r) {
    const int row = (r * P + p) * 4;
    if (dk % 4 == 0) {
      if (row < dk) *reinterpret_cast<float4*>(st + row) = make_float4(S[4 * r], S[4 * r + 1], S[4 * r + 2], S[4 * r + 3]);
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (row + e < dk) st[row + e] = S[4 * r + e];
    }
  }
}

// ------------------------------------------------------------------------------------ long portions
// A portion of more than DC_L tokens runs as chunks of DC_L. Within a chunk that starts from the
// state S0 (transposed here: row c of S0 is column c of S), with G_t the product of the chunk's decays
// up to t and r_ts that of the decays s + 1 .. t, the recurrence unrolls to
//
//   u_t = beta_t v_t - beta_t G_t S0 k_t - sum_(s<t) M_ts u_s,      M_ts = beta_t r_ts (k_s . k_t)
//   o_t = G_t S0 q_t + sum_(s<=t) P_ts u_s,                         P_ts = r_ts (k_s . q_t)
//   S0 <- G_last S0 + sum_t r_(last,t) u_t k_t^T
//
// so that u = U - S0 W with (I + M) U = beta v and (I + M) W = beta G k, unit lower triangular systems that
// do not know S0. Three launches:
//   A  per chunk and head, all side by side: M, P, and U and W by forward substitution;
//   B  per head and slice of DC_B columns, chunk after chunk: u = U - S0 W and the next S0 (the states
//      before each chunk are kept);
//   C  per chunk, head and slice of columns, side by side: the outputs.
// All in float32 (register-tiled products on the CUDA cores); the decays enter as products of
// factors in (0, 1], so nothing overflows. A chunk that is not full is filled up with tokens of
// g = 1, beta = 0 and zero vectors.
constexpr int DC_L = 64, DC_THREADS = 256, DC_B = 16, DC_B_THREADS = 128, DC_N = 64;

struct DeltaChunks {
  const float* qkv;    // as DeltaRule
  const float4* scal;
  float* state;
  float* out;
  const int* cu_q;
  const int* ctx_lens;
  const int* slots;
  int H, G, dk, dv;
  int ldk;             // row length of staged q, k, w and state rows: dk up to a multiple of 8, + 4
  int stages;          // launch B: chunks staged at a time
  // scratch per (chunk, head)
  float* w;            // [64, dk]
  float* u;            // [64, dv]: U, then u
  float* p;            // [64, 64]
  float* s0;           // [dv, dk]: the state before the chunk
  float* coef;         // [2, 64]: G_t, r_(last,t)
};

// First chunk of a sequence in the scratch (only sequences of more than one chunk have any), and its chunks.
__device__ __forceinline__ int dc_first_chunk(const int* cu_q, int seq) {
  int base = 0;
  for (int s = 0; s < seq; ++s) {
    const int n = cu_q[s + 1] - cu_q[s];
    base += n > DC_L ? (n + DC_L - 1) / DC_L : 0;
  }
  return base;
}

// rows t < tn of `len` values, `stride` apart, into rows of `ld` floats; what is left of 64 rows and of `ld` is zero
__device__ __forceinline__ void dc_stage(float* dst, int ld, const float* src, long long stride, int tn, int len,
                                         bool wide, int rows, int tid, int threads) {
  if (wide) {
    const int per = ld / 4, full = len / 4;
    for (int idx = tid; idx < rows * per; idx += threads) {
      const int t = idx / per, i = idx - t * per;
      float* d = dst + (size_t)t * ld + 4 * i;
      if (t < tn && i < full) dr_copy(d, src + (size_t)t * stride + 4 * i, true);
      else *reinterpret_cast<float4*>(d) = make_float4(0.f, 0.f, 0.f, 0.f);
    }
  } else {
    for (int idx = tid; idx < rows * ld; idx += threads) {
      const int t = idx / ld, i = idx - t * ld;
      float* d = dst + (size_t)t * ld + i;
      if (t < tn && i < len) dr_copy(d, src + (size_t)t * stride + i, false);
      else *d = 0.f;
    }
  }
}

// ---- launch A
__global__ void __launch_bounds__(DC_THREADS, 2) delta_chunk_systems_kernel(const DeltaChunks a) {
  extern __shared__ __align__(16) float dc_smem[];
  pdl_trigger();
  const int c = blockIdx.x, h = blockIdx.y, seq = blockIdx.z;
  const int r0 = a.cu_q[seq], n = a.cu_q[seq + 1] - r0;
  const int chunks = n > DC_L ? (n + DC_L - 1) / DC_L : 0;
  if (c >= chunks) {
    pdl_wait();
    return;
  }
  const size_t at = (size_t)(dc_first_chunk(a.cu_q, seq) + c) * a.H + h;
  const int dk = a.dk, dv = a.dv, ld = a.ldk, tid = threadIdx.x;
  const int kh = h / (a.H / a.G), C = 2 * a.G * dk + a.H * dv;
  const int t0 = r0 + c * DC_L, tn = min(DC_L, n - c * DC_L);
  float* ks = dc_smem;                 // [64][ld]
  float* qs = ks + DC_L * ld;          // [64][ld]
  float* ms = qs + DC_L * ld;          // [64][68]: r, then M
  float* gs = ms + DC_L * 68;          // g [64], beta [64], G [64]
  pdl_wait();
  const float* row0 = a.qkv + (size_t)t0 * C + (size_t)kh * dk;
  const bool wide = dk % 4 == 0 && C % 4 == 0;
  dc_stage(qs, ld, row0, C, tn, dk, wide, DC_L, tid, DC_THREADS);
  dc_stage(ks, ld, row0 + (size_t)a.G * dk, C, tn, dk, wide, DC_L, tid, DC_THREADS);
  asm volatile("cp.async.commit_group;\n" ::);
  if (tid < DC_L) {
    const float4 s = tid < tn ? a.scal[(size_t)(t0 + tid) * a.H + h] : make_float4(1.f, 0.f, 0.f, 0.f);
    gs[tid] = s.x;
    gs[DC_L + tid] = s.y;
  }
  __syncthreads();
  if (tid < DC_L) {  // column s of r: the products of the decays behind s
    float r = 1.f;
    for (int t = tid; t < DC_L; ++t) {
      if (t > tid) r *= gs[t];
      ms[t * 68 + tid] = r;
    }
    a.coef[at * 2 * DC_L + DC_L + tid] = r;
  } else if (tid == DC_L) {
    float g = 1.f;
    for (int t = 0; t < DC_L; ++t) {
      g *= gs[t];
      gs[2 * DC_L + t] = g;
    }
  }
  asm volatile("cp.async.wait_group 0;\n" ::);
  __syncthreads();
  if (tid < DC_L) a.coef[at * 2 * DC_L + tid] = gs[2 * DC_L + tid];
  {
    // thread (ty, tx): rows ty + 16 i, columns tx + 16 j of K K^T and Q K^T, the blocks j <= i
    const int ty = tid >> 4, tx = tid & 15;
    float kk[4][4], qk[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) kk[i][j] = qk[i][j] = 0.f;
    for (int d = 0; d < ld - 4; d += 4) {
      float4 kc[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) kc[j] = *reinterpret_cast<const float4*>(ks + (tx + 16 * j) * ld + d);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float4 kr = *reinterpret_cast<const float4*>(ks + (ty + 16 * i) * ld + d);
        const float4 qr = *reinterpret_cast<const float4*>(qs + (ty + 16 * i) * ld + d);
#pragma unroll
        for (int j = 0; j <= i; ++j) {
          kk[i][j] = fmaf(kr.x, kc[j].x, kk[i][j]);
          kk[i][j] = fmaf(kr.y, kc[j].y, kk[i][j]);
          kk[i][j] = fmaf(kr.z, kc[j].z, kk[i][j]);
          kk[i][j] = fmaf(kr.w, kc[j].w, kk[i][j]);
          qk[i][j] = fmaf(qr.x, kc[j].x, qk[i][j]);
          qk[i][j] = fmaf(qr.y, kc[j].y, qk[i][j]);
          qk[i][j] = fmaf(qr.z, kc[j].z, qk[i][j]);
          qk[i][j] = fmaf(qr.w, kc[j].w, qk[i][j]);
        }
      }
    }
    float* pg = a.p + at * DC_L * DC_L;
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int t = ty + 16 * i, s = tx + 16 * j;
        float m = 0.f, p = 0.f;
        if (s <= t) {
          const float r = ms[t * 68 + s];
          p = r * qk[i][j];
          if (s < t) m = gs[DC_L + t] * r * kk[i][j];
        }
        pg[t * DC_L + s] = p;
        ms[t * 68 + s] = m;  // this thread alone reads and writes the element
      }
  }
  __syncthreads();
  // forward substitution, a column of W or U per thread, its 64 values in registers
  for (int col = tid; col < dk + dv; col += DC_THREADS) {
    const bool is_w = col < dk;
    const float* v = a.qkv + (size_t)t0 * C + (size_t)2 * a.G * dk + (size_t)h * dv + (col - dk);
    float* dst = is_w ? a.w + at * DC_L * dk + col : a.u + at * DC_L * dv + (col - dk);
    const int dst_stride = is_w ? dk : dv;
    float x[DC_L];
#pragma unroll
    for (int t = 0; t < DC_L; ++t) {
      float rhs = 0.f;
      if (is_w) rhs = gs[DC_L + t] * gs[2 * DC_L + t] * ks[t * ld + col];
      else if (t < tn) rhs = gs[DC_L + t] * v[(size_t)t * C];
      float e0 = 0.f, e1 = 0.f, e2 = 0.f, e3 = 0.f;
      const float4* m4 = reinterpret_cast<const float4*>(ms + t * 68);
#pragma unroll
      for (int s4 = 0; s4 < (t + 3) / 4; ++s4) {  // entries from t on are zero
        const float4 m = m4[s4];
        e0 = fmaf(m.x, x[4 * s4], e0);
        if (4 * s4 + 1 < t) e1 = fmaf(m.y, x[4 * s4 + 1], e1);
        if (4 * s4 + 2 < t) e2 = fmaf(m.z, x[4 * s4 + 2], e2);
        if (4 * s4 + 3 < t) e3 = fmaf(m.w, x[4 * s4 + 3], e3);
      }
      x[t] = rhs - ((e0 + e1) + (e2 + e3));
      dst[(size_t)t * dst_stride] = x[t];
    }
  }
}

// ---- launch B
__global__ void __launch_bounds__(DC_B_THREADS) delta_chunk_states_kernel(const DeltaChunks a) {
  extern __shared__ __align__(16) float dc_smem[];
  pdl_trigger();
  const int dk = a.dk, dv = a.dv, ld = a.ldk, tid = threadIdx.x;
  const int slices = (dv + DC_B - 1) / DC_B;
  const int h = blockIdx.x / slices, c0 = (blockIdx.x - h * slices) * DC_B, seq = blockIdx.y;
  const int r0 = a.cu_q[seq], n = a.cu_q[seq + 1] - r0;
  if (n <= DC_L) {
    pdl_wait();
    return;
  }
  const int chunks = (n + DC_L - 1) / DC_L;
  const int kh = h / (a.H / a.G), C = 2 * a.G * dk + a.H * dv;
  const int cols = min(DC_B, dv - c0);
  const size_t first = (size_t)dc_first_chunk(a.cu_q, seq) * a.H + h;
  const int per = DC_L * (2 * ld + DC_B + 2);  // a staged chunk: W, K [64][ld], U [64][16], the two factors [64]
  float* Ss = dc_smem + a.stages * per;        // [16][ld]: the state's columns
  float* Vs = Ss + DC_B * ld;                  // [64][20]: r_(last,t) u_t
  float* part = Vs + DC_L * 20;                // [64][20]: the sums of the second half of the key dims
  const bool wide = dk % 4 == 0 && C % 4 == 0, wide_u = dv % 4 == 0;
  pdl_wait();
  auto issue = [&](int c) {
    float* ws = dc_smem + (c % a.stages) * per;
    float* ks = ws + DC_L * ld;
    float* us = ks + DC_L * ld;
    const size_t at = first + (size_t)c * a.H;
    const int t0 = r0 + c * DC_L, tn = min(DC_L, n - c * DC_L);
    dc_stage(ws, ld, a.w + at * DC_L * dk, dk, DC_L, dk, wide, DC_L, tid, DC_B_THREADS);
    dc_stage(ks, ld, a.qkv + (size_t)t0 * C + (size_t)(a.G + kh) * dk, C, tn, dk, wide, DC_L, tid, DC_B_THREADS);
    dc_stage(us, DC_B, a.u + at * DC_L * dv + c0, dv, DC_L, cols, wide_u, DC_L, tid, DC_B_THREADS);
    if (tid < DC_L / 2) dr_copy(us + DC_L * DC_B + 4 * tid, a.coef + at * 2 * DC_L + 4 * tid, true);
    asm volatile("cp.async.commit_group;\n" ::);
  };
  issue(0);
  float* st = a.state + (((size_t)a.slots[seq] * a.H + h) * dv + c0) * dk;
  const bool read = a.ctx_lens[seq] - n > 0;
  for (int idx = tid; idx < DC_B * ld; idx += DC_B_THREADS) {
    const int c = idx / ld, d = idx - c * ld;
    Ss[idx] = (read && c < cols && d < dk) ? __ldcg(st + (size_t)c * dk + d) : 0.f;
  }
  const int grp = tid >> 6, cg = tid & 3, rg = (tid & 63) >> 2;  // first product: half of the key dims, columns, rows
  const int d_half = (ld - 4) / 2;
  for (int c = 0; c < chunks; ++c) {
    if (a.stages > 1 && c + 1 < chunks) {
      issue(c + 1);
      asm volatile("cp.async.wait_group 1;\n" ::);
    } else {
      asm volatile("cp.async.wait_group 0;\n" ::);
    }
    __syncthreads();
    const float* ws = dc_smem + (c % a.stages) * per;
    const float* ks = ws + DC_L * ld;
    float* us = dc_smem + (c % a.stages) * per + 2 * DC_L * ld;
    const float* gam = us + DC_L * DC_B;  // G_t, then r_(last,t)
    const size_t at = first + (size_t)c * a.H;
    float* s0 = a.s0 + (at * dv + c0) * dk;
    if (dk % 4 == 0) {
      for (int idx = tid; idx < cols * (dk / 4); idx += DC_B_THREADS) {
        const int j = idx / (dk / 4), d = (idx - j * (dk / 4)) * 4;
        *reinterpret_cast<float4*>(s0 + (size_t)j * dk + d) = *reinterpret_cast<const float4*>(Ss + j * ld + d);
      }
    } else {
      for (int idx = tid; idx < cols * dk; idx += DC_B_THREADS) {
        const int j = idx / dk, d = idx - j * dk;
        s0[(size_t)j * dk + d] = Ss[j * ld + d];
      }
    }
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
    {
      const float* wp = ws + rg * ld + grp * d_half;
      const float* sp = Ss + cg * ld + grp * d_half;
#pragma unroll 2
      for (int d = 0; d < d_half; d += 4) {
        float4 w[4], s[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) w[i] = *reinterpret_cast<const float4*>(wp + 16 * i * ld + d);
#pragma unroll
        for (int j = 0; j < 4; ++j) s[j] = *reinterpret_cast<const float4*>(sp + 4 * j * ld + d);
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            acc[i][j] = fmaf(w[i].x, s[j].x, acc[i][j]);
            acc[i][j] = fmaf(w[i].y, s[j].y, acc[i][j]);
            acc[i][j] = fmaf(w[i].z, s[j].z, acc[i][j]);
            acc[i][j] = fmaf(w[i].w, s[j].w, acc[i][j]);
          }
      }
    }
    if (grp == 1) {
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) part[(rg + 16 * i) * 20 + cg + 4 * j] = acc[i][j];
    }
    __syncthreads();
    if (grp == 0) {
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int t = rg + 16 * i;
        const float rho = gam[DC_L + t];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int cc = cg + 4 * j;
          const float u = us[t * DC_B + cc] - (acc[i][j] + part[t * 20 + cc]);
          us[t * DC_B + cc] = u;
          Vs[t * 20 + cc] = rho * u;
        }
      }
    }
    __syncthreads();
    {
      float* ug = a.u + at * DC_L * dv + c0;
      for (int idx = tid; idx < DC_L * cols; idx += DC_B_THREADS) {
        const int t = idx / cols, cc = idx - t * cols;
        ug[(size_t)t * dv + cc] = us[t * DC_B + cc];
      }
    }
    const float whole = gam[DC_L - 1];
    // the next state: tiles of four key dims x four columns
    for (int tile = tid; tile < (ld - 4 + 31) / 32 * 32; tile += DC_B_THREADS) {
      const int d = (tile >> 5) * 32 + (tile & 7) * 4, j0 = ((tile >> 3) & 3) * 4;  // a warp: 32 dims x 16 columns
      if (d >= ld - 4) continue;
      float s[4][4];  // [column][dim]
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[j][e] = 0.f;
#pragma unroll 4
      for (int t = 0; t < DC_L; ++t) {
        const float4 k = *reinterpret_cast<const float4*>(ks + t * ld + d);
        const float4 v = *reinterpret_cast<const float4*>(Vs + t * 20 + j0);
        const float vv[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          s[j][0] = fmaf(k.x, vv[j], s[j][0]);
          s[j][1] = fmaf(k.y, vv[j], s[j][1]);
          s[j][2] = fmaf(k.z, vv[j], s[j][2]);
          s[j][3] = fmaf(k.w, vv[j], s[j][3]);
        }
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        float4* p = reinterpret_cast<float4*>(Ss + (j0 + j) * ld + d);
        const float4 o = *p;
        *p = make_float4(fmaf(whole, o.x, s[j][0]), fmaf(whole, o.y, s[j][1]), fmaf(whole, o.z, s[j][2]),
                         fmaf(whole, o.w, s[j][3]));
      }
    }
    __syncthreads();  // the state is whole, and the staged chunk is free
    if (a.stages == 1 && c + 1 < chunks) issue(c + 1);
  }
  for (int idx = tid; idx < cols * dk; idx += DC_B_THREADS) {
    const int c = idx / dk, d = idx - c * dk;
    st[(size_t)c * dk + d] = Ss[c * ld + d];
  }
}

// ---- launch C
__global__ void __launch_bounds__(DC_THREADS) delta_chunk_outputs_kernel(const DeltaChunks a) {
  extern __shared__ __align__(16) float dc_smem[];
  pdl_trigger();
  const int slices = (a.dv + DC_N - 1) / DC_N;
  const int c = blockIdx.x, h = blockIdx.y / slices, c0 = (blockIdx.y - h * slices) * DC_N, seq = blockIdx.z;
  const int r0 = a.cu_q[seq], n = a.cu_q[seq + 1] - r0;
  const int chunks = n > DC_L ? (n + DC_L - 1) / DC_L : 0;
  if (c >= chunks) {
    pdl_wait();
    return;
  }
  const size_t at = (size_t)(dc_first_chunk(a.cu_q, seq) + c) * a.H + h;
  const int dk = a.dk, dv = a.dv, ld = a.ldk, tid = threadIdx.x;
  const int kh = h / (a.H / a.G), C = 2 * a.G * dk + a.H * dv;
  const int t0 = r0 + c * DC_L, tn = min(DC_L, n - c * DC_L), cols = min(DC_N, dv - c0);
  float* qs = dc_smem;            // [64][ld]; then P [64][68]
  float* ss = qs + DC_L * ld;     // [64][ld]: columns of the state; then u [64][68]
  pdl_wait();
  dc_stage(qs, ld, a.qkv + (size_t)t0 * C + (size_t)kh * dk, C, tn, dk, dk % 4 == 0 && C % 4 == 0, DC_L, tid, DC_THREADS);
  dc_stage(ss, ld, a.s0 + (at * dv + c0) * dk, dk, cols, dk, dk % 4 == 0, DC_N, tid, DC_THREADS);
  asm volatile("cp.async.commit_group;\n" ::);
  asm volatile("cp.async.wait_group 0;\n" ::);
  __syncthreads();
  const int ty = tid >> 4, tx = tid & 15;  // rows ty + 16 i, columns tx + 16 j
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
#pragma unroll 2
  for (int d = 0; d < ld - 4; d += 4) {
    float4 q[4], s[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) q[i] = *reinterpret_cast<const float4*>(qs + (ty + 16 * i) * ld + d);
#pragma unroll
    for (int j = 0; j < 4; ++j) s[j] = *reinterpret_cast<const float4*>(ss + (tx + 16 * j) * ld + d);
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        acc[i][j] = fmaf(q[i].x, s[j].x, acc[i][j]);
        acc[i][j] = fmaf(q[i].y, s[j].y, acc[i][j]);
        acc[i][j] = fmaf(q[i].z, s[j].z, acc[i][j]);
        acc[i][j] = fmaf(q[i].w, s[j].w, acc[i][j]);
      }
  }
  __syncthreads();
  float* ps = dc_smem;
  float* us = ps + DC_L * 68;
  dc_stage(ps, 68, a.p + at * DC_L * DC_L, DC_L, DC_L, DC_L, true, DC_L, tid, DC_THREADS);
  dc_stage(us, 68, a.u + at * DC_L * dv + c0, dv, DC_L, cols, dv % 4 == 0, DC_L, tid, DC_THREADS);
  asm volatile("cp.async.commit_group;\n" ::);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float g = __ldg(a.coef + at * 2 * DC_L + ty + 16 * i);
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] *= g;
  }
  asm volatile("cp.async.wait_group 0;\n" ::);
  __syncthreads();
#pragma unroll
  for (int b = 0; b < 4; ++b) {  // keys of block b reach rows of the blocks i >= b
#pragma unroll
    for (int s = 16 * b; s < 16 * b + 16; s += 4) {
      float u[4][4];
#pragma unroll
      for (int e = 0; e < 4; ++e)
#pragma unroll
        for (int j = 0; j < 4; ++j) u[e][j] = us[(s + e) * 68 + tx + 16 * j];
#pragma unroll
      for (int i = b; i < 4; ++i) {
        const float4 p = *reinterpret_cast<const float4*>(ps + (ty + 16 * i) * 68 + s);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          acc[i][j] = fmaf(p.x, u[0][j], acc[i][j]);
          acc[i][j] = fmaf(p.y, u[1][j], acc[i][j]);
          acc[i][j] = fmaf(p.z, u[2][j], acc[i][j]);
          acc[i][j] = fmaf(p.w, u[3][j], acc[i][j]);
        }
      }
    }
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int t = ty + 16 * i;
    if (t >= tn) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (tx + 16 * j < cols)
        a.out[(size_t)(t0 + t) * ((size_t)a.H * dv) + (size_t)h * dv + c0 + tx + 16 * j] = acc[i][j];
  }
}

}  // namespace lse

using namespace lse;

extern "C" int lse_delta_inputs(const float* proj, long long stride, const float* conv, int taps,
                                float* conv_state, const float* A_log, const float* dt_bias, const int* token_seq,
                                const int* cu_q, const int* ctx_lens, const int* slots, float* qkv, float* scal,
                                int T, int H, int G, int dk, int dv, float q_scale,
                                cudaStream_t stream) {
  if (T <= 0) return LSE_OK;
  if (H <= 0 || G <= 0 || H % G || dk <= 0 || dk > DI_MAX || dv <= 0 || taps < 1 || (taps > 1 && !conv_state) ||
      stride < 2LL * G * dk + 2LL * H * dv + 2LL * H)
    return LSE_BAD_ARGUMENT;
  DeltaInputs a;
  a.proj = proj; a.stride = stride; a.conv = conv; a.conv_state = taps > 1 ? conv_state : nullptr;
  a.A_log = A_log; a.dt_bias = dt_bias; a.token_seq = token_seq; a.cu_q = cu_q; a.ctx_lens = ctx_lens;
  a.slots = slots; a.qkv = qkv; a.scal = reinterpret_cast<float4*>(scal);
  a.T = T; a.H = H; a.G = G; a.dk = dk; a.dv = dv; a.taps = taps; a.q_scale = q_scale;
  const int jobs = (G + H + DI_WARPS - 1) / DI_WARPS;
  a.rows = (long long)T * jobs >= 16384 ? 8 : (long long)T * jobs >= 4096 ? 2 : 1;
  const dim3 grid((T + a.rows - 1) / a.rows, jobs);
  if (grid.y > 65535) return LSE_BAD_ARGUMENT;
  auto aligned = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
  // 16-byte accesses: every head starts on one in the projection, the taps, the kept inputs and the result
  const bool vec = dk % 4 == 0 && dv % 4 == 0 && stride % 4 == 0 && aligned(proj) && aligned(conv) &&
                   aligned(conv_state) && aligned(qkv);
  launch(vec ? delta_inputs_kernel<4> : delta_inputs_kernel<1>, grid, DI_WARPS * 32, 0, stream, a);
  return LSE_CHECK_LAUNCH();
}

template <int P>
static int launch_delta_rule(const DeltaRule& a, int num_seqs, cudaStream_t stream) {
  constexpr int CB = DR_THREADS / P;
  constexpr size_t smem =
      (2 * (2 * DR_TT * P * DR_ROWS + DR_TT * CB + DR_TT * 4) + DR_TT * CB) * sizeof(float);
  static bool configured = false;
  if (smem > 48 * 1024 && !configured) {
    if (cudaFuncSetAttribute(delta_rule_kernel<P>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
      return LSE_LAUNCH_FAILED;
    configured = true;
  }
  launch(delta_rule_kernel<P>, dim3(a.H * ((a.dv + CB - 1) / CB), num_seqs), DR_THREADS, smem, stream, a);
  return LSE_CHECK_LAUNCH();
}

// Floats of scratch that one chunk of a portion longer than DC_L tokens needs.
static size_t chunk_floats(int H, int dk, int dv) {
  return (size_t)H * (DC_L * (size_t)(dk + dv + DC_L + 2) + (size_t)dv * dk);
}

extern "C" int lse_delta_rule_chunk(void) { return DC_L; }
extern "C" size_t lse_delta_rule_chunk_floats(int H, int dk, int dv) { return chunk_floats(H, dk, dv); }

template <typename K>
static bool allow_smem(K kernel, size_t bytes) {
  return bytes <= 48 * 1024 ||
         cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes) == cudaSuccess;
}

// The portions of more than DC_L tokens: max_chunks bounds the chunks of any sequence, total_chunks
// those of all such sequences together (what the scratch has room for).
static int launch_delta_chunks(const DeltaRule& r, int num_seqs, int max_chunks, float* scratch, int total_chunks,
                               cudaStream_t stream) {
  DeltaChunks a;
  a.qkv = r.qkv; a.scal = r.scal; a.state = r.state; a.out = r.out; a.cu_q = r.cu_q; a.ctx_lens = r.ctx_lens;
  a.slots = r.slots; a.H = r.H; a.G = r.G; a.dk = r.dk; a.dv = r.dv;
  a.ldk = (r.dk + 7) / 8 * 8 + 4;
  const size_t units = (size_t)total_chunks * r.H;
  // the parts that are read as 16-byte vectors whatever the sizes are come first
  a.coef = scratch;
  a.p = a.coef + units * 2 * DC_L;
  a.w = a.p + units * DC_L * DC_L;
  a.u = a.w + units * DC_L * r.dk;
  a.s0 = a.u + units * DC_L * r.dv;
  if (r.H > 65535 || max_chunks > 65535) return LSE_BAD_ARGUMENT;
  const size_t smem_a = (size_t)(2 * DC_L * a.ldk + DC_L * 68 + 3 * DC_L) * sizeof(float);
  const size_t per = (size_t)DC_L * (2 * a.ldk + DC_B + 2), rest = (size_t)DC_B * a.ldk + 2 * DC_L * 20;
  a.stages = (2 * per + rest) * sizeof(float) <= 227 * 1024 ? 2 : 1;
  const size_t smem_b = (a.stages * per + rest) * sizeof(float);
  size_t smem_c = (size_t)2 * DC_L * a.ldk * sizeof(float);
  if (smem_c < (size_t)2 * DC_L * 68 * sizeof(float)) smem_c = (size_t)2 * DC_L * 68 * sizeof(float);
  if (!allow_smem(delta_chunk_systems_kernel, smem_a) || !allow_smem(delta_chunk_states_kernel, smem_b) ||
      !allow_smem(delta_chunk_outputs_kernel, smem_c))
    return LSE_LAUNCH_FAILED;
  launch(delta_chunk_systems_kernel, dim3(max_chunks, r.H, num_seqs), DC_THREADS, smem_a, stream, a);
  launch(delta_chunk_states_kernel, dim3(r.H * ((r.dv + DC_B - 1) / DC_B), num_seqs), DC_B_THREADS, smem_b, stream, a);
  const int slices = r.H * ((r.dv + DC_N - 1) / DC_N);
  if (slices > 65535) return LSE_BAD_ARGUMENT;
  launch(delta_chunk_outputs_kernel, dim3(max_chunks, slices, num_seqs), DC_THREADS, smem_c, stream, a);
  return LSE_CHECK_LAUNCH();
}

extern "C" int lse_delta_rule(const float* qkv, const float* scal, float* state, float* out, const int* cu_q,
                              const int* ctx_lens, const int* slots, int num_seqs, int H, int G, int dk, int dv,
                              cudaStream_t stream, int max_chunks, float* scratch, int total_chunks, int short_too) {
  if (num_seqs <= 0) return LSE_OK;
  if (max_chunks > 1 && (!scratch || total_chunks < 2)) return LSE_BAD_ARGUMENT;
  if (H <= 0 || G <= 0 || H % G || dk <= 0 || dk > DI_MAX || dv <= 0 || num_seqs > 65535) return LSE_BAD_ARGUMENT;
  DeltaRule a;
  a.qkv = qkv; a.scal = reinterpret_cast<const float4*>(scal); a.state = state; a.out = out; a.cu_q = cu_q;
  a.ctx_lens = ctx_lens; a.slots = slots; a.H = H; a.G = G; a.dk = dk; a.dv = dv;
  a.longest = max_chunks > 1 ? DC_L : 0;
  if (max_chunks > 1) {
    const int code = launch_delta_chunks(a, num_seqs, max_chunks, scratch, total_chunks, stream);
    if (code != LSE_OK || !short_too) return code;
  }
  const int lanes = (dk + DR_ROWS - 1) / DR_ROWS;
  if (lanes <= 1) return launch_delta_rule<1>(a, num_seqs, stream);
  if (lanes <= 2) return launch_delta_rule<2>(a, num_seqs, stream);
  if (lanes <= 4) return launch_delta_rule<4>(a, num_seqs, stream);
  if (lanes <= 8) return launch_delta_rule<8>(a, num_seqs, stream);
  return launch_delta_rule<16>(a, num_seqs, stream);
}
