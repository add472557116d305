// The gated delta rule: linear attention whose state is corrected, not only added to.
//
//   per head, with unit vectors k, q (q also scaled), a decay g and a step size beta per token:
//   S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q            S [dk, dv], float32
//   g is one number per head, or one per head and key channel (row d of S is multiplied by g_d)
//
//   delta_inputs   what enters the recurrence, from the projections of a step's tokens: the short
//                  causal convolution over time per channel (its last inputs kept per request),
//                  silu, unit norms, the query's factor, beta = sigmoid(b),
//                  g = exp(-exp(A_log) softplus(a + dt_bias)) (a, dt_bias and g per head, or per
//                  head and key channel) and the product k . q
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
// decays per channel there is no gate in the row and `a` comes as a tensor of its own (z); H
// more jobs make a value head's dk decays.
//
// The convolution of row i of a portion reads rows i - taps + 1 .. i, the first taps - 1 rows also
// the inputs kept from the step before (state [slots, taps - 1, channels], oldest first). The warp
// of a portion's row 0 makes all of these first rows and then writes the new state of its
// channels, so nobody else touches them. V channels per lane and visit, at most NK visits for a key
// head. TAPS: the number of taps (0: any; their inputs are then fetched one after another). STAGED:
// the inputs of all rows of the warp are fetched together into shared memory.
constexpr int DI_WARPS = 4, DI_MAX = 256;  // DI_MAX: largest key size

struct DeltaInputs {
  const float* proj;
  long long stride;
  const float* conv;    // [taps, C], C = 2 G dk + H dv; the last row is the current token's
  float* conv_state;    // [slots, taps - 1, C], or null when taps == 1
  const float* A_log;   // [H]
  const float* dt_bias; // [H], or [H, dk] beside z
  const int* token_seq;
  const int* cu_q;
  const int* ctx_lens;
  const int* slots;
  float* qkv;           // [T, C]
  float4* scal;         // [T, H]: (g, beta, k . q, 0); g = 1 beside z
  int T, H, G, dk, dv, taps;
  int rows;             // rows per warp
  float q_scale;
  int b_col;            // column of b; a, where it is part of the row, is at b_col + H
  const float* z;       // decays per channel: [T, H dk], rows z_stride apart; null: one decay per head
  long long z_stride;
  float* decay;         // [T, H dk], with z
};

__device__ __forceinline__ float dr_decay(float A, float x) {  // A = exp(A_log)
  const float softplus = fmaxf(x, 0.f) + log1pf(expf(-fabsf(x)));
  return expf(-A * softplus);
}

__device__ __forceinline__ void dr_copy(float* smem, const float* gmem, bool wide) {
  const uint32_t addr = (uint32_t)__cvta_generic_to_shared(smem);
  if (wide) asm volatile("cp.async.ca.shared.global [%0], [%1], 16;\n" ::"r"(addr), "l"(gmem));
  else asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"(addr), "l"(gmem));
}

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

template <int V, int TAPS, int NK, bool STAGED>
__global__ void __launch_bounds__(DI_WARPS * 32) delta_inputs_kernel(const DeltaInputs a) {
  extern __shared__ __align__(16) float di_smem[];
  pdl_trigger();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int job = blockIdx.y * DI_WARPS + warp;
  const bool is_qk = job < a.G;
  const int past = (TAPS > 0 ? TAPS : a.taps) - 1;
  const int C = 2 * a.G * a.dk + a.H * a.dv;
  const int t_begin = blockIdx.x * a.rows, t_end = min(a.T, t_begin + a.rows);
  const int d_lane = lane * V;
  // this warp's channels: one run of q and one of k, or one run of v
  const int len = is_qk ? a.dk : a.dv;
  const int ch0 = is_qk ? job * a.dk : 2 * a.G * a.dk + (job - a.G) * a.dv;
  const int ch1 = is_qk ? (a.G + job) * a.dk : 0;
  // the sequence of the row at hand: looked up again only where the next one starts
  int seq = a.token_seq[t_begin];
  int r0 = a.cu_q[seq], r1 = a.cu_q[seq + 1];
  bool from_zero = a.ctx_lens[seq] - (r1 - r0) == 0;
  float* st = a.conv_state ? a.conv_state + (size_t)a.slots[seq] * past * C : nullptr;
  pdl_wait();
  if (job >= a.G + a.H) {
    const int h = job - a.G - a.H;
    if (!a.z || h >= a.H) return;
    const float A = expf(a.A_log[h]);  // a value head's decays, channel by channel
    for (int t = t_begin; t < t_end; ++t) {
      const float* zp = a.z + (size_t)t * a.z_stride + (size_t)h * a.dk;
      float* out = a.decay + ((size_t)t * a.H + h) * a.dk;
      for (int d = d_lane; d < a.dk; d += 32 * V) {
        float x[V], bias[V];
        di_load<V>(zp + d, x);
        di_load<V>(a.dt_bias + (size_t)h * a.dk + d, bias);
#pragma unroll
        for (int e = 0; e < V; ++e) x[e] = dr_decay(A, x[e] + bias[e]);
        di_store<V>(out + d, x);
      }
    }
    return;
  }
  // STAGED: all inputs of the warp's rows (and of the rows just before them) are on their way together; a lane reads
  // back only what it copied itself
  const int s_begin = max(0, t_begin - past), width = max(2 * a.dk, a.dv);
  float* staged = STAGED ? di_smem + (size_t)warp * (a.rows + past) * width : nullptr;
  if constexpr (STAGED) {
    for (int t = s_begin; t < t_end; ++t) {
      const float* src = a.proj + (size_t)t * a.stride;
      float* dst = staged + (t - s_begin) * width;
      for (int d = d_lane; d < len; d += 32 * V) {
        dr_copy(dst + d, src + ch0 + d, V == 4);
        if (is_qk) dr_copy(dst + a.dk + d, src + ch1 + d, V == 4);
      }
    }
    asm volatile("cp.async.commit_group;\n" ::);
    asm volatile("cp.async.wait_group 0;\n" ::);
  }

  // x_j of row i: the input j rows back, of dims d .. d + V - 1 of run `second` (0: q or v, 1: k)
  auto input = [&](int i, int j, int second, int d, float (&x)[V]) {
    const int ch = (second ? ch1 : ch0) + d;
    const int t = r0 + i - j;
    if (i - j >= 0) {
      if (STAGED && t >= s_begin && t < t_end) di_load<V>(staged + (t - s_begin) * width + second * a.dk + d, x);
      else di_load<V>(a.proj + (size_t)t * a.stride + ch, x);
    } else if (!from_zero) {
      di_load<V>(st + (size_t)(past + i - j) * C + ch, x);
    } else {
#pragma unroll
      for (int e = 0; e < V; ++e) x[e] = 0.f;
    }
  };
  // the convolution of row i, then silu
  auto conv = [&](int i, int second, int d, float (&y)[V]) {
    const int ch = (second ? ch1 : ch0) + d;
    const bool alone = r1 - r0 == 1;  // a single row: the state moves on by one, while the inputs are at hand
    if constexpr (TAPS > 0) {
      float x[TAPS][V], w[TAPS][V];
      const bool direct = STAGED && i >= TAPS - 1 && r0 + i < t_end;  // all of it lies in shared memory
      const float* xp = staged + (direct ? (r0 + i - s_begin) * width + second * a.dk + d : 0);
#pragma unroll
      for (int j = 0; j < TAPS; ++j) {
        if (direct) di_load<V>(xp - j * width, x[j]);
        else input(i, j, second, d, x[j]);
        di_load<V>(a.conv + (size_t)(TAPS - 1 - j) * C + ch, w[j]);
      }
#pragma unroll
      for (int e = 0; e < V; ++e) y[e] = w[0][e] * x[0][e];
#pragma unroll
      for (int j = 1; j < TAPS; ++j)
#pragma unroll
        for (int e = 0; e < V; ++e) y[e] = fmaf(w[j][e], x[j][e], y[e]);
      if (alone)
#pragma unroll
        for (int j = 0; j + 1 < TAPS; ++j) di_store<V>(st + (size_t)(TAPS - 2 - j) * C + ch, x[j]);
    } else {
#pragma unroll
      for (int e = 0; e < V; ++e) y[e] = 0.f;
      for (int j = past; j >= 0; --j) {  // oldest first: a place of the state is read before it is written
        float x[V], w[V];
        input(i, j, second, d, x);
        di_load<V>(a.conv + (size_t)(past - j) * C + ch, w);
#pragma unroll
        for (int e = 0; e < V; ++e) y[e] = fmaf(w[e], x[e], y[e]);
        if (alone && j < past) di_store<V>(st + (size_t)(past - 1 - j) * C + ch, x);
      }
    }
#pragma unroll
    for (int e = 0; e < V; ++e) y[e] = __fdividef(y[e], 1.f + expf(-y[e]));
  };
  // the new state after a portion of several rows: its last inputs, oldest first
  auto keep = [&](int second, int d) {
    for (int s = 0; s < past; ++s) {
      float x[V];
      input(r1 - r0 - 1, past - 1 - s, second, d, x);  // (place s + rows of the old state: not written yet)
      di_store<V>(st + (size_t)s * C + (second ? ch1 : ch0) + d, x);
    }
  };
  // decay, step size and k . q of row t, value head h
  auto numbers = [&](int t, int h, float kq) {
    const float* p = a.proj + (size_t)t * a.stride + a.b_col + h;
    const float g = a.z ? 1.f : dr_decay(expf(a.A_log[h]), p[a.H] + a.dt_bias[h]);
    a.scal[(size_t)t * a.H + h] = make_float4(g, 1.f / (1.f + expf(-p[0])), kq, 0.f);
  };
  const int group = a.H / a.G;
  float kq_mine = 0.f;  // lane r: k . q of the warp's row r
  unsigned made = 0;    // rows of the warp whose numbers are still to be written
  for (int t = t_begin; t < t_end; ++t) {
    if (t >= r1) {
      seq = a.token_seq[t];
      r0 = a.cu_q[seq];
      r1 = a.cu_q[seq + 1];
      from_zero = a.ctx_lens[seq] - (r1 - r0) == 0;
      st = a.conv_state ? a.conv_state + (size_t)a.slots[seq] * past * C : nullptr;
    }
    const int i0 = t - r0, n = r1 - r0;
    if (i0 > 0 && i0 < past) continue;  // made by the warp of row 0
    const int i_end = i0 == 0 ? min(n, max(past, 1)) : i0 + 1;
    for (int i = i0; i < i_end; ++i) {
      float* row = a.qkv + (size_t)(r0 + i) * C;
      if (!is_qk) {
        for (int d = d_lane; d < len; d += 32 * V) {
          float y[V];
          conv(i, 0, d, y);
          di_store<V>(row + ch0 + d, y);
        }
        continue;
      }
      float q[NK][V], k[NK][V];
      float sq = 0.f, sk = 0.f, qk = 0.f;
#pragma unroll
      for (int c = 0; c < NK; ++c) {
        const int d = d_lane + 32 * V * c;
        if (d < len) {
          conv(i, 0, d, q[c]);
          conv(i, 1, d, k[c]);
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
      const float iq = a.q_scale * rsqrtf(sq + 1e-6f), ik = rsqrtf(sk + 1e-6f);
#pragma unroll
      for (int c = 0; c < NK; ++c) {
        const int d = d_lane + 32 * V * c;
        if (d < len) {
#pragma unroll
          for (int e = 0; e < V; ++e) {
            q[c][e] *= iq;
            k[c][e] *= ik;
          }
          di_store<V>(row + ch0 + d, q[c]);
          di_store<V>(row + ch1 + d, k[c]);
        }
      }
      const int r = r0 + i - t_begin;
      if (r < a.rows) {  // one of this warp's rows: its numbers are written at the end, a lane per row and head
        if (lane == r) kq_mine = qk * iq * ik;
        made |= 1u << r;
      } else {
        for (int h = job * group + lane; h < (job + 1) * group; h += 32) numbers(r0 + i, h, qk * iq * ik);
      }
    }
    if (i0 == 0 && n > 1)
      for (int d = d_lane; d < len; d += 32 * V) {
        keep(0, d);
        if (is_qk) keep(1, d);
      }
  }
  if (is_qk)
    for (int base = 0; base < a.rows * group; base += 32) {
      const int idx = base + lane, r = idx / group;
      const float kq = __shfl_sync(0xffffffffu, kq_mine, r & 31);
      if (r < a.rows && (made >> r & 1u)) numbers(t_begin + r, job * group + idx - r * group, kq);
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
// CH: decays per channel, staged beside q and k; the rows of S are multiplied first and the
// number per head is 1.
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
  const float* decay;  // [T, H dk]: a decay per channel; null: scal's number per head
};

template <int P, bool CH>
__global__ void __launch_bounds__(DR_THREADS) delta_rule_kernel(const DeltaRule a) {
  constexpr int CB = DR_THREADS / P;        // columns of this block
  constexpr int LD = P * DR_ROWS;           // a staged q or k row
  constexpr int R4 = DR_ROWS / 4;
  constexpr int PER = (CH ? 3 : 2) * DR_TT * LD + DR_TT * CB + DR_TT * 4;  // floats per buffer
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
    if constexpr (CH) {
      float* gs = ss + DR_TT * 4;
      for (int idx = threadIdx.x; idx < tn * ku; idx += DR_THREADS) {
        const int tt = idx / ku, i = (idx - tt * ku) * kstep;
        dr_copy(gs + tt * LD + i, a.decay + ((size_t)(r0 + t0 + tt) * H + h) * dk + i, wide_k);
      }
    }
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
    const float4* g4 = reinterpret_cast<const float4*>(vs + DR_TT * CB + DR_TT * 4) + p;
#pragma unroll 2
    for (int tt = 0; tt < tn; ++tt, k4 += LD / 4, q4 += LD / 4, g4 += CH ? LD / 4 : 0) {
      float kv[DR_ROWS];
      float kd0 = 0.f, kd1 = 0.f, qd0 = 0.f, qd1 = 0.f;
#pragma unroll
      for (int r = 0; r < R4; ++r) {
        const float4 k = k4[r * P], q = q4[r * P];
        if constexpr (CH) {
          const float4 g = g4[r * P];
          S[4 * r] *= g.x; S[4 * r + 1] *= g.y; S[4 * r + 2] *= g.z; S[4 * r + 3] *= g.w;
        }
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
      if constexpr (CH) {
        const float u = sc.y * (vs[tt * CB + jl] - kd);
#pragma unroll
        for (int r = 0; r < DR_ROWS; ++r) S[r] = fmaf(kv[r], u, S[r]);
        if (p == 0) os[tt * CB + jl] = fmaf(sc.z, u, qd);
      } else {
        const float u = sc.y * (vs[tt * CB + jl] - sc.x * kd);
#pragma unroll
        for (int r = 0; r < DR_ROWS; ++r) S[r] = fmaf(kv[r], u, sc.x * S[r]);
        if (p == 0) os[tt * CB + jl] = fmaf(sc.z, u, sc.x * qd);
      }
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
//
// With a decay per channel (CH) the products k_s . k_t and k_s . q_t are taken with every channel
// multiplied by its own r_ts, and G_t k_t, G_t q_t and r_(last,t) k_t channel by channel. Launch A has
// a form of its own for it; C then reads G q as A left it.
constexpr int DC_L = 64, DC_THREADS = 256, DC_B = 16, DC_B_THREADS = 256, DC_N = 64;
constexpr int DC_MAX_DV = 512;  // value sizes whose rows fit launch A's shared memory; longer ones run token by token

struct DeltaChunks {
  const float* qkv;    // as DeltaRule
  const float4* scal;
  float* state;
  float* out;
  const int* cu_q;
  const int* ctx_lens;
  const int* slots;
  const float* decay;  // [T, H dk] (CH)
  int H, G, dk, dv;
  int ld;              // row length of q, k, W and state rows: dk up to a multiple of 16, + 4 (zeros behind dk)
  int dvp;             // dv up to a multiple of DC_B
  int stages;          // launch B: chunks staged at a time
  // scratch per (chunk, head), laid out as the kernels stage it
  float* wk;           // [2][64][ld]: W, then r_(last,t) k_t
  float* u;            // [dvp / 16][64][16]: U, then u, in the slices of launch B
  float* p;            // [64][DC_LDP]
  float* s0;           // [dvp][ld]: the (transposed) state before the chunk
  float* g;            // [64]: G_t; CH: [ld]: G_last of every channel
  float* qg;           // CH: [64][ld]: G q
};
constexpr int DC_LDP = DC_L + 4;

// First chunk of a sequence in the scratch (only sequences of more than one chunk have any), and its chunks.
__device__ __forceinline__ int dc_first_chunk(const int* cu_q, int seq) {
  int base = 0;
  for (int s = 0; s < seq; ++s) {
    const int n = cu_q[s + 1] - cu_q[s];
    base += n > DC_L ? (n + DC_L - 1) / DC_L : 0;
  }
  return base;
}

// 64 rows, DC_THREADS / 64 threads each: row t < tn has `len` values (rows `stride` apart); what is left of 64 rows of
// `ld` floats is zero
__device__ __forceinline__ void dc_stage(float* dst, int ld, const float* src, long long stride, int tn, int len,
                                         bool wide) {
  constexpr int PER = DC_THREADS / DC_L;
  const int t = threadIdx.x / PER, q = threadIdx.x % PER;
  float* d = dst + t * ld;
  const float* s = src + (size_t)t * stride;
  if (wide) {
    for (int i = 4 * q; i < ld; i += 4 * PER) {
      if (t < tn && i < len) dr_copy(d + i, s + i, true);
      else *reinterpret_cast<float4*>(d + i) = make_float4(0.f, 0.f, 0.f, 0.f);
    }
  } else {
    for (int i = q; i < ld; i += PER) {
      if (t < tn && i < len) dr_copy(d + i, s + i, false);
      else d[i] = 0.f;
    }
  }
}
// n floats (a multiple of 4) as they lie
template <int THREADS>
__device__ __forceinline__ void dc_stage_flat(float* dst, const float* src, int n) {
  for (int i = 4 * threadIdx.x; i < n; i += 4 * THREADS) dr_copy(dst + i, src + i, true);
}
template <int THREADS>
__device__ __forceinline__ void dc_store_flat(float* dst, const float* src, int n) {
  for (int i = 4 * threadIdx.x; i < n; i += 4 * THREADS)
    *reinterpret_cast<float4*>(dst + i) = *reinterpret_cast<const float4*>(src + i);
}

// (I + M) X = factor X, unit lower triangular, X = the dk columns of W in ks (rows ld apart) and the dvp columns of U
// in qs; M in ms (rows DC_LDP apart, its strictly lower part is read); factor(is W, row) scales the right-hand sides.
template <typename F>
__device__ __forceinline__ void dc_solve(float* ks, int ld, int dk, float* qs, int dvp, const float* ms, F factor) {
  // Forward substitution in blocks of 16 rows, in place: two columns of W and U per thread (a row of M is
  // read once for both). What the rows of earlier blocks contribute comes from shared memory, the
  // block's own 16 values stay in registers.
  const int columns = dk + dvp, half = (columns + 1) / 2;
  for (int col = (int)threadIdx.x; col < half; col += DC_THREADS) {
    float* x[2];
    int xs[2];
    bool is_w[2];
#pragma unroll
    for (int v = 0; v < 2; ++v) {
      const int cc = col + v * half < columns ? col + v * half : col;  // (an odd number: one thread has its column twice)
      is_w[v] = cc < dk;
      x[v] = is_w[v] ? ks + cc : qs + (cc - dk);
      xs[v] = is_w[v] ? ld : dvp;
    }
#pragma unroll 1
    for (int b = 0; b < DC_L; b += 16) {
      float acc[2][16];
#pragma unroll
      for (int i = 0; i < 16; ++i) {
#pragma unroll
        for (int v = 0; v < 2; ++v) acc[v][i] = factor(is_w[v], b + i) * x[v][(b + i) * xs[v]];
      }
#pragma unroll 1
      for (int s = 0; s < b; s += 4) {
        float xv[2][4];
#pragma unroll
        for (int v = 0; v < 2; ++v)
#pragma unroll
          for (int e = 0; e < 4; ++e) xv[v][e] = x[v][(s + e) * xs[v]];
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          const float4 m = *reinterpret_cast<const float4*>(ms + (b + i) * DC_LDP + s);
#pragma unroll
          for (int v = 0; v < 2; ++v) {
            acc[v][i] = fmaf(-m.x, xv[v][0], acc[v][i]);
            acc[v][i] = fmaf(-m.y, xv[v][1], acc[v][i]);
            acc[v][i] = fmaf(-m.z, xv[v][2], acc[v][i]);
            acc[v][i] = fmaf(-m.w, xv[v][3], acc[v][i]);
          }
        }
      }
#pragma unroll
      for (int s = 0; s < 16; s += 4) {
        // the block's rows s .. s + 3 are finished one after another, the rows below take them off as they come
#pragma unroll
        for (int i = s + 1; i < 16; ++i) {
          const float4 m = *reinterpret_cast<const float4*>(ms + (b + i) * DC_LDP + b + s);
#pragma unroll
          for (int v = 0; v < 2; ++v) {
            acc[v][i] = fmaf(-m.x, acc[v][s], acc[v][i]);
            if (i > s + 1) acc[v][i] = fmaf(-m.y, acc[v][s + 1], acc[v][i]);
            if (i > s + 2) acc[v][i] = fmaf(-m.z, acc[v][s + 2], acc[v][i]);
            if (i > s + 3) acc[v][i] = fmaf(-m.w, acc[v][s + 3], acc[v][i]);
          }
        }
      }
#pragma unroll
      for (int i = 0; i < 16; ++i)
#pragma unroll
        for (int v = 0; v < 2; ++v) x[v][(b + i) * xs[v]] = acc[v][i];
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
  const int dk = a.dk, dv = a.dv, ld = a.ld, dvp = a.dvp, tid = threadIdx.x;
  const int kh = h / (a.H / a.G), C = 2 * a.G * dk + a.H * dv;
  const int t0 = r0 + c * DC_L, tn = min(DC_L, n - c * DC_L);
  float* ks = dc_smem;                   // [64][ld]: k, then W
  float* qs = ks + DC_L * ld;            // [64][ld]: q; then v and U, [64][dvp]
  float* ms = qs + DC_L * max(ld, dvp);  // [64][DC_LDP]: r, then M
  float* gs = ms + DC_L * DC_LDP;        // g [64], beta [64], G [64], r_(last,t) [64]
  pdl_wait();
  const float* row0 = a.qkv + (size_t)t0 * C;
  const bool wide = dk % 4 == 0 && C % 4 == 0;
  dc_stage(qs, ld, row0 + (size_t)kh * dk, C, tn, dk, wide);
  dc_stage(ks, ld, row0 + (size_t)(a.G + kh) * dk, C, tn, dk, wide);
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
      ms[t * DC_LDP + tid] = r;
    }
    gs[3 * DC_L + tid] = r;
  } else if (tid == DC_L) {
    float g = 1.f;
    for (int t = 0; t < DC_L; ++t) {
      g *= gs[t];
      gs[2 * DC_L + t] = g;
    }
  }
  asm volatile("cp.async.wait_group 0;\n" ::);
  __syncthreads();
  if (tid < DC_L) a.g[at * DC_L + tid] = gs[2 * DC_L + tid];
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
    __syncthreads();  // q is used up: v takes its place
    {
      const int t = tid >> 2;
      float* d = qs + t * dvp;
      const float* s = row0 + (size_t)t * C + (size_t)2 * a.G * dk + (size_t)h * dv;
      const bool wv = wide && dv % 4 == 0;
      const int step = wv ? 4 : 1;
      for (int i = (tid & 3) * step; i < dvp; i += 4 * step) {
        if (t < tn && i < dv) {
          dr_copy(d + i, s + i, wv);
        } else {
          for (int e = 0; e < step; ++e) d[i + e] = 0.f;
        }
      }
    }
    asm volatile("cp.async.commit_group;\n" ::);
    float* pg = a.p + at * DC_L * DC_LDP;
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int t = ty + 16 * i, s = tx + 16 * j;
        float m = 0.f, p = 0.f;
        if (s <= t) {
          const float r = ms[t * DC_LDP + s];
          p = r * qk[i][j];
          if (s < t) m = gs[DC_L + t] * r * kk[i][j];
        }
        pg[t * DC_LDP + s] = p;
        ms[t * DC_LDP + s] = m;  // this thread alone reads and writes the element
      }
  }
  {  // r_(last,t) k_t
    const int t = tid >> 2;
    const float rho = gs[3 * DC_L + t];
    float* kg = a.wk + at * 2 * DC_L * ld + (size_t)(DC_L + t) * ld;
    for (int i = 4 * (tid & 3); i < ld; i += 16) {
      const float4 k = *reinterpret_cast<const float4*>(ks + t * ld + i);
      *reinterpret_cast<float4*>(kg + i) = make_float4(rho * k.x, rho * k.y, rho * k.z, rho * k.w);
    }
  }
  asm volatile("cp.async.wait_group 0;\n" ::);
  __syncthreads();
  dc_solve(ks, ld, dk, qs, dvp, ms, [&](bool is_w, int i) { return is_w ? gs[DC_L + i] * gs[2 * DC_L + i] : gs[DC_L + i]; });
  __syncthreads();
  dc_store_flat<DC_THREADS>(a.wk + at * 2 * DC_L * ld, ks, DC_L * ld);
  float* ug = a.u + at * DC_L * dvp;
  const int t = tid >> 2, q = 4 * (tid & 3);
  for (int c0 = 0; c0 < dvp; c0 += DC_B)
    *reinterpret_cast<float4*>(ug + (size_t)c0 * DC_L + t * DC_B + q) =
        *reinterpret_cast<const float4*>(qs + t * dvp + c0 + q);
}

// ---- launch A, decays per channel
// The chunk is four blocks of 16 tokens. With F_t the product of a block's decays up to and with t, E_s that of
// the decays behind s in its block and B_b a whole block's, a token t of block i and a token s of an
// earlier block j have r_ts = F_t (B_(j+1) .. B_(i-1)) E_s: two products of factors in (0, 1], so a dot
// product of scaled vectors, (F k)_t . B (E k)_s, gives M and P between blocks. Within a block there is no
// such split that cannot underflow: there r_ts k_s is multiplied up token by token, a column s at a time.
// NR: pieces of four channels that a thread has of a column there (8 threads share a column).
constexpr int DC_BLOCK = 16, DC_BLOCKS = DC_L / DC_BLOCK;

static size_t channel_systems_floats(int ld, int dvp) {
  const int third = ld > DC_LDP ? ld : DC_LDP;
  return (size_t)DC_L * (ld + (ld > dvp ? ld : dvp) + third) + DC_BLOCKS * ld + DC_L + DC_BLOCKS * DC_BLOCK * DC_BLOCK;
}

template <int NR>
__global__ void __launch_bounds__(DC_THREADS, 2) delta_channel_systems_kernel(const DeltaChunks a) {
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
  const int dk = a.dk, dv = a.dv, ld = a.ld, dvp = a.dvp, tid = threadIdx.x;
  const int kh = h / (a.H / a.G), C = 2 * a.G * dk + a.H * dv;
  const int t0 = r0 + c * DC_L, tn = min(DC_L, n - c * DC_L);
  float* ks = dc_smem;                        // [64][ld]: k, then F k, then W
  float* qs = ks + DC_L * ld;                 // [64][ld]: q, then F q; then v and U, [64][dvp]
  float* gs = qs + DC_L * max(ld, dvp);       // [64][ld]: g, then E k; then M, [64][DC_LDP]
  float* bs = gs + DC_L * max(ld, DC_LDP);    // [4][ld]: B
  float* betas = bs + DC_BLOCKS * ld;         // [64]
  float* diag = betas + DC_L;                 // [4][16][16]: M within the blocks
  pdl_wait();
  const float* row0 = a.qkv + (size_t)t0 * C;
  const bool wide = dk % 4 == 0 && C % 4 == 0;
  dc_stage(qs, ld, row0 + (size_t)kh * dk, C, tn, dk, wide);
  dc_stage(ks, ld, row0 + (size_t)(a.G + kh) * dk, C, tn, dk, wide);
  dc_stage(gs, ld, a.decay + ((size_t)t0 * a.H + h) * dk, (long long)a.H * dk, tn, dk, wide);
  asm volatile("cp.async.commit_group;\n" ::);
  if (tid < DC_L) betas[tid] = tid < tn ? a.scal[(size_t)(t0 + tid) * a.H + h].y : 0.f;
  __syncwarp();
  if (const int t = tid >> 2; t >= tn)  // tokens that fill the chunk up do not decay (this warp has zeroed the row)
    for (int i = tid & 3; i < ld; i += 4) gs[t * ld + i] = 1.f;
  asm volatile("cp.async.wait_group 0;\n" ::);
  __syncthreads();
  float* pg = a.p + at * DC_L * DC_LDP;
  {
    // within the blocks: a thread has the pieces slice, slice + 8, ... of the columns s and s + 8 of its block
    const int slice = tid & 7, b = tid >> 6, s = (tid >> 3) & 7;
    const float* kb = ks + b * DC_BLOCK * ld;
    const float* qb = qs + b * DC_BLOCK * ld;
    const float* gb = gs + b * DC_BLOCK * ld;
    float run[2][NR][4];
#pragma unroll
    for (int v = 0; v < 2; ++v)
#pragma unroll
      for (int r = 0; r < NR; ++r) {
        const int d = 4 * (slice + 8 * r);
        float4 k = make_float4(0.f, 0.f, 0.f, 0.f);
        if (d < ld - 4) k = *reinterpret_cast<const float4*>(kb + (s + 8 * v) * ld + d);
        run[v][r][0] = k.x; run[v][r][1] = k.y; run[v][r][2] = k.z; run[v][r][3] = k.w;
      }
#pragma unroll 1
    for (int t = 0; t < DC_BLOCK; ++t) {
      float acc[2][2] = {{0.f, 0.f}, {0.f, 0.f}};  // [column][with k_t, with q_t]
#pragma unroll
      for (int r = 0; r < NR; ++r) {
        const int d = 4 * (slice + 8 * r);
        if (d >= ld - 4) continue;
        const float4 g = *reinterpret_cast<const float4*>(gb + t * ld + d);
        const float4 k = *reinterpret_cast<const float4*>(kb + t * ld + d);
        const float4 q = *reinterpret_cast<const float4*>(qb + t * ld + d);
#pragma unroll
        for (int v = 0; v < 2; ++v) {
          if (v == 1 && t < 8) continue;  // its columns have not begun
          if (t > s + 8 * v) {
            run[v][r][0] *= g.x; run[v][r][1] *= g.y; run[v][r][2] *= g.z; run[v][r][3] *= g.w;
          }
          acc[v][0] = fmaf(run[v][r][0], k.x, acc[v][0]);
          acc[v][1] = fmaf(run[v][r][0], q.x, acc[v][1]);
          acc[v][0] = fmaf(run[v][r][1], k.y, acc[v][0]);
          acc[v][1] = fmaf(run[v][r][1], q.y, acc[v][1]);
          acc[v][0] = fmaf(run[v][r][2], k.z, acc[v][0]);
          acc[v][1] = fmaf(run[v][r][2], q.z, acc[v][1]);
          acc[v][0] = fmaf(run[v][r][3], k.w, acc[v][0]);
          acc[v][1] = fmaf(run[v][r][3], q.w, acc[v][1]);
        }
      }
      // four sums over eight lanes: every step halves what a lane still carries
      const bool hi4 = slice & 4, hi2 = slice & 2;
      float x0 = hi4 ? acc[1][0] : acc[0][0], x1 = hi4 ? acc[1][1] : acc[0][1];
      x0 += __shfl_xor_sync(0xffffffffu, hi4 ? acc[0][0] : acc[1][0], 4);
      x1 += __shfl_xor_sync(0xffffffffu, hi4 ? acc[0][1] : acc[1][1], 4);
      float y = hi2 ? x1 : x0;
      y += __shfl_xor_sync(0xffffffffu, hi2 ? x0 : x1, 2);
      y += __shfl_xor_sync(0xffffffffu, y, 1);
      if (!(slice & 1)) {
        const int col = s + (hi4 ? 8 : 0), row = b * DC_BLOCK + t;
        if (hi2) pg[row * DC_LDP + b * DC_BLOCK + col] = col <= t ? y : 0.f;
        else diag[(b * DC_BLOCK + t) * DC_BLOCK + col] = betas[row] * y;  // (read for col < t only)
      }
    }
  }
  __syncthreads();
  for (int idx = tid; idx < DC_BLOCKS * (ld - 4); idx += DC_THREADS) {  // a channel of a block
    const int b = idx / (ld - 4), d = idx - b * (ld - 4);
    float* kp = ks + b * DC_BLOCK * ld + d;
    float* qp = qs + b * DC_BLOCK * ld + d;
    float* gp = gs + b * DC_BLOCK * ld + d;
    float k[DC_BLOCK], g[DC_BLOCK];
#pragma unroll
    for (int t = 0; t < DC_BLOCK; ++t) {
      k[t] = kp[t * ld];
      g[t] = gp[t * ld];
    }
    float f = 1.f, e = 1.f;
#pragma unroll
    for (int t = 0; t < DC_BLOCK; ++t) {
      f *= g[t];
      kp[t * ld] = k[t] * f;
      qp[t * ld] *= f;
    }
    bs[b * ld + d] = f;
#pragma unroll
    for (int t = DC_BLOCK - 1; t >= 0; --t) {
      gp[t * ld] = k[t] * e;
      e *= g[t];
    }
  }
  for (int i = tid; i < DC_L * 4; i += DC_THREADS) gs[(i >> 2) * ld + ld - 4 + (i & 3)] = 0.f;  // (the row's filling)
  if (tid < DC_BLOCKS * 4) bs[(tid >> 2) * ld + ld - 4 + (tid & 3)] = 0.f;
  __syncthreads();
  const int ty = tid >> 4, tx = tid & 15;
  float kk[6], qk[6];  // blocks (1,0) (2,0) (2,1) (3,0) (3,1) (3,2): rows ty + 16 i, columns tx + 16 j
#pragma unroll
  for (int i = 0; i < 6; ++i) kk[i] = qk[i] = 0.f;
  for (int d = 0; d < ld - 4; d += 4) {
    auto row = [&](const float* m, int r) { return *reinterpret_cast<const float4*>(m + r * ld + d); };
    auto mul = [](const float4& x, const float4& y) { return make_float4(x.x * y.x, x.y * y.y, x.z * y.z, x.w * y.w); };
    auto dot = [](const float4& x, const float4& y, float& acc) {
      acc = fmaf(x.x, y.x, acc);
      acc = fmaf(x.y, y.y, acc);
      acc = fmaf(x.z, y.z, acc);
      acc = fmaf(x.w, y.w, acc);
    };
    const float4 b1 = row(bs, 1), b2 = row(bs, 2);
    const float4 c10 = row(gs, tx), c21 = row(gs, tx + 16), c32 = row(gs, tx + 32);
    const float4 c20 = mul(c10, b1), c31 = mul(c21, b2), c30 = mul(c20, b2);
    const float4 k1 = row(ks, ty + 16), k2 = row(ks, ty + 32), k3 = row(ks, ty + 48);
    const float4 q1 = row(qs, ty + 16), q2 = row(qs, ty + 32), q3 = row(qs, ty + 48);
    dot(k1, c10, kk[0]); dot(q1, c10, qk[0]);
    dot(k2, c20, kk[1]); dot(q2, c20, qk[1]);
    dot(k2, c21, kk[2]); dot(q2, c21, qk[2]);
    dot(k3, c30, kk[3]); dot(q3, c30, qk[3]);
    dot(k3, c31, kk[4]); dot(q3, c31, qk[4]);
    dot(k3, c32, kk[5]); dot(q3, c32, qk[5]);
  }
#pragma unroll
  for (int i = 1, e = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < i; ++j, ++e) pg[(ty + 16 * i) * DC_LDP + tx + 16 * j] = qk[e];
  __syncthreads();
  {
    // G q and r_(last,t) k out, and the right-hand side of W: beta G k
    const int t = tid >> 2, b = t / DC_BLOCK;
    const float beta = betas[t];
    float* kg = a.wk + at * 2 * DC_L * ld + (size_t)(DC_L + t) * ld;
    float* qg = a.qg + (at * DC_L + t) * ld;
    for (int i = 4 * (tid & 3); i < ld; i += 16) {
      float4 before = make_float4(1.f, 1.f, 1.f, 1.f), behind = before;
#pragma unroll
      for (int o = 0; o < DC_BLOCKS; ++o) {
        const float4 w = *reinterpret_cast<const float4*>(bs + o * ld + i);
        if (o < b) { before.x *= w.x; before.y *= w.y; before.z *= w.z; before.w *= w.w; }
        if (o > b) { behind.x *= w.x; behind.y *= w.y; behind.z *= w.z; behind.w *= w.w; }
      }
      const float4 e = *reinterpret_cast<const float4*>(gs + t * ld + i);
      const float4 q = *reinterpret_cast<const float4*>(qs + t * ld + i);
      float4* kp = reinterpret_cast<float4*>(ks + t * ld + i);
      const float4 k = *kp;
      *reinterpret_cast<float4*>(kg + i) = make_float4(e.x * behind.x, e.y * behind.y, e.z * behind.z, e.w * behind.w);
      *reinterpret_cast<float4*>(qg + i) = make_float4(q.x * before.x, q.y * before.y, q.z * before.z, q.w * before.w);
      *kp = make_float4(beta * before.x * k.x, beta * before.y * k.y, beta * before.z * k.z, beta * before.w * k.w);
      if (t == 0) {
        const float4 w = *reinterpret_cast<const float4*>(bs + i);
        *reinterpret_cast<float4*>(a.g + at * ld + i) =
            make_float4(w.x * behind.x, w.y * behind.y, w.z * behind.z, w.w * behind.w);
      }
    }
  }
  __syncthreads();
  float* ms = gs;
  {
    const int t = tid >> 2;
    float* d = qs + t * dvp;
    const float* s = row0 + (size_t)t * C + (size_t)2 * a.G * dk + (size_t)h * dv;
    const bool wv = wide && dv % 4 == 0;
    const int step = wv ? 4 : 1;
    for (int i = (tid & 3) * step; i < dvp; i += 4 * step) {
      if (t < tn && i < dv) {
        dr_copy(d + i, s + i, wv);
      } else {
        for (int e = 0; e < step; ++e) d[i + e] = 0.f;
      }
    }
  }
  asm volatile("cp.async.commit_group;\n" ::);
#pragma unroll
  for (int i = 1, e = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < i; ++j, ++e) ms[(ty + 16 * i) * DC_LDP + tx + 16 * j] = betas[ty + 16 * i] * kk[e];
#pragma unroll
  for (int i = 0; i < 4; ++i) ms[(ty + 16 * i) * DC_LDP + tx + 16 * i] = diag[(16 * i + ty) * DC_BLOCK + tx];
  asm volatile("cp.async.wait_group 0;\n" ::);
  __syncthreads();
  dc_solve(ks, ld, dk, qs, dvp, ms, [&](bool is_w, int i) { return is_w ? 1.f : betas[i]; });
  __syncthreads();
  dc_store_flat<DC_THREADS>(a.wk + at * 2 * DC_L * ld, ks, DC_L * ld);
  float* ug = a.u + at * DC_L * dvp;
  const int t = tid >> 2, q = 4 * (tid & 3);
  for (int c0 = 0; c0 < dvp; c0 += DC_B)
    *reinterpret_cast<float4*>(ug + (size_t)c0 * DC_L + t * DC_B + q) =
        *reinterpret_cast<const float4*>(qs + t * dvp + c0 + q);
}

// ---- launch B
template <bool CH>
__global__ void __launch_bounds__(DC_B_THREADS) delta_chunk_states_kernel(const DeltaChunks a) {
  extern __shared__ __align__(16) float dc_smem[];
  pdl_trigger();
  const int dk = a.dk, dv = a.dv, ld = a.ld, tid = threadIdx.x;
  const int slices = a.dvp / DC_B;
  const int h = blockIdx.x / slices, slice = blockIdx.x - h * slices, c0 = slice * DC_B, seq = blockIdx.y;
  const int r0 = a.cu_q[seq], n = a.cu_q[seq + 1] - r0;
  if (n <= DC_L) {
    pdl_wait();
    return;
  }
  const int chunks = (n + DC_L - 1) / DC_L;
  const int cols = min(DC_B, dv - c0);
  const size_t first = (size_t)dc_first_chunk(a.cu_q, seq) * a.H + h;
  const int per = DC_L * (2 * ld + DC_B);  // a staged chunk: W, r k [64][ld] each, U [64][16]
  float* Ss = dc_smem + a.stages * per;    // [16][ld]: the state's columns
  float* part = Ss + DC_B * ld;            // sums of parts: [8][64][20] in the first product, [8][16][32] in the second
  pdl_wait();
  auto issue = [&](int c, float* ws) {
    const size_t at = first + (size_t)c * a.H;
    dc_stage_flat<DC_B_THREADS>(ws, a.wk + at * 2 * DC_L * ld, 2 * DC_L * ld);
    dc_stage_flat<DC_B_THREADS>(ws + 2 * DC_L * ld, a.u + at * DC_L * a.dvp + (size_t)c0 * DC_L, DC_L * DC_B);
    asm volatile("cp.async.commit_group;\n" ::);
  };
  issue(0, dc_smem);
  float* st = a.state + (((size_t)a.slots[seq] * a.H + h) * dv + c0) * dk;
  const bool read = a.ctx_lens[seq] - n > 0;
  for (int j = tid >> 5; j < DC_B; j += DC_B_THREADS / 32)
    for (int d = tid & 31; d < ld; d += 32)
      Ss[j * ld + d] = (read && j < cols && d < dk) ? __ldcg(st + (size_t)j * dk + d) : 0.f;
  // first product: a warp has an eighth of the key dims, its lanes rows rg + 8 i and columns cg + 4 j
  const int warp = tid >> 5, cg = tid & 3, rg = (tid & 31) >> 2;
  const int eighth = ((ld - 4) / 4 + 7) / 8 * 4, d0 = min(warp * eighth, ld - 4), d1 = min(d0 + eighth, ld - 4);
  // second product: a warp covers 32 key dims x 16 columns (tiles of four x four) and a part of the rows
  const int dims = (ld - 4 + 31) / 32;
  const int parts = dims == 1 ? 8 : dims == 2 ? 4 : dims <= 4 ? 2 : 1;
  const int tpart = warp / dims, trows = DC_L / parts;
  const int td = (warp - tpart * dims) * 32 + (tid & 7) * 4, tj = ((tid >> 3) & 3) * 4;
  for (int c = 0; c < chunks; ++c) {
    float* ws = dc_smem + (a.stages > 1 ? (c & 1) * per : 0);
    if (a.stages > 1 && c + 1 < chunks) {
      issue(c + 1, dc_smem + ((c + 1) & 1) * per);
      asm volatile("cp.async.wait_group 1;\n" ::);
    } else {
      asm volatile("cp.async.wait_group 0;\n" ::);
    }
    __syncthreads();
    const float* ks = ws + DC_L * ld;
    float* us = ws + 2 * DC_L * ld;
    const size_t at = first + (size_t)c * a.H;
    const float whole = CH ? 1.f : __ldg(a.g + at * DC_L + DC_L - 1);
    dc_store_flat<DC_B_THREADS>(a.s0 + (at * a.dvp + c0) * ld, Ss, DC_B * ld);
    float acc[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
    for (int d = d0; d < d1; d += 4) {
      float4 s[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) s[j] = *reinterpret_cast<const float4*>(Ss + (cg + 4 * j) * ld + d);
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const float4 w = *reinterpret_cast<const float4*>(ws + (rg + 8 * i) * ld + d);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          acc[i][j] = fmaf(w.x, s[j].x, acc[i][j]);
          acc[i][j] = fmaf(w.y, s[j].y, acc[i][j]);
          acc[i][j] = fmaf(w.z, s[j].z, acc[i][j]);
          acc[i][j] = fmaf(w.w, s[j].w, acc[i][j]);
        }
      }
    }
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) part[(warp * DC_L + rg + 8 * i) * 20 + cg + 4 * j] = acc[i][j];
    __syncthreads();
    {
      const int t = tid >> 2, q = 4 * (tid & 3);
      float4 u = *reinterpret_cast<const float4*>(us + t * DC_B + q);
#pragma unroll
      for (int g = 0; g < 8; ++g) {
        const float4 v = *reinterpret_cast<const float4*>(part + (g * DC_L + t) * 20 + q);
        u.x -= v.x; u.y -= v.y; u.z -= v.z; u.w -= v.w;
      }
      *reinterpret_cast<float4*>(us + t * DC_B + q) = u;
    }
    __syncthreads();
    dc_store_flat<DC_B_THREADS>(a.u + at * DC_L * a.dvp + (size_t)c0 * DC_L, us, DC_L * DC_B);
    if (tpart < parts) {
      float s[4][4];  // [column][dim]
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[j][e] = 0.f;
      const float* kp = ks + tpart * trows * ld + min(td, ld - 4);  // (dims beyond the row's: the zeros behind it)
      const float* up = us + tpart * trows * DC_B + tj;
#pragma unroll 8
      for (int t = 0; t < trows; ++t, kp += ld, up += DC_B) {
        const float4 k = *reinterpret_cast<const float4*>(kp);
        const float4 v = *reinterpret_cast<const float4*>(up);
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
      for (int j = 0; j < 4; ++j) store4<float>(part + (warp * DC_B + tj + j) * 32 + (tid & 7) * 4, s[j]);
    }
    __syncthreads();
    for (int b = tid >> 7; b < dims; b += 2) {
      const int j = (tid >> 3) & 15, d = b * 32 + (tid & 7) * 4;
      if (d >= ld - 4) continue;
      float4* p = reinterpret_cast<float4*>(Ss + j * ld + d);
      float4 o = *p;
      if constexpr (CH) {
        const float4 w = __ldg(reinterpret_cast<const float4*>(a.g + at * ld + d));
        o.x *= w.x; o.y *= w.y; o.z *= w.z; o.w *= w.w;
      } else {
        o.x *= whole; o.y *= whole; o.z *= whole; o.w *= whole;
      }
      for (int g = 0; g < parts; ++g) {
        const float4 v = *reinterpret_cast<const float4*>(part + ((g * dims + b) * DC_B + j) * 32 + (tid & 7) * 4);
        o.x += v.x; o.y += v.y; o.z += v.z; o.w += v.w;
      }
      *p = o;
    }
    __syncthreads();  // the state is whole, and the staged chunk is free
    if (a.stages == 1 && c + 1 < chunks) issue(c + 1, dc_smem);
  }
  for (int j = tid >> 5; j < cols; j += DC_B_THREADS / 32)
    for (int d = tid & 31; d < dk; d += 32) st[(size_t)j * dk + d] = Ss[j * ld + d];
}

// ---- launch C
template <bool CH>
__global__ void __launch_bounds__(DC_THREADS, 3) delta_chunk_outputs_kernel(const DeltaChunks a) {
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
  const int dk = a.dk, dv = a.dv, ld = a.ld, tid = threadIdx.x;
  const int kh = h / (a.H / a.G), C = 2 * a.G * dk + a.H * dv;
  const int t0 = r0 + c * DC_L, tn = min(DC_L, n - c * DC_L), cols = min(DC_N, a.dvp - c0);
  float* qs = dc_smem;            // [64][ld]; then P [64][DC_LDP]
  float* ss = qs + DC_L * ld;     // [64][ld]: columns of the state; then u, up to four slices of [64][16]
  pdl_wait();
  if constexpr (CH) dc_stage_flat<DC_THREADS>(qs, a.qg + at * DC_L * ld, DC_L * ld);
  else dc_stage(qs, ld, a.qkv + (size_t)t0 * C + (size_t)kh * dk, C, tn, dk, dk % 4 == 0 && C % 4 == 0);
  dc_stage_flat<DC_THREADS>(ss, a.s0 + (at * a.dvp + c0) * ld, cols * ld);
  asm volatile("cp.async.commit_group;\n" ::);
  asm volatile("cp.async.wait_group 0;\n" ::);
  __syncthreads();
  const int ty = tid >> 4, tx = tid & 15;  // rows ty + 16 i, columns tx + 16 j
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  // (columns beyond `cols` read what lies there: their sums are never stored)
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
  float* us = ps + DC_L * DC_LDP;
  dc_stage_flat<DC_THREADS>(ps, a.p + at * DC_L * DC_LDP, DC_L * DC_LDP);
  dc_stage_flat<DC_THREADS>(us, a.u + at * DC_L * a.dvp + (size_t)c0 * DC_L, cols * DC_L);
  asm volatile("cp.async.commit_group;\n" ::);
  if constexpr (!CH) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float g = __ldg(a.g + at * DC_L + ty + 16 * i);
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] *= g;
    }
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
        for (int j = 0; j < 4; ++j) u[e][j] = us[(j * DC_L + s + e) * DC_B + tx];
#pragma unroll
      for (int i = b; i < 4; ++i) {
        const float4 p = *reinterpret_cast<const float4*>(ps + (ty + 16 * i) * DC_LDP + s);
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
      if (c0 + tx + 16 * j < dv)
        a.out[(size_t)(t0 + t) * ((size_t)a.H * dv) + (size_t)h * dv + c0 + tx + 16 * j] = acc[i][j];
  }
}

}  // namespace lse

using namespace lse;

extern "C" int lse_delta_inputs(const float* proj, long long stride, const float* conv, int taps,
                                float* conv_state, const float* A_log, const float* dt_bias, const int* token_seq,
                                const int* cu_q, const int* ctx_lens, const int* slots, float* qkv, float* scal,
                                int T, int H, int G, int dk, int dv, float q_scale,
                                cudaStream_t stream, const float* z, long long z_stride, float* decay) {
  if (T <= 0) return LSE_OK;
  if (H <= 0 || G <= 0 || H % G || dk <= 0 || dk > DI_MAX || dv <= 0 || taps < 1 || (taps > 1 && !conv_state) ||
      stride < 2LL * G * dk + (z ? 1LL : 2LL) * H * (dv + 1) || (z && (!decay || z_stride < (long long)H * dk)))
    return LSE_BAD_ARGUMENT;
  DeltaInputs a;
  a.proj = proj; a.stride = stride; a.conv = conv; a.conv_state = taps > 1 ? conv_state : nullptr;
  a.A_log = A_log; a.dt_bias = dt_bias; a.token_seq = token_seq; a.cu_q = cu_q; a.ctx_lens = ctx_lens;
  a.slots = slots; a.qkv = qkv; a.scal = reinterpret_cast<float4*>(scal);
  a.T = T; a.H = H; a.G = G; a.dk = dk; a.dv = dv; a.taps = taps; a.q_scale = q_scale;
  a.b_col = 2 * G * dk + (z ? 1 : 2) * H * dv;
  a.z = z; a.z_stride = z_stride; a.decay = z ? decay : nullptr;
  const int jobs = (G + (z ? 2 : 1) * H + DI_WARPS - 1) / DI_WARPS;
  a.rows = (long long)T * jobs >= 16384 ? 8 : (long long)T * jobs >= 4096 ? 2 : 1;
  const dim3 grid((T + a.rows - 1) / a.rows, jobs);
  if (grid.y > 65535) return LSE_BAD_ARGUMENT;
  auto aligned = [](const void* p) { return reinterpret_cast<uintptr_t>(p) % 16 == 0; };
  // 16-byte accesses: every head starts on one in the projection, the taps, the kept inputs and the result
  const bool vec = dk % 4 == 0 && dv % 4 == 0 && stride % 4 == 0 && aligned(proj) && aligned(conv) &&
                   aligned(conv_state) && aligned(qkv) &&
                   (!z || (z_stride % 4 == 0 && aligned(z) && aligned(dt_bias) && aligned(decay)));
  const size_t smem = (size_t)DI_WARPS * (a.rows + taps - 1) * (2 * dk > dv ? 2 * dk : dv) * sizeof(float);
  const bool staged = vec && a.rows > 1 && smem <= 96 * 1024;
#define LSE_DI_LAUNCH(KERNEL, BYTES)                                                                              \
  do {                                                                                                            \
    if ((BYTES) > 48 * 1024 &&                                                                                    \
        cudaFuncSetAttribute(KERNEL, cudaFuncAttributeMaxDynamicSharedMemorySize, 96 * 1024) != cudaSuccess)      \
      return LSE_LAUNCH_FAILED;                                                                                   \
    launch(KERNEL, grid, DI_WARPS * 32, BYTES, stream, a);                                                        \
  } while (0)
#define LSE_DI(TAPS)                                                          \
  do {                                                                        \
    if (staged && dk <= 128) LSE_DI_LAUNCH((delta_inputs_kernel<4, TAPS, 1, true>), smem); \
    else if (staged) LSE_DI_LAUNCH((delta_inputs_kernel<4, TAPS, 2, true>), smem);         \
    else if (vec && dk <= 128) LSE_DI_LAUNCH((delta_inputs_kernel<4, TAPS, 1, false>), 0); \
    else if (vec) LSE_DI_LAUNCH((delta_inputs_kernel<4, TAPS, 2, false>), 0);              \
    else LSE_DI_LAUNCH((delta_inputs_kernel<1, TAPS, 8, false>), 0);                       \
  } while (0)
  if (taps == 4) LSE_DI(4);
  else if (taps == 3) LSE_DI(3);
  else if (taps == 2) LSE_DI(2);
  else LSE_DI(0);
#undef LSE_DI
#undef LSE_DI_LAUNCH
  return LSE_CHECK_LAUNCH();
}

template <int P, bool CH>
static int launch_delta_rule_form(const DeltaRule& a, int num_seqs, cudaStream_t stream) {
  constexpr int CB = DR_THREADS / P;
  constexpr size_t smem =
      (2 * ((CH ? 3 : 2) * DR_TT * P * DR_ROWS + DR_TT * CB + DR_TT * 4) + DR_TT * CB) * sizeof(float);
  static bool configured = false;
  if (smem > 48 * 1024 && !configured) {
    if (cudaFuncSetAttribute(delta_rule_kernel<P, CH>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
      return LSE_LAUNCH_FAILED;
    configured = true;
  }
  launch(delta_rule_kernel<P, CH>, dim3(a.H * ((a.dv + CB - 1) / CB), num_seqs), DR_THREADS, smem, stream, a);
  return LSE_CHECK_LAUNCH();
}
template <int P>
static int launch_delta_rule(const DeltaRule& a, int num_seqs, cudaStream_t stream) {
  return a.decay ? launch_delta_rule_form<P, true>(a, num_seqs, stream) : launch_delta_rule_form<P, false>(a, num_seqs, stream);
}

// Floats of scratch that one chunk of a portion longer than DC_L tokens needs.
static size_t chunk_floats(int H, int dk, int dv, bool channels) {
  const size_t ld = (dk + 15) / 16 * 16 + 4, dvp = (dv + DC_B - 1) / DC_B * DC_B;
  return (size_t)H * (DC_L * (2 * ld + dvp + DC_LDP) + dvp * ld + (channels ? (DC_L + 1) * ld : DC_L));
}
// Does launch A's working space for decays per channel fit a block? (If not, such portions run token by token.)
static bool channel_chunks_fit(int dk, int dv) {
  const int ld = (dk + 15) / 16 * 16 + 4, dvp = (dv + DC_B - 1) / DC_B * DC_B;
  return channel_systems_floats(ld, dvp) * sizeof(float) <= 227 * 1024;
}

extern "C" int lse_delta_rule_chunk(void) { return DC_L; }
extern "C" size_t lse_delta_rule_chunk_floats(int H, int dk, int dv, int channels) {
  return chunk_floats(H, dk, dv, channels != 0);
}

template <auto KERNEL>
static bool allow_smem(size_t bytes) {
  static size_t allowed = 48 * 1024;
  if (bytes <= allowed) return true;
  if (cudaFuncSetAttribute(KERNEL, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes) != cudaSuccess) return false;
  allowed = bytes;
  return true;
}

// The portions of more than DC_L tokens: max_chunks bounds the chunks of any sequence, total_chunks
// those of all such sequences together (what the scratch has room for).
template <bool CH>
static int launch_delta_chunks(const DeltaRule& r, int num_seqs, int max_chunks, float* scratch, int total_chunks,
                               cudaStream_t stream) {
  DeltaChunks a;
  a.qkv = r.qkv; a.scal = r.scal; a.state = r.state; a.out = r.out; a.cu_q = r.cu_q; a.ctx_lens = r.ctx_lens;
  a.slots = r.slots; a.H = r.H; a.G = r.G; a.dk = r.dk; a.dv = r.dv; a.decay = r.decay;
  a.ld = (r.dk + 15) / 16 * 16 + 4;
  a.dvp = (r.dv + DC_B - 1) / DC_B * DC_B;
  const size_t units = (size_t)total_chunks * r.H;
  a.g = scratch;
  a.p = a.g + units * (CH ? a.ld : DC_L);
  a.u = a.p + units * DC_L * DC_LDP;
  a.wk = a.u + units * DC_L * a.dvp;
  a.s0 = a.wk + units * 2 * DC_L * a.ld;
  a.qg = CH ? a.s0 + units * a.dvp * a.ld : nullptr;
  if (r.H > 65535 || max_chunks > 65535) return LSE_BAD_ARGUMENT;
  const size_t smem_a = CH ? channel_systems_floats(a.ld, a.dvp) * sizeof(float) :
      (size_t)(DC_L * a.ld + DC_L * (a.ld > a.dvp ? a.ld : a.dvp) + DC_L * DC_LDP + 4 * DC_L) * sizeof(float);
  const size_t per = (size_t)DC_L * (2 * a.ld + DC_B), rest = (size_t)DC_B * a.ld + 8 * DC_L * 20;
  a.stages = (2 * per + rest) * sizeof(float) <= 227 * 1024 ? 2 : 1;
  const size_t smem_b = (a.stages * per + rest) * sizeof(float);
  size_t smem_c = (size_t)2 * DC_L * a.ld * sizeof(float);
  const size_t second = (size_t)DC_L * (DC_LDP + DC_N) * sizeof(float);  // what the second product stages in the same place
  if (smem_c < second) smem_c = second;
  if (!allow_smem<delta_chunk_states_kernel<CH>>(smem_b) || !allow_smem<delta_chunk_outputs_kernel<CH>>(smem_c))
    return LSE_LAUNCH_FAILED;
  const dim3 grid_a(max_chunks, r.H, num_seqs);
  if constexpr (CH) {
    const int pieces = (a.ld - 4 + 31) / 32;  // of four channels, per thread
#define LSE_CHANNELS(NR)                                                                             \
  do {                                                                                               \
    if (!allow_smem<delta_channel_systems_kernel<NR>>(smem_a)) return LSE_LAUNCH_FAILED;             \
    launch(delta_channel_systems_kernel<NR>, grid_a, DC_THREADS, smem_a, stream, a);                 \
  } while (0)
    if (pieces <= 1) LSE_CHANNELS(1);
    else if (pieces <= 2) LSE_CHANNELS(2);
    else if (pieces <= 4) LSE_CHANNELS(4);
    else LSE_CHANNELS(8);
#undef LSE_CHANNELS
  } else {
    if (!allow_smem<delta_chunk_systems_kernel>(smem_a)) return LSE_LAUNCH_FAILED;
    launch(delta_chunk_systems_kernel, grid_a, DC_THREADS, smem_a, stream, a);
  }
  launch(delta_chunk_states_kernel<CH>, dim3(r.H * (a.dvp / DC_B), num_seqs), DC_B_THREADS, smem_b, stream, a);
  const int slices = r.H * ((r.dv + DC_N - 1) / DC_N);
  if (slices > 65535) return LSE_BAD_ARGUMENT;
  launch(delta_chunk_outputs_kernel<CH>, dim3(max_chunks, slices, num_seqs), DC_THREADS, smem_c, stream, a);
  return LSE_CHECK_LAUNCH();
}

extern "C" int lse_delta_rule(const float* qkv, const float* scal, float* state, float* out, const int* cu_q,
                              const int* ctx_lens, const int* slots, int num_seqs, int H, int G, int dk, int dv,
                              cudaStream_t stream, int max_chunks, float* scratch, int total_chunks, int short_too,
                              const float* decay) {
  if (num_seqs <= 0) return LSE_OK;
  if (max_chunks > 1 && (!scratch || total_chunks < 2)) return LSE_BAD_ARGUMENT;
  if (H <= 0 || G <= 0 || H % G || dk <= 0 || dk > DI_MAX || dv <= 0 || num_seqs > 65535) return LSE_BAD_ARGUMENT;
  DeltaRule a;
  a.qkv = qkv; a.scal = reinterpret_cast<const float4*>(scal); a.state = state; a.out = out; a.cu_q = cu_q;
  a.ctx_lens = ctx_lens; a.slots = slots; a.H = H; a.G = G; a.dk = dk; a.dv = dv; a.decay = decay;
  const bool chunked = max_chunks > 1 && dv <= DC_MAX_DV && (!decay || channel_chunks_fit(dk, dv));
  a.longest = chunked ? DC_L : 0;
  if (chunked) {
    const int code = decay ? launch_delta_chunks<true>(a, num_seqs, max_chunks, scratch, total_chunks, stream)
                           : launch_delta_chunks<false>(a, num_seqs, max_chunks, scratch, total_chunks, stream);
    if (code != LSE_OK || !short_too) return code;
  }
  const int lanes = (dk + DR_ROWS - 1) / DR_ROWS;
  if (lanes <= 1) return launch_delta_rule<1>(a, num_seqs, stream);
  if (lanes <= 2) return launch_delta_rule<2>(a, num_seqs, stream);
  if (lanes <= 4) return launch_delta_rule<4>(a, num_seqs, stream);
  if (lanes <= 8) return launch_delta_rule<8>(a, num_seqs, stream);
  return launch_delta_rule<16>(a, num_seqs, stream);
}
