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
// | gate (H of dv) | b (H) | a (H). One warp per (row, job): G jobs that make a key head's q and k
// and the numbers of its value heads, then H jobs that make a value head's v.
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
  const int t = blockIdx.x;
  if (job >= a.G + a.H) {
    pdl_wait();
    return;
  }
  const int seq = a.token_seq[t];
  const int r0 = a.cu_q[seq], n = a.cu_q[seq + 1] - r0;
  const int i0 = t - r0;  // this row's place in its portion
  const int past = a.taps - 1;
  pdl_wait();
  if (i0 > 0 && i0 < past) return;  // made by the warp of row 0
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
  const dim3 grid(T, (G + H + DI_WARPS - 1) / DI_WARPS);
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

extern "C" int lse_delta_rule(const float* qkv, const float* scal, float* state, float* out, const int* cu_q,
                              const int* ctx_lens, const int* slots, int num_seqs, int H, int G, int dk, int dv,
                              cudaStream_t stream) {
  if (num_seqs <= 0) return LSE_OK;
  if (H <= 0 || G <= 0 || H % G || dk <= 0 || dk > DI_MAX || dv <= 0 || num_seqs > 65535) return LSE_BAD_ARGUMENT;
  DeltaRule a;
  a.qkv = qkv; a.scal = reinterpret_cast<const float4*>(scal); a.state = state; a.out = out; a.cu_q = cu_q;
  a.ctx_lens = ctx_lens; a.slots = slots; a.H = H; a.G = G; a.dk = dk; a.dv = dv;
  const int lanes = (dk + DR_ROWS - 1) / DR_ROWS;
  if (lanes <= 1) return launch_delta_rule<1>(a, num_seqs, stream);
  if (lanes <= 2) return launch_delta_rule<2>(a, num_seqs, stream);
  if (lanes <= 4) return launch_delta_rule<4>(a, num_seqs, stream);
  if (lanes <= 8) return launch_delta_rule<8>(a, num_seqs, stream);
  return launch_delta_rule<16>(a, num_seqs, stream);
}
