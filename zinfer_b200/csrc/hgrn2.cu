// Gated linear recurrence with a matrix state per head (HGRN2): per head a state S [d, e],
//
//     S_t = diag(f_t) S_{t-1} + (1 - f_t) v_t^T,        o_t = S_t^T q_t,
//
// f_t in (lower, 1) the forget gate per head and channel; 1 - f_t is the share of v_t that enters the state
// (no key projection), q_t = silu(.), v_t plain.  A row of `qfv` holds the three projections of a token,
// [q (H*d) | f (H*d) | v (H*e)], float32 as the contraction left them; hgrn2_gates_kernel turns the first
// two parts, in place, into silu(q) and the gate f = lower + (1 - lower) * sigmoid(z_f + bias), once for
// all the blocks of the recurrence that read them.  Everything here is float32: gate, state, sums.
//
// One kernel serves prompt steps and single-token steps.  A block owns one (sequence, head, 32 value columns)
// and walks the sequence's tokens in order, from the state the step before left in `state[slot]` to the
// state it leaves there.  Its eight warps split the d channels: warp w keeps rows [w*DPT, (w+1)*DPT) of the
// 32 columns of S in registers (lane = column, so the state is read and written in whole lines), adds up its
// part of o_t = sum_i S_t[i, c] q_t[i], and the parts of sixteen tokens at a time meet in shared memory, where
// warp w sums those of tokens w and w + 8 in the order of the warps.  q and f of the next sixteen tokens are fetched into
// registers while the current sixteen are worked on, and go into the other half of a double buffer.  The order of every sum is fixed by the layout alone, so a
// sequence cut into steps gives the same bits as the whole.
//
// The same kernel runs three more recurrences.  KEYED: a retention layer's, a key projection in place of the gate and one
// fixed decay per head, S_t = decay_h S_{t-1} + k_t v_t^T; retention_prepare_kernel rotates q and k and scales k first.
// STEPPED: a state-space layer's (Mamba-2), whose step size dt_t > 0 per head and token sets both the decay and what enters,
// S_t = exp(-exp(A_log_h) dt_t) S_{t-1} + dt_t k_t v_t^T, o_t = S_t^T q_t + skip_h v_t, with k and q shared by the heads of
// a group; lane i of every warp turns the raw step size of a group's token i into dt = softplus(z + bias) and the decay.
// CAPPED: a matrix memory with exponential gates (the mLSTM of xLSTM): the logarithms of the gates, i_t = cap tanh(z_i / cap) and
// f_t = logsigmoid(cap tanh(z_f / cap)), meet in a running maximum m_t = max(f_t + m_{t-1}, i_t), m_0 = 0, and
// S_t = exp(f_t + m_{t-1} - m_t) S_{t-1} + exp(i_t - m_t) k_t v_t^T.  The values get one more column, which is 1 for every token:
// that column of S is the memory's normaliser and its read-out the product of normaliser and query.  Lane i of every warp turns
// the raw gates of a group's token i into logarithms when the group is staged; the maxima of a group are a scan over the lanes
// (a token maps m to max(f + m, i), and such maps compose).
#include "common.cuh"
#include <math.h>

#define HG_R 8             // warps of a block, each with a stretch of the d channels
#define HG_MAX_D 512

enum { REC_GATED = 0, REC_KEYED = 1, REC_STEPPED = 2, REC_CAPPED = 3 };

// Where a STEPPED recurrence's operands lie and its numbers per head.  Rows of the float32 input hold the values [H * e] at
// column 0, the keys [groups * d] at off_k, the queries [groups * d] at off_q; z holds the raw step sizes, rows ld_z apart.
struct Stepped {
  const float *z, *dt_bias, *a_log, *skip;
  int ld_z, off_k, off_q, heads_per_group;
};

// What a CAPPED recurrence needs besides the rows [q (H*d) | k (H*d) | v (H*ev) | ...]: raw gates zi, zf [n, H] (rows ld_z apart),
// their biases [H], the cap; m_out [n, H]: the maximum after every token; max_at: where, behind a slot's matrices, the running
// maxima lie ([H, column blocks]: each block of columns keeps its own copy, so none reads what another has moved on).
struct Capped {
  const float *zi, *zf, *bi, *bf;
  float* m_out;
  float cap;
  int ld_z, ev;
  long long max_at;
};

// In place on the rows of qfv: q <- silu(q), f <- lower + (1 - lower) * sigmoid(f + bias); v is left alone.
__global__ void hgrn2_gates_kernel(float* __restrict__ qfv, int ld, const float* __restrict__ f_bias,
                                   const float* __restrict__ lower, int n, int gate_dim) {
  zk_let_next_start();
  zk_wait_prior();
  const size_t total = (size_t)n * gate_dim;
  for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total; idx += (size_t)gridDim.x * blockDim.x) {
    const size_t t = idx / gate_dim;
    const int i = (int)(idx - t * gate_dim);
    float* row = qfv + t * ld;
    const float zq = row[i], zf = row[gate_dim + i] + f_bias[i], lo = lower[i];
    row[i] = zq / (1.0f + expf(-zq));
    row[gate_dim + i] = lo + (1.0f - lo) * (1.0f / (1.0f + expf(-zf)));
  }
}

// What a retention layer does to its projections before the recurrence, in place on the float32 rows [q (H*d) | k (H*d)
// | ...]: the first n_rot entries of every q and k head are rotated by the token's position (entry i pairs with entry
// i + n_rot/2, angle = float(pos) * inv_freq[i]; inv_freq null = no rotation), then k is multiplied by key_scale.
// Block (t, y) takes `slots_per_block` of token t's 2H heads: the cosines and sines of the position are computed once per
// block (with many tokens one block serves all 2H heads; with few, the heads are spread over more blocks).
__global__ void __launch_bounds__(256)
    retention_prepare_kernel(float* __restrict__ qk, int ld, const float* __restrict__ inv_freq, int n_rot, float key_scale,
                             const int* __restrict__ tok_pos, int H, int d, int slots_per_block) {
  __shared__ float cs[HG_MAX_D / 2], sn[HG_MAX_D / 2];
  zk_let_next_start();
  zk_wait_prior();
  const int t = blockIdx.x;
  const int half = inv_freq ? n_rot >> 1 : 0;
  const float pos = (float)tok_pos[t];
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    const float ang = pos * inv_freq[i];
    cs[i] = cosf(ang);
    sn[i] = sinf(ang);
  }
  __syncthreads();
  const int per_head = d - half;                      // work items of a head: its pairs, then its unrotated entries
  float* row = qk + (size_t)t * ld;
  const int s0 = blockIdx.y * slots_per_block, s_here = min(2 * H, s0 + slots_per_block) - s0;
  for (int idx = threadIdx.x; idx < s_here * per_head; idx += blockDim.x) {
    const int s = s0 + idx / per_head, i = idx % per_head;      // head slot: the H query heads, then the H key heads
    float* head = row + (size_t)s * d;
    const float mul = s >= H ? key_scale : 1.0f;
    if (i < half) {
      const float c = cs[i], sv = sn[i];
      const float u = head[i], v = head[i + half];
      head[i] = (u * c - v * sv) * mul;
      head[i + half] = (v * c + u * sv) * mul;
    } else if (s >= H) {
      head[i + half] *= mul;
    }
  }
}

// DPT: channels per warp; TT: tokens staged at once (sixteen, or eight or four where more do not fit shared memory).
// REC_KEYED: the recurrence of a retention layer instead, S_t = decay_h S_{t-1} + k_t v_t^T with one fixed decay per head
// (`decay` [H]); the row's second part then holds the keys k_t in place of the gates.
template <int DPT, int TT, int REC>
__global__ void __launch_bounds__(HG_R * 32)
    hgrn2_scan_kernel(const float* __restrict__ qfv, int ld, float* __restrict__ state, long long state_stride,
                      float* __restrict__ o, const int* __restrict__ cu_q, const int* __restrict__ seq_slot, int H, int d,
                      int e, const float* __restrict__ decay, Stepped sp, Capped cp) {
  constexpr int DM = HG_R * DPT;                                     // channels the block covers, >= d
  constexpr int NL = (TT * DM + HG_R * 32 - 1) / (HG_R * 32);     // q (and f) values a thread fetches per group of tokens
  __shared__ __align__(16) float qs[2][TT][DM];
  __shared__ __align__(16) float fs[2][TT][DM];
  __shared__ float part[TT][HG_R][32];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int b = blockIdx.x, h = blockIdx.y;
  const int c = blockIdx.z * 32 + lane;
  const bool col = c < e;
  const int row0 = warp * DPT;
  // channels beyond d: q = 0 and f = 0 for good, so they add nothing
  if (d < DM) {
    for (int i = tid; i < 2 * TT * DM; i += HG_R * 32) {
      (&qs[0][0][0])[i] = 0.f;
      (&fs[0][0][0])[i] = 0.f;
    }
    __syncthreads();
  }
  zk_wait_prior();   // qfv is the kernel before's result
  const int t0 = cu_q[b], t1 = cu_q[b + 1];
  const float dk = REC == REC_KEYED ? decay[h] : 0.f;
  const float skip = REC == REC_STEPPED ? sp.skip[h] : 0.f, dt_bias = REC == REC_STEPPED ? sp.dt_bias[h] : 0.f;
  const float rate = REC == REC_STEPPED ? -expf(sp.a_log[h]) : 0.f;
  float* st = state + (size_t)seq_slot[b] * state_stride + (size_t)h * d * e;
  float* st_max = REC == REC_CAPPED ? state + (size_t)seq_slot[b] * state_stride + cp.max_at + (size_t)h * gridDim.z + blockIdx.z : nullptr;
  float m_run = REC == REC_CAPPED ? *st_max : 0.f;      // the running maximum before the group that is staged next
  const float bias_i = REC == REC_CAPPED ? cp.bi[h] : 0.f, bias_f = REC == REC_CAPPED ? cp.bf[h] : 0.f;
  float S[DPT];
#pragma unroll
  for (int k = 0; k < DPT; ++k) S[k] = (col && row0 + k < d) ? st[(size_t)(row0 + k) * e + c] : 0.f;

  const int head_q = REC == REC_STEPPED ? sp.off_q + h / sp.heads_per_group * d : h * d;       // columns of this head's q
  const int off_f = REC == REC_STEPPED ? sp.off_k - sp.off_q : H * d, off_v = REC == REC_STEPPED ? 0 : 2 * H * d;
  float rq[NL], rf[NL], v_cur[TT], v_next[TT];
  // REC_STEPPED: the raw step size, decay and dt of token `lane` of a group; REC_CAPPED: its raw gates, what S keeps and what enters
  float rz = 0.f, rz2 = 0.f, lane_decay = 0.f, lane_dt = 0.f;
  // where a thread's n-th value of a group comes from (relative to the group's first row) and goes to
  int src[NL], dst[NL];
#pragma unroll
  for (int n = 0; n < NL; ++n) {
    const int idx = tid + n * HG_R * 32;
    const int tt = idx / d, i = idx - tt * d;
    src[n] = tt < TT ? tt * ld + head_q + i : -1;
    dst[n] = tt * DM + i;
  }
  auto fetch = [&](int tb) {
    const int nt = min(TT, t1 - tb);
    const float* base = qfv + (size_t)tb * ld;
#pragma unroll
    for (int n = 0; n < NL; ++n) {
      const bool ok = src[n] >= 0 && tid + n * HG_R * 32 < nt * d;
      rq[n] = ok ? base[src[n]] : 0.f;
      rf[n] = ok ? base[src[n] + off_f] : 0.f;
    }
#pragma unroll
    for (int tt = 0; tt < TT; ++tt)
      if (REC == REC_CAPPED) v_next[tt] = (col && tt < nt) ? (c < cp.ev ? base[(size_t)tt * ld + off_v + h * cp.ev + c] : 1.0f) : 0.f;
      else v_next[tt] = (col && tt < nt) ? base[(size_t)tt * ld + off_v + h * e + c] : 0.f;
    if (REC == REC_STEPPED && lane < nt) rz = sp.z[(size_t)(tb + lane) * sp.ld_z + h];
    if (REC == REC_CAPPED && lane < nt) {
      rz = cp.zi[(size_t)(tb + lane) * cp.ld_z + h];
      rz2 = cp.zf[(size_t)(tb + lane) * cp.ld_z + h];
    }
  };
  auto stage = [&](int buf, int tb) {
    const int nt = min(TT, t1 - tb);
#pragma unroll
    for (int n = 0; n < NL; ++n) {
      if (src[n] >= 0 && tid + n * HG_R * 32 < nt * d) {
        (&qs[buf][0][0])[dst[n]] = rq[n];
        (&fs[buf][0][0])[dst[n]] = rf[n];
      }
    }
#pragma unroll
    for (int tt = 0; tt < TT; ++tt) v_cur[tt] = v_next[tt];
    if (REC == REC_STEPPED) {
      const float z = rz + dt_bias;
      lane_dt = fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)));      // softplus
      lane_decay = expf(rate * lane_dt);
    }
    if (REC == REC_CAPPED) {
      const float gi = cp.cap * tanhf((rz + bias_i) / cp.cap), zf = cp.cap * tanhf((rz2 + bias_f) / cp.cap);
      const float gf = -(fmaxf(-zf, 0.f) + log1pf(expf(-fabsf(zf))));      // the logarithm of a sigmoid
      float A = gf, B = gi;            // tokens 0 .. lane as one map of m: max(A + m, B)
#pragma unroll
      for (int s = 1; s < TT; s <<= 1) {
        const float pa = __shfl_up_sync(0xffffffffu, A, s), pb = __shfl_up_sync(0xffffffffu, B, s);
        if (lane >= s) {
          B = fmaxf(A + pb, B);
          A += pa;
        }
      }
      const float m = fmaxf(A + m_run, B);
      float before = __shfl_up_sync(0xffffffffu, m, 1);
      if (lane == 0) before = m_run;
      lane_decay = expf(gf - (m - before));      // in this order what m was rounded by is not lost
      lane_dt = expf(gi - m);
      if (warp == 0 && blockIdx.z == 0 && lane < nt) cp.m_out[(size_t)(tb + lane) * H + h] = m;
      m_run = __shfl_sync(0xffffffffu, m, nt - 1);
    }
  };

  if (t0 < t1) {
    fetch(t0);
    stage(0, t0);
  }
  __syncthreads();
  int buf = 0;
  for (int tb = t0; tb < t1; tb += TT, buf ^= 1) {
    const int nt = min(TT, t1 - tb);
    const bool more = tb + TT < t1;
    if (more) fetch(tb + TT);       // under way while this group is worked on
    auto token = [&](int tt) {
      float v = v_cur[tt], keep = dk;
      float acc = 0.f;
      if (REC == REC_STEPPED) {
        if (warp == 0) acc = skip * v;
        keep = __shfl_sync(0xffffffffu, lane_decay, tt);
        v *= __shfl_sync(0xffffffffu, lane_dt, tt);
      }
      if (REC == REC_CAPPED) {
        keep = __shfl_sync(0xffffffffu, lane_decay, tt);
        v *= __shfl_sync(0xffffffffu, lane_dt, tt);
      }
      if constexpr (DPT % 4 == 0) {
#pragma unroll
        for (int k4 = 0; k4 < DPT; k4 += 4) {
          const float4 f4 = *reinterpret_cast<const float4*>(&fs[buf][tt][row0 + k4]);
          const float4 q4 = *reinterpret_cast<const float4*>(&qs[buf][tt][row0 + k4]);
          const float ff[4] = {f4.x, f4.y, f4.z, f4.w}, qq[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            if (REC != REC_GATED) S[k4 + j] = fmaf(keep, S[k4 + j], ff[j] * v);   // decay S + k v
            else S[k4 + j] = fmaf(ff[j], S[k4 + j], fmaf(-ff[j], v, v));        // f S + (1 - f) v
            acc = fmaf(S[k4 + j], qq[j], acc);
          }
        }
      } else {
#pragma unroll
        for (int k = 0; k < DPT; ++k) {
          const float f = fs[buf][tt][row0 + k];
          if (REC != REC_GATED) S[k] = fmaf(keep, S[k], f * v);
          else S[k] = fmaf(f, S[k], fmaf(-f, v, v));
          acc = fmaf(S[k], qs[buf][tt][row0 + k], acc);
        }
      }
      part[tt][warp][lane] = acc;
    };
    if (nt == TT) {          // a whole group: no branch between the tokens, so their loads and sums interleave
#pragma unroll
      for (int tt = 0; tt < TT; ++tt) token(tt);
    } else {
#pragma unroll
      for (int tt = 0; tt < TT; ++tt)
        if (tt < nt) token(tt);
    }
    __syncthreads();
#pragma unroll
    for (int tt = warp; tt < TT; tt += HG_R) {
      if (tt < nt && col) {
        float sum = 0.f;
#pragma unroll
        for (int r = 0; r < HG_R; ++r) sum += part[tt][r][lane];
        o[(size_t)(tb + tt) * H * e + (size_t)h * e + c] = sum;
      }
    }
    if (more) stage(buf ^ 1, tb + TT);
    __syncthreads();
  }
  // The kernel behind this one may start only now: a block that waits for this long kernel to end would hold
  // an SM's issue slots against it (measured: the recurrence ran at half its speed with the release at its top).
  zk_let_next_start();
  if (col) {
#pragma unroll
    for (int k = 0; k < DPT; ++k)
      if (row0 + k < d) st[(size_t)(row0 + k) * e + c] = S[k];
  }
  if (REC == REC_CAPPED && tid == 0) *st_max = m_run;
}

extern "C" {

int zk_hgrn2_max_dim() { return HG_MAX_D; }

// qfv float32 [n, >= 2*H*d + H*e] with rows `ld` floats apart, whose q and f parts are REPLACED by silu(q) and the
// gate; f_bias, lower float32 [H*d]; state float32, a
// slot's [H, d, e] block `state_stride` floats after the one before; o float32 [n, H*e]; cu_q [n_seqs + 1],
// seq_slot [n_seqs].
int zk_hgrn2_scan(float* qfv, int ld, const float* f_bias, const float* lower, float* state, long long state_stride,
                  float* o, const int* cu_q, const int* seq_slot, int n, int n_seqs, int H, int d, int e, cudaStream_t stream) {
  if (n_seqs <= 0 || n <= 0) return 0;
  if (H <= 0 || d <= 0 || e <= 0 || d > HG_MAX_D || ld < 2 * H * d + H * e || !f_bias || !lower) return ZK_EINVAL;
  {
    const size_t total = (size_t)n * H * d;
    const int threads = 256;
    const size_t want = (total + threads - 1) / threads;
    const int blocks = (int)(want < 148 * 16 ? want : 148 * 16);
    const int rc = zk_launch_dependent(hgrn2_gates_kernel, dim3(blocks), dim3(threads), 0, stream, qfv, ld, f_bias, lower, n, H * d);
    if (rc != 0) return rc;
  }
  dim3 grid(n_seqs, H, (e + 31) / 32);
#define ZK_HG(DP)                                                                                                    \
  return zk_launch_dependent(hgrn2_scan_kernel<DP, (DP > 32 ? 4 : (DP > 16 ? 8 : 16)), REC_GATED>, grid, dim3(HG_R * 32), 0, stream, (const float*)qfv, ld, \
                             state, state_stride, o, cu_q, seq_slot, H, d, e, (const float*)nullptr, Stepped{}, Capped{})
  const int dpt = (d + HG_R - 1) / HG_R;
  if (dpt <= 1) ZK_HG(1);
  if (dpt <= 2) ZK_HG(2);
  if (dpt <= 4) ZK_HG(4);
  if (dpt <= 8) ZK_HG(8);
  if (dpt <= 16) ZK_HG(16);
  if (dpt <= 32) ZK_HG(32);
  ZK_HG(64);
#undef ZK_HG
}

// Retention: per head S_t = decay_h S_{t-1} + k_t v_t^T, o_t = S_t^T q_t.  qkv float32 [n, >= 2*H*d + H*e] with rows `ld`
// floats apart, [q | k | v | ...] as the projections gave them; q and k are REPLACED by their rotated forms (k also
// times key_scale).  decay float32 [H]; inv_freq float32 [n_rot / 2] or null; tok_pos [n]; state, o, cu_q, seq_slot as for
// zk_hgrn2_scan.
int zk_retention_scan(float* qkv, int ld, const float* decay, const float* inv_freq, int n_rot, float key_scale,
                      const int* tok_pos, float* state, long long state_stride, float* o, const int* cu_q,
                      const int* seq_slot, int n, int n_seqs, int H, int d, int e, cudaStream_t stream) {
  if (n_seqs <= 0 || n <= 0) return 0;
  if (H <= 0 || d <= 0 || e <= 0 || d > HG_MAX_D || ld < 2 * H * d + H * e || !decay || !tok_pos) return ZK_EINVAL;
  if (inv_freq && (n_rot <= 0 || (n_rot & 1) || n_rot > d)) return ZK_EINVAL;
  if (inv_freq || key_scale != 1.0f) {
    const int per = n >= 256 ? 2 * H : (2 * H + 7) / 8;       // head slots a block takes
    const int rc = zk_launch_dependent(retention_prepare_kernel, dim3(n, (2 * H + per - 1) / per), dim3(256), 0, stream, qkv, ld,
                                       inv_freq, n_rot, key_scale, tok_pos, H, d, per);
    if (rc != 0) return rc;
  }
  dim3 grid(n_seqs, H, (e + 31) / 32);
#define ZK_RT(DP)                                                                                                    \
  return zk_launch_dependent(hgrn2_scan_kernel<DP, (DP > 32 ? 4 : (DP > 16 ? 8 : 16)), REC_KEYED>, grid, dim3(HG_R * 32), 0, stream, (const float*)qkv, ld, \
                             state, state_stride, o, cu_q, seq_slot, H, d, e, decay, Stepped{}, Capped{})
  const int dpt = (d + HG_R - 1) / HG_R;
  if (dpt <= 1) ZK_RT(1);
  if (dpt <= 2) ZK_RT(2);
  if (dpt <= 4) ZK_RT(4);
  if (dpt <= 8) ZK_RT(8);
  if (dpt <= 16) ZK_RT(16);
  if (dpt <= 32) ZK_RT(32);
  ZK_RT(64);
#undef ZK_RT
}

// State-space recurrence (Mamba-2): xbc float32 [n, >= H*e + 2*groups*d] with rows `ld` floats apart, a row [values (H*e) | keys
// (groups*d) | queries (groups*d)]; z float32 [n, >= H] rows ld_z apart (raw step sizes); dt_bias, a_log, skip float32 [H]; state
// (per slot [H, d, e]), o [n, H*e], cu_q, seq_slot as for zk_hgrn2_scan.  d: state channels, e: values per head.
int zk_ssd_scan(const float* xbc, int ld, const float* z, int ld_z, const float* dt_bias, const float* a_log, const float* skip,
                float* state, long long state_stride, float* o, const int* cu_q, const int* seq_slot, int n, int n_seqs, int H,
                int groups, int d, int e, cudaStream_t stream) {
  if (n_seqs <= 0 || n <= 0) return 0;
  if (H <= 0 || groups <= 0 || H % groups || d <= 0 || e <= 0 || d > HG_MAX_D) return ZK_EINVAL;
  if (ld < H * e + 2 * groups * d || ld_z < H || !z || !dt_bias || !a_log || !skip) return ZK_EINVAL;
  const Stepped sp{z, dt_bias, a_log, skip, ld_z, H * e, H * e + groups * d, H / groups};
  dim3 grid(n_seqs, H, (e + 31) / 32);
#define ZK_SS(DP)                                                                                                    \
  return zk_launch_dependent(hgrn2_scan_kernel<DP, (DP > 32 ? 4 : (DP > 16 ? 8 : 16)), REC_STEPPED>, grid, dim3(HG_R * 32), 0, stream, xbc, ld, \
                             state, state_stride, o, cu_q, seq_slot, H, d, e, (const float*)nullptr, sp, Capped{})
  const int dpt = (d + HG_R - 1) / HG_R;
  if (dpt <= 1) ZK_SS(1);
  if (dpt <= 2) ZK_SS(2);
  if (dpt <= 4) ZK_SS(4);
  if (dpt <= 8) ZK_SS(8);
  if (dpt <= 16) ZK_SS(16);
  if (dpt <= 32) ZK_SS(32);
  ZK_SS(64);
#undef ZK_SS
}

// Floats of state a slot of zk_mlstm_scan needs: matrices [H, d, e + 1] and the running maxima.
int zk_mlstm_state_floats(int H, int d, int e) { return H * d * (e + 1) + H * ((e + 1 + 31) / 32); }

// Matrix memory with exponential gates (mLSTM): qkv float32 [n, >= 2*H*d + H*e] with rows `ld` floats apart, [q | k | v | ...] as the
// projections gave them; zi, zf float32 [n, >= H] raw gates, rows ld_z apart, bi, bf [H]; state float32, a slot's
// zk_mlstm_state_floats `state_stride` floats after the one before, zero when a sequence starts; o float32 [n, H * (e + 1)]: per head
// the e sums S_t^T q_t and, last, the product of normaliser and query; m_out [n, H]: the running maximum after every token.
int zk_mlstm_scan(const float* qkv, int ld, const float* zi, const float* zf, int ld_z, const float* bi, const float* bf, float cap,
                  float* state, long long state_stride, float* o, float* m_out, const int* cu_q, const int* seq_slot, int n,
                  int n_seqs, int H, int d, int e, cudaStream_t stream) {
  if (n_seqs <= 0 || n <= 0) return 0;
  if (H <= 0 || d <= 0 || e <= 0 || d > HG_MAX_D || !(cap > 0.f)) return ZK_EINVAL;
  if (ld < 2 * H * d + H * e || ld_z < H || !zi || !zf || !bi || !bf || !m_out) return ZK_EINVAL;
  const Capped cp{zi, zf, bi, bf, m_out, cap, ld_z, e, (long long)H * d * (e + 1)};
  dim3 grid(n_seqs, H, (e + 1 + 31) / 32);
#define ZK_ML(DP)                                                                                                    \
  return zk_launch_dependent(hgrn2_scan_kernel<DP, (DP > 32 ? 4 : (DP > 16 ? 8 : 16)), REC_CAPPED>, grid, dim3(HG_R * 32), 0, stream, qkv, ld, \
                             state, state_stride, o, cu_q, seq_slot, H, d, e + 1, (const float*)nullptr, Stepped{}, cp)
  const int dpt = (d + HG_R - 1) / HG_R;
  if (dpt <= 1) ZK_ML(1);
  if (dpt <= 2) ZK_ML(2);
  if (dpt <= 4) ZK_ML(4);
  if (dpt <= 8) ZK_ML(8);
  if (dpt <= 16) ZK_ML(16);
  if (dpt <= 32) ZK_ML(32);
  ZK_ML(64);
#undef ZK_ML
}

}  // extern "C"
