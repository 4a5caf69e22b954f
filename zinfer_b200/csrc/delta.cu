// Gated delta rule with one decay per head and key channel.  Per head a state S [d, e] that starts at zero:
//
//     S <- diag(g_t) S        u_t = beta_t (v_t - S^T k_t)        S <- S + k_t u_t^T        o_t = S^T q_t
//
// g_t in (0, 1] per head and channel, beta_t in (0, 1) per head; q and k (unit vectors) may be shared by the heads of a group.
// Everything here is float32.
//
// delta_scan_kernel serves prompt steps and single-token steps.  What a token writes depends on what its key reads of the state
// before it, so the tokens are a chain; its length per token is what the kernel's layout is made for.  A column of S (one value
// channel) is owned by L neighbouring lanes, each of which keeps CH of the d key channels in registers; columns never meet.  The
// read S^T k is a sum in registers and log2(L) shuffles, the write needs nothing of another lane, and the read-out S^T q of one
// token overlaps the next token's read.  The decay is folded into the key for the read (sum (g k) S), so the chain is: read, shuffles,
// one multiplication by beta, one fused multiply-add.  A block owns (sequence, head, COLS columns); q, k, g of the next TT tokens reach
// shared memory with cp.async while the current TT are worked on.  State in memory: [H, e, d4], d4 = d rounded up to a multiple of 4,
// channels side by side, so that a column's lanes read whole lines.  The order of every sum is fixed by the layout alone: a
// sequence cut into steps gives the same bits as the whole.
//
// delta_prepare_kernel comes before it in prompt steps: unit vectors and decays, once for all the blocks that read them.  In
// single-token steps (RAW) the scan does both itself on the one token it has.
#include "common.cuh"
#include <math.h>

#define DL_THREADS 128
#define DL_MAX_D 512
#define DL_UNIT_EPS 1e-6f     // inside the root of the unit vectors' length

__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// In place.  Rows of qkv [q (G*d) | k (G*d) | ...]: every q and k head is divided by sqrt(sum of squares + 1e-6), q then multiplied by
// q_scale.  Rows of a [H*d]: a <- exp(-exp(a_log_h) softplus(a + dt_bias)).  One warp per (token, head slot): G queries, G keys, H decays.
__global__ void __launch_bounds__(256)
    delta_prepare_kernel(float* __restrict__ qkv, int ld, float* __restrict__ a, int ld_a, const float* __restrict__ a_log,
                         const float* __restrict__ dt_bias, long long items, int G, int H, int d, float q_scale) {
  zk_let_next_start();
  zk_wait_prior();
  const int lane = threadIdx.x & 31;
  const long long item = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (item >= items) return;
  const int slots = 2 * G + H;
  const long long t = item / slots;
  const int s = (int)(item - t * slots);
  if (s < 2 * G) {
    float* head = qkv + (size_t)t * ld + (size_t)s * d;
    float ss = 0.f;
    if (d <= 128) {             // the head stays in registers between the sum and the scaling
      float v[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        v[j] = lane + 32 * j < d ? head[lane + 32 * j] : 0.f;
        ss = fmaf(v[j], v[j], ss);
      }
      const float mul = (s < G ? q_scale : 1.0f) / sqrtf(warp_sum(ss) + DL_UNIT_EPS);
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (lane + 32 * j < d) head[lane + 32 * j] = v[j] * mul;
      return;
    }
    for (int i = lane; i < d; i += 32) ss = fmaf(head[i], head[i], ss);
    const float mul = (s < G ? q_scale : 1.0f) / sqrtf(warp_sum(ss) + DL_UNIT_EPS);
    for (int i = lane; i < d; i += 32) head[i] *= mul;
    return;
  }
  const int h = s - 2 * G;
  float* row = a + (size_t)t * ld_a + (size_t)h * d;
  const float* b = dt_bias + (size_t)h * d;
  const float rate = -expf(a_log[h]);
  for (int i = lane; i < d; i += 32) row[i] = expf(rate * softplus_f(row[i] + b[i]));
}

struct DeltaArgs {
  const float *qkv, *g, *zb, *a_log, *dt_bias;      // zb: raw beta logits [n, H], rows ld_b apart; a_log, dt_bias: RAW only
  float *state, *o;
  const int *cu_q, *seq_slot;
  long long state_stride;
  int ld, ld_g, ld_b, H, G, d, e, d4, vec;          // vec: heads start on 16-byte boundaries
  float q_scale;
};

__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async4(void* dst, const void* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((unsigned)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

// L lanes per column, CH channels per lane (a multiple of 4, quads l, l + L, ...), TT tokens staged at once.
template <int L, int CH, int TT, bool RAW>
__global__ void __launch_bounds__(DL_THREADS) delta_scan_kernel(const DeltaArgs p) {
  constexpr int DP = L * CH, NQ = CH / 4, COLS = DL_THREADS / L, WCOLS = 32 / L;
  __shared__ __align__(16) float ks[2][TT][DP], qs[2][TT][DP], gs[2][TT][DP];
  __shared__ float vs[2][TT][COLS], os[TT][COLS], zs[2][TT];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int b = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * COLS;
  const int l = lane % L, wc = warp * WCOLS + lane / L;      // this lane's part of its column, the column within the block
  const int c = c0 + wc;
  const bool col = c < p.e;
  const int hk = h / (p.H / p.G);
  if (p.d < DP) {          // channels beyond d are zero for good
    for (int i = tid; i < 2 * TT * DP; i += DL_THREADS) {
      (&ks[0][0][0])[i] = 0.f;
      (&qs[0][0][0])[i] = 0.f;
      (&gs[0][0][0])[i] = 0.f;
    }
    __syncthreads();
  }
  zk_wait_prior();
  const int t0 = p.cu_q[b], t1 = p.cu_q[b + 1];
  float* st = p.state + (size_t)p.seq_slot[b] * p.state_stride + ((size_t)h * p.e + (col ? c : 0)) * p.d4;
  float4 S[NQ];
#pragma unroll
  for (int j = 0; j < NQ; ++j) {
    const int i = 4 * (l + L * j);
    S[j] = col && i < p.d4 ? *reinterpret_cast<const float4*>(st + i) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  const int off_q = hk * p.d, off_k = (p.G + hk) * p.d, off_v = 2 * p.G * p.d + h * p.e + c0;
  const int cols_here = min(COLS, p.e - c0);
  auto fetch = [&](int buf, int tb) {
    const int nt = min(TT, t1 - tb);
    if (p.vec) {
      const int nq = p.d >> 2;
      for (int i = tid; i < nt * nq; i += DL_THREADS) {
        const int tt = i / nq, x = 4 * (i - tt * nq);
        const float* row = p.qkv + (size_t)(tb + tt) * p.ld;
        cp_async16(&ks[buf][tt][x], row + off_k + x);
        cp_async16(&qs[buf][tt][x], row + off_q + x);
        cp_async16(&gs[buf][tt][x], p.g + (size_t)(tb + tt) * p.ld_g + (size_t)h * p.d + x);
      }
    } else {
      for (int i = tid; i < nt * p.d; i += DL_THREADS) {
        const int tt = i / p.d, x = i - tt * p.d;
        const float* row = p.qkv + (size_t)(tb + tt) * p.ld;
        cp_async4(&ks[buf][tt][x], row + off_k + x);
        cp_async4(&qs[buf][tt][x], row + off_q + x);
        cp_async4(&gs[buf][tt][x], p.g + (size_t)(tb + tt) * p.ld_g + (size_t)h * p.d + x);
      }
    }
    for (int i = tid; i < nt * cols_here; i += DL_THREADS) {
      const int tt = i / cols_here, x = i - tt * cols_here;
      cp_async4(&vs[buf][tt][x], p.qkv + (size_t)(tb + tt) * p.ld + off_v + x);
    }
    if (tid < nt) cp_async4(&zs[buf][tid], p.zb + (size_t)(tb + tid) * p.ld_b + h);
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  auto reduce = [&](float v) {
#pragma unroll
    for (int o = L / 2; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
  };

  if (t0 < t1) fetch(0, t0);
  int buf = 0;
  for (int tb = t0; tb < t1; tb += TT, buf ^= 1) {
    const int nt = min(TT, t1 - tb);
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                  // this group has arrived, and everyone is done with the other buffer
    if (tb + TT < t1) fetch(buf ^ 1, tb + TT);
    const float my_beta = lane < nt ? 1.0f / (1.0f + expf(-zs[buf][lane])) : 0.f;
    if constexpr (RAW) {              // one token as the projections and the convolution gave it
      const float rate = -expf(p.a_log[h]);
      for (int i = tid; i < nt * p.d; i += DL_THREADS) {
        const int tt = i / p.d, x = i - tt * p.d;
        gs[buf][tt][x] = expf(rate * softplus_f(gs[buf][tt][x] + p.dt_bias[(size_t)h * p.d + x]));
      }
      __syncthreads();
    }
    auto token = [&](int tt) {
      float4 k[NQ], q[NQ], g[NQ];
#pragma unroll
      for (int j = 0; j < NQ; ++j) {
        k[j] = *reinterpret_cast<const float4*>(&ks[buf][tt][4 * (l + L * j)]);
        q[j] = *reinterpret_cast<const float4*>(&qs[buf][tt][4 * (l + L * j)]);
        g[j] = *reinterpret_cast<const float4*>(&gs[buf][tt][4 * (l + L * j)]);
      }
      if constexpr (RAW) {
        float sk = 0.f, sq = 0.f;
#pragma unroll
        for (int j = 0; j < NQ; ++j) {
          sk = fmaf(k[j].x, k[j].x, fmaf(k[j].y, k[j].y, fmaf(k[j].z, k[j].z, fmaf(k[j].w, k[j].w, sk))));
          sq = fmaf(q[j].x, q[j].x, fmaf(q[j].y, q[j].y, fmaf(q[j].z, q[j].z, fmaf(q[j].w, q[j].w, sq))));
        }
        const float mk = 1.0f / sqrtf(reduce(sk) + DL_UNIT_EPS), mq = p.q_scale / sqrtf(reduce(sq) + DL_UNIT_EPS);
#pragma unroll
        for (int j = 0; j < NQ; ++j) {
          k[j].x *= mk, k[j].y *= mk, k[j].z *= mk, k[j].w *= mk;
          q[j].x *= mq, q[j].y *= mq, q[j].z *= mq, q[j].w *= mq;
        }
      }
      float4 r = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int j = 0; j < NQ; ++j) {
        r.x = fmaf(S[j].x, g[j].x * k[j].x, r.x);
        r.y = fmaf(S[j].y, g[j].y * k[j].y, r.y);
        r.z = fmaf(S[j].z, g[j].z * k[j].z, r.z);
        r.w = fmaf(S[j].w, g[j].w * k[j].w, r.w);
      }
      const float read = reduce((r.x + r.y) + (r.z + r.w));
      const float u = __shfl_sync(0xffffffffu, my_beta, tt) * ((col ? vs[buf][tt][wc] : 0.f) - read);
      float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int j = 0; j < NQ; ++j) {
        S[j].x = fmaf(k[j].x, u, g[j].x * S[j].x);
        S[j].y = fmaf(k[j].y, u, g[j].y * S[j].y);
        S[j].z = fmaf(k[j].z, u, g[j].z * S[j].z);
        S[j].w = fmaf(k[j].w, u, g[j].w * S[j].w);
        y.x = fmaf(S[j].x, q[j].x, y.x);
        y.y = fmaf(S[j].y, q[j].y, y.y);
        y.z = fmaf(S[j].z, q[j].z, y.z);
        y.w = fmaf(S[j].w, q[j].w, y.w);
      }
      const float out = reduce((y.x + y.y) + (y.z + y.w));
      if (l == 0) os[tt][wc] = out;
    };
    if (nt == TT) {
#pragma unroll
      for (int tt = 0; tt < TT; ++tt) token(tt);
    } else {
      for (int tt = 0; tt < nt; ++tt) token(tt);
    }
    __syncthreads();
    for (int i = tid; i < nt * cols_here; i += DL_THREADS) {
      const int tt = i / cols_here, x = i - tt * cols_here;
      p.o[(size_t)(tb + tt) * p.H * p.e + (size_t)h * p.e + c0 + x] = os[tt][x];
    }
  }
  zk_let_next_start();      // only now: a block that waits for this long kernel would hold an SM's issue slots against it
  if (col) {
#pragma unroll
    for (int j = 0; j < NQ; ++j) {
      const int i = 4 * (l + L * j);
      if (i < p.d4) *reinterpret_cast<float4*>(st + i) = S[j];
    }
  }
}

namespace {

template <int L, int CH, int TT>
int launch_scan(const DeltaArgs& p, int n_seqs, int raw, cudaStream_t stream) {
  constexpr int COLS = DL_THREADS / L;
  const dim3 grid(n_seqs, p.H, (p.e + COLS - 1) / COLS);
  if (raw) return zk_launch_dependent(delta_scan_kernel<L, CH, 1, true>, grid, dim3(DL_THREADS), 0, stream, p);
  return zk_launch_dependent(delta_scan_kernel<L, CH, TT, false>, grid, dim3(DL_THREADS), 0, stream, p);
}

}  // namespace

extern "C" {

int zk_delta_max_dim() { return DL_MAX_D; }

// Floats of state a slot needs: [H, e, d rounded up to a multiple of 4].
int zk_delta_state_floats(int H, int d, int e) { return H * e * ((d + 3) / 4 * 4); }

// qkv float32 [n, >= 2*G*d + H*e], rows `ld` apart, [q | k | v | ...] behind their convolutions; a float32 [n, >= H*d], rows ld_a
// apart: the raw decays; zb float32 [n, >= H], rows ld_b apart: beta's logits; a_log [H], dt_bias [H*d].  state: 16-byte aligned slots
// of zk_delta_state_floats, `state_stride` floats apart (a multiple of 4).  o float32 [n, H*e].  single != 0: every sequence has one
// token, and qkv and a are left as they are; otherwise q, k and a are REPLACED by unit vectors and decays first.
int zk_delta_scan(float* qkv, int ld, float* a, int ld_a, const float* zb, int ld_b, const float* a_log, const float* dt_bias,
                  float* state, long long state_stride, float* o, const int* cu_q, const int* seq_slot, int n, int n_seqs, int H,
                  int G, int d, int e, float q_scale, int single, cudaStream_t stream) {
  if (n_seqs <= 0 || n <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || d <= 0 || e <= 0 || d > DL_MAX_D) return ZK_EINVAL;
  if (ld < 2 * G * d + H * e || ld_a < H * d || ld_b < H || !a_log || !dt_bias || !zb) return ZK_EINVAL;
  if (state_stride % 4 || (uintptr_t)state % 16 || (single && n != n_seqs)) return ZK_EINVAL;
  if (!single) {
    const long long items = (long long)n * (2 * G + H);
    const int rc = zk_launch_dependent(delta_prepare_kernel, dim3((unsigned)((items + 7) / 8)), dim3(256), 0, stream, qkv, ld, a, ld_a,
                                       a_log, dt_bias, items, G, H, d, q_scale);
    if (rc != 0) return rc;
  }
  DeltaArgs p{};
  p.qkv = qkv; p.g = a; p.zb = zb; p.a_log = a_log; p.dt_bias = dt_bias;
  p.state = state; p.o = o; p.cu_q = cu_q; p.seq_slot = seq_slot; p.state_stride = state_stride;
  p.ld = ld; p.ld_g = ld_a; p.ld_b = ld_b; p.H = H; p.G = G; p.d = d; p.e = e; p.d4 = (d + 3) / 4 * 4;
  p.vec = d % 4 == 0 && ld % 4 == 0 && ld_a % 4 == 0 && ((uintptr_t)qkv | (uintptr_t)a) % 16 == 0;
  p.q_scale = q_scale;
  if (d <= 32) return launch_scan<8, 4, 8>(p, n_seqs, single, stream);
  if (d <= 64) return launch_scan<8, 8, 8>(p, n_seqs, single, stream);
  if (d <= 128) return launch_scan<8, 16, 8>(p, n_seqs, single, stream);
  if (d <= 256) return launch_scan<16, 16, 4>(p, n_seqs, single, stream);
  return launch_scan<32, 16, 2>(p, n_seqs, single, stream);
}

}  // extern "C"
