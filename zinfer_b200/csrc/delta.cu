// Gated delta rule with one decay per head and key channel.  Per head a state S [d, e] that starts at zero:
//
//     S <- diag(g_t) S        u_t = beta_t (v_t - S^T k_t)        S <- S + k_t u_t^T        o_t = S^T q_t
//
// g_t in (0, 1] per head and channel, beta_t in (0, 1) per head; q and k (unit vectors) may be shared by the heads of a group.
// Everything here is float32.  State in memory: [H, e, d4], d4 = d rounded up to a multiple of 4, channels side by side.
//
// What a token writes depends on what its key reads of the state before it, so the tokens are a chain.  Prompt steps walk it four
// tokens (a chunk, counted from the sequence's first token of the step) at a time.  With S0 the state before a chunk, c_i the product
// of the decays of its tokens 0..i and p_ij that of tokens j+1..i (per channel):
//
//     read of token i        S^T k_i = S0^T (c_i k_i) + sum_{j<i} A_ij u_j        A_ij = sum_channels k_i p_ij k_j
//     output of token i      o_i = S0^T (c_i q_i) + sum_{j<=i} B_ij u_j           B_ij = sum_channels q_i p_ij k_j
//     state after the chunk  c_3 S0 + sum_j (p_3j k_j) u_j^T
//
// so the four reads and the four outputs of a chunk are sums over S0 that do not wait for one another, and only the four u, a
// small triangular system per column, are a chain.  Products of decays are never divided by, so nothing overflows.
// delta_chunk_prepare_kernel makes the vectors and the numbers A, B once per (chunk, head), with unit vectors, decays and beta on
// the way, as one contiguous record.  delta_chunk_kernel owns (sequence, head, some columns of S) per block and walks the chunks: a
// column lies in L neighbouring lanes, CH channels each, in registers; the records of the next chunks arrive in a ring in shared
// memory, one bulk copy each, counted on an mbarrier.
//
// delta_single_kernel is the single-token step: the recurrence as it stands, unit vectors and decays made on the spot.
#include "tcgen05.cuh"
#include <math.h>

#define DL_THREADS 128
#define DL_MAX_D 512
#define DL_CHUNK 4
#define DL_UNIT_EPS 1e-6f     // inside the root of the unit vectors' length

__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

struct DeltaArgs {
  const float *qkv, *a, *zb, *a_log, *dt_bias;      // as zk_delta_scan takes them
  float* rec;                                       // prompt steps: the records of all chunks, [chunks, H, record_floats(DP, e)]
  float *state, *o;
  int* status;
  const int *cu_q, *seq_slot, *tok_seq;
  long long state_stride;
  int ld, ld_a, ld_b, H, G, d, e, d4;
  float q_scale;
};

// Chunks of all sequences have distinct numbers below n / 4 + n_seqs: that of the chunk of sequence b that starts at row t.
__device__ __forceinline__ int chunk_number(int t0, int t, int b) { return t0 / DL_CHUNK + (t - t0) / DL_CHUNK + b; }

// A record: for each of the four tokens the vectors c_i k_i, c_i q_i, p_3i k_i; then c_3; then, for each token,
// A_i0 A_i1 A_i2 beta_i B_i0 B_i1 B_i2 B_i3 (zeros where j is too large).  Vectors are padded with zeros to DP channels; a token
// that the chunk has not (its sequence ends) is all zeros: it writes nothing.  Behind that lie the chunk's values, column by column:
// [e up to a multiple of 16][4 tokens], of which a block of the chunk kernel takes its own columns.
__host__ __device__ constexpr int vector_floats(int DP) { return 13 * DP + 8 * DL_CHUNK; }
__host__ __device__ __forceinline__ int record_floats(int DP, int e) { return vector_floats(DP) + (e + 15) / 16 * 16 * DL_CHUNK; }

// One warp per (token that starts a chunk, head); the warps of other tokens end at once.  NJ: channels per lane, DP = 32 NJ.
template <int NJ>
__global__ void __launch_bounds__(128) delta_chunk_prepare_kernel(const DeltaArgs p) {
  zk_wait_prior();      // and no early start of the kernel behind: its few long blocks would crowd onto the SMs that have room first
  const int t = blockIdx.x, lane = threadIdx.x & 31, h = blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int b = p.tok_seq[t], t0 = p.cu_q[b];
  if (((t - t0) & (DL_CHUNK - 1)) != 0 || h >= p.H) return;
  const int nt = min(DL_CHUNK, p.cu_q[b + 1] - t);
  const int hk = h / (p.H / p.G);
  const float rate = -expf(p.a_log[h]);
  float q[DL_CHUNK][NJ], k[DL_CHUNK][NJ], g[DL_CHUNK][NJ];
#pragma unroll
  for (int i = 0; i < DL_CHUNK; ++i) {
    const float* row = p.qkv + (size_t)(t + (i < nt ? i : 0)) * p.ld;
    const float* ar = p.a + (size_t)(t + (i < nt ? i : 0)) * p.ld_a + (size_t)h * p.d;
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      const int c = lane + 32 * j;
      const bool ok = i < nt && c < p.d;
      q[i][j] = ok ? row[hk * p.d + c] : 0.f;
      k[i][j] = ok ? row[(p.G + hk) * p.d + c] : 0.f;
      g[i][j] = ok ? expf(rate * softplus_f(ar[c] + p.dt_bias[(size_t)h * p.d + c])) : 1.f;
    }
  }
#pragma unroll
  for (int i = 0; i < DL_CHUNK; ++i) {
    float sq = 0.f, sk = 0.f;
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      sq = fmaf(q[i][j], q[i][j], sq);
      sk = fmaf(k[i][j], k[i][j], sk);
    }
    const float mq = p.q_scale / sqrtf(warp_sum(sq) + DL_UNIT_EPS), mk = 1.0f / sqrtf(warp_sum(sk) + DL_UNIT_EPS);
#pragma unroll
    for (int j = 0; j < NJ; ++j) {
      q[i][j] *= mq;
      k[i][j] *= mk;
    }
  }
  // the sixteen numbers: A_ij at i*i + j, B_ij at i*i + i + j
  float v[16];
#pragma unroll
  for (int x = 0; x < 16; ++x) v[x] = 0.f;
  constexpr int DP = 32 * NJ;
  float* rec = p.rec + ((size_t)chunk_number(t0, t, b) * p.H + h) * record_floats(DP, p.e);
#pragma unroll
  for (int j = 0; j < NJ; ++j) {
    const int c = lane + 32 * j;
    float cum = 1.f;
#pragma unroll
    for (int i = 0; i < DL_CHUNK; ++i) {
      cum *= g[i][j];
      float w = k[i][j];                       // p_li k_i for growing l
      v[i * i + i + i] = fmaf(q[i][j], w, v[i * i + i + i]);
#pragma unroll
      for (int l = i + 1; l < DL_CHUNK; ++l) {
        w *= g[l][j];
        v[l * l + i] = fmaf(k[l][j], w, v[l * l + i]);
        v[l * l + l + i] = fmaf(q[l][j], w, v[l * l + l + i]);
      }
      rec[(3 * i) * DP + c] = cum * k[i][j];
      rec[(3 * i + 1) * DP + c] = cum * q[i][j];
      rec[(3 * i + 2) * DP + c] = w;
    }
    rec[12 * DP + c] = cum;
  }
  // sum all sixteen over the lanes: each exchange halves what a lane holds; lanes 2x and 2x + 1 end with number x
#pragma unroll
  for (int off = 16, n = 8; n >= 1; off >>= 1, n >>= 1) {
    const bool up = lane & off;
#pragma unroll
    for (int x = 0; x < n; ++x) {
      const float send = up ? v[x] : v[x + n], keep = up ? v[x + n] : v[x];
      v[x] = keep + __shfl_xor_sync(0xffffffffu, send, off);
    }
  }
  v[0] += __shfl_xor_sync(0xffffffffu, v[0], 1);
  const int i = lane >> 3, s = lane & 7, j = s < 4 ? s : s - 4;
  const bool is_a = s < 3 && j < i, is_b = s >= 4 && j <= i;
  const float got = __shfl_sync(0xffffffffu, v[0], 2 * (is_a ? i * i + j : (is_b ? i * i + i + j : 0)));
  float out = is_a || is_b ? got : 0.f;
  if (s == 3 && i < nt) out = 1.0f / (1.0f + expf(-p.zb[(size_t)(t + i) * p.ld_b + h]));
  rec[13 * DP + lane] = out;
  const float* values = p.qkv + (size_t)t * p.ld + 2 * p.G * p.d + h * p.e;
  for (int c = lane; c < (p.e + 15) / 16 * 16; c += 32) {
    float x[DL_CHUNK];
#pragma unroll
    for (int i = 0; i < DL_CHUNK; ++i) x[i] = i < nt && c < p.e ? values[(size_t)i * p.ld + c] : 0.f;
    *reinterpret_cast<float4*>(rec + vector_floats(DP) + 4 * c) = make_float4(x[0], x[1], x[2], x[3]);
  }
}

// `bytes` (a multiple of 16, both addresses 16-byte aligned) from global to this block's shared memory, counted on `bar`.
__device__ __forceinline__ void bulk_load(void* dst, const void* src, unsigned bytes, unsigned long long* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(tc5::smem_u32(dst)),
               "l"(src), "r"(bytes), "r"(tc5::smem_u32(bar))
               : "memory");
}
__device__ __forceinline__ float dot4(const float4& a, const float4& b, float acc) {
  return fmaf(a.x, b.x, fmaf(a.y, b.y, fmaf(a.z, b.z, fmaf(a.w, b.w, acc))));
}

// L lanes per column, CH channels per lane (a multiple of 4, quads l, l + L, ...), X neighbouring columns per lane, a ring of ST records.
template <int L, int CH, int X, int ST>
__global__ void __launch_bounds__(DL_THREADS, 1) delta_chunk_kernel(const DeltaArgs p) {
  constexpr int DP = L * CH, NQ = CH / 4, COLS = DL_THREADS / L * X;
  constexpr int VEC = vector_floats(DP), REC = VEC + COLS * DL_CHUNK;      // what a block takes of a record
  extern __shared__ __align__(128) float sm[];       // [ST][REC]
  __shared__ __align__(8) unsigned long long full[ST];
  const int tid = threadIdx.x, l = tid % L, grp = tid / L;
  const int b = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * COLS + grp * X;      // this lane's first column
  if (tid == 0) {
    for (int s = 0; s < ST; ++s) tc5::mbar_init(&full[s], 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
  }
  __syncthreads();
  zk_wait_prior();
  const int t0 = p.cu_q[b], t1 = p.cu_q[b + 1];
  const int n_chunks = (t1 - t0 + DL_CHUNK - 1) / DL_CHUNK;
  const int rec_floats = record_floats(DP, p.e);
  const float* records = p.rec + ((size_t)chunk_number(t0, t0, b) * p.H + h) * rec_floats;      // chunk ch: ch * H records further on
  const size_t rec_step = (size_t)p.H * rec_floats;
  const int col0 = blockIdx.z * COLS;
  const unsigned val_bytes = 4u * DL_CHUNK * min(COLS, (p.e + 15) / 16 * 16 - col0);
  auto fetch = [&](int ch) {
    unsigned long long* bar = &full[ch % ST];
    tc5::mbar_expect_tx(bar, VEC * 4 + val_bytes);
    bulk_load(sm + (size_t)(ch % ST) * REC, records + ch * rec_step, VEC * 4, bar);
    bulk_load(sm + (size_t)(ch % ST) * REC + VEC, records + ch * rec_step + VEC + col0 * DL_CHUNK, val_bytes, bar);
  };
  if (tid == 0)
    for (int ch = 0; ch < ST && ch < n_chunks; ++ch) fetch(ch);
  float* st = p.state + (size_t)p.seq_slot[b] * p.state_stride + (size_t)h * p.e * p.d4;
  float4 S[X][NQ];
#pragma unroll
  for (int x = 0; x < X; ++x) {
#pragma unroll
    for (int j = 0; j < NQ; ++j) {
      const int i = 4 * (l + L * j);
      S[x][j] = c0 + x < p.e && i < p.d4 ? *reinterpret_cast<const float4*>(st + (size_t)(c0 + x) * p.d4 + i) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  }
  float* out = p.o + (size_t)t0 * p.H * p.e + (size_t)h * p.e + c0;
  const int mine = l / (L / 4);                      // the token of a chunk whose outputs this lane ends with
  int ch = 0;
  bool lost = false;
  for (; ch < n_chunks; ++ch) {
    const float* s = sm + (size_t)(ch % ST) * REC;
    const bool here = tc5::mbar_wait(&full[ch % ST], (ch / ST) & 1);
    {
      const float* at = s + 4 * l;                   // this lane's first quad of the chunk's vectors; the next lies 4 * L further on
      const float* num = s + 13 * DP;
      auto load = [&](float4 (&kk)[DL_CHUNK], float4 (&qq)[DL_CHUNK], int j) {
#pragma unroll
        for (int i = 0; i < DL_CHUNK; ++i) {
          kk[i] = *reinterpret_cast<const float4*>(at + (3 * i) * DP + 4 * L * j);
          qq[i] = *reinterpret_cast<const float4*>(at + (3 * i + 1) * DP + 4 * L * j);
        }
      };
      auto load_write = [&](float4 (&kk)[DL_CHUNK], float4& T, int j) {
#pragma unroll
        for (int i = 0; i < DL_CHUNK; ++i) kk[i] = *reinterpret_cast<const float4*>(at + (3 * i + 2) * DP + 4 * L * j);
        T = *reinterpret_cast<const float4*>(at + 12 * DP + 4 * L * j);
      };
      // reads and outputs over S0: the next quad's vectors are under way while one quad is worked on, eight sums at a time
      float4 kk[2][DL_CHUNK], qq[2][DL_CHUNK], T[2];
      float r[X][DL_CHUNK], y[X][DL_CHUNK];
      float4 w[X];                                   // the four tokens' values of each column
      load(kk[0], qq[0], 0);
      float4 A[DL_CHUNK];                            // A_i0 A_i1 A_i2 beta_i
#pragma unroll
      for (int i = 0; i < DL_CHUNK; ++i) {
        A[i] = *reinterpret_cast<const float4*>(num + 8 * i);
#pragma unroll
        for (int x = 0; x < X; ++x) r[x][i] = y[x][i] = 0.f;
      }
#pragma unroll
      for (int x = 0; x < X; ++x) w[x] = *reinterpret_cast<const float4*>(s + VEC + 4 * (grp * X + x));
#pragma unroll
      for (int j = 0; j < NQ; ++j) {
        if (j + 1 < NQ) load(kk[(j + 1) & 1], qq[(j + 1) & 1], j + 1);
#pragma unroll
        for (int x = 0; x < X; ++x)
#pragma unroll
          for (int i = 0; i < DL_CHUNK; ++i) {
            r[x][i] = dot4(S[x][j], kk[j & 1][i], r[x][i]);
            y[x][i] = dot4(S[x][j], qq[j & 1][i], y[x][i]);
          }
      }
      load_write(kk[0], T[0], 0);                    // for the state's update, under way during the exchanges
#pragma unroll
      for (int o = L / 2; o > 0; o >>= 1)
#pragma unroll
        for (int x = 0; x < X; ++x)
#pragma unroll
          for (int i = 0; i < DL_CHUNK; ++i) r[x][i] += __shfl_xor_sync(0xffffffffu, r[x][i], o);
      // the outputs: the four sums of a column need not end in every lane, so two exchanges leave a lane one token's
      float a[X];
#pragma unroll
      for (int x = 0; x < X; ++x) {
        const bool hi = l & (L / 2), lo = l & (L / 4);
        const float a0 = (hi ? y[x][2] : y[x][0]) + __shfl_xor_sync(0xffffffffu, hi ? y[x][0] : y[x][2], L / 2);
        const float a1 = (hi ? y[x][3] : y[x][1]) + __shfl_xor_sync(0xffffffffu, hi ? y[x][1] : y[x][3], L / 2);
        a[x] = (lo ? a1 : a0) + __shfl_xor_sync(0xffffffffu, lo ? a0 : a1, L / 4);
#pragma unroll
        for (int o = L / 8; o > 0; o >>= 1) a[x] += __shfl_xor_sync(0xffffffffu, a[x], o);
      }
      float u[X][DL_CHUNK];
#pragma unroll
      for (int i = 0; i < DL_CHUNK; ++i)
#pragma unroll
        for (int x = 0; x < X; ++x) {
          float z = (i == 0 ? w[x].x : (i == 1 ? w[x].y : (i == 2 ? w[x].z : w[x].w))) - r[x][i];
          if (i > 0) z = fmaf(-A[i].x, u[x][0], z);
          if (i > 1) z = fmaf(-A[i].y, u[x][1], z);
          if (i > 2) z = fmaf(-A[i].z, u[x][2], z);
          u[x][i] = A[i].w * z;
        }
#pragma unroll
      for (int j = 0; j < NQ; ++j) {
        if (j + 1 < NQ) load_write(kk[(j + 1) & 1], T[(j + 1) & 1], j + 1);
        const float4 t4 = T[j & 1];
#pragma unroll
        for (int x = 0; x < X; ++x) S[x][j].x *= t4.x, S[x][j].y *= t4.y, S[x][j].z *= t4.z, S[x][j].w *= t4.w;
#pragma unroll
        for (int i = 0; i < DL_CHUNK; ++i)
#pragma unroll
          for (int x = 0; x < X; ++x) {
            S[x][j].x = fmaf(kk[j & 1][i].x, u[x][i], S[x][j].x);
            S[x][j].y = fmaf(kk[j & 1][i].y, u[x][i], S[x][j].y);
            S[x][j].z = fmaf(kk[j & 1][i].z, u[x][i], S[x][j].z);
            S[x][j].w = fmaf(kk[j & 1][i].w, u[x][i], S[x][j].w);
          }
      }
      const float4 B = *reinterpret_cast<const float4*>(num + 8 * mine + 4);
      const int t = ch * DL_CHUNK + mine;
#pragma unroll
      for (int x = 0; x < X; ++x) {
        a[x] = fmaf(B.x, u[x][0], fmaf(B.y, u[x][1], fmaf(B.z, u[x][2], fmaf(B.w, u[x][3], a[x]))));
        if (l % (L / 4) == 0 && t < t1 - t0 && c0 + x < p.e) out[(size_t)t * p.H * p.e + x] = a[x];
      }
    }
    if (__syncthreads_or(!here)) {                   // everyone is done with this record, or one never came
      lost = true;
      break;
    }
    if (tid == 0 && ch + ST < n_chunks) fetch(ch + ST);
  }
  zk_let_next_start();      // only now: a block that waits for this long kernel would hold an SM's issue slots against it
  if (lost) {
    if (tid == 0) {
      atomicExch(p.status, 19);
      for (int k = ch + 1; k < n_chunks && k < ch + ST; ++k) tc5::mbar_wait(&full[k % ST], (k / ST) & 1);      // the copies under way
    }
    return;
  }
#pragma unroll
  for (int x = 0; x < X; ++x) {
#pragma unroll
    for (int j = 0; j < NQ; ++j) {
      const int i = 4 * (l + L * j);
      if (c0 + x < p.e && i < p.d4) *reinterpret_cast<float4*>(st + (size_t)(c0 + x) * p.d4 + i) = S[x][j];
    }
  }
}

// One token per sequence: row b is sequence b's.  Block (sequence, head, columns); its threads make the decays once, every column's
// lanes read them, and the raw q and k, from shared memory.
template <int L, int CH>
__global__ void __launch_bounds__(DL_THREADS) delta_single_kernel(const DeltaArgs p) {
  constexpr int DP = L * CH, NQ = CH / 4, COLS = DL_THREADS / L;
  __shared__ __align__(16) float ks[DP], qs[DP], gs[DP];
  const int tid = threadIdx.x, l = tid % L, c = blockIdx.z * COLS + tid / L;
  const int b = blockIdx.x, h = blockIdx.y, hk = h / (p.H / p.G);
  const bool col = c < p.e;
  zk_let_next_start();
  zk_wait_prior();
  float* st = p.state + (size_t)p.seq_slot[b] * p.state_stride + ((size_t)h * p.e + (col ? c : 0)) * p.d4;
  float4 S[NQ];
#pragma unroll
  for (int j = 0; j < NQ; ++j) {
    const int i = 4 * (l + L * j);
    S[j] = col && i < p.d4 ? *reinterpret_cast<const float4*>(st + i) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  const float* row = p.qkv + (size_t)b * p.ld;
  const float v = col ? row[2 * p.G * p.d + h * p.e + c] : 0.f;
  const float beta = 1.0f / (1.0f + expf(-p.zb[(size_t)b * p.ld_b + h]));
  const float rate = -expf(p.a_log[h]);
  for (int i = tid; i < DP; i += DL_THREADS) {
    const bool ok = i < p.d;
    qs[i] = ok ? row[hk * p.d + i] : 0.f;
    ks[i] = ok ? row[(p.G + hk) * p.d + i] : 0.f;
    gs[i] = ok ? expf(rate * softplus_f(p.a[(size_t)b * p.ld_a + (size_t)h * p.d + i] + p.dt_bias[(size_t)h * p.d + i])) : 0.f;
  }
  __syncthreads();
  auto reduce = [&](float x) {
#pragma unroll
    for (int o = L / 2; o > 0; o >>= 1) x += __shfl_xor_sync(0xffffffffu, x, o);
    return x;
  };
  float sk = 0.f, sq = 0.f, r = 0.f;
#pragma unroll
  for (int j = 0; j < NQ; ++j) {
    const float4 k = *reinterpret_cast<const float4*>(ks + 4 * (l + L * j)), q = *reinterpret_cast<const float4*>(qs + 4 * (l + L * j));
    const float4 g = *reinterpret_cast<const float4*>(gs + 4 * (l + L * j));
    sk = dot4(k, k, sk);
    sq = dot4(q, q, sq);
    S[j].x *= g.x, S[j].y *= g.y, S[j].z *= g.z, S[j].w *= g.w;
    r = dot4(S[j], k, r);
  }
  const float mk = 1.0f / sqrtf(reduce(sk) + DL_UNIT_EPS), mq = p.q_scale / sqrtf(reduce(sq) + DL_UNIT_EPS);
  const float uk = beta * (v - mk * reduce(r)) * mk;      // times the raw key
  float y = 0.f;
#pragma unroll
  for (int j = 0; j < NQ; ++j) {
    const float4 k = *reinterpret_cast<const float4*>(ks + 4 * (l + L * j)), q = *reinterpret_cast<const float4*>(qs + 4 * (l + L * j));
    S[j].x = fmaf(k.x, uk, S[j].x);
    S[j].y = fmaf(k.y, uk, S[j].y);
    S[j].z = fmaf(k.z, uk, S[j].z);
    S[j].w = fmaf(k.w, uk, S[j].w);
    y = dot4(S[j], q, y);
    const int i = 4 * (l + L * j);
    if (col && i < p.d4) *reinterpret_cast<float4*>(st + i) = S[j];
  }
  y = mq * reduce(y);
  if (col && l == 0) p.o[(size_t)b * p.H * p.e + (size_t)h * p.e + c] = y;
}

namespace {

template <int L, int CH, int X, int ST>
int launch_chunks(const DeltaArgs& p, int n_seqs, cudaStream_t stream) {
  auto kern = delta_chunk_kernel<L, CH, X, ST>;
  constexpr int COLS = DL_THREADS / L * X;
  constexpr size_t smem = sizeof(float) * ST * (vector_floats(L * CH) + COLS * DL_CHUNK);
  if (smem > 40 * 1024) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  return zk_launch_dependent(kern, dim3(n_seqs, p.H, (p.e + COLS - 1) / COLS), dim3(DL_THREADS), smem, stream, p);
}

int padded_channels(int d) { return d <= 32 ? 32 : (d <= 64 ? 64 : (d <= 128 ? 128 : (d <= 256 ? 256 : 512))); }

template <int L, int CH>
int launch_single(const DeltaArgs& p, int n_seqs, cudaStream_t stream) {
  constexpr int COLS = DL_THREADS / L;
  return zk_launch_dependent(delta_single_kernel<L, CH>, dim3(n_seqs, p.H, (p.e + COLS - 1) / COLS), dim3(DL_THREADS), 0, stream, p);
}

int forced_layout = 0;      // lanes per column of the chunk kernel at d of 65..128 (8 or 16); 0 = the library chooses

}  // namespace

extern "C" {

int zk_delta_max_dim() { return DL_MAX_D; }

// Floats of state a slot needs: [H, e, d rounded up to a multiple of 4].
int zk_delta_state_floats(int H, int d, int e) { return H * e * ((d + 3) / 4 * 4); }

// Floats of scratch a prompt step of n tokens and n_seqs sequences needs.
long long zk_delta_scratch_floats(int n, int n_seqs, int H, int d, int e) {
  return (long long)(n / DL_CHUNK + n_seqs) * H * record_floats(padded_channels(d), e);
}

// For measurements: lanes per column (8 or 16) of prompt steps with 65..128 key channels; 0 gives the choice back.
int zk_delta_force_lanes(int lanes) {
  if (lanes != 0 && lanes != 8 && lanes != 16) return ZK_EINVAL;
  forced_layout = lanes;
  return 0;
}

// qkv float32 [n, >= 2*G*d + H*e], rows `ld` apart, [q | k | v | ...] behind their convolutions; a float32 [n, >= H*d], rows ld_a
// apart: the raw decays; zb float32 [n, >= H], rows ld_b apart: beta's logits; a_log [H], dt_bias [H*d].  state: 16-byte aligned slots
// of zk_delta_state_floats, `state_stride` floats apart (a multiple of 4).  o float32 [n, H*e].  scratch: 16-byte aligned, of
// zk_delta_scratch_floats, or null: then every sequence has one token (n = n_seqs, row b sequence b's).
int zk_delta_scan(const float* qkv, int ld, const float* a, int ld_a, const float* zb, int ld_b, const float* a_log,
                  const float* dt_bias, float* state, long long state_stride, float* o, const int* cu_q, const int* seq_slot,
                  const int* tok_seq, int n, int n_seqs, int H, int G, int d, int e, float q_scale, float* scratch,
                  int* status, cudaStream_t stream) {
  if (n_seqs <= 0 || n <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || d <= 0 || e <= 0 || d > DL_MAX_D) return ZK_EINVAL;
  if (ld < 2 * G * d + H * e || ld_a < H * d || ld_b < H || !a_log || !dt_bias || !zb || !status) return ZK_EINVAL;
  if (state_stride % 4 || (uintptr_t)state % 16 || (uintptr_t)scratch % 16 || (!scratch && n != n_seqs)) return ZK_EINVAL;
  DeltaArgs p{};
  p.qkv = qkv; p.a = a; p.zb = zb; p.a_log = a_log; p.dt_bias = dt_bias;
  p.state = state; p.o = o; p.cu_q = cu_q; p.seq_slot = seq_slot; p.tok_seq = tok_seq; p.state_stride = state_stride;
  p.ld = ld; p.ld_a = ld_a; p.ld_b = ld_b; p.H = H; p.G = G; p.d = d; p.e = e; p.d4 = (d + 3) / 4 * 4;
  p.q_scale = q_scale; p.status = status;
  if (!scratch) {
    if (d <= 32) return launch_single<8, 4>(p, n_seqs, stream);
    if (d <= 64) return launch_single<8, 8>(p, n_seqs, stream);
    if (d <= 128) return launch_single<8, 16>(p, n_seqs, stream);
    if (d <= 256) return launch_single<16, 16>(p, n_seqs, stream);
    return launch_single<32, 16>(p, n_seqs, stream);
  }
  p.rec = scratch;
  const dim3 grid(n, (H + 3) / 4), block(128);
  int rc;
  if (d <= 32) rc = zk_launch_dependent(delta_chunk_prepare_kernel<1>, grid, block, 0, stream, p);
  else if (d <= 64) rc = zk_launch_dependent(delta_chunk_prepare_kernel<2>, grid, block, 0, stream, p);
  else if (d <= 128) rc = zk_launch_dependent(delta_chunk_prepare_kernel<4>, grid, block, 0, stream, p);
  else if (d <= 256) rc = zk_launch_dependent(delta_chunk_prepare_kernel<8>, grid, block, 0, stream, p);
  else rc = zk_launch_dependent(delta_chunk_prepare_kernel<16>, grid, block, 0, stream, p);
  if (rc != 0) return rc;
  if (d <= 32) return launch_chunks<8, 4, 1, 8>(p, n_seqs, stream);
  if (d <= 64) return launch_chunks<16, 4, 2, 8>(p, n_seqs, stream);
  if (d <= 128) return forced_layout == 8 ? launch_chunks<8, 16, 1, 6>(p, n_seqs, stream) : launch_chunks<16, 8, 2, 6>(p, n_seqs, stream);
  if (d <= 256) return launch_chunks<16, 16, 2, 4>(p, n_seqs, stream);
  return launch_chunks<32, 16, 2, 4>(p, n_seqs, stream);
}

}  // extern "C"
