// A real-gated linear recurrence on every channel behind a short convolution (the recurrent block of Griffin's form):
//
//     u_t = bias_c + sum_k taps[:, k] x_(t - K + 1 + k),    x = W_x h + b_x  (zeros before a request's first token)
//     r_t = sigmoid(R_b u_b + b_r),   i_t = sigmoid(I_b u_b + b_i)      (b: one of `blocks` equal parts of the channels)
//     log a_t = -decay_scale * r_t * softplus(lam),   S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t,
//     out_t = S_t * gelu_tanh(W_y h + b_y).
//
// What a request carries in its slot: S [C] and the convolution's last K - 1 inputs [K - 1, C], float32.  Everything here
// is float32: the projections [y | x] arrive as float32 rows of one product, u, gates, decays and the recurrence stay
// float32; only out leaves in the activation type.  1 - a^2 is -(a - 1)(a + 1) with a - 1 = expm1(log a) where a is close to 1.
// A decay close to 1 is kept as a - 1 = expm1(log a) and applied as S + ((a - 1) S + x): rounding a itself would be the
// same error at every token of a long memory, and those add up.
//
// The recurrence over a step's tokens is a scan in two kernels over tiles of MT consecutive tokens of the step, whatever
// requests they belong to (a request's first token of the step starts from its slot's S and forgets what came before
// it in the tile, so prompts, portions and single tokens are one case):
//   rglru_gates   a block owns MT tokens and NT channels of one part: the convolution, the two gate products over the
//                 part's channels, decays and inputs, and the scan within the tile: Sl_t (from 0 at the tile's start)
//                 and P_t, the product of the decays since then (0 from a request's first token on).
//   rglru_apply   S_t = Sl_t + P_t S_in, where S_in, the state at the end of the tile before, is put together from the
//                 last rows of the tiles ahead; the output branch; the request's new state and carried inputs.
//
// The gate products in bfloat16 engines (weights bfloat16) run on the tensor cores without losing u's 32 bits: u is the
// exact sum of three bfloat16 numbers (u = hi + mid + lo, 8 bits of the mantissa each), and the three products of
// bfloat16 operands, each exact, are added in float32 (mma.sync m16n8k16).  In float32 engines they run on the FP32 pipes.
#include "common.cuh"

using namespace tkb;

namespace {

using bf16 = __nv_bfloat16;

__device__ __forceinline__ uint32_t smem_u32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void cp_async_wait_all() { asm volatile("cp.async.wait_group 0;" ::: "memory"); }
__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// Two forms of the same functions: EXACT calls CUDA's float32 functions (float32 engines), the other the hardware's
// exponential, reciprocal and square root, each good to a few 1e-7 of its result (bfloat16 engines).
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
constexpr float LOG2E = 1.4426950408889634f;
template <bool EXACT> __device__ __forceinline__ float sigmoid_f(float z) {
  if (EXACT) return 1.f / (1.f + expf(-z));
  float r;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.f + ex2(-LOG2E * z)));
  return r;
}
template <bool EXACT> __device__ __forceinline__ float root_f(float x) {
  if (EXACT) return sqrtf(x);
  float r;
  asm("sqrt.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
  return r;
}
// 0.5 z (1 + tanh(k)) = z sigmoid(2 k)
template <bool EXACT> __device__ __forceinline__ float gelu_tanh_f(float z) {
  return z * sigmoid_f<EXACT>(2.f * 0.7978845608028654f * (z + 0.044715f * z * z * z));
}

struct Step {
  const int* token_seq;
  const int* seq_slot;
  const int* seq_q_start;
  const int* seq_q_len;
  int n_tokens;
};

struct Conv {
  const float* proj;  // [T, stride]: y at column y_off, x at column x_off
  int stride, y_off, x_off;
  const float* y_bias;
  const float* x_bias;
  const float* taps;  // [C, K]
  const float* conv_bias;
  int K;
};

// What a tile's tokens need to know: their request (-1: none), their place among the request's tokens of this step, and where
// the request's slot starts in the state.
struct Rows {
  const int* seq;
  const int* idx;
  const long long* slot;
  __device__ __forceinline__ Rows at(int r) const { return Rows{seq + r, idx + r, slot + r}; }
};

// The raw input of channel c, `back` tokens before token t (row r of the tile): this step's if there is one (with the
// projection's bias), else a carried one; 0 for a token that is none.  One load whatever the case, so that a thread's
// loads can be in flight together.
__device__ __forceinline__ float conv_input(const Conv& cv, const float* __restrict__ state, int C, int c, float bx, int t,
                                            const Rows& rows, int r, int back) {
  const bool live = rows.seq[r] >= 0;
  const int i = rows.idx[r] - back;
  const float* now = cv.proj + (size_t)(live && i >= 0 ? t - back : 0) * cv.stride + cv.x_off + c;
  const float* kept = state + rows.slot[r] + C + (long long)(cv.K - 1 + i) * C + c;
  const float v = *(live && i < 0 ? kept : now);
  return live ? v + (i >= 0 ? bx : 0.f) : 0.f;
}

constexpr int FAST_TAPS = 4;  // convolutions of so many taps keep a run's inputs in registers

// The convolution of one channel over ROWS consecutive tokens of the step (t0 + r).
// Rows past the step's end and padding tokens give 0.  Two halves, so that the loads of a run of channels can be in flight
// while the products of the run before are worked on: fetch() loads what a run inside one request needs (FAST_TAPS taps),
// put() makes the results; other runs (several requests, other taps) are loaded by put() itself, GROUP tokens at a time.
template <int ROWS, int GROUP> struct ConvRun {
  float x[ROWS + FAST_TAPS - 1];
  __device__ __forceinline__ static bool fast(const Conv& cv, const Rows& rows) {
    return cv.K == FAST_TAPS && rows.seq[0] >= 0 && rows.seq[0] == rows.seq[ROWS - 1];
  }
  __device__ __forceinline__ void fetch(const Conv& cv, const float* __restrict__ state, int C, int c, int t0, const Rows& rows) {
    const float bx = cv.x_bias[c];
    const float* col = cv.proj + (size_t)t0 * cv.stride + cv.x_off + c;
#pragma unroll
    for (int j = 0; j < FAST_TAPS - 1; j++) x[j] = conv_input(cv, state, C, c, bx, t0, rows, 0, FAST_TAPS - 1 - j);
#pragma unroll
    for (int r = 0; r < ROWS; r++) x[FAST_TAPS - 1 + r] = col[(size_t)r * cv.stride] + bx;
  }
  template <typename Put>
  __device__ __forceinline__ void put(bool is_fast, const Conv& cv, const float* __restrict__ state, int C, int c, int t0,
                                      const Rows& rows, Put out) {
    const float cb = cv.conv_bias[c];
    const float* w = cv.taps + (size_t)c * cv.K;
    if (is_fast) {
      float wk[FAST_TAPS];
#pragma unroll
      for (int k = 0; k < FAST_TAPS; k++) wk[k] = w[k];
#pragma unroll
      for (int r = 0; r < ROWS; r++) {
        float acc = cb;
#pragma unroll
        for (int k = 0; k < FAST_TAPS; k++) acc = fmaf(wk[k], x[r + k], acc);
        out(r, acc);
      }
      return;
    }
    const float bx = cv.x_bias[c];
    constexpr int G = ROWS < GROUP ? ROWS : GROUP;
#pragma unroll 1
    for (int r0 = 0; r0 < ROWS; r0 += G) {
      float acc[G];
#pragma unroll
      for (int g = 0; g < G; g++) acc[g] = cb;
      int k = 0;
      for (; k + 4 <= cv.K; k += 4) {
        float v[4][G], wv[4];
#pragma unroll
        for (int q = 0; q < 4; q++) {
          wv[q] = w[k + q];
#pragma unroll
          for (int g = 0; g < G; g++) v[q][g] = conv_input(cv, state, C, c, bx, t0 + r0 + g, rows, r0 + g, cv.K - 1 - k - q);
        }
#pragma unroll
        for (int q = 0; q < 4; q++)
#pragma unroll
          for (int g = 0; g < G; g++) acc[g] = fmaf(wv[q], v[q][g], acc[g]);
      }
      for (; k < cv.K; k++) {
        const float wv = w[k];
#pragma unroll
        for (int g = 0; g < G; g++) acc[g] = fmaf(wv, conv_input(cv, state, C, c, bx, t0 + r0 + g, rows, r0 + g, cv.K - 1 - k), acc[g]);
      }
#pragma unroll
      for (int g = 0; g < G; g++) out(r0 + g, rows.seq[r0 + g] >= 0 ? acc[g] : 0.f);
    }
  }
};

// From the gates' sums (biases added) and u: the input x = sqrt(1 - a^2) i u and the decay as one number d: a - 1 (not
// positive) for decays above a half, else a itself (positive, however small).  1 - a^2 = -(a - 1)(a + 1).
template <bool EXACT>
__device__ __forceinline__ void decay_and_input(float r_pre, float i_pre, float u, float neg, float& d, float& x) {
  const float log_a = neg * sigmoid_f<EXACT>(r_pre);
  const bool near = log_a > -0.6931471f;
  const float a = EXACT ? expf(log_a) : ex2(LOG2E * log_a);
  const float e = near ? expm1f(log_a) : a - 1.f;
  d = near ? e : fmaxf(a, 1e-37f);
  x = root_f<EXACT>(-e * (2.f + e)) * sigmoid_f<EXACT>(i_pre) * u;
}
__device__ __forceinline__ float decayed(float d, float S, float x) { return d <= 0.f ? S + fmaf(d, S, x) : fmaf(d, S, x); }

// What a scanning thread needs of its channel, fetched ahead: the biases, the decay's factor, and (short runs) the slots'
// states of its tokens that are the first of their request.
template <int RUN> struct ScanArgs {
  float br, bi, neg, s0[RUN <= 4 ? RUN : 1];
  __device__ __forceinline__ void channel(const float* b_r, const float* b_i, const float* ng, int c) {
    br = b_r[c];
    bi = b_i[c];
    neg = ng[c];
  }
  __device__ __forceinline__ void slots(const float* __restrict__ state, int c, const Rows& rows) {
    if (RUN <= 4) {
#pragma unroll
      for (int r = 0; r < RUN; r++) s0[RUN <= 4 ? r : 0] = rows.seq[r] >= 0 && rows.idx[r] == 0 ? state[rows.slot[r] + c] : 0.f;
    }
  }
};

// Decays, inputs and the scan within a tile.  sr, si [MT][NT + 1]: the gates' sums; own: u; afterwards P and Sl go to
// memory.  Threads: NT channels times SEGS runs of RUN = MT / SEGS tokens.
template <int MT, int NT, int SEGS, bool EXACT>
__device__ __forceinline__ void tile_scan(float* sr, float* si, const float* own, float* ends, const ScanArgs<MT / SEGS>& args,
                                          const float* __restrict__ state, int n_tokens, int C, int c0, int n_ch, int t0,
                                          const Rows& rows, float* __restrict__ Pg, float* __restrict__ Sg) {
  constexpr int RUN = MT / SEGS, LD = NT + 1;
  const int ch = threadIdx.x % NT, seg = threadIdx.x / NT;
  const int c = c0 + ch;
  const bool mine = seg < SEGS && ch < n_ch;
  float S = 0.f, P = 1.f;
  if (mine) {
#pragma unroll 4
    for (int q = 0; q < RUN; q++) {
      const int r = seg * RUN + q;
      if (rows.seq[r] < 0) {
        S = 0.f;
        P = 0.f;
      } else {
        float d, x;
        decay_and_input<EXACT>(sr[r * LD + ch] + args.br, si[r * LD + ch] + args.bi, own[r * LD + ch], args.neg, d, x);
        if (rows.idx[r] == 0) {  // the request's first token of this step starts from its slot
          S = decayed(d, RUN <= 4 ? args.s0[RUN <= 4 ? q : 0] : state[rows.slot[r] + c], x);
          P = 0.f;
        } else {
          S = decayed(d, S, x);
          P = decayed(d, P, 0.f);
        }
      }
      si[r * LD + ch] = S;
      sr[r * LD + ch] = P;
    }
    ends[(seg * NT + ch) * 2] = S;
    ends[(seg * NT + ch) * 2 + 1] = P;
  }
  __syncthreads();
  if (mine) {
    float Sin = 0.f, Pin = 1.f;
    for (int k = 0; k < seg; k++) {
      const float Sk = ends[(k * NT + ch) * 2], Pk = ends[(k * NT + ch) * 2 + 1];
      Sin = fmaf(Pk, Sin, Sk);
      Pin *= Pk;
    }
#pragma unroll 4
    for (int r = seg * RUN; r < (seg + 1) * RUN; r++) {
      if (t0 + r >= n_tokens) break;
      const float p = sr[r * LD + ch];
      Sg[(size_t)(t0 + r) * C + c] = fmaf(p, Sin, si[r * LD + ch]);
      Pg[(size_t)(t0 + r) * C + c] = p * Pin;
    }
  }
}

// ------------------------------------------------------------------------------------------------ bfloat16 weights
// WM row groups of 16 tokens times WN column groups times GS groups of gates; a warp holds 16 tokens times NT / WN channels of
// both gates (GS = 1) or of one (GS = 2).  KC: channels of a part that the products take at a time.
template <int MT, int NT, int KC> struct GatesTC {
  static constexpr int AS = KC + 8;            // row stride in shared memory (bfloat16): 16 bytes of padding keep the banks apart
  static constexpr int WM = MT / 16;
  static constexpr int WN = MT >= 64 ? 2 : 4;
  static constexpr int GS = MT >= 64 ? 1 : 2;
  static constexpr int GW = 2 / GS;            // gates a warp
  static constexpr int THREADS = WM * WN * GS * 32;
  static constexpr int CPW = NT / WN;          // channels a warp
  static constexpr int TILES = CPW / 8;        // 8-column tiles of one gate
  static constexpr int NV = GW * TILES == 1 ? 3 : 1;  // sums a tile (a product waits for the one before it in the same sum)
  static constexpr int SEGS = THREADS / NT > MT ? MT : THREADS / NT;
  static constexpr int RUNS = THREADS / KC, ROWS = MT / RUNS;  // a thread's run of the convolution
  static_assert(THREADS % KC == 0, "a thread owns one channel of a run");
  static constexpr size_t U_BYTES = (size_t)3 * MT * AS * 2;
  static constexpr size_t W_BYTES = (size_t)2 * NT * AS * 2;      // one of two buffers
  static constexpr size_t OWN_BYTES = (size_t)MT * (NT + 1) * 4;  // u of the block's own channels, float32
  static constexpr size_t SCAN_BYTES = (size_t)(2 * MT * (NT + 1) + 2 * SEGS * NT) * 4;
  static constexpr size_t FRONT = (U_BYTES + 2 * W_BYTES > SCAN_BYTES ? U_BYTES + 2 * W_BYTES : SCAN_BYTES + 15) / 16 * 16;
  static constexpr size_t SMEM = FRONT + (OWN_BYTES + 7) / 8 * 8 + MT * (8 + 4 + 4);
  using Run = ConvRun<ROWS, (MT >= 64 ? 2 : 4)>;
};

template <int MT, int NT, int KC>
__global__ void __launch_bounds__(GatesTC<MT, NT, KC>::THREADS, 2)
rglru_gates_tc_kernel(Conv cv, Step st, const float* __restrict__ state, long long slot_stride, int C, int part,
                      const bf16* __restrict__ w_r, const float* __restrict__ b_r, const bf16* __restrict__ w_i,
                      const float* __restrict__ b_i, const float* __restrict__ neg, float* __restrict__ Pg,
                      float* __restrict__ Sg, int wide) {
  using G = GatesTC<MT, NT, KC>;
  constexpr int AS = G::AS;
  extern __shared__ __align__(16) unsigned char smem[];
  bf16* us = reinterpret_cast<bf16*>(smem);  // [3][MT][AS]: hi, mid, lo
  bf16* wbuf = us + 3 * MT * AS;             // two of [gate][NT][AS]
  float* own = reinterpret_cast<float*>(smem + G::FRONT);  // [MT][NT + 1]
  long long* s_slot = reinterpret_cast<long long*>(smem + G::FRONT + (G::OWN_BYTES + 7) / 8 * 8);
  int* s_seq = reinterpret_cast<int*>(s_slot + MT);
  int* s_idx = s_seq + MT;
  const Rows rows{s_seq, s_idx, s_slot};
  trigger_dependents();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t4 = lane & 3;
  const int col_tiles = (part + NT - 1) / NT;
  const int b = blockIdx.x / col_tiles, n0 = (blockIdx.x - b * col_tiles) * NT;  // the part; first channel within it
  const int n_ch = min(NT, part - n0);
  const int t0 = blockIdx.y * MT;
  const bf16* wr = w_r + ((size_t)b * part + n0) * part;  // rows n0 .. of the part's matrix [out, in]
  const bf16* wi = w_i + ((size_t)b * part + n0) * part;
  // the gates' rows of the channels k0 .. of the part (zeros beyond it)
  auto stage_w = [&](int k0, bf16* ws) {
    const int kn = min(KC, part - k0);
    if (wide) {
      for (int idx = tid; idx < 2 * NT * (KC / 8); idx += G::THREADS) {
        const int row = idx / (KC / 8), p = idx - row * (KC / 8);
        const int n = row < NT ? row : row - NT;
        bf16* dst = ws + row * AS + p * 8;
        if (n < n_ch && p * 8 < kn) cp_async16(dst, (row < NT ? wr : wi) + (size_t)n * part + k0 + p * 8);
        else *reinterpret_cast<uint4*>(dst) = make_uint4(0u, 0u, 0u, 0u);
      }
    } else {
      for (int idx = tid; idx < 2 * NT * KC; idx += G::THREADS) {
        const int row = idx / KC, k = idx - row * KC;
        const int n = row < NT ? row : row - NT;
        ws[row * AS + k] = n < n_ch && k < kn ? (row < NT ? wr : wi)[(size_t)n * part + k0 + k] : __float2bfloat16_rn(0.f);
      }
    }
    cp_async_commit();
  };
  stage_w(0, wbuf);  // (no kernel writes weights: they may be fetched while the kernel ahead still runs)
  for (int r = tid; r < MT; r += G::THREADS) {
    const int t = t0 + r;
    const int s = t < st.n_tokens ? st.token_seq[t] : -1;
    s_seq[r] = s;
    s_idx[r] = s >= 0 ? t - st.seq_q_start[s] : 0;
    s_slot[r] = s >= 0 ? (long long)st.seq_slot[s] * slot_stride : 0;
  }
  // what the scan will want of its channel
  const int sch = tid % NT, sseg = tid / NT;
  constexpr int SRUN = MT / G::SEGS;
  ScanArgs<SRUN> args;
  const bool scans = sseg < G::SEGS && sch < n_ch;
  if (scans) args.channel(b_r, b_i, neg, b * part + n0 + sch);
  grid_dependency_wait();
  __syncthreads();
  const int wm = warp % G::WM, wn = (warp / G::WM) % G::WN, q0 = (warp / (G::WM * G::WN)) * G::GW;
  float acc[G::NV][G::GW][G::TILES][4];
#pragma unroll
  for (int v = 0; v < G::NV; v++)
#pragma unroll
    for (int q = 0; q < G::GW; q++)
#pragma unroll
      for (int j = 0; j < G::TILES; j++) acc[v][q][j][0] = acc[v][q][j][1] = acc[v][q][j][2] = acc[v][q][j][3] = 0.f;

  // this thread's channel within a run of KC, and its rows
  const int kt = tid % KC, r0 = (tid / KC) * G::ROWS;
  typename G::Run run;
  const bool is_fast = G::Run::fast(cv, rows.at(r0));
  auto fetch = [&](int k0) {
    if (is_fast && k0 + kt < part) run.fetch(cv, state, C, b * part + k0 + kt, t0 + r0, rows.at(r0));
  };
  auto put_u = [&](int k0) {
    const int k = k0 + kt, n = k - n0;
    const bool keep = n >= 0 && n < n_ch;
    auto put = [&](int r, float u) {
      const bf16 hi = __float2bfloat16_rn(u);
      const float u1 = u - __bfloat162float(hi);
      const bf16 mid = __float2bfloat16_rn(u1);
      us[(r0 + r) * AS + kt] = hi;
      us[(MT + r0 + r) * AS + kt] = mid;
      us[(2 * MT + r0 + r) * AS + kt] = __float2bfloat16_rn(u1 - __bfloat162float(mid));
      if (keep) own[(r0 + r) * (NT + 1) + n] = u;
    };
    if (k < part) run.put(is_fast, cv, state, C, b * part + k, t0 + r0, rows.at(r0), put);
    else
      for (int r = 0; r < G::ROWS; r++) put(r, 0.f);
  };
  if (scans) args.slots(state, b * part + n0 + sch, rows.at(sseg * SRUN));
  fetch(0);
  for (int k0 = 0, it = 0; k0 < part; k0 += KC, it++) {
    const bf16* ws = wbuf + (it & 1) * (G::W_BYTES / 2);
    put_u(k0);
    cp_async_wait_all();
    __syncthreads();
    if (k0 + KC < part) {  // the next run's weights and inputs are on their way during the products
      stage_w(k0 + KC, wbuf + ((it + 1) & 1) * (G::W_BYTES / 2));
      fetch(k0 + KC);
    }
#pragma unroll
    for (int ks = 0; ks < KC; ks += 32) {
      uint32_t af[3][2][4];
#pragma unroll
      for (int q = 0; q < 3; q++)
#pragma unroll
        for (int u = 0; u < 2; u++)
          ldmatrix_x4(af[q][u], smem_u32(us + (q * MT + wm * 16 + (lane & 15)) * AS + ks + u * 16 + (lane >> 4) * 8));
#pragma unroll
      for (int q = 0; q < G::GW; q++) {
        uint32_t bf[G::TILES][4];  // two k-steps of 8 output channels each
#pragma unroll
        for (int j = 0; j < G::TILES; j++)
          ldmatrix_x4(bf[j], smem_u32(ws + ((q0 + q) * NT + wn * G::CPW + j * 8 + (lane & 7)) * AS + ks + (lane >> 3) * 8));
#pragma unroll
        for (int v = 2; v >= 0; v--)  // the small shares first; neighbouring products belong to different sums
#pragma unroll
          for (int u = 0; u < 2; u++)
#pragma unroll
            for (int j = 0; j < G::TILES; j++)
              mma_bf16(acc[G::NV == 3 ? v : 0][q][j], af[v][u], bf[j][2 * u], bf[j][2 * u + 1]);
      }
    }
    __syncthreads();  // us may be filled again
  }
  // the gates' sums, over the buffers that the products have left
  float* sr = reinterpret_cast<float*>(smem);
  float* si = sr + MT * (NT + 1);
  float* ends = si + MT * (NT + 1);
#pragma unroll
  for (int q = 0; q < G::GW; q++) {
    float* dst = q0 + q == 0 ? sr : si;
#pragma unroll
    for (int j = 0; j < G::TILES; j++)
#pragma unroll
      for (int e = 0; e < 4; e++)
        dst[(wm * 16 + g + (e >> 1) * 8) * (NT + 1) + wn * G::CPW + j * 8 + 2 * t4 + (e & 1)] =
            G::NV == 3 ? acc[G::NV - 1][q][j][e] + acc[G::NV / 2][q][j][e] + acc[0][q][j][e] : acc[0][q][j][e];
  }
  __syncthreads();
  tile_scan<MT, NT, G::SEGS, false>(sr, si, own, ends, args, state, st.n_tokens, C, b * part + n0, n_ch, t0, rows, Pg, Sg);
}

// ------------------------------------------------------------------------------------------------ float32 weights
constexpr int FM = 32, FN = 32, FK = 32, FT = 256;  // tokens, channels, channels a time, threads

__global__ void __launch_bounds__(FT)
rglru_gates_f32_kernel(Conv cv, Step st, const float* __restrict__ state, long long slot_stride, int C, int part,
                       const float* __restrict__ w_r, const float* __restrict__ b_r, const float* __restrict__ w_i,
                       const float* __restrict__ b_i, const float* __restrict__ neg, float* __restrict__ Pg,
                       float* __restrict__ Sg) {
  __shared__ float us[FM][FK + 1], ws[2][FN][FK + 1], own[FM * (FN + 1)];
  __shared__ float sa[FM * (FN + 1)], sx[FM * (FN + 1)], ends[2 * (FT / FN) * FN];
  __shared__ int s_seq[FM], s_idx[FM];
  __shared__ long long s_slot[FM];
  trigger_dependents();
  const int tid = threadIdx.x;
  const int col_tiles = (part + FN - 1) / FN;
  const int b = blockIdx.x / col_tiles, n0 = (blockIdx.x - b * col_tiles) * FN;
  const int n_ch = min(FN, part - n0);
  const int t0 = blockIdx.y * FM;
  for (int r = tid; r < FM; r += FT) {
    const int t = t0 + r;
    const int s = t < st.n_tokens ? st.token_seq[t] : -1;
    s_seq[r] = s;
    s_idx[r] = s >= 0 ? t - st.seq_q_start[s] : 0;
    s_slot[r] = s >= 0 ? (long long)st.seq_slot[s] * slot_stride : 0;
  }
  const Rows rows{s_seq, s_idx, s_slot};
  grid_dependency_wait();
  __syncthreads();
  const int n = tid % FN, r4 = (tid / FN) * 4;  // this thread: channel n, four tokens
  float ar[4] = {0.f, 0.f, 0.f, 0.f}, ai[4] = {0.f, 0.f, 0.f, 0.f};
  const float* wr = w_r + ((size_t)b * part + n0) * part;
  const float* wi = w_i + ((size_t)b * part + n0) * part;
  for (int k0 = 0; k0 < part; k0 += FK) {
    const int kn = min(FK, part - k0);
    for (int idx = tid; idx < 2 * FN * FK; idx += FT) {
      const int row = idx / FK, k = idx - row * FK, m = row % FN;
      ws[row / FN][m][k] = m < n_ch && k < kn ? (row < FN ? wr : wi)[(size_t)m * part + k0 + k] : 0.f;
    }
    {
      constexpr int ROWS = FM / (FT / FK);
      const int k = tid % FK, r0 = (tid / FK) * ROWS;
      auto put = [&](int r, float u) {
        us[r0 + r][k] = u;
        const int m = k0 + k - n0;
        if (m >= 0 && m < n_ch) own[(r0 + r) * (FN + 1) + m] = u;
      };
      ConvRun<ROWS, 4> run;
      const bool is_fast = ConvRun<ROWS, 4>::fast(cv, rows.at(r0));
      if (k < kn) {
        if (is_fast) run.fetch(cv, state, C, b * part + k0 + k, t0 + r0, rows.at(r0));
        run.put(is_fast, cv, state, C, b * part + k0 + k, t0 + r0, rows.at(r0), put);
      } else
        for (int r = 0; r < ROWS; r++) put(r, 0.f);
    }
    __syncthreads();
    for (int k = 0; k < kn; k++) {
      const float vr = ws[0][n][k], vi = ws[1][n][k];
#pragma unroll
      for (int r = 0; r < 4; r++) {
        ar[r] = fmaf(us[r4 + r][k], vr, ar[r]);
        ai[r] = fmaf(us[r4 + r][k], vi, ai[r]);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int r = 0; r < 4; r++) {
    sa[(r4 + r) * (FN + 1) + n] = ar[r];
    sx[(r4 + r) * (FN + 1) + n] = ai[r];
  }
  ScanArgs<FM / (FT / FN)> args;
  if (n < n_ch) {
    args.channel(b_r, b_i, neg, b * part + n0 + n);
    args.slots(state, b * part + n0 + n, rows.at((tid / FN) * (FM / (FT / FN))));
  }
  __syncthreads();
  tile_scan<FM, FN, FT / FN, true>(sa, sx, own, ends, args, state, st.n_tokens, C, b * part + n0, n_ch, t0, rows, Pg, Sg);
}

// ------------------------------------------------------------------------------------------------ both
// Block (x, y): 64 channels, the token tile y of MT tokens; four runs of MT / 4 tokens.
constexpr int AC = 64, AR = 4;

template <typename T, int MT>
__global__ void __launch_bounds__(AC * AR)
rglru_apply_kernel(Conv cv, Step st, float* __restrict__ state, long long slot_stride, int C, const float* __restrict__ Pg,
                   const float* __restrict__ Sg, T* __restrict__ out, int write_state) {
  __shared__ float carry[AR][AC][2];
  __shared__ int s_seq[MT], s_len[MT];  // a token's request; the request's tokens in this step, where it is the last of them
  __shared__ long long s_slot[MT];      // where its slot starts
  __shared__ int s_goes_on;             // the tile's first token is not its request's first of this step
  trigger_dependents();
  const int ch = threadIdx.x % AC, run = threadIdx.x / AC;
  const int c = blockIdx.x * AC + ch;
  const int t0 = blockIdx.y * MT;
  for (int r = threadIdx.x; r < MT; r += AC * AR) {
    const int t = t0 + r;
    const int s = t < st.n_tokens ? st.token_seq[t] : -1;
    const int start = s >= 0 ? st.seq_q_start[s] : 0, n = s >= 0 ? st.seq_q_len[s] : 0;
    s_seq[r] = s;
    s_len[r] = s >= 0 && t - start == n - 1 ? n : 0;
    s_slot[r] = s >= 0 ? (long long)st.seq_slot[s] * slot_stride : 0;
    if (r == 0) s_goes_on = s >= 0 && t > start;
  }
  const float by = c < C ? cv.y_bias[c] : 0.f, bx = c < C ? cv.x_bias[c] : 0.f;
  __syncthreads();
  grid_dependency_wait();
  constexpr int PER = MT / AR, BATCH = 4;
  constexpr bool EXACT = sizeof(T) == 4;
  static_assert(PER % BATCH == 0, "whole batches a run");
  // the state at the end of the tile before: S_in = sum of the tiles' own last states, each times the decays behind it.
  // The tiles are shared out among the four runs, the nearest first, and walked back until one has forgotten what came
  // before it (a request's first token did).
  const bool need = blockIdx.y > 0 && s_goes_on != 0;
  if (need) {
    const int per = ((int)blockIdx.y + AR - 1) / AR;
    const int hi = (int)blockIdx.y - 1 - run * per, lo = max(-1, hi - per);  // tiles hi, hi - 1, ... above lo
    float S = 0.f, P = 1.f;
    if (c < C) {
      for (int j = hi; j > lo && P != 0.f; j -= 8) {
        float sv[8], pv[8];
#pragma unroll
        for (int k = 0; k < 8; k++) {
          const bool in = j - k > lo;
          const size_t at = ((size_t)(in ? j - k : 0) * MT + MT - 1) * C + c;
          sv[k] = in ? Sg[at] : 0.f;
          pv[k] = in ? Pg[at] : 1.f;
        }
#pragma unroll
        for (int k = 0; k < 8; k++) {
          S = fmaf(P, sv[k], S);
          P *= pv[k];
        }
      }
    }
    carry[run][ch][0] = S;
    carry[run][ch][1] = P;
  }
  __syncthreads();
  if (c >= C) return;
  float S_in = 0.f;
  if (need) {
#pragma unroll
    for (int q = AR - 1; q >= 0; q--) S_in = fmaf(carry[q][ch][1], S_in, carry[q][ch][0]);
  }
#pragma unroll 1
  for (int b0 = run * PER; b0 < (run + 1) * PER; b0 += BATCH) {
    float P[BATCH], S[BATCH], y[BATCH], v[BATCH][FAST_TAPS - 1];
#pragma unroll
    for (int k = 0; k < BATCH; k++) {
      const size_t t = (size_t)(t0 + b0 + k);
      const bool live = s_seq[b0 + k] >= 0;
      P[k] = live ? Pg[t * C + c] : 0.f;
      S[k] = live ? Sg[t * C + c] : 0.f;
      y[k] = live ? cv.proj[t * cv.stride + cv.y_off + c] + by : 0.f;
    }
    // a request's last token of this step brings its carried inputs forward: [carried ; new] n .. n + K - 2
    if (cv.K == FAST_TAPS) {
#pragma unroll
      for (int k = 0; k < BATCH; k++) {
        const int n = s_len[b0 + k];
        if (n > 0) {
          const float* kept = state + s_slot[b0 + k] + C + c;
          const float* xs = cv.proj + (size_t)(t0 + b0 + k - n + 1) * cv.stride + cv.x_off + c;  // the request's first token of the step
#pragma unroll
          for (int q = 0; q < FAST_TAPS - 1; q++) {
            const int at = n + q;
            v[k][q] = at < FAST_TAPS - 1 ? kept[(size_t)at * C] : xs[(size_t)(at - (FAST_TAPS - 1)) * cv.stride] + bx;
          }
        }
      }
    }
#pragma unroll
    for (int k = 0; k < BATCH; k++) {
      const int n = s_len[b0 + k];
      if (s_seq[b0 + k] < 0) continue;
      const float Sn = fmaf(P[k], S_in, S[k]);
      out[(size_t)(t0 + b0 + k) * C + c] = from_float<T>(Sn * gelu_tanh_f<EXACT>(y[k]));
      if (write_state && n > 0) {
        float* slot = state + s_slot[b0 + k] + c;
        slot[0] = Sn;
        if (cv.K == FAST_TAPS) {
#pragma unroll
          for (int q = 0; q < FAST_TAPS - 1; q++) slot[(size_t)(q + 1) * C] = v[k][q];
        } else {
          const float* xs = cv.proj + (size_t)(t0 + b0 + k - n + 1) * cv.stride + cv.x_off + c;
          for (int q = 0; q < cv.K - 1; q++) {  // ascending: n + q is read before it is written
            const int at = n + q;
            slot[(size_t)(q + 1) * C] = at < cv.K - 1 ? slot[(size_t)(at + 1) * C] : xs[(size_t)(at - (cv.K - 1)) * cv.stride] + bx;
          }
        }
      }
    }
  }
}

template <typename T, int MT>
int apply_launch(const Conv& cv, const Step& sp, float* state, long long slot_stride, int C, const float* P, const float* S, void* out,
                 int write_state, cudaStream_t st) {
  return launch_pdl(rglru_apply_kernel<T, MT>, dim3((C + AC - 1) / AC, (sp.n_tokens + MT - 1) / MT), dim3(AC * AR), 0, st, cv, sp,
                    state, slot_stride, C, P, S, (T*)out, write_state);
}

template <int MT, int NT, int KC>
int gates_tc_launch(const Conv& cv, const Step& sp, const float* state, long long slot_stride, int C, int part, const void* w_r,
                    const float* b_r, const void* w_i, const float* b_i, const float* neg, float* P, float* S,
                    cudaStream_t st) {
  using G = GatesTC<MT, NT, KC>;
  if (G::SMEM > 48 * 1024) {
    static bool done = false;
    if (!done) {
      cudaError_t e = cudaFuncSetAttribute(rglru_gates_tc_kernel<MT, NT, KC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)G::SMEM);
      if (e != cudaSuccess) return (int)e;
      done = true;
    }
  }
  const int wide = part % 8 == 0 && (((uintptr_t)w_r) & 15) == 0 && (((uintptr_t)w_i) & 15) == 0;
  const int tiles = (sp.n_tokens + MT - 1) / MT;
  if (tiles > 65535) return -3;
  return launch_pdl(rglru_gates_tc_kernel<MT, NT, KC>, dim3((C / part) * ((part + NT - 1) / NT), tiles), dim3(G::THREADS), G::SMEM, st,
                    cv, sp, state, slot_stride, C, part, (const bf16*)w_r, b_r, (const bf16*)w_i, b_i, neg, P, S, wide);
}

// few rows: narrow tiles of channels, so that more blocks fetch the gates' weights side by side
constexpr int FEW_ROWS = 64;

template <typename T>
int rglru_launch(Conv cv, Step sp, float* state, long long slot_stride, int C, int parts, const void* w_r, const float* b_r,
                 const void* w_i, const float* b_i, const float* neg, float* P, float* S, void* out, int write_state,
                 cudaStream_t st) {
  if (sp.n_tokens <= 0) return 0;
  if (C <= 0 || parts <= 0 || C % parts || cv.K < 1 || slot_stride < (long long)C * cv.K) return -2;
  const int part = C / parts;
  int rc;
  if (sizeof(T) == 4) {
    const int tiles = (sp.n_tokens + FM - 1) / FM;
    if (tiles > 65535) return -3;
    rc = launch_pdl(rglru_gates_f32_kernel, dim3(parts * ((part + FN - 1) / FN), tiles), dim3(FT), 0, st, cv, sp,
                    (const float*)state, slot_stride, C, part, (const float*)w_r, b_r, (const float*)w_i, b_i, neg, P, S);
    return rc != 0 ? rc : apply_launch<T, FM>(cv, sp, state, slot_stride, C, P, S, out, write_state, st);
  }
  if (sp.n_tokens <= FEW_ROWS) {
    rc = gates_tc_launch<16, 32, 256>(cv, sp, state, slot_stride, C, part, w_r, b_r, w_i, b_i, neg, P, S, st);
    return rc != 0 ? rc : apply_launch<T, 16>(cv, sp, state, slot_stride, C, P, S, out, write_state, st);
  }
  rc = gates_tc_launch<64, 64, 64>(cv, sp, state, slot_stride, C, part, w_r, b_r, w_i, b_i, neg, P, S, st);
  return rc != 0 ? rc : apply_launch<T, 64>(cv, sp, state, slot_stride, C, P, S, out, write_state, st);
}

}  // namespace

// proj float32 [T, stride] with y at column y_off and x at x_off; w_r, w_i [parts, C / parts, C / parts] in the engine's
// type; neg float32 [C] = -decay_scale * softplus(lam); scratch P, S float32 [T, C]; state float32 [slots, slot_stride]:
// S [C], then the carried inputs [K - 1, C]; out [T, C] in the engine's type.
#define TKB_RGLRU_EXPORT(SUF, T)                                                                                      \
  TKB_EXPORT int tkb_rglru_##SUF(const float* proj, int stride, int y_off, int x_off, const float* y_bias,            \
                                 const float* x_bias, const float* taps, const float* conv_bias, int K, int C,        \
                                 int parts, const void* w_r, const float* b_r, const void* w_i, const float* b_i,     \
                                 const float* neg, float* state, long long slot_stride, const int* token_seq,         \
                                 const int* seq_slot, const int* seq_q_start, const int* seq_q_len, int n_tokens,     \
                                 float* P, float* S, void* out, int write_state, void* st) {                          \
    return rglru_launch<T>(Conv{proj, stride, y_off, x_off, y_bias, x_bias, taps, conv_bias, K},                      \
                           Step{token_seq, seq_slot, seq_q_start, seq_q_len, n_tokens}, state, slot_stride, C, parts, \
                           w_r, b_r, w_i, b_i, neg, P, S, out, write_state, (cudaStream_t)st);                        \
  }
TKB_RGLRU_EXPORT(f32, float)
TKB_RGLRU_EXPORT(bf16, __nv_bfloat16)
