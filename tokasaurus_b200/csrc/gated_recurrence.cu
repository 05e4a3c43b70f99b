// A real-gated linear recurrence on every channel behind a short convolution (the recurrent block of Griffin's form):
//
//     u_t = bias_c + sum_k taps[:, k] x_(t - K + 1 + k),    x = W_x h + b_x  (zeros before a request's first token)
//     r_t = sigmoid(R_b u_b + b_r),   i_t = sigmoid(I_b u_b + b_i)      (b: one of `blocks` equal parts of the channels)
//     log a_t = -decay_scale * r_t * softplus(lam),   S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t,
//     out_t = S_t * gelu_tanh(W_y h + b_y).
//
// What a request carries in its slot: S [C] and the convolution's last K - 1 inputs [K - 1, C], float32.  Everything here
// is float32: the projections [y | x] arrive as float32 rows of one product, u, gates, decays and the recurrence stay
// float32; only out leaves in the activation type.  sqrt(1 - a^2) is sqrt(-expm1(2 log a)), exact where a is close to 1.
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
__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float gelu_tanh_f(float z) {
  return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
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

constexpr int KC = 64;       // channels of a part that the products take at a time
constexpr int AS = KC + 8;   // row stride in shared memory (bfloat16): 16 bytes of padding keep the banks apart
constexpr int WINDOW = 8;    // convolutions of up to so many taps keep their inputs in registers

// The convolution at channel c for `rows` consecutive tokens of the step from token t0 on (thread-private); rows past the
// step's end and padding tokens give 0.  put(r, u) takes the results.
template <typename Put>
__device__ __forceinline__ void convolve(const Conv& cv, const Step& st, const float* __restrict__ state, long long slot_stride,
                                         int C, int c, int t0, int rows, const int* s_seq, const int* s_idx, Put put) {
  const float bx = cv.x_bias[c], cb = cv.conv_bias[c];
  const float* col = cv.proj + cv.x_off + c;
  const int K = cv.K;
  // the input `back` tokens before row r: this step's if there is one, else a carried one
  auto input = [&](int r, int back) -> float {
    const int i = s_idx[r] - back;
    if (i >= 0) return col[(size_t)(t0 + r - back) * cv.stride] + bx;
    return state[(size_t)st.seq_slot[s_seq[r]] * slot_stride + C + (size_t)(K - 1 + i) * C + c];
  };
  if (K <= WINDOW) {
    float w[WINDOW], x[WINDOW];  // taps; the last inputs, x[K - 1] the current token's
#pragma unroll
    for (int k = 0; k < WINDOW; k++) {
      w[k] = k < K ? cv.taps[(size_t)c * K + k] : 0.f;
      x[k] = 0.f;
    }
    bool fill = true;
    for (int r = 0; r < rows; r++) {
      if (t0 + r >= st.n_tokens || s_seq[r] < 0) {
        put(r, 0.f);
        fill = true;
        continue;
      }
      if (fill || s_idx[r] == 0) {
#pragma unroll
        for (int k = 0; k < WINDOW; k++)
          if (k < K) x[k] = input(r, K - 1 - k);
        fill = false;
      } else {
#pragma unroll
        for (int k = 0; k + 1 < WINDOW; k++)
          if (k + 1 < K) x[k] = x[k + 1];
        const float now = col[(size_t)(t0 + r) * cv.stride] + bx;
#pragma unroll
        for (int k = 0; k < WINDOW; k++)
          if (k == K - 1) x[k] = now;
      }
      float acc = cb;
#pragma unroll
      for (int k = 0; k < WINDOW; k++)
        if (k < K) acc = fmaf(w[k], x[k], acc);
      put(r, acc);
    }
  } else {
    for (int r = 0; r < rows; r++) {
      float acc = 0.f;
      if (t0 + r < st.n_tokens && s_seq[r] >= 0) {
        acc = cb;
        for (int k = 0; k < K; k++) acc = fmaf(cv.taps[(size_t)c * K + k], input(r, K - 1 - k), acc);
      }
      put(r, acc);
    }
  }
}

// A decay as one number d: a - 1 (not positive) for decays above a half, else a itself (positive, however small).
__device__ __forceinline__ float decay_code(float log_a) {
  return log_a > -0.6931471f ? expm1f(log_a) : fmaxf(expf(log_a), 1e-37f);
}
__device__ __forceinline__ float decayed(float d, float S, float x) { return d <= 0.f ? S + fmaf(d, S, x) : fmaf(d, S, x); }

// The scan within a tile.  sa, sx [MT][NT + 1]: decays (coded) and inputs; afterwards P and Sl go to memory.  Threads: NT
// channels times SEGS runs of MT / SEGS tokens.
template <int MT, int NT, int SEGS>
__device__ __forceinline__ void tile_scan(float* sa, float* sx, float* ends, const Step& st, const float* __restrict__ state,
                                          long long slot_stride, int C, int c0, int n_ch, int t0, const int* s_seq,
                                          const int* s_idx, float* __restrict__ Pg, float* __restrict__ Sg) {
  constexpr int RUN = MT / SEGS, LD = NT + 1;
  const int ch = threadIdx.x % NT, seg = threadIdx.x / NT;
  const int c = c0 + ch;
  const bool mine = seg < SEGS && ch < n_ch;
  float S = 0.f, P = 1.f;
  if (mine) {
    for (int r = seg * RUN; r < (seg + 1) * RUN; r++) {
      if (t0 + r >= st.n_tokens || s_seq[r] < 0) {
        S = 0.f;
        P = 0.f;
      } else {
        const float a = sa[r * LD + ch], x = sx[r * LD + ch];
        if (s_idx[r] == 0) {  // the request's first token of this step starts from its slot
          S = decayed(a, state[(size_t)st.seq_slot[s_seq[r]] * slot_stride + c], x);
          P = 0.f;
        } else {
          S = decayed(a, S, x);
          P = decayed(a, P, 0.f);
        }
      }
      sx[r * LD + ch] = S;
      sa[r * LD + ch] = P;
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
    for (int r = seg * RUN; r < (seg + 1) * RUN; r++) {
      if (t0 + r >= st.n_tokens) break;
      const float p = sa[r * LD + ch];
      Sg[(size_t)(t0 + r) * C + c] = fmaf(p, Sin, sx[r * LD + ch]);
      Pg[(size_t)(t0 + r) * C + c] = p * Pin;
    }
  }
}

__device__ __forceinline__ void decay_and_input(float r_pre, float i_pre, float u, float neg, float& a, float& x) {
  const float log_a = neg * sigmoid_f(r_pre);
  a = decay_code(log_a);
  x = sqrtf(-expm1f(2.f * log_a)) * sigmoid_f(i_pre) * u;
}

// ------------------------------------------------------------------------------------------------ bfloat16 weights
// WM row groups of 16 tokens, WN column groups; a warp holds 16 tokens times NT / WN channels of BOTH gates.
template <int MT, int NT> struct GatesTC {
  static constexpr int WM = MT / 16;
  static constexpr int WN = MT >= 64 ? 2 : 4;
  static constexpr int THREADS = WM * WN * 32;
  static constexpr int CPW = NT / WN;          // channels a warp
  static constexpr int TILES = CPW / 8;        // 8-column tiles of one gate
  static constexpr int SEGS = THREADS / NT;
  static constexpr size_t U_BYTES = (size_t)3 * MT * AS * 2;
  static constexpr size_t W_BYTES = (size_t)2 * NT * AS * 2;
  static constexpr size_t OWN_BYTES = (size_t)MT * (NT + 1) * 4;  // u of the block's own channels, float32
  static constexpr size_t SCAN_BYTES = (size_t)(2 * MT * (NT + 1) + 2 * SEGS * NT) * 4;
  static constexpr size_t FRONT = (U_BYTES + W_BYTES > SCAN_BYTES ? U_BYTES + W_BYTES : SCAN_BYTES + 15) / 16 * 16;
  static constexpr size_t SMEM = FRONT + OWN_BYTES + 2 * MT * 4;
};

template <int MT, int NT>
__global__ void __launch_bounds__(GatesTC<MT, NT>::THREADS)
rglru_gates_tc_kernel(Conv cv, Step st, const float* __restrict__ state, long long slot_stride, int C, int part,
                      const bf16* __restrict__ w_r, const float* __restrict__ b_r, const bf16* __restrict__ w_i,
                      const float* __restrict__ b_i, const float* __restrict__ neg, float* __restrict__ Pg,
                      float* __restrict__ Sg, int wide) {
  using G = GatesTC<MT, NT>;
  extern __shared__ __align__(16) unsigned char smem[];
  bf16* us = reinterpret_cast<bf16*>(smem);  // [3][MT][AS]: hi, mid, lo
  bf16* ws = us + 3 * MT * AS;               // [gate][NT][AS]
  float* own = reinterpret_cast<float*>(smem + G::FRONT);  // [MT][NT + 1]
  int* s_seq = reinterpret_cast<int*>(own + MT * (NT + 1));
  int* s_idx = s_seq + MT;
  trigger_dependents();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t4 = lane & 3;
  const int col_tiles = (part + NT - 1) / NT;
  const int b = blockIdx.x / col_tiles, n0 = (blockIdx.x - b * col_tiles) * NT;  // the part; first channel within it
  const int n_ch = min(NT, part - n0);
  const int t0 = blockIdx.y * MT;
  for (int r = tid; r < MT; r += G::THREADS) {
    const int t = t0 + r;
    const int s = t < st.n_tokens ? st.token_seq[t] : -1;
    s_seq[r] = s;
    s_idx[r] = s >= 0 ? t - st.seq_q_start[s] : 0;
  }
  grid_dependency_wait();
  __syncthreads();
  const int wm = warp / G::WN, wn = warp - wm * G::WN;
  float acc[2][G::TILES][4];
#pragma unroll
  for (int q = 0; q < 2; q++)
#pragma unroll
    for (int j = 0; j < G::TILES; j++) acc[q][j][0] = acc[q][j][1] = acc[q][j][2] = acc[q][j][3] = 0.f;
  const bf16* wr = w_r + ((size_t)b * part + n0) * part;  // rows n0 .. of the part's matrix [out, in]
  const bf16* wi = w_i + ((size_t)b * part + n0) * part;

  for (int k0 = 0; k0 < part; k0 += KC) {
    const int kn = min(KC, part - k0);
    // the gates' rows of this run of channels (zeros beyond the part)
    if (wide) {
      for (int idx = tid; idx < 2 * NT * (KC / 8); idx += G::THREADS) {
        const int row = idx / (KC / 8), p = idx - row * (KC / 8);
        const int n = row < NT ? row : row - NT;
        bf16* dst = ws + row * AS + p * 8;
        if (n < n_ch && p * 8 < kn) cp_async16(dst, (row < NT ? wr : wi) + (size_t)n * part + k0 + p * 8);
        else *reinterpret_cast<uint4*>(dst) = make_uint4(0u, 0u, 0u, 0u);
      }
      cp_async_commit();
    } else {
      for (int idx = tid; idx < 2 * NT * KC; idx += G::THREADS) {
        const int row = idx / KC, k = idx - row * KC;
        const int n = row < NT ? row : row - NT;
        ws[row * AS + k] = n < n_ch && k < kn ? (row < NT ? wr : wi)[(size_t)n * part + k0 + k] : __float2bfloat16_rn(0.f);
      }
    }
    // the convolution of the run's channels, as three bfloat16 numbers; float32 for the block's own channels
    {
      constexpr int RUNS = G::THREADS / KC > 0 ? G::THREADS / KC : 1, ROWS = MT / RUNS;
      const int k = tid % KC, r0 = (tid / KC) * ROWS;
      auto put = [&](int r, float u) {
        const bf16 hi = __float2bfloat16_rn(u);
        const float u1 = u - __bfloat162float(hi);
        const bf16 mid = __float2bfloat16_rn(u1);
        us[(r0 + r) * AS + k] = hi;
        us[(MT + r0 + r) * AS + k] = mid;
        us[(2 * MT + r0 + r) * AS + k] = __float2bfloat16_rn(u1 - __bfloat162float(mid));
        const int n = k0 + k - n0;
        if (n >= 0 && n < n_ch) own[(r0 + r) * (NT + 1) + n] = u;
      };
      if (k < kn) convolve(cv, st, state, slot_stride, C, b * part + k0 + k, t0 + r0, ROWS, s_seq + r0, s_idx + r0, put);
      else
        for (int r = 0; r < ROWS; r++) put(r, 0.f);
    }
    cp_async_wait_all();
    __syncthreads();
#pragma unroll
    for (int ks = 0; ks < KC; ks += 32) {
      uint32_t af[3][2][4];
#pragma unroll
      for (int q = 0; q < 3; q++)
#pragma unroll
        for (int u = 0; u < 2; u++)
          ldmatrix_x4(af[q][u], smem_u32(us + (q * MT + wm * 16 + (lane & 15)) * AS + ks + u * 16 + (lane >> 4) * 8));
#pragma unroll
      for (int q = 0; q < 2; q++)
#pragma unroll
        for (int j = 0; j < G::TILES; j++) {
          uint32_t bf[4];  // two k-steps of 8 output channels
          ldmatrix_x4(bf, smem_u32(ws + (q * NT + wn * G::CPW + j * 8 + (lane & 7)) * AS + ks + (lane >> 3) * 8));
#pragma unroll
          for (int v = 2; v >= 0; v--) {  // the small shares first
            mma_bf16(acc[q][j], af[v][0], bf[0], bf[1]);
            mma_bf16(acc[q][j], af[v][1], bf[2], bf[3]);
          }
        }
    }
    __syncthreads();  // the buffers may be filled again
  }
  // decays and inputs, over the buffers that the products have left
  float* sa = reinterpret_cast<float*>(smem);
  float* sx = sa + MT * (NT + 1);
  float* ends = sx + MT * (NT + 1);
#pragma unroll
  for (int j = 0; j < G::TILES; j++) {
#pragma unroll
    for (int e = 0; e < 4; e++) {
      const int n = wn * G::CPW + j * 8 + 2 * t4 + (e & 1), r = wm * 16 + g + (e >> 1) * 8;
      if (n < n_ch) {
        const int c = b * part + n0 + n;
        float a, x;
        decay_and_input(acc[0][j][e] + b_r[c], acc[1][j][e] + b_i[c], own[r * (NT + 1) + n], neg[c], a, x);
        sa[r * (NT + 1) + n] = a;
        sx[r * (NT + 1) + n] = x;
      }
    }
  }
  __syncthreads();
  tile_scan<MT, NT, G::SEGS>(sa, sx, ends, st, state, slot_stride, C, b * part + n0, n_ch, t0, s_seq, s_idx, Pg, Sg);
}

// ------------------------------------------------------------------------------------------------ float32 weights
constexpr int FM = 32, FN = 32, FK = 32, FT = 256;  // tokens, channels, channels a time, threads

__global__ void __launch_bounds__(FT)
rglru_gates_f32_kernel(Conv cv, Step st, const float* __restrict__ state, long long slot_stride, int C, int part,
                       const float* __restrict__ w_r, const float* __restrict__ b_r, const float* __restrict__ w_i,
                       const float* __restrict__ b_i, const float* __restrict__ neg, float* __restrict__ Pg,
                       float* __restrict__ Sg) {
  __shared__ float us[FM][FK + 1], ws[2][FN][FK + 1], own[FM][FN + 1];
  __shared__ float sa[FM * (FN + 1)], sx[FM * (FN + 1)], ends[2 * (FT / FN) * FN];
  __shared__ int s_seq[FM], s_idx[FM];
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
  }
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
        if (m >= 0 && m < n_ch) own[r0 + r][m] = u;
      };
      if (k < kn) convolve(cv, st, state, slot_stride, C, b * part + k0 + k, t0 + r0, ROWS, s_seq + r0, s_idx + r0, put);
      else
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
  if (n < n_ch) {
    const int c = b * part + n0 + n;
#pragma unroll
    for (int r = 0; r < 4; r++) {
      float a, x;
      decay_and_input(ar[r] + b_r[c], ai[r] + b_i[c], own[r4 + r][n], neg[c], a, x);
      sa[(r4 + r) * (FN + 1) + n] = a;
      sx[(r4 + r) * (FN + 1) + n] = x;
    }
  }
  __syncthreads();
  tile_scan<FM, FN, FT / FN>(sa, sx, ends, st, state, slot_stride, C, b * part + n0, n_ch, t0, s_seq, s_idx, Pg, Sg);
}

// ------------------------------------------------------------------------------------------------ both
// Block (x, y): 64 channels, the token tile y of mt tokens; four runs of mt / 4 tokens.
constexpr int AC = 64, AR = 4;

template <typename T>
__global__ void __launch_bounds__(AC * AR)
rglru_apply_kernel(Conv cv, Step st, float* __restrict__ state, long long slot_stride, int C, const float* __restrict__ Pg,
                   const float* __restrict__ Sg, T* __restrict__ out, int mt, int write_state) {
  __shared__ float carry[AC];
  trigger_dependents();
  const int ch = threadIdx.x % AC, run = threadIdx.x / AC;
  const int c = blockIdx.x * AC + ch;
  const int t0 = blockIdx.y * mt;
  grid_dependency_wait();
  // the state at the end of the tile before; tiles are walked back until one has forgotten what came before it
  const int s0 = st.token_seq[t0];
  const bool need = blockIdx.y > 0 && s0 >= 0 && t0 > st.seq_q_start[s0];
  if (need && run == 0 && c < C) {
    float S = 0.f, P = 1.f;
    constexpr int BATCH = 8;
    for (int j = (int)blockIdx.y - 1; j >= 0 && P != 0.f; j -= BATCH) {
      float sv[BATCH], pv[BATCH];
#pragma unroll
      for (int k = 0; k < BATCH; k++) {
        const bool in = j - k >= 0;
        const size_t at = ((size_t)(in ? j - k : 0) * mt + mt - 1) * C + c;
        sv[k] = in ? Sg[at] : 0.f;
        pv[k] = in ? Pg[at] : 0.f;
      }
#pragma unroll
      for (int k = 0; k < BATCH; k++) {
        S = fmaf(P, sv[k], S);
        P *= pv[k];
      }
    }
    carry[ch] = S;
  }
  __syncthreads();
  if (c >= C) return;
  const float S_in = need ? carry[ch] : 0.f;
  const int per = mt / AR;
  const float by = cv.y_bias[c];
  for (int r = run * per; r < (run + 1) * per; r++) {
    const int t = t0 + r;
    if (t >= st.n_tokens) break;
    const int s = st.token_seq[t];
    if (s < 0) continue;
    const float S = fmaf(Pg[(size_t)t * C + c], S_in, Sg[(size_t)t * C + c]);
    const float y = cv.proj[(size_t)t * cv.stride + cv.y_off + c] + by;
    out[(size_t)t * C + c] = from_float<T>(S * gelu_tanh_f(y));
    const int n = st.seq_q_len[s], start = st.seq_q_start[s];
    if (write_state && t - start == n - 1) {  // the request's last token of this step
      float* slot = state + (size_t)st.seq_slot[s] * slot_stride;
      slot[c] = S;
      float* kept = slot + C;
      const float bx = cv.x_bias[c];
      for (int q = 0; q < cv.K - 1; q++) {  // ascending: input n + q of [carried ; new] is read before it is written
        const int at = n + q;
        kept[(size_t)q * C + c] = at < cv.K - 1 ? kept[(size_t)at * C + c]
                                                : cv.proj[(size_t)(start + at - (cv.K - 1)) * cv.stride + cv.x_off + c] + bx;
      }
    }
  }
}

template <int MT, int NT>
int gates_tc_launch(const Conv& cv, const Step& sp, const float* state, long long slot_stride, int C, int part, const void* w_r,
                    const float* b_r, const void* w_i, const float* b_i, const float* neg, float* P, float* S,
                    cudaStream_t st) {
  using G = GatesTC<MT, NT>;
  if (G::SMEM > 48 * 1024) {
    static bool done = false;
    if (!done) {
      cudaError_t e = cudaFuncSetAttribute(rglru_gates_tc_kernel<MT, NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)G::SMEM);
      if (e != cudaSuccess) return (int)e;
      done = true;
    }
  }
  const int wide = part % 8 == 0 && (((uintptr_t)w_r) & 15) == 0 && (((uintptr_t)w_i) & 15) == 0;
  const int tiles = (sp.n_tokens + MT - 1) / MT;
  if (tiles > 65535) return -3;
  return launch_pdl(rglru_gates_tc_kernel<MT, NT>, dim3((C / part) * ((part + NT - 1) / NT), tiles), dim3(G::THREADS), G::SMEM, st,
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
  int rc, mt;
  if (sizeof(T) == 4) {
    mt = FM;
    const int tiles = (sp.n_tokens + FM - 1) / FM;
    if (tiles > 65535) return -3;
    rc = launch_pdl(rglru_gates_f32_kernel, dim3(parts * ((part + FN - 1) / FN), tiles), dim3(FT), 0, st, cv, sp,
                    (const float*)state, slot_stride, C, part, (const float*)w_r, b_r, (const float*)w_i, b_i, neg, P, S);
  } else if (sp.n_tokens <= FEW_ROWS) {
    mt = 16;
    rc = gates_tc_launch<16, 32>(cv, sp, state, slot_stride, C, part, w_r, b_r, w_i, b_i, neg, P, S, st);
  } else {
    mt = 64;
    rc = gates_tc_launch<64, 64>(cv, sp, state, slot_stride, C, part, w_r, b_r, w_i, b_i, neg, P, S, st);
  }
  if (rc != 0) return rc;
  return launch_pdl(rglru_apply_kernel<T>, dim3((C + AC - 1) / AC, (sp.n_tokens + mt - 1) / mt), dim3(AC * AR), 0, st, cv, sp,
                    state, slot_stride, C, (const float*)P, (const float*)S, (T*)out, mt, write_state);
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
