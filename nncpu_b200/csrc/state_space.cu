// State-space mixers with one decay per head and token (Mamba-2: Dao and Gu, "Transformers are SSMs").  Per head, with a
// state S of N rows and P columns in 32-bit floats, a step size dt > 0, a decay exp(la) with la = -exp(A_log) dt, vectors
// B and C of N lanes (shared by the heads of a group) and x of P lanes:
//     S <- exp(la) S + dt B x^T,        y = S^T C + D x
// Before it, x, B and C pass a causal convolution per channel (taps weights, the last one the current token's, zeros
// before the sequence's start) with a bias, and SiLU; dt <- softplus(dt + dt_bias).  After it, y times silu(z) is
// RMS-normed in equal parts and multiplied by a weight.
//
// A token's row of proj [n_tok, ld] (32-bit) holds z (H P), x (H P), B (G N), C (G N), dt (H), in this order; the
// convolutions' channels are the C_ = H P + 2 G N lanes from column H P on.
//
// A sequence's state is a row of the cache's state area: S of every head, [H, N, P], and behind it (conv_at) a ring of the
// convolutions' inputs, [taps, C_]: the input of position p lies in place p mod taps.  A ring of taps places, one more than
// the taps - 1 inputs a token looks back at, lets a decode step read the old inputs and write the new one in the same
// kernel: the place it writes is none of those it reads, whichever block comes first.
//
// Three kernels for the recurrence: a decode step (convolution, step size, recurrence and read-out in one launch); a scan
// in 32-bit on the CUDA cores that walks the tokens in order (float32 runs, portions of a few tokens); and for prompts a
// chunked form on the tensor cores (below).

#include <math.h>

#define NN_LIB state_space
#include "common.cuh"

namespace {

constexpr int kMaxTaps = 32;

__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(0.0f - z)); }

// The sizes of a mixer, and where things lie.
struct Sizes {
    int H, P, G, N, taps;
    int ld;              // floats a row of proj
    int P8, N8;          // lanes of a head's x and of a group's B and C in the convolved rows (multiples of 8, zeros behind)
    long slot_stride;    // floats a state row
    long conv_at;        // where the ring starts in it
    __host__ __device__ int inner() const { return H * P; }
    __host__ __device__ int channels() const { return H * P + 2 * G * N; }
    __host__ __device__ int row() const { return H * P8 + 2 * G * N8; }       // lanes of a convolved row: x heads, B groups, C groups
};

// The convolution's channel that lane `idx` of a convolved row holds, or -1 (a lane behind a head's or a group's own).
__device__ __forceinline__ int channel_of(const Sizes& z, int idx) {
    const int nx = z.H * z.P8;
    if (idx < nx) {
        const int h = idx / z.P8, p = idx % z.P8;
        return p < z.P ? h * z.P + p : -1;
    }
    const int g = (idx - nx) / z.N8, i = (idx - nx) % z.N8;     // the groups of B, then those of C
    return i < z.N ? z.inner() + g * z.N + i : -1;
}

// What the convolution of a channel reads `back` positions before the token at `t` (place `local` among its sequence's
// tokens of this step, position pos): this step's projections, the ring, or zero before the sequence's start.
__device__ __forceinline__ float conv_input(const float* __restrict__ proj, const Sizes& z, const float* ring, long t, int local,
                                            int pos, int back, int ch) {
    if (local >= back) return proj[(size_t)(t - back) * z.ld + z.inner() + ch];
    if (pos < back) return 0.0f;
    return ring[(size_t)((pos - back) % z.taps) * z.channels() + ch];
}

// The ring after a step, for one channel of one sequence (its last taps inputs that this step brought).
__device__ __forceinline__ void advance_ring(const float* __restrict__ proj, const Sizes& z, float* ring, int t0, int t1, int pos0, int ch) {
    for (int k = 0; k < min(z.taps, t1 - t0); ++k) {
        const int t = t1 - 1 - k, pos = pos0 + t - t0;
        ring[(size_t)(pos % z.taps) * z.channels() + ch] = proj[(size_t)t * z.ld + z.inner() + ch];
    }
}

// The channels that block (head h, columns col0 .. col0 + cols) looks after: its own x lanes, and (the group's first head,
// first columns) the group's B and C.
template <typename F>
__device__ __forceinline__ void own_channels(const Sizes& z, int h, int col0, int cols, bool first_cols, F f) {
    const int n_x = min(cols, z.P - col0);
    const int per = z.H / z.G;
    const int n_bc = (first_cols && h % per == 0) ? 2 * z.N : 0;
    for (int i = threadIdx.x; i < n_x + n_bc; i += blockDim.x) {
        int ch;
        if (i < n_x) ch = h * z.P + col0 + i;
        else {
            const int j = i - n_x;
            ch = z.inner() + (j < z.N ? 0 : z.G * z.N) + (h / per) * z.N + j % z.N;
        }
        f(ch);
    }
}

// ---------------------------------------------------------------------------
// Convolution, SiLU and step sizes of a prompt's tokens.  A thread owns one lane of the convolved row (or one head's step
// size) for kConvTokens tokens in order; with TAPS > 0 (known taps) the inputs it looks back at stay in registers.
// xc [n_tok, row()] in either element type; gd float [n_tok, 2 H]: la, then dt.
// ---------------------------------------------------------------------------
constexpr int kConvTokens = 16;

template <int TAPS>
__global__ void __launch_bounds__(256)
conv_kernel(const float* __restrict__ proj, const Sizes z, const void* __restrict__ conv_w, int w_dt,
            const void* __restrict__ conv_b, int b_dt, const float* __restrict__ state, const int* __restrict__ tok_seq,
            const int* __restrict__ tok_pos, const int* __restrict__ seq_slots, const int* __restrict__ cu_seqlens,
            const void* __restrict__ dt_bias, const void* __restrict__ a_log, int p_dt, void* __restrict__ xc, int xc_dt,
            float* __restrict__ gd, int n_tok) {
    const int idx = blockIdx.x * 256 + threadIdx.x, row = z.row();
    const int t_first = blockIdx.y * kConvTokens, t_end = min(n_tok, t_first + kConvTokens);
    if (idx >= row) {
        const int h = idx - row;
        if (h >= z.H) return;
        const float bias = ld_f(dt_bias, h, p_dt), rate = expf(ld_f(a_log, h, p_dt));
        const int col = z.inner() + z.channels() + h;
        for (int t = t_first; t < t_end; ++t) {
            const float dt = tok_seq[t] < 0 ? 0.0f : softplus_f(proj[(size_t)t * z.ld + col] + bias);
            gd[(size_t)t * 2 * z.H + h] = 0.0f - rate * dt;
            gd[(size_t)t * 2 * z.H + z.H + h] = dt;
        }
        return;
    }
    const int ch = channel_of(z, idx);
    if (ch < 0) {
        for (int t = t_first; t < t_end; ++t) st_f(xc, (size_t)t * row + idx, xc_dt, 0.0f);
        return;
    }
    const float bias = ld_f(conv_b, ch, b_dt);
    constexpr int kKept = TAPS > 0 ? TAPS : 1;
    float w[kKept], past[kKept];                // past[j]: the input j positions back (past[0] is the token's own)
    if (TAPS > 0) {
#pragma unroll
        for (int j = 0; j < kKept; ++j) {
            w[j] = ld_f(conv_w, (size_t)ch * z.taps + z.taps - 1 - j, w_dt);
            past[j] = 0.0f;
        }
    }
    for (int t = t_first; t < t_end; ++t) {
        const int seq = tok_seq[t];
        const int slot = seq < 0 ? -1 : seq_slots[seq];
        if (slot < 0) {
            st_f(xc, (size_t)t * row + idx, xc_dt, 0.0f);
            continue;
        }
        const int local = t - cu_seqlens[seq], pos = tok_pos[t];
        const float* ring = state + (size_t)slot * z.slot_stride + z.conv_at;
        float acc = bias;
        if (TAPS > 0) {
            if (t == t_first || local == 0) {
#pragma unroll
                for (int j = 1; j < kKept; ++j) past[j] = conv_input(proj, z, ring, t, local, pos, j, ch);
            } else {
#pragma unroll
                for (int j = kKept - 1; j > 0; --j) past[j] = past[j - 1];
            }
            past[0] = proj[(size_t)t * z.ld + z.inner() + ch];
#pragma unroll
            for (int j = kKept - 1; j >= 0; --j) acc = fmaf(w[j], past[j], acc);
        } else {
            for (int j = z.taps - 1; j >= 0; --j)
                acc = fmaf(ld_f(conv_w, (size_t)ch * z.taps + z.taps - 1 - j, w_dt), conv_input(proj, z, ring, t, local, pos, j, ch), acc);
        }
        st_f(xc, (size_t)t * row + idx, xc_dt, silu_f(acc));
    }
}

// ---------------------------------------------------------------------------
// The scan in 32-bit.  A block of four warps owns 16 columns of a head's state for one sequence, a warp four of them; a
// lane keeps the rows 32 ii + lane of its warp's columns in registers and walks the tokens in order.  Tokens are staged in
// groups of eight; a lane's partial sums of a group (4 columns x 8 tokens) are added over the warp by one butterfly that
// halves what a lane carries at every stage.  The order of operations of a (sequence, head, column) does not depend on how
// the sequence was cut into steps or on what else the step holds.
// ---------------------------------------------------------------------------
constexpr int kScanCols = 16, kScanGroup = 8;

template <int DR>
__global__ void __launch_bounds__(128)
scan_kernel(const float* __restrict__ proj, const Sizes z, const void* __restrict__ xc, int xc_dt, const float* __restrict__ gd,
            float* state, const int* __restrict__ seq_slots, const int* __restrict__ cu_seqlens, const int* __restrict__ tok_pos,
            const void* __restrict__ d_skip, int p_dt, float* __restrict__ y) {
    constexpr int NP = 32 * DR, TB = kScanGroup;
    extern __shared__ float scan_smem[];                     // B [TB][NP], C [TB][NP]
    __shared__ float xs[TB][kScanCols], las[TB], dts[TB];
    float* bs = scan_smem;
    float* cs = scan_smem + TB * NP;
    const int seq = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int col0 = blockIdx.z * kScanCols, j0 = warp * 4;
    const int t0 = cu_seqlens[seq], t1 = cu_seqlens[seq + 1], slot = seq_slots[seq];
    if (t0 >= t1) return;
    if (slot < 0) {
        for (int i = tid; i < (t1 - t0) * kScanCols; i += 128)
            if (col0 + i % kScanCols < z.P) y[(size_t)(t0 + i / kScanCols) * z.inner() + h * z.P + col0 + i % kScanCols] = 0.0f;
        return;
    }
    const int row = z.row(), g = h / (z.H / z.G);
    const size_t x_at = (size_t)h * z.P8 + col0, b_at = (size_t)z.H * z.P8 + (size_t)g * z.N8, c_at = b_at + (size_t)z.G * z.N8;
    float* s_head = state + (size_t)slot * z.slot_stride + (size_t)h * z.N * z.P;
    const float skip = ld_f(d_skip, h, p_dt);
    float S[DR][4];
#pragma unroll
    for (int ii = 0; ii < DR; ++ii)
#pragma unroll
        for (int c = 0; c < 4; ++c) {
            const int i = ii * 32 + lane, col = col0 + j0 + c;
            S[ii][c] = (i < z.N && col < z.P) ? s_head[(size_t)i * z.P + col] : 0.0f;
        }
    for (int g0 = t0; g0 < t1; g0 += TB) {
        const int nt = min(TB, t1 - g0);
        __syncthreads();
        for (int i = tid; i < TB * NP; i += 128) {
            const int tt = i / NP, n = i % NP;
            const bool in = tt < nt && n < z.N;
            bs[i] = in ? ld_f(xc, (size_t)(g0 + tt) * row + b_at + n, xc_dt) : 0.0f;
            cs[i] = in ? ld_f(xc, (size_t)(g0 + tt) * row + c_at + n, xc_dt) : 0.0f;
        }
        for (int i = tid; i < TB * kScanCols; i += 128) {
            const int tt = i / kScanCols, c = i % kScanCols;
            xs[tt][c] = (tt < nt && col0 + c < z.P) ? ld_f(xc, (size_t)(g0 + tt) * row + x_at + c, xc_dt) : 0.0f;
        }
        if (tid < TB) {
            las[tid] = tid < nt ? gd[(size_t)(g0 + tid) * 2 * z.H + h] : 0.0f;
            dts[tid] = tid < nt ? gd[(size_t)(g0 + tid) * 2 * z.H + z.H + h] : 0.0f;
        }
        __syncthreads();
        float part[4 * TB];
#pragma unroll
        for (int tt = 0; tt < TB; ++tt) {
            const float a = expf(las[tt]), dt = dts[tt];
            float u[4], acc[4];
#pragma unroll
            for (int c = 0; c < 4; ++c) {
                u[c] = dt * xs[tt][j0 + c];
                acc[c] = 0.0f;
            }
            if (tt < nt) {
#pragma unroll
                for (int ii = 0; ii < DR; ++ii) {
                    const float b = bs[tt * NP + ii * 32 + lane], cc = cs[tt * NP + ii * 32 + lane];
#pragma unroll
                    for (int c = 0; c < 4; ++c) {
                        S[ii][c] = fmaf(a, S[ii][c], b * u[c]);
                        acc[c] = fmaf(S[ii][c], cc, acc[c]);
                    }
                }
            }
#pragma unroll
            for (int c = 0; c < 4; ++c) part[4 * tt + c] = acc[c];
        }
#pragma unroll
        for (int m = 16; m >= 1; m >>= 1) {
            const bool up = lane & m;
#pragma unroll
            for (int k = 0; k < m; ++k) {
                const float got = __shfl_xor_sync(0xffffffffu, up ? part[k] : part[k + m], m);
                part[k] = (up ? part[k + m] : part[k]) + got;
            }
        }
        const int tt = lane >> 2, c = lane & 3;               // the sum that this lane ended up with
        if (tt < nt && col0 + j0 + c < z.P)
            y[(size_t)(g0 + tt) * z.inner() + h * z.P + col0 + j0 + c] = fmaf(skip, xs[tt][j0 + c], part[0]);
    }
#pragma unroll
    for (int ii = 0; ii < DR; ++ii)
#pragma unroll
        for (int c = 0; c < 4; ++c) {
            const int i = ii * 32 + lane, col = col0 + j0 + c;
            if (i < z.N && col < z.P) s_head[(size_t)i * z.P + col] = S[ii][c];
        }
    float* ring = state + (size_t)slot * z.slot_stride + z.conv_at;
    const int pos0 = tok_pos[t0];
    own_channels(z, h, col0, kScanCols, blockIdx.z == 0, [&](int ch) { advance_ring(proj, z, ring, t0, t1, pos0, ch); });
}

// ---------------------------------------------------------------------------
// A decode step: one token per sequence, everything from the projections to y in one launch.  A block owns kStepCols
// columns of one (token, head); its threads are groups of VEC neighbouring columns times row groups, so the state is read
// and written at full width with all of a thread's rows in flight.  The convolutions of the head's x and of its group's B
// and C are made by every block that needs them (from the ring and the token's projections); the group's first head writes
// their ring place.
// ---------------------------------------------------------------------------
constexpr int kStepCols = 64, kStepThreads = 256;

template <int VEC>
__global__ void __launch_bounds__(kStepThreads)
step_kernel(const float* __restrict__ proj, const Sizes z, const void* __restrict__ conv_w, int w_dt,
            const void* __restrict__ conv_b, int b_dt, float* state, const int* __restrict__ tok_pos,
            const int* __restrict__ seq_slots, const void* __restrict__ dt_bias, const void* __restrict__ a_log,
            const void* __restrict__ d_skip, int p_dt, float* __restrict__ y) {
    constexpr int kGroups = kStepCols / VEC, kRows = kStepThreads / kGroups;      // column groups, row groups
    extern __shared__ float step_smem[];                          // B [N], C [N]
    __shared__ float xs[kStepCols], red[kRows][kStepCols + 1];
    float* bs = step_smem;
    float* cs = step_smem + z.N;
    const int t = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * kStepCols, tid = threadIdx.x;
    const int slot = seq_slots[t];
    const int cols = min(kStepCols, z.P - col0);
    float* out = y + (size_t)t * z.inner() + (size_t)h * z.P + col0;
    if (slot < 0) {
        for (int i = tid; i < cols; i += kStepThreads) out[i] = 0.0f;
        return;
    }
    const int per = z.H / z.G, g = h / per, pos = tok_pos[t], C = z.channels();
    float* s_head = state + (size_t)slot * z.slot_stride + (size_t)h * z.N * z.P + col0;
    float* ring = state + (size_t)slot * z.slot_stride + z.conv_at;
    const float* own = proj + (size_t)t * z.ld + z.inner();
    // the rows of the state do not wait for anything: the first ones are asked for before the convolutions
    const int cg = tid % kGroups, rg = tid / kGroups;
    const bool col_in = cg * VEC < cols;
    constexpr int kAhead = 8;
    float ahead[kAhead][VEC];
#pragma unroll
    for (int u = 0; u < kAhead; ++u) {
        const int i = rg + u * kRows;
        if (col_in && i < z.N) {
            if (VEC == 4) {
                const float4 v = *reinterpret_cast<const float4*>(s_head + (size_t)i * z.P + cg * VEC);
                ahead[u][0] = v.x; ahead[u][1 % VEC] = v.y; ahead[u][2 % VEC] = v.z; ahead[u][3 % VEC] = v.w;
            } else {
                ahead[u][0] = s_head[(size_t)i * z.P + cg];
            }
        }
    }
    const bool owns_bc = blockIdx.z == 0 && h % per == 0;
    for (int i = tid; i < cols + 2 * z.N; i += kStepThreads) {
        const int j = i - cols;
        const int ch = i < cols ? h * z.P + col0 + i : z.inner() + (j < z.N ? 0 : z.G * z.N) + g * z.N + j % z.N;
        float acc = ld_f(conv_b, ch, b_dt);
        for (int back = z.taps - 1; back > 0; --back)
            if (pos >= back)
                acc = fmaf(ld_f(conv_w, (size_t)ch * z.taps + z.taps - 1 - back, w_dt), ring[(size_t)((pos - back) % z.taps) * C + ch], acc);
        const float now = own[ch];
        acc = fmaf(ld_f(conv_w, (size_t)ch * z.taps + z.taps - 1, w_dt), now, acc);
        const float v = silu_f(acc);
        if (i < cols) xs[i] = v;
        else step_smem[j] = v;
        if (i < cols || owns_bc) ring[(size_t)(pos % z.taps) * C + ch] = now;
    }
    const float dt = softplus_f(proj[(size_t)t * z.ld + z.inner() + C + h] + ld_f(dt_bias, h, p_dt));
    const float a = expf(0.0f - expf(ld_f(a_log, h, p_dt)) * dt);
    __syncthreads();
    float acc[VEC];
#pragma unroll
    for (int c = 0; c < VEC; ++c) acc[c] = 0.0f;
    if (col_in) {
        float u[VEC];
#pragma unroll
        for (int c = 0; c < VEC; ++c) u[c] = dt * xs[cg * VEC + c];
        auto one_row = [&](int i, float (&s)[VEC]) {
            const float b = bs[i], cc = cs[i];
#pragma unroll
            for (int c = 0; c < VEC; ++c) {
                s[c] = fmaf(a, s[c], b * u[c]);
                acc[c] = fmaf(s[c], cc, acc[c]);
            }
            if (VEC == 4)
                *reinterpret_cast<float4*>(s_head + (size_t)i * z.P + cg * VEC) = make_float4(s[0], s[1 % VEC], s[2 % VEC], s[3 % VEC]);
            else
                s_head[(size_t)i * z.P + cg] = s[0];
        };
#pragma unroll
        for (int k = 0; k < kAhead; ++k)
            if (rg + k * kRows < z.N) one_row(rg + k * kRows, ahead[k]);
        for (int i = rg + kAhead * kRows; i < z.N; i += kRows) {
            float s[VEC];
            if (VEC == 4) {
                const float4 v = *reinterpret_cast<const float4*>(s_head + (size_t)i * z.P + cg * VEC);
                s[0] = v.x; s[1 % VEC] = v.y; s[2 % VEC] = v.z; s[3 % VEC] = v.w;
            } else {
                s[0] = s_head[(size_t)i * z.P + cg];
            }
            one_row(i, s);
        }
    }
#pragma unroll
    for (int c = 0; c < VEC; ++c) red[rg][cg * VEC + c] = acc[c];
    __syncthreads();
    if (tid < cols) {
        float sum = 0.0f;
        for (int r = 0; r < kRows; ++r) sum += red[r][tid];
        out[tid] = fmaf(ld_f(d_skip, h, p_dt), xs[tid], sum);
    }
}

// ---------------------------------------------------------------------------
// Gate and norm: u = y silu(z); every one of n_groups equal parts of a token's u over its own root mean square, times the
// weight.  A block per (token, part); a part of up to kGateVec * blockDim lanes stays in registers between the two passes.
// ---------------------------------------------------------------------------
constexpr int kGateVec = 16;

__global__ void __launch_bounds__(256)
gated_norm_kernel(const float* __restrict__ y, const float* __restrict__ proj, int ld, const void* __restrict__ w, int w_dt,
                  float eps, void* __restrict__ out, int out_dt, int inner, int part) {
    __shared__ float scratch[33];
    const int t = blockIdx.x, g0 = blockIdx.y * part;
    const float* ys = y + (size_t)t * inner + g0;
    const float* zs = proj + (size_t)t * ld + g0;
    float v[kGateVec];
    float ss = 0.0f;
#pragma unroll
    for (int j = 0; j < kGateVec; ++j) {
        const int i = threadIdx.x + j * blockDim.x;
        v[j] = i < part ? ys[i] * silu_f(zs[i]) : 0.0f;
        ss = fmaf(v[j], v[j], ss);
    }
    for (int i = threadIdx.x + kGateVec * blockDim.x; i < part; i += blockDim.x) {
        const float u = ys[i] * silu_f(zs[i]);
        ss = fmaf(u, u, ss);
    }
    ss = block_sum(ss, scratch);
    const float scale = 1.0f / sqrtf(ss * (1.0f / (float)part) + eps);
#pragma unroll
    for (int j = 0; j < kGateVec; ++j) {
        const int i = threadIdx.x + j * blockDim.x;
        if (i < part) st_f(out, (size_t)t * inner + g0 + i, out_dt, (v[j] * scale) * ld_f(w, g0 + i, w_dt));
    }
    for (int i = threadIdx.x + kGateVec * blockDim.x; i < part; i += blockDim.x)
        st_f(out, (size_t)t * inner + g0 + i, out_dt, ((ys[i] * silu_f(zs[i])) * scale) * ld_f(w, g0 + i, w_dt));
}

int make_sizes(Sizes* z, int H, int P, int G, int N, int taps, int ld, long slot_stride) {
    NN_CHECK(H > 0 && P > 0 && G > 0 && H % G == 0 && N > 0, "state space: %d heads over %d groups, states of %d x %d", H, G, N, P);
    NN_CHECK(taps >= 1 && taps <= kMaxTaps, "state space: convolutions of %d taps (1 to %d)", taps, kMaxTaps);
    z->H = H; z->P = P; z->G = G; z->N = N; z->taps = taps; z->ld = ld;
    z->P8 = (P + 7) / 8 * 8;
    z->N8 = (N + 7) / 8 * 8;
    z->slot_stride = slot_stride;
    z->conv_at = ((long)H * N * P + 3) / 4 * 4;
    NN_CHECK(ld >= 2 * z->inner() + 2 * G * N + H, "state space: rows of %d floats", ld);
    NN_CHECK(slot_stride >= z->conv_at + (long)taps * z->channels(), "state space: state rows of %ld floats", slot_stride);
    NN_CHECK(H <= 65535 && P <= 65535 * 16, "state space: grid");
    return 0;
}

}  // namespace

// Floats a state row needs, and lanes a convolved row has.
extern "C" long nncpu_ssm_state_floats(int H, int P, int G, int N, int taps) {
    return (((long)H * N * P + 3) / 4 * 4 + (long)taps * ((long)H * P + 2l * G * N) + 3) / 4 * 4;
}
extern "C" int nncpu_ssm_row(int H, int P, int G, int N) { return H * ((P + 7) / 8 * 8) + 2 * G * ((N + 7) / 8 * 8); }

extern "C" int nncpu_ssm_conv(const float* proj, int ld, const void* conv_w, int w_dt, const void* conv_b, int b_dt,
                              const float* state, long slot_stride, const int* tok_seq, const int* tok_pos,
                              const int* seq_slots, const int* cu_seqlens, const void* dt_bias, const void* a_log, int p_dt,
                              void* xc, int xc_dt, float* gd, int n_tok, int H, int P, int G, int N, int taps, void* stream) {
    Sizes z;
    if (int e = make_sizes(&z, H, P, G, N, taps, ld, slot_stride)) return e;
    if (n_tok <= 0) return 0;
    const dim3 grid((z.row() + H + 255) / 256, (n_tok + kConvTokens - 1) / kConvTokens);
    NN_CHECK(grid.y <= 65535, "state space: %d tokens in a step", n_tok);
#define NN_CONV(T)                                                                                                         \
    conv_kernel<T><<<grid, 256, 0, (cudaStream_t)stream>>>(proj, z, conv_w, w_dt, conv_b, b_dt, state, tok_seq, tok_pos,    \
                                                           seq_slots, cu_seqlens, dt_bias, a_log, p_dt, xc, xc_dt, gd, n_tok)
    if (taps == 4) NN_CONV(4);
    else if (taps == 3) NN_CONV(3);
    else if (taps == 2) NN_CONV(2);
    else NN_CONV(0);
#undef NN_CONV
    NN_LAUNCH_OK("state space (convolution)");
    return 0;
}

extern "C" int nncpu_ssm_scan(const float* proj, int ld, const void* xc, int xc_dt, const float* gd, float* state,
                              long slot_stride, const int* seq_slots, const int* cu_seqlens, const int* tok_pos,
                              const void* d_skip, int p_dt, float* y, int n_seqs, int H, int P, int G, int N, int taps,
                              void* stream) {
    Sizes z;
    if (int e = make_sizes(&z, H, P, G, N, taps, ld, slot_stride)) return e;
    NN_CHECK(N <= 512, "state space: states of %d rows (at most 512)", N);
    if (n_seqs <= 0) return 0;
    const dim3 grid(n_seqs, H, (P + kScanCols - 1) / kScanCols);
#define NN_SCAN(DR)                                                                                                        \
    scan_kernel<DR><<<grid, 128, (size_t)2 * kScanGroup * 32 * DR * 4, (cudaStream_t)stream>>>(                             \
        proj, z, xc, xc_dt, gd, state, seq_slots, cu_seqlens, tok_pos, d_skip, p_dt, y)
    if (N <= 32) NN_SCAN(1);
    else if (N <= 64) NN_SCAN(2);
    else if (N <= 128) NN_SCAN(4);
    else if (N <= 256) NN_SCAN(8);
    else NN_SCAN(16);
#undef NN_SCAN
    NN_LAUNCH_OK("state space (scan)");
    return 0;
}

extern "C" int nncpu_ssm_step(const float* proj, int ld, const void* conv_w, int w_dt, const void* conv_b, int b_dt, float* state,
                              long slot_stride, const int* tok_pos, const int* seq_slots, const void* dt_bias,
                              const void* a_log, const void* d_skip, int p_dt, float* y, int n_tok, int H, int P, int G, int N,
                              int taps, void* stream) {
    Sizes z;
    if (int e = make_sizes(&z, H, P, G, N, taps, ld, slot_stride)) return e;
    NN_CHECK(N <= 4096, "state space: states of %d rows (at most 4096)", N);
    if (n_tok <= 0) return 0;
    const dim3 grid(n_tok, H, (P + kStepCols - 1) / kStepCols);
    const size_t smem = (size_t)2 * N * sizeof(float);
    const bool vec = P % 4 == 0 && slot_stride % 4 == 0 && (uintptr_t)state % 16 == 0;
    if (vec)
        step_kernel<4><<<grid, kStepThreads, smem, (cudaStream_t)stream>>>(proj, z, conv_w, w_dt, conv_b, b_dt, state, tok_pos,
                                                                           seq_slots, dt_bias, a_log, d_skip, p_dt, y);
    else
        step_kernel<1><<<grid, kStepThreads, smem, (cudaStream_t)stream>>>(proj, z, conv_w, w_dt, conv_b, b_dt, state, tok_pos,
                                                                           seq_slots, dt_bias, a_log, d_skip, p_dt, y);
    NN_LAUNCH_OK("state space (step)");
    return 0;
}

extern "C" int nncpu_ssm_gated_norm(const float* y, const float* proj, int ld, const void* w, int w_dt, float eps, void* out,
                                    int out_dt, int n_tok, int inner, int n_groups, void* stream) {
    NN_CHECK(n_tok >= 0 && inner > 0 && n_groups > 0 && inner % n_groups == 0 && ld >= inner,
             "gated norm: %d lanes in %d parts", inner, n_groups);
    if (n_tok == 0) return 0;
    const int part = inner / n_groups;
    NN_CHECK(n_groups <= 65535, "gated norm: %d parts", n_groups);
    const int threads = part >= 256 ? 256 : (part + 31) / 32 * 32;
    gated_norm_kernel<<<dim3(n_tok, n_groups), threads, 0, (cudaStream_t)stream>>>(y, proj, ld, w, w_dt, eps, out, out_dt, inner, part);
    NN_LAUNCH_OK("gated norm");
    return 0;
}
