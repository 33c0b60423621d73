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
        // a whole tile of one sequence (a prompt's usual case): all of the tile's inputs are asked for before the first is used
        const int seq = tok_seq[t_first];
        const int slot = seq < 0 ? -1 : seq_slots[seq];
        if (t_end - t_first == kConvTokens && slot >= 0 && tok_seq[t_end - 1] == seq) {
            const int local = t_first - cu_seqlens[seq], pos = tok_pos[t_first];
            const float* ring = state + (size_t)slot * z.slot_stride + z.conv_at;
            float in[kConvTokens + kKept - 1];           // in[k]: the input of the tile's token k - (taps - 1)
#pragma unroll
            for (int k = 0; k < kConvTokens; ++k) in[k + kKept - 1] = proj[(size_t)(t_first + k) * z.ld + z.inner() + ch];
#pragma unroll
            for (int j = 1; j < kKept; ++j) in[kKept - 1 - j] = conv_input(proj, z, ring, t_first, local, pos, j, ch);
#pragma unroll
            for (int k = 0; k < kConvTokens; ++k) {
                float acc = bias;
#pragma unroll
                for (int j = kKept - 1; j >= 0; --j) acc = fmaf(w[j], in[k + kKept - 1 - j], acc);
                st_f(xc, (size_t)(t_first + k) * row + idx, xc_dt, silu_f(acc));
            }
            return;
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
// Prompts of a bfloat16 run: the recurrence over chunks of 64 tokens, as products on the tensor cores (mma.sync).  With
// cum_i the sum of la over the chunk's tokens up to i, S the state before the chunk and a = exp(cum_last):
//     y_i   = sum over j <= i of (C_i . B_j) exp(cum_i - cum_j) dt_j x_j   +   exp(cum_i) S^T C_i   +   D x_i
//     S_new = a S + sum over j of B_j (exp(cum_last - cum_j) dt_j x_j)^T
// x, B and C are bfloat16 as the convolutions left them.  What is 32-bit by design stays so: the state lives in 32-bit
// registers, decays and step sizes are 32-bit, and wherever one of them becomes an operand of a product (the masked
// weights, the scaled x, the state that is read out) it goes in as the sum of two bfloat16 numbers, value and remainder,
// so that a factor keeps 16 bits of mantissa and the products add up in 32-bit.
//
// A block of four warps owns 32 columns of one head's state for one sequence and walks its chunks in order: warp w has the
// chunk's tokens 16 w .. 16 w + 15 as rows of y and a quarter of the state's rows in registers.  B, C and x of the next
// chunk are copied to shared memory (cp.async, two buffers) under this chunk's arithmetic; the state goes through shared
// memory once a chunk, so that every warp can read all of it.  What a token gets does not depend on other sequences;
// where a sequence is cut moves the chunks' borders, which changes rounding only.
// ---------------------------------------------------------------------------
constexpr int kChunk = 64, kChunkCols = 32;

__device__ __forceinline__ uint32_t smem_addr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
// 16 bytes, or zeros where there is nothing to copy
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src, bool in) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(in ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void ldmatrix_x4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldmatrix_x4_trans(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile(
        "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
        : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// Two numbers as bfloat16 pairs: the values, and what rounding them left.
__device__ __forceinline__ void split_pair(float a, float b, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
    const float2 f = __bfloat1622float2(h);
    const __nv_bfloat162 l = __floats2bfloat162_rn(a - f.x, b - f.y);
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = *reinterpret_cast<const uint32_t*>(&l);
}

// Byte offsets of 16-byte pieces in tiles whose rows hold NP (a multiple of 64) or 32 bfloat16, exchanged by the row number
// so that 8 rows' equal pieces lie in 8 bank groups.
template <int NP>
__device__ __forceinline__ uint32_t wide_off(int row, int piece) {
    return (uint32_t)(row * (NP * 2) + (((piece & ~7) | ((piece ^ row) & 7)) << 4));
}
__device__ __forceinline__ uint32_t narrow_off(int row, int piece) { return (uint32_t)(row * 64 + ((piece ^ ((row >> 1) & 3)) << 4)); }

template <int NP>
constexpr int chunk_smem() { return 4 * kChunk * NP * 2 + 4 * kChunk * 64 + 2 * NP * 64; }

template <int NP>
__global__ void __launch_bounds__(128)
chunk_kernel(const float* __restrict__ proj, const Sizes z, const __nv_bfloat16* __restrict__ xc, const float* __restrict__ gd,
             float* state, const int* __restrict__ seq_slots, const int* __restrict__ cu_seqlens, const int* __restrict__ tok_pos,
             const void* __restrict__ d_skip, int p_dt, float* __restrict__ y) {
    constexpr int kWide = kChunk * NP * 2, kNarrow = kChunk * 64;      // bytes of a tile of B or C, of x
    constexpr int MT = NP / 64;                                        // 16-row tiles of the state a warp holds
    extern __shared__ __align__(128) uint8_t chunk_smem_[];
    __shared__ float2 cum_dt[kChunk];
    const uint32_t base = smem_addr(chunk_smem_);
    const uint32_t b_tile = base, c_tile = base + 2 * kWide, x_tile = base + 4 * kWide;      // two buffers each
    const uint32_t xh_tile = x_tile + 2 * kNarrow, xl_tile = xh_tile + kNarrow;              // the scaled x, value and remainder
    const uint32_t sh_tile = xl_tile + kNarrow, sl_tile = sh_tile + NP * 64;                 // the state, value and remainder
    const int seq = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * kChunkCols;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, c = lane & 3, r = lane >> 2;
    const int t0 = cu_seqlens[seq], t1 = cu_seqlens[seq + 1], slot = seq_slots[seq];
    if (t0 >= t1) return;
    const int inner = z.inner();
    float* y_head = y + (size_t)h * z.P + col0;
    if (slot < 0) {
        for (int i = tid; i < (t1 - t0) * kChunkCols; i += 128)
            if (col0 + i % kChunkCols < z.P) y_head[(size_t)(t0 + i / kChunkCols) * inner + i % kChunkCols] = 0.0f;
        return;
    }
    const int row = z.row(), g = h / (z.H / z.G);
    const size_t x_at = (size_t)h * z.P8 + col0, b_at = (size_t)z.H * z.P8 + (size_t)g * z.N8, c_at = b_at + (size_t)z.G * z.N8;
    float* s_head = state + (size_t)slot * z.slot_stride + (size_t)h * z.N * z.P + col0;
    const float skip = ld_f(d_skip, h, p_dt);
    const int cols = min(kChunkCols, z.P - col0);

    auto stage = [&](int g0, int buf) {
        const int nt = t1 - g0;                                        // (may be more than a chunk, or none)
        for (int i = tid; i < kChunk * (NP / 8); i += 128) {
            const int tt = i / (NP / 8), piece = i % (NP / 8);
            const bool in = tt < nt && piece * 8 < z.N8;
            const __nv_bfloat16* src = xc + (in ? (size_t)(g0 + tt) * row + piece * 8 : 0);
            cp_async16(b_tile + buf * kWide + wide_off<NP>(tt, piece), in ? src + b_at : xc, in);
            cp_async16(c_tile + buf * kWide + wide_off<NP>(tt, piece), in ? src + c_at : xc, in);
        }
        for (int i = tid; i < kChunk * 4; i += 128) {
            const int tt = i >> 2, piece = i & 3;
            const bool in = tt < nt && col0 + piece * 8 < z.P8;
            cp_async16(x_tile + buf * kNarrow + narrow_off(tt, piece), in ? xc + (size_t)(g0 + tt) * row + x_at + piece * 8 : xc, in);
        }
    };
    stage(t0, 0);
    cp_async_commit();
    stage(t0 + kChunk, 1);
    cp_async_commit();

    // this warp's rows of the state: m0 + 16 mt + r (and + 8), columns 8 nt + 2 c (and + 1)
    const int m0 = warp * (NP / 4);
    float S[MT][4][4];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int nt = 0; nt < 4; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int i = m0 + 16 * mt + r + 8 * (e >> 1), col = 8 * nt + 2 * c + (e & 1);
                S[mt][nt][e] = (i < z.N && col < cols) ? s_head[(size_t)i * z.P + col] : 0.0f;
            }
    auto publish = [&]() {
#pragma unroll
        for (int mt = 0; mt < MT; ++mt)
#pragma unroll
            for (int nt = 0; nt < 4; ++nt)
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    uint32_t hi, lo;
                    split_pair(S[mt][nt][2 * half], S[mt][nt][2 * half + 1], hi, lo);
                    const uint32_t at = narrow_off(m0 + 16 * mt + r + 8 * half, nt) + 4 * c;
                    asm volatile("st.shared.b32 [%0], %1;" ::"r"(sh_tile + at), "r"(hi) : "memory");
                    asm volatile("st.shared.b32 [%0], %1;" ::"r"(sl_tile + at), "r"(lo) : "memory");
                }
    };
    publish();

    // la and dt of the tokens 2 lane and 2 lane + 1 of a chunk, fetched one chunk ahead
    float la0, la1, dt0, dt1;
    auto fetch = [&](int g0) {
        const float* p = gd + (size_t)(g0 + 2 * lane) * 2 * z.H + h;
        const bool in0 = g0 + 2 * lane < t1, in1 = g0 + 2 * lane + 1 < t1;
        la0 = in0 ? p[0] : 0.0f;
        dt0 = in0 ? p[z.H] : 0.0f;
        la1 = in1 ? p[2 * z.H] : 0.0f;
        dt1 = in1 ? p[3 * z.H] : 0.0f;
    };
    fetch(t0);
    int buf = 0;
    for (int g0 = t0; g0 < t1; g0 += kChunk, buf ^= 1) {
        // sums of la up to every token (tokens beyond the sequence's end add nothing)
        float cum1 = la0 + la1;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float got = __shfl_up_sync(0xffffffffu, cum1, o);
            if (lane >= o) cum1 += got;
        }
        float before = __shfl_up_sync(0xffffffffu, cum1, 1);
        if (lane == 0) before = 0.0f;
        const float cum0 = before + la0;
        const float cum_last = __shfl_sync(0xffffffffu, cum1, 31);
        const float dt_0 = dt0, dt_1 = dt1;
        if (g0 + kChunk < t1) fetch(g0 + kChunk);
        cp_async_wait<1>();                      // this chunk's tiles have landed (the next one's may still fly)
        __syncthreads();                         // everybody's have; the state of the chunk before is published
        if (warp == 0) {
            cum_dt[2 * lane] = make_float2(cum0, dt_0);
            cum_dt[2 * lane + 1] = make_float2(cum1, dt_1);
        }
        {   // x scaled by what is left of a token at the chunk's end: a thread has half of one token's columns
            const int src = 8 * warp + (lane >> 2);
            const bool odd = (lane >> 1) & 1;
            const float cu = __shfl_sync(0xffffffffu, cum0, src), cv = __shfl_sync(0xffffffffu, cum1, src);
            const float du = __shfl_sync(0xffffffffu, dt_0, src), dv = __shfl_sync(0xffffffffu, dt_1, src);
            const float scale = expf(cum_last - (odd ? cv : cu)) * (odd ? dv : du);
            const int tt = tid >> 1;
#pragma unroll
            for (int k = 0; k < 2; ++k) {
                const uint32_t at = narrow_off(tt, 2 * (tid & 1) + k);
                uint32_t v[4], hi[4], lo[4];
                asm volatile("ld.shared.v4.b32 {%0, %1, %2, %3}, [%4];"
                             : "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3]) : "r"(x_tile + buf * kNarrow + at));
#pragma unroll
                for (int q = 0; q < 4; ++q) {
                    const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v[q]));
                    split_pair(f.x * scale, f.y * scale, hi[q], lo[q]);
                }
                asm volatile("st.shared.v4.b32 [%0], {%1, %2, %3, %4};" ::"r"(xh_tile + at), "r"(hi[0]), "r"(hi[1]), "r"(hi[2]), "r"(hi[3]) : "memory");
                asm volatile("st.shared.v4.b32 [%0], {%1, %2, %3, %4};" ::"r"(xl_tile + at), "r"(lo[0]), "r"(lo[1]), "r"(lo[2]), "r"(lo[3]) : "memory");
            }
        }
        __syncthreads();
        // C . B^T (token pairs of this warp's rows, only up to the diagonal) and C . S
        float s[8][4], acc[4][4];
#pragma unroll
        for (int t = 0; t < 8; ++t) s[t][0] = s[t][1] = s[t][2] = s[t][3] = 0.0f;
#pragma unroll
        for (int t = 0; t < 4; ++t) acc[t][0] = acc[t][1] = acc[t][2] = acc[t][3] = 0.0f;
        const uint32_t bt = b_tile + buf * kWide, ct = c_tile + buf * kWide, xt = x_tile + buf * kNarrow;
#pragma unroll 2
        for (int ks = 0; ks < NP / 16; ++ks) {
            if (ks * 16 >= z.N) break;
            uint32_t a[4], b[4];
            ldmatrix_x4(a, ct + wide_off<NP>(16 * warp + ((lane >> 3) & 1) * 8 + (lane & 7), ks * 2 + (lane >> 4)));
#pragma unroll
            for (int tp = 0; tp < 4; ++tp) {
                if (tp <= warp) {
                    ldmatrix_x4(b, bt + wide_off<NP>(tp * 16 + (lane >> 4) * 8 + (lane & 7), ks * 2 + ((lane >> 3) & 1)));
                    mma_bf16(s[2 * tp], a, b[0], b[1]);
                    mma_bf16(s[2 * tp + 1], a, b[2], b[3]);
                }
            }
            const int k_row = ks * 16 + ((lane >> 3) & 1) * 8 + (lane & 7);
#pragma unroll
            for (int dp = 0; dp < 2; ++dp) {
                const uint32_t at = narrow_off(k_row, dp * 2 + (lane >> 4));
                ldmatrix_x4_trans(b, sh_tile + at);
                mma_bf16(acc[2 * dp], a, b[0], b[1]);
                mma_bf16(acc[2 * dp + 1], a, b[2], b[3]);
                ldmatrix_x4_trans(b, sl_tile + at);
                mma_bf16(acc[2 * dp], a, b[0], b[1]);
                mma_bf16(acc[2 * dp + 1], a, b[2], b[3]);
            }
        }
        const int i_lo = 16 * warp + r, i_hi = i_lo + 8;
        const float cum_lo = cum_dt[i_lo].x, cum_hi = cum_dt[i_hi].x;
        const float e_lo = expf(cum_lo), e_hi = expf(cum_hi);
#pragma unroll
        for (int t = 0; t < 4; ++t) {
            acc[t][0] *= e_lo; acc[t][1] *= e_lo; acc[t][2] *= e_hi; acc[t][3] *= e_hi;
        }
        // the weights of the chunk's own tokens, and their sum of x
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {
            if (kk <= warp) {
                uint32_t hi[4], lo[4];
#pragma unroll
                for (int half = 0; half < 2; ++half) {
                    const int t = 2 * kk + half, j = t * 8 + 2 * c;
                    const float4 cd = *reinterpret_cast<const float4*>(&cum_dt[j]);      // (cum, dt) of the tokens j and j + 1
                    const float w0 = j <= i_lo ? s[t][0] * (expf(cum_lo - cd.x) * cd.y) : 0.0f;
                    const float w1 = j + 1 <= i_lo ? s[t][1] * (expf(cum_lo - cd.z) * cd.w) : 0.0f;
                    const float w2 = j <= i_hi ? s[t][2] * (expf(cum_hi - cd.x) * cd.y) : 0.0f;
                    const float w3 = j + 1 <= i_hi ? s[t][3] * (expf(cum_hi - cd.z) * cd.w) : 0.0f;
                    split_pair(w0, w1, hi[2 * half], lo[2 * half]);
                    split_pair(w2, w3, hi[2 * half + 1], lo[2 * half + 1]);
                }
#pragma unroll
                for (int dp = 0; dp < 2; ++dp) {
                    uint32_t b[4];
                    ldmatrix_x4_trans(b, xt + narrow_off(kk * 16 + ((lane >> 3) & 1) * 8 + (lane & 7), dp * 2 + (lane >> 4)));
                    mma_bf16(acc[2 * dp], hi, b[0], b[1]);
                    mma_bf16(acc[2 * dp + 1], hi, b[2], b[3]);
                    mma_bf16(acc[2 * dp], lo, b[0], b[1]);
                    mma_bf16(acc[2 * dp + 1], lo, b[2], b[3]);
                }
            }
        }
        // y, with the token's own x
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int i = half ? i_hi : i_lo;
            if (g0 + i >= t1) continue;
            float* dst = y_head + (size_t)(g0 + i) * inner;
#pragma unroll
            for (int t = 0; t < 4; ++t) {
                const int col = 8 * t + 2 * c;
                uint32_t v;
                asm volatile("ld.shared.b32 %0, [%1];" : "=r"(v) : "r"(xt + narrow_off(i, t) + 4 * c));
                const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v));
                const float o0 = fmaf(skip, f.x, acc[t][2 * half]), o1 = fmaf(skip, f.y, acc[t][2 * half + 1]);
                if (col + 1 < cols && (z.P & 1) == 0) *reinterpret_cast<float2*>(dst + col) = make_float2(o0, o1);
                else {
                    if (col < cols) dst[col] = o0;
                    if (col + 1 < cols) dst[col + 1] = o1;
                }
            }
        }
        // the state after the chunk
        const float a_all = expf(cum_last);
#pragma unroll
        for (int mt = 0; mt < MT; ++mt)
#pragma unroll
            for (int t = 0; t < 4; ++t)
#pragma unroll
                for (int e = 0; e < 4; ++e) S[mt][t][e] *= a_all;
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {
            uint32_t bh[2][4], bl[2][4];
#pragma unroll
            for (int dp = 0; dp < 2; ++dp) {
                const uint32_t at = narrow_off(kk * 16 + ((lane >> 3) & 1) * 8 + (lane & 7), dp * 2 + (lane >> 4));
                ldmatrix_x4_trans(bh[dp], xh_tile + at);
                ldmatrix_x4_trans(bl[dp], xl_tile + at);
            }
#pragma unroll
            for (int mt = 0; mt < MT; ++mt) {
                uint32_t a[4];
                ldmatrix_x4_trans(a, bt + wide_off<NP>(kk * 16 + (lane >> 4) * 8 + (lane & 7), (m0 + 16 * mt) / 8 + ((lane >> 3) & 1)));
#pragma unroll
                for (int dp = 0; dp < 2; ++dp) {
                    mma_bf16(S[mt][2 * dp], a, bh[dp][0], bh[dp][1]);
                    mma_bf16(S[mt][2 * dp + 1], a, bh[dp][2], bh[dp][3]);
                    mma_bf16(S[mt][2 * dp], a, bl[dp][0], bl[dp][1]);
                    mma_bf16(S[mt][2 * dp + 1], a, bl[dp][2], bl[dp][3]);
                }
            }
        }
        __syncthreads();                         // the old state and this chunk's tiles are done with
        publish();
        if (g0 + 2 * kChunk < t1) stage(g0 + 2 * kChunk, buf);
        cp_async_commit();
    }
    cp_async_wait<0>();
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int nt = 0; nt < 4; ++nt)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int i = m0 + 16 * mt + r + 8 * (e >> 1), col = 8 * nt + 2 * c + (e & 1);
                if (i < z.N && col < cols) s_head[(size_t)i * z.P + col] = S[mt][nt][e];
            }
    float* ring = state + (size_t)slot * z.slot_stride + z.conv_at;
    const int pos0 = tok_pos[t0];
    own_channels(z, h, col0, kChunkCols, blockIdx.z == 0, [&](int ch) { advance_ring(proj, z, ring, t0, t1, pos0, ch); });
}

template <int NP>
int launch_chunk(const float* proj, const Sizes& z, const void* xc, const float* gd, float* state, const int* seq_slots,
                 const int* cu_seqlens, const int* tok_pos, const void* d_skip, int p_dt, float* y, int n_seqs, cudaStream_t st) {
    static bool configured[64] = {};
    if (first_use_on_this_device(configured)) {
        const cudaError_t e = cudaFuncSetAttribute(chunk_kernel<NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, chunk_smem<NP>());
        NN_CHECK(e == cudaSuccess, "state space (chunks): cannot reserve shared memory: %s", cudaGetErrorString(e));
    }
    const dim3 grid(n_seqs, z.H, (z.P + kChunkCols - 1) / kChunkCols);
    chunk_kernel<NP><<<grid, 128, chunk_smem<NP>(), st>>>(proj, z, (const __nv_bfloat16*)xc, gd, state, seq_slots, cu_seqlens, tok_pos,
                                                          d_skip, p_dt, y);
    NN_LAUNCH_OK("state space (chunks)");
    return 0;
}

// ---------------------------------------------------------------------------
// A decode step: one token per sequence, everything from the projections to y in one launch.  A block owns kStepCols
// columns of one (token, head); its threads are groups of VEC neighbouring columns times row groups, so the state is read
// and written at full width with all of a thread's rows in flight.  The convolutions of the head's x and of its group's B
// and C are made by every block that needs them (from the ring and the token's projections); the group's first head writes
// their ring place.
// ---------------------------------------------------------------------------
constexpr int kStepCols = 64, kStepThreads = 256;

template <int VEC, int TAPS>
__global__ void __launch_bounds__(kStepThreads, VEC == 4 ? 3 : 1)
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
        const float now = own[ch];
        if (TAPS > 0) {          // (known taps: every input and weight is asked for before the first is used)
            float in[TAPS > 0 ? TAPS : 1], w[TAPS > 0 ? TAPS : 1];
#pragma unroll
            for (int back = TAPS - 1; back >= 0; --back) {
                in[back] = back == 0 ? now : pos >= back ? ring[(size_t)((pos - back) % TAPS) * C + ch] : 0.0f;
                w[back] = ld_f(conv_w, (size_t)ch * TAPS + TAPS - 1 - back, w_dt);
            }
#pragma unroll
            for (int back = TAPS - 1; back >= 0; --back) acc = fmaf(w[back], in[back], acc);
        } else {
            for (int back = z.taps - 1; back > 0; --back)
                if (pos >= back)
                    acc = fmaf(ld_f(conv_w, (size_t)ch * z.taps + z.taps - 1 - back, w_dt), ring[(size_t)((pos - back) % z.taps) * C + ch], acc);
            acc = fmaf(ld_f(conv_w, (size_t)ch * z.taps + z.taps - 1, w_dt), now, acc);
        }
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

// The same for parts that are a multiple of 4 lanes (at most 4 kVec blockDim) in 16-byte rows.
template <int kVec>
__global__ void __launch_bounds__(256)
gated_norm_vec_kernel(const float* __restrict__ y, const float* __restrict__ proj, int ld, const void* __restrict__ w, int w_dt,
                      float eps, void* __restrict__ out, int out_dt, int inner, int part) {
    __shared__ float scratch[33];
    const int t = blockIdx.x, g0 = blockIdx.y * part, n4 = part >> 2;
    const float4* ys = reinterpret_cast<const float4*>(y + (size_t)t * inner + g0);
    const float4* zs = reinterpret_cast<const float4*>(proj + (size_t)t * ld + g0);
    float4 v[kVec], g[kVec];
    float ss = 0.0f;
#pragma unroll
    for (int j = 0; j < kVec; ++j) {
        const int i = threadIdx.x + j * blockDim.x;
        v[j] = i < n4 ? ys[i] : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        g[j] = i < n4 ? zs[i] : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    }
#pragma unroll
    for (int j = 0; j < kVec; ++j) {
        v[j].x *= silu_f(g[j].x); v[j].y *= silu_f(g[j].y); v[j].z *= silu_f(g[j].z); v[j].w *= silu_f(g[j].w);
        ss = fmaf(v[j].x, v[j].x, ss); ss = fmaf(v[j].y, v[j].y, ss);
        ss = fmaf(v[j].z, v[j].z, ss); ss = fmaf(v[j].w, v[j].w, ss);
    }
    ss = block_sum(ss, scratch);
    const float scale = 1.0f / sqrtf(ss * (1.0f / (float)part) + eps);
#pragma unroll
    for (int j = 0; j < kVec; ++j) {
        const int i = threadIdx.x + j * blockDim.x;
        if (i >= n4) continue;
        const int at = g0 + 4 * i;
        const float o[4] = {(v[j].x * scale) * ld_f(w, at, w_dt), (v[j].y * scale) * ld_f(w, at + 1, w_dt),
                            (v[j].z * scale) * ld_f(w, at + 2, w_dt), (v[j].w * scale) * ld_f(w, at + 3, w_dt)};
        if (out_dt == DT_BF16) {
            __nv_bfloat162 h[2] = {__floats2bfloat162_rn(o[0], o[1]), __floats2bfloat162_rn(o[2], o[3])};
            *reinterpret_cast<uint2*>(reinterpret_cast<__nv_bfloat16*>(out) + (size_t)t * inner + at) = *reinterpret_cast<uint2*>(h);
        } else {
            *reinterpret_cast<float4*>(reinterpret_cast<float*>(out) + (size_t)t * inner + at) = make_float4(o[0], o[1], o[2], o[3]);
        }
    }
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

extern "C" int nncpu_ssm_chunk_scan(const float* proj, int ld, const void* xc, const float* gd, float* state, long slot_stride,
                                    const int* seq_slots, const int* cu_seqlens, const int* tok_pos, const void* d_skip,
                                    int p_dt, float* y, int n_seqs, int H, int P, int G, int N, int taps, void* stream) {
    // xc is bfloat16
    Sizes z;
    if (int e = make_sizes(&z, H, P, G, N, taps, ld, slot_stride)) return e;
    NN_CHECK(N <= 256, "state space (chunks): states of %d rows (at most 256)", N);
    NN_CHECK((uintptr_t)xc % 16 == 0 && (uintptr_t)y % 8 == 0, "state space (chunks): rows must be 16-byte aligned");
    if (n_seqs <= 0) return 0;
    cudaStream_t st = (cudaStream_t)stream;
    if (N <= 64) return launch_chunk<64>(proj, z, xc, gd, state, seq_slots, cu_seqlens, tok_pos, d_skip, p_dt, y, n_seqs, st);
    if (N <= 128) return launch_chunk<128>(proj, z, xc, gd, state, seq_slots, cu_seqlens, tok_pos, d_skip, p_dt, y, n_seqs, st);
    return launch_chunk<256>(proj, z, xc, gd, state, seq_slots, cu_seqlens, tok_pos, d_skip, p_dt, y, n_seqs, st);
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
#define NN_STEP(VEC, TAPS)                                                                                                 \
    step_kernel<VEC, TAPS><<<grid, kStepThreads, smem, (cudaStream_t)stream>>>(proj, z, conv_w, w_dt, conv_b, b_dt, state,  \
                                                                               tok_pos, seq_slots, dt_bias, a_log, d_skip, p_dt, y)
    if (vec && taps == 4) NN_STEP(4, 4);
    else if (vec) NN_STEP(4, 0);
    else NN_STEP(1, 0);
#undef NN_STEP
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
    if (part % 4 == 0 && ld % 4 == 0 && part <= 8192 && (((uintptr_t)y | (uintptr_t)proj | (uintptr_t)out) % 16) == 0) {
        const int vec_threads = part >= 1024 ? 256 : (part / 4 + 31) / 32 * 32;
#define NN_GATE(V)                                                                                                         \
    gated_norm_vec_kernel<V><<<dim3(n_tok, n_groups), vec_threads, 0, (cudaStream_t)stream>>>(y, proj, ld, w, w_dt, eps, out, \
                                                                                              out_dt, inner, part)
        if (part <= 1024) NN_GATE(1);
        else if (part <= 2048) NN_GATE(2);
        else if (part <= 4096) NN_GATE(4);
        else NN_GATE(8);
#undef NN_GATE
        NN_LAUNCH_OK("gated norm");
        return 0;
    }
    const int threads = part >= 256 ? 256 : (part + 31) / 32 * 32;
    gated_norm_kernel<<<dim3(n_tok, n_groups), threads, 0, (cudaStream_t)stream>>>(y, proj, ld, w, w_dt, eps, out, out_dt, inner, part);
    NN_LAUNCH_OK("gated norm");
    return 0;
}
