// A matrix memory with exponential gates (the mLSTM of xLSTM).  Per head, with log gates
// i = cap tanh((W_i h + b_i) / cap) and f = logsigmoid(cap tanh((W_f h + b_f) / cap)), a running
// maximum m that starts at 0, a memory S [dim, vdim] and a normaliser n [dim] that start at zero:
//     m_t = max(f + m_{t-1}, i)
//     S_t = exp(f + m_{t-1} - m_t) S_{t-1} + exp(i - m_t) k v^T          n_t likewise with k alone
//     o_t = S_t^T q / (max(|n_t . q|, exp(-m_t)) + floor)                q scaled by dim^-1/2
// All of it float32 (sums of log gates in double), whatever the operand dtype.
//
// Input rows (float32, one per token): [q (H dim) | k (H dim) | v (H vdim) | g (H vdim) | i (H) |
// f (H) | padding].  State per slot: S [H, dim, vdim]; n [2, H, dim] and m [2, H], of which a
// sequence at position p reads number p & 1 and leaves number p' & 1 for its next position p', so that
// the CTAs that share a head may read the old values while one of them writes the new ones.
//
//   memory_step    steps of single tokens: a CTA per (token, head, 32 columns of vdim).
//   memory_gates   prompts, in chunks of 64 tokens of a sequence: with b_t the sum of f over the chunk
//                  up to t and u_t = i_t - b_t, the running maximum is m_t = b_t + M_t,
//                  M_t = max(m_before, u_1 .. u_t): the gates of a chunk need one prefix sum and one
//                  prefix maximum.  A warp per (chunk, head).
//   memory_chunk   what a chunk adds by itself: U = sum_s exp(u_s - max u) k_s v_s^T, and the same of k
//                  alone; all chunks side by side.
//   memory_chain   m between the chunks of a sequence, in order: with M = max(m, max u), m <- b_end + M.
//   memory_carry   S and n between the chunks, in order: S <- exp(m - M) S + exp(max u - M) U; the state
//                  before a chunk replaces the chunk's own U, the last state goes to the slot.
//   memory_out     the outputs, all chunks side by side:
//                  O_t = exp(m_before - M_t) S_before^T q_t + sum_{s <= t} exp(u_s - M_t) (q_t . k_s) v_s,
//                  the denominator the same with n and without v.
//   memory_finish  every head's o divided by its root mean square, times a weight per value, times
//                  sigmoid(g), rounded once to the operand dtype.
//
// A row whose position is -1 (padding) is skipped.
#include "async_copy.cuh"
#include "common.cuh"

namespace nnis {

constexpr int kMemChunk = 64;

__device__ __forceinline__ float log_gate_in(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float log_gate_forget(float z, float cap) {
    const float x = cap * tanhf(z / cap);
    return fminf(x, 0.f) - log1pf(expf(-fabsf(x)));
}

// ---- single tokens ------------------------------------------------------------------------
// Shared memory: q [dim], k [dim] (scaled q).  VEC: four columns a load (vdim a multiple of four).
template <bool VEC>
__global__ void __launch_bounds__(256)
memory_step_kernel(const float* __restrict__ a, int a_cols, const float* __restrict__ i_bias,
                   const float* __restrict__ f_bias, float* state, float* norm_state, float* max_state,
                   const int* __restrict__ token_pos, const int* __restrict__ token_seq,
                   const int* __restrict__ seq_slots, float* __restrict__ o_raw, int H, int dim, int vdim, float cap,
                   float q_scale, float floor_add) {
    extern __shared__ float smem[];
    __shared__ float red[8][32];
    __shared__ float red_n[8];
    pdl_wait();
    pdl_launch_dependents();
    const int n = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int pos = token_pos[n];
    if (pos < 0) return;
    const int slot = seq_slots[token_seq[n]];
    const int now = pos & 1, next = now ^ 1;
    const float* row = a + (size_t)n * a_cols;
    const float* vrow = row + (size_t)2 * H * dim + (size_t)h * vdim;
    const float* gates = row + (size_t)2 * H * dim + (size_t)2 * H * vdim;
    float* qs = smem;
    float* ks = smem + dim;
    const float i = log_gate_in(gates[h] + i_bias[h], cap);
    const float f = log_gate_forget(gates[H + h] + f_bias[h], cap);
    float* m_at = max_state + (size_t)slot * 2 * H + h;
    const float m_old = m_at[now * H];
    const float m_new = fmaxf(f + m_old, i);
    const float keep = expf(f + m_old - m_new), take = expf(i - m_new);
    const float* n_old = norm_state + ((size_t)slot * 2 + now) * H * dim + (size_t)h * dim;
    float* n_new = norm_state + ((size_t)slot * 2 + next) * H * dim + (size_t)h * dim;
    float nq = 0.f;
    for (int d = tid; d < dim; d += 256) {
        const float q = row[(size_t)h * dim + d] * q_scale, k = row[(size_t)H * dim + (size_t)h * dim + d];
        qs[d] = q;
        ks[d] = take * k;
        const float v = fmaf(keep, n_old[d], take * k);
        if (blockIdx.z == 0) n_new[d] = v;
        nq = fmaf(v, q, nq);
    }
    nq = warp_sum(nq);
    if (lane == 0) red_n[warp] = nq;
    __syncthreads();
    float* S = state + ((size_t)slot * H + h) * dim * vdim;
    const int col0 = blockIdx.z * 32;
    float o[4] = {0.f, 0.f, 0.f, 0.f};
    if (VEC) {
        const int c = col0 + (tid & 7) * 4, r = tid >> 3;  // eight lanes to a row of 32 columns
        if (c < vdim) {
            const float4 v = make_float4(vrow[c], vrow[c + 1], vrow[c + 2], vrow[c + 3]);
            for (int d0 = r; d0 < dim; d0 += 128) {
                float4 s[4];
#pragma unroll
                for (int j = 0; j < 4; ++j)
                    if (d0 + 32 * j < dim) s[j] = *reinterpret_cast<const float4*>(S + (size_t)(d0 + 32 * j) * vdim + c);
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const int d = d0 + 32 * j;
                    if (d < dim) {
                        const float k = ks[d], q = qs[d];
                        s[j].x = fmaf(keep, s[j].x, k * v.x);
                        s[j].y = fmaf(keep, s[j].y, k * v.y);
                        s[j].z = fmaf(keep, s[j].z, k * v.z);
                        s[j].w = fmaf(keep, s[j].w, k * v.w);
                        *reinterpret_cast<float4*>(S + (size_t)d * vdim + c) = s[j];
                        o[0] = fmaf(s[j].x, q, o[0]);
                        o[1] = fmaf(s[j].y, q, o[1]);
                        o[2] = fmaf(s[j].z, q, o[2]);
                        o[3] = fmaf(s[j].w, q, o[3]);
                    }
                }
            }
        }
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            o[e] += __shfl_xor_sync(0xffffffffu, o[e], 8);
            o[e] += __shfl_xor_sync(0xffffffffu, o[e], 16);
            if (lane < 8) red[warp][lane * 4 + e] = o[e];
        }
    } else {
        const int c = col0 + lane;
        if (c < vdim) {
            const float v = vrow[c];
            for (int d = warp; d < dim; d += 8) {
                const float s = fmaf(keep, S[(size_t)d * vdim + c], ks[d] * v);
                S[(size_t)d * vdim + c] = s;
                o[0] = fmaf(s, qs[d], o[0]);
            }
        }
        red[warp][lane] = o[0];
    }
    __syncthreads();
    if (warp == 0) {
        float sum = 0.f, total = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) {
            sum += red[w][lane];
            total += red_n[w];
        }
        const float bottom = fmaxf(fabsf(total), expf(-m_new)) + floor_add;
        if (col0 + lane < vdim) o_raw[((size_t)n * H + h) * vdim + col0 + lane] = sum / bottom;
        if (blockIdx.z == 0 && lane == 0) m_at[next * H] = m_new;
    }
}

// ---- prompts ------------------------------------------------------------------------------
struct MemChunk {
    int seq, begin, first, count;  // of the batch; first token within the step's tokens of the sequence; packed row; tokens
};
__device__ __forceinline__ MemChunk mem_chunk(const int* chunks, const int* seq_first_row, const int* seq_count, int c) {
    MemChunk m;
    m.seq = chunks[2 * c];
    m.begin = chunks[2 * c + 1];
    m.first = seq_first_row[m.seq] + m.begin;
    m.count = min(kMemChunk, seq_count[m.seq] - m.begin);
    return m;
}

// b, u, top: double [n_tokens, H] (sum of log forget gates, i - b, prefix maximum of u, all within the chunk);
// ends: double [n_chunks, H, 2] (b of the last token, maximum of u); before: double [n_chunks, H], of which
// this kernel writes the first chunks' (m as the step finds it).
__global__ void __launch_bounds__(256)
memory_gates_kernel(const float* __restrict__ a, int a_cols, const float* __restrict__ i_bias,
                    const float* __restrict__ f_bias, const float* __restrict__ max_state,
                    const int* __restrict__ chunks, const int* __restrict__ seq_slots,
                    const int* __restrict__ seq_first_row, const int* __restrict__ seq_start,
                    const int* __restrict__ seq_count, double* __restrict__ b, double* __restrict__ u,
                    double* __restrict__ top, double* __restrict__ ends, double* __restrict__ before, int H,
                    int gate_off, float cap) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const MemChunk ch = mem_chunk(chunks, seq_first_row, seq_count, blockIdx.x);
    for (int h = blockIdx.y * 8 + warp; h < H; h += gridDim.y * 8) {
        double fs[2];
        float is[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int t = 2 * lane + e;
            fs[e] = 0.0;
            is[e] = -INFINITY;
            if (t < ch.count) {
                const float* g = a + (size_t)(ch.first + t) * a_cols + gate_off;
                is[e] = log_gate_in(g[h] + i_bias[h], cap);
                fs[e] = (double)log_gate_forget(g[H + h] + f_bias[h], cap);
            }
        }
        double sum = fs[0] + fs[1];
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const double x = __shfl_up_sync(0xffffffffu, sum, o);
            if (lane >= o) sum += x;
        }
        const double b1 = sum, b0 = sum - fs[1];
        const double u0 = (double)is[0] - b0, u1 = (double)is[1] - b1;
        double mx = fmax(u0, u1);
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const double x = __shfl_up_sync(0xffffffffu, mx, o);
            if (lane >= o) mx = fmax(mx, x);
        }
        double prev = __shfl_up_sync(0xffffffffu, mx, 1);
        if (lane == 0) prev = -INFINITY;
        const int t = 2 * lane;
        const size_t at = (size_t)(ch.first + t) * H + h;
        if (t < ch.count) {
            b[at] = b0;
            u[at] = u0;
            top[at] = fmax(prev, u0);
        }
        if (t + 1 < ch.count) {
            b[at + H] = b1;
            u[at + H] = u1;
            top[at + H] = mx;
        }
        if (lane == 31) {
            ends[((size_t)blockIdx.x * H + h) * 2] = b1;
            ends[((size_t)blockIdx.x * H + h) * 2 + 1] = mx;
            if (ch.begin == 0)
                before[(size_t)blockIdx.x * H + h] =
                    (double)max_state[((size_t)seq_slots[ch.seq] * 2 + (seq_start[ch.seq] & 1)) * H + h];
        }
    }
}

// A CTA of 256 threads per (chunk, head, 64 rows of dim x BV columns of vdim): 4 columns and BV / 16 rows a thread.
template <int BV>
__global__ void __launch_bounds__(256)
memory_chunk_kernel(const float* __restrict__ a, int a_cols, const double* __restrict__ u,
                    const double* __restrict__ ends, const int* __restrict__ chunks,
                    const int* __restrict__ seq_first_row, const int* __restrict__ seq_count,
                    float* __restrict__ chunk_state, float* __restrict__ chunk_norm, int H, int dim, int vdim) {
    constexpr int TX = BV / 4, RM = BV / 16, STEP = 32;
    __shared__ __align__(16) float Ks[STEP][64];
    __shared__ __align__(16) float Vs[STEP][BV];
    __shared__ float weight[kMemChunk];
    const int c = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
    const int v_tiles = (vdim + BV - 1) / BV;
    const int d0 = blockIdx.z / v_tiles * 64, v0 = blockIdx.z % v_tiles * BV;
    const int tx = tid % TX, ty = tid / TX;
    const MemChunk ch = mem_chunk(chunks, seq_first_row, seq_count, c);
    if (tid < kMemChunk)
        weight[tid] = tid < ch.count
                          ? expf((float)(u[(size_t)(ch.first + tid) * H + h] - ends[((size_t)c * H + h) * 2 + 1]))
                          : 0.f;
    float acc[RM][4] = {};
    float norm = 0.f;
    for (int s0 = 0; s0 < ch.count; s0 += STEP) {
        __syncthreads();
        for (int it = tid; it < STEP * 64; it += 256) {
            const int s = it >> 6, d = it & 63;
            float x = 0.f;
            if (s0 + s < ch.count && d0 + d < dim)
                x = a[(size_t)(ch.first + s0 + s) * a_cols + (size_t)H * dim + (size_t)h * dim + d0 + d] * weight[s0 + s];
            Ks[s][d] = x;
        }
        for (int it = tid; it < STEP * BV; it += 256) {
            const int s = it / BV, j = it % BV;
            float x = 0.f;
            if (s0 + s < ch.count && v0 + j < vdim)
                x = a[(size_t)(ch.first + s0 + s) * a_cols + (size_t)2 * H * dim + (size_t)h * vdim + v0 + j];
            Vs[s][j] = x;
        }
        __syncthreads();
        if (v0 == 0 && tid < 64)
            for (int s = 0; s < STEP; ++s) norm += Ks[s][tid];
#pragma unroll 8
        for (int s = 0; s < STEP; ++s) {
            const float4 v = *reinterpret_cast<const float4*>(&Vs[s][tx * 4]);
#pragma unroll
            for (int r = 0; r < RM; r += 4) {
                const float4 k = *reinterpret_cast<const float4*>(&Ks[s][ty * RM + r]);
                const float kr[4] = {k.x, k.y, k.z, k.w};
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    acc[r + e][0] = fmaf(kr[e], v.x, acc[r + e][0]);
                    acc[r + e][1] = fmaf(kr[e], v.y, acc[r + e][1]);
                    acc[r + e][2] = fmaf(kr[e], v.z, acc[r + e][2]);
                    acc[r + e][3] = fmaf(kr[e], v.w, acc[r + e][3]);
                }
            }
        }
    }
    if (v0 == 0 && tid < 64 && d0 + tid < dim) chunk_norm[((size_t)c * H + h) * dim + d0 + tid] = norm;
    float* out = chunk_state + ((size_t)c * H + h) * dim * vdim;
    const bool whole = (vdim & 3) == 0;
#pragma unroll
    for (int r = 0; r < RM; ++r) {
        const int d = d0 + ty * RM + r, j = v0 + tx * 4;
        if (d >= dim || j >= vdim) continue;
        float* to = out + (size_t)d * vdim + j;
        if (whole) {
            *reinterpret_cast<float4*>(to) = make_float4(acc[r][0], acc[r][1], acc[r][2], acc[r][3]);
        } else {
            for (int e = 0; e < 4; ++e)
                if (j + e < vdim) to[e] = acc[r][e];
        }
    }
}

// The running maximum from chunk to chunk of a sequence, in order (a warp per (sequence, head)): `before` of every chunk
// but the first, the factors of the state before a chunk and of the chunk's own sum (`factors` float [n_chunks, H, 2]), and
// the maximum that the step leaves.
__global__ void __launch_bounds__(32)
memory_chain_kernel(const double* __restrict__ ends, double* before, float* __restrict__ factors,
                    float* __restrict__ max_state, const int* __restrict__ seq_slots, const int* __restrict__ seq_start,
                    const int* __restrict__ seq_count, const int* __restrict__ seq_first_chunk, int H) {
    const int seq = blockIdx.x, h = blockIdx.y, lane = threadIdx.x;
    const int c0 = seq_first_chunk[seq], c1 = seq_first_chunk[seq + 1];
    if (c1 <= c0) return;
    double m = before[(size_t)c0 * H + h];
    for (int c = c0; c < c1; c += 32) {  // 32 chunks at a time: a lane holds one chunk's gates
        const bool in = c + lane < c1;
        const size_t at = (size_t)min(c + lane, c1 - 1) * H + h;
        const double b_end = ends[at * 2], u_max = ends[at * 2 + 1];
        double mine = 0.0;
        for (int j = 0; j < min(32, c1 - c); ++j) {
            if (lane == j) mine = m;
            m = fmax(m, __shfl_sync(0xffffffffu, u_max, j)) + __shfl_sync(0xffffffffu, b_end, j);
        }
        if (in) {
            const double M = fmax(mine, u_max);
            before[at] = mine;
            factors[at * 2] = expf((float)(mine - M));
            factors[at * 2 + 1] = expf((float)(u_max - M));
        }
    }
    if (lane == 0)
        max_state[((size_t)seq_slots[seq] * 2 + ((seq_start[seq] + seq_count[seq]) & 1)) * H + h] = (float)m;
}

// A thread per V elements of S, then of n (V = 4 where dim and dim * vdim are multiples of four).
template <int V>
__global__ void __launch_bounds__(256)
memory_carry_kernel(float* chunk_state, float* chunk_norm, float* state, float* norm_state,
                    const float* __restrict__ factors, const int* __restrict__ seq_slots,
                    const int* __restrict__ seq_start, const int* __restrict__ seq_count,
                    const int* __restrict__ seq_first_chunk, int H, int dim, int vdim) {
    constexpr int AHEAD = 8;
    struct alignas(4 * V) Pack { float x[V]; };
    const int seq = blockIdx.x, h = blockIdx.y, per = dim * vdim;
    const int e = (blockIdx.z * 256 + threadIdx.x) * V;
    if (e >= per + dim) return;
    const int c0 = seq_first_chunk[seq], c1 = seq_first_chunk[seq + 1];
    if (c1 <= c0) return;
    const int slot = seq_slots[seq], start = seq_start[seq], end = start + seq_count[seq];
    const bool is_n = e >= per;
    const size_t step = (size_t)H * (is_n ? dim : per);
    float* own = is_n ? chunk_norm + ((size_t)c0 * H + h) * dim + (e - per) : chunk_state + ((size_t)c0 * H + h) * per + e;
    float* from = is_n ? norm_state + ((size_t)slot * 2 + (start & 1)) * H * dim + (size_t)h * dim + (e - per)
                       : state + ((size_t)slot * H + h) * per + e;
    float* to = is_n ? norm_state + ((size_t)slot * 2 + (end & 1)) * H * dim + (size_t)h * dim + (e - per) : from;
    Pack run = *reinterpret_cast<const Pack*>(from);
    for (int c = c0; c < c1; c += AHEAD) {
        Pack add[AHEAD];
#pragma unroll
        for (int j = 0; j < AHEAD; ++j)
            if (c + j < c1) add[j] = *reinterpret_cast<const Pack*>(own + (size_t)(c - c0 + j) * step);
#pragma unroll
        for (int j = 0; j < AHEAD; ++j) {
            if (c + j >= c1) break;
            const float2 f = *reinterpret_cast<const float2*>(factors + ((size_t)(c + j) * H + h) * 2);
            *reinterpret_cast<Pack*>(own + (size_t)(c - c0 + j) * step) = run;
#pragma unroll
            for (int v = 0; v < V; ++v) run.x[v] = fmaf(f.x, run.x[v], f.y * add[j].x[v]);
        }
    }
    *reinterpret_cast<Pack*>(to) = run;
}

// A CTA of 256 threads per (chunk, head, BV columns of vdim).  Scores: 4 x 4 a thread; outputs: 4 columns and
// BV / 16 rows a thread.
template <int BV>
__global__ void __launch_bounds__(256, 3)
memory_out_kernel(const float* __restrict__ a, int a_cols, const double* __restrict__ b, const double* __restrict__ u,
                  const double* __restrict__ top, const double* __restrict__ before,
                  const float* __restrict__ chunk_state, const float* __restrict__ chunk_norm,
                  const int* __restrict__ chunks, const int* __restrict__ seq_first_row,
                  const int* __restrict__ seq_start, const int* __restrict__ seq_count, float* __restrict__ o_raw,
                  int H, int dim, int vdim, float q_scale, float floor_add) {
    constexpr int C = kMemChunk, STEP = 32, LD = C + 4, TX = BV / 4, RM = BV / 16;
    extern __shared__ __align__(16) float smem[];
    float* Qs = smem;               // [STEP][LD], by place in dim
    float* Ks = Qs + STEP * LD;     // [STEP][LD]
    float* Ps = Ks + STEP * LD;     // [C keys][LD]
    float* Vs = Ps + C * LD;        // [STEP][BV]: rows of the state before the chunk, then of v
    __shared__ double us[C], Mt[C];
    __shared__ float carry[C], least[C], nsum[C], ns[STEP];
    const int c = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * BV, tid = threadIdx.x;
    const MemChunk ch = mem_chunk(chunks, seq_first_row, seq_count, c);
    const bool fresh = ch.begin == 0 && seq_start[ch.seq] == 0;  // nothing before this chunk
    if (tid < C) {
        us[tid] = 0.0;
        Mt[tid] = 0.0;
        carry[tid] = least[tid] = nsum[tid] = 0.f;
        if (tid < ch.count) {
            const size_t at = (size_t)(ch.first + tid) * H + h;
            const double m = before[(size_t)c * H + h], M = fmax(m, top[at]);
            us[tid] = u[at];
            Mt[tid] = M;
            carry[tid] = expf((float)(m - M));
            least[tid] = expf((float)(-(b[at] + M)));
        }
    }
    const int sx = tid & 15, sy = tid >> 4;  // scores: keys 4 sx .., queries 4 sy ..
    const int tx = tid % TX, ty = tid / TX;  // outputs: columns 4 tx .., queries RM ty ..
    float sc[4][4] = {};
    float acc[RM][4] = {};
    float nq = 0.f;
    const float* S = chunk_state + ((size_t)c * H + h) * dim * vdim;
    const int r_lo = tid & 3, k_lo = (tid >> 2) & 7, group = tid >> 5;  // a warp fetches 4 rows x 8 places
    for (int d0 = 0; d0 < dim; d0 += STEP) {
        __syncthreads();
        for (int it = group; it < (C / 4) * (STEP / 8); it += 8) {
            const int t = (it >> 2) * 4 + r_lo, d = (it & 3) * 8 + k_lo;
            float q = 0.f, k = 0.f;
            if (t < ch.count && d0 + d < dim) {
                const float* at = a + (size_t)(ch.first + t) * a_cols + (size_t)h * dim + d0 + d;
                q = at[0] * q_scale;
                k = at[(size_t)H * dim];
            }
            Qs[d * LD + t] = q;
            Ks[d * LD + t] = k;
        }
        if (!fresh) {
            for (int it = tid; it < STEP * BV; it += 256) {
                const int d = it / BV, j = it % BV;
                Vs[it] = d0 + d < dim && v0 + j < vdim ? S[(size_t)(d0 + d) * vdim + v0 + j] : 0.f;
            }
            if (tid < STEP) ns[tid] = d0 + tid < dim ? chunk_norm[((size_t)c * H + h) * dim + d0 + tid] : 0.f;
        }
        __syncthreads();
#pragma unroll 8
        for (int d = 0; d < STEP; ++d) {
            const float4 q = *reinterpret_cast<const float4*>(Qs + d * LD + sy * 4);
            const float4 k = *reinterpret_cast<const float4*>(Ks + d * LD + sx * 4);
            const float qr[4] = {q.x, q.y, q.z, q.w}, kr[4] = {k.x, k.y, k.z, k.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) sc[i][j] = fmaf(qr[i], kr[j], sc[i][j]);
        }
        if (!fresh) {
#pragma unroll 4
            for (int d = 0; d < STEP; ++d) {
                const float4 s = *reinterpret_cast<const float4*>(Vs + d * BV + tx * 4);
#pragma unroll
                for (int r = 0; r < RM; r += 4) {
                    const float4 q = *reinterpret_cast<const float4*>(Qs + d * LD + ty * RM + r);
                    const float qr[4] = {q.x, q.y, q.z, q.w};
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        acc[r + e][0] = fmaf(qr[e], s.x, acc[r + e][0]);
                        acc[r + e][1] = fmaf(qr[e], s.y, acc[r + e][1]);
                        acc[r + e][2] = fmaf(qr[e], s.z, acc[r + e][2]);
                        acc[r + e][3] = fmaf(qr[e], s.w, acc[r + e][3]);
                    }
                }
            }
            if (tid < C)
                for (int d = 0; d < STEP; ++d) nq = fmaf(Qs[d * LD + tid], ns[d], nq);
        }
    }
    // the scores with their gates; their sums are the chunk's share of n . q
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int t = sy * 4 + i;
        float sum = 0.f;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int s = sx * 4 + j;
            sc[i][j] = s <= t && t < ch.count ? sc[i][j] * expf((float)(us[s] - Mt[t])) : 0.f;
            sum += sc[i][j];
        }
        sum = half_warp_sum(sum);
        if (sx == 0) nsum[t] = sum;
    }
#pragma unroll
    for (int j = 0; j < 4; ++j)
        *reinterpret_cast<float4*>(Ps + (sx * 4 + j) * LD + sy * 4) = make_float4(sc[0][j], sc[1][j], sc[2][j], sc[3][j]);
#pragma unroll
    for (int r = 0; r < RM; ++r) {
        const float w = carry[ty * RM + r];
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[r][e] *= w;
    }
    for (int s0 = 0; s0 < ch.count; s0 += STEP) {
        __syncthreads();
        for (int it = tid; it < STEP * BV; it += 256) {
            const int s = it / BV, j = it % BV;
            Vs[it] = s0 + s < ch.count && v0 + j < vdim
                         ? a[(size_t)(ch.first + s0 + s) * a_cols + (size_t)2 * H * dim + (size_t)h * vdim + v0 + j]
                         : 0.f;
        }
        __syncthreads();
#pragma unroll 4
        for (int s = 0; s < STEP; ++s) {
            const float4 v = *reinterpret_cast<const float4*>(Vs + s * BV + tx * 4);
#pragma unroll
            for (int r = 0; r < RM; r += 4) {
                const float4 p = *reinterpret_cast<const float4*>(Ps + (s0 + s) * LD + ty * RM + r);
                const float pr[4] = {p.x, p.y, p.z, p.w};
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    acc[r + e][0] = fmaf(pr[e], v.x, acc[r + e][0]);
                    acc[r + e][1] = fmaf(pr[e], v.y, acc[r + e][1]);
                    acc[r + e][2] = fmaf(pr[e], v.z, acc[r + e][2]);
                    acc[r + e][3] = fmaf(pr[e], v.w, acc[r + e][3]);
                }
            }
        }
    }
    if (tid < C) nsum[tid] = 1.0f / (fmaxf(fabsf(fmaf(carry[tid], nq, nsum[tid])), least[tid]) + floor_add);
    __syncthreads();
#pragma unroll
    for (int r = 0; r < RM; ++r) {
        const int t = ty * RM + r, j = v0 + tx * 4;
        if (t >= ch.count) continue;
        const float inv = nsum[t];
        float* to = o_raw + ((size_t)(ch.first + t) * H + h) * vdim + j;
        if ((vdim & 3) == 0) {
            if (j < vdim)
                *reinterpret_cast<float4*>(to) =
                    make_float4(acc[r][0] * inv, acc[r][1] * inv, acc[r][2] * inv, acc[r][3] * inv);
        } else {
            for (int e = 0; e < 4; ++e)
                if (j + e < vdim) to[e] = acc[r][e] * inv;
        }
    }
}

// A warp per (token, head).
template <typename T>
__global__ void __launch_bounds__(256)
memory_finish_kernel(const float* __restrict__ o_raw, const float* __restrict__ a, int a_cols, int gate_off,
                     const float* __restrict__ w, const int* __restrict__ token_pos, T* __restrict__ out,
                     long long n_units, int H, int vdim, float eps) {
    pdl_wait();
    pdl_launch_dependents();
    const long long unit = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
    if (unit >= n_units) return;
    const int lane = threadIdx.x & 31;
    const long long n = unit / H;
    const int h = (int)(unit - n * H);
    T* dst = out + (size_t)unit * vdim;
    if (token_pos[n] < 0) {
        for (int i = lane; i < vdim; i += 32) dst[i] = from_float<T>(0.f);
        return;
    }
    const float* o = o_raw + (size_t)unit * vdim;
    const float* g = a + (size_t)n * a_cols + gate_off + (size_t)h * vdim;
    const float* wh = w + (size_t)h * vdim;
    float ss = 0.f;
    for (int i = lane; i < vdim; i += 32) ss = fmaf(o[i], o[i], ss);
    const float s = 1.0f / sqrtf(warp_sum(ss) / (float)vdim + eps);
    for (int i = lane; i < vdim; i += 32) dst[i] = from_float<T>((o[i] * s) * wh[i] * (1.0f / (1.0f + expf(-g[i]))));
}

template <int BV>
static cudaError_t launch_memory_prompt(const float* a, int a_cols, float* state, float* norm_state, float* max_state,
                                        const int* chunks, int n_chunks, const int* seq_first_chunk, int n_seqs,
                                        const int* seq_slots, const int* seq_first_row, const int* seq_start,
                                        const int* seq_count, double* gates, double* chunk_gates, int n_tokens,
                                        float* chunk_state, float* chunk_norm, float* o_raw, int H, int dim, int vdim,
                                        float q_scale, float floor_add, cudaStream_t stream) {
    double *b = gates, *u = gates + (size_t)n_tokens * H, *top = gates + (size_t)2 * n_tokens * H;
    double *ends = chunk_gates, *before = chunk_gates + (size_t)2 * n_chunks * H;
    const int v_tiles = (vdim + BV - 1) / BV, d_tiles = (dim + 63) / 64;
    memory_chunk_kernel<BV><<<dim3(n_chunks, H, v_tiles * d_tiles), 256, 0, stream>>>(
        a, a_cols, u, ends, chunks, seq_first_row, seq_count, chunk_state, chunk_norm, H, dim, vdim);
    float* factors = reinterpret_cast<float*>(chunk_gates + (size_t)3 * n_chunks * H);
    memory_chain_kernel<<<dim3(n_seqs, H), 32, 0, stream>>>(ends, before, factors, max_state, seq_slots, seq_start,
                                                            seq_count, seq_first_chunk, H);
    const int elems = dim * vdim + dim;
    if (dim % 4 == 0)
        memory_carry_kernel<4><<<dim3(n_seqs, H, (elems / 4 + 255) / 256), 256, 0, stream>>>(
            chunk_state, chunk_norm, state, norm_state, factors, seq_slots, seq_start, seq_count, seq_first_chunk, H, dim,
            vdim);
    else
        memory_carry_kernel<1><<<dim3(n_seqs, H, (elems + 255) / 256), 256, 0, stream>>>(
            chunk_state, chunk_norm, state, norm_state, factors, seq_slots, seq_start, seq_count, seq_first_chunk, H, dim,
            vdim);
    const size_t smem = (size_t)(2 * 32 * (kMemChunk + 4) + kMemChunk * (kMemChunk + 4) + 32 * BV) * sizeof(float);
    auto kernel = memory_out_kernel<BV>;
    if (smem > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return e;
    }
    cudaError_t carve = cudaFuncSetAttribute(kernel, cudaFuncAttributePreferredSharedMemoryCarveout,
                                             cudaSharedmemCarveoutMaxShared);  // three CTAs an SM
    if (carve != cudaSuccess) return carve;
    kernel<<<dim3(n_chunks, H, v_tiles), 256, smem, stream>>>(a, a_cols, b, u, top, before, chunk_state, chunk_norm,
                                                              chunks, seq_first_row, seq_start, seq_count, o_raw, H,
                                                              dim, vdim, q_scale, floor_add);
    return cudaGetLastError();
}

}  // namespace nnis

using namespace nnis;

NNIS_API int nnis_memory_chunk_tokens() { return kMemChunk; }

// Single tokens: every row of the step is a sequence of its own.  a: float32 [n_tokens, a_cols]; state float32
// [slots, H, dim, vdim], norm_state [slots, 2, H, dim], max_state [slots, 2, H]; o_raw float32 [n_tokens, H * vdim].
NNIS_API int nnis_memory_step(const float* a, int a_cols, const float* i_bias, const float* f_bias, float* state,
                              float* norm_state, float* max_state, const int* token_pos, const int* token_seq,
                              const int* seq_slots, float* o_raw, int n_tokens, int H, int dim, int vdim, float cap,
                              float q_scale, float floor_add, cudaStream_t stream) {
    if (!a || !i_bias || !f_bias || !state || !norm_state || !max_state || !token_pos || !token_seq || !seq_slots ||
        !o_raw || n_tokens <= 0 || H <= 0 || dim <= 0 || vdim <= 0 || !(cap > 0.f) ||
        a_cols < 2 * H * (dim + vdim) + 2 * H)
        return NNIS_ERR_ARGUMENT;
    if (dim > 2048 || H > 65535 || (vdim + 31) / 32 > 65535) return NNIS_ERR_UNSUPPORTED;
    const dim3 grid(n_tokens, H, (vdim + 31) / 32);
    const size_t smem = 2 * (size_t)dim * sizeof(float);
    cudaError_t e = vdim % 4 == 0
        ? launch_dependent(memory_step_kernel<true>, grid, 256, smem, stream, a, a_cols, i_bias, f_bias, state,
                           norm_state, max_state, token_pos, token_seq, seq_slots, o_raw, H, dim, vdim, cap, q_scale,
                           floor_add)
        : launch_dependent(memory_step_kernel<false>, grid, 256, smem, stream, a, a_cols, i_bias, f_bias, state,
                           norm_state, max_state, token_pos, token_seq, seq_slots, o_raw, H, dim, vdim, cap, q_scale,
                           floor_add);
    return e == cudaSuccess ? NNIS_OK : (int)e;
}

// Prompt steps.  chunks: int32 [n_chunks, 2] = (sequence, first token of the chunk among the sequence's tokens of this
// step), 64 tokens each but for a sequence's last, in the order of the sequences; seq_first_chunk
// [n_seqs + 1].  Scratch: gates double [3, n_tokens, H]; chunk_gates double [4, n_chunks, H]; chunk_state
// float32 [n_chunks, H, dim, vdim]; chunk_norm float32 [n_chunks, H, dim].
NNIS_API int nnis_memory_prompt(const float* a, int a_cols, const float* i_bias, const float* f_bias, float* state,
                                float* norm_state, float* max_state, const int* chunks, int n_chunks,
                                const int* seq_first_chunk, int n_seqs, const int* seq_slots, const int* seq_first_row,
                                const int* seq_start, const int* seq_count, double* gates, double* chunk_gates,
                                float* chunk_state, float* chunk_norm, float* o_raw, int n_tokens, int H, int dim,
                                int vdim, float cap, float q_scale, float floor_add, cudaStream_t stream) {
    if (!a || !i_bias || !f_bias || !state || !norm_state || !max_state || !chunks || !seq_first_chunk || !seq_slots ||
        !seq_first_row || !seq_start || !seq_count || !gates || !chunk_gates || !chunk_state || !chunk_norm || !o_raw ||
        n_tokens <= 0 || n_chunks <= 0 || n_seqs <= 0 || H <= 0 || dim <= 0 || vdim <= 0 || !(cap > 0.f) ||
        a_cols < 2 * H * (dim + vdim) + 2 * H)
        return NNIS_ERR_ARGUMENT;
    const long long tiles = (long long)((dim + 63) / 64) * ((vdim + 63) / 64);
    if (H > 65535 || tiles > 65535 || ((long long)dim * vdim + dim + 255) / 256 > 65535) return NNIS_ERR_UNSUPPORTED;
    double *b = gates, *u = gates + (size_t)n_tokens * H, *top = gates + (size_t)2 * n_tokens * H;
    double *ends = chunk_gates, *before = chunk_gates + (size_t)2 * n_chunks * H;
    memory_gates_kernel<<<dim3(n_chunks, (H + 7) / 8), 256, 0, stream>>>(
        a, a_cols, i_bias, f_bias, max_state, chunks, seq_slots, seq_first_row, seq_start, seq_count, b, u, top, ends,
        before, H, 2 * H * (dim + vdim), cap);
    cudaError_t e = vdim > 64
        ? launch_memory_prompt<128>(a, a_cols, state, norm_state, max_state, chunks, n_chunks, seq_first_chunk, n_seqs,
                                    seq_slots, seq_first_row, seq_start, seq_count, gates, chunk_gates, n_tokens,
                                    chunk_state, chunk_norm, o_raw, H, dim, vdim, q_scale, floor_add, stream)
        : launch_memory_prompt<64>(a, a_cols, state, norm_state, max_state, chunks, n_chunks, seq_first_chunk, n_seqs,
                                   seq_slots, seq_first_row, seq_start, seq_count, gates, chunk_gates, n_tokens,
                                   chunk_state, chunk_norm, o_raw, H, dim, vdim, q_scale, floor_add, stream);
    return e == cudaSuccess ? NNIS_OK : (int)e;
}

NNIS_API int nnis_memory_finish(const float* o_raw, const float* a, int a_cols, int gate_off, const float* w,
                                const int* token_pos, void* out, int n_tokens, int H, int vdim, float eps, int dtype,
                                cudaStream_t stream) {
    if (!o_raw || !a || !w || !token_pos || !out || n_tokens <= 0 || H <= 0 || vdim <= 0 || !(eps > 0.f) ||
        gate_off < 0 || a_cols < gate_off + H * vdim)
        return NNIS_ERR_ARGUMENT;
    const long long units = (long long)n_tokens * H;
    const unsigned blocks = (unsigned)((units + 7) / 8);
    cudaError_t e;
    if (dtype == NNIS_DTYPE_F32)
        e = launch_dependent(memory_finish_kernel<float>, blocks, 256, 0, stream, o_raw, a, a_cols, gate_off, w,
                             token_pos, (float*)out, units, H, vdim, eps);
    else if (dtype == NNIS_DTYPE_BF16)
        e = launch_dependent(memory_finish_kernel<bf16>, blocks, 256, 0, stream, o_raw, a, a_cols, gate_off, w,
                             token_pos, (bf16*)out, units, H, vdim, eps);
    else
        return NNIS_ERR_UNSUPPORTED;
    return e == cudaSuccess ? NNIS_OK : (int)e;
}
