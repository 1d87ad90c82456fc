// Prompt attention with a sink on the tensor cores, bfloat16, key and value heads of up to 128
// values (multiples of eight) over the paged cache: the prompt-step form of attention_sink.cu.
// Heads are padded with zeros to 64 or 128 values in shared memory.
//
// A CTA of four warps owns 64 consecutive query tokens of one sequence and one query head,
// each warp 16 rows of m16n8k16 tiles.  It walks the pages (64 keys) that its rows can see:
// the pages of the first `keep` keys, which every row sees, then from the page that holds the
// start of the first row's chunk (or window) to the page of the last row.  K and V pages come into swizzled shared memory by 16-byte cp.async copies, two
// pages ahead; S = Q K^T and O += P V are matrix products; between them, in float32
// registers: score = cap * tanh(scale * s / cap) (cap 0: none) plus the head's bias for the
// distance (a thread's scores of a page lie on 18 distances, read once a page), the mask (causal,
// the row's own chunk counted from position 0 of the sequence, the window, the kept first keys), and the online softmax,
// whose running maximum starts at the head's sink and whose running sum starts at one: the
// sink's own term, which has no key and no value.  The rows leave multiplied by the gate of
// their (token, head).  The host lists the tiles (sequence, first query).
#include <float.h>

#include "mma_helpers.cuh"

namespace nnis {

constexpr int kSinkRows = 64;   // query rows per CTA
constexpr int kSinkPage = 64;
constexpr int kSinkStages = 3;

// DK, DV: sizes in shared memory; PAD: the heads hold fewer values (dk, dv); BIAS: a bias per distance
template <int DK, int DV, bool PAD, bool BIAS>
__global__ void __launch_bounds__(128, (DK <= 64 && DV <= 64) ? 3 : 1)
attn_sink_mma_kernel(const bf16* __restrict__ q, const bf16* __restrict__ k_cache,
                     const bf16* __restrict__ v_cache, const int* __restrict__ tiles,
                     const int* __restrict__ seq_first_row, const int* __restrict__ seq_start,
                     const int* __restrict__ seq_count, const int* __restrict__ page_table, int table_cols,
                     const float* __restrict__ sink, const float* __restrict__ gate, bf16* __restrict__ out,
                     int nq, int nkv, int window, int chunk, float scale, float cap, int gate_elems, int dk_real,
                     int dv_real, int keep, const float* __restrict__ bias, int bias_len) {
    constexpr int NT = DV / 8, KS = DK / 16;
    const int dk = PAD ? dk_real : DK, dv = PAD ? dv_real : DV;
    const int KCH = dk >> 3, VCH = dv >> 3;  // 16-byte chunks of a row
    extern __shared__ __align__(128) unsigned char smem_raw[];
    bf16* q_s = reinterpret_cast<bf16*>(smem_raw);  // [64, DK] swizzled
    bf16* kv_s = q_s + kSinkRows * DK;              // stages x (K [64, DK], V [64, DV])
    constexpr size_t k_elems = (size_t)kSinkPage * DK, v_elems = (size_t)kSinkPage * DV;

    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, tid = threadIdx.x;
    const int seq = tiles[2 * blockIdx.x], q0 = tiles[2 * blockIdx.x + 1];
    const int hq = blockIdx.y, hk = hq / (nq / nkv);
    const int count = seq_count[seq], start = seq_start[seq];
    const int row_base = seq_first_row[seq] + q0;
    const int rows = min(kSinkRows, count - q0);
    const int pos0 = start + q0;
    const int hi = pos0 + rows;
    int lo = window > 0 ? max(0, pos0 - window + 1) : 0;
    if (chunk > 0) lo = max(lo, (pos0 / chunk) * chunk);  // (later rows' chunks start no earlier)
    const int first_page = lo / kSinkPage;
    // pages of the kept first keys that lie before the first page of the rows' own range
    const int kept_pages = keep > 0 ? min((keep - 1) / kSinkPage + 1, first_page) : 0;
    const int n_pages = kept_pages + (hi - 1) / kSinkPage - first_page + 1;
    auto page_of = [&](int it) { return it < kept_pages ? it : first_page + it - kept_pages; };
    const int* table = page_table + (size_t)seq * table_cols;

    if constexpr (PAD) {  // the padding chunks are zero and stay zero
        const uint4 zero = make_uint4(0, 0, 0, 0);
        const int kpad = DK / 8 - KCH, vpad = DV / 8 - VCH;
        for (int c = tid; c < kSinkPage * kpad; c += 128) {
            const int row = c / kpad, part = KCH + c % kpad;
            *reinterpret_cast<uint4*>(q_s + swz<DK>(row, part)) = zero;
            for (int st = 0; st < kSinkStages; ++st)
                *reinterpret_cast<uint4*>(kv_s + st * (k_elems + v_elems) + swz<DK>(row, part)) = zero;
        }
        for (int c = tid; c < kSinkPage * vpad; c += 128) {
            const int row = c / vpad, part = VCH + c % vpad;
            for (int st = 0; st < kSinkStages; ++st)
                *reinterpret_cast<uint4*>(kv_s + st * (k_elems + v_elems) + k_elems + swz<DV>(row, part)) = zero;
        }
    }
    auto load_page = [&](int it) {
        if (it < n_pages) {
            int page = table[page_of(it)];
            const bf16* ksrc = k_cache + (size_t)(page * nkv + hk) * (kSinkPage * dk);
            const bf16* vsrc = v_cache + (size_t)(page * nkv + hk) * (kSinkPage * dv);
            bf16* kd = kv_s + (size_t)(it % kSinkStages) * (k_elems + v_elems);
            bf16* vd = kd + k_elems;
            if (DK == DV && !PAD) {
                for (int c = tid; c < kSinkPage * KCH; c += 128) {
                    int row = c / KCH, part = c % KCH;
                    cp_async16(kd + swz<DK>(row, part), ksrc + (size_t)c * 8);
                    cp_async16(vd + swz<DV>(row, part), vsrc + (size_t)c * 8);
                }
            } else {
                for (int c = tid; c < kSinkPage * KCH; c += 128) {
                    int row = c / KCH, part = c - row * KCH;
                    cp_async16(kd + swz<DK>(row, part), ksrc + (size_t)c * 8);
                }
                for (int c = tid; c < kSinkPage * VCH; c += 128) {
                    int row = c / VCH, part = c - row * VCH;
                    cp_async16(vd + swz<DV>(row, part), vsrc + (size_t)c * 8);
                }
            }
        }
        cp_async_commit();
    };
    for (int it = 0; it < kSinkStages - 1; ++it) load_page(it);

    for (int c = tid; c < kSinkRows * KCH; c += 128) {
        int row = c / KCH, part = c - row * KCH;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (row < rows)
            v = *reinterpret_cast<const uint4*>(q + ((size_t)(row_base + row) * nq + hq) * dk + part * 8);
        *reinterpret_cast<uint4*>(q_s + swz<DK>(row, part)) = v;
    }
    __syncthreads();
    uint32_t qa[KS][4];
#pragma unroll
    for (int kk = 0; kk < KS; ++kk)
        ldmatrix_x4(qa[kk], q_s + swz<DK>(warp * 16 + (lane & 15), kk * 2 + (lane >> 4)));

    const int r_lo = lane >> 2, c_lo = (lane & 3) * 2;
    int pos_r[2], lo_r[2];
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        pos_r[h] = pos0 + warp * 16 + r_lo + h * 8;
        lo_r[h] = window > 0 ? pos_r[h] - window + 1 : 0;
        if (chunk > 0) lo_r[h] = max(lo_r[h], (pos_r[h] / chunk) * chunk);
    }
    // the first key of the warp's last row, the largest of its rows'
    int warp_hi_lo = window > 0 ? pos0 + warp * 16 + 15 - window + 1 : 0;
    if (chunk > 0) warp_hi_lo = max(warp_hi_lo, ((pos0 + warp * 16 + 15) / chunk) * chunk);
    float o[NT][4];
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[j][e] = 0.f;
    // scores are kept times log2(e); the sink is one more score, held by one lane of each row's four
    float m_run[2], l_run[2];
    m_run[0] = m_run[1] = sink ? sink[hq] * kLog2e : -INFINITY;
    l_run[0] = l_run[1] = (sink && (lane & 3) == 0) ? 1.f : 0.f;
    const float cap_in = cap > 0.f ? 2.0f * kLog2e / cap : 0.f, cap_out = cap * kLog2e;
    const float sc = scale * kLog2e;

    for (int it = 0; it < n_pages; ++it) {
        cp_async_wait<kSinkStages - 2>();
        __syncthreads();
        load_page(it + kSinkStages - 1);
        const bf16* kt = kv_s + (size_t)(it % kSinkStages) * (k_elems + v_elems);
        const bf16* vt = kt + k_elems;
        const int t0 = page_of(it) * kSinkPage;
        // a warp whose rows all lie before this page, or whose rows' chunks or windows all start
        // after it, has nothing to see in it (a page of kept keys: all rows after it do)
        if (t0 > pos0 + warp * 16 + 15) continue;
        if (t0 >= keep) {
            if (chunk > 0 && t0 + kSinkPage <= ((pos0 + warp * 16) / chunk) * chunk) continue;
            if (window > 0 && t0 + kSinkPage <= pos0 + warp * 16 - window + 1) continue;
        }
        // every row of the warp sees every key of the page (most pages of a long walk): no mask
        const bool full = t0 + kSinkPage - 1 <= pos0 + warp * 16 && (t0 >= warp_hi_lo || t0 + kSinkPage <= keep);
        // the biases, times log2(e), of the distances that this thread's scores of the page lie on:
        // row r_lo + 8 h against key 8 j + c_lo + e is the distance (of the warp's first row) + r_lo -
        // c_lo + 8 (h - j) - e, so h - j = -7 .. 1 and e = 0, 1
        float near[9][2];
        if (BIAS) {
            const float* table_h = bias + (size_t)hq * bias_len;
            const int d0 = pos0 + warp * 16 + r_lo - t0 - c_lo;
#pragma unroll
            for (int i = 0; i < 9; ++i)
#pragma unroll
                for (int e = 0; e < 2; ++e)
                    near[i][e] = __ldg(table_h + min(max(d0 + 8 * (i - 7) - e, 0), bias_len - 1)) * kLog2e;
        }

        float s[8][4];
#pragma unroll
        for (int j = 0; j < 8; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) s[j][e] = 0.f;
#pragma unroll
        for (int kk = 0; kk < KS; kk += 2) {
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                uint32_t b[4];
                ldmatrix_x4(b, kt + swz<DK>(j * 8 + (lane & 7), kk * 2 + (lane >> 3)));
                mma_bf16(s[j], qa[kk], b[0], b[1]);
                mma_bf16(s[j], qa[kk + 1], b[2], b[3]);
            }
        }
        uint32_t pa[4][4];
        float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int j = 0; j < 8; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                float v;
                if (cap > 0.f) {  // cap * tanh(x / cap) = cap * (1 - 2 / (exp(2 x / cap) + 1))
                    float e2 = exp2f(s[j][e] * scale * cap_in);
                    v = cap_out * (1.0f - __fdividef(2.0f, e2 + 1.0f));
                } else {
                    v = s[j][e] * sc;
                }
                if (BIAS) v += near[(e >> 1) - j + 7][e & 1];
                s[j][e] = v;
            }
        if (!full) {
#pragma unroll
            for (int j = 0; j < 8; ++j)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int key = t0 + j * 8 + c_lo + (e & 1);
                    const bool ok = key <= pos_r[e >> 1] && (key >= lo_r[e >> 1] || key < keep);
                    s[j][e] = ok ? s[j][e] : -INFINITY;
                }
        }
#pragma unroll
        for (int j = 0; j < 8; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) mx[e >> 1] = fmaxf(mx[e >> 1], s[j][e]);
        float alpha[2], base[2];
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
            mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
            float mn = fmaxf(m_run[r], mx[r]);
            base[r] = mn == -INFINITY ? 0.f : mn;
            alpha[r] = exp2f(m_run[r] - base[r]);
            m_run[r] = mn;
        }
        float psum[2] = {0.f, 0.f};
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            float p0v = exp2f(s[j][0] - base[0]), p1v = exp2f(s[j][1] - base[0]);
            float p2v = exp2f(s[j][2] - base[1]), p3v = exp2f(s[j][3] - base[1]);
            psum[0] += p0v + p1v;
            psum[1] += p2v + p3v;
            pa[j >> 1][(j & 1) * 2] = pack_bf16(p0v, p1v);
            pa[j >> 1][(j & 1) * 2 + 1] = pack_bf16(p2v, p3v);
        }
#pragma unroll
        for (int r = 0; r < 2; ++r) l_run[r] = l_run[r] * alpha[r] + psum[r];
#pragma unroll
        for (int jn = 0; jn < NT; ++jn)
#pragma unroll
            for (int e = 0; e < 4; ++e) o[jn][e] *= alpha[e >> 1];
#pragma unroll
        for (int ks = 0; ks < 4; ++ks) {
#pragma unroll
            for (int jn = 0; jn < NT; jn += 2) {
                uint32_t b[4];
                ldmatrix_x4_trans(b, vt + swz<DV>(ks * 16 + (lane & 15), jn + (lane >> 4)));
                mma_bf16(o[jn], pa[ks], b[0], b[1]);
                mma_bf16(o[jn + 1], pa[ks], b[2], b[3]);
            }
        }
    }
    cp_async_wait<0>();
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 1);
        l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 2);
    }
    const int ra = warp * 16 + r_lo, rb = ra + 8;
    float inv_a = l_run[0] > 0.f ? 1.0f / l_run[0] : 0.f;
    float inv_b = l_run[1] > 0.f ? 1.0f / l_run[1] : 0.f;
    const bool by_value = gate && gate_elems > 1;  // a gate per output value: [n, nq * dv]
    if (gate && !by_value) {
        if (ra < rows) inv_a *= gate[(size_t)(row_base + ra) * nq + hq];
        if (rb < rows) inv_b *= gate[(size_t)(row_base + rb) * nq + hq];
    }
#pragma unroll
    for (int jn = 0; jn < NT; ++jn) {
        if (PAD && jn >= VCH) break;
        int col = hq * dv + jn * 8 + c_lo;
        if (ra < rows) {
            float2 g = by_value ? *reinterpret_cast<const float2*>(gate + (size_t)(row_base + ra) * nq * dv + col)
                                : make_float2(1.f, 1.f);
            *reinterpret_cast<uint32_t*>(out + (size_t)(row_base + ra) * nq * dv + col) =
                pack_bf16(o[jn][0] * inv_a * g.x, o[jn][1] * inv_a * g.y);
        }
        if (rb < rows) {
            float2 g = by_value ? *reinterpret_cast<const float2*>(gate + (size_t)(row_base + rb) * nq * dv + col)
                                : make_float2(1.f, 1.f);
            *reinterpret_cast<uint32_t*>(out + (size_t)(row_base + rb) * nq * dv + col) =
                pack_bf16(o[jn][2] * inv_b * g.x, o[jn][3] * inv_b * g.y);
        }
    }
}

template <int DK, int DV, bool PAD, bool BIAS>
static int launch_sink_mma(dim3 grid, cudaStream_t stream, const bf16* q, const bf16* k, const bf16* v,
                           const int* tiles, const int* first_row, const int* start, const int* count,
                           const int* table, int cols, const float* sink, const float* gate, bf16* out, int nq,
                           int nkv, int window, int chunk, float scale, float cap, int gate_elems, int dk, int dv,
                           int keep, const float* bias, int bias_len) {
    size_t smem = ((size_t)kSinkRows * DK + (size_t)kSinkStages * kSinkPage * (DK + DV)) * sizeof(bf16);
    auto kernel = attn_sink_mma_kernel<DK, DV, PAD, BIAS>;
    if (smem > 48 * 1024) {
        cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
    }
    kernel<<<grid, 128, smem, stream>>>(q, k, v, tiles, first_row, start, count, table, cols, sink, gate, out, nq,
                                        nkv, window, chunk, scale, cap, gate_elems, dk, dv, keep, bias, bias_len);
    NNIS_RETURN_LAUNCH();
}

}  // namespace nnis

// 1 if the tensor-core kernel takes these sizes (else the kernel for any sizes runs)
NNIS_API int nnis_attention_sink_mma_takes(int dk, int dv, int page_size) {
    return dk > 0 && dv > 0 && dk % 8 == 0 && dv % 8 == 0 && dk <= 128 && dv <= 128 && page_size == nnis::kSinkPage;
}

// `tiles`: int32 [n_tiles, 2] = (sequence of the batch, first query of the tile within this
// step's tokens of that sequence), 64 queries a tile.  q [n, nq * dk], out [n, nq * dv], caches
// [pages, nkv, 64, dk] and [pages, nkv, 64, dv]; gate float32 [n, nq] or, with gate_elems = dv,
// [n, nq * dv]; keep: first keys of a sequence that every later query sees; bias: float32
// [nq, bias_len] by distance, or null.  Other sizes than nnis_attention_sink_mma_takes: refused.
NNIS_API int nnis_attention_sink_mma(const void* q, const void* k_cache, const void* v_cache, const int* tiles,
                                     int n_tiles, const int* seq_first_row, const int* seq_start,
                                     const int* seq_count, const int* page_table, int table_cols,
                                     const float* sink, const float* gate, void* out, int nq, int nkv, int dk, int dv,
                                     int page_size, int window, int chunk, float scale, float cap, int gate_elems,
                                     int keep, const float* bias, int bias_len, cudaStream_t stream) {
    using namespace nnis;
    if (n_tiles <= 0 || nq <= 0 || nkv <= 0 || nq % nkv || table_cols <= 0 || window < 0 || chunk < 0 ||
        cap < 0.f || keep < 0 || (bias && bias_len <= 0) || !tiles)
        return NNIS_ERR_ARGUMENT;
    if (!nnis_attention_sink_mma_takes(dk, dv, page_size)) return NNIS_ERR_UNSUPPORTED;
    if (nq > 65535) return NNIS_ERR_UNSUPPORTED;
    if (gate_elems > 1 && gate_elems != dv) return NNIS_ERR_ARGUMENT;
    if (((uintptr_t)q | (uintptr_t)k_cache | (uintptr_t)v_cache | (uintptr_t)out) % 16) return NNIS_ERR_ALIGNMENT;
    dim3 grid(n_tiles, nq);
#define NNIS_SINK_MMA(DK, DV, PAD) \
    return bias ? launch_sink_mma<DK, DV, PAD, true>(grid, stream, (const bf16*)q, (const bf16*)k_cache, \
                                                     (const bf16*)v_cache, tiles, seq_first_row, seq_start, \
                                                     seq_count, page_table, table_cols, sink, gate, (bf16*)out, nq, \
                                                     nkv, window, chunk, scale, cap, gate_elems, dk, dv, keep, bias, \
                                                     bias_len) \
                : launch_sink_mma<DK, DV, PAD, false>(grid, stream, (const bf16*)q, (const bf16*)k_cache, \
                                                      (const bf16*)v_cache, tiles, seq_first_row, seq_start, \
                                                      seq_count, page_table, table_cols, sink, gate, (bf16*)out, nq, \
                                                      nkv, window, chunk, scale, cap, gate_elems, dk, dv, keep, bias, \
                                                      bias_len)
    if (dk == 64 && dv == 64) { NNIS_SINK_MMA(64, 64, false); }
    if (dk == 128 && dv == 128) { NNIS_SINK_MMA(128, 128, false); }
    if (dk <= 64 && dv <= 64) { NNIS_SINK_MMA(64, 64, true); }
    if (dk <= 64) { NNIS_SINK_MMA(64, 128, true); }
    if (dv <= 64) { NNIS_SINK_MMA(128, 64, true); }
    NNIS_SINK_MMA(128, 128, true);
#undef NNIS_SINK_MMA
}
