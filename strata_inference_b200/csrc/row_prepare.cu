// What lies between the q|k(|v) product and the attention kernel for mixers that work on whole
// projected rows ahead of their heads (csrc/head_prepare.cu works on single heads):
//
//     u  = proj + bias                                        (q and k; bias optional)
//     c_t = sum_j w[j] u_(t - taps + 1 + j)                   per channel of q and k, zeros before the
//                                                             sequence's start (taps 0: c = u)
//     v  = c of k, head by head  (values are keys), or proj's own v columns + bias
//     x  = c / sqrt(mean over ALL of the row's q (or k) channels of c^2 + eps) * gain   (optional)
//     x  rotated per head: the first `rot` dimensions, half-split or neighbouring pairs, by the
//        angle pos * inv_freq[i], cosine and sine both times `magnitude`
//
// q, k and v go to a packed buffer whose heads are all `pad` wide (zeros behind a narrower
// head), k and v also into the paged cache of that width.  The last taps - 1 rows of u of a
// sequence are per-slot state, 32-bit, oldest first: state[slot] = [taps - 1][q and k channels].
// Everything is 32-bit between the product's output and the packed rows.
//
//   row_prepare          a block per row (or per few rows), the row in shared memory or in registers;
//                        steps of one row per sequence move the state on in the same launch
//   row_prepare_state    the state after any other step, in a launch of its own behind it
//
// Rows of a sequence that holds no slot (slot -1, fillers of a recorded step) see zeros before
// their own rows and leave nothing behind.
// Plain counterpart: tests/plain_simetar.py attention().
#include "common.cuh"

namespace {

struct RowPrepareArgs {
    const void* proj;          // [rows, proj_stride]: q heads | k heads | (v heads) | ...
    void* qkv;                 // [rows, (n_heads + 2 n_kv) * pad]
    const float* bias;         // [nq + nk (+ nv)] or null
    const float* conv;         // [taps, nq + nk] or null
    float* state;              // [slots, state_stride] (taps > 1)
    const float* q_gain;       // [nq] or null: no norm
    const float* k_gain;       // [nk]
    const float* inv_freq;     // [rot / 2] or null
    const int* row_pos;
    const int* row_seq;
    const int* seq_slot;
    const int* seq_start;
    const int* seq_end;
    const int* seq_row0;
    void* k_pool;              // [pages, n_kv, page_tokens, pad]; null: nothing is stored
    void* v_pool;
    const int* page_table;
    long long proj_stride, state_stride;
    int rows, n_heads, n_kv, kd, vd, pad, rot, taps;
    int values_from_keys, neighbours, single;
    int max_pages, page_tokens, ring_tokens, fixed_tokens;
    float eps, magnitude;
};

// The row's cell of kv head 0 in a pool, in elements, or -1 if the row is not stored.
__device__ __forceinline__ long long cell_of_row(const RowPrepareArgs& p, int pos, int b, int slot) {
    if (p.k_pool == nullptr || slot < 0 || !cell_written(pos, p.seq_end[b], p.fixed_tokens, p.ring_tokens)) return -1;
    const int cell = cell_of(pos, p.fixed_tokens, p.ring_tokens);
    const int page = p.page_table[(size_t)slot * p.max_pages + cell / p.page_tokens];
    return ((long long)page * p.n_kv * p.page_tokens + cell % p.page_tokens) * p.pad;
}

// Any sizes: a block per row, the row of q and k channels in shared memory.
template <typename T>
__global__ void __launch_bounds__(256) row_prepare_kernel(RowPrepareArgs p) {
    extern __shared__ float row[];             // [nq + nk]
    __shared__ float scratch[33];
    pdl_trigger();
    const int r = blockIdx.x;
    const int nq = p.n_heads * p.kd, nk = p.n_kv * p.kd, C = nq + nk;
    const int pos = p.row_pos[r], b = p.row_seq[r], slot = p.seq_slot[b];
    const int back = pos - p.seq_start[b];                   // rows of this step before this one
    const long long cell = cell_of_row(p, pos, b, slot);
    pdl_wait();
    const T* src = (const T*)p.proj + (size_t)r * p.proj_stride;
    float* hist = p.taps > 1 && slot >= 0 ? p.state + (size_t)slot * p.state_stride : nullptr;
    float sq = 0.f, sk = 0.f;
    for (int c = threadIdx.x; c < C; c += blockDim.x) {
        const float bias = p.bias ? p.bias[c] : 0.f;
        const float own = to_f32(src[c]) + bias;
        float acc = own;
        if (p.conv) {
            acc = p.conv[(size_t)(p.taps - 1) * C + c] * own;
            for (int d = 1; d < p.taps; ++d) {               // the input d positions back
                float u;
                if (d <= back) u = to_f32(src[c - (long long)d * p.proj_stride]) + bias;
                else if (hist) u = hist[(size_t)(p.taps - 1 + back - d) * C + c];
                else break;                                  // (zeros from here on)
                acc += p.conv[(size_t)(p.taps - 1 - d) * C + c] * u;
            }
            if (p.single && hist)
                for (int k = 0; k < p.taps - 1; ++k)
                    hist[(size_t)k * C + c] = k + 1 < p.taps - 1 ? hist[(size_t)(k + 1) * C + c] : own;
        }
        row[c] = acc;
        if (c < nq) sq += acc * acc;
        else sk += acc * acc;
    }
    float iq = 1.f, ik = 1.f;
    if (p.q_gain) {
        iq = 1.0f / sqrtf(block_sum(sq, scratch) / (float)nq + p.eps);
        ik = 1.0f / sqrtf(block_sum(sk, scratch) / (float)nk + p.eps);
    }
    __syncthreads();
    const int units = p.n_heads + 2 * p.n_kv;
    T* out = (T*)p.qkv + (size_t)r * units * p.pad;
    for (int idx = threadIdx.x; idx < units * p.pad; idx += blockDim.x) {
        const int unit = idx / p.pad, d = idx - unit * p.pad;
        const bool is_q = unit < p.n_heads, is_v = unit >= p.n_heads + p.n_kv;
        float x = 0.f;
        if (is_v) {
            const int g = unit - p.n_heads - p.n_kv;
            if (d < p.vd) {
                if (p.values_from_keys) x = row[nq + g * p.kd + d];
                else x = to_f32(src[C + g * p.vd + d]) + (p.bias ? p.bias[C + g * p.vd + d] : 0.f);
            }
        } else if (d < p.kd) {
            const int c0 = unit * p.kd;                      // (k heads follow the q heads)
            const float inv = is_q ? iq : ik;
            const float* gain = is_q ? p.q_gain : p.k_gain ? p.k_gain - nq : nullptr;
            auto normed = [&](int e) { return gain ? row[c0 + e] * inv * gain[c0 + e] : row[c0 + e]; };
            x = normed(d);
            if (p.inv_freq && d < p.rot) {
                const int half = p.rot / 2;
                const int i = p.neighbours ? d >> 1 : (d < half ? d : d - half);
                const bool first = p.neighbours ? !(d & 1) : d < half;
                const int other = p.neighbours ? d ^ 1 : (d < half ? d + half : d - half);
                const float ang = (float)pos * p.inv_freq[i];
                const float c = cosf(ang) * p.magnitude, s = sinf(ang) * p.magnitude;
                x = first ? x * c - normed(other) * s : x * c + normed(other) * s;
            }
        }
        const T y = from_f32<T>(x);
        out[idx] = y;
        if (!is_q && cell >= 0) {
            const int g = is_v ? unit - p.n_heads - p.n_kv : unit - p.n_heads;
            ((T*)(is_v ? p.v_pool : p.k_pool))[cell + (long long)g * p.page_tokens * p.pad + d] = y;
        }
    }
}

__device__ __forceinline__ void load8(const float* from, float (&o)[8]) {
    const float4 lo = *reinterpret_cast<const float4*>(from), hi = *reinterpret_cast<const float4*>(from + 4);
    o[0] = lo.x; o[1] = lo.y; o[2] = lo.z; o[3] = lo.w;
    o[4] = hi.x; o[5] = hi.y; o[6] = hi.z; o[7] = hi.w;
}
__device__ __forceinline__ void store8(float* to, const float (&o)[8]) {
    *reinterpret_cast<float4*>(to) = make_float4(o[0], o[1], o[2], o[3]);
    *reinterpret_cast<float4*>(to + 4) = make_float4(o[4], o[5], o[6], o[7]);
}
__device__ __forceinline__ void unpack8(const uint4& v, float (&o)[8]) {
    const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        o[2 * i] = __uint_as_float(w[i] << 16);
        o[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
    }
}
__device__ __forceinline__ uint4 pack8(const float (&x)[8]) {
    uint32_t o[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const __nv_bfloat162 pr = __floats2bfloat162_rn(x[2 * i], x[2 * i + 1]);
        o[i] = *reinterpret_cast<const uint32_t*>(&pr);
    }
    return make_uint4(o[0], o[1], o[2], o[3]);
}

// The common case in 16-byte accesses: bfloat16, heads of a multiple of 8 that need no filling
// up, neighbouring pairs.  A thread owns 8 neighbouring channels of q, k or v and takes RUN
// neighbouring rows at once.  A run inside one sequence whose first row has all its predecessors in
// this step asks for its rows together and convolves them tap by tap from registers; in any other
// run each row fetches what lies before it from the step's rows or from the state.  The rows'
// sums cross the block with one barrier.  Where a row is stored, and its cosines and sines, are
// worked out once per block ahead of the wait for the projection (positions and tables are
// written by the host before the step).  TAPS 0: no convolution.
template <int TAPS, int RUN, int THREADS, int BLOCKS>
__global__ void __launch_bounds__(THREADS, BLOCKS) row_prepare_bf16_kernel(RowPrepareArgs p) {
    constexpr int BACK = TAPS > 1 ? TAPS - 1 : 0;          // rows before its own that a row reads
    extern __shared__ float2 turns[];          // [RUN][rot / 2]
    __shared__ float2 sums[RUN][32];
    __shared__ long long cells[RUN];           // the rows' cells of kv head 0, or -1
    __shared__ int slots[RUN], backs[RUN], seqs[RUN];
    pdl_trigger();
    const int nq = p.n_heads * p.kd, nk = p.n_kv * p.kd, C = nq + nk;
    const int units = p.n_heads + 2 * p.n_kv;
    const int c = 8 * threadIdx.x;             // the thread's first channel of the projected row
    const bool live = c < C + (p.values_from_keys ? 0 : nk);
    const bool is_q = c < nq, is_v = c >= C;   // (v channels of their own are passed on)
    const int r0 = blockIdx.x * RUN, n_rows = min(RUN, p.rows - r0);
    const int half = p.inv_freq ? p.rot / 2 : 0;
    if ((int)threadIdx.x < n_rows) {
        const int r = r0 + threadIdx.x, pos = p.row_pos[r], b = p.row_seq[r], slot = p.seq_slot[b];
        cells[threadIdx.x] = cell_of_row(p, pos, b, slot);
        slots[threadIdx.x] = slot;
        backs[threadIdx.x] = pos - p.seq_start[b];
        seqs[threadIdx.x] = b;
    }
    for (int i = threadIdx.x; i < n_rows * half; i += blockDim.x) {
        const int k = i / half;
        const float ang = (float)p.row_pos[r0 + k] * p.inv_freq[i - k * half];
        turns[i] = make_float2(cosf(ang) * p.magnitude, sinf(ang) * p.magnitude);
    }
    float bias[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) bias[e] = 0.f;
    if (live && p.bias) load8(p.bias + c, bias);
    __syncthreads();
    const bool conv = TAPS > 0 && live && !is_v;
    const bool together = n_rows == RUN && seqs[RUN - 1] == seqs[0] && backs[0] >= BACK;
    pdl_wait();
    const __nv_bfloat16* proj = (const __nv_bfloat16*)p.proj + (size_t)r0 * p.proj_stride + c;
    auto fetch = [&](int row) {                // `row`: from the run's first
        return *reinterpret_cast<const uint4*>(proj + (long long)row * p.proj_stride);
    };
    auto input = [&](const uint4& raw, float (&u)[8]) {
        unpack8(raw, u);
#pragma unroll
        for (int e = 0; e < 8; ++e) u[e] += bias[e];
    };
    float acc[RUN][8];
#pragma unroll
    for (int k = 0; k < RUN; ++k)
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[k][e] = 0.f;
    if (conv && together && RUN > 1) {
        uint4 raw[RUN + BACK];
#pragma unroll
        for (int k = 0; k < RUN + BACK; ++k) raw[k] = fetch(k - BACK);
#pragma unroll
        for (int j = TAPS - 1; j >= 0; --j) {
            float w[8];
            load8(p.conv + (size_t)j * C + c, w);
#pragma unroll
            for (int k = 0; k < RUN; ++k) {
                float u[8];
                input(raw[k + j], u);
#pragma unroll
                for (int e = 0; e < 8; ++e) acc[k][e] += w[e] * u[e];
            }
        }
    } else if (conv) {
#pragma unroll
        for (int k = 0; k < RUN; ++k) {
            if (k >= n_rows) break;
            float u[BACK + 1][8];              // u[d]: the input d positions back
            input(fetch(k), u[0]);
            float* hist = BACK > 0 && slots[k] >= 0 ? p.state + (size_t)slots[k] * p.state_stride + c : nullptr;
#pragma unroll
            for (int d = 1; d <= BACK; ++d) {
#pragma unroll
                for (int e = 0; e < 8; ++e) u[d][e] = 0.f;
                if (d <= backs[k]) input(fetch(k - d), u[d]);
                else if (hist) load8(hist + (size_t)(BACK + backs[k] - d) * C, u[d]);
            }
#pragma unroll
            for (int d = 0; d <= BACK; ++d) {
                float w[8];
                load8(p.conv + (size_t)(TAPS > 0 ? TAPS - 1 - d : 0) * C + c, w);
#pragma unroll
                for (int e = 0; e < 8; ++e) acc[k][e] += w[e] * u[d][e];
            }
            if (p.single && hist) {            // one position on
#pragma unroll
                for (int d = 0; d < BACK; ++d) store8(hist + (size_t)(BACK - 1 - d) * C, u[d]);
            }
        }
    } else if (live) {
#pragma unroll
        for (int k = 0; k < RUN; ++k)
            if (k < n_rows) input(fetch(k), acc[k]);
    }
    __nv_bfloat16* dst = (__nv_bfloat16*)p.qkv + (size_t)r0 * units * p.pad + c;
    const int d0 = c % p.kd;                   // the thread's place in its head
    // where the thread's 8 values go in a pool behind a row's cell
    const size_t head_at = (size_t)((is_v ? c - C : c - nq) / p.kd) * p.page_tokens * p.pad + d0;
    if (live && (is_v || (!is_q && p.values_from_keys))) {
#pragma unroll
        for (int k = 0; k < RUN; ++k) {
            if (k >= n_rows) break;
            const uint4 v = pack8(acc[k]);
            *reinterpret_cast<uint4*>(dst + (size_t)k * units * p.pad + (is_v ? 0 : nk)) = v;
            if (cells[k] >= 0) *reinterpret_cast<uint4*>((__nv_bfloat16*)p.v_pool + cells[k] + head_at) = v;
        }
    }
    const int lane = threadIdx.x & 31, n_warps = (blockDim.x + 31) >> 5;
    float gain[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) gain[e] = 1.f;
    if (p.q_gain) {
        // (a warp of q channels alone, or of others alone, sums one number a row)
        const bool any_q = __any_sync(0xffffffffu, is_q), any_k = __any_sync(0xffffffffu, !is_q);
#pragma unroll
        for (int k = 0; k < RUN; ++k) {
            float t = 0.f;
            if (live && !is_v) {
#pragma unroll
                for (int e = 0; e < 8; ++e) t += acc[k][e] * acc[k][e];
            }
            float2 s = make_float2(0.f, 0.f);
            if (any_q) s.x = warp_sum(is_q ? t : 0.f);
            if (any_k) s.y = warp_sum(is_q ? 0.f : t);
            if (lane == 0) sums[k][threadIdx.x >> 5] = s;
        }
        if (live && !is_v) load8(is_q ? p.q_gain + c : p.k_gain + (c - nq), gain);
        __syncthreads();
    }
    if (is_v || !live) return;                 // (neither a barrier nor a shuffle is left)
    const bool rotates = d0 < 2 * half;
#pragma unroll
    for (int k = 0; k < RUN; ++k) {
        if (k >= n_rows) break;
        if (p.q_gain) {
            float total = 0.f;
            for (int w = 0; w < n_warps; ++w) total += is_q ? sums[k][w].x : sums[k][w].y;
            const float inv = 1.0f / sqrtf(total / (float)(is_q ? nq : nk) + p.eps);
#pragma unroll
            for (int e = 0; e < 8; ++e) acc[k][e] = acc[k][e] * inv * gain[e];
        }
        if (rotates) {
            const float2* cs = turns + (size_t)k * half + d0 / 2;
#pragma unroll
            for (int i = 0; i < 4; ++i)
                if (d0 / 2 + i < half) {
                    const float2 t = cs[i];
                    const float u = acc[k][2 * i], v = acc[k][2 * i + 1];
                    acc[k][2 * i] = u * t.x - v * t.y;
                    acc[k][2 * i + 1] = v * t.x + u * t.y;
                }
        }
        const uint4 y = pack8(acc[k]);
        *reinterpret_cast<uint4*>(dst + (size_t)k * units * p.pad) = y;
        if (!is_q && cells[k] >= 0) *reinterpret_cast<uint4*>((__nv_bfloat16*)p.k_pool + cells[k] + head_at) = y;
    }
}

// The state after the step: the last taps - 1 inputs of each sequence.  One thread per (sequence,
// channel), oldest first: a cell that keeps an older input takes it from a later cell of the
// same state, which has not been rewritten yet.
template <typename T>
__global__ void __launch_bounds__(256) row_prepare_state_kernel(RowPrepareArgs p) {
    pdl_trigger();
    pdl_wait();
    const int C = (p.n_heads + p.n_kv) * p.kd;
    const int b = blockIdx.y, slot = p.seq_slot[b];
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    if (slot < 0 || c >= C) return;
    const int n = p.seq_end[b] - p.seq_start[b], row0 = p.seq_row0[b];
    const float bias = p.bias ? p.bias[c] : 0.f;
    float* hist = p.state + (size_t)slot * p.state_stride;
    for (int i = 0; i < p.taps - 1; ++i) {
        const int back = p.taps - 1 - i;             // the input `back` positions before the end
        hist[(size_t)i * C + c] = back <= n
            ? to_f32(((const T*)p.proj)[(size_t)(row0 + n - back) * p.proj_stride + c]) + bias
            : hist[(size_t)(i + n) * C + c];
    }
}

}  // namespace

// `single`: every sequence of the step has exactly one row.  `taps` 0: no convolution.
SIB_EXPORT int sib_row_prepare(
    const void* proj, long long proj_stride, void* qkv, int dtype, const float* bias, const float* conv, int taps,
    float* state, long long state_stride, const float* q_gain, const float* k_gain, float eps,
    const float* inv_freq, int rot, int neighbours, float magnitude, const int* row_pos, const int* row_seq,
    const int* seq_slot, const int* seq_start, const int* seq_end, const int* seq_row0, void* k_pool, void* v_pool,
    const int* page_table, int max_pages, int page_tokens, int ring_tokens, int fixed_tokens, int rows, int n_seqs,
    int n_heads, int n_kv, int kd, int vd, int pad, int values_from_keys, int single, void* stream) {
    if (rows == 0) return 0;
    SIB_REQUIRE(rows > 0 && n_seqs > 0 && n_seqs < 65536 && n_heads > 0 && n_kv > 0 && kd > 0 && vd > 0,
                "row_prepare: rows=%d sequences=%d heads=%d kv_heads=%d key width=%d value width=%d", rows, n_seqs,
                n_heads, n_kv, kd, vd);
    SIB_REQUIRE(pad >= kd && pad >= vd && (!values_from_keys || kd == vd),
                "row_prepare: heads of %d and %d in a width of %d (values that are keys have their width)", kd, vd, pad);
    SIB_REQUIRE(rot >= 0 && rot % 2 == 0 && rot <= kd && (rot == 0 || inv_freq != nullptr),
                "row_prepare: %d rotated dimensions of %d", rot, kd);
    SIB_REQUIRE(proj && qkv && row_pos && row_seq && seq_slot && seq_start && seq_end && seq_row0,
                "row_prepare: an argument is missing");
    SIB_REQUIRE((q_gain != nullptr) == (k_gain != nullptr), "row_prepare: q and k are normed together");
    const int nq = n_heads * kd, nk = n_kv * kd, C = nq + nk;
    SIB_REQUIRE(taps >= 0 && (taps > 0) == (conv != nullptr) &&
                    (taps <= 1 || (state && state_stride >= (long long)(taps - 1) * C)),
                "row_prepare: %d taps need their weights and a state of (taps - 1) * %d numbers", taps, C);
    SIB_REQUIRE(!single || rows == n_seqs, "row_prepare: %d rows of %d sequences are not one each", rows, n_seqs);
    SIB_REQUIRE(k_pool == nullptr || (v_pool && page_table && page_tokens > 0 && max_pages > 0 && fixed_tokens >= 0),
                "row_prepare: incomplete cache description");
    RowPrepareArgs p{proj, qkv, bias, conv, state, q_gain, k_gain, rot ? inv_freq : nullptr, row_pos, row_seq,
                     seq_slot, seq_start, seq_end, seq_row0, k_pool, v_pool, page_table, proj_stride, state_stride,
                     rows, n_heads, n_kv, kd, vd, pad, rot, taps, values_from_keys, neighbours, single,
                     max_pages, page_tokens, ring_tokens, fixed_tokens, eps, magnitude};
    cudaStream_t s = (cudaStream_t)stream;
    auto wide = [](const void* q) { return ((uintptr_t)q % 16) == 0; };
    const int channels = C + (values_from_keys ? 0 : nk);
    if (dtype == SIB_BF16 && kd == vd && kd == pad && kd % 8 == 0 && channels <= 8192 && taps <= 4 &&
        (rot == 0 || neighbours) && proj_stride % 8 == 0 && wide(proj) && wide(qkv) && wide(k_pool) && wide(v_pool) &&
        wide(bias) && wide(conv) && wide(q_gain) && wide(k_gain) && wide(state) && state_stride % 4 == 0) {
        const int threads = (channels / 8 + 31) / 32 * 32;
        // few rows: a block each; many: runs of 2, whose rows share what they read
        const int run = single || rows < 592 ? 1 : 2;
        const dim3 grid((rows + run - 1) / run);
        const size_t smem = (size_t)run * (rot / 2) * sizeof(float2) + 16;
#define GO(TAPS, RUN)                                                                                              \
    do {                                                                                                           \
        if (threads <= 256) sib_launch_chained(row_prepare_bf16_kernel<TAPS, RUN, 256, 3>, grid, dim3(threads), smem, s, p); \
        else if (threads <= 384) sib_launch_chained(row_prepare_bf16_kernel<TAPS, RUN, 384, 2>, grid, dim3(threads), smem, s, p); \
        else if (threads <= 768) sib_launch_chained(row_prepare_bf16_kernel<TAPS, RUN, 768, 1>, grid, dim3(threads), smem, s, p); \
        else sib_launch_chained(row_prepare_bf16_kernel<TAPS, RUN, 1024, 1>, grid, dim3(threads), smem, s, p);     \
    } while (0)
#define BY_RUN(TAPS)              \
    do {                          \
        if (run == 1) GO(TAPS, 1); \
        else GO(TAPS, 2);         \
    } while (0)
        if (taps == 0) BY_RUN(0);
        else if (taps == 1) BY_RUN(1);
        else if (taps == 2) BY_RUN(2);
        else if (taps == 3) BY_RUN(3);
        else BY_RUN(4);
#undef BY_RUN
#undef GO
    } else {
        const size_t smem = (size_t)C * sizeof(float);
        SIB_REQUIRE(smem <= 200 * 1024, "row_prepare: %d channels of q and k are too many", C);
        SIB_DISPATCH_DTYPE(dtype, {
            if (smem > 48 * 1024) {
                cudaError_t e = cudaFuncSetAttribute(row_prepare_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                                     (int)smem);
                SIB_REQUIRE(e == cudaSuccess, "row_prepare: %s", cudaGetErrorString(e));
            }
            sib_launch_chained(row_prepare_kernel<T>, dim3(rows), dim3(256), smem, s, p);
        });
    }
    int rc = sib_check_launch("row_prepare");
    if (rc || single || taps <= 1) return rc;
    SIB_DISPATCH_DTYPE(dtype, sib_launch_chained(row_prepare_state_kernel<T>, dim3((C + 255) / 256, n_seqs), dim3(256), 0,
                                                 s, p));
    return sib_check_launch("row_prepare_state");
}
