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
//   row_prepare          a block per row (or per run of rows), the row in shared memory or in registers;
//                        steps of one row per sequence move the state on in the same launch
//                        steps of prompts leave it as their last rows pass
//   row_prepare_state    the state after any other step, in a launch of its own behind it
//
// Rows of a sequence that holds no slot (slot -1, fillers of a recorded step) see zeros before
// their own rows and leave nothing behind.
// Plain counterpart: tests/plain_simetar.py attention().
#include "common.cuh"

namespace {

constexpr int MAX_RUN = 32;        // the most rows of a block

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
    int fresh;                 // every sequence begins in this step: no history is read, and the last rows
                               // of each leave theirs (else, unless `single`, row_prepare_state does)
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
    const int left = p.seq_end[b] - 1 - pos;                 // rows of the sequence behind this one
    const long long cell = cell_of_row(p, pos, b, slot);
    pdl_wait();
    const T* src = (const T*)p.proj + (size_t)r * p.proj_stride;
    float* state = p.taps > 1 && slot >= 0 ? p.state + (size_t)slot * p.state_stride : nullptr;
    const float* hist = p.fresh ? nullptr : state;
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
            if (p.fresh && state) {
                if (left < p.taps - 1) state[(size_t)(p.taps - 2 - left) * C + c] = own;
            } else if (p.single && state) {
                for (int k = 0; k < p.taps - 1; ++k)
                    state[(size_t)k * C + c] = k + 1 < p.taps - 1 ? state[(size_t)(k + 1) * C + c] : own;
            }
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
// up, neighbouring pairs.  q and k are normed apart, so blockIdx.x's first part takes a row's q
// channels, its second the k channels (and the values that are made of them), its third the v
// channels that a mixer has beside them.  A thread owns 8 neighbouring channels and walks the `run`
// rows of its block: the next row is on its way while one is worked on, a row's shares of the next
// TAPS - 1 rows' sums are added up in registers as it passes, so that it is unpacked once, and a row
// costs one barrier.  Where the rows are stored, their cosines and sines, the taps and (SINGLE: one
// row of each sequence) the history are fetched ahead of the wait for the projection: positions
// and tables are written by the host before the step, the history by an earlier step.
// TAPS 0: no convolution.
template <int TAPS, bool SINGLE, int THREADS, int BLOCKS>
__global__ void __launch_bounds__(THREADS, BLOCKS) row_prepare_bf16_kernel(RowPrepareArgs p, int run, int roles) {
    constexpr int BACK = TAPS > 1 ? TAPS - 1 : 0;          // rows before its own that a row reads
    constexpr int HELD = BACK > 0 ? BACK : 1;
    __shared__ __align__(16) float sums[2][32];            // [row & 1][warp]
    __shared__ long long cells[MAX_RUN];       // the rows' cells of kv head 0, or -1
    __shared__ int slots[MAX_RUN], backs[MAX_RUN], seqs[MAX_RUN], lefts[MAX_RUN];
    extern __shared__ float4 turns[];          // [run][2][groups]: (cos, sin) of a thread's 4 pairs, 2 and 2
    pdl_trigger();
    const int nq = p.n_heads * p.kd, nk = p.n_kv * p.kd, C = nq + nk;
    const int units = p.n_heads + 2 * p.n_kv;
    const int role = blockIdx.x % roles;       // 0: q, 1: k, 2: v of its own
    const bool is_q = role == 0, is_v = role == 2;
    const int width = is_q ? nq : nk, c0 = is_q ? 0 : is_v ? C : nq;
    const int lc = 8 * threadIdx.x, c = c0 + lc;           // the thread's first channel of the projected row
    const bool live = lc < width;
    const int r0 = (blockIdx.x / roles) * run, n_rows = min(run, p.rows - r0);
    const int groups = p.inv_freq && !is_v ? (p.rot + 7) / 8 : 0;
    if ((int)threadIdx.x < n_rows) {
        const int r = r0 + threadIdx.x, pos = p.row_pos[r], b = p.row_seq[r], slot = p.seq_slot[b];
        cells[threadIdx.x] = is_q ? -1 : cell_of_row(p, pos, b, slot);
        slots[threadIdx.x] = slot;
        backs[threadIdx.x] = pos - p.seq_start[b];
        seqs[threadIdx.x] = b;
        lefts[threadIdx.x] = p.seq_end[b] - 1 - pos;       // rows of the sequence behind this one
    }
    for (int i = threadIdx.x; i < 64; i += blockDim.x) (&sums[0][0])[i] = 0.f;      // (warps that are not there)
    for (int i = threadIdx.x; i < n_rows * groups * 4; i += blockDim.x) {
        const int k = i / (groups * 4), pair = i - k * groups * 4;
        float2 t = make_float2(1.f, 0.f);      // (pairs behind the rotated ones pass)
        if (2 * pair < p.rot) {
            const float ang = (float)p.row_pos[r0 + k] * p.inv_freq[pair];
            t = make_float2(cosf(ang) * p.magnitude, sinf(ang) * p.magnitude);
        }
        reinterpret_cast<float2*>(turns + (size_t)(2 * k + ((pair >> 1) & 1)) * groups + (pair >> 2))[pair & 1] = t;
    }
    const bool conv = TAPS > 0 && live && !is_v;
    float bias[8], gain[8], w[TAPS > 0 ? TAPS : 1][8];
#pragma unroll
    for (int e = 0; e < 8; ++e) { bias[e] = 0.f; gain[e] = 1.f; }
    if (live && p.bias) load8(p.bias + c, bias);
    if (live && p.q_gain && !is_v) load8((is_q ? p.q_gain : p.k_gain) + lc, gain);
    if (conv) {
#pragma unroll
        for (int j = 0; j < TAPS; ++j) load8(p.conv + (size_t)j * C + c, w[j]);
    }
    const float inv_n = 1.0f / (float)width;
    const int head = lc / p.kd, d0 = lc - head * p.kd;     // the thread's head and its place there
    const bool rotates = d0 < 8 * groups;
    // where the thread's 8 values go in a pool behind a row's cell
    const size_t head_at = (size_t)head * p.page_tokens * p.pad + d0;
    __syncthreads();
    auto state_of = [&](int slot) {
        return BACK > 0 && slot >= 0 ? p.state + (size_t)slot * p.state_stride + c : nullptr;
    };
    float past[HELD][8];                       // the input d + 1 positions back
    // what the rows passed so far add to the next row's sum, the one behind it, ...
    float ahead[HELD][8];
    auto look_ahead = [&]() {
#pragma unroll
        for (int f = 0; f < BACK; ++f)
#pragma unroll
            for (int e = 0; e < 8; ++e) {
                ahead[f][e] = 0.f;
#pragma unroll
                for (int d = 0; d + f < BACK; ++d) ahead[f][e] += w[TAPS > 1 ? TAPS - 2 - d - f : 0][e] * past[d][e];
            }
    };
    if (SINGLE && conv) {
        const float* hist = state_of(slots[0]);
#pragma unroll
        for (int d = 0; d < BACK; ++d) {
#pragma unroll
            for (int e = 0; e < 8; ++e) past[d][e] = 0.f;
            if (hist) load8(hist + (size_t)(BACK - 1 - d) * C, past[d]);
        }
        look_ahead();
    }
    pdl_wait();
    const __nv_bfloat16* src = (const __nv_bfloat16*)p.proj + (size_t)r0 * p.proj_stride + c;
    uint4 next = live ? *reinterpret_cast<const uint4*>(src) : make_uint4(0, 0, 0, 0);
    auto input = [&](const uint4& raw, float (&u)[8]) {
        unpack8(raw, u);
#pragma unroll
        for (int e = 0; e < 8; ++e) u[e] += bias[e];
    };
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = (width / 8 + 31) >> 5;
    __nv_bfloat16* dst = (__nv_bfloat16*)p.qkv + (size_t)r0 * units * p.pad + c;
#pragma unroll 1
    for (int k = 0; k < n_rows; ++k, dst += (size_t)units * p.pad) {
        const uint4 raw = next;
        if (!SINGLE && live && k + 1 < n_rows)
            next = *reinterpret_cast<const uint4*>(src + (size_t)(k + 1) * p.proj_stride);
        float x[8];
        input(raw, x);
        if (conv) {
            if (SINGLE) {
                float* hist = state_of(slots[0]);
                if (BACK > 0 && hist) {        // one position on
                    store8(hist + (size_t)(BACK - 1) * C, x);
#pragma unroll
                    for (int d = 0; d + 1 < BACK; ++d) store8(hist + (size_t)(BACK - 2 - d) * C, past[d]);
                }
            } else if (BACK > 0 && (k == 0 || seqs[k] != seqs[k - 1])) {
                // the block's first row of a sequence: what lies before it, from the step's rows or the state
                const int back = backs[k];     // rows of this step before this one
                const float* hist = p.fresh ? nullptr : state_of(slots[k]);
#pragma unroll
                for (int d = 0; d < BACK; ++d) {
                    if (d < back) {
                        input(*reinterpret_cast<const uint4*>(src + (long long)(k - d - 1) * p.proj_stride), past[d]);
                    } else {
#pragma unroll
                        for (int e = 0; e < 8; ++e) past[d][e] = 0.f;
                        if (hist) load8(hist + (size_t)(BACK - 1 + back - d) * C, past[d]);
                    }
                }
                look_ahead();
            }
            if (!SINGLE && BACK > 0 && p.fresh && lefts[k] < BACK) {
                float* state = state_of(slots[k]);
                if (state) store8(state + (size_t)(BACK - 1 - lefts[k]) * C, x);
            }
            float y[8];
#pragma unroll
            for (int e = 0; e < 8; ++e) {
                y[e] = w[TAPS > 0 ? TAPS - 1 : 0][e] * x[e];
                if (BACK > 0) y[e] += ahead[0][e];
#pragma unroll
                for (int f = 0; f < BACK; ++f)
                    ahead[f][e] = w[TAPS > 1 ? TAPS - 2 - f : 0][e] * x[e] + (f + 1 < BACK ? ahead[f + 1 < BACK ? f + 1 : 0][e] : 0.f);
            }
#pragma unroll
            for (int e = 0; e < 8; ++e) x[e] = y[e];
        }
        const long long cell = cells[k];
        if (live && (is_v || (!is_q && p.values_from_keys))) {
            const uint4 v = pack8(x);
            *reinterpret_cast<uint4*>(dst + (is_v ? 0 : nk)) = v;
            if (cell >= 0) *reinterpret_cast<uint4*>((__nv_bfloat16*)p.v_pool + cell + head_at) = v;
        }
        if (is_v) continue;                    // (the same for the whole block)
        if (p.q_gain) {
            float t = 0.f;
            if (live) {
#pragma unroll
                for (int e = 0; e < 8; ++e) t += x[e] * x[e];
            }
            t = warp_sum(t);
            if (lane == 0) sums[k & 1][warp] = t;
            __syncthreads();                   // (two rows' sums in turn: one barrier a row is enough)
            float total = 0.f;
            for (int i = 0; i < n_warps; i += 4) {
                const float4 f = *reinterpret_cast<const float4*>(&sums[k & 1][i]);
                total += (f.x + f.y) + (f.z + f.w);
            }
            const float inv = rsqrtf(total * inv_n + p.eps);
#pragma unroll
            for (int e = 0; e < 8; ++e) x[e] = x[e] * inv * gain[e];
        }
        if (live) {
            if (rotates) {
                const float4 lo = turns[(size_t)2 * k * groups + d0 / 8], hi = turns[(size_t)(2 * k + 1) * groups + d0 / 8];
                const float cs[8] = {lo.x, lo.y, lo.z, lo.w, hi.x, hi.y, hi.z, hi.w};
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const float u = x[2 * i], v = x[2 * i + 1];
                    x[2 * i] = u * cs[2 * i] - v * cs[2 * i + 1];
                    x[2 * i + 1] = v * cs[2 * i] + u * cs[2 * i + 1];
                }
            }
            const uint4 y = pack8(x);
            *reinterpret_cast<uint4*>(dst) = y;
            if (cell >= 0) *reinterpret_cast<uint4*>((__nv_bfloat16*)p.k_pool + cell + head_at) = y;
        }
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

// `single`: every sequence of the step has exactly one row.  `fresh`: every sequence begins in this
// step, with a state of zeros.  `taps` 0: no convolution.
SIB_EXPORT int sib_row_prepare(
    const void* proj, long long proj_stride, void* qkv, int dtype, const float* bias, const float* conv, int taps,
    float* state, long long state_stride, const float* q_gain, const float* k_gain, float eps,
    const float* inv_freq, int rot, int neighbours, float magnitude, const int* row_pos, const int* row_seq,
    const int* seq_slot, const int* seq_start, const int* seq_end, const int* seq_row0, void* k_pool, void* v_pool,
    const int* page_table, int max_pages, int page_tokens, int ring_tokens, int fixed_tokens, int rows, int n_seqs,
    int n_heads, int n_kv, int kd, int vd, int pad, int values_from_keys, int single,
    int fresh, void* stream) {
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
                     rows, n_heads, n_kv, kd, vd, pad, rot, taps, values_from_keys, neighbours, single, fresh,
                     max_pages, page_tokens, ring_tokens, fixed_tokens, eps, magnitude};
    cudaStream_t s = (cudaStream_t)stream;
    auto wide = [](const void* q) { return ((uintptr_t)q % 16) == 0; };
    if (dtype == SIB_BF16 && kd == vd && kd == pad && kd % 8 == 0 && nq <= 8192 && nk <= 8192 && taps <= 4 && rows < (1 << 28) &&
        (rot == 0 || neighbours) && proj_stride % 8 == 0 && wide(proj) && wide(qkv) && wide(k_pool) && wide(v_pool) &&
        wide(bias) && wide(conv) && wide(q_gain) && wide(k_gain) && wide(state) && state_stride % 4 == 0) {
        const int threads = ((nq > nk ? nq : nk) / 8 + 31) / 32 * 32;
        const int roles = values_from_keys ? 2 : 3;
        // as many rows a block as spread them over the SMs in one wave (two blocks an SM up to 256 threads)
        const int blocks = 148 * (threads <= 256 ? 2 : 1) / roles, even = (rows + blocks - 1) / blocks;
        const size_t row_bytes = (size_t)2 * ((rot + 7) / 8) * sizeof(float4);
        int run = single ? 1 : even < MAX_RUN ? even : MAX_RUN;
        while (run > 1 && run * row_bytes > 40 * 1024) --run;
        const dim3 grid((unsigned)((rows + run - 1) / run) * roles);
        const size_t smem = run * row_bytes + 16;
#define GO(TAPS, SINGLE, THREADS, BLOCKS)                                                                          \
    sib_launch_chained(row_prepare_bf16_kernel<TAPS, SINGLE, THREADS, BLOCKS>, grid, dim3(threads), smem, s, p, run, roles)
#define BY_STEP(TAPS)                                         \
    do {                                                      \
        if (single && threads <= 512) GO(TAPS, true, 512, 1); \
        else if (single) GO(TAPS, true, 1024, 1);             \
        else if (threads <= 256) GO(TAPS, false, 256, 2);     \
        else if (threads <= 512) GO(TAPS, false, 512, 1);     \
        else GO(TAPS, false, 1024, 1);                        \
    } while (0)
        if (taps == 0) BY_STEP(0);
        else if (taps == 1) BY_STEP(1);
        else if (taps == 2) BY_STEP(2);
        else if (taps == 3) BY_STEP(3);
        else BY_STEP(4);
#undef BY_STEP
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
    if (rc || single || fresh || taps <= 1) return rc;
    SIB_DISPATCH_DTYPE(dtype, sib_launch_chained(row_prepare_state_kernel<T>, dim3((C + 255) / 256, n_seqs), dim3(256), 0,
                                                 s, p));
    return sib_check_launch("row_prepare_state");
}
