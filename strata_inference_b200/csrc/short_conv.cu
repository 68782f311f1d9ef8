// A short causal convolution over time on each channel of a mixer's input, added to the input:
//
//     y[t, c] = x[t, c] + sum_j w[j, c] x[t - taps + 1 + j, c]       (zeros before position 0)
//
// x: the step's normed rows; earlier steps' last taps - 1 rows of each sequence are per-slot
// state, 32-bit, oldest first: state[slot] = [taps - 1][channels].  Sums are 32-bit.
//
//   short_conv        any step: every row reads its taps - 1 predecessors from the step's rows or
//                     from the state, then (its own launch, behind it) the state is brought to
//                     the step's end.  Steps of one row per sequence move the state on in the same launch.
//   add_norm_conv     steps of one row per sequence: the residual step ahead of the mixer and this
//                     convolution as one launch,
//                         h += rms(a) post_gain;  x = rms(h) pre_gain;  y as above
//                     with a thread per 8 channels, the row in registers (csrc/norm.cu's
//                     group kernel), the state's rows asked for before the kernel ahead has finished.
//
// Rows of a sequence that holds no slot (slot -1, fillers of a recorded step) see zeros
// before their own rows and leave nothing behind.
//
// Plain counterpart: tests/plain_kerolorn.py causal_conv().
#include "common.cuh"

namespace {

struct ConvArgs {
    const float* w;            // [taps, channels]
    float* state;              // [slots, state_stride]
    long long state_stride;
    const int* row_pos;
    const int* row_seq;
    const int* seq_slot;
    const int* seq_start;
    const int* seq_end;
    const int* seq_row0;
    int rows, channels, taps;
};

template <typename T> struct Pack;      // V neighbouring channels as one 16-byte access
template <> struct Pack<float> {
    static constexpr int V = 4;
    __device__ static void load(const float* p, float (&o)[4]) {
        const float4 v = *reinterpret_cast<const float4*>(p);
        o[0] = v.x; o[1] = v.y; o[2] = v.z; o[3] = v.w;
    }
    __device__ static void store(float* p, const float (&o)[4]) {
        *reinterpret_cast<float4*>(p) = make_float4(o[0], o[1], o[2], o[3]);
    }
};
template <> struct Pack<__nv_bfloat16> {
    static constexpr int V = 8;
    __device__ static void load(const __nv_bfloat16* p, float (&o)[8]) {
        const uint4 v = *reinterpret_cast<const uint4*>(p);
        const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            o[2 * i] = __uint_as_float(w[i] << 16);
            o[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
        }
    }
    __device__ static void store(__nv_bfloat16* p, const float (&o)[8]) {
        uint32_t w[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const __nv_bfloat162 pr = __floats2bfloat162_rn(o[2 * i], o[2 * i + 1]);
            w[i] = *reinterpret_cast<const uint32_t*>(&pr);
        }
        *reinterpret_cast<uint4*>(p) = make_uint4(w[0], w[1], w[2], w[3]);
    }
};

// A thread takes V channels of RUN neighbouring rows (V 1: any layout).  SINGLE: every sequence
// has one row, and the thread that read a slot's state moves it on.  TAPS > 0 (= p.taps): a run
// inside one sequence whose first row has all its predecessors in this step asks for its rows
// at once and goes from row to row in registers.
template <typename T, int V, int RUN, bool SINGLE, int TAPS = 0>
__global__ void __launch_bounds__(128)
short_conv_kernel(const T* __restrict__ x, T* __restrict__ y, ConvArgs p) {
    pdl_trigger();
    pdl_wait();
    const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V;
    if (c >= p.channels) return;
    const int C = p.channels, taps = p.taps;
    const int r0 = blockIdx.y * RUN, r1 = min(r0 + RUN, p.rows);
    if constexpr (TAPS > 0 && V > 1 && !SINGLE) {
        const int b0 = p.row_seq[r0];
        if (r0 + RUN <= p.rows && p.row_seq[r0 + RUN - 1] == b0 && p.row_pos[r0] - p.seq_start[b0] >= TAPS - 1) {
            float in[RUN + TAPS - 1][V];
#pragma unroll
            for (int k = 0; k < RUN + TAPS - 1; ++k) Pack<T>::load(x + (size_t)(r0 - (TAPS - 1) + k) * C + c, in[k]);
            float acc[RUN][V];
#pragma unroll
            for (int q = 0; q < RUN; ++q)
#pragma unroll
                for (int i = 0; i < V; ++i) acc[q][i] = in[q + TAPS - 1][i];
#pragma unroll
            for (int j = TAPS - 1; j >= 0; --j)
#pragma unroll
                for (int i = 0; i < V; ++i) {
                    const float w = p.w[(size_t)j * C + c + i];
#pragma unroll
                    for (int q = 0; q < RUN; ++q) acc[q][i] += w * in[q + j][i];
                }
#pragma unroll
            for (int q = 0; q < RUN; ++q) Pack<T>::store(y + (size_t)(r0 + q) * C + c, acc[q]);
            return;
        }
    }
    for (int r = r0; r < r1; ++r) {
        const int b = p.row_seq[r], slot = p.seq_slot[b];
        const int back = p.row_pos[r] - p.seq_start[b];          // rows of this step before this one
        float* hist = slot >= 0 ? p.state + (size_t)slot * p.state_stride : nullptr;
        float own[V], acc[V], v[V];
        auto fetch = [&](const T* from) {
            if constexpr (V == 1) v[0] = to_f32(*from);
            else Pack<T>::load(from, v);
        };
        fetch(x + (size_t)r * C + c);
#pragma unroll
        for (int i = 0; i < V; ++i) {
            own[i] = v[i];
            acc[i] = v[i] + p.w[(size_t)(taps - 1) * C + c + i] * v[i];
        }
        for (int j = taps - 2; j >= 0; --j) {
            const int d = taps - 1 - j;                          // the input d positions back
            if (d <= back) {
                fetch(x + (size_t)(r - d) * C + c);
            } else if (hist) {
                const float* from = hist + (size_t)(taps - 1 + back - d) * C + c;
#pragma unroll
                for (int i = 0; i < V; ++i) v[i] = from[i];
            } else {
                break;                                           // (zeros from here on)
            }
#pragma unroll
            for (int i = 0; i < V; ++i) acc[i] += p.w[(size_t)j * C + c + i] * v[i];
        }
        if constexpr (V == 1) y[(size_t)r * C + c] = from_f32<T>(acc[0]);
        else Pack<T>::store(y + (size_t)r * C + c, acc);
        if (SINGLE && hist)
            for (int k = 0; k < taps - 1; ++k)
#pragma unroll
                for (int i = 0; i < V; ++i)
                    hist[(size_t)k * C + c + i] = k + 1 < taps - 1 ? hist[(size_t)(k + 1) * C + c + i] : own[i];
    }
}

// The state after the step: the last taps - 1 inputs of each sequence.  One thread per (sequence,
// channel), oldest first: a cell that keeps an older input takes it from a later cell of the
// same state, which has not been rewritten yet.
template <typename T>
__global__ void __launch_bounds__(256) short_conv_state_kernel(const T* __restrict__ x, ConvArgs p) {
    pdl_trigger();
    pdl_wait();
    const int b = blockIdx.y, slot = p.seq_slot[b];
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    if (slot < 0 || c >= p.channels) return;
    const int n = p.seq_end[b] - p.seq_start[b], row0 = p.seq_row0[b];
    float* hist = p.state + (size_t)slot * p.state_stride;
    for (int i = 0; i < p.taps - 1; ++i) {
        const int back = p.taps - 1 - i;             // the input `back` positions before the end
        hist[(size_t)i * p.channels + c] = back <= n ? to_f32(x[(size_t)(row0 + n - back) * p.channels + c])
                                                     : hist[(size_t)(i + n) * p.channels + c];
    }
}

// One block per row, 8 channels a thread.  HELD: how many of the state's rows are asked for at
// the start (taps - 1 when it is that small and the block leaves the registers for it, else 0:
// each is read where it is used).
// (a, h and y are not marked __restrict__: the compiler may move a load through such a pointer
// ahead of the wait for the kernel that writes there.)
template <int HELD, int THREADS>
__global__ void __launch_bounds__(THREADS)
add_norm_conv_kernel(const __nv_bfloat16* a, const float* __restrict__ post_gain, float post_eps,
                     float* h, const float* __restrict__ pre_gain, float pre_eps,
                     __nv_bfloat16* y, ConvArgs p) {
    __shared__ float scratch[33];
    pdl_trigger();
    const int hidden = p.channels, taps = p.taps, r = blockIdx.x;
    const int c = 8 * threadIdx.x;
    const bool live = c < hidden;
    auto load8 = [](const float* from, float (&o)[8]) {
        const float4 lo = *reinterpret_cast<const float4*>(from), hi = *reinterpret_cast<const float4*>(from + 4);
        o[0] = lo.x; o[1] = lo.y; o[2] = lo.z; o[3] = lo.w;
        o[4] = hi.x; o[5] = hi.y; o[6] = hi.z; o[7] = hi.w;
    };
    auto store8 = [](float* to, const float (&o)[8]) {
        *reinterpret_cast<float4*>(to) = make_float4(o[0], o[1], o[2], o[3]);
        *reinterpret_cast<float4*>(to + 4) = make_float4(o[4], o[5], o[6], o[7]);
    };
    const int slot = p.seq_slot[p.row_seq[r]];
    float* hist = slot >= 0 ? p.state + (size_t)slot * p.state_stride + c : nullptr;
    float pg[8], qg[8], own_w[8], held[HELD > 0 ? HELD : 1][8];
#pragma unroll
    for (int e = 0; e < 8; ++e) pg[e] = qg[e] = own_w[e] = 0.f;
    if (live) {
        if (post_gain) load8(post_gain + c, pg);
        load8(pre_gain + c, qg);
        load8(p.w + (size_t)(taps - 1) * hidden + c, own_w);
        // (the state's rows were written by an earlier step, not by the kernel ahead of this one)
#pragma unroll
        for (int k = 0; k < HELD; ++k)
            if (hist) load8(hist + (size_t)k * hidden, held[k]);
    }
    pdl_wait();
    const size_t base = (size_t)r * hidden + c;
    float v[8], s[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] = s[e] = 0.f;
    if (live) {
        Pack<__nv_bfloat16>::load(a + base, v);
        load8(h + base, s);
    }
    if (post_gain) {
        float ss = 0.f;
#pragma unroll
        for (int e = 0; e < 8; ++e) ss += v[e] * v[e];
        ss = block_sum(ss, scratch);
        const float inv = 1.0f / sqrtf(ss / (float)hidden + post_eps);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] *= inv * pg[e];
    }
    float ss2 = 0.f;
#pragma unroll
    for (int e = 0; e < 8; ++e) {
        s[e] += v[e];
        ss2 += s[e] * s[e];
    }
    if (live) store8(h + base, s);
    ss2 = block_sum(ss2, scratch);
    const float inv2 = 1.0f / sqrtf(ss2 / (float)hidden + pre_eps);
    if (!live) return;
    float x[8], acc[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) {
        x[e] = __bfloat162float(__float2bfloat16_rn(s[e] * inv2 * qg[e]));     // as a normed row is kept
        acc[e] = x[e] + own_w[e] * x[e];
    }
    if (hist) {
        if constexpr (HELD > 0) {
#pragma unroll
            for (int j = HELD - 1; j >= 0; --j) {
                float w[8];
                load8(p.w + (size_t)j * hidden + c, w);
#pragma unroll
                for (int e = 0; e < 8; ++e) acc[e] += w[e] * held[j][e];
                if (j > 0) store8(hist + (size_t)(j - 1) * hidden, held[j]);
            }
        } else {
            for (int j = taps - 2; j >= 0; --j) {
                float old[8], w[8];
                load8(p.w + (size_t)j * hidden + c, w);
                load8(hist + (size_t)j * hidden, old);
#pragma unroll
                for (int e = 0; e < 8; ++e) acc[e] += w[e] * old[e];
            }
            for (int k = 0; k + 1 < taps - 1; ++k) {
                float nx[8];
                load8(hist + (size_t)(k + 1) * hidden, nx);
                store8(hist + (size_t)k * hidden, nx);
            }
        }
        if (taps > 1) store8(hist + (size_t)(taps - 2) * hidden, x);
    }
    Pack<__nv_bfloat16>::store(y + base, acc);
}

}  // namespace

// `single`: every sequence of the step has exactly one row.
SIB_EXPORT int sib_short_conv(const void* x, void* y, int dtype, const float* w, float* state,
                              long long state_stride, const int* row_pos, const int* row_seq,
                              const int* seq_slot, const int* seq_start, const int* seq_end,
                              const int* seq_row0, int rows, int n_seqs, int channels, int taps, int single,
                              void* stream) {
    if (rows == 0) return 0;
    SIB_REQUIRE(rows > 0 && n_seqs > 0 && n_seqs < 65536 && channels > 0 && taps > 0,
                "short_conv: rows=%d sequences=%d channels=%d taps=%d", rows, n_seqs, channels, taps);
    SIB_REQUIRE(x && y && x != y && w && row_pos && row_seq && seq_slot && seq_start && seq_end && seq_row0 &&
                    (taps == 1 || (state && state_stride >= (long long)(taps - 1) * channels)),
                "short_conv: an argument is missing, or the state is too small");
    SIB_REQUIRE(!single || rows == n_seqs, "short_conv: %d rows of %d sequences are not one each", rows, n_seqs);
    ConvArgs p{w, state, state_stride, row_pos, row_seq, seq_slot, seq_start, seq_end, seq_row0, rows, channels, taps};
    cudaStream_t s = (cudaStream_t)stream;
    const int vec = dtype == SIB_F32 ? 4 : 8;
    const bool wide = channels % vec == 0 && ((uintptr_t)x % 16) == 0 && ((uintptr_t)y % 16) == 0;
    constexpr int RUN = 4;
    const int lanes = wide ? channels / vec : channels;
    const int runs = single ? rows : (rows + RUN - 1) / RUN;
    SIB_REQUIRE(runs < 65536, "short_conv: too many rows (%d)", rows);
    const dim3 grid((lanes + 127) / 128, runs);
    SIB_DISPATCH_DTYPE(dtype, {
        if (single && wide)
            sib_launch_chained(short_conv_kernel<T, Pack<T>::V, 1, true>, grid, dim3(128), 0, s, (const T*)x, (T*)y, p);
        else if (single)
            sib_launch_chained(short_conv_kernel<T, 1, 1, true>, grid, dim3(128), 0, s, (const T*)x, (T*)y, p);
        else if (wide && taps == 4)
            sib_launch_chained(short_conv_kernel<T, Pack<T>::V, RUN, false, 4>, grid, dim3(128), 0, s, (const T*)x, (T*)y, p);
        else if (wide && taps == 3)
            sib_launch_chained(short_conv_kernel<T, Pack<T>::V, RUN, false, 3>, grid, dim3(128), 0, s, (const T*)x, (T*)y, p);
        else if (wide && taps == 2)
            sib_launch_chained(short_conv_kernel<T, Pack<T>::V, RUN, false, 2>, grid, dim3(128), 0, s, (const T*)x, (T*)y, p);
        else if (wide)
            sib_launch_chained(short_conv_kernel<T, Pack<T>::V, RUN, false>, grid, dim3(128), 0, s, (const T*)x, (T*)y, p);
        else
            sib_launch_chained(short_conv_kernel<T, 1, RUN, false>, grid, dim3(128), 0, s, (const T*)x, (T*)y, p);
    });
    int rc = sib_check_launch("short_conv");
    if (rc || single || taps == 1) return rc;
    SIB_DISPATCH_DTYPE(dtype, sib_launch_chained(short_conv_state_kernel<T>, dim3((channels + 255) / 256, n_seqs),
                                                 dim3(256), 0, s, (const T*)x, p));
    return sib_check_launch("short_conv_state");
}

// 1 if add_norm_conv takes rows of this width in bfloat16.
SIB_EXPORT int sib_add_norm_conv_supports(int channels) { return channels % 8 == 0 && channels / 8 <= 1024; }

SIB_EXPORT int sib_add_norm_conv(const void* a, const float* post_gain, float post_eps, float* h,
                                 const float* pre_gain, float pre_eps, const float* w, float* state,
                                 long long state_stride, const int* row_seq, const int* seq_slot, void* y,
                                 int rows, int n_seqs, int channels, int taps, void* stream) {
    if (rows == 0) return 0;
    SIB_REQUIRE(rows > 0 && rows == n_seqs && channels > 0 && taps > 0 && sib_add_norm_conv_supports(channels),
                "add_norm_conv: rows=%d sequences=%d (one row each) channels=%d taps=%d", rows, n_seqs, channels, taps);
    SIB_REQUIRE(a && h && pre_gain && w && y && row_seq && seq_slot &&
                    (taps == 1 || (state && state_stride >= (long long)(taps - 1) * channels)),
                "add_norm_conv: an argument is missing, or the state is too small");
    SIB_REQUIRE(((uintptr_t)a % 16) == 0 && ((uintptr_t)h % 16) == 0 && ((uintptr_t)y % 16) == 0 &&
                    ((uintptr_t)post_gain % 16) == 0 && ((uintptr_t)pre_gain % 16) == 0 && ((uintptr_t)w % 16) == 0 &&
                    (taps == 1 || (((uintptr_t)state % 16) == 0 && state_stride % 4 == 0)),
                "add_norm_conv: operands must be 16-byte aligned");
    ConvArgs p{w, state, state_stride, nullptr, row_seq, seq_slot, nullptr, nullptr, nullptr, rows, channels, taps};
    const int threads = (channels / 8 + 31) / 32 * 32;
    cudaStream_t s = (cudaStream_t)stream;
#define LAUNCH(HELD, MOST)                                                                                    \
    sib_launch_chained(add_norm_conv_kernel<HELD, MOST>, dim3(rows), dim3(threads), 0, s, (const __nv_bfloat16*)a, \
                       post_gain, post_eps, h, pre_gain, pre_eps, (__nv_bfloat16*)y, p)
    if (threads > 512) LAUNCH(0, 1024);
    else if (taps == 4) LAUNCH(3, 512);
    else if (taps == 3) LAUNCH(2, 512);
    else if (taps == 2) LAUNCH(1, 512);
    else LAUNCH(0, 512);
#undef LAUNCH
    return sib_check_launch("add_norm_conv");
}
