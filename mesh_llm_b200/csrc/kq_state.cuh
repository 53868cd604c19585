// What the two prompt forms of the matrix-state recurrences share (kq_state_ops.cu, kq_state_chunk.cu): sums over lanes, the
// short convolution's inputs and its ring, the check of a call.
#pragma once
#include "kq_dense.cuh"
#include "kq_tc.cuh"

// N values of every lane summed over groups of L lanes (powers of two).  Each exchange halves the values a lane still carries:
// with p the lane's place in its group, v[i] ends as value p N / L + i (N >= L), v[0] as value p / (L / N) (N < L).
template <int N, int L>
__device__ __forceinline__ void kq_spread_sum(float (&v)[N], int lane) {
    int n = N;
#pragma unroll
    for (int m = L / 2; m >= 1; m /= 2) {
        if (n > 1) {
            n /= 2;
            const bool up = lane & m;
#pragma unroll
            for (int i = 0; i < N / 2; i++)
                if (i < n) {
                    const float send = up ? v[i] : v[i + n], keep = up ? v[i + n] : v[i];
                    v[i] = keep + __shfl_xor_sync(0xffffffffu, send, m);
                }
        } else {
            v[0] += __shfl_xor_sync(0xffffffffu, v[0], m);
        }
    }
}

// the convolution's input at position pos0 + t: this call's rows, the ring, or zero before the start
struct KqConvIn {
    const float *x; // column of row 0 of the sequence
    int64_t ld;
    const float *ring; // column of slot 0
    int64_t channels;
    int taps, pos0;
    __device__ __forceinline__ float at(int t) const {
        if (t >= 0) return x[t * ld];
        const int pos = pos0 + t;
        return pos >= 0 ? ring[(int64_t)(pos % taps) * channels] : 0.f;
    }
};

// the last `taps` inputs of every channel into the ring, shared out over all CTAs of the grid
__device__ __forceinline__ void kq_move_ring(const KqMatState &m, const KqStateIn &in, int64_t n_seq, int T, int pos0, int64_t id, int64_t n_threads) {
    const int64_t channels = kq_state_channels(m), nq = (int64_t)m.kv_heads * m.dim;
    const int keep = min(T, m.taps);
    for (int64_t i = id; i < n_seq * keep * channels; i += n_threads) {
        const int64_t c = i % channels, rest = i / channels, seq = rest / keep;
        const int t = T - keep + (int)(rest % keep);
        const float *x = c < nq ? in.q + c : c < 2 * nq ? in.k + (c - nq) : in.v + (c - 2 * nq);
        m.conv[(seq * m.taps + (pos0 + t) % m.taps) * channels + c] = x[(seq * T + t) * in.ld];
    }
}

static inline b200_status kq_check_state(const KqMatState &m, int n_seq, int T) {
    KQ_REQUIRE(m.heads >= 1 && m.kv_heads >= 1 && m.heads % m.kv_heads == 0 && m.dim >= 1 && m.vdim >= 1 && m.taps >= 0 && n_seq >= 1 && T >= 1 &&
                   m.s && (m.taps == 0 || m.conv),
               "matrix state: bad shape");
    KQ_REQUIRE(m.dim <= KQ_STATE_MAX_DIM && m.heads <= 65535 && n_seq <= 65535, "matrix state: %d heads of %d key dimensions", m.heads, m.dim);
    return B200_OK;
}
