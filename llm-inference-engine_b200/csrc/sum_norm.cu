// sum_norm.cu -- the residual step of B200_NORM_RMS_SUM layers, x <- rmsnorm(alpha * x + sublayer(x')) * g, and the convolution over time
// that makes a sublayer's input: x'_t = x_t + sum_j w_j * x_(t - taps + 1 + j), channel by channel, zeros before position 0.
//
// The convolution's last taps - 1 inputs are state of the sequence: a ring of keep = taps - 1 rows per slot, position p in row p % keep, so
// that a row is written where it stays and nothing is shifted.  Who reads and who writes it:
//   * a token whose tap reaches before its portion reads the ring (the conv kernel, or the fused form below);
//   * the residual kernel, which replaces x (the convolution's input of that sublayer), first saves the row of every token that is among
//     the last keep of its portion.  It runs after every reader of that ring in stream order, and no two tokens share a row.
// Two forms of the convolution: in a batch of one-token portions (decoding) every tap but the token's own comes from the ring, so the
// kernel that writes x -- the residual kernel, or the embedding -- forms x' right away; otherwise conv_input_kernel follows, a thread
// holding a run of tokens of its channels in registers.
// Everything is fp32 but the row handed to the projections.
#include "hybrid_ops.cuh"

#include <algorithm>
#include <initializer_list>

namespace b200 {

template <int N> __device__ __forceinline__ void ld_f32(const float *__restrict__ p, float *v) {
    if constexpr (N == 1) {
        v[0] = p[0];
    } else {
#pragma unroll
        for (int i = 0; i < N; i += 4) {
            const float4 a = *reinterpret_cast<const float4 *>(p + i);
            v[i] = a.x, v[i + 1] = a.y, v[i + 2] = a.z, v[i + 3] = a.w;
        }
    }
}
template <int N> __device__ __forceinline__ void st_f32(float *p, const float *v) {
    if constexpr (N == 1) {
        p[0] = v[0];
    } else {
#pragma unroll
        for (int i = 0; i < N; i += 4) *reinterpret_cast<float4 *>(p + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
    }
}
// N = 1 or one 16-byte piece of T
template <typename T, int N> __device__ __forceinline__ void ld_t(const T *p, float *v) {
    if constexpr (N == 1) v[0] = Elem<T>::to_f(p[0]);
    else unpack16<T>(ld_v4(p), v);
}
template <typename T, int N> __device__ __forceinline__ void st_t(T *p, const float *v) {
    if constexpr (N == 1) p[0] = Elem<T>::from_f(v[0]);
    else st_v4(p, pack16<T>(v));
}

// x' of a one-token portion at position pos for N channels from c on: v holds x and receives x'
template <int N>
__device__ __forceinline__ void conv_from_ring(float *v, int c, int width, int pos, const float *__restrict__ ring, const float *__restrict__ w, int taps) {
    const int keep = taps - 1;
    float own[N], acc[N];
    ld_f32<N>(w + (size_t)keep * width + c, own);
#pragma unroll
    for (int i = 0; i < N; ++i) acc[i] = own[i] * v[i];
    for (int j = 0; j < keep; ++j) {
        const int p = pos - keep + j;
        if (p < 0) continue;  // before the sequence's start
        float in[N], wj[N];
        ld_f32<N>(ring + (size_t)(p % keep) * width + c, in);
        ld_f32<N>(w + (size_t)j * width + c, wj);
#pragma unroll
        for (int i = 0; i < N; ++i) acc[i] = fmaf(wj[i], in[i], acc[i]);
    }
#pragma unroll
    for (int i = 0; i < N; ++i) v[i] += acc[i];
}

// y[t, :] = y_dense[t, :], or sum_k y_rows[pair_row[t, k], :] + shared_gate[t] * y_shared[t, :]   (shared_gate NULL: 1);
// x[t, :] <- rmsnorm(alpha * x + y) * g;   trace too;   own.ring row <- the old x, for the last own.taps - 1 tokens of a portion;
// h_out (optional): next.taps == 0: T(x); one_token: T(x'), x' as the next sublayer's convolution makes it; otherwise nothing.
// One CTA per token; a thread keeps its sums in registers between the two passes when the row is short enough, else forms them again.
template <typename T, bool VEC>
__global__ void __launch_bounds__(512)
sum_norm_kernel(float *x, const T *__restrict__ y_dense, const T *__restrict__ y_rows, const int *__restrict__ pair_row, int top,
                const T *__restrict__ y_shared, const float *__restrict__ shared_gate, float alpha, const float *__restrict__ g, float eps, int width,
                float *__restrict__ trace, T *__restrict__ h_out, RingConv own, RingConv next, int one_token, PortionMap pm) {
    constexpr int N = VEC ? Elem<T>::kVec : 1, KP = VEC ? 2 : 8;
    __shared__ float red[33];
    const int t = blockIdx.x, s = pm.tok_seq[t], pos = pm.tok_pos[t];
    const int slot = pm.seq_slot[s], last = pm.seq_pos0[s] + (pm.seq_start[s + 1] - pm.seq_start[s]) - 1;
    float *xr = x + (size_t)t * width;
    const float sg = (!y_dense && y_shared && shared_gate) ? shared_gate[t] : 1.0f;
    auto total = [&](int c, float *xo, float *v) {  // xo: the old x
        ld_f32<N>(xr + c, xo);
        if (y_dense) {
            ld_t<T, N>(y_dense + (size_t)t * width + c, v);
        } else {
#pragma unroll
            for (int i = 0; i < N; ++i) v[i] = 0.0f;
            for (int k = 0; k < top; ++k) {
                float f[N];
                ld_t<T, N>(y_rows + (size_t)pair_row[(size_t)t * top + k] * width + c, f);
#pragma unroll
                for (int i = 0; i < N; ++i) v[i] += f[i];
            }
            if (y_shared) {
                float f[N];
                ld_t<T, N>(y_shared + (size_t)t * width + c, f);
#pragma unroll
                for (int i = 0; i < N; ++i) v[i] = fmaf(sg, f[i], v[i]);
            }
        }
#pragma unroll
        for (int i = 0; i < N; ++i) v[i] = fmaf(alpha, xo[i], v[i]);
    };
    float *save = nullptr;  // this token's row of the ring
    if (own.taps > 1 && pos > last - (own.taps - 1)) save = own.ring + ((size_t)slot * (own.taps - 1) + pos % (own.taps - 1)) * width;
    const bool held = width <= (int)blockDim.x * N * KP;
    float keep_v[KP][N];
    float ss = 0.0f;
    if (held) {
#pragma unroll
        for (int i = 0; i < KP; ++i) {
            const int c = (threadIdx.x + i * blockDim.x) * N;
            if (c < width) {
                float xo[N];
                total(c, xo, keep_v[i]);
                if (save) st_f32<N>(save + c, xo);
#pragma unroll
                for (int e = 0; e < N; ++e) ss = fmaf(keep_v[i][e], keep_v[i][e], ss);
            }
        }
    } else {
        for (int c = threadIdx.x * N; c < width; c += blockDim.x * N) {
            float xo[N], v[N];
            total(c, xo, v);
            if (save) st_f32<N>(save + c, xo);
#pragma unroll
            for (int e = 0; e < N; ++e) ss = fmaf(v[e], v[e], ss);
        }
    }
    const float inv = rsqrtf(block_sum(ss, red) / (float)width + eps);
    const bool conv = h_out && one_token && next.taps > 0;
    const float *ring = conv && next.taps > 1 ? next.ring + (size_t)slot * (next.taps - 1) * width : nullptr;
    auto finish = [&](int c, float *v) {
        float gv[N];
        ld_f32<N>(g + c, gv);
#pragma unroll
        for (int i = 0; i < N; ++i) v[i] *= inv * gv[i];
        st_f32<N>(xr + c, v);
        if (trace) st_f32<N>(trace + (size_t)t * width + c, v);
        if (conv) conv_from_ring<N>(v, c, width, pos, ring, next.w, next.taps);
        if (h_out && (conv || next.taps == 0)) st_t<T, N>(h_out + (size_t)t * width + c, v);
    };
    if (held) {
#pragma unroll
        for (int i = 0; i < KP; ++i) {
            const int c = (threadIdx.x + i * blockDim.x) * N;
            if (c < width) finish(c, keep_v[i]);
        }
        return;
    }
    for (int c = threadIdx.x * N; c < width; c += blockDim.x * N) {  // (a thread overwrites only the elements it reads)
        float xo[N], v[N];
        total(c, xo, v);
        finish(c, v);
    }
}

// turns[i] = base^(-2i / width) / (2 pi): turns per position of channels 2i and 2i + 1
__global__ void pos_turns_kernel(double *__restrict__ turns, int width, float base) {
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (2 * i < width) turns[i] = exp2(-2.0 * (double)i / (double)width * log2((double)base)) * 0.15915494309189533577;
}

// x[t, :] = table[id] * scale (+ the sinusoidal position vector: channels 2i, 2i + 1 receive sin, cos of p * base^(-2i / width); turns NULL:
// none); h_out as above.  The angle is taken in turns, in fp64, and only its fraction goes to fp32, so that a far position costs no bits.
// grid (tokens, channel blocks); N = 1 or 4 channels per thread.
template <typename T, int N>
__global__ void __launch_bounds__(256)
embed_pos_kernel(const int *__restrict__ ids, const T *__restrict__ table, float *__restrict__ x, T *__restrict__ h_out, int width, int vocab,
                 float scale, const double *__restrict__ turns, RingConv next, int one_token, PortionMap pm) {
    const int t = blockIdx.x, c = (blockIdx.y * blockDim.x + threadIdx.x) * N;
    if (c >= width) return;
    int id = ids[t];
    id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);  // the host has refused ids outside the vocabulary
    const int pos = pm.tok_pos[t];
    float v[N];
    load_n<T, N>(table + (size_t)id * width + c, v);
#pragma unroll
    for (int i = 0; i < N; ++i) v[i] *= scale;
    if (turns) {
#pragma unroll
        for (int i = 0; i < N; i += 2) {
            const double a = (double)pos * turns[(c + i) >> 1];
            float sn, cn;
            sincospif(2.0f * (float)(a - rint(a)), &sn, &cn);
            if constexpr (N == 1) v[0] += (c & 1) ? cn : sn;
            else v[i] += sn, v[i + 1] += cn;
        }
    }
    store_n<float, N>(x + (size_t)t * width + c, v);
    if (!h_out) return;
    if (one_token && next.taps > 0) {
        const int slot = pm.seq_slot[pm.tok_seq[t]];
        conv_from_ring<N>(v, c, width, pos, next.taps > 1 ? next.ring + (size_t)slot * (next.taps - 1) * width : nullptr, next.w, next.taps);
    } else if (next.taps > 0) {
        return;
    }
    store_n<T, N>(h_out + (size_t)t * width + c, v);
}

// h[t, :] = T(x[t, :] + conv(x)[t, :]).  grid (runs of kConvRun packed rows, channel blocks); N channels per thread.  TAPS: taps at compile
// time: a run's rows and the TAPS - 1 before it are loaded at once (independent loads) and every tap that stays inside its portion is a
// register; 0: any number, every tap reads its input again (from L1).
constexpr int kConvRun = 8;
template <typename T, int TAPS, int N>
__global__ void __launch_bounds__(256)
conv_input_kernel(const float *__restrict__ x, T *__restrict__ h, int width, int tokens, RingConv cv, PortionMap pm) {
    const int c = (blockIdx.y * blockDim.x + threadIdx.x) * N;
    if (c >= width) return;
    const int taps = TAPS > 0 ? TAPS : cv.taps, keep = taps - 1;
    const int t0 = blockIdx.x * kConvRun, t1 = min(tokens, t0 + kConvRun);
    // adds tap `back` tokens ago of packed row t, read from where it is: its own portion's row, the ring, or nowhere
    auto add_earlier = [&](int t, int pos, int pos0, int slot, int back, const float *wj, float *acc) {
        const int p = pos - back;
        if (p < 0) return;
        float in[N];
        load_n<float, N>((p >= pos0 ? x + (size_t)(t - back) * width : cv.ring + ((size_t)slot * keep + p % keep) * width) + c, in);
#pragma unroll
        for (int i = 0; i < N; ++i) acc[i] = fmaf(wj[i], in[i], acc[i]);
    };
    if constexpr (TAPS > 1) {
        constexpr int K = TAPS - 1;
        float rows[K + kConvRun][N], wt[TAPS][N];
#pragma unroll
        for (int r = 0; r < K + kConvRun; ++r) load_n<float, N>(x + (size_t)min(max(t0 - K + r, 0), tokens - 1) * width + c, rows[r]);
#pragma unroll
        for (int j = 0; j < TAPS; ++j) load_n<float, N>(cv.w + (size_t)j * width + c, wt[j]);
#pragma unroll
        for (int r = 0; r < kConvRun; ++r) {
            const int t = t0 + r;
            if (t >= t1) break;
            const int s = pm.tok_seq[t], pos = pm.tok_pos[t], pos0 = pm.seq_pos0[s];
            float acc[N];
#pragma unroll
            for (int i = 0; i < N; ++i) acc[i] = wt[K][i] * rows[K + r][i];
            if (pos - K >= pos0) {  // (the whole CTA agrees: it works on one token)
#pragma unroll
                for (int j = 0; j < K; ++j)
#pragma unroll
                    for (int i = 0; i < N; ++i) acc[i] = fmaf(wt[j][i], rows[r + j][i], acc[i]);
            } else {
                const int slot = pm.seq_slot[s];
#pragma unroll
                for (int j = 0; j < K; ++j) add_earlier(t, pos, pos0, slot, K - j, wt[j], acc);
            }
#pragma unroll
            for (int i = 0; i < N; ++i) acc[i] += rows[K + r][i];
            store_n<T, N>(h + (size_t)t * width + c, acc);
        }
    } else {
        for (int t = t0; t < t1; ++t) {
            const int s = pm.tok_seq[t], pos = pm.tok_pos[t], pos0 = pm.seq_pos0[s], slot = pm.seq_slot[s];
            float xv[N], w[N], acc[N];
            load_n<float, N>(x + (size_t)t * width + c, xv);
            load_n<float, N>(cv.w + (size_t)keep * width + c, w);
#pragma unroll
            for (int i = 0; i < N; ++i) acc[i] = w[i] * xv[i];
            for (int j = 0; j < keep; ++j) {
                load_n<float, N>(cv.w + (size_t)j * width + c, w);
                add_earlier(t, pos, pos0, slot, keep - j, w, acc);
            }
#pragma unroll
            for (int i = 0; i < N; ++i) acc[i] += xv[i];
            store_n<T, N>(h + (size_t)t * width + c, acc);
        }
    }
}

int launch_sum_norm(int dtype, float *x, const void *y_dense, const void *y_rows, const int *pair_row, int top, const void *y_shared,
                    const float *shared_gate, float alpha, const float *g, float eps, int width, float *trace, void *h_out, RingConv own, RingConv next,
                    int one_token, PortionMap pm, int tokens, cudaStream_t st) {
    if (tokens == 0) return B200_OK;
    B200_DISPATCH_DTYPE(dtype, {
        const bool vec = width % Elem<T>::kVec == 0 && all_aligned16({x, y_dense, y_rows, y_shared, g, trace, h_out, own.ring, next.ring, next.w});
        const int per = vec ? Elem<T>::kVec : 1;
        const int threads = std::min(512, std::max(32, ((width + per - 1) / per + 31) / 32 * 32));
        auto kern = vec ? sum_norm_kernel<T, true> : sum_norm_kernel<T, false>;
        kern<<<tokens, threads, 0, st>>>(x, (const T *)y_dense, (const T *)y_rows, pair_row, top, (const T *)y_shared, shared_gate, alpha, g, eps, width,
                                         trace, (T *)h_out, own, next, one_token, pm);
    });
    return cuda_status("sum_norm launch");
}

int launch_pos_turns(double *turns, int width, float base, cudaStream_t st) {
    pos_turns_kernel<<<(width + 511) / 512, 256, 0, st>>>(turns, width, base);
    return cuda_status("pos_turns launch");
}

int launch_embed_pos(int dtype, const int *ids, const void *table, float *x, void *h_out, int width, int vocab, float scale, const double *turns,
                     RingConv next, int one_token, PortionMap pm, int tokens, cudaStream_t st) {
    if (tokens == 0) return B200_OK;
    B200_DISPATCH_DTYPE(dtype, {
        const bool vec = width % 4 == 0 && all_aligned16({table, x, h_out, next.ring, next.w});
        const int cols = vec ? width / 4 : width;
        const int threads = std::min(256, (cols + 31) / 32 * 32);
        auto kern = vec ? embed_pos_kernel<T, 4> : embed_pos_kernel<T, 1>;
        kern<<<dim3(tokens, (cols + threads - 1) / threads), threads, 0, st>>>(ids, (const T *)table, x, (T *)h_out, width, vocab, scale, turns, next,
                                                                               one_token, pm);
    });
    return cuda_status("embed_pos launch");
}

template <typename T, int TAPS>
static void launch_conv_taps(const float *x, void *h, int width, RingConv cv, PortionMap pm, int tokens, cudaStream_t st) {
    const bool vec = width % 4 == 0 && all_aligned16({x, h, cv.ring, cv.w});
    const int cols = vec ? width / 4 : width;
    const int threads = std::min(256, (cols + 31) / 32 * 32);
    const dim3 grid((tokens + kConvRun - 1) / kConvRun, (cols + threads - 1) / threads);
    auto kern = vec ? conv_input_kernel<T, TAPS, 4> : conv_input_kernel<T, TAPS, 1>;
    kern<<<grid, threads, 0, st>>>(x, (T *)h, width, tokens, cv, pm);
}

int launch_conv_input(int dtype, const float *x, void *h, int width, RingConv cv, PortionMap pm, int tokens, cudaStream_t st) {
    if (tokens == 0) return B200_OK;
    B200_DISPATCH_DTYPE(dtype, {
        switch (cv.taps) {
            case 2: launch_conv_taps<T, 2>(x, h, width, cv, pm, tokens, st); break;
            case 3: launch_conv_taps<T, 3>(x, h, width, cv, pm, tokens, st); break;
            case 4: launch_conv_taps<T, 4>(x, h, width, cv, pm, tokens, st); break;
            default: launch_conv_taps<T, 0>(x, h, width, cv, pm, tokens, st); break;
        }
    });
    return cuda_status("conv_input launch");
}

}  // namespace b200
