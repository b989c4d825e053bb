// Hyper-connections: the residual stream as `S` parallel 32-bit streams.
//
// A sublayer reads u = sum_s read[s] X_s, runs on norm(u), and its output y is written back into all streams at once:
//   X_to <- sum_from mix[from][to] X_from + write[to] y.
// One kernel does what lies between two sublayers: the write of the sublayer before (its output may come as a tensor, as a
// product's K slices, with a bias, or as the un-summed outputs of a token's routed experts), the read and the norm of the next, so
// that the streams are loaded and stored once per sublayer.  All of it is 32-bit; the norm's output is rounded once.  Where every
// portion of the step is a single token the kernel also runs the sublayer's causal input convolution (h + conv(h)) from the request's
// state and moves that state on.
//
// The causal convolution for longer portions is a kernel of its own (`causal_conv_kernel`), also used without the `h +` for
// convolved projections.
#include "common.cuh"

namespace lb {

constexpr int kMaxStreams = 8;

template <typename T>
struct StreamStep {
    const float* x;        // [rows, S, dim], or [rows, dim] where all streams are still equal (from_one)
    float* x_out;          // [rows, S, dim] (may be x) or null: the new streams are not kept
    const float* mix;      // [S, S] from, to;  null: there is nothing to write
    const float* write;    // [S]
    const float* read;     // [S]
    // y, one of: a tensor [rows, dim]; partial sums of K slices; the outputs of routed experts with their weights
    const T* y;
    const float* partials;
    const float* y_bias;   // [dim], added to y (may be null)
    const float* pair_out;
    const float* pair_weight;
    const int* pair_expert;
    size_t slice_stride;
    int slices, top, experts;
    // the norm of u
    const float* norm_weight;
    float eps;
    T* h;                  // [out_rows, dim]
    const int* rows;       // out row r is row rows[r] of x and y (null: r)
    int dim, from_one;
    // input convolution of single tokens (conv_weight null: none)
    const float* conv_weight;   // [dim, taps], the last column the current token's
    T* conv_state;              // [slots, taps - 1, dim]
    const int* token_segment;
    const int* segment_slot;
    int taps, num_slots;
    int* status;
};

// V consecutive elements as 32-bit values (V = 4: one vector access).
template <int V>
__device__ __forceinline__ void load_floats(const float* source, float (&v)[V]) {
    if constexpr (V == 4) {
        const float4 raw = *reinterpret_cast<const float4*>(source);
        v[0] = raw.x, v[1] = raw.y, v[2] = raw.z, v[3] = raw.w;
    } else {
        v[0] = source[0];
    }
}
template <int V>
__device__ __forceinline__ void store_floats(float* destination, const float (&v)[V]) {
    if constexpr (V == 4) *reinterpret_cast<float4*>(destination) = make_float4(v[0], v[1], v[2], v[3]);
    else destination[0] = v[0];
}
template <int V>
__device__ __forceinline__ void load_elements(const float* source, float (&v)[V]) { load_floats<V>(source, v); }
template <int V>
__device__ __forceinline__ void load_elements(const __nv_bfloat16* source, float (&v)[V]) {
    if constexpr (V == 4) {
        const uint2 raw = *reinterpret_cast<const uint2*>(source);
        const float2 low = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
        const float2 high = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
        v[0] = low.x, v[1] = low.y, v[2] = high.x, v[3] = high.y;
    } else {
        v[0] = to_float(source[0]);
    }
}
template <int V>
__device__ __forceinline__ void store_elements(float* destination, const float (&v)[V]) { store_floats<V>(destination, v); }
template <int V>
__device__ __forceinline__ void store_elements(__nv_bfloat16* destination, const float (&v)[V]) {
    if constexpr (V == 4) {
        const __nv_bfloat162 low = __floats2bfloat162_rn(v[0], v[1]), high = __floats2bfloat162_rn(v[2], v[3]);
        uint2 packed;
        packed.x = *reinterpret_cast<const uint32_t*>(&low);
        packed.y = *reinterpret_cast<const uint32_t*>(&high);
        *reinterpret_cast<uint2*>(destination) = packed;
    } else {
        destination[0] = from_float<__nv_bfloat16>(v[0]);
    }
}

// The sublayer's output at columns d .. d + V - 1 of row `row`.
template <typename T, int V>
__device__ __forceinline__ void load_output(const StreamStep<T>& p, size_t row, int d, float (&y)[V]) {
    if (p.pair_out != nullptr) {
#pragma unroll
        for (int i = 0; i < V; ++i) y[i] = 0.0f;
        for (int k = 0; k < p.top; ++k) {   // in the order of the choice
            const size_t pair = row * p.top + k;
            const int expert = p.pair_expert[pair];
            if (expert < 0 || expert >= p.experts) continue;
            const float weight = p.pair_weight[pair];
            float part[V];
            load_floats<V>(p.pair_out + pair * p.dim + d, part);
#pragma unroll
            for (int i = 0; i < V; ++i) y[i] += weight * part[i];
        }
    } else if (p.slices > 0) {
        // as the product's own epilogue would have stored it: the slices in order, rounded to T; four slices' loads at a time
#pragma unroll
        for (int i = 0; i < V; ++i) y[i] = 0.0f;
        const float* source = p.partials + row * p.dim + d;
        for (int s = 0; s < p.slices; s += 4) {
            float part[4][V];
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                if (s + u < p.slices) load_floats<V>(source + static_cast<size_t>(s + u) * p.slice_stride, part[u]);
            }
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                if (s + u < p.slices) {
#pragma unroll
                    for (int i = 0; i < V; ++i) y[i] += part[u][i];
                }
            }
        }
#pragma unroll
        for (int i = 0; i < V; ++i) y[i] = round_to<T>(y[i]);
    } else {
        load_elements<V>(p.y + row * p.dim + d, y);
    }
    if (p.y_bias != nullptr) {
        float bias[V];
        load_floats<V>(p.y_bias + d, bias);
#pragma unroll
        for (int i = 0; i < V; ++i) y[i] += bias[i];
    }
}

// One block per output row.
constexpr int stream_step_threads(int streams) { return streams <= 4 ? 512 : 256; }   // the coefficients take registers

// MANY: launches of many rows in blocks of at most 256 threads, of which as many as registers allow share an SM.
template <typename T, int S, int V, bool MANY>
__global__ void __launch_bounds__(MANY ? 256 : stream_step_threads(S), MANY ? (S <= 4 ? 4 : 1) : 1) stream_step_kernel(const StreamStep<T> p) {
    extern __shared__ __align__(16) float shared[];
    // Launched to start early; the product after it may then ask for its weights, but not before the kernel before is done.
    wait_for_previous_kernel();
    allow_next_kernel();
    float* u_row = shared;              // dim floats: u
    float* scratch = shared + ((p.dim + 3) & ~3);   // 33 floats
    const int r = blockIdx.x;
    const size_t row = p.rows ? static_cast<size_t>(p.rows[r]) : static_cast<size_t>(r);
    float read[S], write[S], mix[S][S];
#pragma unroll
    for (int s = 0; s < S; ++s) {
        read[s] = p.read[s];
        write[s] = p.mix ? p.write[s] : 0.0f;
#pragma unroll
        for (int to = 0; to < S; ++to) mix[s][to] = p.mix ? p.mix[s * S + to] : (s == to ? 1.0f : 0.0f);
    }
    float squares = 0.0f;
    for (int d = V * threadIdx.x; d < p.dim; d += V * blockDim.x) {
        float old[S][V], u[V];
#pragma unroll
        for (int s = 0; s < S; ++s) {
            if (s == 0 || !p.from_one) load_floats<V>(p.x + (p.from_one ? row : row * S + s) * p.dim + d, old[s]);
        }
        if (p.from_one) {
#pragma unroll
            for (int s = 1; s < S; ++s) {
#pragma unroll
                for (int i = 0; i < V; ++i) old[s][i] = old[0][i];
            }
        }
#pragma unroll
        for (int i = 0; i < V; ++i) u[i] = 0.0f;
        if (p.mix != nullptr) {
            float y[V];
            load_output<T, V>(p, row, d, y);
#pragma unroll
            for (int to = 0; to < S; ++to) {
                float fresh[V];
#pragma unroll
                for (int i = 0; i < V; ++i) {
                    float sum = write[to] * y[i];
#pragma unroll
                    for (int s = 0; s < S; ++s) sum += mix[s][to] * old[s][i];
                    fresh[i] = sum;
                    u[i] += read[to] * sum;
                }
                if (p.x_out != nullptr) store_floats<V>(p.x_out + (row * S + to) * p.dim + d, fresh);
            }
        } else {
#pragma unroll
            for (int s = 0; s < S; ++s) {
#pragma unroll
                for (int i = 0; i < V; ++i) u[i] += read[s] * old[s][i];
            }
        }
        store_floats<V>(u_row + d, u);
#pragma unroll
        for (int i = 0; i < V; ++i) squares += u[i] * u[i];
    }
    const float inv = rsqrtf(block_sum(squares, scratch) / static_cast<float>(p.dim) + p.eps);
    T* state = nullptr;
    if (p.conv_weight != nullptr && p.taps > 1) {
        const int slot = p.segment_slot[p.token_segment[row]];
        if (slot >= 0 && slot < p.num_slots) state = p.conv_state + static_cast<size_t>(slot) * (p.taps - 1) * p.dim;
        else if (threadIdx.x == 0) report_error(p.status, kBadSlot);
    }
    for (int d = V * threadIdx.x; d < p.dim; d += V * blockDim.x) {   // each thread rereads what it wrote
        float u[V], w[V], h[V];
        load_floats<V>(u_row + d, u);
        load_floats<V>(p.norm_weight + d, w);
#pragma unroll
        for (int i = 0; i < V; ++i) h[i] = u[i] * inv * w[i];
        if (p.conv_weight != nullptr) {
            float sum[V], now[V], next[V];
#pragma unroll
            for (int i = 0; i < V; ++i) now[i] = h[i] = round_to<T>(h[i]), sum[i] = 0.0f;
            for (int j = 0; j + 1 < p.taps; ++j) {
#pragma unroll
                for (int i = 0; i < V; ++i) next[i] = 0.0f;
                if (state != nullptr) load_elements<V>(state + static_cast<size_t>(j) * p.dim + d, next);
#pragma unroll
                for (int i = 0; i < V; ++i) sum[i] += p.conv_weight[static_cast<size_t>(d + i) * p.taps + j] * next[i];
                if (state != nullptr && j > 0) store_elements<V>(state + static_cast<size_t>(j - 1) * p.dim + d, next);
            }
            if (state != nullptr) store_elements<V>(state + static_cast<size_t>(p.taps - 2) * p.dim + d, now);
#pragma unroll
            for (int i = 0; i < V; ++i) h[i] += sum[i] + p.conv_weight[static_cast<size_t>(d + i) * p.taps + p.taps - 1] * now[i];
        }
        store_elements<V>(p.h + static_cast<size_t>(r) * p.dim + d, h);
    }
}

template <typename T, int V>
int launch_stream_step(const StreamStep<T>& p, int streams, int out_rows, cudaStream_t stream) {
    int threads = ((p.dim + V - 1) / V + 31) / 32 * 32;
    const int most = out_rows <= 64 ? stream_step_threads(streams) : 256;
    threads = threads < 128 ? 128 : (threads > most ? most : threads);
    const size_t shared = (static_cast<size_t>((p.dim + 3) & ~3) + 33) * sizeof(float);
    if (shared > 200 * 1024) return -2;
    cudaError_t error = cudaSuccess;
    switch (streams) {
#define LB_STREAM_CASE(S)                                                                                                                     \
    case S: {                                                                                                                                 \
        auto kernel = out_rows <= 64 ? stream_step_kernel<T, S, V, false> : stream_step_kernel<T, S, V, true>;                                \
        if (shared > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(shared));          \
        error = launch_overlapped(kernel, dim3(out_rows), dim3(threads), shared, stream, p);                                                  \
        break;                                                                                                                                \
    }
        LB_STREAM_CASE(1) LB_STREAM_CASE(2) LB_STREAM_CASE(3) LB_STREAM_CASE(4) LB_STREAM_CASE(5) LB_STREAM_CASE(6) LB_STREAM_CASE(7) LB_STREAM_CASE(8)
#undef LB_STREAM_CASE
        default: return -2;
    }
    if (error != cudaSuccess) return static_cast<int>(error);
    return LB_LAUNCH_RESULT();
}

// ------------------------------------------------------------------------------------------- causal convolution
// Tokens per block; taps - 1 may not exceed them.  Few, where the number of taps is known: all of a thread's loads leave before the first sum.
template <int TAPS>
struct ConvRows {
    static constexpr int kRows = TAPS > 0 ? 4 : 16;
};

// V consecutive elements, 16 bytes at a time where V elements make that much.
template <typename T, int V>
__device__ __forceinline__ void load_pack(const T* source, float (&v)[V]) {
    if constexpr (V == 8) {
        const uint4 raw = *reinterpret_cast<const uint4*>(source);
        const __nv_bfloat162* pairs = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const float2 two = __bfloat1622float2(pairs[i]);
            v[2 * i] = two.x, v[2 * i + 1] = two.y;
        }
    } else {
        load_elements<V>(source, v);
    }
}
template <typename T, int V>
__device__ __forceinline__ void store_pack(T* destination, const float (&v)[V]) {
    if constexpr (V == 8) {
        uint4 raw;
        __nv_bfloat162* pairs = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
        for (int i = 0; i < 4; ++i) pairs[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
        *reinterpret_cast<uint4*>(destination) = raw;
    } else {
        store_elements<V>(destination, v);
    }
}

// grid (tiles of ConvRows tokens of the longest portion, portions, pieces of the channels); a thread per V channels.
//   out_t = [x_t +] sum_j w[:, j] x_(t - taps + 1 + j), what lies before the portion from the request's state
// A portion's first tile reads all of the state that anyone reads (taps - 1 <= ConvRows) and then moves it on: row i becomes the
// portion's input at len - (taps - 1) + i, or an old row where the portion is shorter than that.  TAPS 0: any number of taps.
template <typename T, int TAPS, int V>
__global__ void causal_conv_kernel(const T* __restrict__ x, int x_stride, T* __restrict__ state, const float* __restrict__ weight, T* __restrict__ out,
                                   int out_stride, int channels, int any_taps, int add_input, const int* __restrict__ segment_start,
                                   const int* __restrict__ segment_length, const int* __restrict__ segment_slot, int num_slots, int* status) {
    wait_for_previous_kernel();
    allow_next_kernel();
    const int taps = TAPS > 0 ? TAPS : any_taps;
    const int segment = blockIdx.y;
    constexpr int kRows = ConvRows<TAPS>::kRows;
    static_assert(TAPS - 1 <= kRows, "a portion's first tile reads all of the state that is read");
    const int first = blockIdx.x * kRows, length = segment_length[segment];
    const int channel = (blockIdx.z * blockDim.x + threadIdx.x) * V;
    if (first >= length || channel >= channels) return;
    const int slot = segment_slot[segment];
    const bool good = slot >= 0 && slot < num_slots;
    if (!good && taps > 1 && channel == 0) report_error(status, kBadSlot);
    T* own_state = good && taps > 1 ? state + static_cast<size_t>(slot) * (taps - 1) * channels + channel : nullptr;
    const T* source = x + static_cast<size_t>(segment_start[segment]) * x_stride + channel;
    T* destination = out + static_cast<size_t>(segment_start[segment]) * out_stride + channel;
    const int end = min(length, first + kRows);
    // the input at local index t, which may lie in the state
    auto input = [&](int t, float (&v)[V]) {
        if (t >= 0) {
            load_pack<T, V>(source + static_cast<size_t>(t) * x_stride, v);
        } else if (own_state != nullptr) {
            load_pack<T, V>(own_state + static_cast<size_t>(taps - 1 + t) * channels, v);
        } else {
#pragma unroll
            for (int i = 0; i < V; ++i) v[i] = 0.0f;
        }
    };
    if constexpr (TAPS > 0) {
        float held[kRows + TAPS - 1][V];   // the inputs at first - (TAPS - 1) ... first + kRows - 1
#pragma unroll
        for (int r = 0; r < kRows + TAPS - 1; ++r) {
            if (first - (TAPS - 1) + r < end) {
                input(first - (TAPS - 1) + r, held[r]);
            } else {
#pragma unroll
                for (int i = 0; i < V; ++i) held[r][i] = 0.0f;
            }
        }
        float w[V * TAPS];   // of this thread's channels, one after the other in memory
        const float* own_weight = weight + static_cast<size_t>(channel) * TAPS;
        if constexpr ((V * TAPS) % 4 == 0) {
#pragma unroll
            for (int i = 0; i < V * TAPS; i += 4) {
                const float4 four = *reinterpret_cast<const float4*>(own_weight + i);
                w[i] = four.x, w[i + 1] = four.y, w[i + 2] = four.z, w[i + 3] = four.w;
            }
        } else {
#pragma unroll
            for (int i = 0; i < V * TAPS; ++i) w[i] = own_weight[i];
        }
#pragma unroll
        for (int r = 0; r < kRows; ++r) {
            if (first + r < end) {
                float sum[V];
#pragma unroll
                for (int i = 0; i < V; ++i) {
                    sum[i] = 0.0f;
#pragma unroll
                    for (int j = 0; j < TAPS; ++j) sum[i] += w[i * TAPS + j] * held[r + j][i];
                    if (add_input) sum[i] += held[r + TAPS - 1][i];
                }
                store_pack<T, V>(destination + static_cast<size_t>(first + r) * out_stride, sum);
            }
        }
    } else {
        for (int t = first; t < end; ++t) {
            float sum[V], v[V];
#pragma unroll
            for (int i = 0; i < V; ++i) sum[i] = 0.0f;
            for (int j = 0; j < taps; ++j) {
                input(t - (taps - 1) + j, v);
#pragma unroll
                for (int i = 0; i < V; ++i) sum[i] += weight[static_cast<size_t>(channel + i) * taps + j] * v[i];
            }
            if (add_input) {   // v is the token's own input
#pragma unroll
                for (int i = 0; i < V; ++i) sum[i] += v[i];
            }
            store_pack<T, V>(destination + static_cast<size_t>(t) * out_stride, sum);
        }
    }
    if (first == 0 && own_state != nullptr) {
        for (int j = 0; j + 1 < taps; ++j) {   // upwards: a row taken from the old state lies further up
            float v[V];
            input(length - (taps - 1) + j, v);
            store_pack<T, V>(own_state + static_cast<size_t>(j) * channels, v);
        }
    }
}

template <typename T, int V>
int launch_causal_conv(const void* x, int x_stride, void* state, const float* weight, void* out, int out_stride, int channels, int taps, int add_input,
                       const int* segment_start, const int* segment_length, const int* segment_slot, int segments, int max_length, int num_slots, int* status,
                       cudaStream_t stream) {
    const int threads_needed = (channels + V - 1) / V;
    const int threads = threads_needed >= 128 ? 128 : (threads_needed + 31) / 32 * 32;
    auto kernel = causal_conv_kernel<T, 0, V>;
    if (taps == 2) kernel = causal_conv_kernel<T, 2, V>;
    if (taps == 3) kernel = causal_conv_kernel<T, 3, V>;
    if (taps == 4) kernel = causal_conv_kernel<T, 4, V>;
    const int rows = taps >= 2 && taps <= 4 ? ConvRows<4>::kRows : ConvRows<0>::kRows;
    const dim3 grid((max_length + rows - 1) / rows, segments, (threads_needed + threads - 1) / threads);
    const cudaError_t error = launch_overlapped(kernel, grid, dim3(threads), 0, stream, static_cast<const T*>(x), x_stride, static_cast<T*>(state), weight,
                                                static_cast<T*>(out), out_stride, channels, taps, add_input, segment_start, segment_length, segment_slot, num_slots,
                                                status);
    if (error != cudaSuccess) return static_cast<int>(error);
    return LB_LAUNCH_RESULT();
}

}  // namespace lb

extern "C" {

// See StreamStep.  x_out may be x (not with from_one); mix null: only read and norm.  Returns 0, a CUDA error, -1 for an unsupported
// type, -2 for sizes the kernel does not take (1 to 8 streams, rows that fit shared memory).
int lb_stream_step(const float* x, float* x_out, int from_one, int streams, const float* mix, const float* write, const float* read, const void* y,
                   const float* partials, int slices, long long slice_stride, const float* y_bias, const float* pair_out, const float* pair_weight,
                   const int* pair_expert, int top, int experts, const float* norm_weight, float eps, void* h, const int* rows, int out_rows, int dim,
                   const float* conv_weight, void* conv_state, const int* token_segment, const int* segment_slot, int taps, int num_slots, int dtype, int* status,
                   cudaStream_t stream) {
    if (out_rows == 0) return 0;
    if (streams < 1 || streams > lb::kMaxStreams || dim < 1) return -2;
    if (mix != nullptr && y == nullptr && pair_out == nullptr && slices < 1) return -2;
    if (from_one && x_out == x && x_out != nullptr) return -2;
    LB_DISPATCH_DTYPE(dtype, {
        lb::StreamStep<T> p{};
        p.x = x;
        p.x_out = x_out;
        p.mix = mix;
        p.write = write;
        p.read = read;
        p.y = static_cast<const T*>(y);
        p.partials = partials;
        p.y_bias = y_bias;
        p.pair_out = pair_out;
        p.pair_weight = pair_weight;
        p.pair_expert = pair_expert;
        p.slice_stride = static_cast<size_t>(slice_stride);
        p.slices = slices;
        p.top = top;
        p.experts = experts;
        p.norm_weight = norm_weight;
        p.eps = eps;
        p.h = static_cast<T*>(h);
        p.rows = rows;
        p.dim = dim;
        p.from_one = from_one;
        p.conv_weight = conv_weight;
        p.conv_state = static_cast<T*>(conv_state);
        p.token_segment = token_segment;
        p.segment_slot = segment_slot;
        p.taps = taps;
        p.num_slots = num_slots;
        p.status = status;
        if (dim % 4 == 0 && slice_stride % 4 == 0) return lb::launch_stream_step<T, 4>(p, streams, out_rows, stream);
        return lb::launch_stream_step<T, 1>(p, streams, out_rows, stream);
    })
    return 0;
}

// state [slots, taps - 1, channels] (not read or written for taps == 1); strides in elements.  add_input: out = x + conv(x).  Returns 0, a
// CUDA error, -1 for an unsupported type, -2 for more than 17 taps.
int lb_causal_conv(const void* x, int x_stride, void* state, const float* weight, void* out, int out_stride, int channels, int taps, int add_input,
                   const int* segment_start, const int* segment_length, const int* segment_slot, int segments, int max_length, int num_slots, int dtype,
                   int* status, cudaStream_t stream) {
    if (segments == 0 || max_length == 0 || channels == 0) return 0;
    if (taps < 1 || taps - 1 > lb::ConvRows<0>::kRows) return -2;
    const bool even8 = channels % 8 == 0 && x_stride % 8 == 0 && out_stride % 8 == 0;
    const bool aligned = ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(state)) & 15) == 0;
    if (dtype == lb::kBFloat16) {
        if (even8 && aligned)
            return lb::launch_causal_conv<__nv_bfloat16, 8>(x, x_stride, state, weight, out, out_stride, channels, taps, add_input, segment_start, segment_length,
                                                            segment_slot, segments, max_length, num_slots, status, stream);
        return lb::launch_causal_conv<__nv_bfloat16, 1>(x, x_stride, state, weight, out, out_stride, channels, taps, add_input, segment_start, segment_length,
                                                        segment_slot, segments, max_length, num_slots, status, stream);
    }
    if (dtype == lb::kFloat32) {
        if (even8 && aligned)
            return lb::launch_causal_conv<float, 4>(x, x_stride, state, weight, out, out_stride, channels, taps, add_input, segment_start, segment_length,
                                                    segment_slot, segments, max_length, num_slots, status, stream);
        return lb::launch_causal_conv<float, 1>(x, x_stride, state, weight, out, out_stride, channels, taps, add_input, segment_start, segment_length,
                                                segment_slot, segments, max_length, num_slots, status, stream);
    }
    return -1;
}

}  // extern "C"
