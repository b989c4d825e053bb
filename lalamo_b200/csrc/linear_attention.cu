// Linear attention with a decaying matrix state per head and no softmax or denominator:
//
//   S_t = diag(a_t) S_(t-1) + k_t v_t^T,     o_t = S_t^T q_t
//
// The decay a_t is one fixed number per head, repeated over the head's key channels, or one number per head and key
// channel made from the token: a = sigmoid(z)^(1 / tau), z a projection of the token plus a bias; or it is a forget gate that also
// says what is written, a = l + (1 - l) sigmoid(z) with a lower bound l per channel and k = 1 - a (HGRN2).  This file holds the
// kernel that lays the recurrence's inputs out in 32-bit (q, k and v as the projection left them, one of q and k
// times key_dim^-1/2, and the decays); the recurrence itself is the scan of gated_delta.cu without its delta-rule
// correction, and the read-out (per-head RMS norm times a gate) is that file's output kernel.
#include "common.cuh"

namespace lb {

// grid (tokens), threads over channels.
//   proj [tokens, stride]: q (heads x dk) | k (heads x dk) | v (heads x dv) | ...
//   z [tokens, z_stride] (may be null): decay logits, heads x dk;  z_bias (may be null): heads x dk
//   fixed_decay (used when z is null): heads
//   lower (may be null): lower bounds of the forget gate, heads x dk; the decay is then lower + (1 - lower) sigmoid(z), the key one
//   minus that, and proj has no k columns: q | v | ...
//   q_silu: q is silu of its columns
//   inv_freq (may be null): channel i of the first 2 `half` channels of every head of q and k turns with channel i + half,
//   (u, v) -> (u cos a - v sin a, v cos a + u sin a), a = positions[token] * inv_freq[i], sines and cosines times `factor`; angles and
//   rotation in 32-bit, nothing rounded before the recurrence reads it
template <typename T>
__global__ void linear_attention_prepare_kernel(const T* __restrict__ proj, int stride, const T* __restrict__ z, int z_stride,
                                                const float* __restrict__ z_bias, const float* __restrict__ fixed_decay, float inverse_tau,
                                                float q_scale, float k_scale, float* __restrict__ q_out, float* __restrict__ k_out,
                                                float* __restrict__ v_out, float* __restrict__ g_out, int heads, int dk, int dv, const float* __restrict__ lower,
                                                int q_silu, const float* __restrict__ inv_freq, const int* __restrict__ positions, int half, float factor) {
    extern __shared__ float turns[];   // cosines, then sines: half of each
    const int token = blockIdx.x;
    const T* row = proj + static_cast<size_t>(token) * stride;
    const int key_width = heads * dk, value_width = heads * dv;
    if (inv_freq != nullptr) {
        const float position = static_cast<float>(positions[token]);
        for (int i = threadIdx.x; i < half; i += blockDim.x) {
            float s, c;
            sincosf(position * inv_freq[i], &s, &c);
            turns[i] = c * factor;
            turns[half + i] = s * factor;
        }
        __syncthreads();
    }
    for (int index = threadIdx.x; index < key_width; index += blockDim.x) {
        float q = to_float(row[index]);
        float k = lower == nullptr ? to_float(row[key_width + index]) : 0.0f;
        if (inv_freq != nullptr) {
            const int d = index % dk;
            if (d < 2 * half) {
                const int i = d < half ? d : d - half, other = d < half ? index + half : index - half;
                const float c = turns[i], s = d < half ? -turns[half + i] : turns[half + i];
                q = q * c + to_float(row[other]) * s;
                k = k * c + to_float(row[key_width + other]) * s;
            }
        }
        if (q_silu) q = q / (1.0f + expf(-q));
        q_out[static_cast<size_t>(token) * key_width + index] = q * q_scale;
        if (lower != nullptr) {
            const float logit = to_float(z[static_cast<size_t>(token) * z_stride + index]) + (z_bias != nullptr ? z_bias[index] : 0.0f);
            const float bound = lower[index];
            // 1 - sigmoid(x) = sigmoid(-x): what is written keeps its precision where the gate is close to one
            g_out[static_cast<size_t>(token) * key_width + index] = bound + (1.0f - bound) / (1.0f + expf(-logit));
            k_out[static_cast<size_t>(token) * key_width + index] = (1.0f - bound) / (1.0f + expf(logit)) * k_scale;
            continue;
        }
        k_out[static_cast<size_t>(token) * key_width + index] = k * k_scale;
        float decay;
        if (z != nullptr) {
            const float logit = to_float(z[static_cast<size_t>(token) * z_stride + index]) + (z_bias != nullptr ? z_bias[index] : 0.0f);
            // log sigmoid(x) = min(x, 0) - log(1 + exp(-|x|)), and sigmoid(x)^(1 / tau) = exp(log sigmoid(x) / tau)
            const float log_sigmoid = fminf(logit, 0.0f) - log1pf(expf(-fabsf(logit)));
            decay = expf(log_sigmoid * inverse_tau);
        } else {
            decay = fixed_decay[index / dk];
        }
        g_out[static_cast<size_t>(token) * key_width + index] = decay;
    }
    for (int index = threadIdx.x; index < value_width; index += blockDim.x)
        v_out[static_cast<size_t>(token) * value_width + index] = to_float(row[(lower != nullptr ? 1 : 2) * key_width + index]);
}

}  // namespace lb

extern "C" {

int lb_linear_attention_prepare(const void* proj, int stride, const void* z, int z_stride, const float* z_bias, const float* fixed_decay, float inverse_tau,
                                float q_scale, float k_scale, float* q_out, float* k_out, float* v_out, float* g_out, int tokens, int heads, int dk, int dv,
                                int dtype, cudaStream_t stream, const float* lower, int q_silu, const float* inv_freq, const int* positions, int rotary_dim,
                                float factor) {
    if (tokens == 0) return 0;
    if (z == nullptr && (fixed_decay == nullptr || lower != nullptr)) return -2;
    if (inv_freq != nullptr && (positions == nullptr || rotary_dim < 2 || rotary_dim % 2 != 0 || rotary_dim > dk || lower != nullptr || q_silu)) return -2;
    const int half = inv_freq != nullptr ? rotary_dim / 2 : 0;
    LB_DISPATCH_DTYPE(dtype, {
        lb::linear_attention_prepare_kernel<T><<<tokens, 256, 2 * half * sizeof(float), stream>>>(static_cast<const T*>(proj), stride, static_cast<const T*>(z), z_stride, z_bias,
                                                                            fixed_decay, inverse_tau, q_scale, k_scale, q_out, k_out, v_out, g_out, heads, dk, dv, lower, q_silu,
                                                                                                    inv_freq, positions, half, factor);
    })
    return LB_LAUNCH_RESULT();
}

}  // extern "C"
