// What a design does to an embedding row before it becomes the residual stream (EmbedPost), shared by the embedding kernels of
// the decode step and of prompt slices.
#pragma once
#include "internal.h"

namespace lumi {

// w: E consecutive elements of a row, the first of them column `col`, at position `pos`.  The angle p * f is formed in double
// and reduced there, so that far positions keep full single precision.
template <int E>
__device__ __forceinline__ void embed_post(const EmbedPost& post, float (&w)[E], int col, int pos) {
    if (post.scale != 1.f) {
#pragma unroll
        for (int e = 0; e < E; ++e) w[e] *= post.scale;
    }
    if (post.freq == nullptr) return;
#pragma unroll
    for (int e = 0; e < E; ++e) {
        const int c = col + e;
        if (c >= post.width) break;
        const double turns = (double)pos * post.freq[c >> 1];            // in half turns: sin(pi t), cos(pi t)
        const float r = (float)(turns - 2.0 * rint(0.5 * turns));
        w[e] += (c & 1) ? cospif(r) : sinpif(r);
    }
}

}  // namespace lumi
