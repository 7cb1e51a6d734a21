// Row-wise kernels over the tokens of one step: embedding, layer norm, layer norm with the input convolution.
#pragma once
#include <cuda_bf16.h>

#include "tg_common.cuh"

namespace tg {

// The rows of a step. A segment is the run of consecutive tokens that one sequence brings; rows of a segment are
// consecutive. `par` selects which of a sequence's two history buffers holds what earlier steps left; a step writes
// the other one, so no row of the step can overwrite what another still has to read.
struct StepDesc {
	const int *tok;      // [R] token ids
	const int *row_seg;  // [R] segment of a row
	const int *seg_seq;  // [S] sequence slot
	const int *seg_row;  // [S] first row
	const int *seg_len;  // [S] rows
	const int *seg_pos;  // [S] position of the first row
	const int *seg_par;  // [S]
};

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }
__device__ __forceinline__ float bf16_lo(uint32_t u) { return __uint_as_float(u << 16); }
__device__ __forceinline__ float bf16_hi(uint32_t u) { return __uint_as_float(u & 0xFFFF0000u); }

__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z))); }

// x[r] = embed[tok[r]], or x[r] += embed[tok[r]] (another pass through a looped block)
static __global__ void __launch_bounds__(256) embed_rows_kernel(float *x, int ldx, const __nv_bfloat16 *embed, int lde, StepDesc d, int D, int V,
                                                                int add, int *err) {
	pdl_trigger();
	pdl_wait();
	const int r = blockIdx.x;
	int tok = d.tok[r];
	if (tok < 0 || tok >= V) {
		if (threadIdx.x == 0) *err = 1;
		tok = 0;
	}
	for (int i = threadIdx.x; i < D; i += 256) {
		const float e = __bfloat162float(embed[size_t(tok) * lde + i]);
		float *p = x + size_t(r) * ldx + i;
		*p = add ? *p + e : e;
	}
}

// mean and 1/sqrt(var + eps) of one row, by one warp (variance from the deviations)
__device__ __forceinline__ float2 warp_ln_stats(const float *x, int D, float eps) {
	const int lane = threadIdx.x & 31;
	float s = 0.0f;
	for (int i = lane; i < D; i += 32) s += x[i];
	const float mean = warp_sum(s) / float(D);
	float v = 0.0f;
	for (int i = lane; i < D; i += 32) {
		const float c = x[i] - mean;
		v = fmaf(c, c, v);
	}
	return make_float2(mean, 1.0f / sqrtf(warp_sum(v) / float(D) + eps));
}

// out[i] = layer_norm(x[row(i)]) for i < n; row(i) = rows ? rows[i] : i. Columns D .. ldo-1 become 0 (operand padding).
// One warp per row.
template <typename OT>
__global__ void __launch_bounds__(256) layer_norm_kernel(OT *out, int ldo, const float *x, int ldx, const float *w, const int *rows, int n, int D, float eps,
                                                         float *out32) {
	pdl_trigger();
	pdl_wait();
	const int i = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
	if (i >= n) return;
	const float *xr = x + size_t(rows ? rows[i] : i) * ldx;
	const float2 st = warp_ln_stats(xr, D, eps);
	for (int c = lane; c < ldo; c += 32) {
		const float y = c < D ? (xr[c] - st.x) * st.y * w[c] : 0.0f;
		out[size_t(i) * ldo + c] = from_f32<OT>(y);
		if (out32 && c < D) out32[size_t(i) * D + c] = y;
	}
}

// h = n + conv(n), n = layer_norm(x): the causal convolution over time on each channel (taps at cw[j][D], the last one
// meets the current row). The taps - 1 normed rows before a segment come from hist[seq][par], and the segment's
// last ones (or, in a shorter segment, the older ones that still matter) are left in hist[seq][par ^ 1], oldest
// first. hist: [B][2][taps-1][D]. Rows before a sequence's start count as zero, whatever hist holds.
// One CTA per LC_ROWS consecutive rows; a thread walks its channels down the rows with the window in registers.
constexpr int LC_ROWS = 8;
template <typename OT, int MT>
__global__ void __launch_bounds__(256) ln_conv_kernel(OT *out, int ldo, const float *x, int ldx, const float *w, const float *cw, float *hist,
                                                      StepDesc d, int R, int D, int taps, float eps) {
	pdl_trigger();
	pdl_wait();
	__shared__ float2 st[LC_ROWS + MT];
	__shared__ int seg_s[LC_ROWS];
	const int r0 = blockIdx.x * LC_ROWS, nr = min(LC_ROWS, R - r0), H = taps - 1;
	const int warp = threadIdx.x >> 5;
	if (threadIdx.x < nr) seg_s[threadIdx.x] = d.row_seg[r0 + threadIdx.x];
	for (int i = warp; i < nr + H; i += 8) {  // rows r0 - H .. r0 + nr - 1
		const int r = r0 - H + i;
		if (r >= 0) {
			const float2 v = warp_ln_stats(x + size_t(r) * ldx, D, eps);
			if ((threadIdx.x & 31) == 0) st[i] = v;
		}
	}
	__syncthreads();
	for (int c = threadIdx.x; c < ldo; c += 256) {
		if (c >= D) {
			for (int i = 0; i < nr; i++) out[size_t(r0 + i) * ldo + c] = from_f32<OT>(0.0f);
			continue;
		}
		const float wc = w[c];
		float cf[MT], win[MT];  // win[MT-1] is the current row; taps are right-aligned
#pragma unroll
		for (int j = 0; j < MT; j++) cf[j] = j >= MT - taps ? cw[size_t(j - (MT - taps)) * D + c] : 0.0f;
		int seg = -1;
		for (int i = 0; i < nr; i++) {
			const int r = r0 + i;
			if (seg_s[i] != seg) {
				seg = seg_s[i];
				const int row0 = d.seg_row[seg], len = d.seg_len[seg], pos = d.seg_pos[seg];
				float *hb = hist + size_t(d.seg_seq[seg]) * 2 * H * D;
				const float *hr = hb + size_t(d.seg_par[seg]) * H * D;
				float *hw = hb + size_t(d.seg_par[seg] ^ 1) * H * D;
				const int t = r - row0;
#pragma unroll
				for (int j = 0; j < MT; j++) {  // slot j of the window before row t: time t - (MT - j)
					const int back = MT - j, tt = t - back;
					float v = 0.0f;
					if (back <= H) {
						if (tt >= 0)
							v = (x[size_t(r - back) * ldx + c] - st[i + H - back].x) * st[i + H - back].y * wc;
						else if (pos + tt >= 0)
							v = hr[size_t(H + tt) * D + c];
					}
					win[j] = v;
				}
				if (t == 0)  // history rows that lie before this segment and stay relevant
					for (int q = 0; q < H; q++) {
						const int tt = len - H + q;
						if (tt < 0) hw[size_t(q) * D + c] = pos + tt >= 0 ? hr[size_t(H + tt) * D + c] : 0.0f;
					}
			}
			const float nv = (x[size_t(r) * ldx + c] - st[i + H].x) * st[i + H].y * wc;
			float y = 0.0f;
#pragma unroll
			for (int j = 0; j < MT - 1; j++) {
				win[j] = win[j + 1];
				y = fmaf(cf[j], win[j], y);
			}
			win[MT - 1] = nv;
			y = fmaf(cf[MT - 1], nv, y);
			out[size_t(r) * ldo + c] = from_f32<OT>(nv + y);
			const int q = (r - d.seg_row[seg]) - (d.seg_len[seg] - H);
			if (q >= 0) hist[(size_t(d.seg_seq[seg]) * 2 + (d.seg_par[seg] ^ 1)) * H * D + size_t(q) * D + c] = nv;
		}
	}
}

}  // namespace tg
