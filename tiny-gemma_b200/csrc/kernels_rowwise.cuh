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

// sum of v over a CTA of NW warps, in every thread
template <int NW> __device__ __forceinline__ float cta_sum(float v, float *red) {
	v = warp_sum(v);
	__syncthreads();
	if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
	__syncthreads();
	float t = 0.0f;
#pragma unroll
	for (int w = 0; w < NW; w++) t += red[w];
	return t;
}
template <typename T> __device__ __forceinline__ void store4(T *p, float4 v);
template <> __device__ __forceinline__ void store4<float>(float *p, float4 v) { *reinterpret_cast<float4 *>(p) = v; }
template <> __device__ __forceinline__ void store4<__nv_bfloat16>(__nv_bfloat16 *p, float4 v) {
	__nv_bfloat162 q[2] = {__floats2bfloat162_rn(v.x, v.y), __floats2bfloat162_rn(v.z, v.w)};
	*reinterpret_cast<uint2 *>(p) = *reinterpret_cast<const uint2 *>(q);
}

// out[i] = layer_norm(x[row(i)]) for i < n; row(i) = rows ? rows[i] : i. Columns D .. ldo-1 become 0 (operand padding).
// One CTA of 128 threads per row, the row in registers while it fits (D <= 4096, D % 4 == 0; ldx, ldo multiples of 4).
template <typename OT>
__global__ void __launch_bounds__(128) layer_norm_kernel(OT *out, int ldo, const float *x, int ldx, const float *w, const int *rows, int n, int D, float eps,
                                                         float *out32) {
	pdl_trigger();
	pdl_wait();
	__shared__ float red[4];
	const int i = blockIdx.x, tid = threadIdx.x;
	const float *xr = x + size_t(rows ? rows[i] : i) * ldx;
	OT *o = out + size_t(i) * ldo;
	if (D <= 4096 && D % 4 == 0) {
		float4 v[8];
		float s = 0.0f;
#pragma unroll
		for (int j = 0; j < 8; j++) {
			const int c = 4 * (tid + 128 * j);
			v[j] = c < D ? *reinterpret_cast<const float4 *>(xr + c) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
			s += (v[j].x + v[j].y) + (v[j].z + v[j].w);
		}
		const float mean = cta_sum<4>(s, red) / float(D);
		float q = 0.0f;
#pragma unroll
		for (int j = 0; j < 8; j++)
			if (4 * (tid + 128 * j) < D) {
				v[j].x -= mean; v[j].y -= mean; v[j].z -= mean; v[j].w -= mean;
				q = fmaf(v[j].x, v[j].x, fmaf(v[j].y, v[j].y, fmaf(v[j].z, v[j].z, fmaf(v[j].w, v[j].w, q))));
			}
		const float f = 1.0f / sqrtf(cta_sum<4>(q, red) / float(D) + eps);
#pragma unroll
		for (int j = 0; j < 8; j++) {
			const int c = 4 * (tid + 128 * j);
			if (c < D) {
				const float4 g = *reinterpret_cast<const float4 *>(w + c);
				const float4 y = make_float4(v[j].x * f * g.x, v[j].y * f * g.y, v[j].z * f * g.z, v[j].w * f * g.w);
				store4<OT>(o + c, y);
				if (out32) *reinterpret_cast<float4 *>(out32 + size_t(i) * D + c) = y;
			} else if (c < ldo) {
				store4<OT>(o + c, make_float4(0.0f, 0.0f, 0.0f, 0.0f));
			}
		}
		return;
	}
	float s = 0.0f, q = 0.0f;
	for (int c = tid; c < D; c += 128) s += xr[c];
	const float mean = cta_sum<4>(s, red) / float(D);
	for (int c = tid; c < D; c += 128) q = fmaf(xr[c] - mean, xr[c] - mean, q);
	const float f = 1.0f / sqrtf(cta_sum<4>(q, red) / float(D) + eps);
	for (int c = tid; c < ldo; c += 128) {
		const float y = c < D ? (xr[c] - mean) * f * w[c] : 0.0f;
		o[c] = from_f32<OT>(y);
		if (out32 && c < D) out32[size_t(i) * D + c] = y;
	}
}

// h = n + conv(n), n = layer_norm(x): the causal convolution over time on each channel (taps at cw[j][D], the last one
// meets the current row). The taps - 1 normed rows before a segment come from hist[seq][par], and the segment's
// last ones (or, in a shorter segment, the older ones that still matter) are left in hist[seq][par ^ 1], oldest
// first. hist: [B][2][taps-1][D]. Rows before a sequence's start count as zero, whatever hist holds.
// One CTA per `rows` (<= LC_ROWS) consecutive rows: its warps norm these rows and the taps - 1 before them into shared
// memory, then a thread walks its channels down the rows with the window in registers.
constexpr int LC_ROWS = 8;
__host__ __device__ inline size_t ln_conv_smem(int rows, int taps, int D) { return size_t(rows + taps - 1) * ((D + 3) & ~3) * 4; }
template <typename OT, int MT>
__global__ void __launch_bounds__(256) ln_conv_kernel(OT *out, int ldo, const float *x, int ldx, const float *w, const float *cw, float *hist,
                                                      StepDesc d, int R, int D, int taps, float eps, int rows) {
	pdl_trigger();
	pdl_wait();
	extern __shared__ __align__(16) float lc_sm[];
	__shared__ int seg_s[LC_ROWS];
	const int r0 = blockIdx.x * rows, nr = min(rows, R - r0), H = taps - 1, ld = (D + 3) & ~3;
	const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
	if (threadIdx.x < nr) seg_s[threadIdx.x] = d.row_seg[r0 + threadIdx.x];
	for (int i = warp; i < nr + H; i += 8) {  // rows r0 - H .. r0 + nr - 1
		const int r = r0 - H + i;
		if (r < 0 || (i < H && d.row_seg[r] != d.row_seg[r0])) continue;  // (another segment's rows are not in any window)
		const float *xr = x + size_t(r) * ldx;
		float *n = lc_sm + size_t(i) * ld;
		float s = 0.0f;
#pragma unroll 8
		for (int c = 4 * lane; c < D; c += 128) {  // (columns D .. ldx - 1 of x are zero)
			const float4 v = *reinterpret_cast<const float4 *>(xr + c);
			*reinterpret_cast<float4 *>(n + c) = v;
			s += (v.x + v.y) + (v.z + v.w);
		}
		const float mean = warp_sum(s) / float(D);
		float q = 0.0f;
#pragma unroll 4
		for (int c = 4 * lane; c < D; c += 128) {
			const float4 v = *reinterpret_cast<const float4 *>(n + c);
			const float a0 = v.x - mean, a1 = c + 1 < D ? v.y - mean : 0.0f, a2 = c + 2 < D ? v.z - mean : 0.0f, a3 = c + 3 < D ? v.w - mean : 0.0f;
			q = fmaf(a0, a0, fmaf(a1, a1, fmaf(a2, a2, fmaf(a3, a3, q))));
		}
		const float f = 1.0f / sqrtf(warp_sum(q) / float(D) + eps);
#pragma unroll 4
		for (int c = lane; c < D; c += 32) n[c] = (n[c] - mean) * f * w[c];
	}
	__syncthreads();
	for (int c = threadIdx.x; c < ldo; c += 256) {
		if (c >= D) {
			for (int i = 0; i < nr; i++) out[size_t(r0 + i) * ldo + c] = from_f32<OT>(0.0f);
			continue;
		}
		float cf[MT], win[MT];  // win[MT-1] is the current row; taps are right-aligned
#pragma unroll
		for (int j = 0; j < MT; j++) cf[j] = j >= MT - taps ? cw[size_t(j - (MT - taps)) * D + c] : 0.0f;
		int seg = -1, row0 = 0, len = 0;
		float *hw = nullptr;
		for (int i = 0; i < nr; i++) {
			const int r = r0 + i;
			if (seg_s[i] != seg) {
				seg = seg_s[i];
				row0 = d.seg_row[seg];
				len = d.seg_len[seg];
				const int pos = d.seg_pos[seg];
				float *hb = hist + size_t(d.seg_seq[seg]) * 2 * H * D;
				const float *hr = hb + size_t(d.seg_par[seg]) * H * D;
				hw = hb + size_t(d.seg_par[seg] ^ 1) * H * D;
				const int t = r - row0;
#pragma unroll
				for (int j = 0; j < MT; j++) {  // slot j of the window before row t: time t - (MT - j)
					const int back = MT - j, tt = t - back;
					float v = 0.0f;
					if (back <= H) {
						if (tt >= 0)
							v = lc_sm[size_t(i + H - back) * ld + c];
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
			const float nv = lc_sm[size_t(i + H) * ld + c];
			float y = 0.0f;
#pragma unroll
			for (int j = 0; j < MT - 1; j++) {
				win[j] = win[j + 1];
				y = fmaf(cf[j], win[j], y);
			}
			win[MT - 1] = nv;
			y = fmaf(cf[MT - 1], nv, y);
			out[size_t(r) * ldo + c] = from_f32<OT>(nv + y);
			const int q = (r - row0) - (len - H);
			if (q >= 0) hw[size_t(q) * D + c] = nv;
		}
	}
}

}  // namespace tg
