// Matrix products with bfloat16 weights stored [N][K] (one row per output):  C[M,N] = A[M,K] . W[N,K]^T
//
//   gemm_bf16_tc_kernel   A bf16: 5th-generation tensor cores. Persistent CTAs walk 128 x BN output tiles; warp 0
//                         fetches A and W in K-blocks of 64 with TMA (128-byte swizzle, ring of stages), one thread
//                         of warp 1 issues tcgen05.mma into one of two TMEM accumulators, warps 2-5 read the other
//                         accumulator back, so a tile's epilogue runs under the next tile's products.
//   gemm_f32_kernel       A fp32: CUDA cores, fp32 FMA (the weights are exact in fp32).
//
// The epilogue is a parameter of both: store, add to the residual stream, gated activation over interleaved
// gate / up columns, soft-capped logits. Trailing columns of a product (gates of a recurrence, router logits) may go to
// an fp32 buffer of their own. Grouped products (GRP): every tile of 128 rows has weights of its own (an expert's).
#pragma once
#include "tc_common.cuh"

namespace tg {

enum GemmEpi {
	GEMM_STORE = 0,   // C = v                                   (C has the type of the activations)
	GEMM_STORE32 = 1, // C = v, fp32
	GEMM_ADD = 2,     // C += v, fp32 (the residual stream)
	GEMM_GLU = 3,     // columns come as blocks of 16 gate, 16 up: C[16 columns] = glu(gate, up)
	GEMM_LOGITS = 4,  // C = cap * tanh(v / cap) (cap = 0: v), fp32; columns N .. ldc-1 are set to -inf
};

// Gated activations
enum GluAct {
	GLU_GELU = 0,   // gelu_tanh(g) u
	GLU_SILU = 1,   // g sigmoid(g) u
	GLU_CLAMP = 2,  // g' sigmoid(1.702 g') (u' + 1), g' = min(g, limit), u' = u within +- limit
};

struct GemmArgs {
	int M, N, K;
	void *C;
	int ldc;
	float cap;
	int m_tiles, n_tiles;
	int *err;
	int act;                 // GEMM_GLU
	float limit;
	int n32;                 // columns n32 .. N-1 (n32 a multiple of 8, of 32 for GEMM_GLU) are stored to C32 as fp32
	float *C32;
	int ld32;
	const int *tile_expert;  // GRP: [row tiles] expert of a tile; its weights are rows expert * N ..
	const int *n_row_tiles;  // GRP: row tiles of this step
	int splits;              // GEMM_STORE32: CTAs that share a tile's K; split s is stored M * ldc * s further on (0, 1: none)
};

__device__ __forceinline__ float gelu_tanh(float z) {
	const float u = 0.7978845608028654f * (z + 0.044715f * z * z * z);
	return 0.5f * z * (1.0f + tanhf(u));
}
__device__ __forceinline__ float glu(int act, float limit, float g, float u) {
	if (act == GLU_GELU) return gelu_tanh(g) * u;
	if (act == GLU_SILU) return g / (1.0f + expf(-g)) * u;
	g = fminf(g, limit);
	u = fminf(fmaxf(u, -limit), limit);
	return g / (1.0f + expf(-1.702f * g)) * (u + 1.0f);
}
// the same for results that are rounded to bf16: z sigmoid(y) with the fast exponential (gelu_tanh(z) = z sigmoid(2 u))
__device__ __forceinline__ float swish_fast(float z, float y) { return __fdividef(z, 1.0f + __expf(-y)); }
template <int ACT> __device__ __forceinline__ float glu_fast(float limit, float g, float u) {
	if (ACT == GLU_GELU) return swish_fast(g, 1.5957691216057308f * (g + 0.044715f * g * g * g)) * u;
	if (ACT == GLU_SILU) return swish_fast(g, g) * u;
	g = fminf(g, limit);
	u = fminf(fmaxf(u, -limit), limit);
	return fmaf(swish_fast(g, 1.702f * g), u, swish_fast(g, 1.702f * g));
}
__device__ __forceinline__ float soft_cap(float v, float cap) { return cap > 0.0f ? cap * tanhf(v / cap) : v; }
__device__ __forceinline__ uint32_t pack_bf16(float a, float b) {
	const __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
	return *reinterpret_cast<const uint32_t *>(&v);
}

constexpr int GB_BM = 128, GB_BK = 64, GB_THREADS = 192;
constexpr int GB_STG = 32 * 36 * 4;  // output staging of one epilogue warp
template <int BN> struct GbShape {
	static constexpr int A_BYTES = GB_BM * GB_BK * 2;
	static constexpr int W_BYTES = BN * GB_BK * 2;
	static constexpr int STAGE = A_BYTES + W_BYTES;
	static constexpr int NS = BN == 256 ? 4 : (BN == 128 ? 6 : 8);
	static constexpr int SMEM = NS * STAGE + 4 * GB_STG + 1024;
};

// shared-memory matrix descriptor, 128-byte swizzle. K-major operand: 8 rows of 128 bytes form a group, groups
// follow each other (sbo = 1024). MN-major operand: 64 consecutive MN elements x 8 k form a group; lbo = distance of
// the next 64 MN elements, sbo = distance of the next 8 k.
__device__ __forceinline__ uint64_t tc_sw128_desc(uint32_t smem_addr, uint32_t lbo, uint32_t sbo) {
	uint64_t d = 0;
	d |= uint64_t((smem_addr & 0x3FFFF) >> 4);
	d |= uint64_t((lbo >> 4) & 0x3FFF) << 16;
	d |= uint64_t((sbo >> 4) & 0x3FFF) << 32;
	d |= uint64_t(1) << 46;
	d |= uint64_t(2) << 61;
	return d;
}
__device__ __forceinline__ void tma_load_2d(void *dst, const CUtensorMap *map, int x, int y, uint64_t *bar) {
	asm volatile(
	    "cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];" ::"r"(smem_u32(dst)),
	    "l"(map), "r"(x), "r"(y), "r"(smem_u32(bar))
	    : "memory");
}
// D fp32, A and B bf16, A K-major, B K-major (b_mn = 0) or MN-major (1), M = 128
__device__ __forceinline__ uint32_t tc_idesc_bf16(int n, int b_mn) {
	return (1u << 4) | (1u << 7) | (1u << 10) | (uint32_t(b_mn) << 16) | (uint32_t(n >> 3) << 17) | (uint32_t(GB_BM >> 4) << 24);
}

template <int BN, int EPI, bool GRP = false>
__global__ void __launch_bounds__(GB_THREADS, 1) gemm_bf16_tc_kernel(const __grid_constant__ CUtensorMap amap,
                                                                     const __grid_constant__ CUtensorMap wmap, GemmArgs a) {
	using SH = GbShape<BN>;
	constexpr int NS = SH::NS;
	pdl_trigger();
	extern __shared__ uint8_t gb_smem_raw[];
	uint8_t *smem = reinterpret_cast<uint8_t *>((uintptr_t(gb_smem_raw) + 1023) & ~uintptr_t(1023));
	__shared__ uint64_t full_bar[NS], free_bar[NS], acc_full[2], acc_free[2];
	__shared__ uint32_t tmem_base_s;
	__shared__ int s_fail, s_issued;
	const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
	const int k_blocks = (a.K + GB_BK - 1) / GB_BK;
	if (GRP) {
		pdl_wait();
		a.m_tiles = *a.n_row_tiles;
	}
	constexpr bool SPLIT = EPI == GEMM_STORE32;
	const int one = a.m_tiles * a.n_tiles, tiles = SPLIT ? one * max(1, a.splits) : one;
	const int share = SPLIT ? (k_blocks + max(1, a.splits) - 1) / max(1, a.splits) : k_blocks;
	// K-blocks of tile t: [kb_lo, kb_hi)
	auto kb_lo = [&](int t) { return SPLIT ? t / one * share : 0; };
	auto kb_hi = [&](int t) { return SPLIT ? min(k_blocks, (t / one + 1) * share) : k_blocks; };
	// first weight row of a tile
	auto w_row = [&](int t) { return (SPLIT ? t % one : t) / a.m_tiles * BN + (GRP ? a.tile_expert[t % a.m_tiles] * a.N : 0); };
	if (tid == 0) {
		for (int s = 0; s < NS; s++) {
			mbar_init(&full_bar[s], 1);
			mbar_init(&free_bar[s], 1);
		}
		for (int i = 0; i < 2; i++) {
			mbar_init(&acc_full[i], 1);
			mbar_init(&acc_free[i], 4);
		}
		s_fail = 0;
		s_issued = 0;
		asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
	}
	if (warp == 1) {
		asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_base_s)), "r"(2 * BN)
		             : "memory");
		asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
	}
	tc_fence_before();
	__syncthreads();
	tc_fence_after();
	const uint32_t tmem_base = tmem_base_s;

	if (warp == 0) {
		if (lane == 0) {
			// The weights are nobody's output: the first stages' W tiles are requested before the wait for the
			// kernel that produces A.
			const int first = int(blockIdx.x);
			int ahead = 0;
			if (first < tiles) {
				ahead = min(NS, kb_hi(first) - kb_lo(first));
				for (int s = 0; s < ahead; s++) {
					mbar_expect_tx(&full_bar[s], SH::STAGE);
					tma_load_2d(smem + s * SH::STAGE + SH::A_BYTES, &wmap, (kb_lo(first) + s) * GB_BK, w_row(first), &full_bar[s]);
				}
			}
			pdl_wait();
			int it = 0;
			for (int t = first; t < tiles && !*(volatile int *)&s_fail; t += gridDim.x) {
				const int m0 = (t % a.m_tiles) * GB_BM, n0 = w_row(t);
				for (int kb = kb_lo(t), k1 = kb_hi(t); kb < k1; kb++, it++) {
					const int s = it % NS, use = it / NS;
					if (use > 0 && !tc_wait(&free_bar[s], (use - 1) & 1, a.err)) {
						s_fail = 1;
						break;
					}
					uint8_t *st = smem + s * SH::STAGE;
					if (it >= ahead) {
						mbar_expect_tx(&full_bar[s], SH::STAGE);
						tma_load_2d(st + SH::A_BYTES, &wmap, kb * GB_BK, n0, &full_bar[s]);
					}
					tma_load_2d(st, &amap, kb * GB_BK, m0, &full_bar[s]);
					s_issued = it + 1;
				}
			}
		}
	} else if (warp == 1) {
		if (lane == 0) {
			const uint32_t idesc = tc_idesc_bf16(BN, 0);
			int it = 0, n = 0;
			for (int t = blockIdx.x; t < tiles && !*(volatile int *)&s_fail; t += gridDim.x, n++) {
				const int buf = n & 1;
				if (n >= 2 && !tc_wait(&acc_free[buf], ((n >> 1) - 1) & 1, a.err)) {
					s_fail = 1;
					break;
				}
				tc_fence_after();
				const uint32_t d = tmem_base + uint32_t(buf * BN);
				bool ok = true;
				const int k0 = kb_lo(t);
				for (int kb = k0, k1 = kb_hi(t); kb < k1; kb++, it++) {
					const int s = it % NS;
					if (!tc_wait(&full_bar[s], (it / NS) & 1, a.err)) {
						s_fail = 1;
						ok = false;
						break;
					}
					tc_fence_after();
					const uint32_t pa = smem_u32(smem + s * SH::STAGE), pw = pa + SH::A_BYTES;
#pragma unroll
					for (int j = 0; j < GB_BK / 16; j++)
						tc_mma(d, tc_sw128_desc(pa + j * 32, 16, 1024), tc_sw128_desc(pw + j * 32, 16, 1024), idesc, (kb > k0 || j > 0) ? 1u : 0u);
					tc_commit(&free_bar[s]);
				}
				if (!ok) break;
				tc_commit(&acc_full[buf]);
			}
		}
	} else {
		pdl_wait();
		const int quad = warp & 3;  // TMEM lanes 32*quad .. belong to this warp
		float *stg = reinterpret_cast<float *>(smem + NS * SH::STAGE + quad * GB_STG);
		int n = 0;
		for (int t = blockIdx.x; t < tiles && !*(volatile int *)&s_fail; t += gridDim.x, n++) {
			const int buf = n & 1;
			// the residual values of a block of 32 columns are requested one block ahead (and the first before the
			// accumulator is complete)
			float4 res[8];
			auto request = [&](int c) {
				const int rr0 = (t % a.m_tiles) * GB_BM + quad * 32, col = (t / a.m_tiles) * BN + c * 32 + (lane & 7) * 4;
#pragma unroll
				for (int i = 0; i < 8; i++) {
					const int row = rr0 + 4 * i + (lane >> 3);
					res[i] = (c < BN / 32 && row < a.M && col < a.N) ? *reinterpret_cast<const float4 *>(reinterpret_cast<const float *>(a.C) + size_t(row) * a.ldc + col)
					                                               : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
				}
			};
			if (EPI == GEMM_ADD) request(0);
			if (!tc_wait(&acc_full[buf], (n >> 1) & 1, a.err)) {
				s_fail = 1;
				break;
			}
			tc_fence_after();
			const int r0 = (t % a.m_tiles) * GB_BM + quad * 32, n0 = (SPLIT ? t % one : t) / a.m_tiles * BN;
			const size_t far = SPLIT ? size_t(t / one) * a.M * a.ldc : 0;
			const uint32_t taddr = tmem_base + (uint32_t(quad * 32) << 16) + uint32_t(buf * BN);
			const int ncol = (EPI == GEMM_LOGITS) ? a.ldc : a.N;
#pragma unroll 1
			for (int c = 0; c < BN / 32; c++) {
				if (n0 + c * 32 >= ncol) break;
				uint32_t r[32];
				tc_ld32(taddr + uint32_t(c * 32), r);
				asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
				const int col = n0 + c * 32;
				const bool tail = (EPI == GEMM_GLU || EPI == GEMM_STORE) && a.C32 && col >= a.n32;
				if (EPI == GEMM_GLU && !tail) {
					const int row = r0 + lane;
					if (row < a.M) {
						uint32_t o[8];
						auto all = [&](auto f) {
#pragma unroll
							for (int i = 0; i < 8; i++)
								o[i] = pack_bf16(f(__uint_as_float(r[2 * i]), __uint_as_float(r[16 + 2 * i])), f(__uint_as_float(r[2 * i + 1]), __uint_as_float(r[17 + 2 * i])));
						};
						if (a.act == GLU_GELU) all([&](float g, float u) { return glu_fast<GLU_GELU>(a.limit, g, u); });
						else if (a.act == GLU_SILU) all([&](float g, float u) { return glu_fast<GLU_SILU>(a.limit, g, u); });
						else all([&](float g, float u) { return glu_fast<GLU_CLAMP>(a.limit, g, u); });
						uint4 *dst = reinterpret_cast<uint4 *>(reinterpret_cast<__nv_bfloat16 *>(a.C) + size_t(row) * a.ldc + col / 2);
						dst[0] = make_uint4(o[0], o[1], o[2], o[3]);
						dst[1] = make_uint4(o[4], o[5], o[6], o[7]);
					}
				} else {
					// a lane owns a row of the block: through shared memory, so that a store covers whole lines
#pragma unroll
					for (int i = 0; i < 8; i++)
						*reinterpret_cast<uint4 *>(stg + lane * 36 + 4 * i) = make_uint4(r[4 * i], r[4 * i + 1], r[4 * i + 2], r[4 * i + 3]);
					__syncwarp();
					if (EPI == GEMM_STORE || EPI == GEMM_GLU) {
						const int cc = (lane & 3) * 8;
#pragma unroll
						for (int i = 0; i < 4; i++) {
							const int rr = 8 * i + (lane >> 2);
							if (r0 + rr < a.M && col + cc < a.N) {
								const float4 u = *reinterpret_cast<const float4 *>(stg + rr * 36 + cc), v = *reinterpret_cast<const float4 *>(stg + rr * 36 + cc + 4);
								if (a.C32 && col + cc >= a.n32) {
									float4 *dst = reinterpret_cast<float4 *>(a.C32 + size_t(r0 + rr) * a.ld32 + col + cc - a.n32);
									dst[0] = u;
									dst[1] = v;
								} else
									*reinterpret_cast<uint4 *>(reinterpret_cast<__nv_bfloat16 *>(a.C) + size_t(r0 + rr) * a.ldc + col + cc) =
								    make_uint4(pack_bf16(u.x, u.y), pack_bf16(u.z, u.w), pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
							}
						}
					} else {
						const int cc = (lane & 7) * 4;
						float4 add[8];
						if (EPI == GEMM_ADD) {
#pragma unroll
							for (int i = 0; i < 8; i++) add[i] = res[i];
							request(c + 1);
						}
#pragma unroll
						for (int i = 0; i < 8; i++) {
							const int rr = 4 * i + (lane >> 3);
							if (r0 + rr < a.M && col + cc < ncol) {
								float4 v = *reinterpret_cast<const float4 *>(stg + rr * 36 + cc);
								float4 *dst = reinterpret_cast<float4 *>(reinterpret_cast<float *>(a.C) + far + size_t(r0 + rr) * a.ldc + col + cc);
								if (EPI == GEMM_ADD) {
									v.x += add[i].x; v.y += add[i].y; v.z += add[i].z; v.w += add[i].w;
								}
								if (EPI == GEMM_LOGITS) {
									v.x = col + cc < a.N ? soft_cap(v.x, a.cap) : -INFINITY;
									v.y = col + cc + 1 < a.N ? soft_cap(v.y, a.cap) : -INFINITY;
									v.z = col + cc + 2 < a.N ? soft_cap(v.z, a.cap) : -INFINITY;
									v.w = col + cc + 3 < a.N ? soft_cap(v.w, a.cap) : -INFINITY;
								}
								*dst = v;
							}
						}
					}
					__syncwarp();
				}
			}
			tc_fence_before();
			__syncwarp();
			if (lane == 0) mbar_arrive(&acc_free[buf]);
		}
	}
	__syncthreads();
	if (s_fail && tid == 0) {  // let the copies in flight land before the CTA's shared memory goes away
		const int last = *(volatile int *)&s_issued;
		for (int it = max(0, last - NS); it < last; it++) tc_wait(&full_bar[it % NS], (it / NS) & 1, a.err);
	}
	__syncthreads();
	tc_fence_after();
	if (warp == 1)
		asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(2 * BN));
}

// ------------------------------------------------------------------ fp32 activations
constexpr int GF_T = 64, GF_K = 16;
template <int EPI, bool GRP = false>
__global__ void __launch_bounds__(256) gemm_f32_kernel(const float *A, int lda, const __nv_bfloat16 *W, int ldw, GemmArgs a) {
	pdl_trigger();
	pdl_wait();
	__shared__ float sa[GF_K][GF_T + 4], sw[GF_K][GF_T + 4];
	const int tid = threadIdx.x, m0 = blockIdx.y * GF_T, n0 = blockIdx.x * GF_T;
	if (GRP) {
		if (m0 / GB_BM >= *a.n_row_tiles) return;
		W += size_t(a.tile_expert[m0 / GB_BM]) * a.N * ldw;
	}
	const int tx = tid & 15, ty = tid >> 4;
	float acc[4][4] = {};
	for (int k0 = 0; k0 < a.K; k0 += GF_K) {
		for (int i = tid; i < GF_T * GF_K; i += 256) {
			const int r = i / GF_K, k = i % GF_K;
			sa[k][r] = (m0 + r < a.M && k0 + k < a.K) ? A[size_t(m0 + r) * lda + k0 + k] : 0.0f;
			sw[k][r] = (n0 + r < a.N && k0 + k < a.K) ? __bfloat162float(W[size_t(n0 + r) * ldw + k0 + k]) : 0.0f;
		}
		__syncthreads();
#pragma unroll
		for (int k = 0; k < GF_K; k++) {
			float x[4], w[4];
#pragma unroll
			for (int i = 0; i < 4; i++) {
				x[i] = sa[k][ty + 16 * i];
				w[i] = sw[k][tx + 16 * i];
			}
#pragma unroll
			for (int i = 0; i < 4; i++)
#pragma unroll
				for (int j = 0; j < 4; j++) acc[i][j] = fmaf(x[i], w[j], acc[i][j]);
		}
		__syncthreads();
	}
	float *C = reinterpret_cast<float *>(a.C);
#pragma unroll
	for (int i = 0; i < 4; i++) {
		const int row = m0 + ty + 16 * i;
		if (row >= a.M) continue;
		if constexpr (EPI == GEMM_GLU) {  // columns n0 + tx + 16 j: j = 0, 2 gate, j = 1, 3 the up values beside them
#pragma unroll
			for (int j = 0; j < 4; j += 2) {
				const int col = n0 + 16 * j + tx;
				if (a.C32 && n0 + 16 * j >= a.n32) {
					if (col < a.N) a.C32[size_t(row) * a.ld32 + col - a.n32] = acc[i][j];
					if (col + 16 < a.N) a.C32[size_t(row) * a.ld32 + col + 16 - a.n32] = acc[i][j + 1];
				} else if (n0 + 16 * j < a.N) {
					C[size_t(row) * a.ldc + (n0 + 16 * j) / 2 + tx] = glu(a.act, a.limit, acc[i][j], acc[i][j + 1]);
				}
			}
		} else {
#pragma unroll
			for (int j = 0; j < 4; j++) {
				const int col = n0 + tx + 16 * j;
				float *dst = C + size_t(row) * a.ldc + col;
				if (EPI == GEMM_LOGITS) {
					if (col < a.ldc) *dst = col < a.N ? soft_cap(acc[i][j], a.cap) : -INFINITY;
				} else if (EPI == GEMM_STORE && a.C32 && col >= a.n32) {
					if (col < a.N) a.C32[size_t(row) * a.ld32 + col - a.n32] = acc[i][j];
				} else if (col < a.N) {
					*dst = EPI == GEMM_ADD ? *dst + acc[i][j] : acc[i][j];
				}
			}
		}
	}
}

}  // namespace tg
