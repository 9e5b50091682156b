// seqgemm_tc.cuh -- the layer-list products on the 5th-generation tensor cores (bf16 mode, many tokens):
//   D[128 weight rows][128 tokens] += W_tile . X_tile^T with tcgen05.mma (kind::f16 on bf16 operands, cta_group::1),
//   fp32 accumulators in TMEM.  Both operands are K-major bf16 matrices in global memory (weights as stored,
//   activations as the producing kernels wrote them) and come in by TMA (cp.async.bulk.tensor, SWIZZLE_128B; edges of M,
//   N and K are zero-filled by the copy).  One lane issues the copies, one lane the MMAs, completion flows through
//   mbarriers (tcgen05.commit); four warps read the accumulators back (tcgen05.ld) and apply the epilogue of the product:
//   fp32 store, activation-type store, or Dynamic-Tanh + residual add.  blockIdx.z walks a batch of per-head products
//   (3-D tensor maps; an operand shared by the batch keeps a 2-D map).
// Every wait is bounded: a stalled pipeline records a code in `err`, every role falls through to the common exit, TMEM
// is released and the host reports the code after the step.
#pragma once

#include <map>
#include <tuple>

#include "seqkernels.cuh"
#include "tc05.cuh"

#define TG_BM 128
#define TG_BN 128
#define TG_BK 64
#define TG_STAGES 3
#define TG_THREADS 192
#define TG_STAGE_BYTES ((TG_BM + TG_BN) * TG_BK * 2)
#define TG_SMEM (TG_STAGES * TG_STAGE_BYTES + 1024)
// kind::f16 instruction descriptor: D = f32 (bit 4), A = B = bf16 (bits 7, 10), both K-major, N at bit 17 (>> 3), M at bit 24 (>> 4)
#define TG_IDESC ((1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(TG_BN >> 3) << 17) | ((uint32_t)(TG_BM >> 4) << 24))

__device__ __forceinline__ void tma_load_3d(void* dst, const CUtensorMap* map, int c0, int c1, int c2, uint64_t* bar) {
	asm volatile("cp.async.bulk.tensor.3d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3, %4}], [%5];" ::"r"(smem_u32(dst)), "l"(map),
	             "r"(c0), "r"(c1), "r"(c2), "r"(smem_u32(bar))
	             : "memory");
}
// about a second at most; false = gave up
__device__ __forceinline__ bool mbar_wait_bounded(uint64_t* bar, uint32_t parity) {
	for (unsigned spins = 0; spins < (1u << 24); ++spins)
		if (mbar_try_wait(bar, parity)) return true;
	return false;
}

// The epilogue of one warp: its 32 weight rows (lane = row m) against the tile's tokens, 32 at a time.  E: what the epilogue does when it is one
// of the plain ones -- a bias at most, and for EPI_F32 columns past `split` in the activation type -- with everything that does not depend on
// the token worked out before the loop; TG_ANY: gemm_store decides per element.
#define TG_ANY (-1)
#define TG_ACT_GATE 100 // EPI_ACT times sigmoid(gate)
template <int E>
__device__ __forceinline__ void tg_epilogue(const GemmArgs& a, int z, const GemmRows& gr, int n0, int m, int lane, uint32_t tmem) {
	const int rows = min(TG_BN, gr.count - n0);
	const bool live = m < a.M;
	const float bias = E != TG_ANY && a.bias && live ? ldf(a.bias + (size_t)z * a.M + m) : 0.f;
	const bool aside = E == EPI_F32 && a.split > 0 && m >= a.split; // this weight row's results go to Y2
	const long ld = aside ? a.ldy2 : a.ldy;
	const size_t o = aside ? (size_t)(gr.base + n0) * a.ldy2 + (m - a.split) : (size_t)z * a.ybs + (size_t)(gr.base + n0) * a.ldy + (E == EPI_GLU ? m >> 1 : m);
	float* const yf = (float*)a.Y + o;
	bf16* const yb = (bf16*)(aside ? a.Y2 : a.Y) + o;
	const float* gate = E == TG_ACT_GATE ? a.gate + (size_t)z * a.gbs + (size_t)(gr.base + n0) * a.ldgate + m : nullptr; // advances with the row pointer
	const size_t gstep = E == TG_ACT_GATE ? a.ldgate : 0;
	for (int c0 = 0; c0 < rows; c0 += 32) {
		float v[32];
		tmem_ld32(tmem + c0, v);
		if constexpr (E == TG_ANY) {
#pragma unroll
			for (int j = 0; j < 32; ++j) gemm_store<bf16>(a, z, gr, n0 + c0 + j, m, v[j]); // lanes = consecutive weight rows: coalesced
		} else {
			const int left = rows - c0;
			// the row pointer advances by one addition per token: 32 separate row offsets would cost the kernel its second CTA per SM
			unsigned char* q = (unsigned char*)(E == EPI_F32 && !aside ? (void*)yf : (void*)yb) + (size_t)c0 * ld * (E == EPI_F32 && !aside ? 4 : 2);
			const size_t step = (size_t)ld * (E == EPI_F32 && !aside ? 4 : 2);
			if constexpr (E == EPI_GLU) { // lanes 2c (gate) and 2c + 1 (up) share the unit's tokens: the even lane forms token j, the odd one token j + 1
				const int odd = lane & 1;
				q += odd ? step : 0;
#pragma unroll
				for (int j = 0; j < 32; j += 2, q += 2 * step) {
					const float x0 = v[j] + bias, x1 = v[j + 1] + bias;
					const float other = __shfl_xor_sync(0xffffffffu, odd ? x0 : x1, 1);
					if (j + odd < left && live) *(bf16*)q = __float2bfloat16_rn(glu_unit(odd ? other : x0, odd ? x1 : other, a.glu_limit, a.glu_mode));
				}
			} else {
#pragma unroll
				for (int j = 0; j < 32; ++j, q += step, gate += gstep) {
					const float x = v[j] + bias;
					if (j >= left || !live) continue;
					if constexpr (E == EPI_F32) {
						if (aside) *(bf16*)q = __float2bfloat16_rn(x);
						else *(float*)q = x;
					} else if constexpr (E == EPI_ACT) *(bf16*)q = __float2bfloat16_rn(x);
					else if constexpr (E == TG_ACT_GATE) *(bf16*)q = __float2bfloat16_rn(x * sigmoidf_(*gate));
					else {
						const bf16 h = __float2bfloat16_rn(x);
						bf16* d = (bf16*)q;
						d[0] = h, d[a.split3] = h, d[2 * a.split3] = __float2bfloat16_rn(x - __bfloat162float(h));
					}
				}
			}
		}
	}
}
// which instance serves a product
static inline int tg_kind(const GemmArgs& a) {
	const bool plain = a.out_scale == 0.f && a.out_cap == 0.f && !a.rs && (a.split == 0 || (a.epi == EPI_F32 && a.split_act == 1));
	if (a.gate) return plain && a.epi == EPI_ACT ? TG_ACT_GATE : TG_ANY;
	return plain && (a.epi == EPI_F32 || a.epi == EPI_ACT || a.epi == EPI_SPLIT3 || a.epi == EPI_GLU) ? a.epi : TG_ANY;
}

template <int E>
__global__ void __launch_bounds__(TG_THREADS, 2) k_seq_gemm_tc(const __grid_constant__ CUtensorMap tm_w, const __grid_constant__ CUtensorMap tm_x, const GemmArgs a, int w3d, int x3d,
                                                             int* err) {
	pdl_enter(); // programmatic dependent launch: let the next kernel's launch overlap this one, then wait for the previous one
	extern __shared__ unsigned char smem_dyn[];
	__shared__ __align__(8) uint64_t full[TG_STAGES], empty[TG_STAGES], accum;
	__shared__ uint32_t tmem_base_s;
	unsigned char* smem = reinterpret_cast<unsigned char*>(((uintptr_t)smem_dyn + 1023) & ~(uintptr_t)1023);
	const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
	const int m0 = blockIdx.x * TG_BM, n0 = blockIdx.y * TG_BN, z = blockIdx.z;
	const int nkb = (a.K + TG_BK - 1) / TG_BK;
	const GemmRows gr = gemm_rows(a, z);
	if (a.band_mode == 1 && !a.band.meets(n0, min(n0 + TG_BN, gr.count) - 1, m0, m0 + TG_BM - 1)) return; // scores that no row of the tile sees
	if (n0 >= gr.count) return; // a grouped product's tile past the end of its group (uniform over the CTA, before any barrier or TMEM allocation)
	// 64-deep step kb of the sum: left out when none of the tile's rows meets its columns
	auto skips = [&](int kb) {
		if (a.band_mode != 2) return false;
		const int c = kb * TG_BK - (a.band_cp > 0 && kb * TG_BK >= a.band_cp ? a.band_cp : 0);
		return !a.band.meets(n0, min(n0 + TG_BN, gr.count) - 1, c, c + TG_BK - 1);
	};
	auto a_tile = [&](int s) { return smem + (size_t)s * TG_STAGE_BYTES; };
	auto b_tile = [&](int s) { return smem + (size_t)s * TG_STAGE_BYTES + TG_BM * TG_BK * 2; };
	if (tid == 0) {
		for (int s = 0; s < TG_STAGES; ++s) mbar_init(&full[s], 1), mbar_init(&empty[s], 1);
		mbar_init(&accum, 1);
		mbar_init_fence();
	}
	if (warp == 1) tmem_alloc(&tmem_base_s, TG_BN);
	tc_fence_before();
	__syncthreads();
	tc_fence_after();
	const uint32_t tmem_base = tmem_base_s;

	if (warp == 0) {
		if (lane == 0) {
			for (int kb = 0, it = 0; kb < nkb; ++kb) {
				if (skips(kb)) continue;
				const int s = it % TG_STAGES;
				if (!mbar_wait_bounded(&empty[s], ((it++ / TG_STAGES) & 1) ^ 1)) {
					atomicExch(err, 1);
					break;
				}
				mbar_expect_tx(&full[s], TG_STAGE_BYTES);
				if (w3d) tma_load_3d(a_tile(s), &tm_w, kb * TG_BK, m0, z, &full[s]);
				else tma_load_2d(a_tile(s), &tm_w, kb * TG_BK, m0, &full[s]);
				if (x3d) tma_load_3d(b_tile(s), &tm_x, kb * TG_BK, n0, z, &full[s]);
				else tma_load_2d(b_tile(s), &tm_x, kb * TG_BK, gr.base + n0, &full[s]); // rows past the group are other groups' (or zero fill): never stored
			}
		}
	} else if (warp == 1) {
		if (lane == 0) {
			bool ok = true;
			for (int kb = 0, it = 0; kb < nkb && ok; ++kb) {
				if (skips(kb)) continue;
				const int s = it % TG_STAGES;
				if (!mbar_wait_bounded(&full[s], (it / TG_STAGES) & 1)) {
					atomicExch(err, 2);
					ok = false;
					break;
				}
				tc_fence_after();
#pragma unroll
				for (int k = 0; k < TG_BK / 16; ++k) // 16 bf16 = 32 bytes along K inside the swizzle atom: +2 in the 16-byte address field
					umma_f16(tmem_base, umma_desc_sw128(a_tile(s)) + 2 * k, umma_desc_sw128(b_tile(s)) + 2 * k, TG_IDESC, (it | k) ? 1u : 0u);
				umma_commit(&empty[s]);
				++it;
			}
			umma_commit(&accum); // arrives when everything issued so far has completed, also after a stall
		}
	} else {
		const bool ok = mbar_wait_bounded(&accum, 0);
		if (!ok && lane == 0) atomicExch(err, 3);
		tc_fence_after();
		if (ok) {
			const int q4 = warp & 3; // the TMEM lane quarter this warp may read
			tg_epilogue<E>(a, z, gr, n0, m0 + q4 * 32 + lane, lane, tmem_base + ((uint32_t)(q4 * 32) << 16));
		}
		tc_fence_before();
	}
	__syncthreads();
	if (warp == 1) {
		tc_fence_after();
		tmem_dealloc(tmem_base, TG_BN);
	}
}

// ---------------------------------------------------------------- host side
typedef CUresult (*TgEncodeFn)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*, const cuuint32_t*, const cuuint32_t*,
                               CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
struct TgState {
	TgEncodeFn encode = nullptr;
	int* err_host = nullptr; // pinned + mapped
	int* err_dev = nullptr;
	std::map<std::tuple<const void*, long, long, long, long, int>, CUtensorMap> maps;
};
static TgState g_tg;

static inline void gemm_tc_setup() {
	if (g_tg.encode) return;
	cudaDriverEntryPointQueryResult qres;
	void* fn = nullptr;
	CUDA_CHECK(cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &fn, cudaEnableDefault, &qres));
	if (!fn || qres != cudaDriverEntryPointSuccess) CALM_FATAL("cuTensorMapEncodeTiled is not available from this driver");
	g_tg.encode = (TgEncodeFn)fn;
	CUDA_CHECK(cudaHostAlloc((void**)&g_tg.err_host, sizeof(int), cudaHostAllocMapped));
	*g_tg.err_host = 0;
	CUDA_CHECK(cudaHostGetDevicePointer((void**)&g_tg.err_dev, g_tg.err_host, 0));
	for (auto k : {k_seq_gemm_tc<TG_ANY>, k_seq_gemm_tc<EPI_F32>, k_seq_gemm_tc<EPI_ACT>, k_seq_gemm_tc<EPI_SPLIT3>, k_seq_gemm_tc<EPI_GLU>, k_seq_gemm_tc<TG_ACT_GATE>})
		CUDA_CHECK(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, TG_SMEM));
}
// a stalled pipeline leaves its code here; read after the stream has been synchronised
static inline int gemm_tc_error() { return g_tg.err_host ? *g_tg.err_host : 0; }

// bf16 [batch][rows][cols] with row stride ld and batch stride bs (elements); box = 64 columns x `box_rows` rows
static inline const CUtensorMap* tg_map(const void* base, long rows, long cols, long ld, long bs, int batch, int box_rows) {
	const auto key = std::make_tuple(base, rows, cols, ld, bs, batch * 1024 + box_rows);
	auto it = g_tg.maps.find(key);
	if (it != g_tg.maps.end()) return &it->second;
	CUtensorMap m;
	const bool three = bs != 0 && batch > 1;
	const cuuint64_t dims[3] = {(cuuint64_t)cols, (cuuint64_t)rows, (cuuint64_t)batch};
	const cuuint64_t strides[2] = {(cuuint64_t)ld * 2, (cuuint64_t)bs * 2};
	const cuuint32_t box[3] = {TG_BK, (cuuint32_t)box_rows, 1}, estr[3] = {1, 1, 1};
	CUresult r = g_tg.encode(&m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, three ? 3 : 2, const_cast<void*>(base), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
	                         CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_128B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
	if (r != CUDA_SUCCESS) return nullptr; // a layout the copy engine does not describe: the caller keeps the mma.sync kernel
	return &(g_tg.maps[key] = m);
}

// shapes the kernel takes: enough tokens to fill its tiles (a matrix of few rows, a router's, fills the rest of its tile with the copy's zeros), 16-byte aligned rows and bases
static inline bool gemm_tc_fits(const GemmArgs& a, int batch) {
	auto al8 = [](long v) { return v % 8 == 0; };
	return a.N >= 64 && a.M >= 8 && a.K >= 32 && al8(a.ldx) && al8(a.ldw) && al8(a.xbs) && al8(a.wbs) && ((uintptr_t)a.X & 15) == 0 && ((uintptr_t)a.W & 15) == 0 &&
	       batch < 65536;
}
// the tensor maps of both operands; false: no map for one of them
static inline bool gemm_tc_maps(const GemmArgs& a, int batch, const CUtensorMap*& mw, const CUtensorMap*& mx) {
	if (g_tg.maps.size() > 8192) g_tg.maps.clear(); // before the look-ups: their results point into the map
	mw = tg_map(a.W, a.M, a.K, a.ldw, a.wbs, batch, TG_BM);
	mx = tg_map(a.X, a.seg ? a.x_rows : a.N, a.K, a.ldx, a.xbs, batch, TG_BN);
	return mw && mx;
}
// false: nothing was launched
static inline bool gemm_tc_launch(const GemmArgs& a, int batch, cudaStream_t stream, bool pdl) {
	const CUtensorMap *mw, *mx;
	if (!gemm_tc_maps(a, batch, mw, mx)) return false;
	const dim3 grid((a.M + TG_BM - 1) / TG_BM, (a.N + TG_BN - 1) / TG_BN, batch);
	cudaLaunchConfig_t cfg = {};
	cfg.gridDim = grid, cfg.blockDim = dim3(TG_THREADS), cfg.dynamicSmemBytes = TG_SMEM, cfg.stream = stream;
	cudaLaunchAttribute at[1];
	at[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
	at[0].val.programmaticStreamSerializationAllowed = 1;
	cfg.attrs = at, cfg.numAttrs = pdl ? 1 : 0;
	auto go = [&](auto kernel) { CUDA_CHECK(cudaLaunchKernelEx(&cfg, kernel, *mw, *mx, a, (int)(a.wbs != 0 && batch > 1), (int)(a.xbs != 0 && batch > 1), g_tg.err_dev)); };
	switch (tg_kind(a)) {
	case EPI_F32: go(k_seq_gemm_tc<EPI_F32>); break;
	case EPI_ACT: go(k_seq_gemm_tc<EPI_ACT>); break;
	case EPI_SPLIT3: go(k_seq_gemm_tc<EPI_SPLIT3>); break;
	case EPI_GLU: go(k_seq_gemm_tc<EPI_GLU>); break;
	case TG_ACT_GATE: go(k_seq_gemm_tc<TG_ACT_GATE>); break;
	default: go(k_seq_gemm_tc<TG_ANY>);
	}
	return true;
}
