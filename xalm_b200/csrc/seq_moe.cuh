// seq_moe.cuh — a mixture of experts as a sublayer of the config.json families: the expert matrices in the engine's layouts, the pass buffers,
// and the kernels of moe_ops.cuh in order.
//
//   router -> [steps of a few tokens: one matvec per (token, slot) pair] or [sort by expert -> tiled fp32 products] or, for long passes of the
//   16-bit mode, [sort -> rows packed in expert order -> grouped tcgen05 GEMM with the activation fused -> grouped tcgen05 GEMM] on the experts'
//   resident fp16 tiles; a shared expert that runs for every token (gated matrices of its own, two row products), optionally with a gate per
//   token that the router's kernel computes; the caller then joins each token's rows (moe_combine, with whatever else its layer adds there).
//
// A family says what differs between designs: how scores become choices and weights (MoeRouteArgs), the activation between an expert's two
// products (RowsEpi), how many of the router's outputs are identity experts.
#pragma once
#include "moe_ops.cuh"
#include "seq_family.cuh"

namespace xalm {
namespace seq {
namespace {

struct MoeWeights {
	int E = 0, identity = 0; // experts with matrices; router outputs behind them that pass the input through
	int top = 0, ff = 0;
	int n_groups = 0, keep_groups = 0; // choice limited to the best expert groups (<= 1: not)
	int up_rows = 0;         // rows of an expert's first matrix: ff, or 2 ff when gate and up rows alternate
	void *w_up = nullptr, *w_down = nullptr, *w_router = nullptr;
	float* correction = nullptr; // (E + identity) or NULL
	float* bias = nullptr;       // (E + identity) of the router's logits, or NULL
	int shared_ff = 0;           // 0: no shared expert
	bool shared_gate = false;    // its output is multiplied by sigmoid(w_sg h): one more row of the router's matrix
	void *w_sup = nullptr, *w_sdown = nullptr;
	WMat m_sup, m_sdown;
	TcWeight t_sup, t_sdown;
	WMat m_up, m_down;
	std::vector<TcWeight> t_up, t_down; // per expert, when long passes run on the tensor cores
	const uint8_t **b_up = nullptr, **b_down = nullptr; // (device) their tiles
	bool on_tc(const SeqModel* m, int n) const { return m->use_tc && !t_up.empty() && n > 1 && n >= m->tc_min_rows; }
};

struct MoeBuffers { // of one pass, sized for the largest mixture of the model
	size_t max_pairs = 0, max_hid = 0, max_shared = 0;
	int max_tiles = 1;
	size_t a_bytes = 0, h_bytes = 0; // operand planes of the tensor-core products: the mixture's input rows in expert order, the hidden rows
	int *idx = nullptr, *sorted = nullptr, *tiles = nullptr, *ntiles = nullptr, *inv = nullptr;
	float *wgt = nullptr, *hid = nullptr, *out = nullptr, *gate = nullptr, *shid = nullptr, *sout = nullptr;
	uint8_t *a_hi = nullptr, *a_lo = nullptr, *hid_hi = nullptr, *hid_lo = nullptr;
};

// tensors of `E` experts under prefix p ("<p>e0." ...): gate (when gated), up, down
void moe_expect(SeqModel* m, const std::string& p, int E, int ff, bool gated) {
	for (int e = 0; e < E; e++) {
		const std::string pe = p + "e" + std::to_string(e) + ".";
		if (gated) expect(m, pe + "gate", {ff, m->width}, true);
		expect(m, pe + "up", {ff, m->width}, true);
		expect(m, pe + "down", {m->width, ff}, true);
	}
}

// tensors of a shared expert under prefix p ("<p>gate" ...); with a gate per token its row is "<p>sg"
void moe_expect_shared(SeqModel* m, const std::string& p, MoeWeights* L, int ff, bool gate) {
	L->shared_ff = ff;
	L->shared_gate = gate;
	expect(m, p + "gate", {ff, m->width}, true);
	expect(m, p + "up", {ff, m->width}, true);
	expect(m, p + "down", {m->width, ff}, true);
	if (gate) expect(m, p + "sg", {1, m->width}, true);
}

// device layouts of the experts (one after the other, gate / up rows alternating) and the router; grows what the buffers must hold
int moe_upload(SeqModel* m, const std::string& p, bool gated, MoeWeights* L, MoeBuffers* b) {
	std::vector<const HostTensor*> up, dn;
	for (int e = 0; e < L->E; e++) {
		const std::string pe = p + "e" + std::to_string(e) + ".";
		if (gated) up.push_back(tensor_or_null(m, pe + "gate"));
		up.push_back(tensor_or_null(m, pe + "up"));
		dn.push_back(tensor_or_null(m, pe + "down"));
	}
	L->up_rows = gated ? 2 * L->ff : L->ff;
	XALM_TRY(upload_rows(m, up, m->width, gated, &L->w_up, &L->m_up));
	XALM_TRY(upload_rows(m, dn, L->ff, false, &L->w_down, &L->m_down));
	XALM_TRY(upload_rows(m, {tensor_or_null(m, p + "router"), L->shared_gate ? tensor_or_null(m, p + "shared.sg") : nullptr}, m->width, false, &L->w_router, nullptr));
	if (L->shared_ff) {
		XALM_TRY(upload_rows(m, {tensor_or_null(m, p + "shared.gate"), tensor_or_null(m, p + "shared.up")}, m->width, true, &L->w_sup, &L->m_sup));
		XALM_TRY(upload_rows(m, {tensor_or_null(m, p + "shared.down")}, L->shared_ff, false, &L->w_sdown, &L->m_sdown));
		b->max_shared = std::max(b->max_shared, (size_t) L->shared_ff);
	}
	XALM_TRY(moe_prepare(m->width, L->E + L->identity, L->n_groups));
	const size_t pairs = (size_t) m->chunk * L->top;
	b->max_pairs = std::max(b->max_pairs, pairs);
	b->max_hid = std::max(b->max_hid, pairs * L->ff);
	b->max_tiles = std::max(b->max_tiles, moe_max_tiles((int) pairs, L->E));
	return XALM_OK;
}

// row tiles of the grouped GEMM over `pairs` rows: every expert may end with a partly filled one
inline int moe_tc_tiles(int pairs, int E) { return pairs / TC_TILE_ROWS + std::min(E, pairs); }

// a mixture whose expert shapes the GEMM takes keeps fp16 tiles per expert for its long passes
int moe_tc_register(SeqModel* m, MoeWeights* L, MoeBuffers* b) {
	const int W = m->width;
	if (L->shared_ff) {
		XALM_TRY(tc_register(m, L->m_sup, &L->t_sup));
		XALM_TRY(tc_register(m, L->m_sdown, &L->t_sdown));
	}
	if (!m->use_tc || !tune("seq_moe_tc") || !tc_shape_ok(L->up_rows, W, L->up_rows) || !tc_shape_ok(W, L->ff, W)) return XALM_OK;
	L->t_up.resize((size_t) L->E);
	L->t_down.resize((size_t) L->E);
	for (int e = 0; e < L->E; e++) {
		WMat up = L->m_up, dn = L->m_down; // this expert's rows of the stacked matrices
		up.rows = L->up_rows;
		up.p0 = static_cast<const uint8_t*>(L->m_up.p0) + (size_t) e * L->up_rows * L->m_up.s0;
		dn.rows = W;
		dn.p0 = static_cast<const uint8_t*>(L->m_down.p0) + (size_t) e * W * L->m_down.s0;
		XALM_TRY(tc_register(m, up, &L->t_up[(size_t) e]));
		XALM_TRY(tc_register(m, dn, &L->t_down[(size_t) e]));
	}
	std::vector<const uint8_t*> up((size_t) L->E), dn((size_t) L->E);
	for (int e = 0; e < L->E; e++) { up[(size_t) e] = L->t_up[(size_t) e].hi; dn[(size_t) e] = L->t_down[(size_t) e].hi; }
	XALM_TRY(dev_alloc(m, &L->b_up, up.size()));
	XALM_TRY(dev_alloc(m, &L->b_down, dn.size()));
	XALM_CUDA_CHECK(cudaMemcpy(L->b_up, up.data(), up.size() * sizeof up[0], cudaMemcpyHostToDevice));
	XALM_CUDA_CHECK(cudaMemcpy(L->b_down, dn.data(), dn.size() * sizeof dn[0], cudaMemcpyHostToDevice));
	const int rows = moe_tc_tiles(m->chunk * L->top, L->E) * TC_TILE_ROWS;
	b->a_bytes = std::max(b->a_bytes, tc_a_plane_bytes(rows, W));
	b->h_bytes = std::max(b->h_bytes, tc_a_plane_bytes(rows, L->ff));
	return XALM_OK;
}

int moe_alloc(SeqModel* m, MoeBuffers* b) {
	if (!b->max_pairs) return XALM_OK;
	const int W = m->width;
	XALM_TRY(dev_alloc(m, &b->idx, b->max_pairs, true));
	XALM_TRY(dev_alloc(m, &b->wgt, b->max_pairs, true));
	XALM_TRY(dev_alloc(m, &b->sorted, b->max_pairs, true));
	XALM_TRY(dev_alloc(m, &b->tiles, (size_t) 3 * b->max_tiles, true));
	XALM_TRY(dev_alloc(m, &b->ntiles, 1, true));
	XALM_TRY(dev_alloc(m, &b->hid, b->max_hid));
	XALM_TRY(dev_alloc(m, &b->out, b->max_pairs * W));
	if (b->max_shared) {
		XALM_TRY(dev_alloc(m, &b->gate, (size_t) m->chunk));
		XALM_TRY(dev_alloc(m, &b->shid, (size_t) m->chunk * b->max_shared));
		XALM_TRY(dev_alloc(m, &b->sout, (size_t) m->chunk * W));
	}
	if (b->a_bytes) {
		XALM_TRY(dev_alloc(m, &b->inv, b->max_pairs, true));
		XALM_TRY(dev_alloc(m, &b->a_hi, b->a_bytes, true));
		XALM_TRY(dev_alloc(m, &b->hid_hi, b->h_bytes, true));
		if (tune("seq_tc") >= 2) {
			XALM_TRY(dev_alloc(m, &b->a_lo, b->a_bytes, true));
			XALM_TRY(dev_alloc(m, &b->hid_lo, b->h_bytes, true));
		}
	}
	return XALM_OK;
}

void moe_free(MoeWeights* L) {
	for (TcWeight& t : L->t_up) tc_weight_free(&t);
	for (TcWeight& t : L->t_down) tc_weight_free(&t);
	tc_weight_free(&L->t_sup);
	tc_weight_free(&L->t_sdown);
}

// The shared expert of n rows h on the main stream: b.sout (and, where the router gave one, its gate) becomes the join's base.
int moe_shared(SeqModel* m, const MoeWeights& L, const MoeBuffers& b, const float* h, int n, RowsEpi act, MoeCombineArgs* ca, int* nl) {
	const int W = m->width;
	act.out = b.shid; act.ldo = L.shared_ff;
	XALM_TRY(rows_product(m, h, W, L.w_sup, &L.t_sup, n, 2 * L.shared_ff, W, act, nl));
	RowsEpi es;
	es.kind = EPI_STORE; es.out = b.sout; es.ldo = W;
	XALM_TRY(rows_product(m, b.shid, L.shared_ff, L.w_sdown, &L.t_sdown, n, W, L.shared_ff, es, nl));
	ca->base = b.sout;
	ca->base_w = L.shared_gate ? b.gate : nullptr;
	return XALM_OK;
}

// Experts of n rows h (n, width) on the main stream.  `route` carries the scoring constants, `act` the epilogue of the first product (kind and
// constants; out and ldo are set here; a shared expert uses the same one).  Afterwards b.wgt and b.idx hold the choice and *ca names the expert
// rows (and the shared expert's) for the caller's moe_combine.  side_free: the side stream has nothing else to do, and the router (one CTA per token)
// and the sort run there beside the shared expert's products.
int moe_experts(SeqModel* m, const MoeWeights& L, const MoeBuffers& b, const float* h, int n, MoeRouteArgs route, RowsEpi act, MoeCombineArgs* ca, int* nl,
                bool side_free = false) {
	cudaStream_t s = m->stream;
	const Fork fk = {m, side_free && L.shared_ff > 0};
	const int W = m->width, total = L.E + L.identity;
	route.h = h; route.ldh = W; route.w = L.w_router; route.w_bf16 = m->w_bf16;
	route.E = total; route.top = L.top; route.K = W; route.correction = L.correction; route.bias = L.bias;
	route.gate_out = L.shared_gate ? b.gate : nullptr;
	route.n_groups = L.n_groups; route.keep_groups = L.keep_groups;
	route.idx = b.idx; route.wgt = b.wgt; route.step = m->d_step;
	XALM_TRY(fk.open());
	XALM_TRY(launch_moe_router(route, n, fk.side()));
	(*nl)++;
	const bool on_tc = L.on_tc(m, n);
	if (on_tc || n * L.top > MOE_MATVEC_PAIRS) { // steps of a few tokens need no tile list
		MoeSortArgs so = {b.idx, L.top, total, m->d_step, b.sorted, b.tiles, b.ntiles, nullptr, b.inv, L.E, on_tc ? TC_TILE_ROWS : 0};
		XALM_TRY(launch_moe_sort(so, fk.side()));
		(*nl)++;
	}
	XALM_TRY(fk.mark());
	if (L.shared_ff) XALM_TRY(moe_shared(m, L, b, h, n, act, ca, nl));
	XALM_TRY(fk.join());
	act.ldo = L.ff;
	if (on_tc) {
		TcGroup up, dn;
		up.b = L.b_up; up.N = L.up_rows; up.K = W;
		up.tiles = b.tiles; up.n_tiles = b.ntiles; up.max_tiles = moe_tc_tiles(n * L.top, L.E);
		dn = up;
		dn.b = L.b_down; dn.N = W; dn.K = L.ff;
		TcAct ta;
		ta.glu = act.kind == EPI_GLU;
		ta.act = ta.glu ? act.glu_act : act.act;
		ta.limit = act.limit; ta.alpha = act.alpha;
		XALM_TRY(tc_group_pack(up, h, b.sorted, L.top, b.a_hi, b.a_lo, s));
		XALM_TRY(tc_group_gemm_act(up, b.a_hi, b.a_lo, ta, b.hid_hi, b.hid_lo, s));
		XALM_TRY(tc_group_gemm(dn, b.hid_hi, b.hid_lo, b.out, W, s));
		*nl += 3;
	} else {
		MoeGemmArgs ga = {};
		ga.A = h; ga.lda = W; ga.a_div = L.top; ga.W = L.w_up; ga.N = L.up_rows; ga.K = W;
		ga.sorted = b.sorted; ga.tiles = b.tiles; ga.n_tiles = b.ntiles;
		ga.idx = b.idx; ga.step = m->d_step; ga.top = L.top; ga.n_experts = L.E;
		ga.e = act; ga.e.out = b.hid;
		XALM_TRY(launch_moe_gemm(ga, m->w_bf16, n * L.top, L.E, s));
		ga.A = b.hid; ga.lda = L.ff; ga.a_div = 1; ga.W = L.w_down; ga.N = W; ga.K = L.ff;
		ga.e = RowsEpi();
		ga.e.kind = EPI_STORE; ga.e.out = b.out; ga.e.ldo = W;
		XALM_TRY(launch_moe_gemm(ga, m->w_bf16, n * L.top, L.E, s));
		*nl += 2;
	}
	ca->y = b.out; ca->ldy = W; ca->top = L.top; ca->width = W; ca->wgt = b.wgt; ca->part_row = on_tc ? b.inv : nullptr;
	ca->step = m->d_step;
	if (L.identity) { ca->idx = b.idx; ca->n_experts = L.E; ca->ident = h; }
	return XALM_OK;
}

} // namespace
} // namespace seq
} // namespace xalm
