// Python bindings of mixture-of-experts feed-forwards with unquantised matrices: an extension of its own, so that a process that serves
// a model without experts compiles and loads nothing of it.
#include "binding_util.h"
#include "experts.h"
#include "launch.h"

namespace {
using namespace llm_binding;

bool aligned16(const Tensor& t) { return reinterpret_cast<uintptr_t>(t.data_ptr()) % 16 == 0; }
const __nv_bfloat16* bf16(const Tensor& t, const char* name) {
    TORCH_CHECK(t.is_cuda() && t.scalar_type() == torch::kBFloat16 && t.is_contiguous() && aligned16(t), name, " must be contiguous, 16-byte aligned bfloat16");
    return reinterpret_cast<const __nv_bfloat16*>(t.data_ptr());
}
int* pair_ints(const Tensor& t, int64_t n, const char* name) {
    TORCH_CHECK(t.numel() == n, name, " must hold one number per pair or expert");
    return const_cast<int*>(ints(t, name));
}

// logits [tokens, experts], or x [tokens, d] and router [experts, d]; counts and ranks number the pairs of every expert
void expert_route(const OptTensor& x, const OptTensor& router, const OptTensor& logits, const OptTensor& bias, const Tensor& ids, const Tensor& weights,
                  const OptTensor& counts, const OptTensor& ranks, int64_t groups, int64_t keep) {
    TORCH_CHECK(ids.dim() == 2 && weights.sizes() == ids.sizes(), "ids / weights must be [tokens, top]");
    TORCH_CHECK(logits || router, "logits, or x with router");
    const int64_t T = ids.size(0), n = logits ? logits->size(-1) : router->size(0);
    if (T == 0) return;
    llm::ExpertRouteParams p = {};
    p.n = n; p.top = ids.size(1); p.groups = groups; p.keep = keep;
    if (bias) p.bias = floats(*bias, n, "bias");
    p.ids = pair_ints(ids, T * p.top, "ids"); p.weights = const_cast<float*>(floats(weights, T * p.top, "weights"));
    TORCH_CHECK(counts.has_value() == ranks.has_value() && logits.has_value() != x.has_value() && x.has_value() == router.has_value(), "counts with ranks; logits, or x with router");
    if (counts) { p.counts = pair_ints(*counts, n, "counts"); p.ranks = pair_ints(*ranks, T * p.top, "ranks"); }
    bool f32 = false;
    if (logits) {
        p.logits = floats(*logits, T * n, "logits");
    } else {
        f32 = is_f32(*x, "x");
        want_like(*router, f32, "router");
        TORCH_CHECK(x->dim() == 2 && x->size(0) == T && x->stride(1) == 1 && router->is_contiguous() && router->size(0) == n && router->size(1) == x->size(1), "x / router");
        p.x = x->data_ptr(); p.x_row = x->stride(0); p.router = router->data_ptr(); p.d = x->size(1);
    }
    check(llm::launch_expert_route(p, T, f32, stream()), "expert_route");
}

void expert_place(const Tensor& x, const Tensor& ids, const Tensor& ranks, const Tensor& counts, const Tensor& place, const Tensor& xs) {
    TORCH_CHECK(ids.dim() == 2 && x.dim() == 2 && x.size(0) == ids.size(0), "x must have a row per token");
    const int64_t P = ids.numel();
    llm::ExpertPlaceParams p = {};
    p.x = bf16(x, "x"); p.x_row = x.stride(0);
    p.top = ids.size(1); p.n = counts.numel(); p.d = x.size(1);
    p.ids = ints(ids, "ids"); p.ranks = pair_ints(ranks, P, "ranks"); p.counts = ints(counts, "counts"); p.place = pair_ints(place, P, "place");
    TORCH_CHECK(xs.dim() == 2 && xs.size(0) == P && xs.size(1) == p.d, "xs must be [pairs, d]");
    p.xs = const_cast<__nv_bfloat16*>(bf16(xs, "xs"));
    check(llm::launch_expert_place(p, x.size(0), stream()), "expert_place");
}

// w [experts, n (pair_act: 2n), k]; out [pairs, n]; pair p reads row p / div of x
llm::ExpertRowsParams rows_params(const Tensor& w, const Tensor& x, const Tensor& ids, const Tensor& out, int64_t div, bool pair_act, double limit) {
    const bool f32 = is_f32(w, "w");
    want_like(x, f32, "x"); want_like(out, f32, "out");
    llm::ExpertRowsParams p = {};
    TORCH_CHECK(w.dim() == 3 && w.is_contiguous() && out.dim() == 2 && out.is_contiguous() && x.dim() == 2 && x.stride(1) == 1, "expert layouts");
    p.w = w.data_ptr(); p.experts = w.size(0); p.n = out.size(1); p.k = w.size(2); p.pair_act = pair_act; p.limit = limit; p.div = div;
    p.pairs = ids.numel();
    TORCH_CHECK(w.size(1) == p.n * (pair_act ? 2 : 1) && x.size(1) == p.k && out.size(0) == p.pairs && div >= 1 && x.size(0) * div >= p.pairs, "expert shapes");
    p.x = x.data_ptr(); p.x_row = x.stride(0); p.ids = ints(ids, "ids"); p.out = out.data_ptr();
    return p;
}
void expert_rows(const Tensor& w, const Tensor& x, const Tensor& ids, const Tensor& out, int64_t div, bool pair_act, double limit) {
    TORCH_CHECK(!is_f32(w, "w") && aligned16(w) && aligned16(x), "expert_rows takes 16-byte aligned bf16 operands");
    check(llm::launch_expert_rows(rows_params(w, x, ids, out, div, pair_act, limit), stream()), "expert_rows");
}
void expert_plain(const Tensor& w, const Tensor& x, const Tensor& ids, const Tensor& out, int64_t div, bool pair_act, double limit) {
    check(llm::launch_expert_plain(rows_params(w, x, ids, out, div, pair_act, limit), is_f32(w, "w"), stream()), "expert_plain");
}

// x [pairs, k] and out [pairs, n] sorted by expert
void expert_grouped(const Tensor& w, const Tensor& x, const Tensor& counts, const Tensor& out, bool pair_act, const Tensor& status, double limit) {
    llm::ExpertGroupedParams p = {};
    p.limit = limit;
    TORCH_CHECK(w.dim() == 3 && x.dim() == 2 && out.dim() == 2 && x.size(0) == out.size(0), "expert layouts");
    p.pairs = x.size(0); p.n = out.size(1); p.k = x.size(1); p.experts = w.size(0);
    TORCH_CHECK(w.size(1) == p.n * (pair_act ? 2 : 1) && w.size(2) == p.k, "expert shapes");
    p.counts = pair_ints(counts, p.experts, "counts");
    p.out = const_cast<__nv_bfloat16*>(bf16(out, "out"));
    want(status, torch::kInt32, "status");
    check(llm::launch_expert_grouped(bf16(w, "w"), bf16(x, "x"), p, pair_act, status.data_ptr<int>(), stream()), "expert_grouped");
}

}  // namespace

PYBIND11_MODULE(TORCH_EXTENSION_NAME, m) {
    m.def("expert_route", &expert_route);
    m.def("expert_place", &expert_place);
    m.def("expert_rows", &expert_rows);
    m.def("expert_plain", &expert_plain);
    m.def("expert_grouped", &expert_grouped);
    m.def("expert_grouped_fits", &llm::expert_grouped_fits);
    m.attr("MAX_PAIRS") = llm::EXPERT_ROWS_MAX_PAIRS;
    m.def("set_pdl", [](bool on) { llm::pdl_enabled() = on; });
    m.def("bounds_status", [](bool reset) { return llm::bounds_status_experts(reset); });
}
