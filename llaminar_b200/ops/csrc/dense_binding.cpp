// Python bindings of what models with unquantised matrices share (dense_ops.cu): an extension of its own, so that a process that
// serves only such a model compiles and loads nothing else.
#include "binding_util.h"
#include "dense.h"
#include "launch.h"

namespace {
using namespace llm_binding;

void resid_norm(const OptTensor& y, const OptTensor& y_rows, const OptTensor& w_post, const Tensor& h, bool add, const OptTensor& w_next,
                const OptTensor& xn, const OptTensor& copy0, const OptTensor& copy1, double eps, const OptTensor& y2, const OptTensor& w_y,
                const OptTensor& w_y2, double factor, bool center_post, bool center_next, const OptTensor& y_w) {
    llm::ResidNormParams p = {};
    want(h, torch::kFloat32, "h");
    const int64_t T = h.size(0), d = h.size(1);
    if (T == 0) return;
    bool f32 = false, typed = false;
    auto elem = [&](const Tensor& t, const char* name) {
        const bool f = is_f32(t, name);
        TORCH_CHECK(!typed || f == f32, name, " has another element type than the other activations");
        f32 = f; typed = true;
        TORCH_CHECK(t.dim() == 2 && t.size(1) == d && t.stride(1) == 1, name, " must be rows of ", d, " values");
    };
    if (y) {
        elem(*y, "y");
        p.y = y->data_ptr(); p.y_stride = y->stride(0);
        if (w_post) p.w_post = floats(*w_post, d, "w_post");
        p.n_y_rows = y->size(0);
        int64_t parts = 1;
        if (y_w) {
            TORCH_CHECK(y_w->dim() == 2 && y_w->size(0) == T && y_w->size(1) >= 1 && !y2, "y_w must be [tokens, parts]");
            parts = y_w->size(1);
            p.y_w = floats(*y_w, T * parts, "y_w"); p.n_parts = parts;
        }
        if (y_rows) {
            p.y_rows = ints(*y_rows, "y_rows");
            TORCH_CHECK(y_rows->numel() == T * parts, "y_rows must name one row per token and part");
        } else {
            TORCH_CHECK(y->size(0) == T * parts, "y must have a row per token and part");
        }
        if (y2) {
            elem(*y2, "y2");
            TORCH_CHECK(!y_rows && y2->size(0) == T, "y2 must have as many rows as h");
            p.y2 = y2->data_ptr(); p.y2_stride = y2->stride(0);
            p.w_y = floats(w_y.value(), d, "w_y"); p.w_y2 = floats(w_y2.value(), d, "w_y2");
        }
    }
    p.h = h.data_ptr<float>(); p.add = add;
    if (w_next) {
        elem(xn.value(), "xn");
        TORCH_CHECK(xn->is_contiguous() && xn->size(0) == T, "xn must be contiguous");
        p.w_next = floats(*w_next, d, "w_next"); p.xn = xn->data_ptr();
    }
    if (copy0) { elem(*copy0, "copy0"); TORCH_CHECK(copy0->size(0) == T, "copy0 rows"); p.copy0 = copy0->data_ptr(); p.copy_stride = copy0->stride(0); }
    if (copy1) {
        elem(*copy1, "copy1");
        TORCH_CHECK(copy1->size(0) == T && (!copy0 || copy1->stride(0) == copy0->stride(0)), "copy1 must have copy0's strides");
        p.copy1 = copy1->data_ptr(); p.copy_stride = copy1->stride(0);
    }
    p.d = d; p.eps = eps; p.factor = factor; p.center_post = center_post; p.center_next = center_next;
    check(llm::launch_resid_norm(p, T, f32, stream()), "resid_norm");
}

// past [streams, tokens, d]: the first n_past streams are summed with weights w, stream n_past receives the update if there is one
void depth_mix(const Tensor& h, bool add, const OptTensor& y, const OptTensor& y_rows, const OptTensor& z, const OptTensor& z_rows, const OptTensor& z_w,
               const OptTensor& past, int64_t n_past, const OptTensor& w, const OptTensor& gain0, const OptTensor& xn0, const OptTensor& gain1, const OptTensor& xn1, double eps) {
    llm::DepthMixParams p = {};
    want(h, torch::kFloat32, "h");
    TORCH_CHECK(h.dim() == 2, "h must be [tokens, width]");
    const int64_t T = h.size(0), d = h.size(1);
    if (T == 0) return;
    bool f32 = false, typed = false;
    auto elem = [&](const Tensor& t, const char* name) {
        const bool f = is_f32(t, name);
        TORCH_CHECK(!typed || f == f32, name, " has another element type than the other activations");
        f32 = f; typed = true;
        TORCH_CHECK(t.dim() == 2 && t.size(1) == d && t.stride(1) == 1, name, " must be rows of ", d, " values");
        TORCH_CHECK(reinterpret_cast<uintptr_t>(t.data_ptr()) % 16 == 0, name, " must be 16-byte aligned");
    };
    if (y) {
        elem(*y, "y");
        p.y = y->data_ptr(); p.y_stride = y->stride(0); p.n_y_rows = y->size(0);
        if (y_rows) p.y_rows = ints(*y_rows, "y_rows");
        TORCH_CHECK((y_rows ? y_rows->numel() : y->size(0)) == T, "y must have a row per token");
    }
    if (z) {
        elem(*z, "z");
        p.z = z->data_ptr(); p.z_stride = z->stride(0); p.n_z_rows = z->size(0);
        int64_t parts = 1;
        if (z_w) {
            TORCH_CHECK(z_w->dim() == 2 && z_w->size(0) == T && z_w->size(1) >= 1, "z_w must be [tokens, parts]");
            parts = z_w->size(1);
            p.z_w = floats(*z_w, T * parts, "z_w"); p.n_parts = parts;
        }
        if (z_rows) p.z_rows = ints(*z_rows, "z_rows");
        TORCH_CHECK((z_rows ? z_rows->numel() : z->size(0)) == T * parts, "z must have a row per token and part");
    }
    p.h = h.data_ptr<float>(); p.add = add;
    TORCH_CHECK(past.has_value() == w.has_value() && n_past >= 0 && (past || n_past == 0), "streams go with weights");
    if (past) {
        TORCH_CHECK(past->is_cuda() && past->scalar_type() == torch::kFloat32 && past->dim() == 3 && past->size(1) == T && past->size(2) == d && past->stride(2) == 1 &&
                        past->stride(1) == d && n_past <= past->size(0) && reinterpret_cast<uintptr_t>(past->data_ptr()) % 16 == 0, "past must be float [streams, tokens, width]");
        p.past = past->data_ptr<float>(); p.past_stride = past->stride(0); p.n_past = n_past;
        p.keep = n_past < past->size(0) && (y || z);
        p.w = floats(*w, n_past + 1, "w");
    }
    auto gain = [&](const OptTensor& g, const OptTensor& xn, const float*& gp, void*& xp) {
        TORCH_CHECK(g.has_value() == xn.has_value(), "a norm has a gain and an output");
        if (!g) return;
        elem(*xn, "xn");
        TORCH_CHECK(xn->is_contiguous() && xn->size(0) == T, "xn must be contiguous");
        want(*g, torch::kFloat32, "gain");
        const int step = g->numel() == 1 ? 0 : 1;
        TORCH_CHECK((step == 0 || g->numel() == d) && (!p.gain0 || p.gain_step == step), "gains must be one number, or one per value, both of a kind");
        p.gain_step = step; gp = g->data_ptr<float>(); xp = xn->data_ptr();
    };
    gain(gain0, xn0, p.gain0, p.xn0);
    gain(gain1, xn1, p.gain1, p.xn1);
    p.d = d; p.eps = eps;
    check(llm::launch_depth_mix(p, T, f32, stream()), "depth_mix");
}

// table [vocabulary, columns]: columns [first, first + cols) belong to this layer
llm::SideTable side_table(const OptTensor& table, int64_t first, int64_t cols, const OptTensor& tokens, int64_t rows, bool f32) {
    llm::SideTable s = {};
    if (!table) return s;
    want_like(*table, f32, "side table");
    TORCH_CHECK(table->dim() == 2 && table->stride(1) == 1 && first >= 0 && first + cols <= table->size(1), "side table columns");
    TORCH_CHECK(tokens ? tokens->numel() == rows : table->size(0) == rows, "one token per row");
    s.table = static_cast<const char*>(table->data_ptr()) + first * table->element_size();
    s.row = table->stride(0); s.cols = cols; s.n_rows = table->size(0);
    if (tokens) s.tokens = ints(*tokens, "tokens");
    return s;
}

// the table of a side input names its rows by token, the one of a gate has the output's rows and columns
void want_table(int64_t act, const OptTensor& table, int64_t cols, const OptTensor& tokens, int64_t n) {
    TORCH_CHECK((act == llm::ACT_GELU_SIDE || act == llm::ACT_GATE) == table.has_value(), "a table goes with the side activation and the gate");
    TORCH_CHECK((act == llm::ACT_GELU_SIDE) == tokens.has_value() && (act != llm::ACT_GATE || cols == n), "tokens / gate columns");
}

void activate(const Tensor& x, const Tensor& act, int64_t kind, const OptTensor& table, int64_t first, int64_t cols, const OptTensor& tokens) {
    const bool f32 = is_f32(x, "x");
    want_like(act, f32, "act");
    TORCH_CHECK(x.dim() == 2 && act.dim() == 2 && x.stride(1) == 1 && act.stride(1) == 1 && x.size(0) == act.size(0), "activation rows");
    TORCH_CHECK((reinterpret_cast<uintptr_t>(x.data_ptr()) | reinterpret_cast<uintptr_t>(act.data_ptr())) % 16 == 0, "activations must be 16-byte aligned");
    TORCH_CHECK(x.size(1) == act.size(1) * (llm::act_pairs(kind) ? 2 : 1), "activation columns");
    want_table(kind, table, cols, tokens, act.size(1));
    if (x.size(0) == 0) return;
    check(llm::launch_activate(x.data_ptr(), x.stride(0), act.data_ptr(), act.stride(0), x.size(0), act.size(1), kind, side_table(table, first, cols, tokens, x.size(0), f32), f32, stream()), "activate");
}

void rope_angles(const Tensor& positions, const Tensor& freqs, double magnitude, const Tensor& out) {
    want(freqs, torch::kFloat64, "freqs");
    const int rows = positions.numel(), half = freqs.numel();
    angle_ptr(out, rows);
    TORCH_CHECK(out.size(1) == half, "angles must have one column per frequency");
    check(llm::launch_rope_angles(ints(positions, "positions"), freqs.data_ptr<double>(), magnitude, reinterpret_cast<float2*>(out.data_ptr<float>()),
                                  rows, half, stream()), "rope_angles");
}

// w [z, n, k] (GELU_MUL, SILU_MUL: [z, 2n, k]), x [z, m, k], out [z, m, n]; the last dimension of each is dense
void gemv_dense(const Tensor& w, const Tensor& x, const Tensor& out, int64_t act, const OptTensor& table, int64_t first, int64_t cols, const OptTensor& tokens) {
    TORCH_CHECK(w.is_cuda() && w.scalar_type() == torch::kBFloat16 && x.scalar_type() == torch::kBFloat16, "gemv_dense takes bf16 operands");
    TORCH_CHECK(w.dim() == 3 && x.dim() == 3 && out.dim() == 3 && w.stride(2) == 1 && x.stride(2) == 1 && out.stride(2) == 1, "gemv_dense layouts");
    llm::GemvDenseParams p = {};
    p.z = w.size(0); p.n = llm::act_pairs(act) ? w.size(1) / 2 : w.size(1); p.k = w.size(2); p.m = x.size(1);
    TORCH_CHECK(x.size(0) == p.z && out.size(0) == p.z && x.size(2) == p.k && out.size(1) == p.m && out.size(2) == p.n, "gemv_dense shapes");
    p.out_f32 = is_f32(out, "out"); p.act = act;
    p.w = reinterpret_cast<const __nv_bfloat16*>(w.data_ptr()); p.w_z = w.stride(0); p.ldw = w.stride(1);
    p.x = reinterpret_cast<const __nv_bfloat16*>(x.data_ptr()); p.x_row = x.stride(1); p.x_z = x.stride(0);
    p.out = out.data_ptr(); p.o_row = out.stride(1); p.o_z = out.stride(0);
    TORCH_CHECK(reinterpret_cast<uintptr_t>(w.data_ptr()) % 16 == 0 && reinterpret_cast<uintptr_t>(x.data_ptr()) % 16 == 0, "gemv_dense operands must be 16-byte aligned");
    want_table(act, table, cols, tokens, (int64_t)p.z * p.n);
    p.side = side_table(table, first, cols, tokens, act == llm::ACT_GATE ? p.m : (int64_t)p.z * p.m, false);
    check(llm::launch_gemv_dense(p, stream()), "gemv_dense");
}

}  // namespace

PYBIND11_MODULE(TORCH_EXTENSION_NAME, m) {
    m.def("resid_norm", &resid_norm);
    m.def("depth_mix", &depth_mix);
    m.def("activate", &activate);
    m.def("rope_angles", &rope_angles);
    m.def("gemv_dense", &gemv_dense);
    m.def("set_pdl", [](bool on) { llm::pdl_enabled() = on; });
    m.def("bounds_status", [](bool reset) { return llm::bounds_status_dense(reset); });
}
