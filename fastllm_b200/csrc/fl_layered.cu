// Layered decoders (FL_ARCH_NIFUNEX, FL_ARCH_ROFETAR, FL_ARCH_TOZARAX, FL_ARCH_MEDULORN, FL_ARCH_LATODRA, FL_ARCH_TUFAZEN): weight layout + ingest, pooled cache (pages of latents or keys | values +
// recurrent-state slots), and the step function for mixed batches (portions of prompts beside single decoded tokens).
#include <cmath>
#include <map>

#include "layered_model.cuh"
#include "layered_ops.cuh"
#include "model.cuh"
#include "synth.cuh"

namespace fl {

static inline size_t up256(size_t x) { return (x + 255) / 256 * 256; }
// grouped-query attention: a launch of few (row, head) pairs splits each row's keys over up to kGqaMaxSplits blocks
constexpr int kGqaMaxSplits = 16, kGqaSplitRows = 4 * 296;
// the softmax between the two attention GEMMs keeps a row's scores in shared memory when the row has at most this many visible keys
constexpr int kSoftmaxKeep = 10240;

static float bits_to_f32(uint16_t b) {
    const uint32_t u = (uint32_t)b << 16;
    float f;
    std::memcpy(&f, &u, 4);
    return f;
}
static uint16_t f32_to_bits(float f) {
    uint32_t b;
    std::memcpy(&b, &f, 4);
    if ((b & 0x7FFFFFFFu) > 0x7F800000u) return (uint16_t)((b >> 16) | 0x40u);
    return (uint16_t)((b + 0x7FFFu + ((b >> 16) & 1u)) >> 16);
}
static float half_to_f32(uint16_t h) {
    const int e = (h >> 10) & 0x1F, m = h & 0x3FF;
    float v = e == 0 ? std::ldexp((float)m, -24) : (e == 31 ? (m ? NAN : INFINITY) : std::ldexp((float)(m + 1024), e - 25));
    return (h & 0x8000) ? -v : v;
}

// where a named tensor goes
struct LyRoute {
    enum Kind { MAT16, F32, UK_T, F32_RAW, F32_FILL } kind;     // F32_RAW: f32 input is kept bit for bit (constants of a design, not
                                                                // weights); F32_FILL: a tensor of ONE element fills rows x cols floats
    void* dst;
    int64_t rows, cols;     // shape handed over
    int heads;              // UK_T: source rows = heads * (rows / heads)
    int64_t ld = 0;         // MAT16: row stride of the destination (0: cols)
    // MAT16 with turn_dims > 0: the rows form blocks of turn_per; inside each, the turn_dims rows from turn_at on hold rotary pairs as two
    // halves (i, i + turn_dims / 2) and are laid out as neighbours (2i, 2i + 1) -- what the latent attention's kernels turn.  A score does
    // not change when query and key channels are reordered alike.
    int turn_per = 0, turn_at = 0, turn_dims = 0;
};
struct LayeredRoutes {
    std::map<std::string, LyRoute> r;
};
static std::map<const LayeredModel*, LayeredRoutes> g_routes;      // built with the model, dropped at finalize
static std::mutex g_routes_mu;

static void check_mixer(const LayeredModel& m, int i, const fl_layer_desc& d, bool second) {
    const std::string at = "layer " + std::to_string(i) + (second ? " (second mixer): " : ": ");
    FL_CHECK(d.heads >= 1 && (d.dim >= 1 || d.mixer == FL_MIXER_MAMBA2) && d.vdim >= 1, FL_ERR_INVALID, at + "heads / dim / vdim must be positive");
    if (second || d.beside)
        FL_CHECK((d.mixer == FL_MIXER_ATTN || d.mixer == FL_MIXER_DELTA || d.mixer == FL_MIXER_LIGHTNING) && d.kv_from < 0, FL_ERR_UNSUPPORTED,
                 at + "mixers side by side: attention, delta rule or lightning attention, each with its own cache");
    if (d.mixer == FL_MIXER_GLA) {
        FL_CHECK(d.decay_rank >= 1 && d.decay_rank <= 4096 && d.tau > 0.f, FL_ERR_INVALID, at + "bad decay rank / tau");
        FL_CHECK(d.dim <= 256, FL_ERR_UNSUPPORTED, at + "gated linear attention: at most 256 key channels per head");
    } else if (d.mixer == FL_MIXER_LATENT_ATTN) {
        FL_CHECK(d.kv_rank >= 1 && d.kv_rank <= 512 && d.rot_dim >= 0 && d.rot_dim <= 128, FL_ERR_UNSUPPORTED,
                 at + "latent attention: kv_rank <= 512 and rot_dim <= 128");
        FL_CHECK(d.rot_dims >= 0 && d.rot_dims <= d.rot_dim && d.rot_dims % 2 == 0, FL_ERR_INVALID, at + "rotated channels must be even and <= rot_dim");
        FL_CHECK(d.window >= 0, FL_ERR_INVALID, at + "negative window");
        FL_CHECK(d.q_rank >= 0 && d.sink >= 0 && d.sink <= 2, FL_ERR_INVALID, at + "bad query latent size / sink kind");
        FL_CHECK(d.out_gate >= 0 && d.out_gate <= 2, FL_ERR_INVALID, at + "unknown gate kind");
        if (d.kv_from >= 0) {
            FL_CHECK(d.kv_from < i, FL_ERR_INVALID, at + "kv_from must name an earlier layer");
            const fl_layer_desc& s = m.layers[d.kv_from].d;
            FL_CHECK(s.mixer == FL_MIXER_LATENT_ATTN && s.kv_from < 0 && s.kv_rank == d.kv_rank && s.rot_dim == d.rot_dim &&
                         s.rot_dims == d.rot_dims && s.rot_halves == d.rot_halves && s.rot_base == d.rot_base && s.yarn_factor == d.yarn_factor &&
                         s.yarn_original == d.yarn_original && s.yarn_fast == d.yarn_fast && s.yarn_slow == d.yarn_slow,
                     FL_ERR_INVALID, at + "kv_from must name a latent-attention layer with its own cache and the same latent / rotary sizes");
        }
    } else if (d.mixer == FL_MIXER_ATTN) {
        const int G = d.kv_heads > 0 ? d.kv_heads : d.heads;
        FL_CHECK(d.heads % G == 0, FL_ERR_INVALID, at + "heads must be a multiple of kv_heads");
        FL_CHECK(d.dim <= 256 && d.vdim <= 256, FL_ERR_UNSUPPORTED, at + "attention: at most 256 channels per head");
        FL_CHECK(d.rot_dims >= 0 && d.rot_dims <= d.dim && d.rot_dims % 2 == 0, FL_ERR_INVALID, at + "rotated channels must be even and <= dim");
        FL_CHECK(d.window >= 0 && d.softcap >= 0.f, FL_ERR_INVALID, at + "negative window / score cap");
        FL_CHECK(d.keep_first >= 0 && d.mask_chunk >= 0 && d.sink >= 0 && d.sink <= 2, FL_ERR_INVALID, at + "bad mask sizes / sink kind");
        FL_CHECK(d.rot_scaling == FL_ROT_SCALE_YARN || d.rot_scaling == FL_ROT_SCALE_BANDS, FL_ERR_INVALID, at + "unknown rotary scaling");
        FL_CHECK(d.out_gate >= 0 && d.out_gate <= 2, FL_ERR_INVALID, at + "unknown gate kind");
        FL_CHECK(!d.v_from_k || (d.no_qk_norm && d.vdim == d.dim && d.kv_from < 0), FL_ERR_UNSUPPORTED,
                 at + "values that are the keys: built without q/k norms, with vdim = dim and a cache of its own");
        FL_CHECK(!(d.qk_norm_whole && d.no_qk_norm), FL_ERR_INVALID, at + "a q/k norm over the whole projection needs the q/k norm");
        FL_CHECK(!(d.qkv_bias && d.kv_from >= 0), FL_ERR_UNSUPPORTED, at + "biased projections are built for layers with their own cache");
        if (d.kv_from >= 0) {
            FL_CHECK(d.kv_from < i, FL_ERR_INVALID, at + "kv_from must name an earlier layer");
            const fl_layer_desc& s = m.layers[d.kv_from].d;
            const int Gs = s.kv_heads > 0 ? s.kv_heads : s.heads;
            FL_CHECK(s.mixer == FL_MIXER_ATTN && s.kv_from < 0 && Gs == G && s.dim == d.dim && s.vdim == d.vdim, FL_ERR_INVALID,
                     at + "kv_from must name an attention layer with its own cache and the same key / value head sizes");
        }
    } else if (d.mixer == FL_MIXER_MAMBA2) {
        FL_CHECK(d.state >= 1 && d.state <= 256, FL_ERR_UNSUPPORTED, at + "Mamba-2: state size must be in 1..256");
        FL_CHECK(d.groups >= 1 && d.heads % d.groups == 0, FL_ERR_INVALID, at + "heads must be a multiple of groups");
        FL_CHECK(d.norm_groups >= 1 && (d.heads * d.vdim) % d.norm_groups == 0, FL_ERR_INVALID, at + "the inner width must divide into norm_groups parts");
        FL_CHECK(d.conv >= 1 && d.conv <= kMaxTaps, FL_ERR_UNSUPPORTED, at + "convolution taps must be in 1..16");
    } else if (d.mixer == FL_MIXER_DELTA) {
        const int G = d.kv_heads > 0 ? d.kv_heads : d.heads;
        FL_CHECK(d.heads % G == 0, FL_ERR_INVALID, at + "heads must be a multiple of kv_heads");
        FL_CHECK(d.dim <= 256, FL_ERR_UNSUPPORTED, at + "delta rule: at most 256 key channels per head");
        FL_CHECK(d.conv >= 1 && d.conv <= kMaxTaps, FL_ERR_UNSUPPORTED, at + "convolution taps must be in 1..16");
    } else if (d.mixer == FL_MIXER_LIGHTNING) {
        FL_CHECK(d.dim <= 256, FL_ERR_UNSUPPORTED, at + "lightning attention: at most 256 key channels per head");
    } else {
        FL_CHECK(false, FL_ERR_INVALID, at + "unknown mixer");
    }
}

static void check_layer(const LayeredModel& m, int i, const fl_layer_desc& d) {
    const std::string at = "layer " + std::to_string(i) + ": ";
    check_mixer(m, i, d, false);
    FL_CHECK(d.ffn_act == FL_ACT_SWISH_CLAMP || d.ffn_act == FL_ACT_GELU_TANH || d.ffn_act == FL_ACT_RELU2 || d.ffn_act == FL_ACT_RELU ||
                 d.ffn_act == FL_ACT_SILU, FL_ERR_INVALID,
             at + "unknown feed-forward activation");
    FL_CHECK(!(d.ffn_act == FL_ACT_RELU && d.ffn_bias), FL_ERR_UNSUPPORTED, at + "the relu-gated feed-forward has no biases");
    FL_CHECK(d.ffn != FL_FFN_MOE || ((d.ffn_act == FL_ACT_SWISH_CLAMP || d.ffn_act == FL_ACT_RELU2 || d.ffn_act == FL_ACT_SILU) && !d.ffn_bias),
             FL_ERR_UNSUPPORTED, at + "experts use the clamped swish, the silu or the squared-relu activation, without biases");
    FL_CHECK(!(d.ffn_act == FL_ACT_RELU2 && d.ffn_bias), FL_ERR_UNSUPPORTED, at + "the squared-relu feed-forward has no biases");
    if (d.ffn == FL_FFN_DENSE) {
        FL_CHECK(d.ff >= 1, FL_ERR_INVALID, at + "ff must be positive");
    } else if (d.ffn == FL_FFN_MOE) {
        FL_CHECK(d.ff >= 1 && d.experts >= 1 && d.experts <= 1024 && d.top >= 1 && d.top <= d.experts && d.shared_ff >= 0, FL_ERR_INVALID,
                 at + "bad expert counts");
        FL_CHECK(d.router == FL_ROUTER_SOFTMAX || d.router == FL_ROUTER_SIGMOID_GROUPS || d.router == FL_ROUTER_SOFTMAX_GROUPS, FL_ERR_INVALID,
                 at + "unknown router");
        if (d.router != FL_ROUTER_SOFTMAX) {
            FL_CHECK(d.route_groups >= 1 && d.experts % d.route_groups == 0 && d.route_keep >= 1 && d.route_keep <= d.route_groups, FL_ERR_INVALID,
                     at + "experts must divide into route_groups groups of which 1..route_groups are kept");
            FL_CHECK(d.top <= d.route_keep * (d.experts / d.route_groups), FL_ERR_INVALID, at + "the kept groups hold fewer than `top` experts");
            FL_CHECK(d.shared_ff == 0 || (d.router == FL_ROUTER_SOFTMAX_GROUPS && d.shared_plain), FL_ERR_UNSUPPORTED,
                     at + "beside a router with groups a shared expert is built for softmax scores, ungated");
            FL_CHECK(!d.router_bias, FL_ERR_UNSUPPORTED, at + "a router with groups has no bias");
        }
    } else {
        FL_CHECK(d.ffn == FL_FFN_NONE, FL_ERR_INVALID, at + "unknown feed-forward kind");
    }
}

void layered_build(LayeredModel& m, const fl_layer_desc* descs) {
    const fl_stack_config& c = m.cfg;
    FL_CHECK(c.arch == FL_ARCH_NIFUNEX || c.arch == FL_ARCH_ROFETAR || c.arch == FL_ARCH_TOZARAX || c.arch == FL_ARCH_MEDULORN ||
                 c.arch == FL_ARCH_LATODRA || c.arch == FL_ARCH_TUFAZEN, FL_ERR_INVALID,
             "layered models: unknown arch");
    FL_CHECK(c.vocab >= 1 && c.width >= 1 && c.n_layers >= 1 && c.n_layers <= 4096, FL_ERR_INVALID, "layered models: sizes must be positive");
    FL_CHECK(c.compute_dtype == FL_DTYPE_BF16 || c.compute_dtype == FL_DTYPE_F32, FL_ERR_INVALID, "compute_dtype must be bf16 or f32");
    FL_CHECK(!(c.no_pre_norm && c.no_post_norm), FL_ERR_INVALID, "a stack norms its sublayers' inputs, their outputs, or both");
    FL_CHECK(c.max_positions >= 0 && c.canon_taps >= 0 && c.canon_taps <= kMaxTaps, FL_ERR_INVALID, "bad position table / input convolution size");
    FL_CHECK(c.no_post_norm || !(c.gated_residual || c.depth_avg), FL_ERR_UNSUPPORTED,
             "gated contributions and the depth average are built for stacks whose sublayer results join the stream un-normed");
    FL_CHECK(!c.post_sum_norm || (c.no_pre_norm && !c.no_post_norm && c.norm_plain), FL_ERR_INVALID,
             "a norm of the sum is built for stacks whose sublayers read the stream itself, with plain norm weights");
    FL_CHECK(!(c.token_shift && c.canon_taps > 0), FL_ERR_UNSUPPORTED, "a stack has a token shift or input convolutions, not both");
    FL_CHECK(!c.token_shift || c.no_pre_norm, FL_ERR_UNSUPPORTED, "the token shift is built for stacks whose mixers read the stream itself");
    FL_CHECK(c.logit_softcap >= 0.f, FL_ERR_INVALID, "negative logit cap");
    const bool both_norms = !c.no_pre_norm && !c.no_post_norm && !c.post_sum_norm;
    FL_CHECK(!c.layer_scale || both_norms, FL_ERR_UNSUPPORTED, "layer scales are built for stacks with a norm before and after every sublayer");
    FL_CHECK(!(c.tied_head && c.max_positions > 0), FL_ERR_UNSUPPORTED, "a tied output projection with a position table is not built");
    FL_CHECK(c.no_post_norm || !(c.parallel_sub || c.norm_tanh || c.token_side > 0), FL_ERR_UNSUPPORTED,
             "parallel sublayers, tanh norms and token vectors are built for stacks whose sublayer results join the stream un-normed");
    FL_CHECK(!c.parallel_sub || (c.canon_taps == 0 && !c.gated_residual && !c.depth_avg && !c.token_shift), FL_ERR_UNSUPPORTED,
             "parallel sublayers are built without input convolutions, gated contributions, depth average and token shift");
    FL_CHECK(c.token_side >= 0 && c.bigram_buckets >= 0 && c.bigram_mul_prev >= 0 && c.bigram_mul_cur >= 0, FL_ERR_INVALID, "bad token vector / bigram sizes");
    // the hash is taken in 64-bit
    FL_CHECK(c.bigram_buckets == 0 || (c.bigram_mul_prev <= INT64_MAX / 2 / c.vocab && c.bigram_mul_cur <= INT64_MAX / 2 / c.vocab), FL_ERR_UNSUPPORTED,
             "bigram multipliers too large");
    FL_CHECK(c.token_side == 0 || !c.depth_avg, FL_ERR_UNSUPPORTED, "token vectors and a depth average do not go together");
    FL_CHECK(c.bigram_buckets == 0 || !(c.embed_norm || c.tied_head), FL_ERR_UNSUPPORTED, "a bigram table is built for plain, untied embeddings");
    if (c.loop_times > 0) {
        FL_CHECK(c.loop_start >= 0 && c.loop_stop > c.loop_start && c.loop_stop <= c.n_layers && c.loop_times <= 4096, FL_ERR_INVALID, "bad loop span");
        FL_CHECK(both_norms || c.no_post_norm || !(c.loop_reinject || c.loop_step), FL_ERR_UNSUPPORTED,
                 "what a loop adds between its passes is built for stacks with a norm before every sublayer");
        FL_CHECK(!c.depth_avg, FL_ERR_UNSUPPORTED, "a loop and a depth average do not go together");
    } else {
        FL_CHECK(c.loop_times == 0 && !c.loop_reinject && !c.loop_step, FL_ERR_INVALID, "loop options without a loop");
    }
    m.W = c.width; m.V = c.vocab; m.L = c.n_layers; m.f32 = c.compute_dtype == FL_DTYPE_F32;
    m.layers.resize(m.L);
    struct Reg { void** pp; size_t bytes; };
    std::vector<Reg> regs;
    auto reg = [&](auto** pp, size_t bytes) { regs.push_back({(void**)pp, bytes}); };
    const size_t W = m.W;
    reg(&m.embed, (size_t)m.V * W * 2); reg(&m.final_norm, W * 4);
    if (!c.tied_head) reg(&m.head, (size_t)m.V * W * 2);
    if (c.embed_norm) reg(&m.embed_norm, W * 4);
    if (c.norm_tanh) { reg(&m.final_bias, W * 4); reg(&m.final_alpha, 4); }
    if (c.bigram_buckets > 0) reg(&m.bigram, ((size_t)c.bigram_buckets + 1) * W * 2);
    if (c.token_side > 0) reg(&m.side_embed, (size_t)m.V * m.L * c.token_side * 2);
    if (c.loop_step) reg(&m.loop_step, (size_t)c.loop_times * W * 4);
    // the order of computation: the layers before the loop, its passes, the layers behind it
    const bool loop = c.loop_times > 0;
    auto passes = [&](int i) { return loop && i >= c.loop_start && i < c.loop_stop ? c.loop_times : 1; };
    for (int i = 0; i < m.L; ++i) {
        if (!loop || i != c.loop_start) { m.runs.push_back({i, 0, false}); continue; }
        for (int t = 0; t < c.loop_times; ++t)
            for (int k = c.loop_start; k < c.loop_stop; ++k) m.runs.push_back({k, t, k == c.loop_start});
        i = c.loop_stop - 1;
    }
    if (c.max_positions > 0) reg(&m.pos, (size_t)c.max_positions * W * 2);
    auto pad8 = [](int n) { return (n + 7) / 8 * 8; };
    // one mixer: its rows inside the layer's stacked input matrix start at `base`; registers its side tables and its cache / state
    auto build_mixer = [&](LayeredLayerW& lw, int i, int base) {
        const fl_layer_desc& d = lw.d;
        const size_t H = d.heads, D = d.dim, Dv = d.vdim;
        auto recurrent = [&]() {                        // a per-slot state [heads][rows][vdim] + the per-head decay parameters
            lw.gla_index = (int)m.gla_layers.size();
            m.gla_layers.insert(m.gla_layers.end(), passes(i), &lw);
            m.max_heads = std::max<int>(m.max_heads, (int)H);
        };
        auto rope = [&]() {
            const RopeSpec rs{d.rot_dims, d.rot_base, d.yarn_factor, d.yarn_original, d.yarn_fast, d.yarn_slow, d.rot_scaling};
            int ri = -1;
            for (size_t k = 0; k < m.ropes.size(); ++k)
                if (m.ropes[k] == rs) ri = (int)k;
            if (ri < 0) { ri = (int)m.ropes.size(); m.ropes.push_back(rs); }
            lw.rope_index = ri;
        };
        if (d.mixer == FL_MIXER_ATTN) {
            if (lw.d.kv_heads <= 0) lw.d.kv_heads = lw.d.heads;
            const size_t G = lw.d.kv_heads;
            lw.off_q = 0; lw.n_in = (int)(H * D); lw.off_k = lw.off_v = lw.off_g = -1;
            if (!d.no_qk_norm) reg(&lw.qnorm, (d.qk_norm_whole ? H * D : D) * 4);
            if (d.qkv_bias) { reg(&lw.bq, H * D * 4); reg(&lw.bk, G * D * 4); reg(&lw.bv, G * Dv * 4); }
            if (d.sink == 2) reg(&lw.sinkv, H * 4);
            m.max_av = std::max<int>(m.max_av, (int)Dv);
            if (d.kv_from < 0) {
                lw.off_k = lw.n_in; lw.n_in += (int)(G * D);
                if (!d.v_from_k) { lw.off_v = lw.n_in; lw.n_in += (int)(G * Dv); }
                if (!d.no_qk_norm) reg(&lw.knorm, (d.qk_norm_whole ? G * D : D) * 4);
                lw.kv_owner = i;
                lw.kv_index = (int)m.kv_layers.size();
                m.kv_layers.insert(m.kv_layers.end(), passes(i), &lw);
            } else {
                FL_CHECK(passes(i) == 1 && passes(d.kv_from) == 1, FL_ERR_UNSUPPORTED, "kv_from is not built for layers of a loop");
                lw.kv_owner = d.kv_from;
                lw.kv_index = m.layers[d.kv_from].kv_index;
            }
            if (d.out_gate) { lw.off_g = lw.n_in; lw.n_in += (int)(d.out_gate == 2 ? H : H * Dv); }
            lw.n_in = pad8(lw.n_in);
            rope();
        } else if (d.mixer == FL_MIXER_MAMBA2) {
            const size_t inner = H * Dv, GN = (size_t)d.groups * d.state;
            lw.off_g = 0;                               // z, the output gate
            lw.off_v = (int)inner; lw.off_k = (int)(2 * inner); lw.off_q = (int)(2 * inner + GN);    // x | B | C
            lw.off_dt = (int)(2 * inner + 2 * GN);
            lw.n_in = pad8(lw.off_dt + (int)H);
            lw.conv_off = (int)inner; lw.conv_ch = (int)(inner + 2 * GN);
            reg(&lw.conv_w, (size_t)lw.conv_ch * d.conv * 4); reg(&lw.conv_b, (size_t)lw.conv_ch * 4);
            reg(&lw.a_log, H * 4); reg(&lw.dt_bias, H * 4); reg(&lw.dskip, H * 4); reg(&lw.hnorm, inner * 4);
            recurrent();
        } else if (d.mixer == FL_MIXER_DELTA) {
            if (lw.d.kv_heads <= 0) lw.d.kv_heads = lw.d.heads;
            const size_t G = lw.d.kv_heads;
            lw.off_q = 0; lw.off_k = (int)(G * D); lw.off_v = (int)(2 * G * D); lw.off_g = lw.off_v + (int)(H * Dv);
            lw.off_b = lw.off_g + (int)(H * Dv); lw.off_a = lw.off_b + (int)H;
            lw.n_in = pad8(lw.off_a + (int)H);
            lw.conv_off = 0; lw.conv_ch = lw.off_g;
            reg(&lw.conv_w, (size_t)lw.conv_ch * d.conv * 4);
            reg(&lw.a_log, H * 4); reg(&lw.dt_bias, H * 4); reg(&lw.hnorm, Dv * 4);
            recurrent();
        } else if (d.mixer == FL_MIXER_LIGHTNING) {
            lw.off_q = 0; lw.off_k = (int)(H * D); lw.off_v = (int)(2 * H * D); lw.off_g = lw.off_v + (int)(H * Dv);
            lw.n_in = pad8(lw.off_g + (int)(H * Dv));
            lw.conv_off = 0; lw.conv_ch = lw.off_g;         // the activated span q | k | v (no convolution: conv = 0 taps)
            reg(&lw.decay, H * 4); reg(&lw.hnorm, H * Dv * 4);
            recurrent();
        } else if (d.mixer == FL_MIXER_GLA) {
            lw.off_q = 0; lw.off_k = (int)(H * D); lw.off_v = (int)(2 * H * D); lw.off_g = lw.off_v + (int)(H * Dv);
            lw.off_a = lw.off_g + (int)(H * Dv);
            lw.n_in = lw.off_a + d.decay_rank;
            reg(&lw.a2, H * D * d.decay_rank * 2); reg(&lw.a2b, H * D * 4); reg(&lw.hnorm, Dv * 4);
            lw.gla_index = (int)m.gla_layers.size();
            m.gla_layers.insert(m.gla_layers.end(), passes(i), &lw);
            m.max_hd = std::max<int>(m.max_hd, (int)(H * D));
        } else {
            const size_t R = d.rot_dim, C = d.kv_rank, Q = d.q_rank;
            lw.off_q = 0; lw.n_in = (int)(Q > 0 ? Q : H * (D + R));
            if (Q > 0) {
                reg(&lw.dq_norm, Q * 4); reg(&lw.uq, H * (D + R) * Q * 2);
                m.max_qr = std::max<int>(m.max_qr, (int)Q); m.max_q = std::max<int>(m.max_q, (int)(H * (D + R)));
            }
            lw.off_dkv = -1; lw.off_g = -1;
            if (d.kv_from < 0) {
                lw.off_dkv = lw.n_in; lw.n_in += (int)(C + R);
                reg(&lw.dkv_norm, C * 4);
                lw.kv_owner = i;
                lw.kv_index = (int)m.kv_layers.size();
                m.kv_layers.insert(m.kv_layers.end(), passes(i), &lw);
            } else {
                FL_CHECK(passes(i) == 1 && passes(d.kv_from) == 1, FL_ERR_UNSUPPORTED, "kv_from is not built for layers of a loop");
                lw.kv_owner = d.kv_from;
                lw.kv_index = m.layers[d.kv_from].kv_index;
            }
            if (d.out_gate) { lw.off_g = lw.n_in; lw.n_in += (int)(d.out_gate == 2 ? H : H * Dv); }
            if (Q > 0 || d.out_gate) lw.n_in = pad8(lw.n_in);
            if (d.sink == 2) reg(&lw.sinkv, H * 4);
            reg(&lw.uk_t, H * C * D * 2); reg(&lw.uv, H * Dv * C * 2);
            rope();
            m.max_hc = std::max<int>(m.max_hc, (int)(H * C));
        }
        if (base > 0) {             // rows of a second mixer: shift its offsets behind the first one's
            for (int* o : {&lw.off_q, &lw.off_k, &lw.off_v, &lw.off_g, &lw.off_a, &lw.off_dkv, &lw.off_b, &lw.off_dt})
                if (*o >= 0) *o += base;
            lw.conv_off += base;
        }
        lw.fx = 0;
        if (c.parallel_sub && d.ffn != FL_FFN_NONE) lw.fx = d.ffn == FL_FFN_DENSE ? d.ff : d.shared_ff;
        lw.u_ld = (int)(H * Dv) + lw.fx;
        if (lw.fx > 0) {
            lw.off_ff = pad8(lw.n_in);
            lw.n_in = pad8(lw.off_ff + (d.ffn_act == FL_ACT_RELU2 ? 1 : 2) * lw.fx);
        }
        reg(&lw.w_o, W * lw.u_ld * 2);
        m.max_u = std::max(m.max_u, lw.u_ld);
        m.max_hv = std::max<int>(m.max_hv, (int)(H * Dv));
        m.max_cv = std::max(m.max_cv, lw.conv_ch);
    };
    int next_desc = 0;
    for (int i = 0; i < m.L; ++i) {
        LayeredLayerW& lw = m.layers[i];
        lw.d = descs[next_desc++];
        const fl_layer_desc& d = lw.d;
        check_layer(m, i, d);
        const bool pre = !c.no_pre_norm, post = !c.no_post_norm;
        if (pre) reg(&lw.norm1, W * 4);
        if (c.norm_tanh) { reg(&lw.norm1_bias, W * 4); reg(&lw.norm1_alpha, 4); }
        if (post) reg(&lw.norm1b, W * 4);
        FL_CHECK(!(c.parallel_sub && (d.beside || d.ffn_bias || (d.ffn == FL_FFN_MOE && d.shared_ff > 0 && !d.shared_plain))), FL_ERR_UNSUPPORTED,
                 "parallel sublayers are built for one mixer, a feed-forward without biases and an ungated shared expert");
        if (c.token_side > 0) {
            const size_t S = c.token_side;
            reg(&lw.side_gate, S * W * 2); reg(&lw.side_proj, W * S * 2); reg(&lw.side_norm, W * 4);
        }
        if (c.layer_scale) reg(&lw.ls1, W * 4);
        if (c.token_shift) reg(&lw.shift, W * 4);
        build_mixer(lw, i, 0);
        if (d.beside) {
            FL_CHECK(d.pair_sum ? c.post_sum_norm != 0 : !post, FL_ERR_UNSUPPORTED,
                     "mixers side by side: their normed mean joins the stream un-normed, or their weighted sum enters a norm of the sum");
            lw.side = std::make_shared<LayeredLayerW>();
            lw.side->d = descs[next_desc++];
            lw.side->d.beside = 0;
            check_mixer(m, i, lw.side->d, true);
            build_mixer(*lw.side, i, lw.n_in);
            lw.n_in += lw.side->n_in;
            lw.side->n_in = lw.n_in;                    // both read rows of the same projected buffer
            if (!d.pair_sum) { reg(&lw.pair_wa, W * 4); reg(&lw.pair_wb, W * 4); }
        }
        reg(&lw.w_in, (size_t)lw.n_in * W * 2);
        m.max_in = std::max(m.max_in, lw.n_in);
        if (c.canon_taps > 0) reg(&lw.canon1, W * c.canon_taps * 4);
        if (c.gated_residual) { reg(&lw.rg1, W * W * 2); reg(&lw.rg1b, W * 4); }
        if (c.depth_avg) reg(&lw.dwa, (size_t)(i + 2) * 4);
        if (d.ffn != FL_FFN_NONE) {
            const bool par = c.parallel_sub != 0;       // one norm per layer; the always-on part lives in w_in and w_o
            if (pre && !par) reg(&lw.norm2, W * 4);
            if (c.norm_tanh && !par) { reg(&lw.norm2_bias, W * 4); reg(&lw.norm2_alpha, 4); }
            if (post) reg(&lw.norm2b, W * 4);
            if (c.layer_scale) reg(&lw.ls2, W * 4);
            if (c.canon_taps > 0) reg(&lw.canon2, W * c.canon_taps * 4);
            if (c.gated_residual) { reg(&lw.rg2, W * W * 2); reg(&lw.rg2b, W * 4); }
            if (d.ffn == FL_FFN_DENSE && d.ffn_bias) { reg(&lw.b_gu, (size_t)2 * d.ff * 4); reg(&lw.b_down, W * 4); }
            const size_t G = d.ffn == FL_FFN_MOE ? d.experts : 1, F = d.ff, GF = d.ffn_act == FL_ACT_RELU2 ? F : 2 * F;
            if (!par || d.ffn == FL_FFN_MOE) { reg(&lw.w_gu, G * GF * W * 2); reg(&lw.w_down, G * W * F * 2); }
            m.max_ff = std::max<int>(m.max_ff, (int)F);
            m.max_top = std::max(m.max_top, d.ffn == FL_FFN_MOE ? d.top : 1);
            if (d.ffn == FL_FFN_MOE) {
                reg(&lw.router, (size_t)d.experts * W * 4);
                if (d.router_bias) reg(&lw.router_b, (size_t)d.experts * 4);
                if (d.router == FL_ROUTER_SIGMOID_GROUPS) reg(&lw.route_corr, (size_t)d.experts * 4);
                m.max_experts = std::max(m.max_experts, d.experts);
                if (d.shared_ff > 0 && !par) {
                    reg(&lw.s_gu, (size_t)2 * d.shared_ff * W * 2); reg(&lw.s_down, W * (size_t)d.shared_ff * 2);
                    if (!d.shared_plain) reg(&lw.shared_gate, W * 4);
                    m.max_ff = std::max(m.max_ff, d.shared_ff);
                }
            }
        }
    }
    size_t total = 0;
    for (const Reg& r : regs) total += up256(r.bytes);
    m.slab.alloc(total, /*zero=*/true);
    size_t off = 0;
    for (const Reg& r : regs) { *r.pp = m.slab.p + off; off += up256(r.bytes); }
    if (c.tied_head) m.head = m.embed;
    m.weight_bytes = total - (c.tied_head ? 0 : up256((size_t)m.V * W * 2)) - (c.max_positions > 0 ? up256((size_t)c.max_positions * W * 2) : 0) -
                     (m.bigram ? up256(((size_t)c.bigram_buckets + 1) * W * 2) : 0) - (m.side_embed ? up256((size_t)m.V * m.L * c.token_side * 2) : 0);

    // names -> destinations
    LayeredRoutes R;
    auto mat = [&](const std::string& n, uint16_t* base, int64_t row0, int64_t rows, int64_t cols) {
        R.r[n] = LyRoute{LyRoute::MAT16, base + row0 * cols, rows, cols, 0};
    };
    auto mat_cols = [&](const std::string& n, uint16_t* base, int64_t ld, int64_t col0, int64_t rows, int64_t cols) {     // columns of a wider matrix
        R.r[n] = LyRoute{LyRoute::MAT16, base + col0, rows, cols, 0, ld};
    };
    // rows whose rotary pairs arrive as halves (see LyRoute)
    auto turned = [&](const std::string& n, const fl_layer_desc& d, int per, int at) {
        if (!d.rot_halves) return;
        LyRoute& r = R.r[n];
        r.turn_per = per; r.turn_at = at; r.turn_dims = d.rot_dims;
    };
    auto vec = [&](const std::string& n, float* base, int64_t rows, int64_t cols) { R.r[n] = LyRoute{LyRoute::F32, base, rows, cols, 0}; };
    // a layer norm's weight: [W], or one number for all channels (norm_scalar), kept as W equal floats so that the kernels index it alike
    auto normw = [&](const std::string& n, float* base) { R.r[n] = LyRoute{c.norm_scalar ? LyRoute::F32_FILL : LyRoute::F32, base, (int64_t)W, 1, 0}; };
    auto tanh_parts = [&](const std::string& n, float* b, float* alpha) {
        if (b != nullptr) { vec(n + ".b", b, W, 1); vec(n + ".alpha", alpha, 1, 1); }
    };
    mat("embed", m.embed, 0, m.V, W); normw("final.norm", m.final_norm);
    tanh_parts("final.norm", m.final_bias, m.final_alpha);
    if (m.bigram != nullptr) mat("bigram", m.bigram, 0, (int64_t)c.bigram_buckets + 1, W);
    if (m.side_embed != nullptr) mat("side.embed", m.side_embed, 0, m.V, (int64_t)m.L * c.token_side);
    if (!c.tied_head) mat("head", m.head, 0, m.V, W);
    if (m.embed_norm != nullptr) normw("embed.norm", m.embed_norm);
    if (m.loop_step != nullptr) vec("loop.step", m.loop_step, c.loop_times, W);
    if (m.pos != nullptr) mat("pos", m.pos, 0, c.max_positions, W);
    // the tensors of one mixer, named p + "q" and so on (p = "l<i>.mix." or "l<i>.mix.left." / "l<i>.mix.right.")
    auto route_mixer = [&](const LayeredLayerW& lw, const std::string& p) {
        const fl_layer_desc& d = lw.d;
        const int64_t H = d.heads, D = d.dim, Dv = d.vdim;
        if (d.mixer == FL_MIXER_ATTN) {
            const int64_t G = d.kv_heads;
            mat(p + "q", lw.w_in, lw.off_q, H * D, W);
            if (!d.no_qk_norm) vec(p + "q.norm", lw.qnorm, d.qk_norm_whole ? H * D : D, 1);
            if (d.kv_from < 0) {
                mat(p + "k", lw.w_in, lw.off_k, G * D, W);
                if (lw.off_v >= 0) mat(p + "v", lw.w_in, lw.off_v, G * Dv, W);
                if (!d.no_qk_norm) vec(p + "k.norm", lw.knorm, d.qk_norm_whole ? G * D : D, 1);
            }
            if (d.qkv_bias) { vec(p + "q.b", lw.bq, H * D, 1); vec(p + "k.b", lw.bk, G * D, 1); }
            if (d.qkv_bias && lw.off_v >= 0) vec(p + "v.b", lw.bv, G * Dv, 1);
            if (d.out_gate) mat(p + "g", lw.w_in, lw.off_g, d.out_gate == 2 ? H : H * Dv, W);
            if (d.sink == 2) vec(p + "sink", lw.sinkv, H, 1);
        } else if (d.mixer == FL_MIXER_MAMBA2) {
            mat(p + "in", lw.w_in, lw.off_g, lw.off_dt - lw.off_g + H, W);
            vec(p + "conv", lw.conv_w, lw.conv_ch, d.conv); vec(p + "conv.b", lw.conv_b, lw.conv_ch, 1);
            vec(p + "dt_bias", lw.dt_bias, H, 1); vec(p + "A_log", lw.a_log, H, 1); vec(p + "D", lw.dskip, H, 1);
            vec(p + "norm", lw.hnorm, H * Dv, 1);
        } else if (d.mixer == FL_MIXER_DELTA) {
            const int64_t G = d.kv_heads;
            mat(p + "q", lw.w_in, lw.off_q, G * D, W); mat(p + "k", lw.w_in, lw.off_k, G * D, W);
            mat(p + "v", lw.w_in, lw.off_v, H * Dv, W); mat(p + "g", lw.w_in, lw.off_g, H * Dv, W);
            mat(p + "b", lw.w_in, lw.off_b, H, W); mat(p + "a", lw.w_in, lw.off_a, H, W);
            vec(p + "q.conv", lw.conv_w + (size_t)(lw.off_q - lw.conv_off) * d.conv, G * D, d.conv);
            vec(p + "k.conv", lw.conv_w + (size_t)(lw.off_k - lw.conv_off) * d.conv, G * D, d.conv);
            vec(p + "v.conv", lw.conv_w + (size_t)(lw.off_v - lw.conv_off) * d.conv, H * Dv, d.conv);
            vec(p + "A_log", lw.a_log, H, 1); vec(p + "dt_bias", lw.dt_bias, H, 1); vec(p + "norm", lw.hnorm, Dv, 1);
        } else if (d.mixer == FL_MIXER_LIGHTNING) {
            mat(p + "q", lw.w_in, lw.off_q, H * D, W); mat(p + "k", lw.w_in, lw.off_k, H * D, W);
            mat(p + "v", lw.w_in, lw.off_v, H * Dv, W); mat(p + "g", lw.w_in, lw.off_g, H * Dv, W);
            vec(p + "norm", lw.hnorm, H * Dv, 1);
            R.r[p + "decay"] = LyRoute{LyRoute::F32_RAW, lw.decay, H, 1, 0};
        } else if (d.mixer == FL_MIXER_GLA) {
            mat(p + "q", lw.w_in, lw.off_q, H * D, W); mat(p + "k", lw.w_in, lw.off_k, H * D, W);
            mat(p + "v", lw.w_in, lw.off_v, H * Dv, W); mat(p + "g", lw.w_in, lw.off_g, H * Dv, W);
            mat(p + "a1", lw.w_in, lw.off_a, d.decay_rank, W);
            mat(p + "a2", lw.a2, 0, H * D, d.decay_rank); vec(p + "a2.b", lw.a2b, H * D, 1); vec(p + "norm", lw.hnorm, Dv, 1);
        } else {
            const int64_t Rr = d.rot_dim, C = d.kv_rank, Q = d.q_rank;
            if (Q > 0) {
                mat(p + "dq", lw.w_in, lw.off_q, Q, W); vec(p + "dq.norm", lw.dq_norm, Q, 1); mat(p + "uq", lw.uq, 0, H * (D + Rr), Q);
                turned(p + "uq", d, (int)(D + Rr), (int)D);
            } else {
                mat(p + "q", lw.w_in, lw.off_q, H * (D + Rr), W);
                turned(p + "q", d, (int)(D + Rr), (int)D);
            }
            if (d.out_gate) mat(p + "g", lw.w_in, lw.off_g, d.out_gate == 2 ? H : H * Dv, W);
            if (d.sink == 2) vec(p + "sink", lw.sinkv, H, 1);
            if (d.kv_from < 0) { mat(p + "dkv", lw.w_in, lw.off_dkv, C + Rr, W); turned(p + "dkv", d, (int)(C + Rr), (int)C); vec(p + "dkv.norm", lw.dkv_norm, C, 1); }
            R.r[p + "uk"] = LyRoute{LyRoute::UK_T, lw.uk_t, H * D, C, (int)H};
            mat(p + "uv", lw.uv, 0, H * Dv, C);
        }
        mat_cols(p + "o", lw.w_o, lw.u_ld, 0, W, H * Dv);
    };
    for (int i = 0; i < m.L; ++i) {
        LayeredLayerW& lw = m.layers[i];
        const fl_layer_desc& d = lw.d;
        const std::string p = "l" + std::to_string(i) + ".";
        const bool pre = !c.no_pre_norm, post = !c.no_post_norm;
        if (pre && post) { normw(p + "norm1", lw.norm1); normw(p + "norm1b", lw.norm1b); }
        else normw(p + "norm1", pre ? lw.norm1 : lw.norm1b);
        tanh_parts(p + "norm1", lw.norm1_bias, lw.norm1_alpha);
        if (lw.side_gate) {
            mat(p + "side.gate", lw.side_gate, 0, c.token_side, W); mat(p + "side.proj", lw.side_proj, 0, W, c.token_side);
            vec(p + "side.norm", lw.side_norm, W, 1);
        }
        if (lw.shift) vec(p + "shift", lw.shift, W, 1);
        if (lw.ls1) vec(p + "ls1", lw.ls1, W, 1);
        if (lw.ls2) vec(p + "ls2", lw.ls2, W, 1);
        if (lw.side) {
            lw.side->w_in = lw.w_in;
            route_mixer(lw, p + "mix.left."); route_mixer(*lw.side, p + "mix.right.");
            if (lw.pair_wa) { vec(p + "mix.left.out", lw.pair_wa, W, 1); vec(p + "mix.right.out", lw.pair_wb, W, 1); }
        } else {
            route_mixer(lw, p + "mix.");
        }
        if (lw.canon1) vec(p + "canon1", lw.canon1, W, c.canon_taps);
        if (lw.rg1) { mat(p + "rg1", lw.rg1, 0, W, W); vec(p + "rg1.b", lw.rg1b, W, 1); }
        if (lw.dwa) vec(p + "dwa", lw.dwa, i + 2, 1);
        if (d.ffn == FL_FFN_NONE) continue;
        if (pre && post) { normw(p + "norm2", lw.norm2); normw(p + "norm2b", lw.norm2b); }
        else if (!c.parallel_sub) normw(p + "norm2", pre ? lw.norm2 : lw.norm2b);
        tanh_parts(p + "norm2", lw.norm2_bias, lw.norm2_alpha);
        // the always-on feed-forward of parallel sublayers: rows of w_in, columns of w_o
        auto always_on = [&](const std::string& q) {
            const bool has_gate = d.ffn_act != FL_ACT_RELU2;
            if (has_gate) mat(q + "gate", lw.w_in, lw.off_ff, lw.fx, W);
            mat(q + "up", lw.w_in, lw.off_ff + (has_gate ? lw.fx : 0), lw.fx, W);
            mat_cols(q + "down", lw.w_o, lw.u_ld, lw.u_ld - lw.fx, W, lw.fx);
        };
        if (lw.canon2) vec(p + "canon2", lw.canon2, W, c.canon_taps);
        if (lw.rg2) { mat(p + "rg2", lw.rg2, 0, W, W); vec(p + "rg2.b", lw.rg2b, W, 1); }
        const int64_t F = d.ff;
        const bool gated = d.ffn_act != FL_ACT_RELU2;
        const int64_t GF = gated ? 2 * F : F;
        if (d.ffn == FL_FFN_DENSE && c.parallel_sub) {
            always_on(p + "mlp.");
        } else if (d.ffn == FL_FFN_DENSE) {
            if (gated) mat(p + "mlp.gate", lw.w_gu, 0, F, W);
            mat(p + "mlp.up", lw.w_gu, gated ? F : 0, F, W); mat(p + "mlp.down", lw.w_down, 0, W, F);
            if (d.ffn_bias) {
                vec(p + "mlp.gate.b", lw.b_gu, F, 1); vec(p + "mlp.up.b", lw.b_gu + F, F, 1); vec(p + "mlp.down.b", lw.b_down, W, 1);
            }
        } else {
            vec(p + "mlp.router", lw.router, d.experts, W);
            if (lw.router_b) vec(p + "mlp.router.b", lw.router_b, d.experts, 1);
            if (lw.route_corr) vec(p + "mlp.correction", lw.route_corr, d.experts, 1);
            for (int e = 0; e < d.experts; ++e) {
                const std::string q = p + "mlp.e" + std::to_string(e) + ".";
                if (gated) mat(q + "gate", lw.w_gu, (int64_t)e * GF, F, W);
                mat(q + "up", lw.w_gu, (int64_t)e * GF + (gated ? F : 0), F, W);
                mat(q + "down", lw.w_down, (int64_t)e * W, W, F);
            }
            if (d.shared_ff > 0 && c.parallel_sub) {
                always_on(p + "mlp.shared.");
            } else if (d.shared_ff > 0) {
                const int64_t Fs = d.shared_ff;
                mat(p + "mlp.shared.gate", lw.s_gu, 0, Fs, W); mat(p + "mlp.shared.up", lw.s_gu, Fs, Fs, W);
                mat(p + "mlp.shared.down", lw.s_down, 0, W, Fs);
                if (lw.shared_gate) vec(p + "mlp.shared.sg", lw.shared_gate, 1, W);
            }
        }
    }
    for (const auto& kv : R.r) m.expected.push_back(kv.first);
    std::lock_guard<std::mutex> g(g_routes_mu);
    g_routes[&m] = std::move(R);
}

static const LyRoute* find_route(const LayeredModel& m, const std::string& name) {
    std::lock_guard<std::mutex> g(g_routes_mu);
    auto it = g_routes.find(&m);
    if (it == g_routes.end()) return nullptr;
    auto jt = it->second.r.find(name);
    return jt == it->second.r.end() ? nullptr : &jt->second;
}

void layered_put_tensor(LayeredModel& m, const char* name, int dtype, const int64_t* shape, int rank, const void* host) {
    FL_CHECK(!m.finalized, FL_ERR_STATE, "model already finalized");
    const LyRoute* r = find_route(m, name);
    if (r == nullptr) { m.ignored++; return; }       // a tensor the layers do not read
    int64_t numel = 1;
    for (int i = 0; i < rank; ++i) numel *= shape[i];
    const bool shape_ok = r->kind == LyRoute::F32_FILL
                              ? numel == 1
                              : numel == r->rows * r->cols && (rank == 0 || rank == 1 || (rank == 2 && (shape[0] == r->rows || r->cols == 1 || r->rows == 1)));
    FL_CHECK(shape_ok, FL_ERR_INVALID, std::string("shape mismatch for ") + name);
    FL_CHECK(dtype == FL_DTYPE_F32 || dtype == FL_DTYPE_BF16 || dtype == FL_DTYPE_F16, FL_ERR_INVALID, "bad dtype");
    if (r->kind == LyRoute::F32_RAW && dtype == FL_DTYPE_F32) {
        FL_CUDA(cudaMemcpy(r->dst, host, (size_t)numel * 4, cudaMemcpyHostToDevice));
        m.have.insert(name);
        return;
    }
    std::vector<uint16_t> bits((size_t)numel);
    if (dtype == FL_DTYPE_BF16) std::memcpy(bits.data(), host, (size_t)numel * 2);
    else if (dtype == FL_DTYPE_F32) for (int64_t i = 0; i < numel; ++i) bits[i] = f32_to_bits(((const float*)host)[i]);
    else for (int64_t i = 0; i < numel; ++i) bits[i] = f32_to_bits(half_to_f32(((const uint16_t*)host)[i]));
    if (r->kind == LyRoute::MAT16) {
        if (r->turn_dims > 0) {
            std::vector<uint16_t> t(bits);
            const int half = r->turn_dims / 2;
            for (int64_t b = 0; b < r->rows; b += r->turn_per)
                for (int i = 0; i < r->turn_dims; ++i)
                    std::memcpy(t.data() + (size_t)(b + r->turn_at + i) * r->cols, bits.data() + (size_t)(b + r->turn_at + (i & 1) * half + i / 2) * r->cols,
                                (size_t)r->cols * 2);
            bits.swap(t);
        }
        const int64_t ld = r->ld > 0 ? r->ld : r->cols;
        FL_CUDA(cudaMemcpy2D(r->dst, (size_t)ld * 2, bits.data(), (size_t)r->cols * 2, (size_t)r->cols * 2, (size_t)r->rows, cudaMemcpyHostToDevice));
    } else if (r->kind == LyRoute::F32 || r->kind == LyRoute::F32_RAW) {
        std::vector<float> v((size_t)numel);
        for (int64_t i = 0; i < numel; ++i) v[i] = bits_to_f32(bits[i]);
        FL_CUDA(cudaMemcpy(r->dst, v.data(), (size_t)numel * 4, cudaMemcpyHostToDevice));
    } else if (r->kind == LyRoute::F32_FILL) {
        std::vector<float> v((size_t)(r->rows * r->cols), bits_to_f32(bits[0]));
        FL_CUDA(cudaMemcpy(r->dst, v.data(), v.size() * 4, cudaMemcpyHostToDevice));
    } else {        // [heads * D, C] -> [heads][C][D]
        const int64_t Hh = r->heads, D = r->rows / Hh, C = r->cols;
        std::vector<uint16_t> t((size_t)numel);
        for (int64_t h = 0; h < Hh; ++h)
            for (int64_t d = 0; d < D; ++d)
                for (int64_t c = 0; c < C; ++c) t[(size_t)((h * C + c) * D + d)] = bits[(size_t)((h * D + d) * C + c)];
        FL_CUDA(cudaMemcpy(r->dst, t.data(), (size_t)numel * 2, cudaMemcpyHostToDevice));
    }
    m.have.insert(name);
}

void layered_random_init(LayeredModel& m, uint64_t seed, float stdv) {
    FL_CHECK(!m.finalized, FL_ERR_STATE, "model already finalized");
    const RowMap ident{0, 0, 0, 0};
    for (const std::string& n : m.expected) {
        const LyRoute* r = find_route(m, n);
        const uint64_t ts = tensor_seed(seed, n.c_str());
        const int64_t numel = r->rows * r->cols;
        if (r->kind == LyRoute::F32 || r->kind == LyRoute::F32_RAW || r->kind == LyRoute::F32_FILL) {
            auto ends = [&](const char* t) { const size_t k = std::strlen(t); return n.size() >= k && n.compare(n.size() - k, k, t) == 0; };
            // a plain norm weight sits around one, a zero-centred one around zero
            const bool around_one = ends("mix.norm") || ends("left.norm") || ends("right.norm") || ends("dkv.norm") || ends("dq.norm") || n == "embed.norm" || ends(".ls1") || ends(".ls2") || ends("side.norm") || ends("q.norm") || ends("k.norm") || ends("mix.D") || ends("left.out") || ends("right.out") ||
                                    (m.cfg.norm_plain && (ends("norm1") || ends("norm2") || ends("norm1b") || ends("norm2b") || n == "final.norm"));
            const bool is_mat = n.find("router") != std::string::npos || n.find("mix.a2") != std::string::npos || n.find("shared.sg") != std::string::npos ||
                                ends(".conv") || ends(".canon1") || ends(".canon2") || n == "loop.step";
            const bool is_bias = n.size() >= 4 && n.compare(n.size() - 4, 4, "a2.b") == 0;
            if (around_one) fill_f32_kernel<<<8, 256>>>((float*)r->dst, numel, 1.0f);
            else if (ends(".decay")) fill_f32_kernel<<<8, 256>>>((float*)r->dst, numel, 0.96875f);
            else if (ends(".alpha")) fill_f32_kernel<<<8, 256>>>((float*)r->dst, numel, 0.5f);
            else if (ends(".shift")) fill_f32_kernel<<<8, 256>>>((float*)r->dst, numel, 0.25f);
            else if (ends(".dwa")) fill_f32_kernel<<<8, 256>>>((float*)r->dst, numel, 1.0f / (float)numel);     // a plain mean over the outputs so far
            else if (is_bias) fill_f32_kernel<<<8, 256>>>((float*)r->dst, numel, 3.0f);
            else if (is_mat) synth_fill_f32_kernel<<<kNumSMs, 256>>>((float*)r->dst, numel, ts, stdv, ident);
            else fill_f32_kernel<<<8, 256>>>((float*)r->dst, numel, 0.0f);
        } else {
            const bool unit = (n == "embed" && !m.cfg.tied_head) || n == "bigram" || n == "side.embed";
            if (r->ld > 0) synth_fill_bf16_kernel<<<kNumSMs * 8, 256>>>((uint16_t*)r->dst, r->rows, r->cols, r->ld, ts, stdv, ident);
            else synth_fill_bf16_kernel<<<kNumSMs * 8, 256>>>((uint16_t*)r->dst, 1, numel, numel, ts, unit ? 1.0f : stdv, ident);
        }
        g_launches.fetch_add(1);
        m.have.insert(n);
    }
    FL_CUDA(cudaGetLastError());
    FL_CUDA(cudaDeviceSynchronize());
}

void layered_finalize(LayeredModel& m) {
    FL_CHECK(!m.finalized, FL_ERR_STATE, "model already finalized");
    for (const std::string& n : m.expected) FL_CHECK(m.have.count(n), FL_ERR_STATE, "missing tensor: " + n);
    {
        std::lock_guard<std::mutex> g(g_routes_mu);
        g_routes.erase(&m);
    }
    // serving precision: the projections whose rows are whole 16-byte pieces run on the tcgen05 GEMM (a K that ends inside a 64-column
    // k block is filled up with zeros by the tensor maps of both operands); everything else, and every product of the exact mode, stays on the f32 FMA kernel
    if (!m.f32 && !env_flag("FL_LAYERED_NO_TC")) {
        auto fits = [](int N, int K) { return K % 8 == 0 && N % 8 == 0; };
        auto map = [&](const uint16_t* p, int N, int K, CUtensorMap& tm, bool& ok) {
            ok = p != nullptr && fits(N, K);
            if (ok) tm = make_tmap_bf16(p, (uint64_t)N, (uint64_t)K, (uint64_t)K, 128);
        };
        for (LayeredLayerW& lw : m.layers) {
            const fl_layer_desc& d = lw.d;
            map(lw.w_in, lw.n_in, m.W, lw.tm_in, lw.tc_in);
            map(lw.w_o, m.W, lw.u_ld, lw.tm_o, lw.tc_o);
            if (d.mixer == FL_MIXER_LATENT_ATTN) {
                // sizes in multiples of 8 may end inside a k block (the tensor maps fill its rest with zeros)
                const int H = d.heads, D = d.dim, Dv = d.vdim, C = d.kv_rank, R = d.rot_dim;
                lw.lat_tc = D % 8 == 0 && Dv % 8 == 0 && C % 8 == 0 && R % 8 == 0 && m.W % 8 == 0 && lw.u_ld % 8 == 0 &&
                            (d.out_gate != 1 || lw.off_g % 4 == 0) && lw.n_in % 4 == 0;
                if (lw.lat_tc) {
                    lw.tm_uk = make_tmap_bf16(lw.uk_t, (uint64_t)H * C, (uint64_t)D, (uint64_t)D, 128);
                    lw.tm_uv = make_tmap_bf16(lw.uv, (uint64_t)H * Dv, (uint64_t)C, (uint64_t)C, 128);
                    m.max_hp = std::max(m.max_hp, H * D); m.max_hq = std::max(m.max_hq, H * ((C + R + 63) / 64 * 64)); m.max_c = std::max(m.max_c, C);
                }
            }
            // (a query latent may end inside a k block: the tensor maps fill its rest with zeros)
            lw.tc_uq = lw.uq != nullptr && d.q_rank % 8 == 0 && d.heads * (d.dim + d.rot_dim) % 8 == 0;
            if (lw.tc_uq) {
                const uint64_t nq = (uint64_t)d.heads * (d.dim + d.rot_dim), Q = d.q_rank;
                lw.tm_uq = make_tmap_bf16(lw.uq, nq, Q, Q, 128);
            }
            if (lw.side) map(lw.side->w_o, m.W, lw.side->d.heads * lw.side->d.vdim, lw.side->tm_o, lw.side->tc_o);
            map(lw.rg1, m.W, m.W, lw.tm_rg1, lw.tc_rg1); map(lw.rg2, m.W, m.W, lw.tm_rg2, lw.tc_rg2);
            const int GF = d.ffn_act == FL_ACT_RELU2 ? d.ff : 2 * d.ff;       // rows of the first feed-forward matrix: up, or gate | up
            map(lw.side_gate, m.cfg.token_side, m.W, lw.tm_tgate, lw.tc_tgate); map(lw.side_proj, m.W, m.cfg.token_side, lw.tm_tproj, lw.tc_tproj);
            if (d.ffn == FL_FFN_DENSE) { map(lw.w_gu, GF, m.W, lw.tm_gu, lw.tc_gu); map(lw.w_down, m.W, d.ff, lw.tm_down, lw.tc_down); }
            if (d.ffn == FL_FFN_MOE && d.shared_ff > 0) {
                map(lw.s_gu, 2 * d.shared_ff, m.W, lw.tm_sgu, lw.tc_sgu); map(lw.s_down, m.W, d.shared_ff, lw.tm_sdown, lw.tc_sdown);
            }
            if (d.ffn == FL_FFN_MOE && fits(GF, m.W) && fits(m.W, d.ff)) {
                lw.tc_moe = true;
                lw.tm_gu = make_tmap_bf16(lw.w_gu, (uint64_t)d.experts * GF, (uint64_t)m.W, (uint64_t)m.W, 128);
                lw.tm_down = make_tmap_bf16(lw.w_down, (uint64_t)d.experts * m.W, (uint64_t)d.ff, (uint64_t)d.ff, 128);
                for (int e = 0; e < d.experts; ++e) {
                    lw.tm_egu.push_back(make_tmap_bf16(lw.w_gu + (size_t)e * GF * m.W, (uint64_t)GF, (uint64_t)m.W, (uint64_t)m.W, 128));
                    lw.tm_edown.push_back(make_tmap_bf16(lw.w_down + (size_t)e * m.W * d.ff, (uint64_t)m.W, (uint64_t)d.ff, (uint64_t)d.ff, 128));
                }
            }
        }
        map(m.head, m.V, m.W, m.tm_head, m.tc_head);
    }
    // the norms behind a sublayer park a row in shared memory: above the default 48 KB the kernels are told so once
    if ((!m.cfg.no_post_norm || m.cfg.token_side > 0) && (size_t)m.W * 4 > 48 * 1024) {
        FL_CHECK((size_t)m.W * 4 <= 200 * 1024, FL_ERR_UNSUPPORTED, "norms behind a sublayer are built for widths up to 51200");
        FL_CUDA(cudaFuncSetAttribute(ly_post_norm_kernel<4>, cudaFuncAttributeMaxDynamicSharedMemorySize, m.W * 4));
        FL_CUDA(cudaFuncSetAttribute(ly_post_norm_kernel<1>, cudaFuncAttributeMaxDynamicSharedMemorySize, m.W * 4));
        FL_CUDA(cudaFuncSetAttribute(ly_sum_norm_kernel<4>, cudaFuncAttributeMaxDynamicSharedMemorySize, m.W * 4));
        FL_CUDA(cudaFuncSetAttribute(ly_sum_norm_kernel<1>, cudaFuncAttributeMaxDynamicSharedMemorySize, m.W * 4));
    }
    m.finalized = true;
}

// ---- cache -------------------------------------------------------------------------------------------------------------------
static void rope_tables(const RopeSpec& rs, int max_seq, std::vector<float>& cs, std::vector<float>& sn) {
    const int half = rs.dims / 2;
    std::vector<double> f(half);
    double mult = 1.0;
    for (int i = 0; i < half; ++i) f[i] = std::pow(rs.base, -2.0 * i / (double)rs.dims);
    if (rs.yarn_factor > 0.f && rs.scaling == FL_ROT_SCALE_BANDS) {
        // bands of wavelength: short ones (below original / fast) keep their frequency, long ones (above original / slow) are slowed
        // by the factor, between the two a linear blend in original / wavelength; magnitude 1
        const double factor = rs.yarn_factor, orig = rs.yarn_original, hi = rs.yarn_fast, lo = rs.yarn_slow;
        for (int i = 0; i < half; ++i) {
            const double wl = 2.0 * M_PI / f[i];
            if (wl < orig / hi) continue;
            if (wl > orig / lo) { f[i] /= factor; continue; }
            const double sm = (orig / wl - lo) / (hi - lo);
            f[i] = (1.0 - sm) * f[i] / factor + sm * f[i];
        }
    } else if (rs.yarn_factor > 0.f) {
        // YaRN: pairs that complete many turns inside the original context keep their frequency, slow pairs are stretched by the
        // factor, a linear ramp between the two pair indices; cos and sin grow by 0.1 ln(factor) + 1
        const double factor = rs.yarn_factor, orig = rs.yarn_original;
        auto corr = [&](double turns) { return rs.dims * std::log(orig / (2.0 * M_PI * turns)) / (2.0 * std::log(rs.base)); };
        const double lo = std::max(std::floor(corr(rs.yarn_fast)), 0.0), hi = std::min(std::ceil(corr(rs.yarn_slow)), (double)rs.dims - 1.0);
        for (int i = 0; i < half; ++i) {
            const double ramp = std::min(1.0, std::max(0.0, (i - lo) / std::max(hi - lo, 0.001)));
            f[i] = f[i] / factor * ramp + f[i] * (1.0 - ramp);
        }
        mult = 0.1 * std::log(factor) + 1.0;
    }
    cs.resize((size_t)max_seq * half); sn.resize((size_t)max_seq * half);
    for (int p = 0; p < max_seq; ++p)
        for (int i = 0; i < half; ++i) {
            cs[(size_t)p * half + i] = (float)(std::cos(p * f[i]) * mult);
            sn[(size_t)p * half + i] = (float)(std::sin(p * f[i]) * mult);
        }
}

static KvLayout kv_layout(const fl_layer_desc& d) {
    const int G = d.kv_heads, D = d.dim, Dv = d.vdim, r = d.rot_dims;
    if (d.v_from_k) return KvLayout{G * (D + r), D + r, r, D + r, r == D ? 0 : r};
    return KvLayout{G * (D + Dv), D, G * D, Dv, 0};
}

void layered_cache_create(fl_cache& c, int max_slots, int max_seq, int pool_tokens) {
    const LayeredModel& m = *c.lm;
    FL_CHECK(m.finalized, FL_ERR_STATE, "model not finalized");
    FL_CHECK(max_slots >= 1 && max_slots <= kMaxBatch && max_seq >= 1 && pool_tokens >= 1, FL_ERR_INVALID, "bad cache dimensions");
    c.max_batch = max_slots; c.max_seq = max_seq;
    c.pages_per_seq = (max_seq + kKvPage - 1) / kKvPage;
    FL_CUDA(cudaStreamCreateWithFlags(&c.stream, cudaStreamNonBlocking));
    c.ly.reset(new LayeredCache);
    LayeredCache& y = *c.ly;
    y.f32 = m.f32;
    const int pages = (pool_tokens + kKvPage - 1) / kKvPage;
    y.pool = PagePool(pages, max_slots, c.pages_per_seq, kKvPage);
    const size_t esz = m.f32 ? 4 : 2;
    y.kv_store.resize(m.kv_layers.size());
    for (size_t k = 0; k < m.kv_layers.size(); ++k) {
        const fl_layer_desc& d = m.kv_layers[k]->d;
        const size_t width = d.mixer == FL_MIXER_ATTN ? (size_t)kv_layout(d).E : (size_t)(d.kv_rank + d.rot_dim);
        y.kv_store[k].alloc((size_t)pages * kKvPage * width * esz, true);
        y.kv_pool.push_back(y.kv_store[k].p);
    }
    y.gla_state.resize(m.gla_layers.size());
    y.conv_state.resize(m.gla_layers.size());
    for (size_t k = 0; k < m.gla_layers.size(); ++k) {
        const LayeredLayerW& lw = *m.gla_layers[k];
        const fl_layer_desc& d = lw.d;
        const size_t rows = d.mixer == FL_MIXER_MAMBA2 ? d.state : d.dim;
        y.gla_state[k].alloc((size_t)max_slots * d.heads * rows * d.vdim, true);
        if (lw.conv_ch > 0 && d.conv > 1) y.conv_state[k].alloc((size_t)max_slots * (d.conv - 1) * lw.conv_ch, true);
    }
    if (m.cfg.canon_taps > 1) {
        y.canon_state.resize(m.runs.size());
        for (size_t i = 0; i < m.runs.size(); ++i) y.canon_state[i].alloc((size_t)2 * max_slots * (m.cfg.canon_taps - 1) * m.W, true);
    }
    if (m.cfg.token_shift) {
        y.shift_state.resize(m.runs.size());
        for (size_t i = 0; i < m.runs.size(); ++i) y.shift_state[i].alloc((size_t)max_slots * m.W, true);
    }
    y.rope_cos.resize(m.ropes.size()); y.rope_sin.resize(m.ropes.size());
    for (size_t k = 0; k < m.ropes.size(); ++k) {
        std::vector<float> cs, sn;
        rope_tables(m.ropes[k], max_seq, cs, sn);
        y.rope_cos[k].alloc(std::max<size_t>(cs.size(), 1)); y.rope_sin[k].alloc(std::max<size_t>(sn.size(), 1));
        if (!cs.empty()) {
            FL_CUDA(cudaMemcpy(y.rope_cos[k].p, cs.data(), cs.size() * 4, cudaMemcpyHostToDevice));
            FL_CUDA(cudaMemcpy(y.rope_sin[k].p, sn.data(), sn.size() * 4, cudaMemcpyHostToDevice));
        }
    }
    y.page_table.alloc((size_t)max_slots * c.pages_per_seq, true);
    {
        size_t part = m.max_av > 0 && !m.f32 ? (size_t)kGqaSplitRows * kGqaMaxSplits * (m.max_av + 2) : 0;
        if (m.max_c > 0) part = std::max(part, (size_t)kNumSMs * 32 * (m.max_c + 2));
        y.at_part.alloc(part);
    }
    c.slot_len.assign(max_slots, 0);
    y.slot_last.assign(max_slots, -1);
    FL_CUDA(cudaDeviceSynchronize());
}

void layered_slot_reset(fl_cache& c, int slot) {
    c.ly->pool.release(slot);       // the recurrent state needs no clearing: a sequence that starts at position 0 starts from zero
    c.slot_len[slot] = 0;
    c.ly->slot_last[slot] = -1;
}

void layered_cache_reset(fl_cache& c) {
    for (int s = 0; s < c.max_batch; ++s) layered_slot_reset(c, s);
}

// captured decode steps hold workspace pointers: they go when a buffer they name is reallocated
static void drop_graphs(fl_cache& c) {
    for (auto& kv : c.graphs)
        if (kv.second.exec) cudaGraphExecDestroy(kv.second.exec);
    c.graphs.clear();
}

static void ensure_ws(fl_cache& c, size_t T, size_t n_want) {
    const LayeredModel& m = *c.lm;
    LayeredCache& y = *c.ly;
    if (T > y.rows) {
        FL_CUDA(cudaStreamSynchronize(c.stream));
        drop_graphs(c);
        const size_t R = std::max<size_t>(T, 2 * y.rows), W = m.W, P = R * std::max(m.max_top, 1);
        y.x.alloc(R * W); y.h.alloc(R * W); y.y.alloc(R * W);
        y.proj.alloc(R * m.max_in); y.u.alloc(R * std::max(m.max_u, 1)); y.go.alloc(R * std::max(m.max_hv, 1));
        y.la.alloc(R * std::max(m.max_hd, 1));
        y.cv.alloc(R * std::max(m.max_cv, 1)); y.rs.alloc(R * 2 * std::max(m.max_heads, 1));
        if (m.cfg.canon_taps > 0 || m.cfg.token_shift) y.hc.alloc(R * W);
        if (m.cfg.gated_residual) y.gz.alloc(R * W);
        if (m.cfg.depth_avg) y.xs.alloc((size_t)(m.L + 1) * R * W);
        else if (m.cfg.loop_reinject) y.xs.alloc(R * W);
        if (m.max_qr > 0) { y.cq.alloc(R * m.max_qr); y.qx.alloc(R * m.max_q); }
        if (m.cfg.token_side > 0) { y.tz.alloc(R * m.cfg.token_side); y.ta.alloc(R * m.cfg.token_side); }
        for (const LayeredLayerW& lw : m.layers)
            if ((lw.side || (m.cfg.parallel_sub && lw.d.ffn == FL_FFN_MOE)) && y.y2.n < R * W) y.y2.alloc(R * W);
        bool plain_latent = false;          // a latent attention that is not on the tensor cores keeps f32 query / value rows
        for (const LayeredLayerW& lw : m.layers) plain_latent |= lw.d.mixer == FL_MIXER_LATENT_ATTN && !lw.lat_tc;
        if (plain_latent) { y.qa.alloc(R * m.max_hc); y.ol.alloc(R * m.max_hc); }
        if (m.max_hq > 0) {
            y.qp_hi.alloc(R * m.max_hp); y.qp_lo.alloc(R * m.max_hp); y.qo_hi.alloc(R * m.max_hq); y.qo_lo.alloc(R * m.max_hq);
            y.ol_hi.alloc(R * m.max_hc); y.ol_lo.alloc(R * m.max_hc);
        }
        y.gu.alloc(P * 2 * std::max(m.max_ff, 1)); y.act.alloc(P * std::max(m.max_ff, 1)); y.eo.alloc(P * W);
        y.sh_gu.alloc(R * 2 * std::max(m.max_ff, 1)); y.sh_act.alloc(R * std::max(m.max_ff, 1)); y.sh_o.alloc(R * W);
        y.route_w.alloc(P); y.route_sel.alloc(P); y.sgate.alloc(R);
        y.pair_row.alloc(P); y.pair_of.alloc(P); y.grp_off.alloc((size_t)m.max_experts + 2);
        if (!m.f32) {
            y.h_hi.alloc(R * W); y.h_lo.alloc(R * W);
            if (m.max_qr > 0) { y.cq_hi.alloc(R * m.max_qr); y.cq_lo.alloc(R * m.max_qr); }
            y.u_hi.alloc(R * std::max(m.max_u, 1)); y.u_lo.alloc(R * std::max(m.max_u, 1));
            if (m.cfg.token_side > 0) { y.ta_hi.alloc(R * m.cfg.token_side); y.ta_lo.alloc(R * m.cfg.token_side); }
            y.act_hi.alloc(R * std::max(m.max_ff, 1)); y.act_lo.alloc(R * std::max(m.max_ff, 1));
            // split-K slices of a tensor-core GEMM with <= 128 rows: ks * rows <= 256 (see pick_ksplit)
            const size_t nmax = std::max<size_t>(std::max<size_t>(std::max(m.max_in, m.max_q), W), std::max<size_t>(std::max<size_t>(2 * (size_t)m.max_ff, m.cfg.token_side), m.V));
            size_t need = 256 * nmax;
            size_t gx_rows = 0;
            for (const LayeredLayerW& lw : m.layers) {          // grouped expert GEMMs: [slices][experts * cap rows][2 ff | W]
                if (!lw.tc_moe) continue;
                const int E = lw.d.experts, F = lw.d.ff, GF = lw.d.ffn_act == FL_ACT_RELU2 ? F : 2 * F;
                gx_rows = std::max<size_t>(gx_rows, (size_t)E * 128);
                for (int cap = 16; cap <= 128; cap *= 2) {
                    const int k1 = pick_ksplit(E * ((GF + 127) / 128), (int)(W + 63) / 64, cap), k2 = pick_ksplit(E * ((int)(W + 127) / 128), (F + 63) / 64, cap);
                    need = std::max(need, std::max((size_t)k1 * E * cap * GF, (size_t)k2 * E * cap * W));
                }
            }
            if (y.gemm_out.n < need) y.gemm_out.alloc(need);
            if (gx_rows > 0 && y.gx_hi.n == 0) {
                y.gx_hi.alloc(gx_rows * W, true); y.gx_lo.alloc(gx_rows * W, true);
                y.ga_hi.alloc(gx_rows * std::max(m.max_ff, 1), true); y.ga_lo.alloc(gx_rows * std::max(m.max_ff, 1), true);
                y.grp_cnt.alloc((size_t)m.max_experts + 1, true);
            }
        }
        y.rows = R;
    }
    if (n_want > y.want_cap) {
        FL_CUDA(cudaStreamSynchronize(c.stream));
        drop_graphs(c);
        const size_t N = std::max<size_t>(n_want, 2 * y.want_cap);
        y.hf.alloc(N * m.W); y.logits.alloc(N * m.V); y.h_logits.alloc(N * m.V);
        if (!m.f32) { y.hf_hi.alloc(N * m.W); y.hf_lo.alloc(N * m.W); }
        y.want_cap = N;
    }
}

// The FMA-chain GEMM: f32 accumulators where it stands in for the tensor-core GEMM on shapes outside its tiles (serving precision),
// f64 accumulators in the exact mode.
static void gemm(LaunchCtx& lc, const char* tag, const float* A, int lda, const uint16_t* Wt, int N, int K, float* Y, int ldy, int R) {
    if (R <= 0) return;
    LyGemm g{A, 0, lda, nullptr, Wt, 0, N, K, Y, 0, ldy, nullptr, R};
    const dim3 grid((N + kLyBN - 1) / kLyBN, (R + kLyBM - 1) / kLyBM, 1);
    if (lc.exact) launch(lc, tag, (uint64_t)N * K * 2, ly_gemm_kernel<double>, grid, dim3(256), 0, g);
    else launch(lc, tag, (uint64_t)N * K * 2, ly_gemm_kernel<float>, grid, dim3(256), 0, g);
}
// Y[R, N] = A[R, K] . Wt[N, K]^T on the tensor cores when the matrix has a descriptor (serving precision; A as hi | lo halves),
// else on the exact kernel.  A tensor-core GEMM of few rows may leave split-K slices in the shared scratch: the caller hands them to
// the kernel that reads the result next (before another split GEMM runs), which folds them in slice order.
static Slices gemm_slices(fl_cache& c, LaunchCtx& lc, const char* tag, const float* A, const uint16_t* ahi, const uint16_t* alo, const uint16_t* Wt,
                          const CUtensorMap& tm, bool tc, int N, int K, float* Y, int R) {
    if (R <= 0) return Slices{Y, 1, 0};
    if (!tc || ahi == nullptr) { gemm(lc, tag, A, K, Wt, N, K, Y, N, R); return Slices{Y, 1, 0}; }
    LayeredCache& y = *c.ly;
    int ks_plan = R <= 128 ? pick_ksplit((N + 127) / 128, (K + 63) / 64, R) : 1;
    if (R > 128) {              // many rows but few output tiles (a narrow matrix): cut K as long as the slices fit the scratch
        const int tiles = ((R + 127) / 128) * ((N + 255) / 256), nk = (K + 63) / 64;
        // (up to eight slices of at least eight k blocks: none of them is empty)
        while (ks_plan < 8 && 2 * ks_plan * tiles <= kNumSMs && nk / (2 * ks_plan) >= 8 && (size_t)(2 * ks_plan) * R * N <= y.gemm_out.n) ks_plan *= 2;
    }
    float* out = ks_plan == 1 ? Y : y.gemm_out.p;
    FL_CHECK(ks_plan == 1 || (size_t)ks_plan * R * N <= y.gemm_out.n, FL_ERR_STATE, "internal: split-K scratch too small");
    const int ks = dense_gemm(c, lc, tag, R, N, K, tm, out, ahi, alo, nullptr, nullptr, R > 128 ? ks_plan : 1);
    FL_CHECK(ks == ks_plan, FL_ERR_STATE, "internal: split-K plan mismatch");
    return Slices{out, ks, (size_t)R * N};
}
// the same with the slices folded into Y
static void gemm_tc_or_exact(fl_cache& c, LaunchCtx& lc, const char* tag, const float* A, const uint16_t* ahi, const uint16_t* alo, const uint16_t* Wt,
                             const CUtensorMap& tm, bool tc, int N, int K, float* Y, int R) {
    const Slices s = gemm_slices(c, lc, tag, A, ahi, alo, Wt, tm, tc, N, K, Y, R);
    if (s.n > 1)
        launch(lc, "sum_slices", 0, ly_sum_slices_kernel, dim3((unsigned)std::min<size_t>(4 * kNumSMs, (s.stride + 255) / 256)), dim3(256), 0,
               s.p, s.n, s.stride, s.stride, Y);
}
// feed-forward activation of `rows` rows (see ly_glu_kernel)
// (ldg, ldo: row strides of gu and of the output; 0 = dense rows.  gu.p, out, hi, lo may start inside a row.)
static void launch_glu(LaunchCtx& lc, const Slices& gu, int rows, int F, float limit, int act, const float* bias, float* out, uint16_t* hi, uint16_t* lo, int ldg = 0,
                       int ldo = 0) {
    if (rows <= 0) return;
    if (ldg == 0) ldg = act == FL_ACT_RELU2 ? F : 2 * F;
    if (ldo == 0) ldo = F;
    auto al = [](const void* p, size_t n) { return (reinterpret_cast<uintptr_t>(p) & (n - 1)) == 0; };
    if (((F | ldg | ldo) & 3) == 0 && (gu.stride & 3) == 0 && al(gu.p, 16) && al(out, 16) && al(hi, 8) && al(lo, 8))
        launch(lc, "glu", 0, ly_glu_kernel<4>, dim3(rows, (F + 1023) / 1024), dim3(256), 0, gu, ldg, ldo, F, limit, act, bias, out, hi, lo);
    else
        launch(lc, "glu", 0, ly_glu_kernel<1>, dim3(rows, (F + 255) / 256), dim3(256), 0, gu, ldg, ldo, F, limit, act, bias, out, hi, lo);
}

static void gemm_groups(LaunchCtx& lc, const char* tag, const LyGemm& g, int groups, int max_rows) {
    if (max_rows <= 0) return;
    const dim3 grid((g.N + kLyBN - 1) / kLyBN, (max_rows + kLyBM - 1) / kLyBM, groups);
    if (lc.exact) launch(lc, tag, (uint64_t)groups * g.N * g.K * 2, ly_gemm_kernel<double>, grid, dim3(256), 0, g);
    else launch(lc, tag, (uint64_t)groups * g.N * g.K * 2, ly_gemm_kernel<float>, grid, dim3(256), 0, g);
}

template <typename CT>
static void launch_latent_attn(LaunchCtx& lc, const LatentAttnArgs& a, int T) {
    const int cpl = (a.C + 31) / 32;
    const size_t smem = ((size_t)kLatWarps * a.C + 2 * kLatWarps) * 4;
    const dim3 g(T, a.H), b(kLatWarps * 32);
    const uint64_t bytes = 0;
    if (cpl <= 1) launch(lc, "latent_attn", bytes, ly_latent_attn_kernel<CT, 1>, g, b, smem, a);
    else if (cpl <= 2) launch(lc, "latent_attn", bytes, ly_latent_attn_kernel<CT, 2>, g, b, smem, a);
    else if (cpl <= 4) launch(lc, "latent_attn", bytes, ly_latent_attn_kernel<CT, 4>, g, b, smem, a);
    else if (cpl <= 8) launch(lc, "latent_attn", bytes, ly_latent_attn_kernel<CT, 8>, g, b, smem, a);
    else launch(lc, "latent_attn", bytes, ly_latent_attn_kernel<CT, 16>, g, b, smem, a);
}

template <int MT, int NT>
static void launch_latent_mma_t(LaunchCtx& lc, const LatMmaArgs& a, int T, int splits) {
    static bool attr_set = false;
    if (!attr_set) {
        FL_CUDA(cudaFuncSetAttribute(ly_latent_mma_kernel<MT, NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kLatSmemMax));
        attr_set = true;
    }
    launch(lc, "latent_attn", 0, ly_latent_mma_kernel<MT, NT>, dim3(T, (a.H + 16 * MT - 1) / (16 * MT), splits), dim3(256), lat_mma_smem(a.Ep, MT), a);
}
// max_keys: the most keys a row of the launch can see.  Few (row, head group) pairs split each row's pages over several blocks.
static void launch_latent_mma(LaunchCtx& lc, const LatMmaArgs& a, int T, int max_keys) {
    if (T <= 0) return;
    const bool wide = a.H > 16 && lat_mma_smem(a.Ep, 2) <= kLatSmemMax;        // two groups of 16 heads share a block's tiles
    const int groups = wide ? (a.H + 31) / 32 : (a.H + 15) / 16;
    int splits = std::max(1, std::min(kGqaMaxSplits, kNumSMs / (T * groups)));
    splits = std::min(splits, (max_keys + kLatTile - 1) / kLatTile);
    auto go = [&](auto mt) {
        constexpr int MT = decltype(mt)::value;
        if (a.C <= 64) launch_latent_mma_t<MT, 1>(lc, a, T, splits);
        else if (a.C <= 128) launch_latent_mma_t<MT, 2>(lc, a, T, splits);
        else if (a.C <= 256) launch_latent_mma_t<MT, 4>(lc, a, T, splits);
        else launch_latent_mma_t<MT, 8>(lc, a, T, splits);
    };
    if (wide) go(std::integral_constant<int, 2>{}); else go(std::integral_constant<int, 1>{});
    if (splits > 1)
        launch(lc, "latent_merge", 0, ly_gqa_merge_kernel, dim3(T, a.H), dim3(std::min(256, (a.C + 31) / 32 * 32)), 0, (const float*)a.part, splits, a.H, a.C, a.sink,
               a.sinkv, a.row_base, a.H * a.C, 0, OutGate{}, (float*)nullptr, a.ohi, a.olo);
}

static void launch_gla_scan(LaunchCtx& lc, const GlaArgs& a, int n) {
    const int rpt = (a.D + kGlaDG - 1) / kGlaDG;
    const size_t smem = ((size_t)6 * a.D + 2 * kGlaVS + 2 * kGlaDG * kGlaVS) * 4;
    const dim3 g(n, a.H, (a.Dv + kGlaVS - 1) / kGlaVS), b(kGlaVS * kGlaDG);
    if (rpt <= 1) launch(lc, "gla_scan", 0, ly_gla_scan_kernel<1>, g, b, smem, a);
    else if (rpt <= 2) launch(lc, "gla_scan", 0, ly_gla_scan_kernel<2>, g, b, smem, a);
    else if (rpt <= 4) launch(lc, "gla_scan", 0, ly_gla_scan_kernel<4>, g, b, smem, a);
    else if (rpt <= 8) launch(lc, "gla_scan", 0, ly_gla_scan_kernel<8>, g, b, smem, a);
    else if (rpt <= 16) launch(lc, "gla_scan", 0, ly_gla_scan_kernel<16>, g, b, smem, a);
    else launch(lc, "gla_scan", 0, ly_gla_scan_kernel<32>, g, b, smem, a);
}

template <typename CT, int RB>
static void launch_gqa_attn_rb(LaunchCtx& lc, const GqaAttnArgs& a, int T, int splits) {
    const int cpl = (std::max(a.D, a.Dv) + 31) / 32;
    const size_t smem = ((size_t)kGqaWarps * RB * (a.Dv + 2)) * 4;
    const dim3 g(T, a.H / RB, splits), b(kGqaWarps * 32);
    auto go = [&](auto c) {
        constexpr int CPL = decltype(c)::value;
        const size_t al = std::min<size_t>(16, CPL * sizeof(CT)) - 1, es = sizeof(CT);
        const bool vec = a.D % CPL == 0 && a.Dv % CPL == 0 && (((size_t)a.kv.E * es | (size_t)a.kv.ks * es | (size_t)a.kv.vo * es | (size_t)a.kv.vs * es) & al) == 0;
        if (vec) launch(lc, "gqa_attn", 0, ly_gqa_attn_kernel<CT, CPL, RB, true>, g, b, smem, a);
        else launch(lc, "gqa_attn", 0, ly_gqa_attn_kernel<CT, CPL, RB, false>, g, b, smem, a);
    };
    if (cpl <= 1) go(std::integral_constant<int, 1>{});
    else if (cpl <= 2) go(std::integral_constant<int, 2>{});
    else if (cpl <= 4) go(std::integral_constant<int, 4>{});
    else go(std::integral_constant<int, 8>{});
}
// max_keys: the most keys a row of the launch can see (bounds the useful number of key splits).  The exact mode never splits: there
// a position's result is bitwise the same whatever else the launch holds.
template <typename CT>
static void launch_gqa_attn(LaunchCtx& lc, const GqaAttnArgs& a, int T, int max_keys, bool may_split) {
    if (T <= 0) return;
    const int rep = a.H / a.G, rb = rep % 4 == 0 ? 4 : (rep % 2 == 0 ? 2 : 1);
    int splits = 1;
    if (may_split && a.part != nullptr && (long long)T * a.H <= kGqaSplitRows) {
        const int blocks = T * (a.H / rb);
        splits = std::min(kGqaMaxSplits, std::max(1, 2 * kNumSMs / std::max(blocks, 1)));
        splits = std::max(1, std::min(splits, max_keys / (kGqaWarps * 16)));        // at least 16 keys per warp
    }
    if (rb == 4) launch_gqa_attn_rb<CT, 4>(lc, a, T, splits);
    else if (rb == 2) launch_gqa_attn_rb<CT, 2>(lc, a, T, splits);
    else launch_gqa_attn_rb<CT, 1>(lc, a, T, splits);
    if (splits > 1)
        launch(lc, "gqa_merge", 0, ly_gqa_merge_kernel, dim3(T, a.H), dim3(std::min(256, std::max(32, (a.Dv + 31) / 32 * 32))), 0, (const float*)a.part, splits,
               a.H, a.Dv, a.sink, a.sinkv, a.row_base, a.ldo, a.kv.roll, a.gate, a.out, a.ohi, a.olo);
}

template <bool DELTA>
static void launch_rec_scan(LaunchCtx& lc, const RecArgs& a, int n) {
    const int rpt = (a.D + kRecParts - 1) / kRecParts;
    auto go = [&](auto kern, int RPT) {
        const size_t smem = (size_t)4 * (RPT >= 64 ? 4 : 8) * (2 * kRecParts * (RPT + 4) + 12) * 4;       // [4 warps][ring][slot] floats
        launch(lc, DELTA ? "delta_scan" : "ssm_scan", 0, kern, dim3(n, a.H, (a.Dv + kRecCols - 1) / kRecCols), dim3(128), smem, a);
    };
    if (rpt <= 2) go(ly_rec_scan_kernel<2, DELTA>, 2);
    else if (rpt <= 4) go(ly_rec_scan_kernel<4, DELTA>, 4);
    else if (rpt <= 8) go(ly_rec_scan_kernel<8, DELTA>, 8);
    else if (rpt <= 16) go(ly_rec_scan_kernel<16, DELTA>, 16);
    else if (rpt <= 32) go(ly_rec_scan_kernel<32, DELTA>, 32);
    else go(ly_rec_scan_kernel<64, DELTA>, 64);
}

// P = softmax of the score block's rows (see ly_attn_softmax_kernel)
static void launch_attn_softmax(LayeredCache& y, LaunchCtx& lc, const int* row_pos, int row0, int H, int rows, int k_lo, int n_first, int nk, int nkp, int window,
                                int keep_first, int chunk, float softcap, int sink, const float* sinkv) {
    if (n_first == 0 && (keep_first == 0 || window == 0) && nkp <= 2048) {
        auto go = [&](auto kern) {
            launch(lc, "attn_softmax", 0, kern, dim3((rows + 7) / 8), dim3(256), 0, (const float*)y.at_s.p, row_pos, row0, H, rows, k_lo, nk, nkp, window, chunk, softcap,
                   sink, sinkv, y.at_phi.p, y.at_plo.p);
        };
        if (nkp <= 512) go(ly_attn_softmax_warp_kernel<4>);
        else if (nkp <= 1024) go(ly_attn_softmax_warp_kernel<8>);
        else go(ly_attn_softmax_warp_kernel<16>);
        return;
    }
    const int keep = std::min(nkp, kSoftmaxKeep);
    launch(lc, "attn_softmax", 0, ly_attn_softmax_kernel, dim3(rows), dim3(256), (size_t)keep * 4, (const float*)y.at_s.p, row_pos, row0, H, k_lo, n_first, nk, nkp,
           window, keep_first, chunk, softcap, sink, sinkv, keep, y.at_phi.p, y.at_plo.p);
}

// Latent attention of rows [r0, r0 + Ts) -- one sequence's portion, positions pos0.. -- on the tensor-core GEMM, in blocks of query
// rows small enough that a block's score matrix stays within a fixed scratch budget.  A block only gathers the keys its rows'
// windows reach, so long prompts with short windows never touch fully masked regions.
// mma != nullptr: the step's query operand exists already and the result goes to hi | lo halves (the mixer runs on the tensor cores).
static void latent_attn_tc(fl_cache& c, LaunchCtx& lc, const LatentAttnArgs& a, const LatMmaArgs* mma, int r0, int Ts, int pos0, int slot) {
    LayeredCache& y = *c.ly;
    const int H = a.H, C = a.C, R = a.R, E = C + R, Ep = (E + 63) / 64 * 64;
    const size_t budget = (size_t)48 << 20;                // floats in a score block (192 MB); P halves take the same again
    auto keys_for = [&](int qb, int first) {               // padded key count of the block of qb rows starting at local row `first`
        const int p_lo = pos0 + first, p_hi = pos0 + std::min(Ts, first + qb);      // positions [p_lo, p_hi)
        const int k_lo = (a.window > 0 && p_lo - a.window + 1 > 0) ? p_lo - a.window + 1 : 0;
        return ((p_hi - k_lo) + 63) / 64 * 64;
    };
    int qb = 512;
    while (qb > 8 && (size_t)qb * H * keys_for(qb, std::max(0, Ts - qb)) > budget) qb /= 2;
    const size_t rows_max = (size_t)std::min(qb, Ts) * H;
    size_t nkp_max = 0;
    for (int f = 0; f < Ts; f += qb) nkp_max = std::max<size_t>(nkp_max, keys_for(qb, f));
    auto need = [&](auto& buf, size_t n) { if (buf.n < n) { FL_CUDA(cudaStreamSynchronize(c.stream)); buf.alloc(n + n / 4); } };
    need(y.at_kc, nkp_max * Ep); need(y.at_kct, (size_t)C * nkp_max);
    if (mma == nullptr) { need(y.at_qhi, rows_max * Ep); need(y.at_qlo, rows_max * Ep); }
    need(y.at_s, rows_max * nkp_max); need(y.at_phi, rows_max * nkp_max); need(y.at_plo, rows_max * nkp_max);
    const int* page_row = y.page_table.p + (size_t)slot * c.pages_per_seq;
    for (int f = 0; f < Ts; f += qb) {
        const int nq = std::min(qb, Ts - f), p_lo = pos0 + f, p_hi = p_lo + nq;
        const int k_lo = (a.window > 0 && p_lo - a.window + 1 > 0) ? p_lo - a.window + 1 : 0, nk = p_hi - k_lo, nkp = (nk + 63) / 64 * 64;
        const int rows = nq * H;
        if (rows <= 128) {          // a short tail: the per-(row, head) kernel
            if (mma != nullptr) {
                LatMmaArgs t = *mma;
                t.row_base = r0 + f;
                launch_latent_mma(lc, t, nq, p_hi);
            } else {
                LatentAttnArgs t = a;
                t.row_base = r0 + f;
                launch_latent_attn<uint16_t>(lc, t, nq);
            }
            continue;
        }
        // without a window every block's keys are a prefix of the last block's: they are gathered once (a later key meets a zero
        // probability)
        const int ldt = a.window > 0 ? nkp : (int)nkp_max;
        if (a.window > 0)
            launch(lc, "attn_gather_keys", 0, ly_attn_gather_keys_kernel, dim3(nkp / 64, Ep / 64), dim3(256), 0, (const uint16_t*)a.pool, page_row, k_lo, nk, nkp, C, E,
                   Ep, y.at_kc.p, y.at_kct.p);
        else if (f == 0)
            launch(lc, "attn_gather_keys", 0, ly_attn_gather_keys_kernel, dim3(ldt / 64, Ep / 64), dim3(256), 0, (const uint16_t*)a.pool, page_row, 0, pos0 + Ts, ldt, C,
                   E, Ep, y.at_kc.p, y.at_kct.p);
        const size_t q0 = (size_t)(r0 + f) * H;
        if (mma == nullptr)
            launch(lc, "attn_build_q", 0, ly_attn_build_q_kernel, dim3(nq, H), dim3(128), 0, a.qa, a.proj, a.ldp, a.off_q, r0 + f, H, a.D, R, C, Ep, a.scale,
                   y.at_qhi.p, y.at_qlo.p);
        const CUtensorMap tk = make_tmap_bf16(y.at_kc.p, (uint64_t)nkp, (uint64_t)Ep, (uint64_t)Ep, 128);
        dense_gemm(c, lc, "gemm_tc_attn_scores", rows, nkp, Ep, tk, y.at_s.p, mma ? mma->qhi + q0 * Ep : y.at_qhi.p, mma ? mma->qlo + q0 * Ep : y.at_qlo.p);
        launch_attn_softmax(y, lc, a.row_pos, r0 + f, H, rows, k_lo, 0, nk, nkp, a.window, 0, 0, 0.f, a.sink, a.sinkv);
        const CUtensorMap tv = make_tmap_bf16(y.at_kct.p, (uint64_t)C, (uint64_t)nkp, (uint64_t)ldt, 128);
        if (mma != nullptr)
            dense_gemm_blocks(c, lc, "gemm_tc_attn_values", rows, 1, C, nkp, tv, y.at_phi.p, y.at_plo.p, mma->ohi + q0 * C, mma->olo + q0 * C, C, 0);
        else
            dense_gemm(c, lc, "gemm_tc_attn_values", rows, C, nkp, tv, a.ol + q0 * C, y.at_phi.p, y.at_plo.p);
    }
}

// Grouped-query attention of rows [r0, r0 + Ts) -- one sequence's portion, positions pos0.. -- on the tensor-core GEMM: per block of
// query rows and per key/value head a score GEMM whose rows are (token, query head of the group) pairs, an f32 softmax (score cap,
// sink, causal mask) and a value GEMM; the block size keeps a score block within a fixed scratch budget.
static void gqa_attn_tc(fl_cache& c, LaunchCtx& lc, const GqaAttnArgs& a, int r0, int Ts, int pos0, int slot) {
    LayeredCache& y = *c.ly;
    const int H = a.H, G = a.G, rep = H / G, D = a.D, Dv = a.Dv, Dp = (D + 63) / 64 * 64;
    const size_t budget = (size_t)48 << 20;                // floats in a score block (192 MB); P halves take the same again
    // first key of the contiguous range a position reads (window and chunk starts only grow with the position, so a block of
    // rows needs the keys from its first row's start on), and the kept first keys that lie before it
    auto start_of = [&](int p) {
        const int lo_w = (a.window > 0 && p - a.window + 1 > 0) ? p - a.window + 1 : 0, lo_c = a.chunk > 0 ? p / a.chunk * a.chunk : 0;
        return std::max(lo_w, lo_c);
    };
    auto first_of = [&](int k_lo) { return a.window > 0 ? std::min(a.keep_first, k_lo) : 0; };
    auto keys_for = [&](int qb, int first) {
        const int p_lo = pos0 + first, p_hi = pos0 + std::min(Ts, first + qb);
        const int k_lo = start_of(p_lo);
        return ((p_hi - k_lo) + first_of(k_lo) + 63) / 64 * 64;
    };
    int qb = 1024;
    while (qb > 8 && (size_t)qb * rep * keys_for(qb, std::max(0, Ts - qb)) > budget) qb /= 2;
    const size_t rows_max = (size_t)std::min(qb, Ts) * rep;
    size_t nkp_max = 0;
    for (int f = 0; f < Ts; f += qb) nkp_max = std::max<size_t>(nkp_max, keys_for(qb, f));
    auto need = [&](auto& buf, size_t n) { if (buf.n < n) { FL_CUDA(cudaStreamSynchronize(c.stream)); buf.alloc(n + n / 4); } };
    need(y.at_kc, nkp_max * Dp); need(y.at_kct, (size_t)Dv * nkp_max);
    need(y.at_qhi, rows_max * Dp); need(y.at_qlo, rows_max * Dp);
    need(y.at_s, rows_max * nkp_max); need(y.at_phi, rows_max * nkp_max); need(y.at_plo, rows_max * nkp_max);
    need(y.at_o, rows_max * G * Dv);
    const int* page_row = y.page_table.p + (size_t)slot * c.pages_per_seq;
    for (int f = 0; f < Ts; f += qb) {
        const int nq = std::min(qb, Ts - f), p_lo = pos0 + f, p_hi = p_lo + nq;
        const int k_lo = start_of(p_lo), n_first = first_of(k_lo), nk = p_hi - k_lo, nkp = (n_first + nk + 63) / 64 * 64;
        const int rows = nq * rep;
        if (rows <= 128) {          // a short tail: the per-(row, head) kernel
            GqaAttnArgs t = a;
            t.row_base = r0 + f;
            launch_gqa_attn<uint16_t>(lc, t, nq, p_hi, true);
            continue;
        }
        for (int g = 0; g < G; ++g) {
            launch(lc, "gqa_gather_kv", 0, ly_gqa_gather_kv_kernel, dim3(nkp), dim3(128), 0, (const uint16_t*)a.pool, page_row, k_lo, n_first, nk, nkp, a.kv.E,
                   g * a.kv.ks, D, Dp, a.kv.vo + g * a.kv.vs, Dv, a.kv.roll, y.at_kc.p, y.at_kct.p);
            launch(lc, "gqa_build_q", 0, ly_gqa_build_q_kernel, dim3(nq, rep), dim3(128), 0, a.proj, a.ldp, a.off_q, r0 + f, rep, g, D, Dp, a.scale, y.at_qhi.p,
                   y.at_qlo.p);
            const CUtensorMap tk = make_tmap_bf16(y.at_kc.p, (uint64_t)nkp, (uint64_t)Dp, (uint64_t)Dp, 128);
            dense_gemm(c, lc, "gemm_tc_attn_scores", rows, nkp, Dp, tk, y.at_s.p, y.at_qhi.p, y.at_qlo.p);
            launch_attn_softmax(y, lc, a.row_pos, r0 + f, rep, rows, k_lo, n_first, nk, nkp, a.window, a.keep_first, a.chunk, a.softcap, a.sink,
                                a.sinkv ? a.sinkv + g * rep : (const float*)nullptr);
            const CUtensorMap tv = make_tmap_bf16(y.at_kct.p, (uint64_t)Dv, (uint64_t)nkp, (uint64_t)nkp, 128);
            dense_gemm(c, lc, "gemm_tc_attn_values", rows, Dv, nkp, tv, y.at_o.p + (size_t)g * rows * Dv, y.at_phi.p, y.at_plo.p);
        }
        const size_t no = (size_t)nq * H * Dv;
        launch(lc, "gqa_scatter", 0, ly_gqa_scatter_kernel, dim3((unsigned)std::min<size_t>(4 * kNumSMs, (no + 255) / 256)), dim3(256), 0, (const float*)y.at_o.p, nq,
               G, rep, Dv, r0 + f, a.ldo, a.gate, a.out, a.ohi, a.olo);
    }
}

static void enqueue_step(fl_cache& c, LaunchCtx& lc, const StepTab& st, const int* slots, const int* counts, int n, const int* h_row0,
                         const int* h_pos0);

void layered_forward(fl_cache& c, const int* slots, const int* counts, int n, const uint32_t* ids, const int* want, int n_want) {
    const LayeredModel& m = *c.lm;
    LayeredCache& y = *c.ly;
    FL_CHECK(!c.poisoned, FL_ERR_CUDA, "cache poisoned by an earlier CUDA error");
    FL_CHECK(slots && counts && ids && (want || n_want == 0), FL_ERR_INVALID, "NULL argument");
    FL_CHECK(n >= 1 && n <= c.max_batch && n_want >= 0, FL_ERR_INVALID, "bad batch");
    // ---- host: validate, take pages, lay out the step tables ----
    long long T = 0;
    std::vector<char> seen(c.max_batch, 0);
    int need_pages = 0;
    for (int i = 0; i < n; ++i) {
        const int sl = slots[i];
        FL_CHECK(sl >= 0 && sl < c.max_batch, FL_ERR_INVALID, "slot index out of range");
        FL_CHECK(!seen[sl], FL_ERR_INVALID, "a slot appears twice in one call");
        seen[sl] = 1;
        FL_CHECK(counts[i] >= 1, FL_ERR_INVALID, "every sequence of a step brings at least one token");
        FL_CHECK(c.slot_len[sl] + counts[i] <= c.max_seq, FL_ERR_STATE, "sequence longer than the cache's max_seq");
        FL_CHECK(m.cfg.max_positions <= 0 || c.slot_len[sl] + counts[i] <= m.cfg.max_positions, FL_ERR_STATE, "sequence longer than the model's position table");
        need_pages += y.pool.missing(sl, c.slot_len[sl] + counts[i]);
        T += counts[i];
    }
    FL_CHECK(need_pages <= y.pool.pages_free(), FL_ERR_STATE, "cache page pool exhausted");
    for (long long i = 0; i < T; ++i) FL_CHECK(ids[i] < (uint32_t)m.V, FL_ERR_INVALID, "token id out of range");
    for (int k = 0; k < n_want; ++k) FL_CHECK(want[k] >= 0 && want[k] < T, FL_ERR_INVALID, "wanted row out of range");
    ensure_ws(c, (size_t)T, (size_t)n_want);
    const size_t tab_ints = (size_t)4 * T + 3 * (size_t)n + 1 + (size_t)n_want;
    if (tab_ints > y.tab_cap) {
        FL_CUDA(cudaStreamSynchronize(c.stream));
        drop_graphs(c);
        y.tab_cap = std::max(tab_ints, 2 * y.tab_cap);
        y.step_tab.alloc(y.tab_cap); y.h_step_tab.alloc(y.tab_cap);
    }
    FL_CUDA(cudaStreamSynchronize(c.stream));      // the pinned staging buffers of the previous step are free again
    int* ht = y.h_step_tab.p;
    int *h_tok = ht, *h_rseq = ht + T, *h_rpos = ht + 2 * T, *h_row0 = ht + 3 * T, *h_slot = h_row0 + n + 1, *h_pos0 = h_slot + n,
        *h_want = h_pos0 + n, *h_prev = h_want + n_want;
    int row = 0;
    for (int i = 0; i < n; ++i) {
        const int sl = slots[i];
        h_row0[i] = row; h_slot[i] = sl; h_pos0[i] = c.slot_len[sl];
        int before_tok = y.slot_last[sl];           // -1 for a slot that holds nothing
        for (int k = 0; k < counts[i]; ++k, ++row) {
            h_prev[row] = before_tok;
            before_tok = (int)ids[row]; h_tok[row] = (int)ids[row]; h_rseq[row] = i; h_rpos[row] = c.slot_len[sl] + k; }
        const int before = y.pool.held(sl);
        y.pool.grow(sl, c.slot_len[sl] + counts[i]);
        if (y.pool.held(sl) != before)
            FL_CUDA(cudaMemcpyAsync(y.page_table.p + (size_t)sl * c.pages_per_seq + before, y.pool.row(sl) + before,
                                    (size_t)(y.pool.held(sl) - before) * 4, cudaMemcpyHostToDevice, c.stream));
    }
    h_row0[n] = row;
    for (int k = 0; k < n_want; ++k) h_want[k] = want[k];
    FL_CUDA(cudaMemcpyAsync(y.step_tab.p, ht, tab_ints * 4, cudaMemcpyHostToDevice, c.stream));
    const int* dt = y.step_tab.p;
    StepTab st{dt, dt + T, dt + 2 * T, dt + 3 * T, dt + 3 * T + n + 1, dt + 3 * T + 2 * n + 1, dt + 3 * T + 3 * n + 1, dt + 3 * T + 3 * n + 1 + n_want, (int)T, n, n_want};

    // ---- device: layer by layer over all rows of the step ----
    LaunchCtx lc;
    lc.stream = c.stream;
    lc.pdl = false;
    lc.exact = m.f32;
    // A step in which every sequence brings ONE token has a launch geometry that depends on (sequences, wanted rows) alone --
    // positions, slots and pages are read from the device tables -- so it is captured into a CUDA graph the second time the pair is
    // seen and replayed from then on (FL_NO_GRAPH=1 keeps eager launches).
    static const bool no_graph = env_flag("FL_NO_GRAPH");
    if (T == n && !g_prof.on && !no_graph) {
        const GraphKey key{n, 1000 + n_want};
        auto it = c.graphs.find(key);
        if (it == c.graphs.end()) {
            c.graphs[key] = GraphEntry{};               // first sight: run eagerly (one-time kernel attributes, lazy loading)
            enqueue_step(c, lc, st, slots, counts, n, h_row0, h_pos0);
        } else {
            if (it->second.exec == nullptr) {
                lc.capturing = true;
                cudaGraph_t graph = nullptr;
                FL_CUDA(cudaStreamBeginCapture(c.stream, cudaStreamCaptureModeThreadLocal));
                try {
                    enqueue_step(c, lc, st, slots, counts, n, h_row0, h_pos0);
                } catch (...) {
                    cudaStreamEndCapture(c.stream, &graph);
                    if (graph) cudaGraphDestroy(graph);
                    throw;
                }
                FL_CUDA(cudaStreamEndCapture(c.stream, &graph));
                GraphEntry e;
                FL_CUDA(cudaGraphInstantiate(&e.exec, graph, 0));
                FL_CUDA(cudaGraphDestroy(graph));
                e.kernels = lc.captured;
                it->second = e;
            }
            FL_CUDA(cudaGraphLaunch(it->second.exec, c.stream));
            g_launches.fetch_add(it->second.kernels, std::memory_order_relaxed);
        }
    } else {
        enqueue_step(c, lc, st, slots, counts, n, h_row0, h_pos0);
    }
    if (n_want > 0)
        FL_CUDA(cudaMemcpyAsync(y.h_logits.p, y.logits.p, (size_t)n_want * m.V * 4, cudaMemcpyDeviceToHost, c.stream));
    for (int i = 0, r = 0; i < n; ++i) {
        c.slot_len[slots[i]] += counts[i];
        r += counts[i];
        y.slot_last[slots[i]] = (int)ids[r - 1];
    }
}

// One mixer over all rows of the step (`pass`: which pass of a loop, 0 elsewhere -- its own cache and state): reads its columns of the projected buffer y.proj (row stride lw.n_in; `in`: the same as
// the GEMM left it, perhaps in slices), its cache pages / state
// slots, and leaves the mixer's inner output (what its output projection reads) in y.u with the hi | lo halves when that
// projection runs on the tensor cores.
static void run_mixer(fl_cache& c, LaunchCtx& lc, const StepTab& st, const LayeredLayerW& lw, const Slices& in, int pass, const int* slots, const int* counts, int n,
                      const int* h_row0, const int* h_pos0) {
    const LayeredModel& m = *c.lm;
    LayeredCache& y = *c.ly;
    const fl_layer_desc& d = lw.d;
    const int Ti = st.T, H = d.heads, D = d.dim, Dv = d.vdim;
    const float eps = m.cfg.norm_eps;
    const int kv_index = lw.kv_index + pass, gla_index = lw.gla_index + pass;
    uint16_t *uhi = m.f32 ? nullptr : y.u_hi.p, *ulo = m.f32 ? nullptr : y.u_lo.p;
    const int ldu = lw.u_ld;
    const OutGate gate = d.out_gate ? OutGate{y.proj.p + lw.off_g, lw.n_in, d.out_gate == 2 ? 1 : Dv, d.out_gate == 2 ? 0 : 1} : OutGate{};
    const int n_gate = d.out_gate == 0 ? 0 : (d.out_gate == 2 ? H : H * Dv);
    if (d.mixer == FL_MIXER_ATTN) {
        const int G = d.kv_heads;
        const KvLayout kv = kv_layout(d);
        AttnPrepArgs pa{y.proj.p, lw.n_in, lw.off_q, lw.off_k, lw.off_v, lw.qnorm, lw.knorm, eps, y.kv_pool[kv_index], y.page_table.p,
                        c.pages_per_seq, st.row_seq, st.row_pos, st.seq_slot, y.rope_cos[lw.rope_index].p, y.rope_sin[lw.rope_index].p,
                        H, G, D, Dv, d.rot_dims, d.rot_halves, lw.bq, lw.bk, lw.bv, d.qk_norm_whole, kv, in, lw.off_g, n_gate};
        // eight warps per block take the heads in turn; steps of few rows spread a row's heads and gate columns over up to eight blocks (not with a
        // norm over the whole projection: its sums read every head before any is rewritten in place, which one block orders)
        const size_t psm = (size_t)8 * D * 4;
        const int heads_all = H + (lw.off_k >= 0 ? G : 0), py = (Ti <= 64 && !d.qk_norm_whole) ? std::max(1, std::min(8, std::max((heads_all + 7) / 8, n_gate / 512))) : 1;
        if (m.f32) launch(lc, "attn_prep", 0, ly_attn_prep_kernel<float>, dim3(Ti, py), dim3(256), psm, pa);
        else launch(lc, "attn_prep", 0, ly_attn_prep_kernel<uint16_t>, dim3(Ti, py), dim3(256), psm, pa);
        GqaAttnArgs at{y.proj.p, lw.n_in, lw.off_q, y.kv_pool[kv_index], y.page_table.p, c.pages_per_seq, st.row_seq, st.row_pos, st.seq_slot,
                       y.u.p, lw.tc_o ? uhi : (uint16_t*)nullptr, ulo, H, G, D, Dv, d.window, d.scale, d.softcap, d.sink, 0, y.at_part.p,
                       d.keep_first, d.mask_chunk, lw.sinkv, kv, ldu, gate};
        // a step of single tokens is replayed from a captured graph whatever the contexts' lengths: its split count must not follow them
        int max_keys = c.max_seq;
        if (Ti != n) {
            max_keys = 1;
            for (int si = 0; si < n; ++si) max_keys = std::max(max_keys, h_pos0[si] + counts[si]);
        }
        if (d.window > 0) max_keys = std::min(max_keys, d.window + d.keep_first);
        if (d.mask_chunk > 0) max_keys = std::min(max_keys, d.mask_chunk);
        // masks that leave a row few keys: the per-row kernel reads just those, the GEMM path would compute a block's whole rectangle
        const bool few_keys = (d.window > 0 && d.window + d.keep_first <= 256) || (d.mask_chunk > 0 && d.mask_chunk <= 256);
        // long portions (serving precision): scores and weighted sums as tensor-core GEMMs; decoded tokens, short portions and
        // the exact mode on the per-(row, head) kernel.  Rows are taken in order.
        static const bool tc_attn_off = env_flag("FL_LAYERED_NO_TC_ATTN");
        int done = 0;
        for (int si = 0; si < n; ++si) {
            const int r0 = h_row0[si], Ts = counts[si];
            if (m.f32 || tc_attn_off || few_keys || Dv % 8 != 0 || Ts < 64 || (long long)Ts * (H / G) <= 128) continue;
            if (r0 > done) {
                at.row_base = done;
                launch_gqa_attn<uint16_t>(lc, at, r0 - done, max_keys, true);
            }
            gqa_attn_tc(c, lc, at, r0, Ts, h_pos0[si], slots[si]);
            done = r0 + Ts;
        }
        if (done < Ti) {
            at.row_base = done;
            if (m.f32) launch_gqa_attn<float>(lc, at, Ti - done, max_keys, false); else launch_gqa_attn<uint16_t>(lc, at, Ti - done, max_keys, true);
        }
    } else if (d.mixer == FL_MIXER_MAMBA2 || d.mixer == FL_MIXER_DELTA) {
        const bool delta = d.mixer == FL_MIXER_DELTA;
        const int G = delta ? d.kv_heads : d.groups, rows = delta ? D : d.state;
        float* cstate = d.conv > 1 ? y.conv_state[gla_index].p : nullptr;
        ConvArgs ca{y.proj.p, lw.n_in, lw.conv_off, lw.conv_w, lw.conv_b, cstate, st.row_seq, st.row_pos, st.seq_row0, st.seq_slot, st.seq_pos0,
                    lw.conv_ch, d.conv, y.cv.p};
        // channel chunks per row: whole q / k heads for the delta rule (they are normalised inside one block)
        const int chunk = delta ? D * std::max(1, 512 / D) : 512, nchunk = (lw.conv_ch + chunk - 1) / chunk;
        if (delta)
            launch(lc, "delta_prep", 0, ly_delta_prep_kernel, dim3(Ti, nchunk), dim3(256), 0, ca, chunk, lw.off_b, lw.off_a, (const float*)lw.dt_bias,
                   (const float*)lw.a_log, H, G, D, (float)(1.0 / std::sqrt((double)D)), y.rs.p);
        else
            launch(lc, "ssm_prep", 0, ly_mamba_prep_kernel, dim3(Ti, nchunk), dim3(256), 0, ca, chunk, lw.off_dt, (const float*)lw.dt_bias,
                   (const float*)lw.a_log, H, y.rs.p);
        if (d.conv > 1) launch(lc, "conv_state", 0, ly_conv_state_kernel, dim3(n, (lw.conv_ch + 127) / 128), dim3(128), 0, ca);
        // column offsets inside cv (the convolved span starts at conv_off)
        RecArgs ra{y.cv.p, lw.conv_ch, lw.off_q - lw.conv_off, lw.off_k - lw.conv_off, lw.off_v - lw.conv_off, y.rs.p,
                   delta ? (const float*)nullptr : (const float*)lw.dskip, y.go.p, y.gla_state[gla_index].p, st.seq_row0, st.seq_slot, st.seq_pos0,
                   H, G, rows, Dv};
        if (delta) {
            launch_rec_scan<true>(lc, ra, n);
            launch(lc, "gla_out", 0, ly_gla_out_kernel, dim3((Ti * H + 7) / 8), dim3(256), 0, (const float*)y.go.p, (const float*)y.proj.p, lw.n_in, lw.off_g,
                   (const float*)lw.hnorm, eps, Ti, H, Dv, ldu, y.u.p, lw.tc_o ? uhi : (uint16_t*)nullptr, ulo);
        } else {
            launch_rec_scan<false>(lc, ra, n);
            const int inner = H * Dv, part = inner / d.norm_groups;
            launch(lc, "gated_group_norm", 0, ly_gated_group_norm_kernel, dim3(Ti, d.norm_groups), dim3(std::min(1024, std::max(64, (part + 31) / 32 * 32))), 0,
                   (const float*)y.go.p, (const float*)y.proj.p, lw.n_in, lw.off_g, (const float*)lw.hnorm, eps, inner, d.norm_groups, 0, ldu, y.u.p,
                   lw.tc_o ? uhi : (uint16_t*)nullptr, ulo);
        }
    } else if (d.mixer == FL_MIXER_LIGHTNING) {
        const int chunk = 512, nchunk = (lw.conv_ch + chunk - 1) / chunk, inner = H * Dv;
        launch(lc, "lightning_prep", 0, ly_lightning_prep_kernel, dim3(Ti, nchunk), dim3(256), 0, (const float*)y.proj.p, lw.n_in, lw.conv_off, lw.conv_ch, chunk,
               (const float*)lw.decay, H, y.cv.p, y.rs.p);
        RecArgs ra{y.cv.p, lw.conv_ch, lw.off_q - lw.conv_off, lw.off_k - lw.conv_off, lw.off_v - lw.conv_off, y.rs.p, (const float*)nullptr, y.go.p,
                   y.gla_state[gla_index].p, st.seq_row0, st.seq_slot, st.seq_pos0, H, H, D, Dv};
        launch_rec_scan<false>(lc, ra, n);
        const bool v4 = ((inner | lw.n_in | lw.off_g | ldu) & 3) == 0;       // four channels per thread
        launch(lc, "gated_group_norm", 0, ly_gated_group_norm_kernel, dim3(Ti, 1), dim3(std::min(v4 ? 256 : 1024, std::max(64, ((v4 ? inner / 4 : inner) + 31) / 32 * 32))), 0,
               (const float*)y.go.p, (const float*)y.proj.p, lw.n_in, lw.off_g, (const float*)lw.hnorm, eps, inner, 1, 1, ldu, y.u.p,
               lw.tc_o ? uhi : (uint16_t*)nullptr, ulo);
    } else if (d.mixer == FL_MIXER_GLA) {
        // decay pre-activation through the rank-r bottleneck: z = W_a2 a (the bias and the sigmoid^(1/tau) are applied by the scan)
        gemm(lc, "gemm_gla_decay", y.proj.p + lw.off_a, lw.n_in, lw.a2, H * D, d.decay_rank, y.la.p, H * D, Ti);
        GlaArgs ga{y.proj.p, lw.n_in, lw.off_q, lw.off_k, lw.off_v, y.la.p, lw.a2b, 1.f / d.tau, y.go.p, y.gla_state[gla_index].p, st.seq_row0,
                   st.seq_slot, st.seq_pos0, H, D, Dv, (float)(1.0 / std::sqrt((double)D))};
        launch_gla_scan(lc, ga, n);
        launch(lc, "gla_out", 0, ly_gla_out_kernel, dim3((Ti * H + 7) / 8), dim3(256), 0, (const float*)ga.o, (const float*)y.proj.p, lw.n_in, lw.off_g,
               (const float*)lw.hnorm, eps, Ti, H, Dv, ldu, y.u.p, lw.tc_o ? uhi : (uint16_t*)nullptr, ulo);
    } else {
        const int R = d.rot_dim, C = d.kv_rank, Q = d.q_rank;
        LatentAppendArgs aa{y.proj.p, lw.n_in, lw.off_q, lw.off_dkv, lw.dkv_norm, eps, y.kv_pool[kv_index], y.page_table.p, c.pages_per_seq,
                            st.row_seq, st.row_pos, st.seq_slot, y.rope_cos[lw.rope_index].p, y.rope_sin[lw.rope_index].p, H, D, R, C, d.rot_dims, lw.off_q, Q, lw.dq_norm, lw.tc_uq ? (float*)nullptr : y.cq.p,
                            lw.tc_uq ? y.cq_hi.p : (uint16_t*)nullptr, y.cq_lo.p, in, lw.off_g, n_gate};
        const int ath = Ti <= 2 * kNumSMs ? std::min(1024, std::max(128, (Q + C + 31) / 32 * 32)) : 128;
        if (m.f32) launch(lc, "latent_append", 0, ly_latent_append_kernel<float>, dim3(Ti), dim3(ath), 0, aa);
        else launch(lc, "latent_append", 0, ly_latent_append_kernel<uint16_t>, dim3(Ti), dim3(ath), 0, aa);
        // queries [T][H][D + R]: columns of the projected buffer, or expanded from the normed query latent
        float* q = y.proj.p + lw.off_q;
        int ldq = lw.n_in;
        Slices qs{q, 1, 0};
        if (Q > 0) {
            q = y.qx.p; ldq = H * (D + R);
            qs = gemm_slices(c, lc, "gemm_q_up", y.cq.p, y.cq_hi.p, y.cq_lo.p, lw.uq, lw.tm_uq, lw.tc_uq, ldq, Q, q, Ti);
            if (qs.n > 1 && !lw.lat_tc) {
                launch(lc, "sum_slices", 0, ly_sum_slices_kernel, dim3((unsigned)std::min<size_t>(4 * kNumSMs, (qs.stride + 255) / 256)), dim3(256), 0, qs.p, qs.n,
                       qs.stride, qs.stride, q);
            }
            if (d.rot_dims > 0 && !lw.lat_tc)
                launch(lc, "rotate_q", 0, ly_rotate_q_kernel, dim3(Ti), dim3(128), 0, q, ldq, st.row_pos, (const float*)y.rope_cos[lw.rope_index].p,
                       (const float*)y.rope_sin[lw.rope_index].p, H, D, R, d.rot_dims);
        }
        static const bool tc_attn_off = env_flag("FL_LAYERED_NO_TC_ATTN");
        // Rows are taken in order: long portions (serving precision) run scores and weighted sums as tensor-core GEMMs over the
        // gathered window, everything else goes to `rest`(first row, rows).
        auto walk = [&](const LatentAttnArgs& at, const LatMmaArgs* mma, bool gemms, auto&& rest) {
            int done = 0;           // rows [0, done) are finished
            for (int si = 0; si < n; ++si) {
                const int r0 = h_row0[si], Ts = counts[si];
                if (!gemms || Ts < 64 || (long long)Ts * H <= 128) continue;
                if (r0 > done) rest(done, r0 - done);
                latent_attn_tc(c, lc, at, mma, r0, Ts, h_pos0[si], slots[si]);
                done = r0 + Ts;
            }
            if (done < Ti) rest(done, Ti - done);
        };
        if (lw.lat_tc) {
            // the whole mixer over hi | lo halves: split queries -> W_uk absorbed (one block per head) -> attention -> W_uv (and the
            // gate) -> the output projection's operand
            const int Ep = (C + R + 63) / 64 * 64;
            const bool turn = Q > 0 && d.rot_dims > 0;
            launch(lc, "latent_split_q", 0, ly_latent_split_q_kernel, dim3(Ti, Ti <= kNumSMs ? 4 : 1), dim3(256), 0, qs, ldq, st.row_pos,
                   turn ? (const float*)y.rope_cos[lw.rope_index].p : (const float*)nullptr, (const float*)y.rope_sin[lw.rope_index].p, H, D, R, d.rot_dims, C, Ep,
                   d.scale, y.qp_hi.p, y.qp_lo.p, y.qo_hi.p, y.qo_lo.p);
            dense_gemm_blocks(c, lc, "gemm_q_absorb", Ti, H, C, D, lw.tm_uk, y.qp_hi.p, y.qp_lo.p, y.qo_hi.p, y.qo_lo.p, H * Ep, Ep);
            LatentAttnArgs at{nullptr, q, ldq, 0, y.kv_pool[kv_index], y.page_table.p, c.pages_per_seq, st.row_seq, st.row_pos,
                              st.seq_slot, nullptr, H, D, R, C, d.window, d.scale, 0, d.sink, lw.sinkv};
            LatMmaArgs ma{y.qo_hi.p, y.qo_lo.p, (const uint16_t*)y.kv_pool[kv_index], y.page_table.p, c.pages_per_seq, st.row_seq, st.row_pos, st.seq_slot,
                          y.ol_hi.p, y.ol_lo.p, y.at_part.p, H, C, R, Ep, d.window, 0, d.sink, lw.sinkv};
            // a step of single tokens is replayed from a captured graph whatever the contexts' lengths: its split count must not follow them
            int max_keys = c.max_seq;
            if (Ti != n) {
                max_keys = 1;
                for (int si = 0; si < n; ++si) max_keys = std::max(max_keys, h_pos0[si] + counts[si]);
            }
            if (d.window > 0) max_keys = std::min(max_keys, d.window + kLatTile);
            walk(at, &ma, !tc_attn_off, [&](int first, int rows) {
                LatMmaArgs t = ma;
                t.row_base = first;
                launch_latent_mma(lc, t, rows, max_keys);
            });
            dense_gemm_blocks(c, lc, "gemm_v_expand", Ti, H, Dv, C, lw.tm_uv, y.ol_hi.p, y.ol_lo.p, uhi, ulo, ldu, Dv, gate.g,
                              gate.ld, d.out_gate == 2);
            return;
        }
        // q~[row, h, :] = W_uk[h]^T q_plain[row, h, :]: the score against the latent needs no per-head keys
        LyGemm qa{q, D + R, ldq, nullptr, lw.uk_t, (long long)C * D, C, D, y.qa.p, C, H * C, nullptr, Ti};
        gemm_groups(lc, "gemm_q_absorb", qa, H, Ti);
        LatentAttnArgs at{y.qa.p, q, ldq, 0, y.kv_pool[kv_index], y.page_table.p, c.pages_per_seq, st.row_seq, st.row_pos,
                          st.seq_slot, y.ol.p, H, D, R, C, d.window, d.scale, 0, d.sink, lw.sinkv};
        walk(at, nullptr, !m.f32 && !tc_attn_off && C % 8 == 0, [&](int first, int rows) {      // the exact mode: everything on the per-(row, head) kernel
            LatentAttnArgs t = at;
            t.row_base = first;
            if (m.f32) launch_latent_attn<float>(lc, t, rows); else launch_latent_attn<uint16_t>(lc, t, rows);
        });
        // value expansion after the softmax: out[row, h, :] = W_uv[h] (sum_j p_j c_j)
        LyGemm ov{y.ol.p, C, H * C, nullptr, lw.uv, (long long)Dv * C, Dv, C, y.u.p, Dv, ldu, nullptr, Ti};
        gemm_groups(lc, "gemm_v_expand", ov, H, Ti);
        if (d.out_gate || lw.tc_o)
            launch(lc, d.out_gate ? "out_gate" : "split_hi_lo", 0, ly_out_gate_kernel, dim3((unsigned)std::min<size_t>(4 * kNumSMs, ((size_t)Ti * H * Dv + 255) / 256)),
                   dim3(256), 0, y.u.p, ldu, gate, H, Dv, Ti, lw.tc_o ? uhi : (uint16_t*)nullptr, ulo);
    }
}

// The device part of a step: every layer over all rows, then the vocabulary projection of the wanted rows.
static void enqueue_step(fl_cache& c, LaunchCtx& lc, const StepTab& st, const int* slots, const int* counts, int n, const int* h_row0,
                         const int* h_pos0) {
    const LayeredModel& m = *c.lm;
    LayeredCache& y = *c.ly;
    const int n_want = st.n_want;
    const int Ti = st.T, W = m.W;
    const float eps = m.cfg.norm_eps;
    const int nthr = std::min(1024, std::max(64, (W + 31) / 32 * 32));
    uint16_t *hhi = m.f32 ? nullptr : y.h_hi.p, *hlo = m.f32 ? nullptr : y.h_lo.p, *uhi = m.f32 ? nullptr : y.u_hi.p, *ulo = m.f32 ? nullptr : y.u_lo.p,
             *ahi = m.f32 ? nullptr : y.act_hi.p, *alo = m.f32 ? nullptr : y.act_lo.p;
    // pre-norm stacks: a sublayer reads h = norm(x) (written by the kernel that last touched x); otherwise it reads x itself and
    // the same kernel writes x's hi | lo halves for the tensor-core GEMMs.  With an input convolution the sublayer reads
    // hc = h + conv(h) instead (the convolution kernel rewrites the hi | lo halves after the gate's GEMM has read those of h).
    const bool pre = !m.cfg.no_pre_norm, post = !m.cfg.no_post_norm, canon = m.cfg.canon_taps > 0, gated = m.cfg.gated_residual != 0,
               depth = m.cfg.depth_avg != 0;
    const int plain = m.cfg.norm_plain ? 1 : 0, split_x = pre ? 0 : 1;
    const bool par = m.cfg.parallel_sub != 0, tside = m.cfg.token_side > 0;
    auto norm_of = [&](const float* w, const float* b, const float* alpha) { return NormW{w, b, alpha, plain}; };
    auto norm1_of = [&](int r) { const LayeredLayerW& l = m.layers[m.runs[r].layer]; return norm_of(l.norm1, l.norm1_bias, l.norm1_alpha); };
    // whether a run's mixer input is read as hi | lo halves only (routed experts' routers and the FMA kernels read f32 rows)
    auto halves_only = [&](int r) {
        const LayeredLayerW& l = m.layers[m.runs[r].layer];
        return l.tc_in && !canon && !gated && !(par && l.d.ffn == FL_FFN_MOE);
    };
    const float* norm_out = pre ? y.h.p : y.x.p;                // what the arrangement hands to a sublayer
    const float* sub_in = canon ? y.hc.p : norm_out;            // what the sublayer's own matrices read
    const size_t hist_stride = y.rows * (size_t)W;
    launch(lc, "embed_norm", 0, ly_embed_norm_kernel, dim3(Ti), dim3(nthr), 0, (const uint16_t*)m.embed, st.tok, W,
           pre ? norm1_of(0) : NormW{}, eps, plain, (const uint16_t*)m.pos, st.row_pos, m.cfg.embed_scale, (const float*)m.embed_norm,
           BigramTab{m.bigram, st.prev, m.cfg.bigram_buckets, (long long)m.cfg.bigram_mul_prev, (long long)m.cfg.bigram_mul_cur},
           m.runs[0].pass_start ? (const float*)m.loop_step : (const float*)nullptr, y.x.p, depth || m.cfg.loop_reinject ? y.xs.p : (float*)nullptr, y.h.p, hhi, hlo);
    // in front of a sublayer: the gate's pre-activation from the normed input, then the input convolution (and its carried inputs)
    auto sublayer_front = [&](const LayeredLayerW& lw, int run, int sub) {
        if (gated) {
            const uint16_t* rg = sub == 0 ? lw.rg1 : lw.rg2;
            gemm_tc_or_exact(c, lc, "gemm_gate", norm_out, hhi, hlo, rg, sub == 0 ? lw.tm_rg1 : lw.tm_rg2, sub == 0 ? lw.tc_rg1 : lw.tc_rg2, W, W, y.gz.p, Ti);
        }
        if (canon) {
            const int taps = m.cfg.canon_taps;
            float* cs = taps > 1 ? y.canon_state[run].p + (size_t)sub * c.max_batch * (taps - 1) * W : nullptr;
            ConvArgs ca{norm_out, W, 0, sub == 0 ? lw.canon1 : lw.canon2, nullptr, cs, st.row_seq, st.row_pos, st.seq_row0, st.seq_slot, st.seq_pos0, W, taps, nullptr};
            // few rows: one row per block; long steps: a block walks 8 rows with its taps staged once
            const int rpb = Ti >= 1024 ? 8 : 1;
            if (W % 4 == 0)
                launch(lc, "input_conv", 0, ly_input_conv_kernel<4>, dim3((Ti + rpb - 1) / rpb, (W / 4 + 127) / 128), dim3(128), (size_t)taps * 128 * 4 * 4, ca, rpb, Ti,
                       y.hc.p, hhi, hlo);
            else
                launch(lc, "input_conv", 0, ly_input_conv_kernel<1>, dim3((Ti + rpb - 1) / rpb, (W + 127) / 128), dim3(128), (size_t)taps * 128 * 4, ca, rpb, Ti,
                       y.hc.p, hhi, hlo);
            if (taps > 1) launch(lc, "conv_state", 0, ly_conv_state_kernel, dim3(n, (W + 127) / 128), dim3(128), 0, ca);
        }
    };
    // stacks with a token shift: the mixer reads hc = x + (x_prev - x) * shift (x_prev from the row before, or the slot's carried
    // row); the slot then keeps this step's last row of x.  The shift kernel rewrites the hi | lo halves with those of hc.
    const bool shifted = m.cfg.token_shift != 0, sum_norm = m.cfg.post_sum_norm != 0;
    auto shift_front = [&](const LayeredLayerW& lw, int run) {
        ConvArgs ca{y.x.p, W, 0, nullptr, nullptr, y.shift_state[run].p, st.row_seq, st.row_pos, st.seq_row0, st.seq_slot, st.seq_pos0, W, 2, nullptr};
        if (W % 4 == 0)
            launch(lc, "token_shift", 0, ly_token_shift_kernel<4>, dim3(Ti, (W / 4 + 127) / 128), dim3(128), 0, ca, (const float*)lw.shift, y.hc.p, hhi, hlo);
        else
            launch(lc, "token_shift", 0, ly_token_shift_kernel<1>, dim3(Ti, (W + 127) / 128), dim3(128), 0, ca, (const float*)lw.shift, y.hc.p, hhi, hlo);
        launch(lc, "conv_state", 0, ly_conv_state_kernel, dim3(n, (W + 127) / 128), dim3(128), 0, ca);
    };
    // the norm of the sum: x <- norm(alpha x + sa y (+ sb y2)); split: whether another sublayer reads the new x through the tensor cores
    auto sum_norm_join = [&](const float* yb, const float* y2, float sa, float sb, const float* w, int split) {
        if (W % 4 == 0)
            launch(lc, "sum_norm", 0, ly_sum_norm_kernel<4>, dim3(Ti), dim3(std::min(256, std::max(32, (W / 4 + 31) / 32 * 32))), (size_t)W * 4, y.x.p,
                   (const float*)y.y.p, yb, y2, m.cfg.residual_alpha, sa, sb, w, eps, W, plain, split, hhi, hlo);
        else
            launch(lc, "sum_norm", 0, ly_sum_norm_kernel<1>, dim3(Ti), dim3(nthr), (size_t)W * 4, y.x.p, (const float*)y.y.p, yb, y2, m.cfg.residual_alpha, sa, sb,
                   w, eps, W, plain, split, hhi, hlo);
    };
    // a sublayer's result (and y2 beside it) joins the stream; four channels per thread when the rows are 16-byte multiples
    // (hout == nullptr: what comes next reads the hi | lo halves alone; split: without a next norm, the halves of the stream itself)
    auto join = [&](const Slices& yv, const float* y2, const float* wa, const float* wb, const float* gate_bias, int hist_slot, const float* dw, const float* x0,
                    const float* step, NormW next, int split, float* hout) {
        const float* gz = gated ? (const float*)y.gz.p : (const float*)nullptr;
        if (W % 4 == 0)
            launch(lc, "join", 0, ly_join_kernel<4>, dim3(Ti), dim3(std::min(Ti <= kNumSMs ? 1024 : 256, std::max(32, (W / 4 + 31) / 32 * 32))), 0, y.x.p, yv, y2, wa, wb,
                   gz, gate_bias, y.xs.p, hist_stride, hist_slot, dw, x0, step, next, eps, W, split, hout, hhi, hlo);
        else
            launch(lc, "join", 0, ly_join_kernel<1>, dim3(Ti), dim3(nthr), 0, y.x.p, yv, y2, wa, wb, gz, gate_bias, y.xs.p, hist_stride, hist_slot, dw, x0, step, next,
                   eps, W, split, hout, hhi, hlo);
    };
    // a sublayer's result (still in split-K slices, perhaps) is normed (weight wb, wplain) and joins the stream
    // (hout as above)
    auto post_norm = [&](const Slices& yv, const float* yb, const float* wb, int wplain, NormW next, const float* ls, const float* x0, const float* step, int split,
                         float* hout) {
        if (W % 4 == 0)
            launch(lc, "post_norm", 0, ly_post_norm_kernel<4>, dim3(Ti), dim3(std::min(Ti <= kNumSMs ? 1024 : 256, std::max(32, (W / 4 + 31) / 32 * 32))), (size_t)W * 4,
                   y.x.p, yv, yb, wb, next, ls, x0, step, eps, W, wplain, split, hout, hhi, hlo);
        else
            launch(lc, "post_norm", 0, ly_post_norm_kernel<1>, dim3(Ti), dim3(nthr), (size_t)W * 4, y.x.p, yv, yb, wb, next, ls, x0, step, eps, W, wplain, split, hout,
                   hhi, hlo);
    };
    // the other arrangements read the folded rows
    auto fold = [&](Slices& s) {
        if (s.n > 1)
            launch(lc, "sum_slices", 0, ly_sum_slices_kernel, dim3((unsigned)std::min<size_t>(4 * kNumSMs, (s.stride + 255) / 256)), dim3(256), 0, s.p, s.n, s.stride,
                   s.stride, y.y.p);
        s = Slices{y.y.p, 1, 0};
    };
    // the experts of a layer over all rows: out[row] = sum of the chosen ones' weighted outputs (+ the shared one)
    auto experts = [&](const LayeredLayerW& lw, float* out) {
        const fl_layer_desc& d = lw.d;
        const int F = d.ff, act = d.ffn_act, GF = act == FL_ACT_RELU2 ? F : 2 * F;
        const int E = d.experts, top = d.top, P = Ti * top;
        if (d.router != FL_ROUTER_SOFTMAX) {
            auto route = [&](auto kern, int rb) {
                launch(lc, "moe_router", 0, kern, dim3((Ti + rb - 1) / rb), dim3(256), (size_t)rb * (2 * E + d.route_groups) * 4, sub_in, W, (const float*)lw.router, E, top,
                       d.router == FL_ROUTER_SOFTMAX_GROUPS ? 1 : 0, (const float*)lw.route_corr, d.route_groups, d.route_keep, d.route_best ? 0 : 1, d.route_renorm, Ti,
                       y.route_sel.p, y.route_w.p);
            };
            if (Ti >= 1024) route(ly_router_groups_kernel<4>, 4);       // (at most 48 KB of shared memory: E <= 1024)
            else route(ly_router_groups_kernel<1>, 1);
        }
        else
            launch(lc, "moe_router", 0, ly_router_kernel, dim3(Ti), dim3(256), (size_t)E * 4, sub_in, W, (const float*)lw.router, (const float*)lw.router_b, E, top,
                   (const float*)lw.shared_gate, y.route_sel.p, y.route_w.p, y.sgate.p);
        const float* sg = lw.shared_gate ? (const float*)y.sgate.p : (const float*)nullptr;    // nullptr: the shared expert counts fully
        const float* sh = nullptr;
        if (d.shared_ff > 0 && !par) {  // the always-on expert first (parallel sublayers hold it in the mixer's matrices): its split-K scratch is free again before the routed experts run
            const int Fs = d.shared_ff;
            const Slices gu = gemm_slices(c, lc, "gemm_shared_in", sub_in, hhi, hlo, lw.s_gu, lw.tm_sgu, lw.tc_sgu, 2 * Fs, W, y.sh_gu.p, Ti);
            launch_glu(lc, gu, Ti, Fs, d.shared_limit, act, nullptr, lw.tc_sdown ? (float*)nullptr : y.sh_act.p, lw.tc_sdown ? ahi : (uint16_t*)nullptr, alo);
            gemm_tc_or_exact(c, lc, "gemm_shared_out", y.sh_act.p, ahi, alo, lw.s_down, lw.tm_sdown, lw.tc_sdown, W, Fs, y.sh_o.p, Ti);
            sh = y.sh_o.p;
        }
        const dim3 gw((W + 255) / 256, Ti);
        if (lw.tc_moe && Ti > 128) {
            // many rows: every expert over all rows on the tensor cores, kept where the row picked it (ascending expert order)
            for (int e = 0; e < E; ++e) {
                dense_gemm(c, lc, "gemm_tc_moe_in", Ti, GF, W, lw.tm_egu[e], y.gu.p, hhi, hlo);
                launch_glu(lc, Slices{y.gu.p, 1, 0}, Ti, F, d.limit, act, nullptr, nullptr, ahi, alo);
                dense_gemm(c, lc, "gemm_tc_moe_out", Ti, W, F, lw.tm_edown[e], y.eo.p, ahi, alo);
                launch(lc, "moe_accum", 0, ly_moe_accum_kernel, gw, dim3(256), 0, (const float*)y.eo.p, (const int*)y.route_sel.p,
                       (const float*)y.route_w.p, top, e, (const float*)nullptr, e == 0 ? 1 : 0, W, out);
            }
            if (sh != nullptr)
                launch(lc, "moe_accum", 0, ly_moe_accum_kernel, gw, dim3(256), 0, sh, (const int*)nullptr, (const float*)nullptr, 0, -1,
                       sg, 0, W, out);
        } else {
            launch(lc, "moe_lists", 0, ly_moe_lists_kernel, dim3(E), dim3(32), 0, (const int*)y.route_sel.p, Ti, top, E, y.grp_off.p, y.pair_row.p,
                   y.pair_of.p);
            if (lw.tc_moe) {
                // few rows: ONE grouped GEMM pair over (expert, weight tile, k slice) items; an expert without rows costs nothing
                const int cap = Ti <= 16 ? 16 : (Ti <= 32 ? 32 : (Ti <= 64 ? 64 : 128));
                launch(lc, "moe_gather", 0, ly_moe_gather_kernel, dim3(E, std::min(Ti, 16)), dim3(256), 0, (const uint16_t*)hhi, (const uint16_t*)hlo, W,
                       (const int*)y.grp_off.p, (const int*)y.pair_row.p, cap, y.gx_hi.p, y.gx_lo.p, y.grp_cnt.p);
                int ks = dense_gemm_grouped(c, lc, "gemm_tc_moe_in", E, cap, GF, W, lw.tm_gu, y.gemm_out.p, y.gx_hi.p, y.gx_lo.p, y.grp_cnt.p);
                FL_CHECK((size_t)ks * E * cap * GF <= y.gemm_out.n, FL_ERR_STATE, "internal: grouped GEMM scratch too small");
                launch(lc, "glu_grouped", 0, ly_glu_grouped_kernel, dim3((F + 255) / 256, E * cap), dim3(256), 0, (const float*)y.gemm_out.p, ks,
                       (size_t)E * cap * GF, F, d.limit, act, (const int*)y.grp_cnt.p, cap, y.ga_hi.p, y.ga_lo.p);
                ks = dense_gemm_grouped(c, lc, "gemm_tc_moe_out", E, cap, W, F, lw.tm_down, y.gemm_out.p, y.ga_hi.p, y.ga_lo.p, y.grp_cnt.p);
                FL_CHECK((size_t)ks * E * cap * W <= y.gemm_out.n, FL_ERR_STATE, "internal: grouped GEMM scratch too small");
                launch(lc, "moe_combine", 0, ly_moe_combine_grouped_kernel, gw, dim3(256), 0, (const float*)y.gemm_out.p, ks, (size_t)E * cap * W,
                       (const int*)y.route_sel.p, (const int*)y.pair_of.p, (const int*)y.grp_off.p, cap, (const float*)y.route_w.p, top, sh,
                       sg, W, out);
            } else {
                LyGemm g1{sub_in, 0, W, y.pair_row.p, lw.w_gu, (long long)GF * W, GF, W, y.gu.p, 0, GF, y.grp_off.p, P};
                gemm_groups(lc, "gemm_moe_in", g1, E, P);
                launch_glu(lc, Slices{y.gu.p, 1, 0}, P, F, d.limit, act, nullptr, y.act.p, nullptr, nullptr);
                LyGemm g2{y.act.p, 0, F, nullptr, lw.w_down, (long long)W * F, W, F, y.eo.p, 0, W, y.grp_off.p, P};
                gemm_groups(lc, "gemm_moe_out", g2, E, P);
                launch(lc, "moe_combine", 0, ly_moe_combine_kernel, gw, dim3(256), 0, (const float*)y.eo.p, (const int*)y.pair_of.p,
                       (const float*)y.route_w.p, top, sh, sg, W, out);
            }
        }
    };
    const int n_runs = (int)m.runs.size();
    for (int run = 0; run < n_runs; ++run) {
        const int li = m.runs[run].layer, pass = m.runs[run].pass;
        const LayeredLayerW& lw = m.layers[li];
        const fl_layer_desc& d = lw.d;
        const int H = d.heads, Dv = d.vdim;
        sublayer_front(lw, run, 0);
        if (shifted) shift_front(lw, run);
        Slices in = gemm_slices(c, lc, "gemm_mix_in", shifted ? (const float*)y.hc.p : sub_in, hhi, hlo, lw.w_in, lw.tm_in, lw.tc_in, lw.n_in, W, y.proj.p, Ti);
        const bool folds = !lw.side && (d.mixer == FL_MIXER_ATTN || (d.mixer == FL_MIXER_LATENT_ATTN && d.q_rank > 0));     // mixers that fold the slices themselves
        if (in.n > 1 && !folds) {
            launch(lc, "sum_slices", 0, ly_sum_slices_kernel, dim3((unsigned)std::min<size_t>(4 * kNumSMs, (in.stride + 255) / 256)), dim3(256), 0, in.p, in.n, in.stride,
                   in.stride, y.proj.p);
            in = Slices{y.proj.p, 1, 0};
        }
        const bool last = run + 1 == n_runs, has_ff = d.ffn != FL_FFN_NONE;
        const NormW next1 = (pre && !last) ? norm1_of(run + 1) : NormW{};
        const int more = last ? 0 : split_x;               // whether another sublayer reads x after this layer
        // what joins the stream between this layer and the next run when that one starts a pass of the loop
        const bool into_pass = !last && m.runs[run + 1].pass_start;
        const int next_pass = into_pass ? m.runs[run + 1].pass : 0;
        const float* again = (into_pass && next_pass > 0 && m.cfg.loop_reinject) ? (const float*)y.xs.p : (const float*)nullptr;
        const float* pstep = (into_pass && m.cfg.loop_step) ? (const float*)m.loop_step + (size_t)next_pass * W : (const float*)nullptr;
        float* h_next = !last && halves_only(run + 1) ? nullptr : y.h.p;
        // the layer's last join: behind it (or, with token vectors, behind theirs) the stream gains what a loop adds and the next norm follows
        auto last_join = [&](const Slices& yv, const float* y2, const float* wa, const float* wb, const float* gate_bias) {
            const int hist = depth ? li + 1 : -1;
            if (!tside) { join(yv, y2, wa, wb, gate_bias, hist, lw.dwa, again, pstep, next1, more, h_next); return; }
            join(yv, y2, wa, wb, gate_bias, -1, nullptr, nullptr, nullptr, NormW{}, lw.tc_tgate ? 1 : 0, nullptr);
            const int S = m.cfg.token_side;
            const Slices z = gemm_slices(c, lc, "gemm_side_gate", y.x.p, hhi, hlo, lw.side_gate, lw.tm_tgate, lw.tc_tgate, S, W, y.tz.p, Ti);
            launch(lc, "token_side", 0, ly_token_side_kernel, dim3(Ti), dim3(std::min(256, (S + 31) / 32 * 32)), 0, z, st.tok,
                   (const uint16_t*)m.side_embed + (size_t)li * S, (size_t)m.L * S, S, lw.tc_tproj ? (float*)nullptr : y.ta.p,
                   lw.tc_tproj ? y.ta_hi.p : (uint16_t*)nullptr, y.ta_lo.p);
            const Slices v = gemm_slices(c, lc, "gemm_side_proj", y.ta.p, y.ta_hi.p, y.ta_lo.p, lw.side_proj, lw.tm_tproj, lw.tc_tproj, W, S, y.y.p, Ti);
            post_norm(v, nullptr, lw.side_norm, 1, next1, nullptr, again, pstep, more, h_next);
        };
        if (par) {          // mixer and feed-forward read the same h and join together
            const int off = lw.u_ld - lw.fx;
            if (lw.fx > 0)
                launch_glu(lc, Slices{in.p + lw.off_ff, in.n, in.stride}, Ti, lw.fx, d.ffn == FL_FFN_MOE ? d.shared_limit : d.limit, d.ffn_act, nullptr,
                           lw.tc_o ? (float*)nullptr : y.u.p + off, lw.tc_o ? uhi + off : (uint16_t*)nullptr, lw.tc_o ? ulo + off : (uint16_t*)nullptr, lw.n_in, lw.u_ld);
            run_mixer(c, lc, st, lw, in, pass, slots, counts, n, h_row0, h_pos0);
            if (d.ffn == FL_FFN_MOE) experts(lw, y.y2.p);
            const Slices both = gemm_slices(c, lc, "gemm_mix_out", y.u.p, uhi, ulo, lw.w_o, lw.tm_o, lw.tc_o, W, lw.u_ld, y.y.p, Ti);
            last_join(both, d.ffn == FL_FFN_MOE ? (const float*)y.y2.p : (const float*)nullptr, nullptr, nullptr, nullptr);
            continue;
        }
        run_mixer(c, lc, st, lw, in, pass, slots, counts, n, h_row0, h_pos0);
        Slices mix = gemm_slices(c, lc, "gemm_mix_out", y.u.p, uhi, ulo, lw.w_o, lw.tm_o, lw.tc_o, W, H * Dv, y.y.p, Ti), ff{y.y.p, 1, 0};
        if (sum_norm || lw.side) fold(mix);
        if (lw.side) {
            const LayeredLayerW& sw = *lw.side;
            run_mixer(c, lc, st, sw, in, pass, slots, counts, n, h_row0, h_pos0);
            gemm_tc_or_exact(c, lc, "gemm_mix_out", y.u.p, uhi, ulo, sw.w_o, sw.tm_o, sw.tc_o, W, sw.d.heads * sw.d.vdim, y.y2.p, Ti);
        }
        // whether the feed-forward takes its input as hi | lo halves only
        const bool ff_halves = lw.tc_gu && d.ffn == FL_FFN_DENSE && !canon && !gated;
        const NormW norm2 = norm_of(lw.norm2, lw.norm2_bias, lw.norm2_alpha);
        float* h_ff = ff_halves ? nullptr : y.h.p;
        if (sum_norm)
            sum_norm_join(nullptr, lw.side ? (const float*)y.y2.p : (const float*)nullptr, lw.side ? d.out_scale : 1.f, lw.side ? lw.side->d.out_scale : 0.f,
                          lw.norm1b, (has_ff || !shifted) ? (has_ff ? split_x : more) : 0);
        else if (post)
            post_norm(mix, nullptr, lw.norm1b, plain, has_ff ? norm2 : next1, lw.ls1, has_ff ? nullptr : again, has_ff ? nullptr : pstep, has_ff ? split_x : more,
                      has_ff ? h_ff : h_next);
        else if (has_ff)
            join(mix, lw.side ? (const float*)y.y2.p : (const float*)nullptr, lw.pair_wa, lw.pair_wb, lw.rg1b, -1, nullptr, nullptr, nullptr, norm2, 0, h_ff);
        else
            last_join(mix, lw.side ? (const float*)y.y2.p : (const float*)nullptr, lw.pair_wa, lw.pair_wb, lw.rg1b);
        if (!has_ff) continue;
        sublayer_front(lw, run, 1);
        const int F = d.ff, act = d.ffn_act, GF = act == FL_ACT_RELU2 ? F : 2 * F;
        if (d.ffn == FL_FFN_DENSE) {
            const Slices gu = gemm_slices(c, lc, "gemm_ff_in", sub_in, hhi, hlo, lw.w_gu, lw.tm_gu, lw.tc_gu, GF, W, y.gu.p, Ti);
            launch_glu(lc, gu, Ti, F, d.limit, act, lw.b_gu, lw.tc_down ? (float*)nullptr : y.act.p, lw.tc_down ? ahi : (uint16_t*)nullptr, alo);
            ff = gemm_slices(c, lc, "gemm_ff_out", y.act.p, ahi, alo, lw.w_down, lw.tm_down, lw.tc_down, W, F, y.y.p, Ti);
            if (sum_norm) fold(ff);
        } else {
            experts(lw, y.y.p);
        }
        if (sum_norm)
            sum_norm_join(lw.b_down, nullptr, 1.f, 0.f, lw.norm2b, shifted ? 0 : more);
        else if (post)
            post_norm(ff, lw.b_down, lw.norm2b, plain, next1, lw.ls2, again, pstep, more, h_next);
        else
            last_join(ff, nullptr, nullptr, nullptr, lw.rg2b);
    }
    if (n_want > 0) {
        launch(lc, "final_norm", 0, ly_final_norm_kernel, dim3(n_want), dim3(nthr), 0, (const float*)y.x.p, st.want, norm_of(m.final_norm, m.final_bias, m.final_alpha),
               eps, W, m.cfg.logit_scale != 0.f ? m.cfg.logit_scale : 1.f, y.hf.p,
               m.tc_head ? y.hf_hi.p : (uint16_t*)nullptr, y.hf_lo.p);
        gemm_tc_or_exact(c, lc, "gemm_head", y.hf.p, m.tc_head ? y.hf_hi.p : nullptr, y.hf_lo.p, m.head, m.tm_head, m.tc_head, m.V, W, y.logits.p, n_want);
        if (m.cfg.logit_softcap > 0.f) {
            const size_t nl = (size_t)n_want * m.V;
            launch(lc, "logit_cap", 0, ly_softcap_kernel, dim3((unsigned)std::min<size_t>(4 * kNumSMs, (nl + 255) / 256)), dim3(256), 0, y.logits.p, nl,
                   m.cfg.logit_softcap);
        }
    }
}

}  // namespace fl
