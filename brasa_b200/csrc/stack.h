// Layer-stack models: a residual stream through a list of layers, each a mixer (attention, recurrence, ..) and an optional
// feed-forward, described entry by entry in the model's configuration. The stack (stack.cu) owns the embedding, the norms,
// the feed-forward, the residual stream, the head, the workspace and the bookkeeping of positions; a mixer (latent.cu,
// attention.cu, delta.cu, ssm.cu, and parallel.cu, which sets two of them side by side) owns its weights and its per-sequence
// state.
#pragma once
#include <memory>

#include "host_util.h"
#include "linear.h"
#include "model_internal.h"

namespace brasa_stack {

struct Weight {  // bf16 [rows][ld], zero between cols and ld
    const uint16_t *p = nullptr;
    uint32_t rows = 0, cols = 0, ld = 0;
};
inline uint32_t up8(uint32_t n) { return (n + 7) / 8 * 8; }
inline LinearSeg segment(const Weight &w, const void *x, uint32_t ldx) { return LinearSeg{w.p, w.ld, x, ldx, w.cols}; }

// An output projection of a mixer. parts > 0: of one token the mixer leaves the vector un-normed, and the product norms it on the
// way in (GemvInput::parts).
struct MixerOut : Weight {
    uint32_t parts = 0;
    const float *part_w = nullptr;
    float part_scale = 1.0f;
};

// Everything a model allocates goes through this: with m == nullptr it only adds up what would be allocated, so that the
// memory plan and the model are the same code.
struct Builder {
    enum Class { WEIGHTS, STATE, WORKSPACE };
    brasa_model *m = nullptr;
    const brasa::WeightFile *file = nullptr;
    brasa_cmd *cmd = nullptr;
    brasa_buf *staging = nullptr;
    brasa_limits limits{};
    bool f32 = false;       // 32-bit mode: activations, caches and products in f32
    uint64_t bytes[3] = {0, 0, 0};
    std::string err;

    uint32_t elem() const { return f32 ? 4 : 2; }
    int32_t fail(const std::string &what);
    int32_t get(Class c, uint64_t n, void **out);
    // bf16 matrix [rows][cols]; rows or cols 0 takes the tensor's own
    int32_t matrix(const std::string &name, uint32_t rows, uint32_t cols, Weight *out);
    // two matrices [rows][cols] in alternating blocks of 32 rows of each (LINEAR_ACT_SWIGLU), zero rows behind the last ones
    int32_t interleaved(const std::string &first, const std::string &second, uint32_t rows, uint32_t cols, Weight *out);
    // bf16 tensor of n values (any shape) as an f32 vector
    int32_t vector(const std::string &name, uint64_t n, const float **out);
    // cos and sin of p * base^(-2i / dims), [limits.ctx][dims / 2]; shared by the layers that ask for the same
    int32_t rope(double base, uint32_t dims, const float **cos_t, const float **sin_t);

  private:
    struct Table {
        double base;
        uint32_t dims;
        const float *c, *s;
    };
    std::vector<Table> tables_;
};

// One forward over `tokens` tokens of the sequence. dev_pos != nullptr: one token whose position is read from the device (the
// step is recorded once and replayed); all vectors are then f32.
struct Run {
    brasa_cmd *cmd;
    uint32_t tokens, pos0;
    const uint32_t *dev_pos;
    bool f32;
    const void *h;  // the mixer's normed input [tokens][ldh], f32 or bf16 (unused with dev_pos)
    uint32_t ldh;
    void *out[2];   // the mixer's results ahead of its output projections [tokens][ldo]; f32 with dev_pos
    uint32_t ldo[2];
    uint8_t *scratch;
};

class Mixer {
  public:
    virtual ~Mixer() {}
    // reads the layer's "mixer" object; width: of the residual stream
    virtual bool configure(const brasa::Json &c, uint32_t width, float eps, std::string &err) = 0;
    virtual int32_t build(Builder &b, const std::string &prefix) = 0;  // weights and per-sequence state
    virtual uint64_t scratch_bytes() const = 0;  // known once built
    virtual void project(const Run &r, std::vector<GemvProblem> &out) = 0;  // the products that read the normed input
    virtual int32_t mix(const Run &r) = 0;                                  // from those products to r.out
    virtual bool scale_output(float) { return false; }                     // results times a constant; false: not offered
    std::vector<MixerOut> outs;  // one or two; the mixer's output is the sum of these products

  protected:
    // the product of w with the normed input, f32, to the scratch area at `at`
    static void add_projection(const Run &r, const Weight &w, uint64_t at, uint32_t ld, std::vector<GemvProblem> &out) {
        GemvProblem g;
        g.p.seg[0] = segment(w, r.h, r.ldh);
        g.p.rows = w.rows;
        g.p.tokens = r.tokens;
        g.p.y = r.scratch + at;
        g.p.ldy = ld;
        out.push_back(g);
    }
};
// the mixer a configuration entry names, or null (stack.cu)
std::unique_ptr<Mixer> make_mixer(const std::string &type);
std::unique_ptr<Mixer> make_latent_attention();
std::unique_ptr<Mixer> make_channel_delta();
std::unique_ptr<Mixer> make_delta();
std::unique_ptr<Mixer> make_window_attention();
std::unique_ptr<Mixer> make_state_space();
std::unique_ptr<Mixer> make_parallel();

// readers of a configuration entry; false and a message when it is absent or out of range
bool read_u32(const brasa::Json &c, const char *key, uint32_t *out, std::string &err);
bool read_f64(const brasa::Json &c, const char *key, double *out, std::string &err);

// places in the scratch area, 256-byte aligned
struct Carver {
    uint64_t at = 0;
    uint64_t take(uint64_t n) {
        const uint64_t p = at;
        at += (n + 255) / 256 * 256;
        return p;
    }
};

}  // namespace brasa_stack
