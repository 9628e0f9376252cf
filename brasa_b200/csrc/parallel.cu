// Two mixers side by side on the same input ("parallel"): windowed attention and a state-space mixer, each with a constant factor.
// Their projections go into one launch, and the sum of their output projections is one product over the concatenation of their
// results (the factors are applied to the results, in f32).
#include "stack.h"

namespace brasa_stack {
namespace {

class Parallel : public Mixer {
  public:
    bool configure(const brasa::Json &c, uint32_t width, float eps, std::string &err) override {
        static const char *const SIDE[2] = {"left", "right"};
        side_[0] = make_window_attention();
        side_[1] = make_state_space();
        for (int i = 0; i < 2; ++i) {
            const brasa::Json *j = c.get(SIDE[i]);
            double f;
            if (!j || j->kind != brasa::Json::Obj) return err = std::string("parallel: ") + SIDE[i] + " is missing", false;
            if (!read_f64(c, i ? "right_scale" : "left_scale", &f, err) || !side_[i]->configure(*j, width, eps, err)) return false;
            if (!side_[i]->scale_output((float)f)) return err = std::string("parallel: ") + SIDE[i] + " cannot be scaled", false;
        }
        return true;
    }

    int32_t build(Builder &b, const std::string &x) override {
        BRASA_TRY(side_[0]->build(b, x + "left."));
        BRASA_TRY(side_[1]->build(b, x + "right."));
        outs = {side_[0]->outs[0], side_[1]->outs[0]};
        return BRASA_OK;
    }

    uint64_t scratch_bytes() const override { return offset(side_[0]->scratch_bytes()) + side_[1]->scratch_bytes(); }

    void project(const Run &r, std::vector<GemvProblem> &out) override {
        side_[0]->project(of(r, 0), out);
        side_[1]->project(of(r, 1), out);
    }

    int32_t mix(const Run &r) override {
        BRASA_TRY(side_[0]->mix(of(r, 0)));
        return side_[1]->mix(of(r, 1));
    }

  private:
    static uint64_t offset(uint64_t n) { return (n + 255) / 256 * 256; }
    Run of(const Run &r, int i) const {
        Run s = r;
        s.out[0] = r.out[i];
        s.ldo[0] = r.ldo[i];
        if (i) s.scratch += offset(side_[0]->scratch_bytes());
        return s;
    }

    std::unique_ptr<Mixer> side_[2];
};

}  // namespace

std::unique_ptr<Mixer> make_parallel() { return std::unique_ptr<Mixer>(new Parallel()); }

}  // namespace brasa_stack
