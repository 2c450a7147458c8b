/*
 * vb_lm_config.h - what a decoder language model is made of, as read from a model folder's
 * config.json, and the registry of designs that are read this way.
 *
 * A model is an embedding, a list of layers (mixer + optional feed-forward), an optional loop over
 * a part of the list, a final norm and a head. Every mechanism carries its constants as
 * parameters, so that a design is a combination of them.
 */
#ifndef VB_LM_CONFIG_H
#define VB_LM_CONFIG_H

#include <string>
#include <vector>

#include "vb_json.h"

namespace vb {

enum LmMixerKind { LM_MIXER_ATTENTION = 0, LM_MIXER_DELTA = 1 };

/* Rotary positions on the first `dims` dimensions of a head, i paired with i + dims / 2. */
struct LmRope {
    int dims = 0;                          /* 0: no rotation */
    double base = 0.0;
    bool yarn = false;                     /* frequency blend + magnitude, parameters below */
    double factor = 1.0, original = 0.0, fast = 0.0, slow = 0.0;
    /* Angle per position of every rotated pair, and the factor on cos and sin. */
    std::vector<double> frequencies() const;
    double magnitude() const;
};

/* Which keys a query sees, besides j <= i: all of them (window == 0), or the last `window` ones
 * (itself included) and the first `keep_first` of the sequence. */
struct LmMask {
    int window = 0, keep_first = 0;
};

struct LmMixer {
    LmMixerKind kind = LM_MIXER_ATTENTION;
    int heads = 0, kv_heads = 0, dim = 0, vdim = 0;
    /* attention */
    LmRope rope;
    LmMask mask;
    double scale = 0.0, softcap = 0.0;     /* softcap 0: none */
    /* delta rule */
    int taps = 0;                          /* short convolution, current token included */
};

struct LmLayer {
    LmMixer mixer;
    int ff = 0;                            /* gated feed-forward size; 0: the layer has none */
};

struct LmConfig {
    std::string architecture;
    int vocab = 0, width = 0;
    double eps = 0.0;
    std::vector<LmLayer> layers;
    int loop_start = 0, loop_stop = 0, loop_times = 0;   /* loop_times 0: no loop */

    /* Layers in execution order: index of the layer, and whether a pass of the loop begins there
     * (the loop's input projection runs right before it). Every entry owns its cache or state. */
    struct Run { int layer; bool begins_pass; };
    std::vector<Run> runs() const;
};

/* A registered design: the name in config.json's "architecture" and the reader of its keys. */
struct LmArchitecture {
    const char *name;
    bool (*read)(const Json &config, LmConfig *out, std::string *err);
};
const LmArchitecture *lm_architecture(const std::string &name);

/* Parses a config.json text and dispatches on its architecture. */
bool lm_config_from_text(const std::string &text, LmConfig *out, std::string *err);

} // namespace vb

#endif
