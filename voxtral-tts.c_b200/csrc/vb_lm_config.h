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

enum LmMixerKind { LM_MIXER_ATTENTION = 0, LM_MIXER_DELTA = 1, LM_MIXER_LATENT = 2 };

/* Rotary positions on the first `dims` dimensions of a head (latent attention: of the rotated part).
 * Pairs: i with i + dims / 2 in an attention, 2i with 2i + 1 in a latent attention. */
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
    /* latent attention: queries through a latent of q_rank, keys and values out of a latent of kv_rank that
     * is cached with a rotated key part of rot_dim shared by the heads; `dim` is the unrotated part */
    int q_rank = 0, kv_rank = 0, rot_dim = 0;
    int kv_from = -1;                      /* layer whose latent and key part this one reads; -1: its own */
};

enum LmMlpKind { LM_MLP_NONE = 0, LM_MLP_SWIGLU = 1, LM_MLP_RELU2 = 2 };

/* Feed-forward: one of size ff, or `experts` of that size of which a token uses `top` (chosen by the
 * largest router logits, weighted by the softmax over the chosen ones). */
struct LmMlp {
    LmMlpKind kind = LM_MLP_NONE;
    int ff = 0;
    int experts = 0, top = 0;              /* experts 0: dense */
};

struct LmLayer {
    LmMixer mixer;
    LmMlp mlp;
};

/* How a layer's sublayers meet the residual stream. */
enum LmBlockKind {
    LM_BLOCK_SANDWICH = 0,                 /* x += post(mixer(pre(x))), then the same with the feed-forward */
    LM_BLOCK_PARALLEL = 1                  /* h = norm(x); x += mixer(h) + feed_forward(h) */
};
enum LmNormKind { LM_NORM_LAYER = 0, LM_NORM_RMS = 1 };   /* the norms of the stream, no bias */

struct LmConfig {
    std::string architecture;
    int vocab = 0, width = 0;
    double eps = 0.0;
    LmBlockKind block = LM_BLOCK_SANDWICH;
    LmNormKind norm = LM_NORM_LAYER;
    std::vector<LmLayer> layers;
    int loop_start = 0, loop_stop = 0, loop_times = 0;   /* loop_times 0: no loop */

    /* Layers in execution order: index of the layer, and whether a pass of the loop begins there
     * (the loop's input projection runs right before it). Every entry owns its cache or state. */
    struct Run { int layer; bool begins_pass; };
    std::vector<Run> runs() const;
    /* Longest look-back of the layers that read layer i's cache (its own included): 0 when one of them
     * sees every earlier key. */
    int cache_window(int i) const;
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
