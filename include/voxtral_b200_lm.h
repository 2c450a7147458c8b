/*
 * voxtral_b200_lm.h - decoder language models loaded from a model folder (config.json +
 * model.safetensors). No counterpart in mudler/voxtral-tts.c.
 *
 * The design is chosen by the "architecture" key of config.json. A model handle owns its weights, a
 * stream, and `max_seqs` slots; a slot holds the caches and recurrent states of one sequence, of
 * constant size for windowed and recurrent layers. Tokens are fed in portions of any length, cut
 * anywhere; logits are those of the whole sequence whatever the cuts.
 *
 * Every call returns 0 (or a count) on success and a negative value on failure, with the reason in
 * vb200_lm_error(). There is no CPU fallback. All pointers are host memory.
 */
#ifndef VOXTRAL_B200_LM_H
#define VOXTRAL_B200_LM_H

#include <stddef.h>
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

typedef struct vb200_lm vb200_lm_t;

enum { VB200_LM_BF16 = 0, VB200_LM_F32 = 1 };

typedef struct {
    int dtype;        /* VB200_LM_BF16: tensor-core GEMMs on the BF16 weights, fp32 activations as BF16 terms;
                         VB200_LM_F32: every product on the fp32 pipes */
    int max_seqs;     /* slots (0: 1) */
    int max_tokens;   /* longest sequence a slot can hold (0: 8192) */
    int block_rows;   /* longest stretch of a portion that runs at once (0: chosen by the library) */
} vb200_lm_options_t;

typedef struct {
    int vocab, width, layers, runs;   /* runs: layers counted as often as a loop repeats them */
    int max_seqs, max_tokens, block_rows, dtype;
    size_t weight_bytes, state_bytes_per_seq;
} vb200_lm_info_t;

vb200_lm_t *vb200_lm_open(const char *model_dir, const vb200_lm_options_t *options);
void vb200_lm_close(vb200_lm_t *lm);
int vb200_lm_info(vb200_lm_t *lm, vb200_lm_info_t *info);
const char *vb200_lm_error(void);

/* A free slot (>= 0), to be given back with seq_close. */
int vb200_lm_seq_open(vb200_lm_t *lm);
int vb200_lm_seq_close(vb200_lm_t *lm, int seq);
int vb200_lm_seq_length(vb200_lm_t *lm, int seq);

/* The next n tokens of a sequence. want: ascending places in [0, n) whose logits go to logits_out
 * ([n_want][vocab]); n_want may be 0. */
int vb200_lm_step(vb200_lm_t *lm, int seq, const int *tokens, int n, const int *want, int n_want, float *logits_out);

/* Greedy continuation: the n prompt tokens, then n_new tokens chosen on the device (largest logit, the
 * first one on a tie) without a host round trip per token. The last one is returned but not fed. */
int vb200_lm_generate(vb200_lm_t *lm, int seq, const int *prompt, int n, int n_new, int *out);
/* Device time in milliseconds (CUDA events) of the last generate call: its prompt, and its decoding loop. */
int vb200_lm_last_ms(vb200_lm_t *lm, float *prompt_ms, float *decode_ms);

/* Residual stream after every layer run, for parity checks: once enabled, a step of at most
 * block_rows tokens leaves [runs][n][width] to be read. */
int vb200_lm_tap_enable(vb200_lm_t *lm, int on);
int vb200_lm_tap_read(vb200_lm_t *lm, float *out, int n);

/* A model of the given config.json text with hashed random weights made on the device
 * (measurements need no file). */
vb200_lm_t *vb200_lm_open_random(const char *config_json, const vb200_lm_options_t *options, unsigned seed);
/* Host arithmetic only: 0 when the text is a configuration the library can run. */
int vb200_lm_check_config(const char *config_json);

#ifdef __cplusplus
}
#endif
#endif
