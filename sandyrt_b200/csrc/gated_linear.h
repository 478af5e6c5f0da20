// What tells one recurrence with a decay per key channel from another (gated_linear.cu), in one structure that its entry
// points take.  Zeros: gated linear attention with as many query/key heads as heads (inv_tau is then still to be given).
#pragma once

enum SandyFadeKind { SANDY_FADE_ADD = 0, SANDY_FADE_BONUS = 1, SANDY_FADE_DELTA = 2 };
enum SandyDecayForm { SANDY_DECAY_LOGSIGMOID = 0, SANDY_DECAY_EXP = 1, SANDY_DECAY_SOFTPLUS = 2 };

typedef struct SandyFadeRule {
    int kind;               // how a token enters the state and is read (SandyFadeKind)
    int decay;              // the decay's logarithm: logsigmoid(z) * inv_tau, -exp(z) or -exp(a_log[h]) * softplus(z)
    float inv_tau;
    int tanh_low;           // 1: z = W2 tanh(low) + bias, 0: z = W2 low + bias
    const float* a_log;     // float32 [H] (softplus form)
    const float* bonus;     // float32 [H * qk_dim] (bonus): the current token's own factor per key channel
    const float* beta;      // float32 [T, ld_beta] (delta): pre-activations of the step size, one per head
    int ld_beta;
    int n_qk_heads;         // query/key heads; head h reads query/key head h / (H / n_qk_heads).  0: one for every head
} SandyFadeRule;
