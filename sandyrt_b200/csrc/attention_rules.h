// What an attention layer may add to plain causal softmax attention, in one structure that every attention entry point
// with a form for it takes (the `*_rules` entries).  Zeros mean: none of it.
#pragma once

typedef struct SandyAttentionRules {
    int window;              // > 0: a query at position pos sees keys pos - window + 1 .. pos; 0: all up to pos
    int keep_first;          // with a window: keys 0 .. keep_first - 1 stay visible behind it
    float softcap;           // > 0: a score becomes softcap * tanh(score / softcap)
    int chunk;               // > 0: a query sees only keys of its own chunk of positions (not together with keep_first)
    const float* sink;       // float32 [H] or null: exp(sink[h]) joins the softmax's denominator
    const float* out_gate;   // float32 [T, H] or null: a factor on each head's output
    const float* dist_bias;  // float32 [H, n_dist] or null: entry min(pos - j, n_dist - 1) joins the score of key j
    int n_dist;
    const void* elem_gate;   // pre-activations of the query's type, or null: element i < gate_dim of head h is multiplied by
    int ld_elem_gate;        // sigmoid(elem_gate[t * ld_elem_gate + h * gate_dim + i])
    int gate_dim;
} SandyAttentionRules;
