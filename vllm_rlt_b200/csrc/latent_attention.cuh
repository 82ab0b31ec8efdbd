// Arguments of the prompt kernel over packed keys and values (attention_latent_prompt_sm100.cu explains the operands).
#pragma once

#include "attention.cuh"

namespace rlt {

// Up to 256 consecutive query rows of one sequence; eight words, built on the host.
struct PromptTile {
  int q_row;       // first row in the packed queries
  int count;
  int position;    // of the first row in its sequence
  int key_row;     // packed key row of position key_first
  int key_first;   // first position of the sequence that is among the packed keys
  int kept;        // positions 0 .. kept - 1 are packed in front of key_row
  int pad[2];
};

struct LatentPromptArgs {
  void* out; int64_t out_stride;
  int heads, share, vdim;   // query heads, query heads per key/value head
  const PromptTile* tiles; int tile_count;
  float scale; int window;
  const float* sink;                                               // [heads], or null
  const void* gate; int64_t gate_stride; bool gate_per_head;       // null: no gate
  unsigned* error;   // set when a bounded wait gave up
};

bool latent_prompt_supported(int dim, int rot_dim, int vdim, int dtype);

}  // namespace rlt
