// Layer-stack models (host only): the configuration of a decoder whose config.json lists its layers one by one, each with a mixer
// and a feed-forward of its own, and the registry that maps the file's "architecture" to the design it names.
//
// A design is a set of rules fixed in code (its norm, its activation, how a residual block is put together) plus the numbers of
// its config.json; a mixer is named by the layer's "type".  Both are looked up in tables (stack_config.cpp), so that another
// design adds a table entry and the mechanisms it needs.
#pragma once
#include <cstdint>
#include <string>
#include <vector>

namespace l2b {

enum class MixerKind { LatentAttention, DifferentialAttention, Mlstm };
enum class MlpKind { None, GatedGeluTanh, GatedSilu };
enum class NormKind { DynamicTanh, Rms };

struct RotaryConfig {  // pair i < dims/2 is turned by position * base^(-2i/dims); which two dimensions form it is the mixer's
    double base = 10000.0;
    int dims = 0;
};

struct MixerConfig {
    MixerKind kind = MixerKind::LatentAttention;
    int heads = 0;
    int dim = 0;      // query / key dimensions per head (latent attention: the unrotated ones; differential attention: per map)
    int vdim = 0;     // value dimensions per head
    float scale = 1.f;
    RotaryConfig rot;
    // latent attention
    int rot_dim = 0;  // rotated dimensions; the rotated key part is shared by all heads
    int kv_rank = 0;  // size of the cached latent
    // differential attention
    int kv_heads = 0;
    int chunk = 0;      // a position sees its own chunk of this many positions (0: everything before it)
    float diff = 0.f;   // constant part of the second map's weight
    int kv_from = -1;   // layer whose cached keys and values are used (-1: this layer has its own)
    // matrix memory (mLSTM)
    float gate_cap = 1.f;
};

struct StackLayerConfig {
    MixerConfig mix;
    MlpKind mlp = MlpKind::None;
    int ff = 0;
};

struct LayerRun {
    int layer;
    int pass;  // number of the loop pass this run begins, or -1
};

struct StackConfig {
    std::string architecture;
    int vocab = 0, width = 0;
    float embed_scale = 1.f;
    int max_positions = 0;   // rows of the table of learned position vectors (0: there is none)
    float logit_scale = 1.f;
    NormKind norm = NormKind::DynamicTanh;
    bool post_norm = false;  // the result of a sublayer is normed before it is added to the residual stream
    float eps = 1e-5f;
    int loop_start = 0, loop_stop = 0, loop_times = 0;  // layers start .. stop-1 run `times` times in a row (0 times: no loop)
    int side_dim = 0;                                   // per-layer token input (0: none)
    std::vector<StackLayerConfig> layers;
    bool has_loop() const { return loop_times > 0; }
    bool recurrent() const;              // some layer carries a state from position to position
    std::vector<LayerRun> runs() const;  // the layers in the order they run; every run has a cache of its own
};

// False (with a message) when the text is not JSON, names an unknown architecture, or misses or contradicts something.
bool parse_stack_config(const char* json, size_t n, StackConfig& out, std::string& err);

}  // namespace l2b
