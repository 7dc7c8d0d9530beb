// Constants of the ragged-step plans that host description and kernels share.
#pragma once

namespace tmb {

constexpr int kGluUnit = 16;          // a packed gate/up matrix alternates this many gate rows and up rows
constexpr int kMaxHeadDim = 256;      // query/key (and attention value) columns of a head
constexpr int kMaxLatent = 1024;      // columns of a cached latent row
constexpr int kMaxStreams = 16;       // residual streams
constexpr int kMaxTaps = 16;          // of a short convolution
constexpr int kMaxConvWidth = 8192;   // residual columns of models with grouped norms, short convolutions or side inputs
constexpr int kRaggedBlock = 16;      // positions per KV pool block
constexpr int kMaxExperts = 1024;     // of a layer
constexpr int kMaxTop = 32;           // experts a token uses
constexpr double kMostDecay = 4;       // of a delta rule in bf16 plans: largest scale of the log decays
constexpr int kRetentionChunk = 64;   // positions a retention state advances by at once inside a prompt portion

}  // namespace tmb
