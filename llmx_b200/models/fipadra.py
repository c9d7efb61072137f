"""Fipadra put together from the parts, and its registration.

The embedding's rows pass an RMS norm of their own before the first layer.  A layer is a parallel block with two norms:
the mixer reads one RMS norm of the stream and the feed-forward another (each with a weight of its own), and both add
into the float32 residual.  The mixer is one of three, as the configuration's layer list says, in any order:
  * `retention`: linear attention with a constant decay per head, q and k rotated in the two-halves pairing, no
    activation, every head's output divided by its root mean square, a silu gate;
  * `delta`: the gated delta rule with one decay per head behind a short filter, a silu gate;
  * `latent_attention`: softmax attention over cached latents under a sliding window, neighbouring pairs rotated.
The feed-forward is a dense unit whose activation is the square of relu, or a mixture of experts: clamped gated units
chosen by a softmax over all of the router's outputs plus a correction that counts for the choice alone, groups of
experts of which the best are kept, identity experts, and a shared unit under a sigmoid gate.  The logits are made with
the embedding's table and carry a factor.
Tensor names: `embed`, `embed.norm`, `l<i>.norm1`, `l<i>.norm2`, `l<i>.mix.<role>`, `l<i>.mlp.<role>`, `final.norm`.

The design has no context limit of its own; positions are int32 and their angles 32-bit floats, exact up to 2^24.
"""
from __future__ import annotations

from ..config.fipadra import DeltaMixer, DenseMlp, FipadraConfig, LatentMixer, RetentionMixer, RoutedMlp
from ..parts import (ActivatedMLP, ClampedGLU, DecayedLinearAttention, GatedDeltaRule, LatentAttention, LogitsHead, ParallelBlock,
                     RMSNorm, RoutedExperts, TokenEmbedding)
from ..registry import register_architecture
from .model import Model

MAX_POSITIONS = 1 << 24
ALPHA = 1.702                      # of the clamped units' sigmoid


def _mixer(cfg: FipadraConfig, m):
    E, eps = cfg.width, cfg.norm_eps
    if isinstance(m, RetentionMixer):
        return DecayedLinearAttention(E, m.heads, m.dim, m.vdim, m.decay, eps, activation=None, rot_dims=m.rot_dims, rot_base=m.rot_base,
                                      key_factor=m.dim ** -0.5, norm="heads", gate="silu")
    if isinstance(m, DeltaMixer):
        return GatedDeltaRule(E, m.heads, m.kv_heads, m.dim, m.vdim, m.conv, eps)
    if isinstance(m, LatentMixer):
        return LatentAttention(E, m.heads, m.dim, m.rot_dim, m.vdim, m.q_rank, m.kv_rank, m.scale, m.rot_base, m.rot_dims,
                               eps, window=m.window)
    raise TypeError(type(m).__name__)


def _feed_forward(cfg: FipadraConfig, m):
    E = cfg.width
    if m is None:
        return None
    if isinstance(m, DenseMlp):
        return ActivatedMLP(E, m.ff, activation="relu2", names=("up", "down"))
    if isinstance(m, RoutedMlp):
        shared = None if m.shared is None else ClampedGLU(E, m.shared.ff, m.shared.limit, alpha=ALPHA)
        return RoutedExperts(E, m.experts, m.top, m.expert.ff, shared=shared, shared_gate=True, router_bias_role=None,
                             scores="all", correction_role="correction", groups=(m.group_count, m.group_keep), identity=m.identity,
                             weight_scale=m.scale, clamp=(m.expert.limit, ALPHA))
    raise TypeError(type(m).__name__)


def build_fipadra(cfg: FipadraConfig) -> Model:
    E, eps = cfg.width, cfg.norm_eps
    blocks = []
    for layer in cfg.layers:
        ffn = _feed_forward(cfg, layer.mlp)
        blocks.append(ParallelBlock(RMSNorm(E, eps, role=""), _mixer(cfg, layer.mixer), ffn, names=("norm1", "mix", "mlp"),
                                    ffn_norm=None if ffn is None else RMSNorm(E, eps, role=""), ffn_norm_name="norm2"))
    embedding = TokenEmbedding(cfg.vocab, E, role="", norm=RMSNorm(E, eps, role=""))
    head = LogitsHead(RMSNorm(E, eps, role=""), cfg.vocab, E, tied_to=embedding, scale=cfg.logit_scale)
    # A layer without a feed-forward has no use for a second norm; a file may hold its weight all the same.
    unused = [f"l{i}.norm2" for i, layer in enumerate(cfg.layers) if layer.mlp is None]
    return Model(embedding=embedding, blocks=blocks, head=head, vocab_size=cfg.vocab, max_positions=MAX_POSITIONS,
                 block_prefix=lambda i: f"l{i}.", embedding_prefix="embed.", head_norm_prefix="final.norm.", head_prefix="head.",
                 ignorable=unused)


register_architecture(("Fipadra", "fipadra"), FipadraConfig, build_fipadra)
