"""Dikusun put together from the parts, and its registration.

A layer is a post-norm block: the sublayers read the float32 stream itself, and each one's output passes an RMS norm before it
is added.  The mixer is one of three, as the configuration's layer list says, in any order:
  * `latent_attention`: softmax attention over cached latents without positions;
  * `attention`: differential softmax attention (two maps a head over the same values, each query and key normed and rotated
    by itself) under a sliding window with capped scores, biases on its four products and a gate per head;
  * `gla`: linear attention whose state decays by a gate per key channel, a silu gate on the heads' normed outputs.
The feed-forward is a dense clamped gated unit, or none.  A layer may use another layer's weights (mixer, feed-forward and
norms): the order then runs that layer's block once more, with a cache entry of its own.
Tensor names: `embed`, `l<i>.norm1`, `l<i>.norm2`, `l<i>.mix.<role>`, `l<i>.mlp.gate|up|down`, `final.norm`, `head`.

The design has no context limit of its own; positions are int32 and their angles 32-bit floats, exact up to 2^24.
"""
from __future__ import annotations

from ..config.dikusun import DifferentialMixer, DikusunConfig, GlaMixer, LatentMixer
from ..parts import ClampedGLU, GatedLinearAttention, LatentAttention, LogitsHead, MaskedAttention, PostNormBlock, RMSNorm, TokenEmbedding
from ..registry import register_architecture
from .model import LayerStep, Model

MAX_POSITIONS = 1 << 24
ALPHA = 1.702                      # of the clamped unit's sigmoid


def _mixer(cfg: DikusunConfig, m):
    E, eps = cfg.width, cfg.norm_eps
    if isinstance(m, LatentMixer):
        return LatentAttention(E, m.heads, m.dim, 0, m.vdim, m.q_rank, m.kv_rank, m.scale, 1.0, 0, eps)
    if isinstance(m, DifferentialMixer):
        return MaskedAttention(E, m.heads, m.kv_heads, m.dim, m.vdim, scale=m.scale, qk_norm_eps=eps, rot_dims=m.rot_dims,
                               rot_base=m.rot_base, window=m.window, bias=True, softcap=m.softcap, difference=m.diff,
                               difference_eps=eps, head_gate=True)
    if isinstance(m, GlaMixer):
        return GatedLinearAttention(E, m.heads, m.dim, m.vdim, m.tau, eps, decay_rank=m.decay_rank or -1)
    raise TypeError(type(m).__name__)


def build_dikusun(cfg: DikusunConfig) -> Model:
    E, eps = cfg.width, cfg.norm_eps
    owners = [i for i, layer in enumerate(cfg.layers) if layer.weights_of is None]
    blocks = []
    for i in owners:
        layer = cfg.layers[i]
        ffn = None if layer.mlp is None else ClampedGLU(E, layer.mlp.ff, layer.mlp.limit, alpha=ALPHA)
        blocks.append(PostNormBlock(_mixer(cfg, layer.mixer), RMSNorm(E, eps, role=""), ffn, None if ffn is None else RMSNorm(E, eps, role="")))
    order = [LayerStep(owners.index(cfg.owner(i)), i) for i in range(len(cfg.layers))]
    embedding = TokenEmbedding(cfg.vocab, E, scale=cfg.embedding_scale, role="")
    head = LogitsHead(RMSNorm(E, eps, role=""), cfg.vocab, E, role="")
    # A layer without a feed-forward has no use for a second norm; a file may hold its weight all the same.
    unused = [f"l{i}.norm2" for i in owners if cfg.layers[i].mlp is None]
    return Model(embedding=embedding, blocks=blocks, head=head, order=order, vocab_size=cfg.vocab, max_positions=MAX_POSITIONS,
                 block_prefix=lambda b: f"l{owners[b]}.", embedding_prefix="embed.", head_norm_prefix="final.norm.", head_prefix="head.",
                 ignorable=unused)


register_architecture(("Dikusun", "dikusun"), DikusunConfig, build_dikusun)
