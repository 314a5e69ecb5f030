"""Sogodra put together from the parts.

A decoder whose layers each hold a mixer and, unless the layer has none, a feed-forward, with an RMS norm on each sublayer's
output only: the sublayers read the stream itself (``parts.PostNormBlock``).  The mixer is

* ``delta`` (``parts.GatedDeltaRule``): the gated delta rule with one decay per head and a SiLU gate;
* ``mingru`` (``parts.MinGru``): a recurrence per channel whose gates read the current token only;
* ``parallel`` (``parts.ParallelMixer``): attention in a sliding window (``parts.GroupedQueryAttention``: a norm per q and k head
  before the rotation, the leading entries of every head rotated in half-split pairs with long wavelengths stretched over a ramp,
  a learned sink per head) beside the gated delta rule with a decay per row of the state and a sigmoid gate through thin
  matrices, each with a factor.

The feed-forward clamps gate and up (``parts.GatedMlp`` with ``swiglu_clamp``).  The head is a matrix of its own.

Checkpoint names: ``embed``, ``head``, ``final.norm`` and per layer ``l<i>.norm1`` / ``norm2``, ``l<i>.mix.{q, k, v, q.conv,
k.conv, v.conv, b, a, A_log, dt_bias, g, norm, o}``, ``l<i>.mix.{z, z.b, x, x.b, g, o}`` or ``l<i>.mix.left.{q, k, v, q.norm, k.norm,
sink, o}`` with ``l<i>.mix.right.{q, k, v, q.conv, k.conv, v.conv, b, a1, a2, A_log, dt_bias, g1, g2, norm, o}``, and
``l<i>.mlp.{gate, up, down}``.
Fixed by the design, not by config.json: the feed-forward's activation and its 1.702, SiLU behind the convolution, the 1e-6 beside
the unit vectors' sums of squares, the two kinds of gate.
"""
from __future__ import annotations

from ..config.model_config import ConfigError
from ..config.registry import register_architecture
from ..parts import (AttentionNames, DeltaNames, GatedDeltaRule, GatedMlp, GatedMlpNames, GroupedQueryAttention, GroupedRmsNorm, MinGru,
                     MinGruNames, NoPositionEncoding, OutputHead, ParallelMixer, PostNormBlock, RampScaling, RotaryEncoding,
                     TokenEmbedding)
from .decoder import DecoderModel
from .sogodra_config import ARCHITECTURE, DELTA_TYPE, MINGRU_TYPE, SogodraConfig


def build_sogodra(config: SogodraConfig) -> DecoderModel:
    try:
        return _build(config)
    except ValueError as error:
        if isinstance(error, ConfigError):
            raise
        raise ConfigError(ARCHITECTURE, str(error)) from None


def _delta(width: int, m, eps: float, p: str, channels: bool) -> GatedDeltaRule:
    names = dict(q=p + "q", k=p + "k", v=p + "v", q_conv=p + "q.conv", k_conv=p + "k.conv", v_conv=p + "v.conv", beta=p + "b",
                 a_log=p + "A_log", dt_bias=p + "dt_bias", norm=p + "norm", o=p + "o")
    if channels:
        names.update(decay_down=p + "a1", decay_up=p + "a2", gate_down=p + "g1", gate_up=p + "g2")
    else:
        names.update(decay=p + "a", gate=p + "g")
    return GatedDeltaRule(width, m.heads, m.kv_heads, m.dim, m.vdim, m.conv, eps, DeltaNames(**names), channel_decay=channels,
                          gate="sigmoid_low_rank" if channels else "silu")


def _build(config: SogodraConfig) -> DecoderModel:
    width, eps = config.width, config.norm_eps
    rotations = {}          # layers with the same rotation share one table of frequencies

    def rotation(spec, head_dim: int):
        if spec is None:
            return NoPositionEncoding()
        if (head_dim, spec) not in rotations:
            scaling = RampScaling(*spec.scaling) if spec.scaling else None
            rotations[head_dim, spec] = RotaryEncoding(head_dim, spec.base, rotary_dim=spec.dims, scaling=scaling)
        return rotations[head_dim, spec]
    layers = []
    for index, spec in enumerate(config.layers):
        p, m = f"l{index}.", spec.mixer
        if spec.kind == DELTA_TYPE:
            mixer = _delta(width, m, eps, p + "mix.", False)
        elif spec.kind == MINGRU_TYPE:
            mixer = MinGru(width, m.width, MinGruNames(z=p + "mix.z", z_bias=p + "mix.z.b", x=p + "mix.x", x_bias=p + "mix.x.b",
                                                       gate=p + "mix.g", o=p + "mix.o"))
        else:
            left, at = m.left, p + "mix.left."
            attention = GroupedQueryAttention(
                width, left.heads, left.kv_heads, left.dim, left.scale, rotation(left.rot, left.dim),
                AttentionNames(q=at + "q", k=at + "k", v=at + "v", o=at + "o", q_norm=at + "q.norm", k_norm=at + "k.norm",
                               sink=at + "sink"),
                qk_norm_eps=eps, window=left.window, value_dim=left.vdim)
            mixer = ParallelMixer(attention, _delta(width, m.right, eps, p + "mix.right.", True), m.left_scale, m.right_scale)
        norm_1 = GroupedRmsNorm(width, eps, p + "norm1")
        if spec.mlp is None:
            layers.append(PostNormBlock(mixer, norm_1))
            continue
        feed_forward = GatedMlp(width, spec.mlp.ff, "swiglu_clamp",
                                GatedMlpNames(gate=p + "mlp.gate", up=p + "mlp.up", down=p + "mlp.down"),
                                activation_param=spec.mlp.limit)
        layers.append(PostNormBlock(mixer, norm_1, feed_forward, GroupedRmsNorm(width, eps, p + "norm2")))
    # a layer without a feed-forward has no second norm; checkpoints may carry one all the same
    ignored = [f"l{i}.norm2" for i, spec in enumerate(config.layers) if spec.mlp is None]
    return DecoderModel(TokenEmbedding(config.vocab, width, "embed"), layers, GroupedRmsNorm(width, eps, "final.norm"),
                        OutputHead(config.vocab, width, "head"), vocab_size=config.vocab, max_positions=config.max_positions,
                        eos_token_ids=config.eos_token_ids, ignored_tensors=ignored)


register_architecture(ARCHITECTURE, SogodraConfig.from_raw, build_sogodra, replace=True)
