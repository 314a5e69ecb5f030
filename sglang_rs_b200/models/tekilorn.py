"""Tekilorn put together from the parts.

A pre-norm decoder (``parts.PreNormBlock``; a layer may end after its mixer) whose mixer is

* ``attention`` (``parts.GroupedQueryAttention(maps=)``): differential attention, two maps per head over the same values whose
  results are subtracted and normed, no rotation, a query temperature that grows with the position, a cap on the scores, every
  key up to the row's own; or
* ``attention_2`` (``parts.GroupedQueryAttention``): grouped heads, the leading entries of every head rotated in interleaved
  pairs, a sliding window that keeps the sequence's first tokens, a sigmoid gate per head on the result.

The feed-forward is a clamped gated one (``parts.GatedMlp``) or routed experts of that form (``parts.RoutedExperts``): sigmoid
scores, the chosen scores as they are on the experts' inputs, a shared expert behind a sigmoid gate per token.  A stretch of
layers may be walked several times with the same weights, each pass with caches of its own; every pass, also the first, is
opened by adding the pass's own vector to the stream (``parts.PassStep``).  The norms are RMS norms with a plain weight
(``parts.GroupedRmsNorm``: its kernel takes the 32-bit sums of the experts, partial sums of few-row products and the passes'
vectors) and the head is a matrix of its own.

Checkpoint names: ``embed``, ``head``, ``final.norm``, ``loop.step`` and per layer ``l<i>.norm1`` / ``norm2``,
``l<i>.mix.{q, k, v, o}`` with ``l<i>.mix.{lq1, lk1, lq2, lk2}`` or ``l<i>.mix.g``, ``l<i>.mlp.{gate, up, down}`` or
``l<i>.mlp.router``, ``l<i>.mlp.e<j>.{gate, up, down}``, ``l<i>.mlp.shared.{gate, up, down, sg}``.
Fixed by the design, not by config.json: the activation, unnormalised router weights on the inputs, the pairing of the
rotation, the layout of the maps.
"""
from __future__ import annotations

from ..config.model_config import ConfigError
from ..config.registry import register_architecture
from ..parts import (AttentionNames, DifferentialMaps, GatedMlp, GatedMlpNames, GroupedQueryAttention, GroupedRmsNorm,
                     NoPositionEncoding, OutputHead, PassStep, PreNormBlock, RotaryEncoding, RoutedExperts, TokenEmbedding)
from .decoder import DecoderModel, LayerCall
from .tekilorn_config import ARCHITECTURE, DIFFERENTIAL_TYPE, ClampedSizes, TekilornConfig

#: min(g, limit) sigmoid(1.702 min(g, limit)) (clamp(u, -limit, limit) + 1)
ACTIVATION = "swiglu_clamp"


def layer_program(config: TekilornConfig):
    """The layer calls of one forward pass: the layers ahead of the stretch, the stretch ``times`` times (the first call of
    every walk opens the pass), the layers behind it."""
    count, loop = len(config.layers), config.loop
    if loop is None:
        return [LayerCall(i) for i in range(count)]
    calls = [LayerCall(i) for i in range(loop.start)]
    for t in range(loop.times):
        calls += [LayerCall(i, entry=0 if i == loop.start else None, pass_index=t) for i in range(loop.start, loop.stop)]
    return calls + [LayerCall(i) for i in range(loop.stop, count)]


def build_tekilorn(config: TekilornConfig) -> DecoderModel:
    try:
        return _build(config)
    except ValueError as error:
        if isinstance(error, ConfigError):
            raise
        raise ConfigError(ARCHITECTURE, str(error)) from None


def _build(config: TekilornConfig) -> DecoderModel:
    width, eps = config.width, config.norm_eps
    rotations = {}          # layers with the same rotation share one table of frequencies

    def rotation(spec, head_dim: int):
        if spec is None:
            return NoPositionEncoding()
        key = (head_dim, spec)
        if key not in rotations:
            rotations[key] = RotaryEncoding(head_dim, spec.base, rotary_dim=spec.dims, interleaved=True)
        return rotations[key]

    def clamped(sizes: ClampedSizes, prefix: str, float_result: bool = False) -> GatedMlp:
        return GatedMlp(width, sizes.ff, ACTIVATION, GatedMlpNames(gate=prefix + "gate", up=prefix + "up", down=prefix + "down"),
                        float_result=float_result, activation_param=sizes.limit)
    layers = []
    for index, spec in enumerate(config.layers):
        p, m = f"l{index}.", spec.mixer
        names = dict(q=p + "mix.q", k=p + "mix.k", v=p + "mix.v", o=p + "mix.o")
        if spec.kind == DIFFERENTIAL_TYPE:
            maps = DifferentialMaps(m.diff, eps, *(p + "mix." + name for name in ("lq1", "lk1", "lq2", "lk2")))
            mixer = GroupedQueryAttention(width, m.heads, m.kv_heads, 2 * m.dim, m.scale, NoPositionEncoding(),
                                          AttentionNames(**names), value_dim=m.vdim, softcap=m.softcap,
                                          temperature=m.temperature, maps=maps)
        else:
            mixer = GroupedQueryAttention(width, m.heads, m.kv_heads, m.dim, m.scale, rotation(m.rot, m.dim),
                                          AttentionNames(gate=p + "mix.g", **names), value_dim=m.vdim, window=m.window,
                                          keep_first=m.keep_first)
        f, norm_1 = spec.mlp, GroupedRmsNorm(width, eps, p + "norm1")
        if f is None:
            layers.append(PreNormBlock(norm_1, mixer))
            continue
        if isinstance(f, ClampedSizes):
            feed_forward = clamped(f, p + "mlp.")
        else:
            shared = clamped(f.shared, p + "mlp.shared.", float_result=True) if f.shared is not None else None
            feed_forward = RoutedExperts(
                width, f.expert.ff, f.experts, f.top, ACTIVATION, p + "mlp.router",
                lambda e, p=p: GatedMlpNames(gate=f"{p}mlp.e{e}.gate", up=f"{p}mlp.e{e}.up", down=f"{p}mlp.e{e}.down"),
                scoring="sigmoid", activation_param=f.expert.limit, weigh_inputs=True, shared=shared,
                shared_gate_name=p + "mlp.shared.sg" if shared is not None else None)
        layers.append(PreNormBlock(norm_1, mixer, GroupedRmsNorm(width, eps, p + "norm2"), feed_forward))
    entries = [PassStep(width, config.loop.times, "loop.step")] if config.loop is not None else []
    # a layer without a feed-forward has no second norm; checkpoints may carry it all the same
    ignored = [f"l{i}.norm2" for i, spec in enumerate(config.layers) if spec.mlp is None]
    return DecoderModel(TokenEmbedding(config.vocab, width, "embed"), layers, GroupedRmsNorm(width, eps, "final.norm"),
                        OutputHead(config.vocab, width, "head"), vocab_size=config.vocab, max_positions=config.max_positions,
                        eos_token_ids=config.eos_token_ids, program=layer_program(config), pass_entries=entries,
                        ignored_tensors=ignored)


register_architecture(ARCHITECTURE, TekilornConfig.from_raw, build_tekilorn, replace=True)
