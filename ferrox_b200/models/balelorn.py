"""Balelorn as a description made of parts.

A decoder of attention layers with a norm before and after each sublayer and a scale per channel on what is added; the
embedding rows are RMS-normed:

    h += ls1 * norm1b(mixer(norm1(h)));   h += ls2 * norm2b(ffn(norm2(h)))      norm: z / sqrt(mean(z^2) + eps) * w

* attention: grouped query heads, keys and values of different widths; the first ``rot.dims`` elements of every query
  and key head rotated on pairs (i, i + dims/2); a query sees the keys of its own chunk of positions only; a learned
  number per head in the softmax's denominator; from the second layer that mixes its values on, what is cached is
  (1 - lambda) v + lambda v_first with the first such layer's values of the same token; the concatenated heads are
  multiplied by sigmoid(g x) before the output projection.
* feed-forward: gated with the tanh form of GELU, or experts without a router: a table names each token id's experts,
  all with the same weight; an expert is down(min(g, l) sigmoid(1.702 min(g, l)) (clamp(u, -l, l) + 1)) with g, u its
  gate and up products and l its limit.

Tensor names: ``embed``, ``embed.norm``, ``l<i>.{norm1,norm1b,ls1,norm2,norm2b,ls2}``, ``l<i>.mix.{q,k,v,g,o,sink,
vmix}``, ``l<i>.mlp.{gate,up,down}`` or ``l<i>.mlp.{table, e<k>.{gate,up,down}}``, ``final.norm``, ``head``.
"""
from __future__ import annotations

from ..config.balelorn import ARCHITECTURE, AttentionConfig, BalelornConfig, DenseConfig
from ..config.registry import register_architecture
from ..parts.specs import (
    AttentionSpec,
    DenseMlpSpec,
    ModelSpec,
    MoeSpec,
    NormSpec,
    SandwichBlockSpec,
    ScaledRotarySpec,
    ScheduleEntry,
    ValueMixSpec,
)

GATE_ALPHA = 1.702          # the experts' gate passes through g * sigmoid(GATE_ALPHA * g)


def _mixer(cfg: BalelornConfig, m: AttentionConfig, prefix: str, first_of_mix: bool):
    return AttentionSpec(
        hidden=cfg.width, n_heads=m.heads, n_kv_heads=m.kv_heads, head_dim=m.dim, value_dim=m.vdim, qkv_bias=False,
        position=ScaledRotarySpec(m.rot.dims, m.rot.base) if m.rot is not None else None, window=None, prefix=prefix,
        softmax_scale=m.scale, tensor_names=(("q", "q"), ("k", "k"), ("v", "v"), ("o", "o")), output_gate="g",
        chunk=m.chunk, sink="sink", value_mix=ValueMixSpec("vmix", source=first_of_mix) if m.v_mix else None,
    )


def _ffn(cfg: BalelornConfig, f, prefix: str):
    if isinstance(f, DenseConfig):
        return DenseMlpSpec(hidden=cfg.width, intermediate=f.ff, prefix=prefix, activation="gelu_tanh",
                            tensor_names=("gate", "up", "down"))
    return MoeSpec(
        hidden=cfg.width, n_experts=f.experts, top_k=f.top, expert_intermediate=f.ff, shared_intermediate=0,
        norm_topk_prob=False, shared_gate=False, prefix=prefix, activation=("clamped_swish", f.limit, GATE_ALPHA),
        tensor_names=("", "e{e}.{part}", ""), table="table", vocab=cfg.vocab,
    )


def model_spec(cfg: BalelornConfig) -> ModelSpec:
    W, eps = cfg.width, cfg.norm_eps
    blocks = []
    first_mix = next((i for i, layer in enumerate(cfg.layers) if layer.mixer.v_mix), None)
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        has_ffn = layer.mlp is not None

        def norm(name, scale=None):
            return NormSpec(W, eps, p, name=p + name, scale_name=p + scale if scale else None)

        blocks.append(SandwichBlockSpec(
            norm1=norm("norm1"),
            mixer=_mixer(cfg, layer.mixer, p + "mix.", i == first_mix),
            post1=norm("norm1b", "ls1"),
            norm2=norm("norm2") if has_ffn else None,
            ffn=_ffn(cfg, layer.mlp, p + "mlp.") if has_ffn else None,
            post2=norm("norm2b", "ls2") if has_ffn else None,
            unused_tensors=() if has_ffn else tuple((p + n, (W,)) for n in ("norm2", "norm2b", "ls2")),
        ))
    return ModelSpec(
        architecture=ARCHITECTURE,
        vocab_size=cfg.vocab,
        hidden=W,
        max_positions=cfg.max_positions,
        layers=tuple(blocks),
        schedule=tuple(ScheduleEntry(layer=i, cache=i) for i in range(len(blocks))),
        final_norm=NormSpec(W, eps, "final.", name="final.norm"),
        embedding_name="embed",
        embedding_norm=NormSpec(W, eps, "embed.", name="embed.norm"),
        head_name="head",
    )


register_architecture(ARCHITECTURE, BalelornConfig.from_json, model_spec, replace=True)
