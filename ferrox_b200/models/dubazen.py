"""Dubazen as a description made of parts.

A decoder whose residual is several streams: before each sublayer the streams are summed with weights of the layer's own
and RMS-normed with one number as weight; its result goes back into every stream, which are mixed at the same time; the
embedding rows are multiplied by a constant and start every stream, and the streams' sum is what the head reads.

* ``parallel``: attention beside lightning attention, summed with constants.  Attention: grouped query heads, keys and
  values of different widths, biases on q, k, v and the output; the first ``rot.dims`` elements of every query and key
  head rotated on pairs (i, i + dims/2), then each head divided by its root mean square; values rotated over their whole
  width before they are cached and a head's result rotated back; a learned number per head in the softmax's denominator;
  an output gate.  Lightning attention: one fixed decay per head on SiLU(q, k, v), the read-outs normed together and gated.
* ``gla``: linear attention with a decay per key channel that depends on the token.
* ``mamba1``: a selective state space behind a short causal convolution.
* feed-forward: experts down(min(g, l) sigmoid(1.702 min(g, l)) (clamp(u, -l, l) + 1)) with g, u their gate and up
  products and l a limit, chosen by the largest softmax scores, weighted by those divided by their sum; a shared expert of
  the same form, with a limit of its own, is added for every token.

Tensor names: ``embed``, ``l<i>.{norm1,norm2}``, ``l<i>.hc{1,2}.{in,out,mix}``, ``l<i>.mix.*`` (``parallel``:
``l<i>.mix.{left,right}.*``), ``l<i>.mlp.{router, e<k>.{gate,up,down}, shared.{gate,up,down}}``, ``final.norm``, ``head``.
"""
from __future__ import annotations

from ..config.dubazen import ARCHITECTURE, DubazenConfig, GlaConfig, MambaConfig, ParallelConfig
from ..config.registry import register_architecture
from ..parts.specs import (
    AttentionSpec,
    DecayedLinearAttentionSpec,
    GatedLinearAttentionSpec,
    HyperBlockSpec,
    MixerSumSpec,
    ModelSpec,
    MoeSpec,
    NormSpec,
    ScaledRotarySpec,
    ScheduleEntry,
    SelectiveScanSpec,
    StreamNormSpec,
)

GATE_ALPHA = 1.702          # an expert's gate passes through g * sigmoid(GATE_ALPHA * g)
RENORM_EPS = 1e-20          # added to the sum of the chosen experts' scores before they are divided by it
DEFAULT_DECAY_RANK = 16     # inner width of a gla layer's decay, where neither a checkpoint nor the configuration says it


def _mixer(cfg: DubazenConfig, m, prefix: str, shapes):
    W, eps = cfg.width, cfg.norm_eps
    if isinstance(m, ParallelConfig):
        a, r = m.left, m.right
        left = AttentionSpec(
            hidden=W, n_heads=a.heads, n_kv_heads=a.kv_heads, head_dim=a.dim, value_dim=a.vdim, qkv_bias=True,
            position=ScaledRotarySpec(a.rot_dims, a.rot_base) if a.rot_dims else None, window=None,
            prefix=prefix + "left.", softmax_scale=a.scale,
            tensor_names=(("q", "q"), ("k", "k"), ("v", "v"), ("o", "o"), ("q_bias", "q.b"), ("k_bias", "k.b"),
                          ("v_bias", "v.b"), ("o_bias", "o.b")),
            output_gate="g", sink="sink", rotated_norm_eps=eps, value_turn=(a.rot_base, "halves"), o_bias=True)
        right = DecayedLinearAttentionSpec(hidden=W, n_heads=r.heads, head_dim=r.dim, value_dim=r.vdim, decay=r.decay,
                                           norm_eps=eps, prefix=prefix + "right.")
        return MixerSumSpec(mixers=(left, right), scales=(m.left_scale, m.right_scale))
    if isinstance(m, GlaConfig):
        rank = m.decay_rank or DEFAULT_DECAY_RANK
        if shapes is not None and prefix + "a1" in shapes:
            rank = int(shapes[prefix + "a1"][0])
        return GatedLinearAttentionSpec(hidden=W, n_heads=m.heads, head_dim=m.dim, value_dim=m.vdim, decay_rank=rank,
                                        tau=m.tau, norm_eps=eps, prefix=prefix)
    assert isinstance(m, MambaConfig)
    return SelectiveScanSpec(hidden=W, inner=m.inner, n_state=m.state, dt_rank=m.dt_rank, conv_taps=m.conv, prefix=prefix)


def _ffn(cfg: DubazenConfig, f, prefix: str):
    if f is None:
        return None
    return MoeSpec(
        hidden=cfg.width, n_experts=f.experts, top_k=f.top, expert_intermediate=f.ff, shared_intermediate=f.shared_ff,
        norm_topk_prob=True, shared_gate=False, prefix=prefix, activation=("clamped_swish", f.limit, GATE_ALPHA),
        shared_activation=("clamped_swish", f.shared_limit, GATE_ALPHA) if f.shared_ff else None,
        tensor_names=("router", "e{e}.{part}", "shared.{part}"), renorm_eps=RENORM_EPS)


def model_spec(cfg: DubazenConfig, tensor_shapes=None) -> ModelSpec:
    """``tensor_shapes`` (name -> shape, optional): the checkpoint's, for the one size that ``config.json`` may leave to
    them (the inner width of a gla layer's decay, the rows of ``l<i>.mix.a1``)."""
    W, S = cfg.width, cfg.streams
    blocks = []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."

        def norm(q):
            return StreamNormSpec(NormSpec(W, cfg.norm_eps, p, name=f"{p}norm{q}", scalar=True), S, f"{p}hc{q}.in")

        has_ffn = layer.mlp is not None
        blocks.append(HyperBlockSpec(
            norm1=norm(1),
            mixer=_mixer(cfg, layer.mixer, p + "mix.", tensor_shapes),
            norm2=norm(2) if has_ffn else None,
            ffn=_ffn(cfg, layer.mlp, p + "mlp."),
            streams=S,
            connections=tuple((f"{p}hc{q}.mix", f"{p}hc{q}.out") for q in ((1, 2) if has_ffn else (1,))),
            unused_tensors=() if has_ffn else ((p + "norm2", ()), (p + "hc2.in", (S,)), (p + "hc2.out", (S,)),
                                               (p + "hc2.mix", (S, S))),
        ))
    return ModelSpec(
        architecture=ARCHITECTURE,
        vocab_size=cfg.vocab,
        hidden=W,
        max_positions=cfg.max_positions,
        layers=tuple(blocks),
        schedule=tuple(ScheduleEntry(layer=i, cache=i) for i in range(len(blocks))),
        final_norm=StreamNormSpec(NormSpec(W, cfg.norm_eps, "final.", name="final.norm", scalar=True), S),
        embedding_name="embed",
        head_name="head",
        embedding_scale=cfg.embedding_scale,
        streams=S,
    )


register_architecture(ARCHITECTURE, DubazenConfig.from_json, model_spec, replace=True, reads_shapes=True)
