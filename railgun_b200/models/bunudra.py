"""Bunudra as a description in parts.

Layers in the order the configuration lists them.  A layer is a mixer and
(unless it has none) a feed-forward, each with a layer norm on its OUTPUT
only (arrangement "postnorm"): every part reads the 32-bit stream and adds the
normed result to it.

Mixers: "attention", grouped-query attention ("gqa_attention") with an RMS
norm per head on q and k and half-layout rotation, in which a query sees its
own chunk of positions only; "latent_attention" with an interleaved rotation
by YaRN's frequencies, a sliding window and a sigmoid gate on the heads'
outputs; "mlstm", the matrix memory of xLSTM.

The feed-forward is a mixture of experts without gates (exact gelu): a
softmax router, a choice limited to the experts of the best groups, weights
that are the scores times a constant, and a shared expert behind a sigmoid
gate of one number per token.  The embedding is multiplied by a constant;
final layer norm, then a head of its own.

Tensor names: ``embed``, ``l<i>.norm1``, ``l<i>.norm1.b``, ``l<i>.norm2``,
``l<i>.norm2.b``, ``l<i>.mix.*``, ``l<i>.mlp.e<j>.up|down``,
``l<i>.mlp.router``, ``l<i>.mlp.shared.up|down|sg``, ``final.norm``,
``final.norm.b``, ``head``.
"""
from __future__ import annotations

from ..config.bunudra import BunudraConfig
from ..config.registry import Architecture, register_architecture
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, SubLayer


def _mixer_spec(c: BunudraConfig, L) -> PartSpec:
    W, m = c.width, L.mixer
    if L.type == "mlstm":
        return PartSpec("mlstm", dict(hidden_size=W, num_heads=m.heads, head_dim=m.dim, v_dim=m.vdim, gate_cap=m.gate_cap,
                                      eps=c.norm_eps))
    if L.type == "latent_attention":
        s = m.rot.scaling
        yarn = dict(factor=s.factor, original=s.original, fast=s.fast, slow=s.slow) if s else None
        return PartSpec("latent_attention", dict(
            hidden_size=W, num_heads=m.heads, head_dim=m.dim, rot_dim=m.rot_dim, v_dim=m.vdim, kv_rank=m.kv_rank,
            scale=m.scale, rot_dims=m.rot.dims, rot_base=m.rot.base, rot_layout="interleaved", yarn=yarn, eps=c.norm_eps,
            window=m.size, out_gate=True))
    return PartSpec("gqa_attention", dict(
        hidden_size=W, num_heads=m.heads, num_kv_heads=m.kv_heads, head_dim=m.dim, v_dim=m.vdim, scale=m.scale,
        rot_dims=m.rot.dims, rot_base=m.rot.base, rot_layout="half", eps=c.norm_eps, chunk=m.size, bias=False,
        qk_norm=True, head_temp=False))


def bunudra_model_spec(c: BunudraConfig) -> ModelSpec:
    W = c.width
    none = PartSpec("identity", {})

    def norm(name):
        return PartSpec("layernorm", dict(size=W, eps=c.norm_eps, name=name))

    layers = []
    for i, L in enumerate(c.layers):
        subs = [SubLayer(none, _mixer_spec(c, L), "mixer", post_norm=norm("norm1"))]
        if L.mlp is not None:
            e = L.mlp
            ffn = PartSpec("routed_experts", dict(
                hidden_size=W, experts=e.experts, identity=0, top=e.top, expert_size=e.expert_ff,
                shared_size=e.shared_ff or None, gated=False, activation="gelu", correction=False, renormalize=False,
                weight_scale=e.scale, groups=e.groups, shared_gate=bool(e.shared_ff)))
            subs.append(SubLayer(none, ffn, "ffn", post_norm=norm("norm2")))
        layers.append(LayerSpec(prefix=f"l{i}.", sublayers=tuple(subs), arrangement="postnorm"))
    return ModelSpec(
        hidden_size=W, vocab_size=c.vocab, max_position=c.max_position,
        embedding=PartSpec("token_embedding", dict(vocab_size=c.vocab, hidden_size=W, name="embed", scale=c.embedding_scale)),
        layers=tuple(layers),
        final_norm=norm("final.norm"),
        head=PartSpec("lm_head", dict(vocab_size=c.vocab, hidden_size=W, name="head")),
    )


BUNUDRA = register_architecture(Architecture(
    name="Bunudra",
    config_from_dict=BunudraConfig.from_dict,
    model_spec=bunudra_model_spec,
    # a layer without a feed-forward has no use for its second norm
    allow_unexpected=lambda c: tuple(f"l{i}.norm2{b}" for i, L in enumerate(c.layers) if L.mlp is None for b in ("", ".b")),
    description="layer norms on the sublayers' outputs only; attention in chunks, windowed latent attention or xLSTM's "
                "matrix memory; experts chosen from the best groups beside a gated shared expert",
    family="Bunudra",
), replace=True)
