"""Sagizen as a description in parts.

Layers in the order the configuration lists them.  A layer is a mixer and
(unless it has none) a feed-forward, each with a norm on its OUTPUT only
(arrangement "postnorm"): x <- x + norm1(mixer(h)), x <- x + norm2(ff(x)).
The mixer's input h is the stream mixed with the previous token's, element
by element ("token_shift"): h = x + (x' - x) shift.

Mixers: "mamba2" (scalar decay per token and head, B and C shared by groups
of heads, the gate before a norm in equal parts), and "parallel", two mixers
that read the same h, their outputs times a constant each and added: on the
left grouped-query attention ("gqa_attention") with biases on q, k and v,
half-layout rotation of part of each head with linearly scaled frequencies,
q and k divided by their root mean square, and a sliding window beside which
blocks of tokens that lie wholly before it are seen as the means of their
keys and values; on the right RWKV-style time mixing ("rwkv").

The feed-forward is down(silu(gate x) * up x).  Final norm, then a head of
its own.

Tensor names: ``embed``, ``l<i>.shift``, ``l<i>.norm1``, ``l<i>.norm2``,
``l<i>.mix.*`` (``.left.*`` and ``.right.*`` in a parallel mixer),
``l<i>.mlp.gate|up|down``, ``final.norm``, ``head``.
"""
from __future__ import annotations

from ..config.registry import Architecture, register_architecture
from ..config.sagizen import SagizenConfig
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, SubLayer


def _mixer_spec(c: SagizenConfig, L) -> PartSpec:
    W, m = c.width, L.mixer
    if L.type == "mamba2":
        return PartSpec("mamba2", dict(hidden_size=W, num_heads=m.heads, v_dim=m.vdim, state=m.state, groups=m.groups,
                                       taps=m.conv, norm_groups=m.norm_groups, eps=c.norm_eps))
    a, s = m.left, m.right
    left = PartSpec("gqa_attention", dict(
        hidden_size=W, num_heads=a.heads, num_kv_heads=a.kv_heads, head_dim=a.dim, v_dim=a.vdim, scale=a.scale,
        rot_dims=a.rot_dims, rot_base=a.rot_base, rot_factor=a.rot_factor, rot_layout="half", eps=c.norm_eps,
        window=a.size, pool=a.pool, bias="qkv", bias_in="rows", qk_norm="unit", head_temp=False, base="mix.left."))
    right = PartSpec("rwkv", dict(hidden_size=W, num_heads=s.heads, head_dim=s.dim, eps=c.norm_eps, base="mix.right."))
    return PartSpec("parallel", dict(branches=((left, m.left_scale), (right, m.right_scale))))


def sagizen_model_spec(c: SagizenConfig) -> ModelSpec:
    W = c.width
    none = PartSpec("identity", {})

    def norm(name):
        return PartSpec("rmsnorm", dict(size=W, eps=c.norm_eps, name=name))

    layers = []
    for i, L in enumerate(c.layers):
        shifted = PartSpec("token_shift", dict(hidden_size=W, name="shift", inner=_mixer_spec(c, L)))
        subs = [SubLayer(none, shifted, "mixer", post_norm=norm("norm1"))]
        if L.ff:
            ffn = PartSpec("swiglu", dict(hidden_size=W, intermediate_size=L.ff, activation="silu",
                                          names=("mlp.gate", "mlp.up", "mlp.down")))
            subs.append(SubLayer(none, ffn, "ffn", post_norm=norm("norm2")))
        layers.append(LayerSpec(prefix=f"l{i}.", sublayers=tuple(subs), arrangement="postnorm"))
    return ModelSpec(
        hidden_size=W, vocab_size=c.vocab, max_position=c.max_position,
        embedding=PartSpec("token_embedding", dict(vocab_size=c.vocab, hidden_size=W, name="embed")),
        layers=tuple(layers),
        final_norm=norm("final.norm"),
        head=PartSpec("lm_head", dict(vocab_size=c.vocab, hidden_size=W, name="head")),
    )


SAGIZEN = register_architecture(Architecture(
    name="Sagizen",
    config_from_dict=SagizenConfig.from_dict,
    model_spec=sagizen_model_spec,
    # a layer without a feed-forward has no use for its second norm
    allow_unexpected=lambda c: tuple(f"l{i}.norm2" for i, L in enumerate(c.layers) if not L.ff),
    description="norms on the sublayers' outputs only, a token shift in front of every mixer; Mamba-2, or windowed "
                "attention with pooled blocks beside RWKV-style time mixing; dense feed-forward",
    family="Sagizen",
), replace=True)
