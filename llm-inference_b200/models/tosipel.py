"""Tosipel as a recipe of parts.

``x = table[token] * scale``; each layer is ``x += norm1(mixer(x)); x += norm2(ff(x))`` over a 32-bit stream that the sublayers read
directly, with norms whose weights are stored around zero. The mixer is one of three: attention in a sliding window with one
norm over all of q and one over all of k, rotation, a sink and a gate per head; attention over cached latents, without positions,
whose queries come out of a latent of their own; a gated delta rule with one decay per head. The feed-forward is a gated unit
(tanh gelu) or absent. A layer may run another layer's tensors against a cache or state of its own. A last norm, then an
untied head. Every size, constant and the order of the layers come from the configuration.
"""

from __future__ import annotations

from ..config.registry import register_architecture
from ..config.tosipel_config import TosipelConfig
from ..parts.base import PartSpec
from ..parts.model import LayerCall, ModelRecipe


def tosipel_mixer(kind: str, sizes: dict, prefix: str, hidden: int, eps: float) -> PartSpec:
    """The mixer of one layer."""
    common = dict(prefix=prefix, hidden_size=hidden, heads=sizes["heads"], dim=sizes["dim"], vdim=sizes["vdim"], eps=eps)
    if kind == "delta":
        return PartSpec("head_delta", dict(common, kv_heads=sizes["kv_heads"], taps=sizes["conv"]))
    if kind == "latent_attention":
        return PartSpec("latent_attention", dict(common, rot_dim=0, rank=sizes["kv_rank"], q_rank=sizes["q_rank"], scale=sizes["scale"], sink=False, gate=False))
    rot = sizes.get("rot")
    position = PartSpec("rotary", dict(head_dim=sizes["dim"], theta=rot["base"], rotary_dims=rot["dims"])) if rot and rot["dims"] else None
    return PartSpec(
        "shaped_attention",
        dict(common, kv_heads=sizes["kv_heads"], scale=sizes["scale"], qk_norm=True, position=position, window=(sizes.get("mask") or {}).get("size", 0),
             sink=True, gate="head"),
    )


def tosipel_recipe(config: TosipelConfig) -> ModelRecipe:
    hidden, eps = config.hidden_size, config.norm_eps

    def norm(name: str) -> PartSpec:
        return PartSpec("grouped_rmsnorm", dict(name=name, hidden_size=hidden, groups=1, eps=eps, around_zero=True))

    layers: list[PartSpec] = []
    block_of: dict[int, int] = {}  # layer that owns tensors -> its place among the blocks
    for index, layer in enumerate(config.layers):
        if config.owner(index) != index:
            continue
        prefix, mlp = f"l{index}.", layer.get("mlp")
        feed_forward = PartSpec("geglu", dict(prefix=prefix + "mlp.", hidden_size=hidden, intermediate_size=mlp["ff"])) if mlp is not None else None
        block_of[index] = len(layers)
        layers.append(
            PartSpec(
                "post_norm_residual",
                dict(
                    mixer=tosipel_mixer(layer["type"], layer["mixer"], prefix + "mix.", hidden, eps), feed_forward=feed_forward,
                    mixer_norm=norm(prefix + "norm1"), feed_forward_norm=norm(prefix + "norm2") if mlp is not None else None, hidden_size=hidden,
                    unused=() if mlp is not None else (prefix + "norm2",),
                ),
            )
        )
    # Every layer of the configuration is one call; a layer that names another's tensors runs that block
    # against the cache entry with its own number.
    return ModelRecipe(
        config=config,
        embedding=PartSpec(
            "token_embedding",
            dict(name="embed", suffix="", vocab_size=config.vocab_size, hidden_size=hidden, scale=config.embedding_scale, cast=True),
        ),
        layers=layers,
        final_norm=norm("final.norm"),
        head=PartSpec("linear_head", dict(name="head", suffix="", vocab_size=config.vocab_size, hidden_size=hidden)),
        schedule=[LayerCall(block_of[config.owner(index)], cache=index) for index in range(len(config.layers))],
    )


register_architecture(TosipelConfig.ARCHITECTURE, TosipelConfig.from_json_dict, tosipel_recipe, model_types=(TosipelConfig.MODEL_TYPE,))
