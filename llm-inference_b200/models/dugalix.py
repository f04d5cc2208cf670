"""Dugalix as a recipe of parts.

Each layer is ``x += m * norm1b(mixer(h)); x += m * norm2b(ff(norm2(x)))`` with norms whose weights are stored around zero and
``h`` the rows of ``norm1(x)`` blended with the previous token's (a factor per column). The mixer is one of two: softmax
attention with biases, rotation, a sliding window and kept first tokens beside a matrix memory (xLSTM's mLSTM), their
outputs added with a constant factor each; or attention whose values are its keys before rotation and whose weights are
sigmoids, in a sliding window. The feed-forward is a squared-relu unit, or a mixture of such units and of identity experts
(softmax scores over all, a correction for the choice, groups) with a gated shared expert, or absent. A last norm, then
an untied head. Every size, constant and the order of the layers come from the configuration.
"""

from __future__ import annotations

from ..config.dugalix_config import DugalixConfig
from ..config.registry import register_architecture
from ..parts.base import PartSpec
from ..parts.model import ModelRecipe


def _attention(sizes: dict, prefix: str, hidden: int, eps: float, **more) -> PartSpec:
    rot, mask = sizes.get("rot"), sizes.get("mask") or {}
    position = None
    if rot and rot["dims"]:
        position = PartSpec("rotary", dict(head_dim=sizes["dim"], theta=rot["base"], rotary_dims=rot["dims"],
                                           scaling=dict(factor=(rot.get("scaling") or {}).get("factor", 1.0))))
    return PartSpec(
        "shaped_attention",
        dict(
            prefix=prefix, hidden_size=hidden, heads=sizes["heads"], kv_heads=sizes["kv_heads"], dim=sizes["dim"], vdim=sizes["vdim"],
            scale=sizes["scale"], eps=eps, qk_norm=False, position=position, window=mask.get("size", 0), keep_first=mask.get("keep_first", 0), **more,
        ),
    )


def dugalix_mixer(kind: str, sizes: dict, prefix: str, hidden: int, eps: float) -> PartSpec:
    """The mixer of one layer."""
    if kind == "attention":
        return _attention(sizes, prefix, hidden, eps, values="keys", weights="sigmoid")
    right = sizes["right"]
    return PartSpec(
        "parallel_mixers",
        dict(
            first=_attention(sizes["left"], prefix + "left.", hidden, eps, qk_bias=True, v_bias=True, out_bias=True),
            second=PartSpec("matrix_memory", dict(prefix=prefix + "right.", hidden_size=hidden, heads=right["heads"], dim=right["dim"],
                                                  vdim=right["vdim"], gate_cap=right["gate_cap"], eps=eps)),
            hidden_size=hidden, scales=(sizes["left_scale"], sizes["right_scale"]),
        ),
    )


def dugalix_feed_forward(mlp: dict | None, prefix: str, hidden: int) -> PartSpec | None:
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return PartSpec("squared_relu", dict(prefix=prefix, hidden_size=hidden, intermediate_size=mlp["ff"]))
    router, shared = mlp["router"], mlp.get("shared")
    groups = router.get("groups") or {"count": 1, "keep": 1}
    return PartSpec(
        "routed_experts",
        dict(
            prefix=prefix, hidden_size=hidden, experts=router["experts"], top=router["top"], intermediate_size=mlp["expert"]["ff"], limit=0.0,
            group_count=groups["count"], group_keep=groups["keep"], router="softmax_all", router_bias=True, activation="squared_relu",
            identity=router.get("identity", 0), shared_size=shared["ff"] if shared else None, shared_gate=bool(shared),
        ),
    )


def dugalix_recipe(config: DugalixConfig) -> ModelRecipe:
    hidden, eps = config.hidden_size, config.norm_eps

    def norm(name: str) -> PartSpec:
        return PartSpec("grouped_rmsnorm", dict(name=name, hidden_size=hidden, groups=1, eps=eps, around_zero=True))

    layers = []
    for index, layer in enumerate(config.layers):
        prefix = f"l{index}."
        feed_forward = dugalix_feed_forward(layer.get("mlp"), prefix + "mlp.", hidden)
        second = feed_forward is not None
        layers.append(
            PartSpec(
                "sandwich_residual",
                dict(
                    mixer=dugalix_mixer(layer["type"], layer["mixer"], prefix + "mix.", hidden, eps), feed_forward=feed_forward,
                    mixer_norm=norm(prefix + "norm1"), mixer_out_norm=norm(prefix + "norm1b"),
                    feed_forward_norm=norm(prefix + "norm2") if second else None, feed_forward_out_norm=norm(prefix + "norm2b") if second else None,
                    hidden_size=hidden, mult=config.residual_mult, shift=prefix + "shift",
                    unused=() if second else (prefix + "norm2", prefix + "norm2b"),
                ),
            )
        )
    return ModelRecipe(
        config=config,
        embedding=PartSpec("token_embedding", dict(name="embed", suffix="", vocab_size=config.vocab_size, hidden_size=hidden)),
        layers=layers,
        final_norm=norm("final.norm"),
        head=PartSpec("linear_head", dict(name="head", suffix="", vocab_size=config.vocab_size, hidden_size=hidden)),
    )


register_architecture(DugalixConfig.ARCHITECTURE, DugalixConfig.from_json_dict, dugalix_recipe, model_types=(DugalixConfig.MODEL_TYPE,))
