"""Rolevik: how a ``RolevikConfig`` becomes a ``ModelSpec``.

Every layer is a "branchnorm" block on a float32 stream: x <- x + ls1 * ln(mixer(x); norm1), then, where the layer has a
feed-forward, x <- x + ls2 * ln(ff(x); norm2), with layer norms that have no bias and a weight per channel behind them; the
sublayers read the stream itself. Layer types: "parallel", softmax attention in chunks (biased projections, q and k normed over
all heads together, partial rotary positions, keys and values of their own sizes) beside a gated delta rule with one decay per
head, half the sum of the two results, each RMS-normed; and "rglru", a real-gated linear recurrent unit behind a short filter,
beside a GELU gate. The feed-forward is a gated one with GELU, or experts with SiLU, chosen by corrected softmax scores within
the best groups, some of the choices being the input itself, beside an expert every token uses. The embedding is scaled going in;
going out the logits are the final norm's rows times the (unscaled) embedding table, times a constant. Tensor names: ``embed``,
``final.norm`` and per layer ``l<i>.`` + ``norm1``, ``norm2``, ``ls1``, ``ls2``, ``mix.left.*``, ``mix.right.*`` or ``mix.*``, ``mlp.*``.
"""
from __future__ import annotations

from ..config.base import register_architecture
from ..config.rolevik import RolevikConfig
from ..parts.spec import (AttentionSpec, BlockSpec, GatedDeltaSpec, GatedMlpSpec, LayerScaleSpec, ModelSpec, NormSpec, ParallelMixerSpec,
                          PositionSpec, RgLruSpec, RoutedExpertsSpec)

DECAY_RATE = 8.0      # c of the recurrent unit's a = exp(-c r softplus(lambda))


def _pad8(n: int) -> int:
    return (n + 7) & ~7


def _mixer(cfg: RolevikConfig, layer: dict, eps: float):
    W, m = cfg.width, layer["mixer"]
    if layer["type"] == "rglru":
        return RgLruSpec(hidden_size=W, channels=int(m["width"]), blocks=int(m["blocks"]), conv_taps=int(m["conv"]), rate=DECAY_RATE)
    left, right = m["left"], m["right"]
    dim, vdim, rot, mask = int(left["dim"]), int(left["vdim"]), left.get("rot"), left.get("mask")
    position = PositionSpec(kind="none") if not rot else PositionSpec(
        kind="rope", rotary_dim=int(rot["dims"]), theta=float(rot["base"]), max_positions=cfg.max_position_embeddings, precise=True)
    attention = AttentionSpec(
        hidden_size=W, num_heads=int(left["heads"]), num_kv_heads=int(left["kv_heads"]), head_dim=_pad8(max(dim, vdim)),
        softmax_scale=float(left["scale"]), position=position, window=int(mask["size"]) if mask else None, chunked=bool(mask),
        qk_dim=dim, v_dim=vdim, q_name="q", k_name="k", v_name="v", o_name="o", q_norm_name="q.norm", k_norm_name="k.norm",
        qkv_bias=True, joint_norm_eps=eps)
    delta = GatedDeltaSpec(
        hidden_size=W, num_heads=int(right["heads"]), num_kv_heads=int(right["kv_heads"]), qk_dim=int(right["dim"]),
        v_dim=int(right["vdim"]), conv_taps=int(right["conv"]), eps=eps, decay_per="head", gate_activation="silu")
    return ParallelMixerSpec(left=attention, right=delta, left_scale=0.5, right_scale=0.5, out_norm_eps=eps)


def _feed_forward(cfg: RolevikConfig, mlp):
    if not mlp:
        return None

    def gated(ff: int, activation: str) -> GatedMlpSpec:
        return GatedMlpSpec(hidden_size=cfg.width, intermediate_size=ff, activation=activation, gate_name="gate", up_name="up", down_name="down")

    if mlp["kind"] == "dense":
        return gated(int(mlp["ff"]), "gelu_tanh")
    router = mlp["router"]
    groups = router.get("groups") or {"count": 1, "keep": 1}
    scale = router.get("scale")
    return RoutedExpertsSpec(
        hidden_size=cfg.width, intermediate_size=int(mlp["expert"]["ff"]), experts=int(router["experts"]), top=int(router["top"]),
        activation="silu", routing="softmax_groups", groups=int(groups["count"]), keep_groups=int(groups["keep"]),
        identity=int(router.get("identity") or 0), weight_scale=1.0 if scale is None else float(scale),
        shared=gated(int(mlp["shared"]["ff"]), "silu") if mlp.get("shared") else None)


def build_spec(cfg: RolevikConfig) -> ModelSpec:
    eps = float(cfg.norm["eps"])
    W = cfg.width
    norm, scale = NormSpec(kind="layer", size=W, eps=eps, param_name=""), LayerScaleSpec(size=W)
    blocks = []
    for i, layer in enumerate(cfg.layers):
        ff = _feed_forward(cfg, layer.get("mlp"))
        blocks.append(BlockSpec(
            kind="branchnorm", name=f"l{i}.", mixer=_mixer(cfg, layer, eps), feed_forward=ff, input_norm=norm,
            post_norm=norm if ff is not None else None, mixer_scale=scale, feed_forward_scale=scale if ff is not None else None,
            mixer_name="mix.", feed_forward_name="mlp.", input_norm_name="norm1", post_norm_name="norm2"))
    return ModelSpec(
        vocab_size=cfg.vocab, hidden_size=W, blocks=tuple(blocks), order=tuple(range(len(blocks))), final_norm=norm,
        embedding_name="embed", final_norm_name="final.norm", head_name=None, max_positions=cfg.max_position_embeddings,
        stop_token_ids=tuple(cfg.stop_token_ids), embedding_scale=float(cfg.embedding["scale"]), logit_scale=float(cfg.logit_scale),
        residual_dtype="float32")


register_architecture(RolevikConfig.architecture, RolevikConfig, build_spec)
