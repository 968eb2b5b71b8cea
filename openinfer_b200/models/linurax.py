"""Linurax: how a ``LinuraxConfig`` becomes a ``ModelSpec``.

Every layer is a "branchnorm" block on a float32 stream: x <- x + rms(mixer(x); norm1), then, where the layer has a
feed-forward, x <- x + rms(ff(x); norm2); the sublayers read the stream itself. The embedding is scaled going in; going out
the logits are the final norm's rows times the (unscaled) embedding table. Layer types: "attention" (weights sigmoid(score +
bias) that are not normalised over the keys, scores mixed between the heads, keys that serve as values before their norm and
rotation, a norm over all heads together, a gate per output number) and "mingru" (a gated recurrence per channel). The
feed-forward is a gated one with SiLU. Tensor names: ``embed``, ``final.norm`` and per layer ``l<i>.`` + ``norm1``, ``norm2``,
``mix.{q,k,q.norm,k.norm,talk,pb,g,o}`` or ``mix.{z,z.b,x,x.b,g,o}``, ``mlp.{gate,up,down}``.
"""
from __future__ import annotations

from ..config.base import register_architecture
from ..config.linurax import LinuraxConfig
from ..parts.spec import BlockSpec, GatedMlpSpec, MinGruSpec, ModelSpec, NormSpec, PositionSpec, SigmoidAttentionSpec


def _mixer(cfg: LinuraxConfig, layer: dict, eps: float):
    m = layer["mixer"]
    if layer["type"] == "mingru":
        return MinGruSpec(hidden_size=cfg.width, channels=int(m["width"]))
    rot = m.get("rot")
    position = PositionSpec(kind="none") if rot is None else PositionSpec(
        kind="rope", rotary_dim=int(rot["dims"]), theta=float(rot["base"]), max_positions=cfg.max_position_embeddings,
        interleaved=True, precise=True)
    return SigmoidAttentionSpec(
        hidden_size=cfg.width, num_heads=int(m["heads"]), num_kv_heads=int(m["kv_heads"]), qk_dim=int(m["dim"]),
        v_dim=int(m["vdim"]), score_scale=float(m["scale"]), position=position, joint_norm_eps=eps, values_from_keys=True,
        mix_heads=True, score_bias=True, output_gate=True)


def build_spec(cfg: LinuraxConfig) -> ModelSpec:
    eps = float(cfg.norm["eps"])
    W = cfg.width
    norm = NormSpec(kind="rms", size=W, eps=eps, param_name="")
    blocks = []
    for i, layer in enumerate(cfg.layers):
        mlp = layer.get("mlp")
        ff = GatedMlpSpec(hidden_size=W, intermediate_size=int(mlp["ff"]), activation="silu", gate_name="gate", up_name="up",
                          down_name="down") if mlp else None
        blocks.append(BlockSpec(
            kind="branchnorm", name=f"l{i}.", mixer=_mixer(cfg, layer, eps), feed_forward=ff, input_norm=norm,
            post_norm=norm if ff is not None else None, mixer_name="mix.", feed_forward_name="mlp.",
            input_norm_name="norm1", post_norm_name="norm2"))
    return ModelSpec(
        vocab_size=cfg.vocab, hidden_size=W, blocks=tuple(blocks), order=tuple(range(len(blocks))), final_norm=norm,
        embedding_name="embed", final_norm_name="final.norm", head_name=None, max_positions=cfg.max_position_embeddings,
        stop_token_ids=tuple(cfg.stop_token_ids), embedding_scale=float(cfg.embedding["scale"]), residual_dtype="float32")


register_architecture(LinuraxConfig.architecture, LinuraxConfig, build_spec)
