"""Tidenex as a plan of parts.

Every layer is a pre-norm block (``pre_norm``) with layer norms that have weight and bias.  The mixer is attention by the difference
of two maps (``differential_attention``) or two mixers side by side (``side_by_side``): biased grouped-query attention whose q
and k are normed over the whole projection, with a temperature by position and a bias by distance instead of a rotation
(``masked_sink_attention``), and the HGRN2 recurrence (``hgrn2``).  The feed-forward is W_down gelu(W_up h) (``activation_mlp``) or
absent.  A range of layers may run several times in a row with the same weights: every pass has cache and state slots of its own, and
in front of every pass but the first the embedding output joins the stream again.  The embedding is also the output matrix.
Layer i's tensors are ``l<i>.*``; all numbers come from the configuration.
"""
from __future__ import annotations

from ..config.model_config import TidenexConfig
from ..config.registry import Architecture, register_architecture
from ..parts import BlockSpec, LayerCall, ModelPlan, PartSpec, SharedRef


def tidenex_plan(cfg: TidenexConfig) -> ModelPlan:
    W, eps = cfg.hidden_size, cfg.norm_eps

    def norm(name: str) -> PartSpec:
        return PartSpec("layernorm", {"size": W, "eps": eps, "param": name, "bias": name + ".b"})
    blocks, shared = [], {}
    for layer in cfg.layers:
        m = layer["mixer"]
        if layer["type"] == "attention":
            rope = None
            if m.get("rot") and m["rot"]["dims"]:
                key = f"rot_{m['rot']['dims']}_{m['rot']['base']!r}"          # layers with the same rotation share one object
                shared.setdefault(key, PartSpec("rope_frequencies", {"rotary_dim": m["rot"]["dims"], "theta": m["rot"]["base"]}))
                rope = SharedRef(key)
            mixer = PartSpec("differential_attention", {
                "hidden_size": W, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "dim": m["dim"], "vdim": m["vdim"],
                "scale": m["scale"], "diff": m["diff"], "norm_eps": eps, "position_encoding": rope})
        else:
            left, right, temp = m["left"], m["right"], m["left"].get("q_temp")
            mixer = PartSpec("side_by_side", {"hidden_size": W, "mixers": [
                ("left.", PartSpec("masked_sink_attention", {
                    "hidden_size": W, "num_heads": left["heads"], "num_kv_heads": left["kv_heads"], "dim": left["dim"], "vdim": left["vdim"],
                    "scale": left["scale"], "norm_eps": eps, "qk_norm": "row", "bias": True, "sink": False, "distance_bias": True,
                    "temperature": (temp["coef"], temp["every"]) if temp else None, "out_scale": m["left_scale"], "pad_rows": True})),
                ("right.", PartSpec("hgrn2", {
                    "hidden_size": W, "num_heads": right["heads"], "dim": right["dim"], "vdim": right["vdim"], "norm_eps": eps,
                    "out_scale": m["right_scale"]}))]})
        ffn = None
        if layer["mlp"] is not None:
            ffn = PartSpec("activation_mlp", {"hidden_size": W, "intermediate_size": layer["mlp"]["ff"], "activation": "gelu", "in_product": True})
        blocks.append(BlockSpec(mixer=mixer, feed_forward=ffn, kind="pre_norm", mixer_norm=norm("norm1"), feed_forward_norm=norm("norm2"),
                                mixer_prefix="mix.", feed_forward_prefix="mlp.", mixer_norm_prefix="", feed_forward_norm_prefix=""))
    # every run of a layer has a cache slot of its own: a looped layer keeps one cache or state per pass
    schedule = [LayerCall(i, slot, True, add_embedding=rejoin) for slot, (i, rejoin) in enumerate(cfg.layer_runs())]
    return ModelPlan(
        vocab_size=cfg.vocab_size, hidden_size=W, blocks=blocks, schedule=schedule, final_norm=norm("final.norm"),
        tie_word_embeddings=True, max_position=cfg.max_position_embeddings, shared=shared,
        embed_prefix="", block_prefix="l{i}.", final_norm_prefix="", head_prefix="", embed_param="embed", head_param="head")


register_architecture(Architecture("Tidenex", TidenexConfig.from_dict, tidenex_plan), replace=True)
