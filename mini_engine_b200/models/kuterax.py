"""Kuterax as a plan of parts.

Every layer is a ``parallel`` block with ONE RMS norm (weight stored around zero) that both sub-layers read, and a scale for each of their
outputs.  The mixer is retention (``retention``) or two mixers side by side (``side_by_side``) whose outputs are normed over the width and
averaged: windowed grouped-query attention with biased projections, a weighted norm of q and k in front of a YaRN rotation, a one in the
softmax's denominator and a gate a head (``masked_sink_attention``), and Mamba-2 (``mamba2``).  The feed-forward is routed squared-relu experts
chosen by a softmax over all of them within the best groups, with a gated shared expert (``routed_experts``), or absent.  A range of layers may
be looped over: every pass has cache and state slots of its own, and in front of it the stream becomes a
product of itself and the embedding output, plus the pass's vector.  The embedding has a learned vector for every position.  Layer i's
tensors are ``l<i>.*``; all numbers come from the configuration.
"""
from __future__ import annotations

from ..config.model_config import KuteraxConfig
from ..config.registry import Architecture, register_architecture
from ..parts import BlockSpec, LayerCall, ModelPlan, PartSpec, SharedRef


def _rotation(m: dict, shared: dict):
    rot = m.get("rot")
    if not rot or not rot["dims"]:
        return None
    sc = rot.get("scaling")
    key = f"rot_{rot['dims']}_{rot['base']!r}_{sorted(sc.items()) if sc else None}"      # layers with the same rotation share one object
    shared.setdefault(key, PartSpec("rope_frequencies", {"rotary_dim": rot["dims"], "theta": rot["base"], "scaling": sc}))
    return SharedRef(key)


def kuterax_plan(cfg: KuteraxConfig) -> ModelPlan:
    W, eps = cfg.hidden_size, cfg.norm_eps

    def norm(name: str) -> PartSpec:
        return PartSpec("rmsnorm", {"size": W, "eps": eps, "param": name, "unit_offset": True})
    blocks, shared = [], {}
    for layer in cfg.layers:
        m = layer["mixer"]
        if layer["type"] == "retention":
            mixer = PartSpec("retention", {"hidden_size": W, "num_heads": m["heads"], "dim": m["dim"], "vdim": m["vdim"], "decay": m["decay"],
                                           "norm_eps": eps})
        else:
            left, right = m["left"], m["right"]
            mixer = PartSpec("side_by_side", {"hidden_size": W, "mixers": [
                ("left.", PartSpec("masked_sink_attention", {
                    "hidden_size": W, "num_heads": left["heads"], "num_kv_heads": left["kv_heads"], "dim": left["dim"], "vdim": left["vdim"],
                    "scale": left["scale"], "norm_eps": eps, "position_encoding": _rotation(left, shared), "qk_norm": "before", "bias": True,
                    "output_bias": False, "sink": "one", "head_gate": True, "pad_rows": True,
                    "mask": ("window", left["mask"]["size"]) if left.get("mask") else None})),
                ("right.", PartSpec("mamba2", {
                    "hidden_size": W, "num_heads": right["heads"], "vdim": right["vdim"], "state": right["state"], "groups": right["groups"],
                    "taps": right["conv"], "norm_groups": right["norm_groups"], "norm_eps": eps}))],
                "output_norms": {"names": ["left.out", "right.out"], "eps": eps, "mean": True}})
        mlp, ffn = layer["mlp"], None
        if mlp is not None:
            r = mlp["router"]
            ffn = PartSpec("routed_experts", {
                "hidden_size": W, "num_experts": r["experts"], "top": r["top"], "expert_size": mlp["expert"]["ff"], "router_bias": False,
                "routing": "softmax_groups", "groups": (r["groups"]["count"], r["groups"]["keep"]), "weight_scale": r["scale"],
                "activation": "relu_squared",
                **({"shared": {"intermediate_size": mlp["shared"]["ff"], "activation": "relu_squared"}, "shared_gate": "shared.sg"}
                   if mlp.get("shared") else {})})
        blocks.append(BlockSpec(mixer=mixer, feed_forward=ffn, kind="parallel", mixer_norm=norm("norm1"), mixer_prefix="mix.",
                                feed_forward_prefix="mlp.", mixer_norm_prefix="",
                                args={"one_norm": True, "scales": {"mixer": "ls1", "feed_forward": "ls2", "width": W}}))
    # every run of a layer has a cache slot of its own: a looped layer keeps one cache and state per pass
    schedule = [LayerCall(i, slot, True, add_row=t, join_embedding=t is not None) for slot, (i, t) in enumerate(cfg.layer_runs())]
    return ModelPlan(
        vocab_size=cfg.vocab_size, hidden_size=W, blocks=blocks, schedule=schedule, final_norm=norm("final.norm"),
        tie_word_embeddings=False, max_position=cfg.max_position_embeddings, shared=shared,
        embed_prefix="", block_prefix="l{i}.", final_norm_prefix="", head_prefix="", embed_param="embed", head_param="head",
        position_table=("pos", cfg.max_position_embeddings), pass_vectors=("loop.step", cfg.loop["times"]) if cfg.loop else None,
        pass_input="loop.in" if cfg.loop else None)


register_architecture(Architecture("Kuterax", KuteraxConfig.from_dict, kuterax_plan), replace=True)
