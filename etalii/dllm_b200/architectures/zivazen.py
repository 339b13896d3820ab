"""The Zivazen design as data: which parts each layer has, the order they run in, and the checkpoint's tensor names.

The embedding's rows are RMS-normed on the way into the stream. A layer has one RMS norm, whose output both of its parts
read: x += mixer(h) + feed_forward(h), h = norm1(x) (a layer may have no feed-forward). The mixer is one of
  attention: grouped-query softmax attention with biases on q, k, v and the output, RMS norms per query and key head,
             rotary positions (halves, optionally with long wavelengths stretched), chunks, one more in the softmax's
             denominator, and values mixed with those of the first layer that mixes;
  parallel:  grouped-query softmax attention over a sliding window beside a Mamba-2 branch, each output with a factor.
The feed-forward is dense, down(silu(gate(h)) * up(h)) with biases, or a mixture of relu-squared experts chosen by sigmoid
scores with a correction inside the best groups, and a shared expert. Tensor names: `embed`, `embed.norm`, `head`,
`final.norm`, and per layer i `l<i>.norm1`, `l<i>.mix.*`, `l<i>.mlp.*`; a bias is its matrix's name with `.b` behind."""
from __future__ import annotations

from ..config.registry import register_architecture
from ..config.zivazen import ZivazenConfig, mixes_values
from ..parts.spec import LayerSpec, ModelSpec, PartSpec


def _position(m: dict) -> PartSpec | None:
    rot = m.get("rot")
    if rot is None or not rot["dims"]:
        return None
    params = {"head_dim": m["dim"], "theta": float(rot["base"]), "rotary_dim": int(rot["dims"]), "pairing": "halves"}
    scaling = rot.get("scaling")
    if scaling is not None:
        params["scaling"] = {"rope_type": "llama3", "factor": float(scaling["factor"]),
                             "low_freq_factor": float(scaling["low"]), "high_freq_factor": float(scaling["high"]),
                             "original_max_position_embeddings": float(scaling["original"])}
    return PartSpec("rotary", params)


def _mask_size(m: dict) -> int | None:
    return int(m["mask"]["size"]) if m.get("mask") is not None else None


def attention_spec(width: int, eps: float, m: dict, p: str, value_mix: str | None) -> PartSpec:
    names = {name: p + name for name in ("q", "k", "v", "o")}
    names.update({name + "_bias": f"{p}{name}.b" for name in ("q", "k", "v", "o")})
    names.update({"q_norm": p + "q.norm", "k_norm": p + "k.norm"})
    if value_mix is not None:
        names["share"] = p + "vmix"
    return PartSpec("sink_attention", {
        "hidden_size": width, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "dim": m["dim"],
        "vdim": m["vdim"], "scale": float(m["scale"]), "chunk": _mask_size(m), "position": _position(m), "qk_eps": eps,
        "biases": True, "output_bias": True, "ones_column": True, "sink": "unit", "value_mix": value_mix}, names)


def window_spec(width: int, m: dict) -> PartSpec:
    """The softmax branch of a parallel mixer: the plain attention part where keys and values have one size that its
    kernels take, else the one that takes any."""
    common = {"hidden_size": width, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "scale": float(m["scale"]),
              "window": _mask_size(m), "position": _position(m)}
    if m["dim"] == m["vdim"] and m["dim"] % 16 == 0 and m["dim"] <= 128:
        return PartSpec("attention", {**common, "head_dim": m["dim"]})
    return PartSpec("sink_attention", {**common, "dim": m["dim"], "vdim": m["vdim"], "sink": False})


def mixer_spec(width: int, eps: float, layer: dict, prefix: str, value_mix: str | None) -> PartSpec:
    m, p = layer["mixer"], prefix + "mix."
    if layer["type"] == "attention":
        return attention_spec(width, eps, m, p, value_mix)
    right = m["right"]
    names = {f"left.{name}": f"{p}left.{name}" for name in ("q", "k", "v", "o")}
    names.update({f"right.{name}": f"{p}right.{name}" for name in ("in", "conv", "dt_bias", "A_log", "D", "norm", "o")})
    names["right.conv_bias"] = p + "right.conv.b"
    return PartSpec("parallel", {
        "hidden_size": width, "eps": eps, "scales": (float(m["left_scale"]), float(m["right_scale"])),
        "left": window_spec(width, m["left"]),
        "right": PartSpec("state_space_duality", {
            "hidden_size": width, "heads": right["heads"], "vdim": right["vdim"], "state": right["state"],
            "groups": right["groups"], "conv": right["conv"], "norm_groups": right["norm_groups"], "eps": eps})}, names)


def feed_forward_spec(width: int, mlp: dict, prefix: str) -> PartSpec:
    p = prefix + "mlp."
    if mlp["kind"] == "dense":
        names = {name: p + name for name in ("gate", "up", "down")}
        names.update({name + "_bias": f"{p}{name}.b" for name in ("gate", "up", "down")})
        return PartSpec("swiglu", {"hidden_size": width, "intermediate_size": int(mlp["ff"]), "pad": True,
                                   "biases": True}, names)
    router = mlp["router"]
    names = {"router": p + "router", "correction": p + "correction"}
    for e in range(int(router["experts"])):
        names.update({f"e{e}.{part}": f"{p}e{e}.{part}" for part in ("up", "down")})
    shared = None
    if mlp.get("shared") is not None:
        shared = PartSpec("activation_mlp", {"hidden_size": width, "intermediate_size": int(mlp["shared"]["ff"]),
                                             "activation": "relu_squared"})
        names.update({f"shared.{part}": f"{p}shared.{part}" for part in ("up", "down")})
    groups = router.get("groups") or {"count": 1, "keep": 1}
    return PartSpec("activation_experts", {
        "hidden_size": width, "intermediate_size": int(mlp["expert"]["ff"]), "experts": int(router["experts"]),
        "top": int(router["top"]), "activation": "relu_squared", "weights": "sigmoid_groups",
        "groups": (int(groups["count"]), int(groups["keep"])), "weight_factor": float(router["scale"]),
        "shared": shared}, names)


def build_spec(config: ZivazenConfig) -> ModelSpec:
    width, eps = config.width, config.norm_eps
    layers = []
    mixing = [index for index, layer in enumerate(config.layers) if mixes_values(layer)]
    for index, layer in enumerate(config.layers):
        prefix = f"l{index}."
        value_mix = None if index not in mixing else ("keep" if index == mixing[0] else "mix")
        parts = {"mixer": mixer_spec(width, eps, layer, prefix, value_mix),
                 "mixer_norm": PartSpec("rmsnorm", {"hidden_size": width, "eps": eps}, {"weight": prefix + "norm1"})}
        if layer.get("mlp") is not None:
            parts["feed_forward"] = feed_forward_spec(width, layer["mlp"], prefix)
        layers.append(LayerSpec(block="shared_norm", parts=parts))
    return ModelSpec(
        vocab_size=config.vocab, hidden_size=width, max_position=config.max_position,
        embedding=PartSpec("token_embedding", {"vocab_size": config.vocab, "hidden_size": width, "norm_eps": eps},
                           {"weight": "embed", "norm": "embed.norm"}),
        layers=tuple(layers),
        final_norm=PartSpec("rmsnorm", {"hidden_size": width, "eps": eps}, {"weight": "final.norm"}),
        head=PartSpec("linear", {"vocab_size": config.vocab, "hidden_size": width}, {"weight": "head"}),
        stop_token_ids=tuple(config.eos_token_ids),
    )


register_architecture("Zivazen", ZivazenConfig, build_spec)
