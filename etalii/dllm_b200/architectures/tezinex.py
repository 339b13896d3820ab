"""The Tezinex design as data: which parts each layer has, the order they run in, and the checkpoint's tensor names.

The embedding's rows get a sinusoidal position vector. Every sublayer is normed before and after, x += m
norm1b(mixer(norm1(x))) and then (a layer may have none) x += m norm2b(feed_forward(norm2(x))), with RMS norms whose
weights are stored around zero and one multiplier m for the model; behind every layer the stream becomes a weighted
sum of the embedding's output and all layers' results so far. The mixer is one of
  channel_delta: the gated delta rule behind short convolutions with one decay per head and key channel, the decays and
                 the read-out's sigmoid gate through low-rank projections;
  attention:     grouped-query softmax attention with biases on q, k and v, no rotation, capped scores, a sink per head,
                 and a sliding window that also keeps the sequence's first tokens. A layer with `kv_from: j` projects
                 no keys and values: it reads what layer j's cache holds, so the two share one cache entry.
The feed-forward is down(silu(gate(h)) * up(h)); the head is the embedding's table, its logits capped. Tensor names:
`embed`, `final.norm`, and per layer i `l<i>.norm1`, `l<i>.norm1b`, `l<i>.norm2`, `l<i>.norm2b`, `l<i>.dwa`, `l<i>.mix.*`,
`l<i>.mlp.{gate,up,down}`."""
from __future__ import annotations

from ..config.registry import register_architecture
from ..config.tezinex import TezinexConfig
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

POSITION_BASE = 10000.0


def mixer_spec(width: int, eps: float, layer: dict, prefix: str, readers=()) -> PartSpec:
    m, p = layer["mixer"], prefix + "mix."
    if layer["type"] == "channel_delta":
        names = {name: p + name for name in ("q", "k", "v", "b", "a1", "a2", "g1", "g2", "A_log", "dt_bias", "norm", "o")}
        names.update({"q_conv": p + "q.conv", "k_conv": p + "k.conv", "v_conv": p + "v.conv"})
        return PartSpec("channel_delta_rule", {
            "hidden_size": width, "heads": m["heads"], "qk_heads": m["kv_heads"], "dim": m["dim"], "vdim": m["vdim"],
            "conv": m["conv"], "eps": eps}, names)
    shares = m.get("kv_from") is not None
    names = {name: p + name for name in ("q", "o", "sink")}
    names["q_bias"] = p + "q.b"
    if not shares:
        names.update({"k": p + "k", "v": p + "v", "k_bias": p + "k.b", "v_bias": p + "v.b"})
    mask = m.get("mask")
    return PartSpec("sink_attention", {
        "hidden_size": width, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "dim": m["dim"],
        "vdim": m["vdim"], "scale": float(m["scale"]),
        "softcap": float(m["softcap"]) if m.get("softcap") is not None else 0.0,
        "window": int(mask["size"]) if mask is not None else None,
        "keep_first": int(mask.get("keep_first", 0)) if mask is not None else 0, "biases": True, "sink": True,
        "shares_keys": shares, "readers": tuple(readers)}, names)


def _mask_of(mixer: dict) -> tuple[int | None, int]:
    mask = mixer.get("mask")
    return (None, 0) if mask is None else (int(mask["size"]), int(mask.get("keep_first", 0)))


def build_spec(config: TezinexConfig) -> ModelSpec:
    width, eps = config.width, config.norm_eps
    layers, schedule, entry_of = [], [], {}
    for index, layer in enumerate(config.layers):
        prefix = f"l{index}."

        def norm(name, factor=1.0):
            return PartSpec("rmsnorm", {"hidden_size": width, "eps": eps, "zero_centred": True, "factor": factor},
                            {"weight": prefix + name})

        # a layer's cache entry is read by itself and by the layers that borrow it, each with a mask of its own
        readers = [_mask_of(other["mixer"]) for j, other in enumerate(config.layers)
                   if j == index or other["mixer"].get("kv_from") == index]
        parts = {"mixer": mixer_spec(width, eps, layer, prefix, readers), "mixer_norm": norm("norm1"),
                 "mixer_output_norm": norm("norm1b", config.residual_mult),
                 "depth_average": PartSpec("depth_average", {"index": index, "layers": len(config.layers)},
                                           {"weight": prefix + "dwa"})}
        if layer.get("mlp") is not None:
            parts["feed_forward"] = PartSpec(
                "swiglu", {"hidden_size": width, "intermediate_size": int(layer["mlp"]["ff"]), "pad": True},
                {name: f"{prefix}mlp.{name}" for name in ("gate", "up", "down")})
            parts["feed_forward_norm"] = norm("norm2")
            parts["feed_forward_output_norm"] = norm("norm2b", config.residual_mult)
        layers.append(LayerSpec(block="sandwich_norm", parts=parts))
        source = layer["mixer"].get("kv_from")
        if source is None:
            entry_of[index] = len(entry_of)  # a cache entry of its own
            schedule.append(ScheduleEntry(index, entry_of[index], True))
        else:
            schedule.append(ScheduleEntry(index, entry_of[source], False))
    return ModelSpec(
        vocab_size=config.vocab, hidden_size=width, max_position=config.max_position,
        embedding=PartSpec("token_embedding", {
            "vocab_size": config.vocab, "hidden_size": width,
            "position": PartSpec("sinusoidal", {"hidden_size": width, "base": POSITION_BASE})}, {"weight": "embed"}),
        layers=tuple(layers),
        final_norm=PartSpec("rmsnorm", {"hidden_size": width, "eps": eps, "zero_centred": True}, {"weight": "final.norm"}),
        head=PartSpec("linear", {"vocab_size": config.vocab, "hidden_size": width,
                                 "softcap": config.logit_softcap or 0.0}, {"weight": "embed"}),
        schedule=tuple(schedule), stop_token_ids=tuple(config.eos_token_ids),
        # (a layer without a feed-forward has no use for its norms; a checkpoint that stores them all the same loads)
        ignored_suffixes=tuple(f"l{i}.{name}" for i, layer in enumerate(config.layers) if layer.get("mlp") is None
                               for name in ("norm2", "norm2b")),
    )


register_architecture("Tezinex", TezinexConfig, build_spec)
