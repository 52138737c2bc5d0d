"""The Goridra decoder as data: GoridraConfig -> ModelSpec.

Every layer is h = norm1(x); x += mixer(h) + ffn(h) (`parallel_sublayers`; the feed-forward is optional) with a layer
norm that has a weight and a bias.  The mixer is grouped-query attention in chunks: a query sees the keys of its own chunk
of positions up to its own; a part of every query and key head is turned by its position; a layer may read the keys and
values of an earlier one (`cache_from` in the schedule, `reads_cache` in the mixer) with a mask of its own.  Heads whose
keys and values have one even size are a `gqa_attention` (one cache tensor, the tensor-memory prompt kernel and the
one-launch decode kernel), others a `capped_attention` without a cap (two cache tensors).  The feed-forward is a dense
`gelu` or a mixture of squared-ReLU experts chosen by groups (`moe_relu2`).  A final layer norm; the head is the embedding
table, with a cap on the logits.
Tensor names: `embed`, `final.norm[.b]`, `l<i>.norm1[.b]`, `l<i>.mix.q|k|v|o`, `l<i>.mlp.up|down`,
`l<i>.mlp.router`, `l<i>.mlp.e<n>.up|down`.
"""
from __future__ import annotations

from ..config.base import register_architecture
from ..config.goridra import GoridraConfig
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

NO_POSITION_LIMIT = 1 << 30        # the design has no largest position; the cache's size bounds a sequence


def build_spec(cfg: GoridraConfig, max_positions: int | None = None) -> ModelSpec:
    D, eps = cfg.width, cfg.norm_eps
    max_pos = NO_POSITION_LIMIT if max_positions is None else min(max_positions, NO_POSITION_LIMIT)
    positions, layers, schedule = {}, [], []

    def norm(name):
        return PartSpec("layer_norm", {"size": D, "eps": eps, "name": name})

    def position(rot, head_dim):
        """The name of the rotary tables of a rotation; equal rotations share one."""
        if rot is None:
            return None
        key = f"rot:{head_dim}:{rot['dims']}:{rot['base']!r}"
        positions.setdefault(key, PartSpec("rotary", {"head_dim": head_dim, "dims": rot["dims"], "theta": rot["base"],
                                                      "scaling": None, "max_positions": max_pos}))
        return key

    for i, layer in enumerate(cfg.layers):
        m, mlp = layer["mixer"], layer["mlp"]
        params = {"hidden_size": D, "num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "scale": m["scale"],
                  "chunk": (m["mask"] or {}).get("size", 0), "reads_cache": m["kv_from"] is not None,
                  "tensor_names": {k: "mix." + k for k in ("q", "k", "v", "o")}}
        if m["dim"] == m["vdim"] and m["dim"] % 2 == 0:
            mixer = PartSpec("gqa_attention", {**params, "head_dim": m["dim"], "position": position(m["rot"], m["dim"])})
        else:
            # this mixer's kernels turn a part of a head by themselves: tables of the turned dimensions only
            mixer = PartSpec("capped_attention", {**params, "key_dim": m["dim"], "value_dim": m["vdim"],
                                                  "position": position(m["rot"], m["rot"]["dims"] if m["rot"] else 0)})
        if mlp is None:
            ffn = None
        elif mlp["kind"] == "dense":
            ffn = PartSpec("gelu", {"hidden_size": D, "intermediate_size": mlp["ff"],
                                    "tensor_names": {"up": "mlp.up", "down": "mlp.down"}})
        else:
            router = mlp["router"]
            ffn = PartSpec("moe_relu2", {"hidden_size": D, "num_experts": router["experts"], "top": router["top"],
                                         "expert_size": mlp["expert"]["ff"], "groups": router["groups"]})
        layers.append(LayerSpec(prefix=f"l{i}.", mixer=mixer, feed_forward=ffn, mixer_norm=norm("norm1"), ffn_norm=None,
                                block="parallel_sublayers"))
        schedule.append(ScheduleEntry(i, cache_from=m["kv_from"]))
    return ModelSpec(
        architecture=cfg.architecture, hidden_size=D, vocab_size=cfg.vocab, max_positions=max_pos,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": D, "name": "embed"}),
        final_norm=norm("final.norm"),
        head=PartSpec("lm_head", {"vocab_size": cfg.vocab, "hidden_size": D, "tied": True, "name": "embed",
                                  "softcap": cfg.logit_softcap}),
        positions=positions, layers=tuple(layers), schedule=tuple(schedule))


register_architecture("Goridra", GoridraConfig, build_spec)
