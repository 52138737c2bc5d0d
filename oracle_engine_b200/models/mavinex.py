"""The Mavinex decoder as data: MavinexConfig -> ModelSpec.

Every layer norms the SUM of the stream and a sublayer's output (`norm_of_sum`): x <- norm1(alpha x + mixer(x)),
x <- norm2(alpha x + ffn(x)), the feed-forward being optional; the norms are RMS norms whose weight is kept around zero.
A "parallel" layer's mixer is the mean of two normed mixers that read the same input (`parallel_mixers`): an attention with
queries and keys normed over the whole projection, a window and an output gate (`gated_attention`) and a selective scan
(`selective_scan`).  A "latent_attention" layer attends over cached latents with a window, a learned sink and one gate per
head (`latent_attention`).  The feed-forward is `moe_swiglu` with a bias on the router's logits.  A layer with `weights_of`
is one more entry of the schedule that names the owner's layer: the weights are shared, cache and state are its own.
Tensor names: `embed`, `head`, `final.norm`, `l<i>.norm1|norm2`, `l<i>.mix.left.*`, `l<i>.mix.right.*`, `l<i>.mix.*`,
`l<i>.mlp.router[.b]`, `l<i>.mlp.e<n>.gate|up|down`.
"""
from __future__ import annotations

from ..config.base import register_architecture
from ..config.mavinex import MavinexConfig
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

NO_POSITION_LIMIT = 1 << 30        # the design has no largest position; the cache's size bounds a sequence


def build_spec(cfg: MavinexConfig, max_positions: int | None = None) -> ModelSpec:
    D, eps = cfg.width, cfg.norm_eps
    max_pos = NO_POSITION_LIMIT if max_positions is None else min(max_positions, NO_POSITION_LIMIT)
    positions, layers, index_of, schedule = {}, [], {}, []

    def norm(name):
        return PartSpec("rms_norm", {"size": D, "eps": eps, "name": name, "offset": 1.0})

    def position(rot):
        """The name of the rotary tables of a rotation; equal rotations share one."""
        if rot is None:
            return None
        key = f"rot:{rot['dims']}:{rot['base']!r}:{rot['scaling']!r}"
        sc = rot["scaling"]
        if sc is not None and "low" in sc:
            sc = {"factor": sc["factor"], "low_freq_factor": sc["low"], "high_freq_factor": sc["high"],
                  "original_max_position_embeddings": sc["original"]}
        elif sc is not None:
            sc = {"kind": "yarn", **sc}
        positions.setdefault(key, PartSpec("rotary", {"head_dim": rot["dims"], "theta": rot["base"], "scaling": sc,
                                                      "max_positions": max_pos}))
        return key

    def window(m):
        return 0 if m["mask"] is None else m["mask"]["size"]

    def parallel(m):
        left, right = m["left"], m["right"]
        return PartSpec("parallel_mixers", {"hidden_size": D, "eps": eps, "branches": [
            {"tag": "left", "kind": "gated_attention", "prefix": "mix.left.", "out_norm": "mix.left.out",
             "params": {"hidden_size": D, "num_heads": left["heads"], "num_kv_heads": left["kv_heads"],
                        "key_dim": left["dim"], "value_dim": left["vdim"], "scale": left["scale"], "eps": eps,
                        "window": window(left), "position": position(left["rot"]), "pairing": "interleaved"}},
            {"tag": "right", "kind": "selective_scan", "prefix": "mix.right.", "out_norm": "mix.right.out",
             "params": {"hidden_size": D, "inner": right["inner"], "state": right["state"], "dt_rank": right["dt_rank"],
                        "conv_taps": right["conv"]}}]})

    def latent(m):
        return PartSpec("latent_attention", {
            "hidden_size": D, "num_heads": m["heads"], "key_dim": m["dim"], "value_dim": m["vdim"], "kv_rank": m["kv_rank"],
            "scale": m["scale"], "eps": eps, "rot_dim": m["rot_dim"], "position": position(m["rot"]), "pairing": "halves",
            "window": window(m), "sink": True, "gate": "head", "joined": True,
            "tensor_names": {k: "mix." + v for k, v in {
                "q": "q", "dkv": "dkv", "dkv_norm": "dkv.norm", "uk": "uk", "uv": "uv", "g": "g", "o": "o",
                "sink": "sink"}.items()}})

    for i, layer in enumerate(cfg.layers):
        j = cfg.owner(i)
        if j not in index_of:
            m, mlp = cfg.layers[j]["mixer"], cfg.layers[j]["mlp"]
            ffn = None if mlp is None else PartSpec("moe_swiglu", {
                "hidden_size": D, "num_experts": mlp["router"]["experts"], "top": mlp["router"]["top"],
                "expert_size": mlp["expert"]["ff"], "router_bias": True})
            index_of[j] = len(layers)
            layers.append(LayerSpec(
                prefix=f"l{j}.", mixer=(parallel if cfg.layers[j]["type"] == "parallel" else latent)(m), feed_forward=ffn,
                mixer_norm=norm("norm1"), ffn_norm=None if ffn is None else norm("norm2"), block="norm_of_sum",
                block_params={"alpha": cfg.postln_alpha}))
        schedule.append(ScheduleEntry(index_of[j]))
    return ModelSpec(
        architecture=cfg.architecture, hidden_size=D, vocab_size=cfg.vocab, max_positions=max_pos,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": D, "name": "embed",
                                               "scale": cfg.embedding_scale}),
        final_norm=norm("final.norm"),
        head=PartSpec("lm_head", {"vocab_size": cfg.vocab, "hidden_size": D, "tied": False, "name": "head"}),
        positions=positions, layers=tuple(layers), schedule=tuple(schedule),
        # a layer without a feed-forward does not read this, whether its file holds it or not
        ignored_tensors=(".norm2",))


register_architecture("Mavinex", MavinexConfig, build_spec)
