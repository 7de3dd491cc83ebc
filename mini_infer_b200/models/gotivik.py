"""``Gotivik``: a decoder with a norm in front of and a norm behind every branch:
``x += m * norm1b(mixer(norm1(x)))``, then ``x += m * norm2b(ff(norm2(x)))``, RMS norms, ``m`` one factor for the
model.  A layer's mixer is either softmax attention over a sliding window that keeps the first tokens of the
sequence visible, with a short causal convolution on its queries, keys and values and a rotation whose
frequencies may be rescaled, or differential attention over the whole past (two maps per head over the same
values, capped scores, queries that grow with the position, a gate per head).  The feed-forward is a squared
ReLU between two products, or absent.  A layer may run another layer's weights with a cache of its own.  The
head is the embedding table.

This file is the only place that knows the architecture: it turns a ``GotivikConfig`` into a ``ModelSpec`` of
generic parts and names the checkpoint tensors (``embed``, ``l{i}.norm1``, ``l{i}.norm1b``, ``l{i}.norm2``,
``l{i}.norm2b``, ``l{i}.mix.*``, ``l{i}.mlp.*``, ``final.norm``).
"""

from __future__ import annotations

from ..config.gotivik import GotivikConfig, WindowAttentionConfig
from ..config.registry import register_architecture
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry


def _front(H: int, eps: float, name: str) -> PartSpec:
    return PartSpec("rmsnorm", {"hidden_size": H, "eps": eps}, rename={"weight": name})


def _behind(H: int, eps: float, mult: float, name: str) -> PartSpec:
    return PartSpec("branch_rmsnorm", {"hidden_size": H, "eps": eps, "mult": mult}, rename={"weight": name})


def _rotary(m: WindowAttentionConfig) -> PartSpec | None:
    if not m.rot_dims:
        return None
    scaling = None
    if m.rot_scaling is not None:
        s = m.rot_scaling
        scaling = {"type": "yarn", "factor": s.factor, "original_max_position_embeddings": s.original,
                   "beta_fast": s.fast, "beta_slow": s.slow}
    return PartSpec("rotary", {"head_dim": m.dim, "theta": m.rot_base, "rotary_dim": m.rot_dims, "span": "rotated",
                               "scaling": scaling})


def assemble(cfg: GotivikConfig) -> ModelSpec:
    H, eps, mult = cfg.width, cfg.eps, cfg.residual_mult
    layers, place, unread = [], {}, []       # place: a layer with tensors of its own -> its index in `layers`
    for i, layer in enumerate(cfg.layers):
        if layer.weights != i:
            continue
        p, m, position = f"l{i}.", layer.mixer, None
        if isinstance(m, WindowAttentionConfig):
            mixer = PartSpec("conv_attention",
                             {"hidden_size": H, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim,
                              "value_dim": m.vdim, "scale": m.scale, "conv_taps": m.conv, "window": m.window,
                              "keep_first": m.keep_first}, prefix=p + "mix.")
            position = _rotary(m)
        else:
            mixer = PartSpec("differential_attention",
                             {"hidden_size": H, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim,
                              "value_dim": m.vdim, "scale": m.scale, "softcap": m.softcap, "diff": m.diff, "eps": eps,
                              "temp_coef": m.temp_coef, "temp_every": m.temp_every, "head_gate": True},
                             prefix=p + "mix.")
        if layer.ff:
            feed_forward = PartSpec("activated_mlp", {"hidden_size": H, "intermediate_size": layer.ff,
                                                      "activation": "relu2"}, prefix=p + "mlp.")
            ff_front, ff_behind = _front(H, eps, p + "norm2"), _behind(H, eps, mult, p + "norm2b")
        else:
            feed_forward, ff_front, ff_behind = PartSpec("no_feed_forward"), PartSpec("no_norm"), PartSpec("no_norm")
            unread += [p + "norm2", p + "norm2b"]    # a layer without a feed-forward has no second branch
        place[i] = len(layers)
        layers.append(LayerSpec(mixer=mixer, feed_forward=feed_forward, mixer_norm=_front(H, eps, p + "norm1"),
                                feed_forward_norm=ff_front, position=position, arrangement="sandwich_norm",
                                mixer_branch_norm=_behind(H, eps, mult, p + "norm1b"),
                                feed_forward_branch_norm=ff_behind))
    return ModelSpec(
        hidden_size=H,
        vocab_size=cfg.vocab,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": H}, rename={"weight": "embed"}),
        layers=tuple(layers),
        final_norm=_front(H, eps, "final.norm"),
        head=PartSpec("linear_head", {"vocab_size": cfg.vocab, "hidden_size": H, "tied": True},
                      rename={"weight": "head"}),
        schedule=tuple(ScheduleEntry(layer=place[layer.weights], cache=i) for i, layer in enumerate(cfg.layers)),
        max_positions=None,
        ignorable=tuple(unread),
    )


register_architecture("Gotivik", GotivikConfig.from_json, assemble, replace=True)
