"""``Zinesun``: a decoder whose branches read the residual stream itself and whose layer norms, each with a
scale per channel, stand behind the branches: ``x += s1 * norm1(mixer(h))`` with ``h`` the stream plus a
short causal convolution of it, then ``x += s2 * norm2(ff(x))``; what a layer hands on is a weighted sum
of the embedding's output and of every layer's result so far.  The mixer is attention in a low-rank latent
space over a sliding window (queries through a latent of their own, interleaved rotation, one sigmoid gate
per head).  The feed-forward is a dense unit with the xIELU activation, a mixture of experts (softmax over the
chosen logits, a bias on the router), or absent.  The embedding is scaled; its table is the head.

This file is the only place that knows the architecture: it turns a ``ZinesunConfig`` into a ``ModelSpec``
of generic parts and names the checkpoint tensors (``embed``, ``l{i}.norm1``, ``l{i}.norm1.b``, ``l{i}.ls1``,
``l{i}.norm2`` ..., ``l{i}.canon1``, ``l{i}.dwa``, ``l{i}.mix.*``, ``l{i}.mlp.*``, ``final.norm``, ``final.norm.b``).
"""

from __future__ import annotations

from ..config.registry import register_architecture
from ..config.zinesun import DenseConfig, ExpertsConfig, ZinesunConfig
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry


def _branch_norm(H: int, eps: float, norm: str, scale: str) -> PartSpec:
    return PartSpec("branch_layernorm", {"hidden_size": H, "eps": eps, "layer_scale": True},
                    rename={"weight": norm, "bias": norm + ".b", "scale": scale})


def assemble(cfg: ZinesunConfig) -> ModelSpec:
    H, eps = cfg.width, cfg.eps
    layers, schedule = [], []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        m = layer.mixer
        mixer = PartSpec("latent_attention",
                         {"hidden_size": H, "num_heads": m.heads, "head_dim": m.dim, "rot_dim": m.rot_dim,
                          "value_dim": m.vdim, "kv_rank": m.kv_rank, "q_rank": m.q_rank, "theta": m.rot_base,
                          "rotary_dim": m.rot_dims, "interleaved": True, "scale": m.scale, "eps": eps,
                          "window": m.window, "gate": "sigmoid", "gate_per_head": True}, prefix=p + "mix.")
        e = layer.mlp
        ff_norm = _branch_norm(H, eps, p + "norm2", p + "ls2")
        if e is None:
            feed_forward, ff_norm = PartSpec("no_feed_forward"), PartSpec("no_norm")
        elif isinstance(e, DenseConfig):
            feed_forward = PartSpec("activated_mlp", {"hidden_size": H, "intermediate_size": e.ff, "activation": "xielu"},
                                    prefix=p + "mlp.")
        else:
            assert isinstance(e, ExpertsConfig)
            feed_forward = PartSpec("routed_experts",
                                    {"hidden_size": H, "experts": e.experts, "top": e.top, "expert_ff": e.ff,
                                     "activation": "silu", "scores": "chosen", "router_bias": True}, prefix=p + "mlp.")
        layers.append(LayerSpec(
            mixer=mixer, feed_forward=feed_forward, mixer_norm=_branch_norm(H, eps, p + "norm1", p + "ls1"),
            feed_forward_norm=ff_norm, arrangement="branch_norm",
            mixer_input=PartSpec("causal_input_conv", {"hidden_size": H, "taps": cfg.taps}, rename={"weight": p + "canon1"})))
        after = PartSpec("depth_average", {"hidden_size": H, "index": i, "layers": len(cfg.layers)},
                         rename={"weights": p + "dwa"})
        schedule.append(ScheduleEntry(layer=i, cache=i, writes_cache=True, after=after))
    return ModelSpec(
        hidden_size=H,
        vocab_size=cfg.vocab,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": H, "scale": cfg.embedding_scale},
                           rename={"weight": "embed"}),
        layers=tuple(layers),
        final_norm=PartSpec("layernorm", {"hidden_size": H, "eps": eps},
                            rename={"weight": "final.norm", "bias": "final.norm.b"}),
        head=PartSpec("linear_head", {"vocab_size": cfg.vocab, "hidden_size": H, "tied": True}, rename={"weight": "head"}),
        schedule=tuple(schedule),
        max_positions=None,
    )


register_architecture("Zinesun", ZinesunConfig.from_json, assemble, replace=True)
