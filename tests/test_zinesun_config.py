"""CPU checks of the Zinesun architecture: configuration reader, assembly into parts, tensor names and
shapes against a checkpoint's, what the cache manager is asked to keep, and the plain implementation's own
consistency."""

import copy

import pytest
import torch

import plain_zinesun as P
from zinesun_configs import CONFIGS, config, dense, latent, prompt, random_state

from mini_infer_b200.cache.manager import CacheManager
from mini_infer_b200.config import ConfigError, load_config
from mini_infer_b200.parts import DecoderModel, KVNeed, LayerSpec, ModelSpec, PartSpec, StateNeed
from mini_infer_b200.weights.loader import WeightLoadError, check_names


def build(which):
    arch, cfg = load_config(CONFIGS[which])
    return cfg, DecoderModel(arch.assemble(cfg))


@pytest.mark.parametrize("which", list(CONFIGS))
def test_names_and_shapes_fit_a_checkpoint(which):
    cfg, model = build(which)
    state = random_state(CONFIGS[which], seed=1)
    check_names(model, {n: tuple(t.shape) for n, t in state.items()})
    assert len(model.blocks) == len(cfg.layers)
    assert model.graph_safe()
    broken = {n: tuple(t.shape) for n, t in state.items()}
    broken["embed"] = broken["embed"][::-1]
    del broken["final.norm.b"]
    broken["surplus"] = (1,)
    with pytest.raises(WeightLoadError) as e:
        check_names(model, broken)
    assert e.value.missing == ["final.norm.b"] and e.value.unexpected == ["surplus"]
    assert [m[0] for m in e.value.mismatched] == ["embed"]


def test_what_the_cache_keeps():
    _, model = build("A")
    needs = model.cache_needs()
    windows = [9, 17, 30, 64]
    rows = [24 + 6, 40 + 4, 16 + 10, 36 + 2]
    assert [n.kv for n in needs[:4]] == [KVNeed(1, r, w, 0, None) for r, w in zip(rows, windows)]
    assert all(n.state is None for n in needs[:4])
    # the inputs of every layer's convolution, under indices behind the cache layers' (and the embedding's)
    assert [(n.index, n.kv, n.state) for n in needs[4:]] == \
        [(model.input_state_index(i), None, StateNeed((2, 48), torch.float32)) for i in range(4)]
    assert len({n.index for n in needs}) == len(needs)
    _, model = build("C")                                 # one tap: nothing to keep
    assert len(model.cache_needs()) == 3
    names = {e.name for e in model.expected_tensors()}
    assert "l0.norm2" not in names and "l0.ls2" not in names and "l1.ls2" in names
    assert [p.index for p in model.after] == [0, 1, 2] and [p.layers for p in model.after] == [3, 3, 3]


def test_windows_give_pages_back():
    """A request decodes far past its pools: every layer's group keeps the pages of its own window only."""
    _, model = build("C")
    cm = CacheManager(model.cache_needs(), page_size=4, num_pages=14, max_requests=2)
    assert [g.window for g in cm.groups] == [1, 2, 45]
    cm.add_request("a")
    for _ in range(300):
        cm.plan_append([("a", 1)])
        cm.check()
    held = [sum(p >= 0 for p in cm.table("a", g)) for g in range(3)]
    assert held[0] <= 2 and held[1] <= 2 and held[2] <= 13
    cm.free_request("a")
    assert all(cm.num_free_pages(g) == 14 for g in range(3))


def test_configurations_that_are_refused():
    base = CONFIGS["A"]
    cases = [
        lambda c: c.pop("canon"), lambda c: c["canon"].update(taps=0), lambda c: c["embedding"].pop("scale"),
        lambda c: c["norm"].pop("eps"), lambda c: c.update(layers=[]),
        lambda c: c["layers"][1].update(type="attention"),
        lambda c: c["layers"][1]["mixer"].pop("q_rank"), lambda c: c["layers"][1]["mixer"].pop("mask"),
        lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), lambda c: c["layers"][1]["mixer"]["rot"].update(dims=5),
        lambda c: c["layers"][1]["mixer"]["rot"].update(dims=6), lambda c: c["layers"][1]["mixer"].update(heads=True),
        lambda c: c["layers"][1]["mlp"]["router"].update(top=7), lambda c: c["layers"][0]["mlp"].update(kind="gated"),
        lambda c: c["layers"][1]["mlp"].pop("expert"),
    ]
    for change in cases:
        cfg = copy.deepcopy(base)
        change(cfg)
        with pytest.raises(ConfigError):
            load_config(cfg)


def test_an_input_part_needs_an_arrangement_that_runs_it():
    norm = PartSpec("rmsnorm", {"hidden_size": 8, "eps": 1e-6})
    layer = LayerSpec(mixer=PartSpec("gqa_attention", {"hidden_size": 8, "num_heads": 1, "num_kv_heads": 1, "head_dim": 16}),
                      feed_forward=PartSpec("no_feed_forward"), mixer_norm=norm, feed_forward_norm=PartSpec("no_norm"),
                      mixer_input=PartSpec("causal_input_conv", {"hidden_size": 8, "taps": 2}), arrangement="prenorm")
    spec = ModelSpec(8, 5, PartSpec("token_embedding", {"vocab_size": 5, "hidden_size": 8}), (layer,), norm,
                     PartSpec("linear_head", {"vocab_size": 5, "hidden_size": 8}))
    with pytest.raises(ValueError, match="input part"):
        DecoderModel(spec)


# ----------------------------------------------------------------------------- the plain implementation itself


def test_plain_prefixes_windows_and_averages():
    """A prefix's logits do not depend on what follows; a token just outside the only layer's window changes
    nothing but what the convolution carries, one just inside does."""
    cfg = CONFIGS["A"]
    state = random_state(cfg, seed=2)
    toks = prompt(cfg, 24, salt=1)
    streams = []
    full = P.zinesun_logits(state, cfg, toks, streams=streams)
    assert torch.allclose(P.zinesun_logits(state, cfg, toks[:9]), full[:9], atol=1e-9)
    assert len(streams) == len(cfg["layers"])
    one = config([latent(2, 8, 4, 6, 10, 12, 5, 0.5, 10.0, dense(12))], vocab=31, width=16, eps=1e-5, taps=1, scale=1.0)
    state = random_state(one, seed=3)
    toks = prompt(one, 12, salt=2)
    base = P.zinesun_logits(state, one, toks)
    other = list(toks)
    other[6] = (other[6] + 1) % 31
    moved = (P.zinesun_logits(state, one, other) - base).abs().max(dim=1).values
    assert (moved[:6] == 0).all() and (moved[6:11] > 1e-6).all() and (moved[11:] == 0).all()     # seen from 6 to 6 + 4
    # weights (1, 0 ... 0): only the embedding's output is handed on
    s2 = {k: v.clone() for k, v in state.items()}
    s2["l0.dwa"] = torch.tensor([1.0, 0.0])
    x = s2["embed"][torch.tensor(toks)].double()
    want = P.layer_norm(x, s2["final.norm"].double(), s2["final.norm.b"].double(), 1e-5) @ s2["embed"].double().T
    assert torch.allclose(P.zinesun_logits(s2, one, toks), want, atol=1e-12)


def test_plain_mechanisms_on_known_numbers():
    z = torch.tensor([-3.0, -1e-3, 0.0, 1e-3, 2.0], dtype=torch.float64)
    p, q = torch.tensor(0.0, dtype=torch.float64), torch.tensor(1.0, dtype=torch.float64)
    want = [(0.5 + torch.log1p(torch.exp(q))) * (torch.exp(v) - 1 - v) + v / 2 if v <= 0
            else torch.log(torch.tensor(2.0, dtype=torch.float64)) * v * v + v / 2 for v in z]
    assert torch.allclose(P.xielu(z, p, q), torch.stack(want), atol=1e-15)
    x = torch.tensor([[[1.0, 0.0, 0.0, 2.0, 5.0]]], dtype=torch.float64)       # pairs (0, 1), (2, 3); the last passes
    got = P.rotate_pairs(x, [1], {"dims": 4, "base": 16.0})[0, 0]
    a, b = torch.tensor(1.0, dtype=torch.float64), torch.tensor(0.25, dtype=torch.float64)
    assert torch.allclose(got, torch.stack([a.cos(), a.sin(), -2 * b.sin(), 2 * b.cos(), x[0, 0, 4]]), atol=1e-15)
    h = torch.arange(5, dtype=torch.float64)[:, None] + 1
    w = torch.tensor([[100.0, 10.0, 1.0]], dtype=torch.float64)
    assert P.input_convolution(h, w)[:, 0].tolist() == [2.0, 14.0, 126.0, 238.0, 350.0]
    ids, weights, margin = P.choose_experts(torch.tensor([0.0, 2.0, 1.0, -1.0]), 2)
    assert ids == [1, 2] and abs(sum(weights) - 1) < 1e-6 and abs(weights[0] / weights[1] - 2.7182818) < 1e-5
    assert abs(margin - 1.0) < 1e-6
