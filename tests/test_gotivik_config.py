"""CPU checks of the Gotivik architecture: configuration reader, assembly into parts, tensor names and shapes against
a checkpoint's, what the cache manager is asked to keep and gives back, the rescaled rotation's numbers, and the plain
implementation's own consistency."""

import copy
import math

import pytest
import torch

import plain_gotivik as P
from gotivik_configs import CONFIGS, again, config, differential, owner, prompt, random_state, window, yarn

from mini_infer_b200.cache.manager import CacheManager
from mini_infer_b200.config import ConfigError, load_config
from mini_infer_b200.parts import DecoderModel, KVNeed, LayerSpec, ModelSpec, PartSpec, StateNeed, build_part
from mini_infer_b200.weights.loader import WeightLoadError, check_names


def build(which):
    arch, cfg = load_config(CONFIGS[which])
    return cfg, DecoderModel(arch.assemble(cfg))


@pytest.mark.parametrize("which", list(CONFIGS))
def test_names_and_shapes_fit_a_checkpoint(which):
    cfg, model = build(which)
    state = random_state(CONFIGS[which], seed=1)
    check_names(model, {n: tuple(t.shape) for n, t in state.items()})
    owners = [owner(CONFIGS[which], i) for i in range(len(cfg.layers))]
    assert [layer.weights for layer in cfg.layers] == owners
    own = sorted(set(owners))
    assert len(model.blocks) == len(own) and model.graph_safe()
    # every entry runs its owner's block with a cache layer of its own
    assert [own[e.layer] for e in model.schedule] == owners
    assert [e.cache for e in model.schedule] == list(range(len(owners)))
    broken = {n: tuple(t.shape) for n, t in state.items()}
    broken["embed"] = broken["embed"][::-1]
    del broken["final.norm"]
    broken["surplus"] = (1,)
    with pytest.raises(WeightLoadError) as e:
        check_names(model, broken)
    assert e.value.missing == ["final.norm"] and e.value.unexpected == ["surplus"]
    assert [m[0] for m in e.value.mismatched] == ["embed"]


def test_layers_without_a_feed_forward_may_carry_its_norms():
    _, model = build("C")
    state = random_state(CONFIGS["C"], seed=1)
    shapes = {n: tuple(t.shape) for n, t in state.items()}
    assert "l0.norm2" not in shapes and "l1.norm2b" in shapes
    shapes.update({"l0.norm2": (36,), "l0.norm2b": (36,)})
    check_names(model, shapes)


def test_what_the_cache_keeps():
    _, model = build("A")
    needs = model.cache_needs()
    kv = [KVNeed(2, 12, 9, 20, keep_first=2), KVNeed(1, 32, None, 14), KVNeed(3, 16, None, 9), KVNeed(5, 6, 17, None)]
    assert [n.kv for n in needs] == kv + [kv[1], kv[0]]       # a key's two maps in one row, padded to a multiple of 16
    states = [StateNeed((2 * (6 * 12 + 2 * 20),), torch.float32), None, None, StateNeed((15 * 6,), torch.float32)]
    assert [n.state for n in needs] == states + [None, states[0]]
    _, model = build("C")                                      # one tap: nothing to keep
    assert model.cache_needs()[0].state is None and model.cache_needs()[0].kv == KVNeed(1, 6, 1, 10, keep_first=3)


def test_windows_give_pages_back_but_keep_the_first_ones():
    """A request decodes far past its pools: a window's group keeps the pages of the window and those of the first
    tokens, in a pool that holds no more; the pages given back are used again, also within the step."""
    _, model = build("C")
    cm = CacheManager(model.cache_needs(), page_size=4, num_pages=[3, 80, 2, 13], max_requests=2)
    assert [(g.window, g.keep_first) for g in cm.groups] == [(1, 3), (None, 0), (2, 0), (5, 40)]
    for rid in ("a", "b"):
        cm.add_request(rid)
        for n in range(300):
            cm.plan_append([(rid, 1)])
            cm.check()
            for gi, g in enumerate(cm.groups):
                table = cm.table(rid, gi)
                seen = [j for j in range(n + 1) if g.window is None or n - j < g.window or j < g.keep_first]
                assert all(table[j // 4] >= 0 for j in seen)
        held = [sum(p >= 0 for p in cm.table(rid, gi)) for gi in range(4)]
        assert held[0] <= 3 and held[1] == 75 and held[2] <= 2 and held[3] <= 13
        cm.free_request(rid)
    assert [cm.num_free_pages(g) for g in range(4)] == [3, 80, 2, 13]


def test_pages_needed_counts_kept_pages_once():
    cm = CacheManager([type("N", (), dict(index=0, kv=KVNeed(1, 8, 6, keep_first=5), state=None))()], page_size=4,
                      num_pages=6, max_requests=1)
    cm.add_request("a")
    cm.plan_append([("a", 17)])                    # five pages
    assert cm.pages_needed([("a", 4)]) == [0]      # a sixth; page 2 comes back, pages 0 and 1 are kept
    cm.plan_append([("a", 4)])
    table = cm.table("a")
    assert [p >= 0 for p in table] == [True, True, False, True, True, True]
    cm.check()


@pytest.mark.parametrize("rot", [{"base": 50.0, "dims": 8, "scaling": yarn(3.0, 40, 4.0, 0.5)},
                                 {"base": 20.0, "dims": 2, "scaling": yarn(8.0, 16, 2.0, 0.9)},
                                 {"base": 500000.0, "dims": 64, "scaling": yarn(4.0, 8192, 32.0, 1.0)},
                                 {"base": 100.0, "dims": 6, "scaling": yarn(2.0, 10, 1e-4, 1e-5)},
                                 {"base": 100.0, "dims": 6, "scaling": yarn(1.0, 50, 2.0, 2.0)},
                                 {"base": 777.0, "dims": 10}])
def test_rescaled_rotation_frequencies(rot):
    """Frequencies and the factor on sines and cosines, also where both edges fall outside the pairs or on one."""
    sc = rot.get("scaling")
    scaling = {"type": "yarn", "factor": sc["factor"], "original_max_position_embeddings": sc["original"],
               "beta_fast": sc["fast"], "beta_slow": sc["slow"]} if sc else None
    part = build_part("position", PartSpec("rotary", {"head_dim": 80, "theta": rot["base"], "rotary_dim": rot["dims"],
                                                      "span": "rotated", "scaling": scaling}))
    part.bind({}, torch.float32, torch.device("cpu"))
    freqs, mult = P.yarn_frequencies(rot)
    assert part.freq64.tolist() == pytest.approx(freqs, rel=1e-14) and part.multiplier == pytest.approx(mult, rel=1e-15)
    if sc and sc["factor"] > 1:
        assert rot["dims"] < 8 or any(abs(a - rot["base"] ** (-2 * i / rot["dims"])) > 1e-9 for i, a in enumerate(freqs))


def test_configurations_that_are_refused():
    cases = [
        lambda c: c.pop("residual_mult"), lambda c: c["norm"].pop("eps"), lambda c: c.update(layers=[]),
        lambda c: c["layers"][2].update(type="attention_3"), lambda c: c["layers"][2]["mixer"].pop("diff"),
        lambda c: c["layers"][2]["mixer"].update(softcap=0), lambda c: c["layers"][2]["mixer"]["q_temp"].update(every=0),
        lambda c: c["layers"][2]["mixer"].update(kv_heads=4), lambda c: c["layers"][3]["mixer"].pop("mask"),
        lambda c: c["layers"][3]["mixer"]["mask"].pop("keep_first"), lambda c: c["layers"][3]["mixer"]["mask"].update(size=0),
        lambda c: c["layers"][3]["mixer"]["mask"].update(keep_first=-1), lambda c: c["layers"][3]["mixer"].pop("conv"),
        lambda c: c["layers"][3]["mixer"]["rot"].update(dims=5), lambda c: c["layers"][3]["mixer"]["rot"].update(dims=8),
        lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"), lambda c: c["layers"][3]["mlp"].update(kind="moe"),
        lambda c: c["layers"][3].update(weights_of=9), lambda c: c["layers"][3].update(weights_of=3),
        lambda c: c["layers"][4].update(weights_of=2), lambda c: c["layers"][4].update(weights_of=True),
        lambda c: c["layers"][1].update(weights_of=4),       # two layers that name one another
    ]
    for change in cases:
        cfg = copy.deepcopy(CONFIGS["A"])
        change(cfg)
        with pytest.raises(ConfigError):
            load_config(cfg)
    bad = copy.deepcopy(CONFIGS["A"])
    bad["layers"][3]["mixer"]["conv"] = 17               # more taps than the kernel's tile has tokens
    arch, cfg = load_config(bad)
    with pytest.raises(ValueError, match="taps"):
        DecoderModel(arch.assemble(cfg))


def test_branch_norms_need_an_arrangement_with_places_for_them():
    norm = PartSpec("rmsnorm", {"hidden_size": 8, "eps": 1e-6})
    behind = PartSpec("branch_rmsnorm", {"hidden_size": 8, "eps": 1e-6})

    def model(arrangement, **norms):
        layer = LayerSpec(mixer=PartSpec("gqa_attention", {"hidden_size": 8, "num_heads": 1, "num_kv_heads": 1, "head_dim": 16}),
                          feed_forward=PartSpec("no_feed_forward"), mixer_norm=norm, feed_forward_norm=PartSpec("no_norm"),
                          arrangement=arrangement, **norms)
        return DecoderModel(ModelSpec(8, 5, PartSpec("token_embedding", {"vocab_size": 5, "hidden_size": 8}), (layer,), norm,
                                      PartSpec("linear_head", {"vocab_size": 5, "hidden_size": 8})))

    with pytest.raises(ValueError, match="no place"):
        model("prenorm", mixer_branch_norm=behind)
    with pytest.raises(ValueError, match="needs"):
        model("sandwich_norm")
    assert len(model("sandwich_norm", mixer_branch_norm=behind, feed_forward_branch_norm=PartSpec("no_norm")).blocks) == 1


# ----------------------------------------------------------------------------- the plain implementation itself


def test_plain_prefixes_and_windows():
    """A prefix's logits do not depend on what follows; with one windowed layer a changed token moves the positions
    that see it, those whose convolution carries it, and no others, unless it is one of the kept first ones."""
    cfg = CONFIGS["A"]
    state = random_state(cfg, seed=2)
    toks = prompt(cfg, 22, salt=1)
    full = P.gotivik_logits(state, cfg, toks)
    assert torch.allclose(P.gotivik_logits(state, cfg, toks[:9]), full[:9], atol=1e-9)
    assert len(P.gotivik_streams(state, cfg, toks)) == len(cfg["layers"]) + 1
    one = config([window(2, 1, 8, 6, 0.5, 2, 4, 2, (10.0, 4), 0)], vocab=31, width=16, eps=1e-5, mult=1.0)
    state = random_state(one, seed=3)
    toks = prompt(one, 16, salt=2)
    base = P.gotivik_logits(state, one, toks)
    for at, last in ((6, 6 + 1 + 3), (1, 15), (2, 2 + 1 + 3)):      # its key reaches one token on, then three more see that
        other = list(toks)
        other[at] = (other[at] + 1) % 31
        moved = (P.gotivik_logits(state, one, other) - base).abs().max(dim=1).values
        assert (moved[:at] == 0).all() and (moved[at:last + 1] > 1e-9).all() and (moved[last + 1:] == 0).all()


def test_plain_layers_that_share_weights():
    L = [differential(2, 1, 4, 6, 0.5, 3.0, 0.3, 0.2, 3, 12), window(2, 2, 4, 4, 0.5, 2, 3, 1, (10.0, 4), 8)]
    cfg = config(L + [again(L, 0)], vocab=23, width=12, eps=1e-5, mult=0.5)
    state = random_state(cfg, seed=4)
    spelled = {n.replace("l0.", "l2.") if n.startswith("l0.") else n: t for n, t in state.items()} | state
    toks = prompt(cfg, 9, salt=3)
    same = dict(cfg, layers=L + [L[0]])
    assert torch.equal(P.gotivik_logits(state, cfg, toks), P.gotivik_logits(spelled, same, toks))


def test_plain_mechanisms_on_known_numbers():
    u = torch.arange(5, dtype=torch.float64)[:, None] + 1
    w = torch.tensor([[100.0, 10.0, 1.0]], dtype=torch.float64)
    assert P.short_convolution(u, w)[:, 0].tolist() == [1.0, 12.0, 123.0, 234.0, 345.0]
    assert P.sees(9, {"size": 3, "keep_first": 2}) == [0, 1, 7, 8, 9] and P.sees(1, {"size": 1, "keep_first": 4}) == [0, 1]
    x = torch.tensor([[[1.0, 0.0, 0.0, 2.0, 5.0]]], dtype=torch.float64)       # pairs (0, 2), (1, 3); the last passes
    got = P.rotate_halves(x, [1], {"dims": 4, "base": 16.0})[0, 0]
    a, b = 1.0, 0.25
    assert got.tolist() == pytest.approx([math.cos(a), -2 * math.sin(b), math.sin(a), 2 * math.cos(b), 5.0])
    m = {"q_temp": {"coef": 2.0, "every": 3}}
    assert P.query_temperature([0, 1, 2, 5], m, torch.float64).tolist() == pytest.approx(
        [1.0, 1.0, 1 + 2 * math.log(2), 1 + 2 * math.log(3)])
    one = torch.ones(2, dtype=torch.float64)
    assert float(P.map_weight({"lq1": one, "lk1": one * 0.5, "lq2": one, "lk2": one * 0}, 0.25)) == pytest.approx(math.e - 0.75)
    q = k = torch.tensor([[0.0], [10.0]], dtype=torch.float64)
    v = torch.tensor([[0.0], [1.0]], dtype=torch.float64)
    got = P.attend(q, k, v, 1.0, None, softcap=2.0)[1, 0]            # scores 0 and 2 tanh(50)
    assert float(got) == pytest.approx(1 / (1 + math.exp(-2.0)))
