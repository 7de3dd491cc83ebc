"""The Gotivik architecture in the engine against the plain implementation (``plain_gotivik``): every mechanism alone
at the kernel level, then whole models of four small configurations under every way of cutting the work, in float32
and bfloat16, long decoding, and greedy generation through the scheduler.  Weights and inputs are made so that a fault
shows: one key that stands out at every edge of windows, kept tokens, chunks and pages, scores that a cap bites,
convolution states in slots between poisoned ones, caches and states filled with NaN where nothing was written, slots
and pages that are used again."""

import copy
import json
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_gotivik as P
import trace_util as T
from gotivik_configs import CONFIGS, PAGE_SIZE, config, differential, prompt, random_state, window, yarn

pytestmark = pytest.mark.gpu
DEV = "cuda:0"

LENGTHS = {"A": [3, 19, 64, 90, 41], "B": [150, 2, 37, 201, 70], "C": [50, 1, 33, 81], "D": [1, 2, 40, 17, 5]}


def ops():
    from mini_infer_b200.csrc import ops as o
    return o


def requests_for(which):
    return {f"r{i}": prompt(CONFIGS[which], n, salt=i) for i, n in enumerate(LENGTHS[which])}


_plain_cache = {}


def plain_for(which):
    if which not in _plain_cache:
        state = random_state(CONFIGS[which], seed=21)
        _plain_cache[which] = (state, {rid: P.gotivik_logits(state, CONFIGS[which], toks).numpy()
                                       for rid, toks in requests_for(which).items()})
    return _plain_cache[which]


def poisoned(runner):
    for st in runner.cache.storage:
        st.fill_(float("nan"))            # a slot that was never written must never be read
    for arena in runner.cache.state_arenas.values():
        arena.fill_(float("nan"))         # a state must be zeroed when its slot is handed out
    return runner


def make_runner(which, dtype, steps=None, num_blocks=None, max_requests=4, cuda_graph=False):
    from mini_infer_b200.engine import ModelRunner

    state, _ = plain_for(which)
    ps = PAGE_SIZE[which]
    if num_blocks is None:
        num_blocks = T.max_tokens_needed(steps) // ps
    return poisoned(ModelRunner.from_state_dict(CONFIGS[which], state, dtype=dtype, block_size=ps,
                                                num_blocks=num_blocks, max_requests=max_requests,
                                                cuda_graph=cuda_graph))


def bound_for(dtype, want):
    return T.tolerance(dtype, max(float(np.abs(w).max()) for w in want))


def compare(which, dtype, got):
    _, want = plain_for(which)
    tol = bound_for(dtype, want.values())
    for rid, w in want.items():
        assert got[rid].shape == w.shape
        assert np.isfinite(got[rid]).all(), f"{rid}: non-finite logits"
        bad = T.first_bad(got[rid], w, tol)
        assert bad is None, f"{which} {dtype} {rid}: position {bad} differs by " \
                            f"{np.abs(got[rid][bad] - w[bad]).max():.3g} (bound {float(tol):.3g})"


CUTTINGS = {"whole": T.cut_whole, "last_decoded": T.cut_last_decoded, "portions": T.cut_portions,
            "mixed": T.cut_mixed}


@pytest.mark.parametrize("cutting", list(CUTTINGS))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", list(CONFIGS))
def test_engine_matches_plain_under_every_cutting(which, dtype, cutting):
    """Whole prompts, prefill then token-by-token decoding, portions down to two tokens, and mixed batches of unequal
    requests in which slots and pages are freed and used again."""
    requests = requests_for(which)
    steps = CUTTINGS[cutting](requests)
    runner = make_runner(which, dtype, steps)
    got = T.collect(steps, T.replay_in_process(runner, steps), CONFIGS[which]["vocab"])
    runner.cache.check()
    assert runner.cache.num_requests == 0
    for gi, pool in enumerate(runner.cache.pools):
        assert runner.cache.num_free_pages(gi) == pool.num_pages
    compare(which, dtype, got)


@pytest.mark.parametrize("which", list(CONFIGS))
def test_float32_logits_do_not_depend_on_the_cutting(which):
    """In float32 every sum runs in an order that depends on the position alone: the logits of a position are the same
    bits whole, in portions, decoded, or beside other requests."""
    requests = requests_for(which)
    results = {}
    for name, cut in CUTTINGS.items():
        steps = cut(requests)
        runner = make_runner(which, "float32", steps)
        results[name] = T.collect(steps, T.replay_in_process(runner, steps), CONFIGS[which]["vocab"])
    for name in ("last_decoded", "portions", "mixed"):
        for rid in requests:
            assert np.array_equal(results[name][rid], results["whole"][rid]), f"{which} {name} {rid}"


@pytest.mark.parametrize("which,tokens", [("A", 200), ("B", 330), ("C", 200)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_and_captured_steps(which, tokens, dtype):
    """One short prompt, then everything else token by token over every window's end, kernel by kernel and as captured
    graphs."""
    from mini_infer_b200.engine import StepEntry

    cfg = CONFIGS[which]
    state, _ = plain_for(which)
    toks = prompt(cfg, tokens, salt=91)
    want = P.gotivik_logits(state, cfg, toks).numpy()
    tol = bound_for(dtype, [want])
    results = []
    for graph in (False, True):
        runner = make_runner(which, dtype, num_blocks=-(-tokens // PAGE_SIZE[which]), cuda_graph=graph)
        runner.add_request("a")
        rows = [runner.step([StepEntry("a", toks[:6], list(range(6)))]).logits.cpu().numpy()]
        for t in toks[6:]:
            rows.append(runner.step([StepEntry("a", [t], [0])]).logits.cpu().numpy())
        got = np.concatenate(rows)
        assert T.first_bad(got, want, tol) is None
        for gi, g in enumerate(runner.cache.groups):      # windows have given their pages back, the first ones are kept
            if g.window is not None:
                held = sum(p >= 0 for p in runner.cache.table("a", gi))
                assert held <= -(-g.window // PAGE_SIZE[which]) + 1 + -(-g.keep_first // PAGE_SIZE[which])
        runner.free_request("a")
        runner.cache.check()
        results.append(got)
    if dtype == "float32":
        assert np.array_equal(results[0], results[1])    # a captured step computes what the step itself does
    else:       # a captured step cuts the keys into runs for the longest context, the step itself for today's: rounding
        assert T.first_bad(results[0], results[1], tol) is None


def test_windowed_layers_decode_in_a_pool_of_their_window():
    """Windows with kept first tokens alone: a request runs far past its pool, on pages that come back."""
    from mini_infer_b200.engine import ModelRunner, StepEntry

    cfg = config([window(4, 2, 16, 16, 0.4, 3, 11, 6, (50.0, 8), 24), window(2, 1, 32, 32, 0.3, 4, 20, 3, (90.0, 16), 24)],
                 vocab=41, width=32, eps=1e-5, mult=0.6)
    state = random_state(cfg, seed=8)
    toks = prompt(cfg, 150, salt=4)
    want = P.gotivik_logits(state, cfg, toks).numpy()
    for dtype in ("float32", "bfloat16"):
        runner = poisoned(ModelRunner.from_state_dict(cfg, state, dtype=dtype, block_size=4, num_blocks=9, max_requests=1))
        runner.add_request("a")
        pieces = [toks[:7], toks[7:19], *([t] for t in toks[19:])]
        got = np.concatenate([runner.step([StepEntry("a", p, list(range(len(p))))]).logits.cpu().numpy() for p in pieces])
        assert T.first_bad(got, want, bound_for(dtype, [want])) is None


def test_greedy_generation_through_the_scheduler():
    """Greedy tokens from the engine's own entry point (scheduler, sampler, cache) equal the plain implementation's, fed
    its own tokens, for several prompts generated together."""
    from mini_infer_b200.engine import ContinuousScheduler, Request
    from mini_infer_b200.sampling import SamplingParams

    for which in ("A", "C"):
        cfg = CONFIGS[which]
        state, _ = plain_for(which)
        prompts = [prompt(cfg, n, salt=200 + i) for i, n in enumerate([4, 21, 9])]
        n_new = 14
        runner = make_runner(which, "float32", num_blocks=64)
        sched = ContinuousScheduler(runner, max_concurrent=3, max_tokens_per_step=16)
        results = sched.generate([Request(prompt=p, sampling_params=SamplingParams(), max_tokens=n_new) for p in prompts])
        sched.stop()
        for p, r in zip(prompts, results):
            assert len(r.tokens) == n_new
            check_greedy(state, cfg, p, r.tokens)
        runner.cache.check()
        assert runner.cache.num_requests == 0


def check_greedy(state, cfg, p, tokens):
    logits = P.gotivik_logits(state, cfg, list(p) + list(tokens))
    for i, tok in enumerate(tokens):
        row = logits[len(p) - 1 + i]
        top2 = torch.topk(row, 2).values
        if float(top2[0] - top2[1]) > 1e-3:         # the plain choice is not a close call
            assert tok == int(row.argmax()), f"after {len(p) + i} tokens"


def test_generation_from_a_model_folder(tmp_path):
    """A folder with config.json and model.safetensors through ``generate_ids``, the call behind the command line."""
    from mini_infer_b200.engine.api import generate_ids
    from mini_infer_b200.weights.safetensors_io import write_safetensors

    cfg = CONFIGS["D"]
    state = random_state(cfg, seed=21)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(tmp_path / "model.safetensors"), state)
    p = prompt(cfg, 11, salt=300)
    got = generate_ids(str(tmp_path), [p], max_tokens=6, dtype="float32", device=DEV)[0]
    check_greedy(state, cfg, p, got)


def test_first_tokens_of_a_sequence_and_slots_used_again():
    """A request's first tokens (alone, as a pair, as a longer prompt) start from empty convolutions whatever the slot
    held before: the same prompt gives the same logits in a fresh runner and in slots and pages that other requests
    have just left."""
    from mini_infer_b200.engine import StepEntry

    for which in ("A", "C"):
        cfg = CONFIGS[which]
        toks, other = prompt(cfg, 40, salt=5), prompt(cfg, 55, salt=6)
        fresh = make_runner(which, "float32", num_blocks=40)
        fresh.add_request("x")
        want = fresh.step([StepEntry("x", toks, list(range(len(toks))))]).logits.cpu().numpy()
        runner = make_runner(which, "float32", num_blocks=40, max_requests=2)
        for first in (1, 2, 17):
            for rid in ("p", "q"):                               # fill both slots and leave them
                runner.add_request(rid)
                runner.step([StepEntry(rid, other, [])])
            runner.free_request("q")
            runner.free_request("p")
            runner.add_request("a")
            rows = [runner.step([StepEntry("a", toks[:first], list(range(first)))]).logits.cpu().numpy(),
                    runner.step([StepEntry("a", toks[first:], list(range(len(toks) - first)))]).logits.cpu().numpy()]
            runner.free_request("a")
            assert np.array_equal(np.concatenate(rows), want), f"{which}: first portion of {first}"
        runner.cache.check()


# ----------------------------------------------------------------------------- mechanisms alone


def rnd(*shape, seed, scale=1.0, dtype=torch.float32):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * scale).to(dtype)


def i32(a):
    return torch.tensor(np.asarray(a, dtype=np.int32), device=DEV)


def ctx_for(q_lens, slots, held=None):
    """The part of a step context that the kernels around an attention read; tiles of 16 tokens, the last ones first
    (their order is the planner's business)."""
    starts = np.concatenate([[0], np.cumsum(q_lens)[:-1]]).astype(np.int32)
    tiles = [(b, t) for b, n in enumerate(q_lens) for t in range(0, n, 16)][::-1]
    tile_lists = (i32([b for b, _ in tiles]), i32([t for _, t in tiles]), len(tiles))
    positions = np.concatenate([np.arange(n) + h for n, h in zip(q_lens, held or [0] * len(q_lens))])
    return SimpleNamespace(q_start=i32(starts), q_len=i32(q_lens), state_slot=i32(slots), n_requests=len(q_lens),
                           n_tokens=int(sum(q_lens)), decode_only=all(n == 1 for n in q_lens), positions=i32(positions),
                           q_tiles=lambda n: tile_lists, scratch={})


def rotary(rot, d):
    from mini_infer_b200.parts import PartSpec, build_part

    sc = rot.get("scaling")
    scaling = {"type": "yarn", "factor": sc["factor"], "original_max_position_embeddings": sc["original"],
               "beta_fast": sc["fast"], "beta_slow": sc["slow"]} if sc else None
    part = build_part("position", PartSpec("rotary", {"head_dim": d, "theta": rot["base"], "rotary_dim": rot["dims"],
                                                      "span": "rotated", "scaling": scaling}))
    part.bind({}, torch.float32, torch.device(DEV))
    return part


def test_angles_of_far_positions():
    rot = {"base": 5000.0, "dims": 12, "scaling": yarn(4.0, 1000, 16.0, 1.0)}
    pos = [0, 1, 77, 4095, 999_999, 3_000_000]
    got = rotary(rot, 16).step_angles(SimpleNamespace(positions=i32(pos), scratch={})).double().cpu()
    freqs, mult = P.yarn_frequencies(rot)
    a = torch.tensor(pos, dtype=torch.float64)[:, None] * torch.tensor(freqs, dtype=torch.float64)
    want = torch.cat([a.sin(), a.cos()], dim=1) * mult
    assert (got - want).abs().max() <= 5e-7


CONV_SIZES = [(3, 1, 16, 16, 8), (2, 2, 24, 8, 16), (4, 2, 12, 20, 8), (3, 3, 7, 9, 4), (1, 1, 5, 300, 0), (2, 1, 128, 128, 24),
              (1, 1, 130, 5, 130)]


@pytest.mark.parametrize("nq,nkv,d,dv,rot", CONV_SIZES)
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5, 16])
@pytest.mark.parametrize("dtype,bound", [(torch.float32, 3e-6), (torch.bfloat16, 1e-2)])
def test_convolved_and_rotated_queries_keys_and_values_through_portions(nq, nkv, d, dv, rot, taps, dtype, bound):
    """Two requests of unequal portions (1, 2 and more tokens, across tiles and pages) in slots between poisoned ones,
    against the plain functions over the whole sequences; a state holds the last projected rows unrounded."""
    portions = [(1, 4), (2, 1), (17, 20), (1, 1), (1, 2), (40, 1), (3, 33)]
    C, page = (nq + nkv) * d + nkv * dv, 4
    w = rnd(C, taps, seed=11, scale=0.5)
    totals = [sum(p[r] for p in portions) for r in range(2)]
    xs = [rnd(n, C + 3, seed=12 + r, scale=2.0).to(dtype) for r, n in enumerate(totals)]     # three columns of something else
    rotp = {"base": 30.0, "dims": rot, "scaling": yarn(2.0, 40, 4.0, 1.0)} if rot else None
    part = rotary(rotp, d) if rot else None
    want = []
    for x in xs:
        y = P.short_convolution(x[:, :C].double(), w.double())
        pos = range(len(x))
        want.append((P.rotate_halves(y[:, :nq * d].reshape(-1, nq, d), pos, rotp).reshape(-1, nq * d),
                     P.rotate_halves(y[:, nq * d:(nq + nkv) * d].reshape(-1, nkv, d), pos, rotp),
                     y[:, (nq + nkv) * d:].reshape(-1, nkv, dv)))
    n_pages = sum(-(-n // page) for n in totals)
    pages = torch.randperm(n_pages, generator=torch.Generator().manual_seed(5)).tolist()
    table = [pages[:-(-totals[0] // page)], pages[-(-totals[0] // page):]]
    kc = torch.full((n_pages, nkv, page, d), float("nan"), dtype=dtype, device=DEV)
    vc = torch.full((n_pages, nkv, page, dv), float("nan"), dtype=dtype, device=DEV)
    state = torch.full((5, max(taps - 1, 1) * C), float("nan"), device=DEV)
    slots = [3, 1]
    state[slots] = 0.0
    at, got = [0, 0], [[], []]
    for p in portions:
        rows = torch.cat([xs[r][at[r]:at[r] + p[r]] for r in range(2)]).to(DEV)
        ctx = ctx_for(list(p), slots, at)
        where = [table[r][j // page] * page + j % page for r in range(2) for j in range(at[r], at[r] + p[r])]
        q = torch.full((sum(p), nq * d), float("nan"), dtype=dtype, device=DEV)
        before = rows.clone()
        ops().conv_rope_store(rows, q, w.t().contiguous().to(DEV), state if taps > 1 else None, ctx, nq, nkv, d, dv, rot=rot,
                              angles=part.step_angles(ctx) if rot else None, slots=i32(where), kcache=kc, vcache=vc)
        assert torch.equal(rows, before)
        got[0].append(q[:p[0]].double().cpu())
        got[1].append(q[p[0]:].double().cpu())
        at = [at[r] + p[r] for r in range(2)]
    keys, values = (ops().unpack_cache_pages(c).double().cpu() for c in (kc, vc))      # [slots, nkv, size]
    for r in range(2):
        where = [table[r][j // page] * page + j % page for j in range(totals[r])]
        for g, t in zip((torch.cat(got[r]), keys[where], values[where]), want[r]):
            assert (g - t).abs().max() <= bound * t.abs().max()
        if taps > 1:
            last = torch.cat([torch.zeros(taps, C), xs[r][:, :C].float()])[-(taps - 1):]
            assert torch.equal(state[slots[r]].cpu(), last.reshape(-1))
    assert torch.isnan(state[[0, 2, 4]]).all()             # nobody else's slot is touched
    free = sorted(set(range(n_pages * page)) - {table[r][j // page] * page + j % page for r in range(2) for j in range(totals[r])})
    assert torch.isnan(keys[free]).all() and torch.isnan(values[free]).all()


@pytest.mark.parametrize("nq,nkv,d,row,dv", [(4, 2, 8, 16, 16), (3, 1, 10, 32, 14), (6, 3, 7, 16, 9), (2, 2, 64, 128, 128),
                                             (8, 1, 24, 48, 300), (2, 1, 4, 16, 4)])
@pytest.mark.parametrize("M", [1, 9, 300])
@pytest.mark.parametrize("dtype,bound", [(torch.float32, 1e-6), (torch.bfloat16, 5e-3)])
def test_two_maps_into_rows_with_a_query_temperature(nq, nkv, d, row, dv, M, dtype, bound):
    page, coef, every = 8, 0.37, 5
    pos = ([0, 3, 4, 5, 9, 100, 4095, 1_000_000, 17] + list(range(20, 311)))[:M]
    width = 2 * (nq + nkv) * d + nkv * dv
    x = rnd(M, width + nq, seed=31).to(dtype)
    slots = torch.randperm(2 * M + 8, generator=torch.Generator().manual_seed(6))[:M].tolist()
    n_pages = -(-(2 * M + 8) // page)
    kc = torch.full((n_pages, nkv, page, row), float("nan"), dtype=dtype, device=DEV)
    vc = torch.full((n_pages, nkv, page, dv), float("nan"), dtype=dtype, device=DEV)
    q = torch.full((M, 2 * nq * row), float("nan"), dtype=dtype, device=DEV)
    k_off, v_off = 2 * nq * d, 2 * (nq + nkv) * d
    ops().split_maps_store(x.to(DEV), q, k_off, v_off, nq, nkv, d, row, dv, positions=i32(pos), temp_coef=coef, temp_every=every,
                           slots=i32(slots), kcache=kc, vcache=vc)
    temp = P.query_temperature(pos, {"q_temp": {"coef": coef, "every": every}}, torch.float64)
    qd = x[:, :k_off].double().reshape(M, nq, 2, d) * temp[:, None, None, None]
    want = torch.zeros(M, nq, 2, row, dtype=torch.float64)
    want[:, :, 0, :d], want[:, :, 1, d:2 * d] = qd[:, :, 0], qd[:, :, 1]
    assert (q.double().cpu() - want.reshape(M, -1)).abs().max() <= bound * want.abs().max()
    keys, values = ops().unpack_cache_pages(kc).cpu(), ops().unpack_cache_pages(vc).cpu()
    assert torch.equal(keys[slots][:, :, :2 * d], x[:, k_off:v_off].reshape(M, nkv, 2 * d))
    assert (keys[slots][:, :, 2 * d:] == 0).all()
    assert torch.equal(values[slots], x[:, v_off:v_off + nkv * dv].reshape(M, nkv, dv))
    rest = [s for s in range(n_pages * page) if s not in set(slots)]
    assert torch.isnan(keys[rest]).all() and torch.isnan(values[rest]).all()


@pytest.mark.parametrize("nq,dv", [(3, 16), (2, 64), (5, 96), (4, 128), (1, 14), (2, 9), (3, 256), (1, 512)])
@pytest.mark.parametrize("M", [1, 37])
@pytest.mark.parametrize("dtype,bound", [(torch.float32, 3e-6), (torch.bfloat16, 1e-2)])
def test_two_maps_combined_normed_and_gated(nq, dv, M, dtype, bound):
    """Heads so small that the epsilon counts and maps that nearly cancel, with and without the gate, also into a range
    of columns."""
    eps, lam, mult = 1e-5, 0.83, 0.65
    heads = rnd(M, nq, 2, dv, seed=41)
    heads[0, 0] *= 1e-3
    heads[-1, -1, 1] = heads[-1, -1, 0] * 1.1
    heads = heads.to(dtype)
    gate = rnd(M, nq + 2, seed=42, scale=3.0).to(dtype)
    o = heads[:, :, 0].double() - lam * heads[:, :, 1].double()
    plain = P.unit_rms(o, eps) * mult
    for with_gate in (False, True):
        wide = torch.full((M, nq * dv + 8), float("nan"), dtype=dtype, device=DEV)
        out = wide[:, 8:] if dv % 8 == 0 else torch.empty((M, nq * dv), dtype=dtype, device=DEV)
        ops().combine_maps(heads.reshape(M, -1).to(DEV), gate.to(DEV)[:, 1:nq + 1] if with_gate else None, out, nq, dv, lam, eps, mult)
        want = plain * torch.sigmoid(gate[:, 1:nq + 1].double())[:, :, None] if with_gate else plain
        assert (out.double().cpu().reshape(M, nq, dv) - want).abs().max() <= bound * want.abs().max()
        assert torch.isnan(wide[:, :8]).all()


@pytest.mark.parametrize("H", [7, 48, 328, 1000, 2048, 4096, 8192, 8200])
@pytest.mark.parametrize("dtype,bound", [(torch.float32, 3e-6), (torch.bfloat16, 1e-2)])
def test_the_norm_behind_a_branch_the_sum_and_the_next_norm(H, dtype, bound):
    """Both norms and the sum in one pass against the plain functions, all rows in place and some rows alone; branches
    so small that their epsilon counts."""
    from mini_infer_b200.parts import PartSpec, build_part
    from mini_infer_b200.parts.base import PendingBranch

    M, e1, e2, mult = 6, 1e-5, 1e-3, 0.4
    stream, y = rnd(M, H, seed=51, scale=2.0), rnd(M, H, seed=52, scale=0.01).to(dtype)
    g1, g2 = rnd(H, seed=53) * 0.3 + 1, rnd(H, seed=54) * 0.3 + 1
    behind = build_part("norm", PartSpec("branch_rmsnorm", {"hidden_size": H, "eps": e1, "mult": mult}))
    front = build_part("norm", PartSpec("rmsnorm", {"hidden_size": H, "eps": e2}))
    behind.bind({"weight": g1.to(DEV)}, dtype, torch.device(DEV))
    front.bind({"weight": g2.to(DEV)}, dtype, torch.device(DEV))
    r = stream.double() + mult * P.unit_rms(y.double(), e1) * g1.double()
    want = P.unit_rms(r, e2) * g2.double()
    dev = stream.to(DEV).clone()
    rows = i32([4, 0, 4])
    out, res = front.forward(PendingBranch.of(behind, y.to(DEV)), dev, rows=rows)
    assert res is None and torch.equal(dev.cpu(), stream)
    assert (out.double().cpu() - want[[4, 0, 4]]).abs().max() <= bound * want.abs().max()
    full, res = front.forward(PendingBranch.of(behind, y.to(DEV)), dev)
    assert res is dev and (dev.double().cpu() - r).abs().max() <= 3e-6 * r.abs().max()
    assert full.dtype == dtype and (full.double().cpu() - want).abs().max() <= bound * want.abs().max()
    assert torch.equal(full[[4, 0, 4]], out)


@pytest.mark.parametrize("M,I,H", [(1, 40, 64), (9, 136, 48), (16, 200, 256), (17, 64, 40), (200, 88, 64), (5, 21, 30)])
@pytest.mark.parametrize("dtype,bound", [(torch.float32, 1e-5), (torch.bfloat16, 2e-2)])
def test_squared_relu_unit(M, I, H, dtype, bound):
    """Both routes (the streaming product's epilogue, the kernel behind the product), large and small values."""
    from mini_infer_b200.parts import PartSpec, build_part

    W = {"up": rnd(I, H, seed=61, scale=2.0 * H ** -0.5).to(dtype), "down": rnd(H, I, seed=62, scale=0.2).to(dtype)}
    x = rnd(M, H, seed=63).to(dtype)
    x[0] *= 8.0
    part = build_part("feed_forward", PartSpec("activated_mlp", {"hidden_size": H, "intermediate_size": I, "activation": "relu2"}))
    assert set(part.param_decls()) == {"up", "down"}
    part.bind({k: v.to(DEV) for k, v in W.items()}, dtype, torch.device(DEV))
    W64 = {k: v.double() for k, v in W.items()}
    z = x.double() @ W64["up"].T
    act = ops().linear_activated(x.to(DEV), part.up, "relu2", part.act_params).double().cpu()
    want = torch.clamp(z, min=0) ** 2
    assert (act[z < -1e-2 * z.abs().max()] == 0).all() and (act - want).abs().max() <= bound * want.abs().max()
    got = part.forward(x.to(DEV), SimpleNamespace())
    want = P.squared_relu_unit(x.double(), W64)
    assert (got.double().cpu() - want).abs().max() <= bound * want.abs().max()


def dense_attention(q, k, v, scale, mask, cap):
    """All rows at once: ``q [T, nq, d]``, ``k [T, nkv, d]``, ``v [T, nkv, dv]``; the mask from ``plain_gotivik.sees``."""
    total, group = q.shape[0], q.shape[1] // k.shape[1]
    hidden = torch.ones(total, total, dtype=torch.bool)
    for i in range(total):
        hidden[i, P.sees(i, mask)] = False
    out = []
    for h in range(q.shape[1]):
        s = q[:, h] @ k[:, h // group].T * scale
        if cap:
            s = cap * torch.tanh(s / cap)
        out.append(torch.softmax(s.masked_fill(hidden, float("-inf")), dim=1) @ v[:, h // group])
    return torch.stack(out, dim=1)


def cut(total, kind):
    if kind == "whole":
        return [total]
    if kind == "decode":
        return [total - 100] + [1] * 100
    sizes, rest = [], total
    for s in (5, 2, 33, 1, 3, 29, 2, 17, 7, 1) * 20:
        if rest <= 0:
            break
        sizes.append(min(s, rest))
        rest -= sizes[-1]
    return sizes


# heads, key/value heads, key size, value size, page: the tcgen05 kernel (64, 128), mma.sync (other sizes, pages or groups),
# the kernel for keys and values of two sizes, the CUDA-core kernel
ATTENTIONS = [(8, 2, 64, 64, 16), (4, 1, 128, 128, 16), (2, 2, 64, 64, 8), (12, 1, 64, 64, 16), (6, 2, 48, 48, 4), (4, 1, 128, 128, 3),
              (2, 1, 256, 256, 16), (24, 1, 16, 16, 16), (4, 2, 32, 64, 16), (5, 1, 16, 96, 8), (3, 3, 12, 20, 8), (2, 1, 40, 40, 16)]
MASKS = [(None, 0), (1, 3), (9, 0), (40, 6), (64, 64), (70, 66), (21, 150), (130, 1)]


@pytest.mark.parametrize("sizes", ATTENTIONS)
@pytest.mark.parametrize("dtype,bound", [("float32", 2e-5), ("bfloat16", 2.5e-2)])
def test_windows_with_kept_tokens_and_capped_scores(sizes, dtype, bound):
    """Every query points at one key: just inside or just outside its window, the last kept token or the first that is
    not, a border of a chunk or a page, itself; scores far above the cap and far below it.  Two requests in one step, cut
    differently, so that single tokens run beside portions; pages that a window gives back go to the other request."""
    from mini_infer_b200.engine import ModelRunner, StepEntry

    nq, nkv, d, dv, page = sizes
    td = torch.float32 if dtype == "float32" else torch.bfloat16
    totals = {"a": 203, "b": 171}
    scale = 0.9 / d ** 0.5
    for case, (size, keep) in enumerate(MASKS):
        cap, strength = [(0.0, 9.0), (3.0, 8.0), (50.0, 14.0), (20.0, 90.0)][case % 4]
        layer = window(nq, nkv, d, dv, scale, 1, size or 999, keep, (10.0, 2), 0)
        cfg = config([layer], vocab=8, width=16, eps=1e-6, mult=1.0)
        data = {}
        for n, (rid, total) in enumerate(totals.items()):
            k = rnd(total, nkv, d, seed=60 + n)
            k = k / k.norm(dim=-1, keepdim=True) * d ** 0.5
            q = rnd(total, nq, d, seed=70 + n, scale=0.3)
            w = size or total
            for i in range(total):
                target = [i - w + 1, i - w, keep - 1, keep, i, 0, 63, 64, i - w + 2, (i // page) * page, (i // page) * page - 1,
                          i // 2][(i * 5 + i // 12) % 12]
                if 0 <= target <= i:
                    q[i] = k[target].repeat_interleave(nq // nkv, dim=0) * (strength / (scale * d))
            v = rnd(total, nkv, dv, seed=80 + n)
            q, k, v = (t.to(td) for t in (q, k, v))
            mask = {"size": size, "keep_first": keep} if size else None
            data[rid] = (torch.cat([q.flatten(1), k.flatten(1), v.flatten(1)], dim=1),
                         dense_attention(q.double(), k.double(), v.double(), scale, mask, cap))
        for kinds in (("whole", "whole"), ("decode", "portions"), ("portions", "decode")):
            runner = poisoned(ModelRunner.from_state_dict(cfg, random_state(cfg, seed=3), dtype=dtype, block_size=page,
                                                          num_blocks=sum(-(-t // page) for t in totals.values()), max_requests=2))
            mixer = runner.model.blocks[0].mixer
            mixer.s_cap = cap
            if size is None:
                mixer.s_window = None
            ones = torch.ones(1, data["a"][0].shape[1], device=DEV)
            at = dict.fromkeys(totals, 0)
            todo = {rid: cut(total, kind) for (rid, total), kind in zip(totals.items(), kinds)}
            got = {rid: [] for rid in totals}
            for rid in totals:
                runner.add_request(rid)
            while any(todo.values()):
                now = {rid: todo[rid].pop(0) for rid in totals if todo[rid]}
                ctx, caches, _, _ = runner.stepper.plan([StepEntry(rid, [0] * n, []) for rid, n in now.items()])
                runner.stepper.apply_table_updates(ctx)
                cache, M = caches[0], sum(now.values())
                x = torch.cat([data[rid][0][at[rid]:at[rid] + n] for rid, n in now.items()]).to(DEV)
                q = torch.empty((M, nq * d), dtype=td, device=DEV)
                ops().conv_rope_store(x, q, ones, None, ctx, nq, nkv, d, dv, rot=0, angles=None,
                                      slots=ctx.groups[cache.group].slots, kcache=cache.k, vcache=cache.v)
                out = torch.full((M, nq * dv), float("nan"), dtype=td, device=DEV)
                mixer._attend(q, out, cache, ctx)
                for rid, rows in zip(now, out.double().cpu().split(list(now.values()))):
                    got[rid].append(rows)
                    at[rid] += now[rid]
            runner.cache.check()
            for rid, total in totals.items():
                err = (torch.cat(got[rid]).reshape(total, nq, dv) - data[rid][1]).abs().amax(dim=(1, 2))
                bad = torch.nonzero(~(err <= bound * 3.0)).ravel().tolist()       # values reach about three
                assert not bad, (size, keep, cap, kinds, rid, bad[:6], err[bad[:6]].tolist())
