"""The Zinesun architecture in the engine against the plain implementation (``plain_zinesun``): every
mechanism alone at the kernel level, then whole models of four small configurations under every way of
cutting the work, in float32 and bfloat16, long decoding, and greedy generation through the scheduler.
Weights and inputs are made so that a fault shows: a key that stands out just inside and just outside a
window and at page borders, convolution inputs in slots between poisoned ones, caches and states filled with
NaN where nothing was written, slots and pages that are used again."""

from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_zinesun as P
import trace_util as T
from zinesun_configs import CONFIGS, PAGE_SIZE, config, latent, prompt, random_state

pytestmark = pytest.mark.gpu
DEV = "cuda:0"

LENGTHS = {"A": [3, 19, 64, 90, 41], "B": [150, 2, 37, 201, 70], "C": [50, 1, 33, 81], "D": [1, 2, 40, 17, 5]}
# A router logit this close to the first one left out is a close call: the other expert is as good an answer,
# and through keys, convolutions and depth averages it reaches the tokens behind.  In float32 a request is
# compared up to its first close call; in bfloat16, where they are many, every row whose own routing is none.
CLOSE_CALL = {"float32": 2e-4, "bfloat16": 0.05}


def ops():
    from mini_infer_b200.csrc import ops as o
    return o


def requests_for(which):
    return {f"r{i}": prompt(CONFIGS[which], n, salt=i) for i, n in enumerate(LENGTHS[which])}


_plain_cache = {}


def plain_with_margins(state, cfg, toks):
    m = []
    logits = P.zinesun_logits(state, cfg, toks, torch.float64, margins=m).numpy()
    n_moe = sum(1 for l in cfg["layers"] if l["mlp"] and l["mlp"]["kind"] == "moe")
    margin = np.array(m).reshape(n_moe, len(toks)).min(axis=0) if n_moe else np.full(len(toks), np.inf)
    return logits, margin


def plain_for(which):
    """float64 logits of every request, and per request and position its closest router call."""
    if which not in _plain_cache:
        state = random_state(CONFIGS[which], seed=21)
        logits, margins = {}, {}
        for rid, toks in requests_for(which).items():
            logits[rid], margins[rid] = plain_with_margins(state, CONFIGS[which], toks)
        _plain_cache[which] = (state, logits, margins)
    return _plain_cache[which]


def poisoned(runner):
    for st in runner.cache.storage:
        st.fill_(float("nan"))            # a slot that was never written must never be read
    for arena in runner.cache.state_arenas.values():
        arena.fill_(float("nan"))         # a state must be zeroed when its slot is handed out
    return runner


def make_runner(which, dtype, steps=None, num_blocks=None, max_requests=4, cuda_graph=False):
    from mini_infer_b200.engine import ModelRunner

    state, _, _ = plain_for(which)
    ps = PAGE_SIZE[which]
    if num_blocks is None:
        num_blocks = T.max_tokens_needed(steps) // ps
    return poisoned(ModelRunner.from_state_dict(CONFIGS[which], state, dtype=dtype, block_size=ps,
                                                num_blocks=num_blocks, max_requests=max_requests,
                                                cuda_graph=cuda_graph))


def compare(which, dtype, got):
    _, want, margins = plain_for(which)
    scale = max(float(np.abs(w).max()) for w in want.values())
    tol = T.tolerance(dtype, scale)
    checked = total = over = far_over = 0
    for rid, w in want.items():
        assert got[rid].shape == w.shape
        close = margins[rid] < CLOSE_CALL[dtype]
        total += len(w)
        assert np.isfinite(got[rid]).all(), f"{rid}: non-finite logits"
        if dtype == "bfloat16":
            keep = np.nonzero(~close)[0]
            checked += len(keep)
            err = np.abs(got[rid][keep] - w[keep]).max(axis=1)
            over += int((err > float(tol)).sum())
            far_over += int((err > 4 * float(tol)).sum())
            continue
        keep = np.arange(int(np.nonzero(close)[0][0]) if close.any() else len(w))
        checked += len(keep)
        bad = T.first_bad(got[rid][keep], w[keep], tol)
        assert bad is None, f"{which} {dtype} {rid}: position {keep[bad]} differs by " \
                            f"{np.abs(got[rid][keep[bad]] - w[keep[bad]]).max():.3g} (bound {float(tol):.3g})"
    # another expert at an earlier token reaches a later row weakly; a wrong key, page or state moves most rows far
    assert over <= max(3, 0.08 * checked), f"{over} of {checked} rows are over the bound"
    assert far_over <= max(2, 0.02 * checked), f"{far_over} of {checked} rows are far over the bound"
    assert checked >= 0.5 * total, f"only {checked} of {total} rows were compared"


CUTTINGS = {"whole": T.cut_whole, "last_decoded": T.cut_last_decoded, "portions": T.cut_portions,
            "mixed": T.cut_mixed}


@pytest.mark.parametrize("cutting", list(CUTTINGS))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", list(CONFIGS))
def test_engine_matches_plain_under_every_cutting(which, dtype, cutting):
    """Whole prompts, prefill then token-by-token decoding, portions down to two tokens, and mixed
    batches of unequal requests in which slots and pages are freed and used again."""
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
    """In float32 every sum runs in an order that depends on the position alone: the logits of a
    position are the same bits whole, in portions, decoded, or beside other requests."""
    requests = requests_for(which)
    results = {}
    for name, cut in CUTTINGS.items():
        steps = cut(requests)
        runner = make_runner(which, "float32", steps)
        results[name] = T.collect(steps, T.replay_in_process(runner, steps), CONFIGS[which]["vocab"])
    for name in ("last_decoded", "portions", "mixed"):
        for rid in requests:
            assert np.array_equal(results[name][rid], results["whole"][rid]), f"{which} {name} {rid}"


@pytest.mark.parametrize("which,n_pages", [("A", 10), ("B", 11), ("C", 14)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_and_captured_steps(which, n_pages, dtype):
    """One short prompt, then 190 tokens one by one over every window's end, in a pool that holds a window's
    pages only, kernel by kernel and as captured graphs."""
    from mini_infer_b200.engine import StepEntry

    cfg = CONFIGS[which]
    state, _, _ = plain_for(which)
    toks = prompt(cfg, 196, salt={"A": 91, "B": 92, "C": 93}[which])
    want, margin = plain_with_margins(state, cfg, toks)
    close = margin < CLOSE_CALL[dtype]
    tol = T.tolerance(dtype, float(np.abs(want).max()))
    results = []
    for graph in (False, True):
        runner = make_runner(which, dtype, num_blocks=n_pages, cuda_graph=graph)
        runner.add_request("a")
        rows = [runner.step([StepEntry("a", toks[:6], list(range(6)))]).logits.cpu().numpy()]
        for t in toks[6:]:
            rows.append(runner.step([StepEntry("a", [t], [0])]).logits.cpu().numpy())
        got = np.concatenate(rows)
        if dtype == "float32":
            upto = int(np.nonzero(close)[0][0]) if close.any() else len(toks)
            assert upto > 60
            assert T.first_bad(got[:upto], want[:upto], tol) is None
        else:
            err = np.abs(got - want).max(axis=1)[~close]
            assert (err > float(tol)).mean() <= 0.08 and (err > 4 * float(tol)).mean() <= 0.02
        runner.free_request("a")
        runner.cache.check()
        results.append(got)
    if dtype == "float32":
        assert np.array_equal(results[0], results[1])    # a captured step computes what the step itself does
    else:       # a captured step cuts the keys into runs for the longest context, the step itself for today's: rounding
        assert (np.abs(results[0] - results[1]).max(axis=1)[~close] > float(tol)).mean() <= 0.05


def test_greedy_generation_through_the_scheduler():
    """Greedy tokens from the engine's own entry point (scheduler, sampler, cache) equal the plain
    implementation's, fed its own tokens, for several prompts generated together."""
    from mini_infer_b200.engine import ContinuousScheduler, Request
    from mini_infer_b200.sampling import SamplingParams

    which = "A"
    cfg = CONFIGS[which]
    state, _, _ = plain_for(which)
    prompts = [prompt(cfg, n, salt=200 + i) for i, n in enumerate([4, 21, 9])]
    n_new = 14
    runner = make_runner(which, "float32", num_blocks=32)
    sched = ContinuousScheduler(runner, max_concurrent=3, max_tokens_per_step=16)
    results = sched.generate([Request(prompt=p, sampling_params=SamplingParams(), max_tokens=n_new) for p in prompts])
    sched.stop()
    for p, r in zip(prompts, results):
        assert len(r.tokens) == n_new
        check_greedy(state, cfg, p, r.tokens)
    runner.cache.check()
    assert runner.cache.num_requests == 0


def check_greedy(state, cfg, p, tokens):
    seq = list(p)
    for tok in tokens:
        logits = P.zinesun_logits(state, cfg, seq, torch.float64)[-1]
        top2 = torch.topk(logits, 2).values
        if float(top2[0] - top2[1]) > 1e-3:         # the plain choice is not a close call
            assert tok == int(logits.argmax()), f"after {len(seq)} tokens"
        seq.append(tok)


def test_generation_from_a_model_folder(tmp_path):
    """A folder with config.json and model.safetensors through ``generate_ids``, the call behind the command line."""
    import json

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
    """A request's first tokens (alone, as a pair, as a longer prompt) start from empty convolution inputs
    whatever the slot held before: the same prompt gives the same logits in a fresh runner and in slots and
    pages that other requests have just left."""
    from mini_infer_b200.engine import StepEntry

    for which in ("A", "D"):
        cfg = CONFIGS[which]
        toks, other = prompt(cfg, 40, salt=5), prompt(cfg, 55, salt=6)
        fresh = make_runner(which, "float32", num_blocks=16)
        fresh.add_request("x")
        want = fresh.step([StepEntry("x", toks, list(range(len(toks))))]).logits.cpu().numpy()
        runner = make_runner(which, "float32", num_blocks=16, max_requests=2)
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


def ctx_for(q_lens, slots):
    """The part of a step context the state kernels read."""
    starts = np.concatenate([[0], np.cumsum(q_lens)[:-1]]).astype(np.int32)
    return SimpleNamespace(q_start=i32(starts), q_len=i32(q_lens), state_slot=i32(slots), n_requests=len(q_lens),
                           n_tokens=int(sum(q_lens)), decode_only=all(n == 1 for n in q_lens),
                           host_q_len=list(q_lens))


SIZES = [(48, torch.float32, 3e-6), (40, torch.bfloat16, 1e-2), (1000, torch.bfloat16, 1e-2), (7, torch.float32, 3e-6),
         (2050, torch.float32, 3e-6), (5, torch.bfloat16, 1e-2)]


@pytest.mark.parametrize("H,dtype,bound", SIZES)
def test_a_layer_norm_behind_its_branch_adds_to_the_stream(H, dtype, bound):
    """``stream += s * (layernorm(y) w + b)`` in fp32, in place or beside a stream that is kept, with the stream's
    copy in the compute dtype; the rows are so small that the epsilon counts, and far from a mean of zero."""
    from mini_infer_b200.parts import PartSpec, build_part

    M, eps = 13, 1e-5
    stream = rnd(M, H, seed=1, scale=3.0)
    y = (rnd(M, H, seed=2, scale=0.01) + 0.3).to(dtype)
    W = {"weight": rnd(H, seed=3, scale=0.3) + 1, "bias": rnd(H, seed=4), "scale": rnd(H, seed=5) * 0.7}
    part = build_part("norm", PartSpec("branch_layernorm", {"hidden_size": H, "eps": eps, "layer_scale": True}))
    part.bind({k: v.to(DEV) for k, v in W.items()}, dtype, torch.device(DEV))
    want = stream.double() + P.layer_norm(y.double(), W["weight"].double(), W["bias"].double(), eps) * W["scale"].double()
    tol = 1e-5 * want.abs().max()             # the deviations are a thirtieth of the values they are taken from
    dev = stream.to(DEV).clone()
    kept, copy = part.add_branch(dev, y.to(DEV), keep=True)
    assert torch.equal(dev.cpu(), stream) and (kept.cpu().double() - want).abs().max() <= tol
    out, copy = part.add_branch(dev, y.to(DEV))
    assert out is dev and torch.equal(dev, kept)
    assert copy.dtype == dtype and (copy.float().cpu().double() - want).abs().max() <= max(float(tol), bound * float(want.abs().max()))
    plain = build_part("norm", PartSpec("branch_layernorm", {"hidden_size": H, "eps": eps}))
    assert set(plain.param_decls()) == {"weight", "bias"}


@pytest.mark.parametrize("H,taps", [(48, 3), (7, 5), (1000, 4), (64, 1), (30, 2), (256, 16)])
@pytest.mark.parametrize("x_dtype,dtype,bound", [(torch.float32, torch.float32, 2e-6), (torch.float32, torch.bfloat16, 1e-2),
                                                 (torch.bfloat16, torch.bfloat16, 1e-2)])
def test_input_convolution_through_portions(H, taps, x_dtype, dtype, bound):
    """The convolution through portions of 1, 2 and more tokens, two requests of unequal portions side by side
    in slots between poisoned ones, against the plain function over the whole sequences; the state holds the
    last inputs unrounded."""
    portions = [(1, 4), (2, 1), (17, 20), (1, 1), (1, 2), (40, 1), (3, 33)]
    w = rnd(H, taps, seed=11, scale=0.5)
    totals = [sum(p[r] for p in portions) for r in range(2)]
    xs = [rnd(n, H, seed=12 + r, scale=2.0).to(x_dtype) for r, n in enumerate(totals)]
    want = [P.input_convolution(x.double(), w.double()) for x in xs]
    state = torch.full((5, max(taps - 1, 1), H), float("nan"), device=DEV)
    slots = [3, 1]
    state[slots] = 0.0
    at, got = [0, 0], [[], []]
    for p in portions:
        rows = torch.cat([xs[r][at[r]:at[r] + p[r]] for r in range(2)]).to(DEV)
        out = ops().input_conv(rows, w.t().contiguous().to(DEV), state if taps > 1 else None, ctx_for(list(p), slots), dtype)
        got[0].append(out[:p[0]].float().cpu().double())
        got[1].append(out[p[0]:].float().cpu().double())
        at = [at[r] + p[r] for r in range(2)]
    for r in range(2):
        g = torch.cat(got[r])
        assert (g - want[r]).abs().max() <= bound * want[r].abs().max()
        if taps > 1:
            assert torch.equal(state[slots[r]].cpu(), xs[r][totals[r] - taps + 1:].float())
    assert torch.isnan(state[[0, 2, 4]]).all()             # nobody else's slot is touched


@pytest.mark.parametrize("H,dtype,bound", SIZES)
@pytest.mark.parametrize("index,layers", [(0, 3), (1, 3), (2, 3), (4, 6), (9, 10), (0, 1)])
def test_depth_average_with_the_norm_and_the_next_convolution(H, dtype, bound, index, layers):
    """The average over the embedding's output and every result so far, the layer's last norm in front of it
    and, in a step of single tokens, the next layer's convolution behind it: against the plain functions, and
    bit-equal to the convolution's own kernel."""
    from mini_infer_b200.parts import PartSpec, build_part
    from mini_infer_b200.parts.base import LayerCache, PendingBranch, StreamCopy

    M, eps, taps = 6, 1e-5, 4
    results = [rnd(M, H, seed=30 + j) for j in range(index + 1)]          # X_0 ... X_index
    stream, y = rnd(M, H, seed=50), rnd(M, H, seed=51).to(dtype)
    W = {"weight": rnd(H, seed=52) + 1, "bias": rnd(H, seed=53), "scale": rnd(H, seed=54)}
    a = rnd(index + 2, seed=55)
    norm = build_part("norm", PartSpec("branch_layernorm", {"hidden_size": H, "eps": eps, "layer_scale": True}))
    norm.bind({k: v.to(DEV) for k, v in W.items()}, dtype, torch.device(DEV))
    part = build_part("stream", PartSpec("depth_average", {"hidden_size": H, "index": index, "layers": layers}))
    part.bind({"weights": a.to(DEV)}, dtype, torch.device(DEV))
    conv = build_part("input", PartSpec("causal_input_conv", {"hidden_size": H, "taps": taps}))
    w = rnd(H, taps, seed=56)
    conv.bind({"weight": w.to(DEV)}, dtype, torch.device(DEV))
    X = stream.double() + P.layer_norm(y.double(), W["weight"].double(), W["bias"].double(), eps) * W["scale"].double()
    want = P.depth_average(a.double(), [r.double() for r in results] + [X])
    before = rnd(M, taps - 1, H, seed=57)

    def run(following, decode_only, pending):
        first = results[0].to(DEV)
        history = torch.full((layers - 1, M, H), float("nan"), device=DEV)
        for j in range(index):
            history[j] = results[j + 1].to(DEV)
        ctx = ctx_for([1] * M, [4, 0, 7, 1, 2, 6])
        ctx.decode_only, ctx.scratch = decode_only, {"depth_results": history, "embedded": first}
        state = torch.full((8, taps - 1, H), float("nan"), device=DEV)
        state[ctx.state_slot.long()] = before.to(DEV)
        cache = LayerCache(input_state=state)
        s = stream.to(DEV).clone()
        x = PendingBranch.of(norm, y.to(DEV)) if pending else StreamCopy.of(None)
        out, res = part.forward(x, s, ctx, first, following=(conv, cache) if following else None)
        assert torch.equal(s.cpu(), stream) and torch.equal(first.cpu(), results[0])
        return out, res, history, state, ctx, cache

    out, res, history, state, ctx, cache = run(True, True, True)
    assert (res.cpu().double() - want).abs().max() <= 5e-6 * want.abs().max()
    if index < layers - 1:
        assert (history[index].cpu().double() - X).abs().max() <= 5e-6 * X.abs().max()
    assert torch.isnan(history[index + 1:]).all()
    for r in range(M):
        seq = torch.cat([before[r].double(), want[r:r + 1]])
        ref = P.input_convolution(seq, w.double())[-1]
        assert (out.prepared[r].float().cpu().double() - ref).abs().max() <= max(bound, 5e-6) * ref.abs().max()
    out2, res2, _, state2, ctx2, cache2 = run(False, True, True)
    assert out2.prepared is None and torch.equal(res2, res)
    h = conv.forward(res2, ctx2, cache2)
    assert torch.equal(h, out.prepared) and torch.equal(state2.nan_to_num(7.0), state.nan_to_num(7.0))
    out3, res3, *_ = run(True, False, True)                # a step with prompt portions leaves the convolution to the layer
    assert out3.prepared is None and torch.equal(res3, res)
    _, res4, *_ = run(False, False, False)                 # without a branch the stream itself is the layer's result
    want4 = P.depth_average(a.double(), [r.double() for r in results] + [stream.double()])
    assert (res4.cpu().double() - want4).abs().max() <= 5e-6 * want4.abs().max()


@pytest.mark.parametrize("M,I,H", [(1, 40, 64), (9, 136, 48), (16, 200, 256), (17, 64, 40), (200, 88, 64), (5, 21, 30)])
@pytest.mark.parametrize("dtype,bound", [(torch.float32, 1e-5), (torch.bfloat16, 2e-2)])
@pytest.mark.parametrize("pq", [(0.5, -1.0), (-2.0, 3.0)])
def test_dense_unit_with_xielu(M, I, H, dtype, bound, pq):
    """Both routes (the streaming product's epilogue, the kernel behind the product), pre-activations on both
    sides of zero, large and close to it, two different numbers for the sides."""
    from mini_infer_b200.parts import PartSpec, build_part

    W = {"up": rnd(I, H, seed=61, scale=2.0 * H ** -0.5).to(dtype), "down": rnd(H, I, seed=62, scale=0.2).to(dtype),
         "act": torch.tensor(pq)}
    x = rnd(M, H, seed=63).to(dtype)
    x[0] *= 8.0
    if M > 1:
        x[-1] *= 1e-2
    part = build_part("feed_forward", PartSpec("activated_mlp", {"hidden_size": H, "intermediate_size": I, "activation": "xielu"}))
    part.bind({k: v.to(DEV) for k, v in W.items()}, dtype, torch.device(DEV))
    z = x.double() @ W["up"].double().T
    assert (z > 3).any() and (z < -3).any()
    act = ops().linear_activated(x.to(DEV), part.up, "xielu", part.act_params).float().cpu().double()
    want = P.xielu(z, *W["act"].double())
    # a pre-activation is off by some roundings of its row's size, however small it is itself
    assert ((act - want).abs() <= bound * (want.abs() + z.abs().amax(dim=1, keepdim=True))).all()
    assert (act - want).abs().max() <= bound * want.abs().max()
    got = part.forward(x.to(DEV), SimpleNamespace())
    want = P.dense_unit(x.double(), {k: v.double() for k, v in W.items()})
    assert (got.float().cpu().double() - want).abs().max() <= bound * want.abs().max()


@pytest.mark.parametrize("E,top,ff,H,M", [(6, 2, 20, 40, 33), (8, 3, 16, 48, 150), (5, 1, 12, 36, 5), (4, 4, 16, 40, 9),
                                          (64, 6, 24, 64, 50), (16, 5, 88, 176, 40)])
@pytest.mark.parametrize("dtype,bound", [(torch.float32, 1e-5), (torch.bfloat16, 2e-2)])
def test_router_bias_and_softmax_over_the_chosen(E, top, ff, H, M, dtype, bound):
    """The bias on the logits decides choices and enters the weights; against the plain token loop."""
    from mini_infer_b200.parts import PartSpec, build_part

    x = rnd(M, H, seed=70).to(dtype)
    W = {"router": rnd(E, H, seed=71, scale=0.4).to(dtype), "router.b": rnd(E, seed=72, scale=2.0).to(dtype)}
    for e in range(E):
        W[f"e{e}.gate"] = rnd(ff, H, seed=100 + e, scale=0.3).to(dtype)
        W[f"e{e}.up"] = rnd(ff, H, seed=200 + e, scale=0.3).to(dtype)
        W[f"e{e}.down"] = rnd(H, ff, seed=300 + e, scale=0.2).to(dtype)
    W64 = {k: v.double() for k, v in W.items()}
    mlp = {"kind": "moe", "router": {"experts": E, "top": top}, "expert": {"ff": ff}}
    margins = []
    want = P.mixture_of_experts(x.double(), W64, mlp, margins)
    ok = torch.tensor(margins) > (1e-4 if dtype == torch.float32 else 1e-2)
    assert ok.sum() >= 0.6 * M
    if top < E:
        z = x.double() @ W64["router"].T
        moved = [set(P.choose_experts(z[t], top)[0]) != set(P.choose_experts(z[t] + W64["router.b"], top)[0]) for t in range(M)]
        assert sum(moved) >= 0.3 * M             # the bias counts
    part = build_part("feed_forward", PartSpec("routed_experts", {"hidden_size": H, "experts": E, "top": top, "expert_ff": ff,
                                                                 "activation": "silu", "scores": "chosen", "router_bias": True}))
    part.bind({k: v.to(DEV) for k, v in W.items()}, dtype, torch.device(DEV))
    out = part.forward(x.to(DEV), SimpleNamespace())
    assert (out.float().cpu().double() - want)[ok].abs().max() <= bound * max(1.0, want.abs().max())


@pytest.mark.parametrize("n,d,rd,dv,rank,qr", [(3, 7, 6, 9, 15, 11), (4, 12, 8, 20, 24, 40), (20, 24, 32, 32, 96, 56), (1, 16, 2, 28, 36, 12)])
@pytest.mark.parametrize("dtype,bound", [(torch.float32, 3e-6), (torch.bfloat16, 1e-2)])
def test_latent_rows_and_queries_through_a_latent(n, d, rd, dv, rank, qr, dtype, bound):
    """The cache row (normed latent, interleaved rotation of the key part), the queries' normed latent and their
    rotated parts, at positions from 0 to a million, against the plain functions."""
    M, H, eps, page = 9, 40, 1e-5, 4
    pos = [0, 1, 2, 3, 100, 101, 4095, 1000000, 8]
    m = {"heads": n, "dim": d, "rot_dim": rd, "kv_rank": rank, "rot": {"base": 300.0, "dims": rd}}
    proj = rnd(M, qr + rank + rd + 3, seed=80).to(dtype)
    cg, qg = rnd(rank, seed=81) + 1, rnd(qr, seed=82) + 1
    freq = torch.tensor([300.0 ** (-2.0 * i / rd) for i in range(rd // 2)], dtype=torch.float64, device=DEV)
    kc = torch.full((4, 1, page, rank + rd), float("nan"), dtype=dtype, device=DEV)
    slots = [5, 0, 15, 3, 8, 9, 1, 12, 7]
    cq = torch.full((M, qr), float("nan"), dtype=dtype, device=DEV)
    common = dict(positions=i32(pos), freq=freq, eps=eps, interleaved=True)
    ops().latent_prepare(proj.to(DEV), 0, 0, d + rd, d, qr, rank, rd, rd, c_gain=cg.to(DEV), qfull=None, slots=i32(slots),
                         kcache=kc, cq_gain=qg.to(DEV), cq_out=cq, **common)
    x = proj.double()
    # the plain functions project first; identity matrices make the packed columns their projections
    W = {"dkv": torch.eye(rank + rd, dtype=torch.float64), "dkv.norm": cg.double(), "dq": torch.eye(qr, dtype=torch.float64),
         "dq.norm": qg.double(), "uq": torch.eye(n * (d + rd), dtype=torch.float64)}
    c, r = P.latent_rows(x[:, qr:qr + rank + rd], W, m, pos, eps)
    rows = ops().unpack_cache_pages(kc).float().cpu().double().reshape(16, rank + rd)
    want = torch.cat([c, r], dim=1)
    assert (rows[slots] - want).abs().max() <= bound * want.abs().max()
    assert torch.isnan(rows[[s for s in range(16) if s not in slots]]).all()
    want = P.rms_norm(x[:, :qr], qg.double(), eps)
    assert (cq.float().cpu().double() - want).abs().max() <= bound * want.abs().max()
    q = rnd(M, n * (d + rd), seed=83).to(dtype)
    qfull = torch.full((M, n, rank + rd), float("nan"), dtype=dtype, device=DEV)
    ops().latent_prepare(q.to(DEV), 0, n, d + rd, d, 0, rank, rd, rd, c_gain=None, qfull=qfull, **common)
    want = P.rotate_pairs(q.double().reshape(M, n, d + rd)[:, :, d:], pos, m["rot"])
    assert (qfull[:, :, rank:].float().cpu().double() - want).abs().max() <= bound * want.abs().max()
    assert torch.isnan(qfull[:, :, :rank]).all()             # the mapped part is the next product's


def attention_runner(n_tokens, page, dtype, sizes, window):
    """A runner of one layer (``sizes``: heads, rotated part, latent) whose planner, pages and choice of kernel the
    kernel-level test borrows."""
    from mini_infer_b200.engine import ModelRunner

    n, rd, rank = sizes
    cfg = config([latent(n, 8, rd, 8, rank, 8, window, 1.0, 10.0, None)], vocab=8, width=16, eps=1e-12, taps=1, scale=1.0)
    return poisoned(ModelRunner.from_state_dict(cfg, random_state(cfg, seed=3), dtype=dtype, block_size=page,
                                                num_blocks=-(-n_tokens // page) + 1, max_requests=2))


# the tensor-core kernel in bfloat16 (keys a multiple of 16, latents of 32): groups of heads that divide its rows or not,
# and more heads than its rows; a latent it does not take
@pytest.mark.parametrize("sizes", [(6, 16, 32), (16, 16, 64), (20, 32, 96), (70, 16, 32), (3, 6, 20), (1, 64, 512)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_windows_page_borders_and_far_keys(dtype, sizes):
    """One token's latent points where the queries point, all others across; a query that sees it returns its
    row, one that does not returns the others'.  Windows of one token up to the whole sequence, the marked token
    at a page's last and first slot and at position 0, looked at from just inside and just outside the window and
    from hundreds of tokens behind; as one prompt, in portions, and one by one in a pool that gives pages back."""
    from mini_infer_b200.engine import StepEntry

    n, rd, rank = sizes
    td = torch.float32 if dtype == "float32" else torch.bfloat16
    unit = rank ** 0.5                                       # a latent (unit, 0, ...) is its own RMS norm

    def run(total, marked, page, window, portions):
        runner = attention_runner(total, page, dtype, sizes, window)
        mixer = runner.model.blocks[0].mixer
        assert mixer.window == window
        runner.add_request("a")
        rows = torch.zeros(total, rank + rd)
        rows[:, 1] = unit
        rows[marked, 1], rows[marked, 0] = 0.0, unit
        q = torch.zeros(total, n, rank + rd)
        q[:, :, 0] = 40.0 / unit
        outs, t0 = [], 0
        for cnt in portions:
            ctx, caches, _, _ = runner.stepper.plan([StepEntry("a", [0] * cnt, [])])
            runner.stepper.apply_table_updates(ctx)
            cache = caches[0]
            ops().latent_prepare(rows[t0:t0 + cnt].to(td).to(DEV), 0, 0, 1, 0, 0, rank, rd, 0, positions=ctx.positions,
                                 freq=None, c_gain=torch.ones(rank, device=DEV), eps=1e-12, qfull=None,
                                 slots=ctx.groups[cache.group].slots, kcache=cache.k)
            out = torch.full((cnt, n * rank), float("nan"), dtype=td, device=DEV)
            ops().attention_ext(q[t0:t0 + cnt].reshape(cnt, -1).to(td).to(DEV), out, cache, ctx, n, 1, rank + rd, rank, 1.0,
                                window=window, values_in_keys=True)
            outs.append(out.float().cpu().reshape(cnt, n, rank))
            t0 += cnt
        assert t0 == total
        runner.cache.check()
        out = torch.cat(outs)
        pos = torch.arange(total)
        seen = (pos >= marked) & (pos - marked < window)
        want = torch.zeros(total, rank)
        want[seen, 0] = unit
        want[~seen, 1] = unit
        bad = (out - want[:, None]).abs().amax(dim=(1, 2)) > 0.02 * unit
        assert not bad.any(), (page, window, marked, portions[:4], torch.nonzero(bad)[:5].ravel().tolist())

    def mixed(total):
        sizes_, rest = [], total
        for s in (5, 2, 13, 1, 3, 29, 2, 17, 7) * 10:
            if rest <= 0:
                break
            sizes_.append(min(s, rest))
            rest -= sizes_[-1]
        return sizes_

    cases = [(8, 15, 9), (8, 16, 1), (16, 31, 33), (4, 13, 2), (8, 0, 64), (16, 39, 30), (16, 2, 65), (8, 7, 200)]
    for page, marked, window in cases if rank < 512 else cases[2:6:3]:
        for portions in ([100], mixed(100), [36] + [1] * 64):
            run(100, marked, page, window, portions)
    for portions in ([420], [300] + [1] * 120, [130, 290]):
        run(420, 67, 16, 301, portions)                      # the window's edge lies 300 tokens behind


@pytest.mark.parametrize("n,dn,rd,dv,rank", [(2, 64, 32, 64, 64), (3, 128, 64, 128, 96), (16, 8, 8, 16, 32), (1, 72, 16, 96, 40),
                                             (5, 24, 0, 48, 24), (4, 120, 40, 80, 512)])
@pytest.mark.parametrize("window,sink", [(0, False), (1, False), (50, True), (200, False), (333, True)])
def test_prompt_portions_on_expanded_rows(n, dn, rd, dv, rank, window, sink):
    """The tcgen05 kernel on keys and values expanded from gathered cache rows: three requests of unequal portions
    in one step, one of them a single token that stays out of it, pages handed out from the far end and NaN
    everywhere else; per-head gates, sinks, and a key that stands out at the window's first position of one token,
    against the plain softmax over expanded keys."""
    o = ops()
    page, scale = 8, 0.7
    assert o.expanded_latent_supported(n, dn, rd, dv, rank)
    starts, portions = [0, 77, 301], [131, 1, 200]              # tokens held before, tokens brought
    lens = [a + b for a, b in zip(starts, portions)]
    width = rank + rd
    kc = torch.full((sum(-(-x // page) for x in lens) + 2, 1, page, width), float("nan"), dtype=torch.bfloat16, device=DEV)
    table = torch.full((4, 80), -1, dtype=torch.int32, device=DEV)
    table_rows, free = [2, 0, 3], list(range(kc.shape[0] - 1, 0, -1))
    w_k = rnd(n * dn, rank, seed=90, scale=rank ** -0.5).bfloat16()
    w_v = rnd(n * dv, rank, seed=91, scale=rank ** -0.5).bfloat16()
    M = sum(portions)
    q = rnd(M, n, dn + rd, seed=92, scale=(dn + rd) ** -0.5).bfloat16()
    gate = rnd(M, n, seed=93).bfloat16()
    sinks = torch.linspace(-2.0, 3.0, n, dtype=torch.float64) if sink else None
    rows = [rnd(x, width, seed=94 + i).bfloat16() for i, x in enumerate(lens)]
    if window > 1:      # request 2: the token at 301 + 150 points at the first key of its window, which stands out
        target = 451 - window + 1
        k = (w_k.double() @ rows[2][target, :rank].double()).reshape(n, dn)
        q[portions[0] + 1 + 150, :, :dn] = (k * 12.0 / (k * k).sum(dim=1, keepdim=True)).bfloat16()
    by_slot = o.unpack_cache_pages(kc)
    for i, x in enumerate(lens):
        first = max(0, starts[i] - window + 1) if window else 0
        held = []
        for p in range(-(-x // page)):
            held.append(free.pop())
            table[table_rows[i], p] = held[-1]
        slots = [held[j // page] * page + j % page for j in range(x)]
        keep = list(range(first, x))                             # what lies before every window was given back
        by_slot[[slots[j] for j in keep], 0] = rows[i][keep].to(DEV)
    kc.copy_(o.pack_cache_pages(by_slot, page))
    tiles = [(i, t) for i, x in enumerate(portions) if x > 1 for t in range(0, x, 128)][::-1]
    ctx = SimpleNamespace(
        groups=[SimpleNamespace(block_table=table, page_size=page, table_rows=i32(table_rows))], n_requests=3, n_single=1,
        q_start=i32(np.cumsum([0] + portions[:-1])), q_len=i32(portions), kv_len=i32(lens), host_q_len=portions, host_kv_len=lens,
        tiles={}, tiles_multi={128: (i32([t[0] for t in tiles]), i32([t[1] for t in tiles]), len(tiles))})
    lat = o.latent_gather(SimpleNamespace(group=0, k=kc), ctx, rank, rd, window)
    assert lat.rows.shape[0] % 64 == 0 and torch.isfinite(lat.rows).all()
    out = torch.full((M, n * dv), float("nan"), dtype=torch.bfloat16, device=DEV)
    o.attention_expanded(q.reshape(M, -1).to(DEV), out, lat, torch.cat([w_k, w_v]).to(DEV), ctx, n, dn, rd, dv, scale,
                         window=window, sinks=sinks.float().to(DEV) if sink else None, gate=gate.to(DEV))
    assert o.attention_tc_status() == 0
    got = out.float().cpu().double().reshape(M, n, dv)
    t0 = 0
    for i, (a, b) in enumerate(zip(starts, portions)):
        if b == 1:
            assert torch.isnan(got[t0]).all()                    # a single token's row is somebody else's
            t0 += b
            continue
        c, r = rows[i][:, :rank].double(), rows[i][:, rank:].double()
        k = (c @ w_k.double().T).reshape(-1, n, dn)
        v = (c @ w_v.double().T).reshape(-1, n, dv)
        qq = q[t0:t0 + b].double()
        s = (torch.einsum("thd,jhd->thj", qq[..., :dn], k) + torch.einsum("thd,jd->thj", qq[..., dn:], r)) * scale
        pos, j = torch.arange(a, a + b)[:, None], torch.arange(a + b)[None]
        seen = (j <= pos) & ((pos - j < window) if window else torch.ones_like(j <= pos))
        s = s.masked_fill(~seen[:, None], float("-inf"))
        if sink:
            s = torch.cat([s, sinks[None, :, None].expand(b, n, 1)], dim=2)
        p = torch.softmax(s, dim=2)[..., :a + b]
        want = torch.einsum("thj,jhd->thd", p, v) * torch.sigmoid(gate[t0:t0 + b].double())[..., None]
        err = (got[t0:t0 + b] - want).abs().amax(dim=(1, 2))
        assert err.max() <= 2e-2 * max(1.0, want.abs().max()), (i, torch.nonzero(err > 2e-2).ravel()[:5].tolist(), float(err.max()))
        t0 += b


@pytest.mark.parametrize("n,d,rd,dv,rank", [(16, 128, 64, 128, 512), (20, 24, 16, 40, 96), (3, 8, 16, 17, 32), (70, 16, 0, 8, 64)])
@pytest.mark.parametrize("lens,window,sink,act,per_head,out_scale", [
    ([1, 64, 65, 700, 3, 130], 0, True, "sigmoid", False, 1.0), ([90, 33, 1, 500], 65, False, "sigmoid", True, 1.0),
    ([40], 9, False, "silu", False, 0.6), ([1200, 7], 1, False, None, False, 1.5), (list(range(5, 21)), 0, True, "sigmoid", True, 1.0)])
def test_single_tokens_through_the_fused_products(n, d, rd, dv, rank, lens, window, sink, act, per_head, out_scale):
    """The query's mapping with its rotation, attention cut into runs of keys, and the runs' merge with expansion
    and gate, against the plain formulas (keys and values expanded), with NaN in every cache row no one may see."""
    o = ops()
    page, scale, M = 16, 0.6, len(lens)
    width = rank + rd
    kc = torch.full((sum(-(-x // page) for x in lens) + 1, 1, page, width), float("nan"), dtype=torch.bfloat16, device=DEV)
    table = torch.full((M + 2, 80), -1, dtype=torch.int32, device=DEV)
    table_rows, free = list(range(M + 1, 1, -1)), list(range(kc.shape[0] - 1, 0, -1))
    rows = [rnd(x, width, seed=40 + i).bfloat16() for i, x in enumerate(lens)]
    by_slot = o.unpack_cache_pages(kc)
    for i, x in enumerate(lens):
        held = [free.pop() for _ in range(-(-x // page))]
        table[table_rows[i], :len(held)] = i32(held)
        keep = list(range(max(0, x - window) if window else 0, x))
        by_slot[[held[j // page] * page + j % page for j in keep], 0] = rows[i][keep].to(DEV)
    kc.copy_(o.pack_cache_pages(by_slot, page))
    uk, uv = rnd(n, d, rank, seed=31, scale=rank ** -0.5).bfloat16(), rnd(n, dv, rank, seed=32, scale=rank ** -0.5).bfloat16()
    q = rnd(M, n, d + rd, seed=33, scale=(d + rd) ** -0.5).bfloat16()
    gate = rnd(M, n if per_head else n * dv, seed=34).bfloat16() if act else None
    sinks = torch.linspace(-2.0, 3.0, n, dtype=torch.float64) if sink else None
    pos = [x - 1 for x in lens]
    freq = torch.tensor([50.0 ** (-2.0 * i / rd) for i in range(rd // 2)], dtype=torch.float64)
    ctx = SimpleNamespace(
        groups=[SimpleNamespace(block_table=table, page_size=page, table_rows=i32(table_rows))], decode_only=True, n_tokens=M,
        q_start=i32(range(M)), q_len=i32([1] * M), kv_len=i32(lens), max_kv_len=max(lens), tiles={t: None for t in range(1, 17)})
    qd = q.reshape(M, -1).to(DEV)
    assert o.latent_decode_fusable(torch.bfloat16, ctx, n, d, rd, dv, rank, qd)
    for interleaved in (True, False):
        qfull = o.latent_query(qd, uk.transpose(1, 2).contiguous().to(DEV), n, d, rd, rd, positions=i32(pos), freq=freq.to(DEV),
                               interleaved=interleaved)
        qq = q.double()
        want_map = torch.einsum("tnd,ndr->tnr", qq[..., :d], uk.double())
        assert (qfull[..., :rank].float().cpu().double() - want_map).abs().max() <= 1e-2 * want_map.abs().max()
        order = list(range(rd)) if interleaved else [j for i in range(rd // 2) for j in (i, i + rd // 2)]
        turned = torch.zeros(M, n, rd, dtype=torch.float64)
        if rd:
            turned[..., order] = P.rotate_pairs(qq[..., d:][..., order], pos, {"dims": rd, "base": 50.0})
            assert (qfull[..., rank:].float().cpu().double() - turned).abs().max() <= 1e-2 * turned.abs().max()
        runs = o.attention_latent_runs(qfull.view(M, -1), SimpleNamespace(group=0, k=kc), ctx, n, width, rank, scale,
                                       window=window, sinks=sinks.float().to(DEV) if sink else None)
        out = torch.full((M, n * dv), float("nan"), dtype=torch.bfloat16, device=DEV)
        o.latent_value(runs, sinks.float().to(DEV) if sink else None, uv.to(DEV), out, n,
                       gate=gate.to(DEV) if act else None, act=act, scale=out_scale)
        got = out.float().cpu().double().reshape(M, n, dv)
        for i, x in enumerate(lens):
            lo = max(0, x - window) if window else 0
            c, r = rows[i][lo:, :rank].double(), rows[i][lo:, rank:].double()
            s = (torch.einsum("nr,jr->nj", want_map[i], c) + turned[i] @ r.T) * scale
            if sink:
                s = torch.cat([s, sinks[:, None]], dim=1)
            p = torch.softmax(s, dim=1)[:, :x - lo]
            want = torch.einsum("nj,jr,nvr->nv", p, c, uv.double()) * out_scale
            if act:
                g = gate[i].double().reshape(n, -1)
                want = want * torch.sigmoid(g) * (g if act == "silu" else 1.0)
            assert (got[i] - want).abs().max() <= 2e-2 * max(1.0, want.abs().max()), (i, x)


def test_configurations_take_both_attention_kernels():
    o = ops()
    taken = {which: [o.rows_attention_supported(l["mixer"]["heads"], 1, l["mixer"]["kv_rank"] + l["mixer"]["rot_dim"],
                                                l["mixer"]["kv_rank"], True) for l in cfg["layers"]]
             for which, cfg in CONFIGS.items()}
    assert all(taken["B"]) and not any(taken["A"] + taken["C"] + taken["D"])
