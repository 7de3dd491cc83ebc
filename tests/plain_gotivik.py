"""A plain, slow implementation of the Gotivik decoder, for tests only.

Whole sequences from position 0, no cache, no batching, loops over heads and tokens, one function per
mechanism, sharing no code with the package under test.  Everything runs on the CPU in the dtype of the
tensors it is given (tests use float64).

Notation: ``h [T, width]`` is what a mixer or feed-forward reads; a stored ``[out, in]`` matrix ``W`` applied
to rows is written ``h @ W.T``.  ``W`` in an argument list holds the tensors of one part under their local
names, ``m`` its part of the raw configuration.
"""

from __future__ import annotations

import math

import torch


# ------------------------------------------------------------------------------- small pieces


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """``x / sqrt(mean(x^2) + eps)`` over the last dimension."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def short_convolution(u: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """Per channel ``y_t = sum_j w[:, j] u_(t - taps + 1 + j)``, nothing before the start."""
    T, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for t in range(T):
        for j in range(taps):
            src = t - taps + 1 + j
            if src >= 0:
                y[t] = y[t] + w[:, j] * u[src]
    return y


def yarn_frequencies(rot: dict) -> tuple[list[float], float]:
    """``(frequency of each rotated pair, factor on cosines and sines)``.

    Pair ``i`` of ``dims / 2`` turns with ``base^(-2i/dims)``; with a rescale, pairs below ``lo`` keep that, pairs
    from ``hi`` on turn ``factor`` times slower and the ramp between is linear in ``i``; ``lo`` and ``hi`` are the
    (fractional) pairs that make ``fast`` and ``slow`` turns over the original length, rounded outwards."""
    dims, base = int(rot["dims"]), float(rot["base"])
    plain = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return plain, 1.0
    factor, original = float(sc["factor"]), float(sc["original"])

    def pair_with(turns: float) -> float:
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(pair_with(float(sc["fast"]))), 0)
    hi = min(math.ceil(pair_with(float(sc["slow"]))), dims - 1)
    out = []
    for i, f in enumerate(plain):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(factor) + 1.0


def rotate_halves(x: torch.Tensor, positions, rot: dict | None) -> torch.Tensor:
    """``x [T, heads, d]``: of the first ``dims`` dimensions, ``i`` and ``i + dims/2`` are one pair."""
    if not rot:
        return x
    freqs, mult = yarn_frequencies(rot)
    half = len(freqs)
    out = x.clone()
    p = torch.as_tensor(positions, dtype=x.dtype)
    for i, f in enumerate(freqs):
        c, s = (torch.cos(p * f) * mult)[:, None], (torch.sin(p * f) * mult)[:, None]
        u, v = x[..., i], x[..., half + i]
        out[..., i] = u * c - v * s
        out[..., half + i] = v * c + u * s
    return out


def sees(i: int, mask: dict | None) -> list[int]:
    """The positions that position ``i`` sees: itself and the ``size - 1`` before it, and the first ``keep_first``
    of the sequence; without a mask all up to ``i``."""
    if mask is None:
        return list(range(i + 1))
    size, keep = int(mask["size"]), int(mask["keep_first"])
    return [j for j in range(i + 1) if i - j < size or j < keep]


def attend(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, mask: dict | None,
           softcap: float | None = None) -> torch.Tensor:
    """One head: ``q, k [T, d]``, ``v [T, dv]``; softmax over what each position sees."""
    T = q.shape[0]
    out = torch.zeros(T, v.shape[1], dtype=q.dtype)
    for i in range(T):
        js = sees(i, mask)
        s = (k[js] @ q[i]) * scale
        if softcap is not None:
            s = softcap * torch.tanh(s / softcap)
        out[i] = torch.softmax(s, dim=0) @ v[js]
    return out


# ------------------------------------------------------------------------------- mixers


def window_attention(h: torch.Tensor, W: dict, m: dict, positions, eps: float) -> torch.Tensor:
    T, H, G = h.shape[0], int(m["heads"]), int(m["kv_heads"])
    proj = {}
    for name in ("q", "k", "v"):
        u = h @ W[name].T
        proj[name] = short_convolution(u, W[name + ".conv"]) if name + ".conv" in W else u
    q = rotate_halves(proj["q"].reshape(T, H, -1), positions, m.get("rot"))
    k = rotate_halves(proj["k"].reshape(T, G, -1), positions, m.get("rot"))
    v = proj["v"].reshape(T, G, -1)
    heads = [attend(q[:, a], k[:, a // (H // G)], v[:, a // (H // G)], float(m["scale"]), m.get("mask"))
             for a in range(H)]
    return torch.cat(heads, dim=1) @ W["o"].T


def map_weight(W: dict, diff: float) -> torch.Tensor:
    """What the second map is taken off with."""
    return torch.exp((W["lq1"] * W["lk1"]).sum()) - torch.exp((W["lq2"] * W["lk2"]).sum()) + diff


def query_temperature(positions, m: dict, dtype) -> torch.Tensor:
    t = m.get("q_temp")
    if not t:
        return torch.ones(len(positions), dtype=dtype)
    return torch.tensor([1.0 + float(t["coef"]) * math.log((p + 1) // int(t["every"]) + 1) for p in positions],
                        dtype=dtype)


def differential_attention(h: torch.Tensor, W: dict, m: dict, positions, eps: float) -> torch.Tensor:
    T, H, G, d = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
    q = (h @ W["q"].T).reshape(T, H, 2, d) * query_temperature(positions, m, h.dtype)[:, None, None, None]
    k = (h @ W["k"].T).reshape(T, G, 2, d)
    v = (h @ W["v"].T).reshape(T, G, -1)
    lam, diff, cap = map_weight(W, float(m["diff"])), float(m["diff"]), m.get("softcap")
    gate = torch.sigmoid(h @ W["g"].T)
    heads = []
    for a in range(H):
        b = a // (H // G)
        one, two = (attend(q[:, a, w], k[:, b, w], v[:, b], float(m["scale"]), None, cap) for w in (0, 1))
        heads.append(unit_rms(one - lam * two, eps) * (1.0 - diff) * gate[:, a:a + 1])
    return torch.cat(heads, dim=1) @ W["o"].T


MIXERS = {"attention": window_attention, "attention_2": differential_attention}


# ------------------------------------------------------------------------------- the model


def squared_relu_unit(h: torch.Tensor, W: dict) -> torch.Tensor:
    return torch.clamp(h @ W["up"].T, min=0.0) ** 2 @ W["down"].T


def _local(state: dict, prefix: str, dtype) -> dict:
    return {n[len(prefix):]: t.to(dtype) for n, t in state.items() if n.startswith(prefix)}


def owner_of(layers: list[dict], i: int) -> int:
    while layers[i].get("weights_of") is not None:
        i = int(layers[i]["weights_of"])
    return i


def gotivik_streams(state: dict, cfg: dict, tokens, dtype=torch.float64) -> list[torch.Tensor]:
    """The residual stream behind the embedding and behind every layer."""
    eps, mult = float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
    positions = list(range(len(tokens)))
    x = state["embed"].to(dtype)[torch.as_tensor(tokens)]
    streams = [x]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{owner_of(cfg['layers'], i)}."
        g = {n: state[p + n].to(dtype) for n in ("norm1", "norm1b", "norm2", "norm2b") if p + n in state}
        y = MIXERS[layer["type"]](unit_rms(x, eps) * g["norm1"], _local(state, p + "mix.", dtype), layer["mixer"],
                                  positions, eps)
        x = x + mult * unit_rms(y, eps) * g["norm1b"]
        if layer.get("mlp") is not None:
            y = squared_relu_unit(unit_rms(x, eps) * g["norm2"], _local(state, p + "mlp.", dtype))
            x = x + mult * unit_rms(y, eps) * g["norm2b"]
        streams.append(x)
    return streams


def gotivik_logits(state: dict, cfg: dict, tokens, dtype=torch.float64) -> torch.Tensor:
    x = gotivik_streams(state, cfg, tokens, dtype)[-1]
    return unit_rms(x, float(cfg["norm"]["eps"])) * state["final.norm"].to(dtype) @ state["embed"].to(dtype).T
