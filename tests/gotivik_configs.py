"""Small Gotivik configurations and random weights for tests (none of them a real model's sizes).

The configurations differ from one another, and their layers among themselves, in every size: head counts from 1 to
20, one and several key/value heads, key and value sizes equal and different, multiples of 16 and not, windows from one
token to 130 with no, some, and more kept first tokens than the window is long, one to five convolution taps, plain and
rescaled rotations over all and part of a head, caps that bite and caps that do not, temperatures that grow at every
position and rarely, layers without a feed-forward, layers that run the weights of an earlier one, of a later one, and
through another such layer.
"""

from __future__ import annotations

import torch


def yarn(factor, original, fast, slow):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def window(heads, kv, dim, vdim, scale, taps, size, keep, rot, ff, **extra):
    """``rot``: ``(base, dims)`` or ``(base, dims, yarn(...))``."""
    r = {"base": rot[0], "dims": rot[1], **({"scaling": rot[2]} if len(rot) > 2 else {})}
    return {"type": "attention", "mlp": {"kind": "dense", "ff": ff} if ff else None, **extra,
            "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "conv": taps,
                      "mask": {"size": size, "keep_first": keep}, "rot": r}}


def differential(heads, kv, dim, vdim, scale, cap, diff, coef, every, ff, **extra):
    return {"type": "attention_2", "mlp": {"kind": "dense", "ff": ff} if ff else None, **extra,
            "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "softcap": cap,
                      "diff": diff, "q_temp": {"coef": coef, "every": every}}}


def again(layers, j):
    """An entry that runs layer ``j``'s weights."""
    return dict(layers[j], weights_of=j)


def config(layers, *, vocab, width, eps, mult):
    return {"architecture": "Gotivik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult,
            "layers": layers}


def _a():
    L = [window(4, 2, 12, 20, 0.4, 3, 9, 2, (50.0, 8, yarn(3.0, 40, 4.0, 0.5)), 40),
         differential(3, 1, 10, 14, 0.5, 3.0, 0.35, 0.4, 1, 28),
         differential(6, 3, 7, 9, 0.3, 30.0, 0.1, 0.2, 7, 0),
         window(5, 5, 6, 6, 0.5, 2, 17, 0, (10.0, 6), 24)]
    L += [again(L, 1), again(L, 0)]
    return config(L, vocab=59, width=48, eps=1e-5, mult=0.5)


def _b():
    # sizes the tensor-core kernels take: tcgen05 (64 and 128), mma.sync (48, 80), keys and values of two sizes
    L = [differential(4, 2, 32, 64, 0.2, 5.0, 0.3, 0.3, 16, 72),
         window(8, 2, 64, 64, 0.15, 4, 21, 5, (300.0, 32, yarn(2.0, 128, 8.0, 1.0)), 64),
         differential(6, 2, 24, 48, 0.25, 40.0, 0.2, 0.1, 3, 40),
         window(6, 1, 48, 48, 0.2, 3, 70, 66, (1000.0, 48), 48),
         differential(2, 1, 16, 96, 0.3, 2.0, 0.45, 0.5, 50, 56),
         window(4, 4, 32, 64, 0.25, 2, 130, 1, (100.0, 16), 40),
         differential(2, 2, 64, 128, 0.15, 50.0, 0.25, 0.2, 32, 64)]
    L += [again(L, 1), again(L, 0)]
    return config(L, vocab=61, width=64, eps=1e-6, mult=0.4)


def _c():
    # one tap (no state), windows of one and two tokens, kept tokens beyond the window, a chain of shared weights
    L = [window(2, 1, 6, 10, 0.5, 1, 1, 3, (7.0, 2), 0),
         differential(7, 7, 5, 6, 0.35, 1.5, 0.6, 0.7, 2, 28),
         window(20, 4, 10, 4, 0.35, 5, 2, 0, (100.0, 8, yarn(1.0, 30, 3.0, 1.0)), 20),
         window(2, 2, 8, 8, 0.3, 4, 5, 40, (50.0, 4, yarn(8.0, 16, 2.0, 0.9)), 0)]
    L += [dict(L[3], weights_of=5), again(L, 3), dict(L[1], weights_of=1), dict(L[1], weights_of=6)]
    return config(L, vocab=47, width=36, eps=1e-5, mult=1.0)


def _d():
    return config([differential(3, 3, 9, 11, 0.4, 4.0, 0.5, 0.3, 4, 21)], vocab=37, width=30, eps=1e-4, mult=0.7)


CONFIGS = {"A": _a(), "B": _b(), "C": _c(), "D": _d()}
PAGE_SIZE = {"A": 8, "B": 16, "C": 4, "D": 16}


def owner(cfg: dict, i: int) -> int:
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


def random_state(cfg: dict, seed: int) -> dict[str, torch.Tensor]:
    """Random weights as a checkpoint would hold them (values that bfloat16 represents exactly, so that both engine
    dtypes and the float64 plain implementation start from the same numbers)."""
    g = torch.Generator().manual_seed(seed)
    H = cfg["width"]

    def mat(*shape, std=None):
        std = std if std is not None else shape[-1] ** -0.5
        return (torch.randn(*shape, generator=g) * std).to(torch.bfloat16)

    def vec(n, mean=0.0, std=0.1):
        return (mean + torch.randn(n, generator=g) * std).to(torch.bfloat16)

    st = {"embed": mat(cfg["vocab"], H, std=1.0), "final.norm": vec(H, 1.0)}
    for i, layer in enumerate(cfg["layers"]):
        if owner(cfg, i) != i:
            continue
        p, m = f"l{i}.", layer["mixer"]
        names = ("norm1", "norm1b") + (("norm2", "norm2b") if layer["mlp"] else ())
        st.update({p + n: vec(H, 1.0, 0.3) for n in names})
        q, n, kv, d, dv = p + "mix.", m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        maps = 2 if layer["type"] == "attention_2" else 1
        rows = {"q": n * maps * d, "k": kv * maps * d, "v": kv * dv}
        st.update({q + a: mat(r, H, std=1.3 * H ** -0.5) for a, r in rows.items()})
        st[q + "o"] = mat(H, n * dv)
        if maps == 2:
            st.update({q + a: vec(d, 0.0, 0.3) for a in ("lq1", "lk1", "lq2", "lk2")})
            st[q + "g"] = mat(n, H, std=2.0 * H ** -0.5)
        elif m["conv"] >= 1:
            st.update({q + a + ".conv": mat(r, m["conv"], std=0.6) for a, r in rows.items()})
        if layer["mlp"]:
            ff = layer["mlp"]["ff"]
            st.update({p + "mlp.up": mat(ff, H, std=1.5 * H ** -0.5), p + "mlp.down": mat(H, ff)})
    return st


def prompt(cfg: dict, n: int, salt: int) -> list[int]:
    g = torch.Generator().manual_seed(7000 + salt)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()
