"""Small Zinesun configurations and random weights for tests (none of them a real model's sizes).

The configurations differ from one another, and their layers among themselves, in every size: head counts
from 1 to 20 (with and without a common divisor with the tensor-core kernel's rows), unrotated, rotated and
value sizes that are all different, latents of the queries below and above those of the keys, windows from 1
to 130 positions, one to five convolution taps, widths that are no multiple of 8 or 4, one expert per token
and all of them, layers without a feed-forward (also the first and the last one), one layer and several.
"""

from __future__ import annotations

import torch


def dense(ff):
    return {"kind": "dense", "ff": ff}


def experts(n, top, ff):
    return {"kind": "moe", "router": {"experts": n, "top": top}, "expert": {"ff": ff}}


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, window, scale, base, mlp):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
                      "mask": {"size": window}, "scale": scale, "rot": {"base": base, "dims": rot_dim}}}


def config(layers, *, vocab, width, eps, taps, scale):
    return {"architecture": "Zinesun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "canon": {"taps": taps},
            "embedding": {"scale": scale}, "layers": layers}


CONFIGS = {
    # small odd sizes: the CUDA-core attention kernel in both dtypes
    "A": config([latent(4, 12, 6, 20, 24, 18, 9, 0.3, 1000.0, dense(40)),
                 latent(3, 20, 4, 8, 40, 50, 17, 0.2, 30.0, experts(6, 2, 16)),
                 latent(5, 8, 10, 12, 16, 9, 30, 0.4, 500.0, None),
                 latent(1, 16, 2, 28, 36, 12, 64, 0.25, 10.0, experts(4, 4, 8))],
                vocab=59, width=48, eps=1e-5, taps=3, scale=3.5),
    # sizes the tensor-core attention kernel takes in bfloat16: groups that divide its rows and that do not
    "B": config([latent(6, 16, 16, 24, 32, 40, 21, 0.2, 10000.0, experts(8, 3, 16)),
                 latent(16, 32, 16, 16, 64, 24, 70, 0.15, 300.0, dense(72)),
                 latent(20, 24, 32, 32, 96, 56, 130, 0.12, 2000.0, experts(5, 1, 24))],
                vocab=61, width=64, eps=1e-6, taps=4, scale=1.0),
    # one tap (no state), windows of one and two tokens, layers without a feed-forward at both ends
    "C": config([latent(2, 6, 4, 10, 12, 20, 1, 0.5, 7.0, None),
                 latent(7, 10, 8, 6, 20, 14, 2, 0.35, 100.0, dense(28)),
                 latent(2, 14, 2, 18, 28, 16, 45, 0.3, 50.0, None)],
                vocab=47, width=36, eps=1e-5, taps=1, scale=0.5),
    # one layer, five taps, rows that are no whole number of four values
    "D": config([latent(3, 7, 6, 9, 15, 11, 12, 0.4, 20.0, dense(21))], vocab=37, width=30, eps=1e-4, taps=5, scale=2.0),
}

PAGE_SIZE = {"A": 8, "B": 16, "C": 4, "D": 16}


def random_state(cfg: dict, seed: int) -> dict[str, torch.Tensor]:
    """Random weights as a checkpoint would hold them (values that bfloat16 represents exactly, so
    that both engine dtypes and the float64 plain implementation start from the same numbers)."""
    g = torch.Generator().manual_seed(seed)
    H = cfg["width"]

    def mat(*shape, std=None):
        std = std if std is not None else shape[-1] ** -0.5
        return (torch.randn(*shape, generator=g) * std).to(torch.bfloat16)

    def vec(n, mean=0.0, std=0.1):
        return (mean + torch.randn(n, generator=g) * std).to(torch.bfloat16)

    st = {"embed": mat(cfg["vocab"], H, std=1.0), "final.norm": vec(H, 1.0), "final.norm.b": vec(H)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        n, d, rd, dv, rank, qr = (m[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank"))
        st.update({p + "norm1": vec(H, 1.0, 0.3), p + "norm1.b": vec(H, 0.0, 0.3), p + "ls1": vec(H, 0.8, 0.3),
                   p + "canon1": mat(H, cfg["canon"]["taps"], std=0.4),
                   p + "dwa": torch.cat([vec(i + 1, 0.0, 0.4), vec(1, 0.8, 0.1)])})
        q = p + "mix."
        st.update({q + "dq": mat(qr, H), q + "dq.norm": vec(qr, 1.0, 0.3), q + "uq": mat(n * (d + rd), qr),
                   q + "dkv": mat(rank + rd, H), q + "dkv.norm": vec(rank, 1.0, 0.3), q + "uk": mat(n * d, rank),
                   q + "uv": mat(n * dv, rank), q + "g": mat(n, H, std=2.0 * H ** -0.5), q + "o": mat(H, n * dv)})
        mlp = layer["mlp"]
        q = p + "mlp."
        if mlp is None:
            continue
        st.update({p + "norm2": vec(H, 1.0, 0.3), p + "norm2.b": vec(H, 0.0, 0.3), p + "ls2": vec(H, 0.8, 0.3)})
        if mlp["kind"] == "dense":
            st.update({q + "up": mat(mlp["ff"], H), q + "down": mat(H, mlp["ff"]), q + "act": vec(2, 0.3, 0.8)})
        else:
            ff, E = mlp["expert"]["ff"], mlp["router"]["experts"]
            st.update({q + "router": mat(E, H, std=3.0 * H ** -0.5), q + "router.b": vec(E, 0.0, 1.0)})
            for e in range(E):
                st.update({f"{q}e{e}.gate": mat(ff, H), f"{q}e{e}.up": mat(ff, H), f"{q}e{e}.down": mat(H, ff)})
    return st


def prompt(cfg: dict, n: int, salt: int) -> list[int]:
    g = torch.Generator().manual_seed(5000 + salt)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()
