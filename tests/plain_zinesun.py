"""A plain, slow implementation of the Zinesun decoder, for tests only.

Whole sequences from position 0, no cache, no batching, loops over heads, tokens and experts, one
function per mechanism, sharing no code with the package under test.  Everything runs on the CPU in
the dtype of the tensors it is given (tests use float64).

Notation: ``h [T, width]`` is what a mixer or feed-forward reads; a stored ``[out, in]`` matrix ``W``
applied to rows is written ``h @ W.T``.  ``W`` in an argument list holds the tensors of one part under
their local names, ``m`` its part of the raw configuration.
"""

from __future__ import annotations

import math

import torch


# ------------------------------------------------------------------------------- small pieces


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """``x / sqrt(mean(x^2) + eps) * w`` over the last dimension."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w


def layer_norm(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor, eps: float) -> torch.Tensor:
    """``(x - mu) / sqrt(var + eps) * w + b``, ``var`` the mean of the squared deviations from ``mu``."""
    dev = x - x.mean(dim=-1, keepdim=True)
    return dev / torch.sqrt((dev * dev).mean(dim=-1, keepdim=True) + eps) * w + b


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.logaddexp(z, torch.zeros_like(z))


def xielu(z: torch.Tensor, p: torch.Tensor, q: torch.Tensor) -> torch.Tensor:
    """Positive side ``softplus(p) z^2 + z / 2``, negative side (and zero)
    ``(softplus(q) + 1/2) (e^z - 1 - z) + z / 2``."""
    neg = torch.clamp(z, max=0.0)                    # the other side's exponential must not overflow
    above = softplus(p) * z * z + 0.5 * z
    below = (0.5 + softplus(q)) * (torch.expm1(neg) - neg) + 0.5 * neg
    return torch.where(z > 0, above, below)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def rotate_pairs(x: torch.Tensor, positions, rot: dict) -> torch.Tensor:
    """``x [T, heads, d]``: of the first ``dims`` dimensions, ``2i`` and ``2i + 1`` are one pair ``(u, v)``,
    turned by ``a = p base^(-2i/dims)`` into ``(u cos a - v sin a, v cos a + u sin a)``."""
    dims, base = int(rot["dims"]), float(rot["base"])
    out = x.clone()
    p = torch.as_tensor(positions, dtype=x.dtype)
    for i in range(dims // 2):
        a = p * base ** (-2.0 * i / dims)
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def input_convolution(h: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """``h_t + sum_j w[:, j] h_(t - taps + 1 + j)``, nothing before the start: the last column of ``w``
    meets the current token."""
    T, taps = h.shape[0], w.shape[1]
    out = h.clone()
    for t in range(T):
        for j in range(taps):
            src = t - taps + 1 + j
            if src >= 0:
                out[t] = out[t] + w[:, j] * h[src]
    return out


# ------------------------------------------------------------------------------- mixer


def latent_rows(h: torch.Tensor, W: dict, m: dict, positions, eps: float):
    """What a token leaves for later ones: its normed latent ``c [T, kv_rank]`` and its rotated key part
    ``r [T, rot_dim]``, shared by the heads."""
    rank = int(m["kv_rank"])
    raw = h @ W["dkv"].T
    c = rms_norm(raw[:, :rank], W["dkv.norm"], eps)
    r = rotate_pairs(raw[:, None, rank:], positions, m["rot"])[:, 0]
    return c, r


def latent_queries(h: torch.Tensor, W: dict, m: dict, positions, eps: float):
    """``(unrotated [T, H, dim], rotated [T, H, rot_dim])``: queries through a low-rank, normed latent."""
    T, H, d, rd = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["rot_dim"])
    q = (rms_norm(h @ W["dq"].T, W["dq.norm"], eps) @ W["uq"].T).reshape(T, H, d + rd)
    return q[..., :d], rotate_pairs(q[..., d:], positions, m["rot"])


def latent_attention(h: torch.Tensor, W: dict, m: dict, positions, eps: float) -> torch.Tensor:
    """Keys and values are expanded per head from the latent rows; token ``i`` sees ``j`` with ``0 <= i - j <
    mask.size``; softmax over these; head ``a`` times ``sigmoid(W_g h)_a``; the heads side by side through ``W_o``."""
    T, H, d, dv = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["vdim"])
    size, scale = int(m["mask"]["size"]), float(m["scale"])
    qu, qr = latent_queries(h, W, m, positions, eps)
    c, r = latent_rows(h, W, m, positions, eps)
    k = (c @ W["uk"].T).reshape(T, H, d)
    v = (c @ W["uv"].T).reshape(T, H, dv)
    gate = torch.sigmoid(h @ W["g"].T)
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for a in range(H):
        for i in range(T):
            lo = max(0, i - size + 1)
            s = (k[lo:i + 1, a] @ qu[i, a] + r[lo:i + 1] @ qr[i, a]) * scale
            out[i, a] = (torch.softmax(s, dim=0) @ v[lo:i + 1, a]) * gate[i, a]
    return out.reshape(T, H * dv) @ W["o"].T


# ------------------------------------------------------------------------------- feed-forwards


def dense_unit(h: torch.Tensor, W: dict) -> torch.Tensor:
    return xielu(h @ W["up"].T, W["act"][0], W["act"][1]) @ W["down"].T


def choose_experts(z: torch.Tensor, top: int):
    """One token's logits: the ``top`` largest, their weights (the softmax over these alone), and how close
    the call was (the gap between the last one taken and the first one left)."""
    order = torch.sort(z, descending=True)
    ids = order.indices[:top]
    margin = float(order.values[top - 1] - order.values[top]) if top < z.shape[0] else math.inf
    return ids.tolist(), torch.softmax(z[ids], dim=0).tolist(), margin


def mixture_of_experts(h: torch.Tensor, W: dict, mlp: dict, margins: list | None = None) -> torch.Tensor:
    """``margins`` (a list) receives, per token, how close the router's call was."""
    z = h @ W["router"].T + W["router.b"]
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        ids, weights, margin = choose_experts(z[t], int(mlp["router"]["top"]))
        if margins is not None:
            margins.append(margin)
        for e, w in zip(ids, weights):
            x = h[t]
            act = silu(W[f"e{e}.gate"] @ x) * (W[f"e{e}.up"] @ x)
            out[t] = out[t] + w * (W[f"e{e}.down"] @ act)
    return out


# ------------------------------------------------------------------------------- the model


def part(state: dict, prefix: str) -> dict:
    return {k[len(prefix):]: v for k, v in state.items() if k.startswith(prefix)}


def depth_average(weights: torch.Tensor, results: list) -> torch.Tensor:
    """``sum_j weights[j] X_j`` over the embedding output and every layer's result so far."""
    assert weights.shape[0] == len(results)
    out = torch.zeros_like(results[0])
    for w, x in zip(weights, results):
        out = out + w * x
    return out


def zinesun_logits(state: dict, cfg: dict, tokens, dtype=torch.float64, streams: list | None = None,
                   margins: list | None = None) -> torch.Tensor:
    """Logits ``[T, vocab]`` of one sequence from position 0.  ``streams`` (a list) receives the residual
    stream after every layer's depth average, ``margins`` (a list) the routers' closest calls, layer by
    layer, token by token."""
    st = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in state.items()}
    eps = float(cfg["norm"]["eps"])
    positions = list(range(len(tokens)))
    x = st["embed"][torch.as_tensor(tokens, dtype=torch.long)] * float(cfg["embedding"]["scale"])
    results = [x]

    def norm(y, name):
        return layer_norm(y, st[name], st[name + ".b"], eps)

    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = input_convolution(x, st[p + "canon1"])
        y = latent_attention(h, part(st, p + "mix."), layer["mixer"], positions, eps)
        x = x + norm(y, p + "norm1") * st[p + "ls1"]
        mlp = layer.get("mlp")
        if mlp is not None:
            W = part(st, p + "mlp.")
            f = dense_unit(x, W) if mlp["kind"] == "dense" else mixture_of_experts(x, W, mlp, margins)
            x = x + norm(f, p + "norm2") * st[p + "ls2"]
        results.append(x)
        x = depth_average(st[p + "dwa"], results)
        if streams is not None:
            streams.append(x.clone())
    return norm(x, "final.norm") @ st["embed"].T
