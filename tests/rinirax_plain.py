"""Rinirax, written out plainly: one function per mechanism, whole sequences, no cache, float64
unless told otherwise. It shares nothing with the package; the engine is compared with it.

Notation: a sequence is T tokens; D the model width; H query heads in G key/value groups; dk the
query/key size of a head, dv its value size; tensors are a dict by checkpoint name; `p` is a
tensor-name prefix such as "l3.mix."; `m` is that mixer's entry of the configuration.
"""

from __future__ import annotations

import math

import torch


def lin(x: torch.Tensor, W: dict, name: str) -> torch.Tensor:
    """W x, plus the bias stored beside W when there is one."""
    y = x @ W[name].to(x.dtype).T
    return y + W[name + ".b"].to(x.dtype) if name + ".b" in W else y


def rms(x: torch.Tensor, eps: float, w: torch.Tensor | None = None) -> torch.Tensor:
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w.to(x.dtype)


def layer_norm(x: torch.Tensor, W: dict, name: str, eps: float) -> torch.Tensor:
    centred = x - x.mean(-1, keepdim=True)
    y = centred / torch.sqrt((centred * centred).mean(-1, keepdim=True) + eps)
    return y * W[name].to(x.dtype) + W[name + ".b"].to(x.dtype)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def causal_conv(u: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """u [T, C], w [C, K]: y_t = sum_j w[:, j] u_(t - K + 1 + j), nothing ahead of the start."""
    T, K = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for back in range(min(K, T)):
        y[back:] += u[: T - back] * w[:, K - 1 - back].to(u.dtype)
    return y


def frequencies(dims: int, base: float, scaling: dict | None, dtype) -> tuple[torch.Tensor, float]:
    """-> (angle per position of each pair, factor of cos and sin): base^(-2i / dims), or with `scaling`
    the blend of those with themselves divided by `factor`, by how often a pair turns over `original`
    positions."""
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=dtype)
    if scaling is None:
        return f, 1.0

    def dim_of(turns: float) -> float:
        return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(dim_of(scaling["fast"])), 0)
    hi = min(math.ceil(dim_of(scaling["slow"])), dims - 1)
    ramp = ((torch.arange(dims // 2, dtype=dtype) - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return f / scaling["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(scaling["factor"]) + 1.0


def rotate(x: torch.Tensor, rot: dict, interleaved: bool) -> torch.Tensor:
    """x [T, heads, d], its row t at position t: the first rot.dims dims of every head in pairs, (2i, 2i + 1)
    or (i, i + dims / 2), by the pair's angle; the other dims pass."""
    dims = rot["dims"]
    if dims == 0:
        return x
    f, amount = frequencies(dims, rot["base"], rot.get("scaling"), x.dtype)
    angle = torch.arange(x.shape[0], dtype=x.dtype)[:, None, None] * f
    c, s = torch.cos(angle) * amount, torch.sin(angle) * amount
    first = slice(0, dims, 2) if interleaved else slice(0, dims // 2)
    second = slice(1, dims, 2) if interleaved else slice(dims // 2, dims)
    u, v = x[..., first], x[..., second]
    y = x.clone()
    y[..., first], y[..., second] = u * c - v * s, v * c + u * s
    return y


def softmax_map(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, window: int | None = None) -> torch.Tensor:
    """One head: q [T, dk], k [T, dk], v [T, dv]; position i sees j <= i, and with a window only the last
    `window` of them. -> [T, dv]"""
    i, j = torch.arange(q.shape[0])[:, None], torch.arange(k.shape[0])[None, :]
    hidden = j > i
    if window is not None:
        hidden = hidden | (i - j >= window)
    return torch.softmax(((q @ k.T) * scale).masked_fill(hidden, -math.inf), dim=-1) @ v


def lambda_of(W: dict, p: str, diff: float, dtype) -> torch.Tensor:
    a, b, c, d = (W[p + name].to(dtype) for name in ("lq1", "lk1", "lq2", "lk2"))
    return torch.exp((a * b).sum()) - torch.exp((c * d).sum()) + diff


def projected_keys_values(h, W, p: str, m: dict) -> tuple[torch.Tensor, torch.Tensor]:
    """What a layer of differential attention keeps: keys [T, G, 2, dk] behind their convolution and
    rotation, values [T, G, dv] behind their convolution."""
    T, G, dk, dv = h.shape[0], m["kv_heads"], m["dim"], m["vdim"]
    k = causal_conv(lin(h, W, p + "k"), W[p + "k.conv"]).view(T, G * 2, dk)
    v = causal_conv(lin(h, W, p + "v"), W[p + "v.conv"]).view(T, G, dv)
    return rotate(k, m["rot"], True).view(T, G, 2, dk), v


def differential_heads(q, k, v, scale: float, lam, diff: float, eps: float) -> torch.Tensor:
    """q [T, H, 2, dk], k [T, G, 2, dk], v [T, G, dv]: per head the first map's output minus lambda times
    the second's, divided by its own root mean square, times (1 - diff). -> [T, H, dv]"""
    T, H = q.shape[:2]
    G, dv = v.shape[1:]
    out = torch.zeros(T, H, dv, dtype=q.dtype)
    for head in range(H):
        g = head // (H // G)
        a1, a2 = (softmax_map(q[:, head, i], k[:, g, i], v[:, g], scale) for i in (0, 1))
        out[:, head] = rms(a1 - lam * a2, eps) * (1.0 - diff)
    return out


def differential_attention(h, W, p: str, m: dict, eps: float, kept: tuple | None = None):
    """-> (branch, (keys, values)); `kept`: another layer's keys and values instead of own ones."""
    T, H, dk = h.shape[0], m["heads"], m["dim"]
    k, v = projected_keys_values(h, W, p, m) if kept is None else kept
    q = causal_conv(lin(h, W, p + "q"), W[p + "q.conv"]).view(T, H * 2, dk)
    q = rotate(q, m["rot"], True).view(T, H, 2, dk)
    o = differential_heads(q, k, v, m["scale"], lambda_of(W, p, m["diff"], h.dtype), m["diff"], eps)
    return lin(o.reshape(T, -1), W, p + "o"), (k, v)


def latent_attention(h, W, p: str, m: dict, eps: float) -> torch.Tensor:
    """Queries through a latent of their own; keys and values expanded from one latent per token, the
    rotated key part shared by the heads; the last `mask.size` positions are seen."""
    T, H, dn, dr, dv, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = lin(rms(lin(h, W, p + "dq"), eps, W[p + "dq.norm"]), W, p + "uq").view(T, H, dn + dr)
    down = lin(h, W, p + "dkv")
    c = rms(down[:, :rank], eps, W[p + "dkv.norm"])
    shared = rotate(down[:, None, rank:], m["rot"], False)
    q_rot = rotate(q[..., dn:], m["rot"], False)
    k, v = lin(c, W, p + "uk").view(T, H, dn), lin(c, W, p + "uv").view(T, H, dv)
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for head in range(H):
        out[:, head] = softmax_map(torch.cat([q[:, head, :dn], q_rot[:, head]], -1),
                                   torch.cat([k[:, head], shared[:, 0]], -1), v[:, head], m["scale"],
                                   (m.get("mask") or {}).get("size"))
    return lin(out.reshape(T, -1), W, p + "o")


def min_gru_states(z: torch.Tensor, u: torch.Tensor, S0: torch.Tensor | None = None) -> torch.Tensor:
    """z (gate logits) and u [T, C]: S_t = (1 - sigmoid(z_t)) S_(t-1) + sigmoid(z_t) candidate(u_t), the
    candidate being u + 1/2 from zero on and sigmoid(u) below. -> [T, C]"""
    keep, take = torch.sigmoid(-z), torch.sigmoid(z)
    candidate = torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
    S = torch.zeros(z.shape[1], dtype=z.dtype) if S0 is None else S0.clone()
    out = []
    for t in range(z.shape[0]):
        S = keep[t] * S + take[t] * candidate[t]
        out.append(S)
    return torch.stack(out)


def min_gru(h, W, p: str) -> torch.Tensor:
    S = min_gru_states(lin(h, W, p + "z"), lin(h, W, p + "x"))
    return lin(S * silu(lin(h, W, p + "g")), W, p + "o")


def xielu(z: torch.Tensor, p: torch.Tensor, q: torch.Tensor) -> torch.Tensor:
    rise, fall = torch.nn.functional.softplus(p.to(z.dtype)), torch.nn.functional.softplus(q.to(z.dtype))
    below = (0.5 + fall) * (torch.exp(z.clamp(max=0.0)) - 1.0 - z) + 0.5 * z
    return torch.where(z > 0, rise * z * z + 0.5 * z, below)


def dense(h, W, p: str) -> torch.Tensor:
    act = W[p + "act"]
    return lin(xielu(lin(h, W, p + "up"), act[0], act[1]), W, p + "down")


def route(z: torch.Tensor, correction: torch.Tensor, r: dict) -> tuple[torch.Tensor, torch.Tensor]:
    """z [T, experts] router logits -> (experts chosen [T, top], their weights): sigmoid scores, chosen by
    score + correction among the `keep` groups whose two largest choice scores sum highest, weighted by the
    scores over their sum, times `scale`."""
    s = torch.sigmoid(z)
    pick = s + correction.to(z.dtype)
    T, E = z.shape
    groups, keep = r["groups"]["count"], r["groups"]["keep"]
    by_group = pick.view(T, groups, E // groups)
    best = by_group.sort(-1, descending=True).values[..., :2].sum(-1).topk(keep, dim=-1).indices
    allowed = torch.zeros(T, groups, dtype=torch.bool).scatter(1, best, True)
    pick = pick.masked_fill(~allowed.repeat_interleave(E // groups, dim=1), -math.inf)
    chosen = pick.topk(r["top"], dim=-1).indices
    w = s.gather(1, chosen)
    return chosen, w / (w.sum(-1, keepdim=True) + 1e-20) * r["scale"]


def routed_experts(h, W, p: str, mlp: dict, chosen_out: list | None = None) -> torch.Tensor:
    r = mlp["router"]
    chosen, weight = route(lin(h, W, p + "router"), W[p + "correction"], r)
    if chosen_out is not None:
        chosen_out.append(chosen)
    out = torch.zeros_like(h)
    for e in range(r["experts"]):
        rows, place = (chosen == e).nonzero(as_tuple=True)
        if len(rows):
            y = lin(silu(lin(h[rows], W, p + f"e{e}.gate")) * lin(h[rows], W, p + f"e{e}.up"), W, p + f"e{e}.down")
            out[rows] += weight[rows, place][:, None] * y
    return out


def depth_average(history: list[torch.Tensor], weights: torch.Tensor) -> torch.Tensor:
    """sum_j weights[j] history[j] of the embedding output and every layer's result so far."""
    return sum(w * x for w, x in zip(weights.to(history[0].dtype), history))


def forward(tokens: list[int], W: dict, cfg: dict, dtype=torch.float64, layers_out: list | None = None) -> torch.Tensor:
    """Logits [T, vocab] of a whole sequence."""
    eps = cfg["norm"]["eps"]
    x = W["embed"].to(dtype)[torch.tensor(tokens)]
    history, kept = [x], {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = layer_norm(x, W, p + "norm1", eps)
        if layer["type"] == "attention":
            branch, kept[i] = differential_attention(h, W, p + "mix.", m, eps, kept.get(m.get("kv_from")))
        elif layer["type"] == "mingru":
            branch = min_gru(h, W, p + "mix.")
        elif layer["type"] == "latent_attention":
            branch = latent_attention(h, W, p + "mix.", m, eps)
        else:
            raise ValueError(layer["type"])
        mlp = layer.get("mlp")
        if mlp is not None:
            branch = branch + (dense(h, W, p + "mlp.") if mlp["kind"] == "dense" else routed_experts(h, W, p + "mlp.", mlp))
        history.append(x + branch)
        x = depth_average(history, W[p + "dwa"])
        if layers_out is not None:
            layers_out.append(x.clone())
    return layer_norm(x, W, "final.norm", eps) @ W["head"].to(dtype).T
