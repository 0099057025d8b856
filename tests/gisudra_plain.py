"""Gisudra, written out plainly: one function per mechanism, whole sequences, no cache, float64
unless told otherwise. It shares nothing with the package; the engine is compared with it.

Notation: a sequence is T tokens; D the model width; H query heads in G key/value groups; dk the
query/key size of a head, dv its value size; N the rows of a recurrent head's state; tensors are a
dict by checkpoint name; `p` is a tensor-name prefix such as "l3.mix."; `m` is that mixer's entry of
the configuration.
"""

from __future__ import annotations

import math

import torch


def lin(x: torch.Tensor, W: dict, name: str) -> torch.Tensor:
    return x @ W[name].to(x.dtype).T


def rms(x: torch.Tensor, eps: float, w: torch.Tensor | None = None) -> torch.Tensor:
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w.to(x.dtype)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z * z * z)))


def gelu_erf(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def causal_conv(u: torch.Tensor, w: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """u [T, C], w [C, K]: y_t = b + sum_j w[:, j] u_(t - K + 1 + j), nothing ahead of the start."""
    T, K = u.shape[0], w.shape[1]
    y = b.to(u.dtype).expand(T, -1).clone()
    for back in range(min(K, T)):
        y[back:] += u[: T - back] * w[:, K - 1 - back].to(u.dtype)
    return y


def rotate(x: torch.Tensor, base: float, dims: int) -> torch.Tensor:
    """x [T, heads, d], row t at position t: the first `dims` dims in pairs (2i, 2i + 1), by t base^(-2i / dims)."""
    if dims == 0:
        return x
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=x.dtype)
    angle = torch.arange(x.shape[0], dtype=x.dtype)[:, None, None] * f
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    y = x.clone()
    y[..., 0:dims:2] = u * torch.cos(angle) - v * torch.sin(angle)
    y[..., 1:dims:2] = v * torch.cos(angle) + u * torch.sin(angle)
    return y


def visible(T: int, mask: dict | None) -> torch.Tensor:
    """[T, T]: whether position i (row) sees position j: the last `size`, and the first `keep_first`."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    sees = j <= i
    if mask is not None:
        sees = sees & ((i - j < mask["size"]) | (j < mask.get("keep_first", 0)))
    return sees


def softmax_head(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, sees: torch.Tensor) -> torch.Tensor:
    """One head: q [T, dk], k [T, dk], v [T, dv] -> [T, dv]."""
    return torch.softmax(((q @ k.T) * scale).masked_fill(~sees, -math.inf), dim=-1) @ v


def mixed_values(v: torch.Tensor, first: torch.Tensor | None, lam: torch.Tensor) -> torch.Tensor:
    """The values a layer keeps: its own, or (1 - lambda) of them and lambda of the first mixing layer's."""
    return v if first is None else (1.0 - lam.to(v.dtype)) * v + lam.to(v.dtype) * first


def attention(h, W, p: str, m: dict, eps: float, first: torch.Tensor | None) -> tuple[torch.Tensor, torch.Tensor]:
    """-> (branch, this layer's unmixed values [T, G, dv]). `first`: the first mixing layer's values, or None
    where this layer mixes nothing (it is the first, or its configuration says so)."""
    T, H, G, dk, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms(lin(h, W, p + "q").view(T, H, dk), eps, W[p + "q.norm"])
    k = rms(lin(h, W, p + "k").view(T, G, dk), eps, W[p + "k.norm"])
    own = lin(h, W, p + "v").view(T, G, dv)
    v = mixed_values(own, first, W.get(p + "vmix"))
    sees = visible(T, m.get("mask"))
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for head in range(H):
        g = head // (H // G)
        out[:, head] = softmax_head(q[:, head], k[:, g], v[:, g], m["scale"], sees)
    return lin(out.reshape(T, -1) * torch.sigmoid(lin(h, W, p + "g")), W, p + "o"), own


def latent_attention(h, W, p: str, m: dict, eps: float) -> torch.Tensor:
    """Keys and values expanded from one latent per token, the rotated key part shared by the heads."""
    T, H, dn, dr, dv, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = lin(h, W, p + "q").view(T, H, dn + dr)
    down = lin(h, W, p + "dkv")
    c = rms(down[:, :rank], eps, W[p + "dkv.norm"])
    base, dims = m["rot"]["base"], m["rot"]["dims"]
    shared, q_rot = rotate(down[:, None, rank:], base, dims), rotate(q[..., dn:], base, dims)
    k, v = lin(c, W, p + "uk").view(T, H, dn), lin(c, W, p + "uv").view(T, H, dv)
    sees = visible(T, m.get("mask"))
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for head in range(H):
        out[:, head] = softmax_head(torch.cat([q[:, head, :dn], q_rot[:, head]], -1),
                                    torch.cat([k[:, head], shared[:, 0]], -1), v[:, head], m["scale"], sees)
    return lin(out.reshape(T, -1) * torch.sigmoid(lin(h, W, p + "g")), W, p + "o")


def state_space(x: torch.Tensor, B: torch.Tensor, C: torch.Tensor, dt: torch.Tensor, A_log: torch.Tensor, D: torch.Tensor,
                S0: torch.Tensor | None = None) -> tuple[torch.Tensor, torch.Tensor]:
    """x [T, H, dv], B and C [T, G, N], dt [T, H] (behind the softplus): per head
    S_t = exp(-exp(A_log) dt_t) S_(t-1) + dt_t B_t x_t^T, y_t = S_t^T C_t + D x_t. -> (y [T, H, dv], S [H, N, dv])"""
    T, H, dv = x.shape
    G, N = B.shape[1:]
    S = torch.zeros(H, N, dv, dtype=x.dtype) if S0 is None else S0.clone()
    A, D = torch.exp(A_log.to(x.dtype)), D.to(x.dtype)
    of = torch.arange(H) // (H // G)
    out = []
    for t in range(T):
        b, c = B[t, of], C[t, of]  # [H, N]
        S = torch.exp(-A * dt[t])[:, None, None] * S + dt[t][:, None, None] * b[:, :, None] * x[t][:, None, :]
        out.append((c[:, :, None] * S).sum(1) + D[:, None] * x[t])
    return torch.stack(out), S


def gated_group_norm(y: torch.Tensor, z: torch.Tensor, groups: int, eps: float, w: torch.Tensor) -> torch.Tensor:
    """y silu(z), each of `groups` equal parts divided by its own root mean square, times w."""
    g = (y * silu(z)).view(y.shape[0], groups, -1)
    return rms(g, eps).reshape(y.shape) * w.to(y.dtype)


def mamba2(h, W, p: str, m: dict, eps: float) -> torch.Tensor:
    T, H, dv, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * dv
    z, xbc, dt = torch.split(lin(h, W, p + "in"), [inner, inner + 2 * G * N, H], dim=-1)
    xbc = silu(causal_conv(xbc, W[p + "conv"], W[p + "conv.b"]))
    x, B, C = torch.split(xbc, [inner, G * N, G * N], dim=-1)
    dt = softplus(dt + W[p + "dt_bias"].to(h.dtype))
    y, _ = state_space(x.view(T, H, dv), B.view(T, G, N), C.view(T, G, N), dt, W[p + "A_log"], W[p + "D"])
    return lin(gated_group_norm(y.reshape(T, inner), z, m["norm_groups"], eps, W[p + "norm"]), W, p + "o")


def dense(h, W, p: str) -> torch.Tensor:
    return lin(gelu_tanh(lin(h, W, p + "gate")) * lin(h, W, p + "up"), W, p + "down")


def route(z: torch.Tensor, top: int) -> tuple[torch.Tensor, torch.Tensor]:
    """z [T, experts] router logits -> (experts chosen [T, top], the softmax over the chosen logits)."""
    best = z.topk(top, dim=-1)
    return best.indices, torch.softmax(best.values, dim=-1)


def experts(h, W, p: str, mlp: dict, chosen_out: list | None = None) -> torch.Tensor:
    r = mlp["router"]
    chosen, weight = route(lin(h, W, p + "router") + W[p + "router.b"].to(h.dtype), r["top"])
    if chosen_out is not None:
        chosen_out.append(chosen)
    unit = lambda rows, name: lin(gelu_erf(lin(rows, W, p + name + ".up")), W, p + name + ".down")  # noqa: E731
    out = torch.zeros_like(h)
    for e in range(r["experts"]):
        rows, place = (chosen == e).nonzero(as_tuple=True)
        if len(rows):
            out[rows] += weight[rows, place][:, None] * unit(h[rows], f"e{e}")
    if mlp.get("shared") is not None:
        out = out + torch.sigmoid(lin(h, W, p + "shared.sg")) * unit(h, "shared")
    return out


def forward(tokens: list[int], W: dict, cfg: dict, dtype=torch.float64, layers_out: list | None = None) -> torch.Tensor:
    """Logits [T, vocab] of a whole sequence."""
    eps = cfg["norm"]["eps"]
    x = W["embed"].to(dtype)[torch.tensor(tokens)]
    first = None
    for i, layer in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
        h = rms(x, eps, W[p + "norm1"])
        if layer["type"] == "attention":
            mixes = bool(m.get("v_mix"))
            branch, own = attention(h, W, p + "mix.", m, eps, first if mixes else None)
            if mixes and first is None:
                first = own
        elif layer["type"] == "latent_attention":
            branch = latent_attention(h, W, p + "mix.", m, eps)
        elif layer["type"] == "mamba2":
            branch = mamba2(h, W, p + "mix.", m, eps)
        else:
            raise ValueError(layer["type"])
        x = x + branch
        if mlp is not None:
            h = rms(x, eps, W[p + "norm2"])
            x = x + (dense(h, W, p + "mlp.") if mlp["kind"] == "dense" else experts(h, W, p + "mlp.", mlp))
        if layers_out is not None:
            layers_out.append(x.clone())
    return rms(x, eps, W["final.norm"]) @ W["head"].to(dtype).T
