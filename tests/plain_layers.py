"""Plain, slow restatement of layer-list models (Talizen) for the tests: one function per mechanism, whole sequences, float64.

Nothing here is shared with the product path: no kernels, no cache, no batching, no code of the package.  Every function takes the
complete sequence of one request and returns a value per token.
"""
from __future__ import annotations

import torch

F = torch.float64


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def grouped_norm(x: torch.Tensor, w: torch.Tensor, groups: int, eps: float) -> torch.Tensor:
    """Every one of `groups` consecutive parts of the vector is divided by its own root mean square; w spans the whole vector."""
    parts = x.reshape(*x.shape[:-1], groups, x.shape[-1] // groups)
    return rms(parts, eps).reshape(x.shape) * w


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1 + torch.tanh((2 / torch.pi) ** 0.5 * (z + 0.044715 * z ** 3)))


def hgrn2_gates(z: torch.Tensor, lower: torch.Tensor) -> torch.Tensor:
    """Forget gate: the sigmoid of z squeezed into [lower, 1]."""
    return lower + (1 - lower) / (1 + torch.exp(-z))


def hgrn2_scan(q: torch.Tensor, f: torch.Tensor, v: torch.Tensor, state: torch.Tensor | None = None):
    """q, f [T, H, d], v [T, H, dv] -> o [T, H, dv] and the last state [H, d, dv].  What the gate forgets on channel d is replaced by v."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    out = []
    for t in range(T):
        S = f[t][:, :, None] * S + (1 - f[t])[:, :, None] * v[t][:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out), S


def hgrn2_mixer(h: torch.Tensor, w: dict, heads: int, dim: int, vdim: int, eps: float) -> torch.Tensor:
    T = h.shape[0]
    zq = h @ w["q"].T
    q = (zq / (1 + torch.exp(-zq))).reshape(T, heads, dim)
    f = hgrn2_gates(h @ w["f"].T + w["f.b"], w["lower"]).reshape(T, heads, dim)
    v = (h @ w["v"].T).reshape(T, heads, vdim)
    o, _ = hgrn2_scan(q, f, v)
    return (rms(o, eps) * w["norm"]).reshape(T, heads * vdim) @ w["o"].T


def causal_softmax_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float) -> torch.Tensor:
    """q, k [T, H, d], v [T, H, dv]: position i sees the keys 0 .. i."""
    T = q.shape[0]
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    s = s.masked_fill(torch.ones(T, T, dtype=torch.bool).triu(1), float("-inf"))
    return torch.einsum("hij,jhv->ihv", torch.softmax(s, -1), v)


def latent_mixer(h: torch.Tensor, w: dict, heads: int, dim: int, vdim: int, scale: float, eps: float) -> torch.Tensor:
    T = h.shape[0]
    c = rms(h @ w["dkv"].T, eps) * w["dkv.norm"]
    q = (h @ w["q"].T).reshape(T, heads, dim)
    k = (c @ w["uk"].T).reshape(T, heads, dim)
    v = (c @ w["uv"].T).reshape(T, heads, vdim)
    o = causal_softmax_attention(q, k, v, scale)
    gate = 1 / (1 + torch.exp(-(h @ w["g"].T)))
    return (o * gate[:, :, None]).reshape(T, heads * vdim) @ w["o"].T


def gated_mlp(h: torch.Tensor, w: dict) -> torch.Tensor:
    return (gelu_tanh(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def layer(x: torch.Tensor, spec: dict, w: dict, norm: dict) -> torch.Tensor:
    """Both sublayers read x as it is; their outputs are normalised before they are added."""
    m = spec["mixer"]
    mix = {k[4:]: v for k, v in w.items() if k.startswith("mix.")}
    if spec["type"] == "hgrn2":
        y = hgrn2_mixer(x, mix, m["heads"], m["dim"], m["vdim"], norm["eps"])
    elif spec["type"] == "latent_attention":
        y = latent_mixer(x, mix, m["heads"], m["dim"], m["vdim"], m["scale"], norm["eps"])
    else:
        raise ValueError(spec["type"])
    x = x + grouped_norm(y, w["norm1"], norm["groups"], norm["eps"])
    if spec["mlp"] is not None:
        y = gated_mlp(x, {k[4:]: v for k, v in w.items() if k.startswith("mlp.")})
        x = x + grouped_norm(y, w["norm2"], norm["groups"], norm["eps"])
    return x


def forward(cfg: dict, w: dict[str, torch.Tensor], tokens, dtype=F):
    """Logits [T, vocab] and the residual stream after every layer [layers, T, width] of one whole sequence."""
    w = {k: v.to(dtype) for k, v in w.items()}
    x = w["embed"][torch.as_tensor(list(tokens))]
    after = []
    for i, spec in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = layer(x, spec, {k[len(p):]: v for k, v in w.items() if k.startswith(p)}, cfg["norm"])
        after.append(x)
    x = grouped_norm(x, w["final.norm"], cfg["norm"]["groups"], cfg["norm"]["eps"])
    return x @ w["head"].T, torch.stack(after)


def greedy(cfg: dict, w: dict[str, torch.Tensor], prompt, n: int) -> tuple[list[int], list[float]]:
    """Greedy continuation by whole-sequence forwards, with the gap between the two best logits at every step."""
    ids, out, gaps = list(prompt), [], []
    for _ in range(n):
        lg = forward(cfg, w, ids)[0][-1]
        top = lg.topk(2).values
        out.append(int(lg.argmax()))
        gaps.append(float(top[0] - top[1]))
        ids.append(out[-1])
    return out, gaps
