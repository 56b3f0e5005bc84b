"""Plain, slow restatement of layer-list models (Talizen, Vozinex, Nifalorn, Rigalorn) for the tests: one function per mechanism, whole sequences, float64.

Nothing here is shared with the product path: no kernels, no cache, no batching, no code of the package.  Every function takes the
complete sequence of one request and returns a value per token.
"""
from __future__ import annotations

import functools
import math

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


def layer_norm(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor, eps: float) -> torch.Tensor:
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def rotate_half(x: torch.Tensor, dims: int, base: float, pos: torch.Tensor) -> torch.Tensor:
    """x [T, H, d] at positions pos: dimension i < dims / 2 turns with dimension i + dims / 2, the rest stays."""
    n = dims // 2
    a = pos.to(x.dtype)[:, None] * base ** (-2 * torch.arange(n, dtype=x.dtype) / dims)
    c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
    u, v = x[..., :n], x[..., n:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], -1)


def window_mask(T: int, size: int, keep_first: int) -> torch.Tensor:
    """[query, key]: the last `size` keys up to the query itself, and the first `keep_first` of the sequence."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None]
    return (j <= i) & ((i - j < size) | (j < keep_first))


def masked_softmax_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, seen: torch.Tensor) -> torch.Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, dv]: consecutive groups of H / G query heads share a key / value head."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = torch.empty(T, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        s = (q[:, h] @ k[:, h // (H // G)].T * scale).masked_fill(~seen, float("-inf"))
        out[:, h] = torch.softmax(s, -1) @ v[:, h // (H // G)]
    return out


def attention_mixer(h: torch.Tensor, w: dict, m: dict, eps: float) -> torch.Tensor:
    """Grouped-query attention: q and k are normalised over the whole projection, then rotated; sliding window with kept first tokens."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    pos = torch.arange(T)
    q = (rms(h @ w["q"].T, eps) * w["q.norm"]).reshape(T, H, m["dim"])
    k = (rms(h @ w["k"].T, eps) * w["k.norm"]).reshape(T, G, m["dim"])
    q, k = (rotate_half(x, m["rot"]["dims"], m["rot"]["base"], pos) for x in (q, k))
    v = (h @ w["v"].T).reshape(T, G, m["vdim"])
    o = masked_softmax_attention(q, k, v, m["scale"], window_mask(T, m["mask"]["size"], m["mask"]["keep_first"]))
    return o.reshape(T, H * m["vdim"]) @ w["o"].T


def route(h: torch.Tensor, w: torch.Tensor, b: torch.Tensor, top: int):
    """Chosen experts [T, top] and their weights: softmax over the chosen logits only."""
    z, ids = (h @ w.T + b).sort(dim=-1, descending=True, stable=True)
    return ids[:, :top], torch.softmax(z[:, :top], -1)


def expert(h: torch.Tensor, up: torch.Tensor, down: torch.Tensor) -> torch.Tensor:
    return torch.clamp(h @ up.T, min=0) ** 2 @ down.T


def moe_mlp(h: torch.Tensor, w: dict, top: int) -> torch.Tensor:
    ids, p = route(h, w["router"], w["router.b"], top)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, x in zip(ids[t].tolist(), p[t]):
            out[t] += x * expert(h[t], w[f"e{e}.up"], w[f"e{e}.down"])
    return out


def silu(z: torch.Tensor) -> torch.Tensor:
    return z / (1 + torch.exp(-z))


def sigmoid(z: torch.Tensor) -> torch.Tensor:
    return 1 / (1 + torch.exp(-z))


def decayed_scan(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: torch.Tensor, state: torch.Tensor | None = None):
    """q, k [T, H, d], v [T, H, dv], decay [T, H] -> o [T, H, dv] and the last state [H, d, dv]: one factor per head and token, no other scale."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    out = []
    for t in range(T):
        S = decay[t][:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out), S


def lightning_mixer(h: torch.Tensor, w: dict, m: dict, eps: float) -> torch.Tensor:
    """A constant decay per head; all heads share one root mean square, then the gate."""
    T, H = h.shape[0], m["heads"]
    q, k, v = (silu(h @ w[n].T).reshape(T, H, -1) for n in ("q", "k", "v"))
    o, _ = decayed_scan(q, k, v, torch.tensor(m["decay"], dtype=h.dtype).expand(T, H))
    return (rms(o.reshape(T, -1), eps) * w["norm"] * sigmoid(h @ w["g"].T)) @ w["o"].T


def causal_conv(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor, before: torch.Tensor | None = None) -> torch.Tensor:
    """x [T, channels], w [channels, taps]: every channel on its own, the last tap belongs to the token itself; `before`: the taps - 1 inputs in front."""
    T, taps = x.shape[0], w.shape[1]
    x = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=x.dtype) if before is None else before, x])
    return torch.stack([(x[t:t + taps] * w.T).sum(0) + b for t in range(T)])


def mamba2_steps(z: torch.Tensor, dt_bias: torch.Tensor, A_log: torch.Tensor):
    """Step sizes (softplus) and decays [T, H]."""
    dt = torch.log1p(torch.exp(-z.add(dt_bias).abs())) + torch.clamp(z + dt_bias, min=0)
    return dt, torch.exp(-torch.exp(A_log) * dt)


def mamba2_mixer(h: torch.Tensor, w: dict, m: dict, eps: float) -> torch.Tensor:
    T, H, V, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * V
    z, xbc, dt = (h @ w["in"].T).split([inner, inner + 2 * G * N, H], dim=-1)
    x, B, C = silu(causal_conv(xbc, w["conv"], w["conv.b"])).split([inner, G * N, G * N], dim=-1)
    x = x.reshape(T, H, V)
    B, C = (y.reshape(T, G, N).repeat_interleave(H // G, 1) for y in (B, C))
    dt, decay = mamba2_steps(dt, w["dt_bias"], w["A_log"])
    y, _ = decayed_scan(C, B * dt[:, :, None], x, decay)
    y = (y + w["D"][:, None] * x).reshape(T, inner) * silu(z)
    return grouped_norm(y, w["norm"], m["norm_groups"], eps) @ w["o"].T


def scaled_frequencies(rot: dict) -> torch.Tensor:
    """Rotation frequencies; short wavelengths keep theirs, long ones turn slower by `factor`, a linear blend in between."""
    f = torch.tensor([rot["base"] ** (-2 * i / rot["dims"]) for i in range(rot["dims"] // 2)], dtype=F)
    s = rot.get("scaling")
    if not s:
        return f
    out = []
    for x in f.tolist():
        length = 2 * math.pi / x
        if length < s["original"] / s["high"]:
            out.append(x)
        elif length > s["original"] / s["low"]:
            out.append(x / s["factor"])
        else:
            t = (s["original"] / length - s["low"]) / (s["high"] - s["low"])
            out.append((1 - t) * x / s["factor"] + t * x)
    return torch.tensor(out, dtype=F)


def rotate_pairs(x: torch.Tensor, freqs: torch.Tensor, pos: torch.Tensor) -> torch.Tensor:
    """x [T, H, d]: neighbouring dimensions 2i, 2i+1 turn together by pos * freqs[i], the rest stays."""
    n = 2 * len(freqs)
    a = pos.to(x.dtype)[:, None] * freqs.to(x.dtype)
    c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    return torch.cat([torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2), x[..., n:]], -1)


def chunk_mask(T: int, size: int) -> torch.Tensor:
    """[query, key]: keys up to the query in the query's own chunk, chunks counted from the first token."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None]
    return (j <= i) & (i // size == j // size)


def differential_lambda(w: dict, diff: float) -> torch.Tensor:
    return torch.exp((w["lq1"] * w["lk1"]).sum()) - torch.exp((w["lq2"] * w["lk2"]).sum()) + diff


def differential_mixer(h: torch.Tensor, w: dict, m: dict, eps: float) -> torch.Tensor:
    """Two softmax maps per head over the same values; the second one, weighted by lambda, is taken off the first."""
    T, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    pos, f = torch.arange(T), scaled_frequencies(m["rot"])
    q, k = (h @ w["q"].T).reshape(T, H, 2, D), (h @ w["k"].T).reshape(T, G, 2, D)
    v = (h @ w["v"].T).reshape(T, G, -1)
    a1, a2 = (masked_softmax_attention(rotate_pairs(q[:, :, i], f, pos), rotate_pairs(k[:, :, i], f, pos), v, m["scale"], chunk_mask(T, m["mask"]["size"])) for i in (0, 1))
    o = rms(a1 - differential_lambda(w, m["diff"]) * a2, eps) * (1 - m["diff"])
    return o.reshape(T, -1) @ w["o"].T


def group_route(h: torch.Tensor, w: torch.Tensor, correction: torch.Tensor, top: int, count: int, keep: int, scale: float):
    """Sigmoid scores; the corrected ones choose `keep` groups of neighbouring experts (by their two best) and then `top` experts among them;
    the weights are the chosen scores without the correction, divided by their sum, times `scale`."""
    s = sigmoid(h @ w.T)
    T, n = s.shape
    ids, p = torch.empty(T, top, dtype=torch.long), torch.empty(T, top, dtype=s.dtype)
    for t in range(T):
        c = (s[t] + correction).reshape(count, n // count)
        best = c.sort(-1, descending=True).values[:, :2].sum(-1).sort(descending=True, stable=True).indices[:keep]
        open_ = torch.full_like(c, -math.inf)
        open_[best] = c[best]
        ids[t] = open_.flatten().sort(descending=True, stable=True).indices[:top]
        p[t] = s[t][ids[t]]
    return ids, p / (p.sum(-1, keepdim=True) + 1e-20) * scale


def gated_expert(h: torch.Tensor, gate: torch.Tensor, up: torch.Tensor, down: torch.Tensor) -> torch.Tensor:
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def shared_moe_mlp(h: torch.Tensor, w: dict, r: dict) -> torch.Tensor:
    """Routed gated experts and one that every token uses, weighted by its own gate."""
    ids, p = group_route(h, w["router"], w["correction"], r["top"], r["groups"]["count"], r["groups"]["keep"], r["scale"])
    out = gated_expert(h, w["shared.gate"], w["shared.up"], w["shared.down"]) * sigmoid(h @ w["shared.sg"].T)
    for t in range(h.shape[0]):
        for e, x in zip(ids[t].tolist(), p[t]):
            out[t] += x * gated_expert(h[t], *(w[f"e{e}.{n}"] for n in ("gate", "up", "down")))
    return out


def relu2_mlp(h: torch.Tensor, w: dict) -> torch.Tensor:
    return torch.clamp(h @ w["up"].T, min=0) ** 2 @ w["down"].T


def nifalorn_layer(x: torch.Tensor, spec: dict, w: dict, norm: dict) -> torch.Tensor:
    """RMS norms with weights around zero in front of the sublayers."""
    sub = {p: {k[4:]: v for k, v in w.items() if k.startswith(p + ".")} for p in ("mix", "mlp")}
    mixer = {"lightning": lightning_mixer, "mamba2": mamba2_mixer, "attention": differential_mixer}[spec["type"]]
    x = x + mixer(rms(x, norm["eps"]) * (1 + w["norm1"]), sub["mix"], spec["mixer"], norm["eps"])
    if spec["mlp"] is not None:
        h = rms(x, norm["eps"]) * (1 + w["norm2"])
        x = x + (relu2_mlp(h, sub["mlp"]) if spec["mlp"]["kind"] == "dense" else shared_moe_mlp(h, sub["mlp"], spec["mlp"]["router"]))
    return x


def yarn_rotation(rot: dict) -> tuple[torch.Tensor, float]:
    """Rotation frequencies and the factor on both cosine and sine.  With YaRN scaling, pairs that turn more than `fast` times within the
    original context keep their frequency, those below `slow` turns are slowed down by `factor`, with a linear ramp over the pair number between."""
    n, base = rot["dims"], rot["base"]
    f = [base ** (-2 * i / n) for i in range(n // 2)]
    s = rot.get("scaling")
    if not s:
        return torch.tensor(f, dtype=F), 1.0

    def pair_of(turns):
        return n * math.log(s["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(pair_of(s["fast"])), 0), min(math.ceil(pair_of(s["slow"])), n - 1)
    out = []
    for i, x in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(x / s["factor"] * ramp + x * (1 - ramp))
    return torch.tensor(out, dtype=F), 0.1 * math.log(s["factor"]) + 1


def turn_half(x: torch.Tensor, rot: dict, pos: torch.Tensor) -> torch.Tensor:
    """x [T, H, d]: dimension i turns with dimension i + dims / 2 at the (scaled) frequencies of `rot`."""
    f, amp = yarn_rotation(rot)
    n = len(f)
    a = pos.to(x.dtype)[:, None] * f.to(x.dtype)
    c, s = amp * torch.cos(a)[:, None], amp * torch.sin(a)[:, None]
    u, v = x[..., :n], x[..., n:2 * n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * n:]], -1)


def mix_values(v: torch.Tensor, first: torch.Tensor | None, lam: torch.Tensor) -> torch.Tensor:
    """The first mixing layer keeps its values; the later ones blend them in."""
    return v if first is None else (1 - lam) * v + lam * first


def biased_attention_mixer(h: torch.Tensor, w: dict, m: dict, first: torch.Tensor | None = None):
    """Grouped-query attention with biases on q, k and v, a sliding window, and values mixed with those of the first mixing layer.  Returns
    the output and the layer's own values (before mixing)."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    pos = torch.arange(T)
    q, k, v = (h @ w[n].T + w[n + ".b"] for n in ("q", "k", "v"))
    q, k = turn_half(q.reshape(T, H, m["dim"]), m["rot"], pos), turn_half(k.reshape(T, G, m["dim"]), m["rot"], pos)
    mixed = mix_values(v, first, w["vmix"]) if m.get("v_mix") else v
    o = masked_softmax_attention(q, k, mixed.reshape(T, G, m["vdim"]), m["scale"], window_mask(T, m["mask"]["size"], 0))
    return o.reshape(T, H * m["vdim"]) @ w["o"].T, v


def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.log1p(torch.exp(-z.abs())) + torch.clamp(z, min=0)


def delta_scan(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, g: torch.Tensor, beta: torch.Tensor, state: torch.Tensor | None = None):
    """q, k [T, H, d], v [T, H, dv], decay g and write strength beta [T, H] -> o [T, H, dv] and the last state [H, d, dv].  What the decayed
    state already answers to k is taken off v before it is written."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    out = []
    for t in range(T):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - (S * k[t][:, :, None]).sum(1))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out), S


def delta_mixer(h: torch.Tensor, w: dict, m: dict, eps: float) -> torch.Tensor:
    T, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q, k, v = (silu(causal_conv(h @ w[n].T, w[n + ".conv"], torch.zeros(w[n].shape[0], dtype=h.dtype))) for n in ("q", "k", "v"))
    q, k = (unit(x.reshape(T, G, D)).repeat_interleave(H // G, 1) for x in (q, k))
    g = torch.exp(-torch.exp(w["A_log"]) * softplus(h @ w["a"].T + w["dt_bias"]))
    o, _ = delta_scan(q * D ** -0.5, k, v.reshape(T, H, m["vdim"]), g, sigmoid(h @ w["b"].T))
    return (rms(o, eps) * w["norm"]).reshape(T, -1) * silu(h @ w["g"].T) @ w["o"].T


def low_rank_latent_mixer(h: torch.Tensor, w: dict, m: dict, eps: float) -> torch.Tensor:
    """Latent attention whose queries pass a latent too; every head has a part with positions (neighbouring pairs), its key shared by all heads."""
    T, H, D, V, R, P = h.shape[0], m["heads"], m["dim"], m["vdim"], m["kv_rank"], m["rot_dim"]
    pos, (f, amp) = torch.arange(T), yarn_rotation(m["rot"])
    q = ((rms(h @ w["dq"].T, eps) * w["dq.norm"]) @ w["uq"].T).reshape(T, H, D + P)
    kv = h @ w["dkv"].T
    c, kr = rms(kv[:, :R], eps) * w["dkv.norm"], amp * rotate_pairs(kv[:, None, R:], f, pos)
    q = torch.cat([q[..., :D], amp * rotate_pairs(q[..., D:], f, pos)], -1)
    k = torch.cat([(c @ w["uk"].T).reshape(T, H, D), kr.expand(T, H, P)], -1)
    o = masked_softmax_attention(q, k, (c @ w["uv"].T).reshape(T, H, V), m["scale"], window_mask(T, m["mask"]["size"], 0))
    return o.reshape(T, H * V) @ w["o"].T


def xielu(z: torch.Tensor, p: torch.Tensor, q: torch.Tensor) -> torch.Tensor:
    return z / 2 + torch.where(z > 0, softplus(p) * z * z, (0.5 + softplus(q)) * (torch.expm1(torch.clamp(z, max=0)) - z))


def xielu_mlp(h: torch.Tensor, w: dict) -> torch.Tensor:
    return xielu(h @ w["up"].T, w["act"][0], w["act"][1]) @ w["down"].T


def rigalorn_layer(x: torch.Tensor, spec: dict, w: dict, norm: dict, kept: dict) -> torch.Tensor:
    """One norm; mixer and feed-forward both read its output.  `kept`: values of the first layer that mixes them."""
    sub = {p: {k[4:]: v for k, v in w.items() if k.startswith(p + ".")} for p in ("mix", "mlp")}
    m = spec["mixer"]
    h = rms(x, norm["eps"]) * w["norm1"]
    if spec["type"] == "attention":
        y, v = biased_attention_mixer(h, sub["mix"], m, kept.get("v"))
        if m.get("v_mix"):
            kept.setdefault("v", v)
    else:
        y = {"delta": delta_mixer, "latent_attention": low_rank_latent_mixer}[spec["type"]](h, sub["mix"], m, norm["eps"])
    return x + (y + xielu_mlp(h, sub["mlp"]) if spec["mlp"] is not None else y)


def layer(x: torch.Tensor, spec: dict, w: dict, norm: dict) -> torch.Tensor:
    """Talizen: both sublayers read x as it is; their outputs are normalised before they are added."""
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


def pre_norm_layer(x: torch.Tensor, spec: dict, w: dict, norm: dict) -> torch.Tensor:
    """Vozinex: layer norms in front of the sublayers, whose outputs are added as they are."""
    sub = {p: {k[4:]: v for k, v in w.items() if k.startswith(p + ".")} for p in ("mix", "mlp")}
    x = x + attention_mixer(layer_norm(x, w["norm1"], w["norm1.b"], norm["eps"]), sub["mix"], spec["mixer"], norm["eps"])
    if spec["mlp"] is not None:
        x = x + moe_mlp(layer_norm(x, w["norm2"], w["norm2.b"], norm["eps"]), sub["mlp"], spec["mlp"]["router"]["top"])
    return x


def layer_runs(cfg: dict) -> list[tuple[int, bool]]:
    """(layer, whether the embedding output is added in front of it) in the order of execution."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return [(i, False) for i in range(n)]
    inner, rejoin = list(range(lp["start"], lp["stop"])), cfg["architecture"] == "Vozinex"
    passes = [(i, rejoin and p > 0 and i == inner[0]) for p in range(lp["times"]) for i in inner]
    return [(i, False) for i in range(lp["start"])] + passes + [(i, False) for i in range(lp["stop"], n)]


def final_rows(cfg: dict, w: dict, x: torch.Tensor) -> torch.Tensor:
    """The last norm."""
    eps = cfg["norm"]["eps"]
    if cfg["architecture"] == "Vozinex":
        return layer_norm(x, w["final.norm"], w["final.norm.b"], eps)
    if cfg["architecture"] == "Nifalorn":
        return rms(x, eps) * (1 + w["final.norm"])
    if cfg["architecture"] == "Rigalorn":
        return rms(x, eps) * w["final.norm"]
    return grouped_norm(x, w["final.norm"], cfg["norm"]["groups"], eps)


def forward(cfg: dict, w: dict[str, torch.Tensor], tokens, dtype=F):
    """Logits [T, vocab] and the residual stream after every layer run [runs, T, width] of one whole sequence."""
    w = {k: v.to(dtype) for k, v in w.items()}
    kept = {}
    run = {"Talizen": layer, "Vozinex": pre_norm_layer, "Nifalorn": nifalorn_layer, "Rigalorn": functools.partial(rigalorn_layer, kept=kept)}[cfg["architecture"]]
    emb = x = w["embed"][torch.as_tensor(list(tokens))] * cfg.get("embedding", {}).get("scale", 1.0)
    after = []
    for i, again in layer_runs(cfg):
        p = f"l{i}."
        if again:
            x = x + emb
        x = run(x, cfg["layers"][i], {k[len(p):]: v for k, v in w.items() if k.startswith(p)}, cfg["norm"])
        after.append(x)
    return final_rows(cfg, w, x) @ w["head"].T * cfg.get("logit_scale", 1.0), torch.stack(after)


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
