"""Token mixers and feed-forwards of layer-list models: their weights, what they keep per sequence, and their launches.

A mixer multiplies the layer input by one stacked matrix (`w_in`), mixes over the tokens of every request in the batch (`mix`), and
hands the rows of its output product (`w_out`) back.  What it keeps between steps is declared, not allocated: `planes` are per-token
rows of the paged cache, `states` are fp32 tensors per sequence (models/engine.py PagedKVCache, RecurrentState).  A layer that runs
several times in one forward keeps them once per run (`run` below).

A feed-forward takes the rows in front of it and leaves its output in the engine's `y` (`apply`).  Where both read the same rows and their
outputs are added, `Joined` runs them as one input and one output product.
"""
from __future__ import annotations

import math
from dataclasses import dataclass

import torch

from ..ops import layers as lops


def pad_to(n: int, m: int) -> int:
    return (n + m - 1) // m * m


@dataclass
class Dense:
    """Weight rows [N, Kp] in the storage type; columns K .. Kp-1 are zero (the kernels read 16-byte pieces)."""
    t: torch.Tensor
    K: int

    @classmethod
    def make(cls, w: torch.Tensor, device, dtype) -> "Dense":
        N, K = w.shape
        t = torch.zeros(N, pad_to(K, 8), dtype=dtype, device=device)
        t[:, :K] = w.to(device)
        return cls(t, K)

    @property
    def N(self) -> int:
        return self.t.shape[0]

    @property
    def Kp(self) -> int:
        return self.t.shape[1]

    @property
    def nbytes(self) -> int:
        return self.t.numel() * self.t.element_size()


@dataclass
class Rows:
    """Input rows of a product: activation-typed `x`, or fp32 `x` with the residual sum / norms of ops.layers.RowStage in front."""
    x: torch.Tensor
    K: int
    y: torch.Tensor | None = None
    w1: torch.Tensor | None = None
    w2: torch.Tensor | None = None
    groups2: int = 1
    h_out: torch.Tensor | None = None
    b2: torch.Tensor | None = None      # with it the norm in front is a layer norm
    e: torch.Tensor | None = None       # a second addend
    pair: int = 0                       # x holds two vectors of this many values per head: x1 - lam * x2
    lam: float = 0.0
    g: torch.Tensor | None = None       # gate logits (ops.layers.GATE_*)
    gate: int = 0
    tail: torch.Tensor | None = None    # activation-typed columns behind the row as they are (mat-vec sizes)


class Mixer:
    """What the engine asks of every mixer."""
    planes: dict = {}
    states: dict = {}
    bias: torch.Tensor | None = None    # fp32 [rows of w_in], added in the input product

    def weights(self):
        return [self.w_in, self.w_out]


class Hgrn2(Mixer):
    """Gated linear recurrence with state expansion: the forget gate decides what is written; fp32 state [heads, dim, vdim]."""

    def __init__(self, m: dict, get, device, dtype, eps: float):
        self.H, self.D, self.V = m["heads"], m["dim"], m["vdim"]
        f32 = dict(device=device, dtype=torch.float32)
        self.w_in = Dense.make(torch.cat([get("q"), get("f"), get("v")], 0), device, dtype)
        self.w_out = Dense.make(get("o"), device, dtype)
        self.fbias, self.lower, self.norm = (get(n).to(**f32).contiguous() for n in ("f.b", "lower", "norm"))
        for name, t, n in (("f.b", self.fbias, self.H * self.D), ("lower", self.lower, self.H * self.D), ("norm", self.norm, self.V)):
            if t.numel() != n:
                raise ValueError(f"{name} has {t.numel()} values, expected {n}")
        if self.w_in.N != self.H * (2 * self.D + self.V) or self.w_out.K != self.H * self.V:
            raise ValueError("hgrn2: a projection does not fit heads, dim and vdim")
        self.states = {"s": (self.H, self.D, self.V)}
        self.chunk = lops.HGRN2_CHUNK if self.D <= 128 else 0          # the chunk kernels keep a head's channels in one block

    def buffers(self, rows: int) -> dict[str, int]:
        return {"o": rows * self.H * self.V}

    def mix(self, eng, run: int, proj: torch.Tensor, b) -> Rows:
        o = eng.buf("o", b.T, self.H * self.V)
        state = eng.rstate.parts["s"][run]
        for s in (b.short, b.long):
            if s is not None:
                chunks = (*s.chunks[self.chunk], *eng.chunk_ws) if s is b.long and self.chunk else None
                lops.hgrn2(proj, self.fbias, self.lower, state, s.range, s.slot, s.n, b.pos, o, chunks)
        return Rows(o, self.H * self.V, w2=self.norm, groups2=self.H)


class ScalarDecay(Mixer):
    """What recurrences with one decay per head and token share (ops.layers.ssd): state [heads, dim, vdim], forms by segment length."""
    H: int
    D: int
    V: int

    @property
    def chunk(self) -> int:
        """Tokens per chunk of long segments (0: they are scanned token by token)."""
        return lops.SSD_CHUNK if self.D <= lops.SSD_DIM else 0

    def scan(self, eng, run: int, rows, hpg: int, b, o: torch.Tensor, **kw):
        """Every segment of the batch: single tokens of a decode step, short ones token by token, long ones in chunks."""
        state = eng.rstate.parts["s"][run]
        for s in (b.short, b.long):
            if s is not None:
                chunks = (*s.chunks[self.chunk], *eng.chunk_ws) if s is b.long and self.chunk else None
                lops.ssd(rows, hpg, state, self.decay, self.log_decay, s.range, s.slot, s.n, b.pos, o, chunks=chunks, single=b.decode and lops.ssd_single_fits(self.D, self.V), **kw)


class Lightning(ScalarDecay):
    """Linear attention with a constant decay per head; the heads are normalised together and gated."""

    def __init__(self, m: dict, get, device, dtype, eps: float):
        self.H, self.D, self.V = m["heads"], m["dim"], m["vdim"]
        H, D, V = self.H, self.D, self.V
        f32 = dict(device=device, dtype=torch.float32)
        parts = [get("q"), get("k"), get("v"), get("g")]
        self.norm = get("norm").to(**f32).contiguous()
        if [p.shape[0] for p in parts] != [H * D, H * D, H * V, H * V] or self.norm.numel() != H * V or len(m["decay"]) != H:
            raise ValueError("lightning: a projection, the norm or the decays do not fit heads, dim and vdim")
        self.w_in = Dense.make(torch.cat(parts, 0), device, dtype)
        self.w_out = Dense.make(get("o"), device, dtype)
        if self.w_out.K != H * V:
            raise ValueError("lightning: the output matrix does not fit heads and vdim")
        decay = torch.tensor(m["decay"], dtype=torch.float64)
        self.decay = decay.to(**f32)
        self.log_decay = torch.log(decay).clamp(min=-1e30).to(**f32)        # (a decay of zero: exponents stay finite)
        self.states = {"s": (H, D, V)}

    def buffers(self, rows: int) -> dict[str, int]:
        return {"o": rows * self.H * self.V}

    def mix(self, eng, run: int, proj: torch.Tensor, b) -> Rows:
        HD, HV = self.H * self.D, self.H * self.V
        o = eng.buf("o", b.T, HV)
        self.scan(eng, run, (proj[:, :HD], proj[:, HD:2 * HD], proj[:, 2 * HD:2 * HD + HV]), 1, b, o, act=True)
        return Rows(o, HV, w2=self.norm, g=proj[:, 2 * HD + HV:], gate=lops.GATE_SIGMOID_AFTER)


class Mamba2(ScalarDecay):
    """State-space duality: step sizes and decays from the input, keys and queries shared by groups of heads, a short convolution in front,
    a gate in front of the norm (in groups)."""

    def __init__(self, m: dict, get, device, dtype, eps: float):
        self.H, self.D, self.V, self.G, self.taps, self.norm_groups = m["heads"], m["state"], m["vdim"], m["groups"], m["conv"], m["norm_groups"]
        H, V = self.H, self.V
        self.inner, gn = H * V, self.G * self.D
        self.channels = self.inner + 2 * gn
        f32 = dict(device=device, dtype=torch.float32)
        self.w_in = Dense.make(get("in"), device, dtype)
        self.w_out = Dense.make(get("o"), device, dtype)
        conv = get("conv")
        self.conv_b, self.dt_bias, self.skip, self.norm, a_log = (get(n).to(**f32).contiguous() for n in ("conv.b", "dt_bias", "D", "norm", "A_log"))
        if self.w_in.N != self.inner + self.channels + H or self.w_out.K != self.inner or conv.shape != (self.channels, self.taps):
            raise ValueError("mamba2: a projection or the convolution does not fit heads, vdim, groups and state")
        for name, t, n in (("conv.b", self.conv_b, self.channels), ("dt_bias", self.dt_bias, H), ("D", self.skip, H), ("A_log", a_log, H), ("norm", self.norm, self.inner)):
            if t.numel() != n:
                raise ValueError(f"mamba2: {name} has {t.numel()} values, expected {n}")
        self.conv_w = conv.to(**f32).T.contiguous()               # [taps, channels]
        self.decay, self.log_decay = None, -torch.exp(a_log)      # per unit of step size
        self.states = {"s": (H, self.D, V), "conv": (self.taps, self.channels)}

    def buffers(self, rows: int) -> dict[str, int]:
        return {"o": rows * self.inner, "xbc": rows * pad_to(self.channels, 8)}

    def mix(self, eng, run: int, proj: torch.Tensor, b) -> Rows:
        I, gn, T = self.inner, self.G * self.D, b.T
        o = eng.buf("o", T, I)
        ring, raw = eng.rstate.parts["conv"][run], proj[:, I:I + self.channels]
        cols = lambda x: (x[:, I + gn:], x[:, I:I + gn], x)       # (C, B, x) as query, key and value
        steps = (proj[:, I + self.channels:], self.dt_bias)
        if b.decode and lops.ssd_single_fits(self.D, self.V):
            self.scan(eng, run, cols(raw), self.H // self.G, b, o, steps=steps, skip=self.skip, conv=lops.conv_args(raw, self.conv_w, self.conv_b, ring))
        else:
            xbc = eng.buf("xbc", T, pad_to(self.channels, 8))
            for s in (b.short, b.long):
                if s is not None:
                    lops.conv_rows(raw, self.conv_w, self.conv_b, ring, s.range, s.slot, s.n, s.longest, b.pos, xbc)
            self.scan(eng, run, cols(xbc), self.H // self.G, b, o, steps=steps, skip=self.skip)
        return Rows(o, I, w2=self.norm, groups2=self.norm_groups, g=proj[:, :I], gate=lops.GATE_SILU_BEFORE)


class Delta(Mixer):
    """Gated delta rule: what the decayed state answers to a key is taken off the value before it is written; unit queries and keys behind short
    convolutions, shared by groups of heads; a norm per head and a gate behind it."""
    UNIT_EPS = 1e-6         # inside the root that makes a unit vector
    WORKSPACES = tuple("delta_" + n for n in ("states", "keys", "solve", "weights", "u", "gates"))

    def __init__(self, m: dict, get, device, dtype, eps: float):
        self.H, self.G, self.D, self.V, self.taps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
        H, G, D, V = self.H, self.G, self.D, self.V
        self.channels = 2 * G * D + H * V
        f32 = dict(device=device, dtype=torch.float32)
        parts, convs = [get(n) for n in ("q", "k", "v", "g", "b", "a")], [get(n + ".conv") for n in ("q", "k", "v")]
        if [p.shape[0] for p in parts] != [G * D, G * D, H * V, H * V, H, H]:
            raise ValueError("delta: a projection does not fit heads, kv_heads, dim and vdim")
        if [tuple(c.shape) for c in convs] != [(p.shape[0], self.taps) for p in parts[:3]]:
            raise ValueError("delta: a convolution does not fit its projection")
        self.w_in = Dense.make(torch.cat(parts, 0), device, dtype)
        self.w_out = Dense.make(get("o"), device, dtype)
        self.norm, self.dt_bias, a_log = (get(n).to(**f32).contiguous() for n in ("norm", "dt_bias", "A_log"))
        if self.w_out.K != H * V or self.norm.numel() != V or self.dt_bias.numel() != H or a_log.numel() != H:
            raise ValueError("delta: the output matrix, the norm or the decays do not fit heads and vdim")
        self.log_decay = -torch.exp(a_log)                        # per unit of step size
        self.conv_w = torch.cat(convs, 0).to(**f32).T.contiguous()          # [taps, channels]
        self.chunk = lops.DELTA_CHUNK if D <= lops.DELTA_DIM and dtype == torch.bfloat16 else 0
        self.states = {"s": (H, D, V), "conv": (self.taps, self.channels)}

    def buffers(self, rows: int) -> dict[str, int]:
        out = {"o": rows * self.H * self.V, "xbc": rows * pad_to(self.channels, 8)}
        if self.chunk:
            out |= {n: b // 4 for n, b in zip(self.WORKSPACES, lops.delta_workspace(lops.most_chunks(rows, self.chunk), self.H, self.G, self.D, self.V))}
        return out

    def mix(self, eng, run: int, proj: torch.Tensor, b) -> Rows:
        H, GD, HV, ch, T = self.H, self.G * self.D, self.H * self.V, self.channels, b.T
        o = eng.buf("o", T, HV)
        ring, state, raw = eng.rstate.parts["conv"][run], eng.rstate.parts["s"][run], proj[:, :ch]
        gate, wb, wa = proj[:, ch:ch + HV], proj[:, ch + HV:ch + HV + H], proj[:, ch + HV + H:ch + HV + 2 * H]
        cols = lambda x: (x, x[:, GD:], x[:, 2 * GD:])

        def scan(rows, s, **kw):
            lops.delta(rows, H // self.G, state, wa, wb, self.log_decay, self.dt_bias, s.range, s.slot, s.n, b.pos, o, self.UNIT_EPS, **kw)
        if b.decode and lops.ssd_single_fits(self.D, self.V):
            scan(cols(raw), b.short, conv=lops.conv_args(raw, self.conv_w, None, ring), single=True)
        else:
            xbc = eng.buf("xbc", T, pad_to(ch, 8))
            for s in (b.short, b.long):
                if s is not None:
                    lops.conv_rows(raw, self.conv_w, None, ring, s.range, s.slot, s.n, s.longest, b.pos, xbc)
                    ws = (*s.chunks[self.chunk], *(eng.flat(n) for n in self.WORKSPACES)) if s is b.long and self.chunk else None
                    scan(cols(xbc), s, chunks=ws)
        return Rows(o, HV, w2=self.norm, groups2=H, g=gate, gate=lops.GATE_SILU_AFTER)


class LatentAttention(Mixer):
    """Softmax attention over one cached latent row per token, shared by all heads.  Queries are multiplied into the latent space (key matrix
    absorbed), the attended latent is expanded per head.  What the layer's entry may ask for: queries through a normalised latent of their own
    (`q_rank`); a part of every query with positions, whose key the heads share (`rot_dim`; it lies behind the latent in the cached row, so that one
    dot product covers both parts); a sliding window; a gate per head."""

    def __init__(self, m: dict, get, device, dtype, eps: float):
        self.H, self.D, self.V, self.R, self.scale, self.eps = m["heads"], m["dim"], m["vdim"], m["kv_rank"], float(m["scale"]), eps
        self.P, self.gated, self.window = m.get("rot_dim", 0), bool(m.get("gate")), (m.get("mask") or {}).get("size", lops.NO_WINDOW)
        H, D, V, R, P = self.H, self.D, self.V, self.R, self.P
        self.Dq = D + P
        self.Rc, self.Vc = pad_to(R + P, 32), pad_to(R, 32)           # row length of the latent cache, and of what is attended of it
        self.planes = {"c": (1, self.Rc)}
        f32 = dict(device=device, dtype=torch.float32)
        self.w_uq = self.q_norm = None
        wq, wd = get("dq" if m.get("q_rank") else "q"), get("dkv")
        if m.get("q_rank"):
            self.w_uq, self.q_norm = Dense.make(get("uq"), device, dtype), get("dq.norm").to(**f32).contiguous()
            if wq.shape[0] != m["q_rank"] or self.w_uq.K != m["q_rank"] or self.q_norm.numel() != m["q_rank"]:
                raise ValueError("latent attention: a query projection does not fit q_rank")
        self.dkv0 = wq.shape[0]                       # first latent column of the projection
        if (wq if self.w_uq is None else self.w_uq.t).shape[0] != H * self.Dq or wd.shape[0] != R + P:
            raise ValueError("latent attention: a projection does not fit heads, dim and kv_rank")
        parts = [wq, wd]
        if self.gated:
            parts.append(get("g"))
            if parts[-1].shape[0] != H:
                raise ValueError("latent attention: the gate does not fit heads")
        self.w_in = Dense.make(torch.cat(parts, 0), device, dtype)
        self.w_out = Dense.make(get("o"), device, dtype)
        self.c_norm = get("dkv.norm").to(**f32).contiguous()
        if self.c_norm.numel() != R or self.w_out.K != H * V:
            raise ValueError("latent attention: the norm or the output matrix does not fit kv_rank, heads and vdim")
        if P:
            f, self.rot_scale = rotation(m["rot"])
            self.inv_freq = f.to(**f32)
        uk, uv = get("uk").to(device).view(H, D, R), get("uv").to(device).view(H, V, R)
        self.uk = torch.zeros(H, self.Rc, pad_to(self.Dq, 32), dtype=dtype, device=device)      # per head [cached row, query]: the part with positions as it is
        self.uk[:, :R, :D] = uk.transpose(1, 2)
        self.uk[:, range(R, R + P), range(D, D + P)] = 1
        self.uv = torch.zeros(H, V, self.Vc, dtype=dtype, device=device)                  # per head [vdim, latent]
        self.uv[:, :, :R] = uv
        # long prompt portions expand keys and values per head instead (tensor-core flash kernel; heads padded to multiples of 64)
        self.expand = dtype == torch.bfloat16 and self.Dq <= lops.ROWS_FLASH_KEY and V <= lops.ROWS_FLASH_VALUE
        self.Dp, self.Vp = pad_to(self.Dq, 64), pad_to(V, 64)
        if self.expand:
            ukv = torch.zeros(H * (self.Dp + self.Vp), self.Rc, dtype=dtype, device=device)
            keys = ukv[:H * self.Dp].view(H, self.Dp, self.Rc)
            keys[:, :D, :R] = uk
            keys[:, range(D, D + P), range(R, R + P)] = 1
            ukv[H * self.Dp:].view(H, self.Vp, self.Rc)[:, :V, :R] = uv
            self.ukv = Dense(ukv, R + P)

    @property
    def kind(self) -> tuple:
        """What the row tiles of a batch depend on."""
        return self.H, self.window, self.Rc

    def weights(self):
        extra = [w for w in (self.w_uq, self.ukv if self.expand else None) if w is not None]
        return [self.w_in, self.w_out, Dense(self.uk.view(-1, self.uk.shape[2]), self.Dq), Dense(self.uv.view(-1, self.Vc), self.R), *extra]

    def buffers(self, rows: int) -> dict[str, int]:
        return {"q": rows * self.H * self.Rc, "ctx": rows * self.H * self.Vc, "att": rows * self.w_out.Kp, **({"q_up": rows * self.H * self.Dq} if self.w_uq is not None else {})}

    def mix(self, eng, run: int, proj: torch.Tensor, b) -> Rows:
        H, Dq, R, Rc, V, Vc = self.H, self.Dq, self.R, self.Rc, self.V, self.Vc
        cache = eng.kv.planes["c"][run]
        qx = proj[:, :H * Dq]
        if self.w_uq is not None:
            qx = eng.product(Rows(proj[:, :self.dkv0], self.dkv0, w2=self.q_norm), self.w_uq, eng.buf("q_up", b.T, H * Dq), b.T)
        c0 = self.dkv0
        lops.latent_write(proj[:, c0:c0 + R + self.P], self.c_norm, self.eps, R, b.slot, cache, b.T, **(dict(rot=(b.pos, self.inv_freq, self.rot_scale), q=qx, heads=H) if self.P else {}))
        gate = proj[:, c0 + R + self.P:] if self.gated else None
        att = eng.buf("att", b.T, self.w_out.Kp, eng.dtype)
        long = b.long if self.expand else None
        T = b.T_short if long is not None else b.T           # short segments come first
        if T:
            q = eng.buf("q", T, H * Rc, eng.dtype)
            lops.head_matmul(qx, Dq, Dq, self.uk, Rc, q, Rc, T)
            ctx = eng.buf("ctx", T, H * Vc, eng.dtype)
            t = b.tiles[self.kind, long is not None]
            lops.latent_attention(q, cache, eng.kv.block_table, b.tok_slot, b.pos, t.row0, t.rows, t.n, t.bm, H, T, self.scale, ctx, n_splits=t.n_splits,
                                  workspace=eng.latent_ws, window=self.window)
            lops.head_matmul(ctx, Vc, Vc, self.uv, V, att, V, T, gate=gate)
        for sid, lo, hi, S in (long.host if long is not None else ()):
            pos0 = S - (hi - lo)
            page0 = max(0, pos0 - self.window + 1) // eng.page_size         # the first page whose rows are seen
            S, pos0 = S - page0 * eng.page_size, pos0 - page0 * eng.page_size
            c = eng.grow("c_rows", S, Rc)
            lops.latent_gather(cache, eng.kv.block_table[sid, page0:], S, c)
            kv = lops.linear(c, self.ukv.t, eng.grow("kv_rows", S, self.ukv.N))
            q = lops.head_rows(qx[lo:hi], H, Dq, self.Dp, eng.grow("q_rows", hi - lo, H * self.Dp))
            lops.rows_attention(q, kv, S, pos0, H, self.Dp, self.Vp, V, self.scale, att[lo:hi], gate=gate[lo:hi] if gate is not None else None, window=self.window)
        return Rows(att, H * V)


def rotation_frequencies(dims: int, base: float, scaling: dict | None = None) -> torch.Tensor:
    """Frequency of every rotated pair (fp64).  scaling: pairs whose wavelength exceeds original / low turn `factor` times slower, those below
    original / high keep their frequency, in between the two are blended linearly in original / wavelength."""
    f = base ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims)
    if not scaling:
        return f
    turns = scaling["original"] * f / (2 * math.pi)               # within the original context
    keep = ((turns - scaling["low"]) / (scaling["high"] - scaling["low"])).clamp(0, 1)
    slow = f / scaling["factor"]
    return torch.where(turns > scaling["high"], f, torch.where(turns < scaling["low"], slow, (1 - keep) * slow + keep * f))


def yarn_frequencies(dims: int, base: float, scaling: dict) -> torch.Tensor:
    """YaRN: pairs that turn at least `fast` times within the original context keep their frequency, those of at most `slow` turns get `factor` times
    slower, with a linear ramp over the pair number in between (fp64)."""
    f = rotation_frequencies(dims, base)

    def pair(turns):           # (not whole) number of the pair that turns this often
        return dims * math.log(scaling["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(pair(scaling["fast"])), 0), min(math.ceil(pair(scaling["slow"])), dims - 1)
    ramp = ((torch.arange(dims // 2, dtype=torch.float64) - lo) / max(hi - lo, 0.001)).clamp(0, 1)
    return f / scaling["factor"] * ramp + f * (1 - ramp)


def rotation(rot: dict) -> tuple[torch.Tensor, float]:
    """Frequencies of a layer's rotation (fp64) and the factor on cosine and sine."""
    scaling = rot.get("scaling")
    if scaling and "fast" in scaling:
        return yarn_frequencies(rot["dims"], float(rot["base"]), scaling), 0.1 * math.log(scaling["factor"]) + 1
    return rotation_frequencies(rot["dims"], float(rot["base"]), scaling), 1.0


class Attention(Mixer):
    """Grouped-query softmax attention over cached keys and values.  What the layer's entry may ask for: RMS norm of queries and keys over their
    whole projection; biases; rotation of the first `rot.dims` dimensions of a head, half-split or adjacent pairs, with scaled frequencies; a sliding
    window with kept first tokens; chunks; values mixed with those of the first layer that asks for it (`v_mix`: "first", then "later"); two maps
    per head over the same values, of which the second is taken off the first with a learned weight and the rest normalised per head
    (differential attention).  With two maps `H` counts (head, map) query rows."""

    def __init__(self, m: dict, get, device, dtype, eps: float):
        self.heads, self.G, self.D, self.V, self.scale, self.eps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"]), eps
        self.maps = 2 if "diff" in m else 1
        self.H = self.heads * self.maps
        self.R = self.H // self.G                     # query rows per key / value head
        rot, mask = m["rot"], m.get("mask") or {}
        self.rot, self.adjacent = rot["dims"], bool(rot.get("adjacent"))
        self.window, self.keep, self.chunk = mask.get("size", lops.NO_WINDOW), mask.get("keep_first", 0), mask.get("chunk", 0)
        self.Dc, self.Vc = pad_to(self.D, 16), pad_to(self.V, 16)        # cached rows
        self.planes = {"k": (self.G * self.maps, self.Dc), "v": (self.G, self.Vc)}
        parts = [get("q"), get("k"), get("v")]
        if [p.shape[0] for p in parts] != [self.H * self.D, self.G * self.maps * self.D, self.G * self.V]:
            raise ValueError("attention: a projection does not fit heads, kv_heads, dim and vdim")
        self.w_in = Dense.make(torch.cat(parts, 0), device, dtype)
        self.w_out = Dense.make(get("o"), device, dtype)
        if self.w_out.K != self.heads * self.V:
            raise ValueError("attention: the output matrix does not fit heads and vdim")
        f32 = dict(device=device, dtype=torch.float32)
        self.q_norm = self.k_norm = None
        if m.get("qk_norm"):
            self.q_norm, self.k_norm = (get(n).to(**f32).contiguous() for n in ("q.norm", "k.norm"))
            if self.q_norm.numel() != self.H * self.D or self.k_norm.numel() != self.G * self.D:
                raise ValueError("attention: a norm does not span its projection")
        if m.get("bias"):
            self.bias = torch.cat([get(n + ".b") for n in ("q", "k", "v")], 0).to(**f32)
            if self.bias.numel() != self.w_in.N:
                raise ValueError("attention: the biases do not fit their projections")
        self.v_mix, self.share = bool(m.get("v_mix")), float(get("vmix")) if m.get("v_mix") == "later" else None
        self.base = float(rot["base"])
        f, self.rot_scale = rotation(rot)
        self.inv_freq = f.to(**f32)
        if self.maps == 2:
            lq1, lk1, lq2, lk2 = (get(n).double().cpu() for n in ("lq1", "lk1", "lq2", "lk2"))
            if any(t.numel() != self.D for t in (lq1, lk1, lq2, lk2)):
                raise ValueError("attention: the vectors behind lambda do not fit dim")
            self.lam = float(torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum()) + m["diff"])
            self.o_norm = torch.full((self.V,), 1.0 - m["diff"], **f32)
        # tensor-core tiles; prompt portions from 128 tokens on take the tcgen05 flash kernel (bf16 storage, heads up to 128 wide)
        self.mma = dtype == torch.bfloat16 and max(self.maps * self.Dc, self.Vc) <= lops.GQA_MMA_DIM
        self.flash = dtype == torch.bfloat16 and max(self.Dc, self.Vc) <= lops.GQA_FLASH_DIM

    def buffers(self, rows: int) -> dict[str, int]:
        out = {"att": rows * self.w_out.Kp} if self.maps == 1 else {"o": rows * self.H * self.V}
        if self.v_mix:
            out["v_first"] = rows * self.G * self.V
        return {"q": rows * self.H * self.Dc, **out}

    def visible(self, length: int) -> int:
        """Most keys a token sees in a sequence of this length."""
        return min(length, self.window + self.keep, self.chunk or length)

    def rows(self, att: torch.Tensor) -> Rows:
        """Input rows of the output matrix: the attended values, or the difference of a head's two maps, normalised."""
        n = self.heads * self.V
        return Rows(att, n) if self.maps == 1 else Rows(att, n, w2=self.o_norm, groups2=self.heads, pair=self.V, lam=self.lam)

    def mix(self, eng, run: int, proj: torch.Tensor, b) -> Rows:
        kc, vc = eng.kv.planes["k"][run], eng.kv.planes["v"][run]
        bt, T = eng.kv.block_table, b.T
        att = eng.buf("att", T, self.w_out.Kp, eng.dtype) if self.maps == 1 else eng.buf("o", T, self.H * self.V)
        mix = (eng.buf("v_first", T, self.G * self.V), self.share) if self.v_mix else None
        if b.decode and self.mma:
            t = b.tiles["tokens", self.R, False]
            lops.gqa_decode(self, proj, kc, vc, bt, b.tok_slot, b.pos, t.table, b.key_ranges(self, t), att, T, mix=mix)
            return self.rows(att)
        q = eng.buf("q", T, self.H * self.Dc, eng.dtype)
        lops.gqa_prepare(self, proj, kc, vc, bt, b.tok_slot, b.pos, b.slot, q, T, mix=mix)
        flash = b.long is not None and self.flash
        if not flash or b.short is not None:
            t = b.tiles["tokens", self.R, flash]
            lops.gqa_attention(self, q, kc, vc, bt, b.tok_slot, b.pos, t.table, t.bm, b.key_ranges(self, t) if self.mma else 1, att, T)
        if flash:
            lops.gqa_flash(self, q, kc, vc, bt, b.tok_slot, b.pos, b.tiles["flash"].table, att, T)
        return self.rows(att)


class GatedMlp:
    """W_down (act(W_gate h) * W_up h) with the tanh form of gelu; gate and up rows are interleaved."""

    def __init__(self, m: dict, get, device, dtype, width: int):
        gate, up = get("gate"), get("up")
        if gate.shape != up.shape or gate.shape[0] != m["ff"]:
            raise ValueError("feed-forward: gate / up do not fit ff")
        self.w_gu = Dense.make(interleave(gate, up), device, dtype)
        self.w_down = Dense.make(get("down"), device, dtype)

    def weights(self):
        return [self.w_gu, self.w_down]

    def buffers(self, rows: int) -> dict[str, int]:
        return {"act": rows * self.w_down.Kp}

    def apply(self, eng, r: Rows, T: int):
        act = eng.product(r, self.w_gu, eng.buf("act", T, self.w_down.Kp), T, lops.OUT_GEGLU)
        eng.product(Rows(act, self.w_down.K), self.w_down, eng.y[:T], T)


class Relu2Mlp:
    """W_down max(W_up h, 0)^2."""

    def __init__(self, m: dict, get, device, dtype, width: int):
        self.w_up, self.w_down = Dense.make(get("up"), device, dtype), Dense.make(get("down"), device, dtype)
        if self.w_up.N != m["ff"] or self.w_up.K != width or self.w_down.K != m["ff"] or self.w_down.N != width:
            raise ValueError("feed-forward: up / down do not fit width and ff")

    def weights(self):
        return [self.w_up, self.w_down]

    def buffers(self, rows: int) -> dict[str, int]:
        return {"act": rows * self.w_down.Kp}

    def apply(self, eng, r: Rows, T: int):
        act = eng.product(r, self.w_up, eng.buf("act", T, self.w_down.Kp), T, lops.OUT_RELU2)
        eng.product(Rows(act, self.w_down.K), self.w_down, eng.y[:T], T)


class XieluMlp:
    """W_down xIELU(W_up h); the activation's two coefficients are learned."""

    def __init__(self, m: dict, get, device, dtype, width: int):
        self.w_up, self.w_down = Dense.make(get("up"), device, dtype), Dense.make(get("down"), device, dtype)
        act = get("act").double()
        if self.w_up.N != m["ff"] or self.w_up.K != width or self.w_down.K != m["ff"] or self.w_down.N != width or act.numel() != 2:
            raise ValueError("feed-forward: up / down / act do not fit width and ff")
        pos, neg = torch.nn.functional.softplus(act, threshold=100.0).tolist()
        self.act = pos, 0.5 + neg               # ops.layers.OutTail

    def weights(self):
        return [self.w_up, self.w_down]

    def buffers(self, rows: int) -> dict[str, int]:
        return {"act": rows * self.w_down.Kp}

    def apply(self, eng, r: Rows, T: int):
        act = eng.buf("act", T, self.w_down.Kp)
        eng.product(r, self.w_up, act, T, tail=lops.out_tail(n2=0, out2=act, act=self.act))
        eng.product(Rows(act, self.w_down.K), self.w_down, eng.y[:T], T)


class Joined:
    """A mixer and a feed-forward that read the same rows and whose outputs are added.  The input matrices are stacked to one product, which leaves
    the mixer's columns in the projection and the others behind their activation; the output product runs over the mixer's rows and those side by
    side (`att`), so that the sum is part of it."""

    def __init__(self, mixer, mlp: XieluMlp):
        self.mixer, self.act = mixer, mlp.act
        self.n, self.k = pad_to(mixer.w_in.N, 32), mixer.w_out.Kp
        w = torch.zeros(self.n + mlp.w_up.N, mlp.w_up.Kp, dtype=mlp.w_up.t.dtype, device=mlp.w_up.t.device)
        w[:mixer.w_in.N], w[self.n:] = mixer.w_in.t, mlp.w_up.t
        self.bias = None
        if mixer.bias is not None:
            self.bias = torch.zeros(self.n + mlp.w_up.N, dtype=torch.float32, device=w.device)
            self.bias[:mixer.bias.numel()] = mixer.bias
        self.w_in = mixer.w_in = Dense(w, mlp.w_up.K)
        self.w_out = mixer.w_out = Dense(torch.cat([mixer.w_out.t, mlp.w_down.t], 1), self.k + mlp.w_down.K)

    def buffers(self, rows: int) -> dict[str, int]:
        return {"att": rows * self.w_out.Kp}

    def apply(self, eng, run: int, r: Rows, b):
        T = b.T
        both = eng.buf("att", T, self.w_out.Kp)
        mine, act = both[:, :self.k], both[:, self.k:]
        proj = eng.product(r, self.w_in, eng.buf("proj", T, self.n), T, tail=lops.out_tail(self.bias, self.n, act, self.act))
        r = self.mixer.mix(eng, run, proj, b)
        if r.x.data_ptr() != both.data_ptr():            # rows that are still to be prepared
            if eng.matvec_rows(T, self.w_out):
                r.tail = act
                eng.product(r, self.w_out, eng.y[:T], T)
                return
            lops.stage_rows(eng.stage(r, self.k), mine, T)
        eng.product(Rows(both, self.w_out.Kp), self.w_out, eng.y[:T], T)


class RoutedExperts:
    """Each token uses the `top` of `experts` small feed-forwards: W_down max(W_up h, 0)^2, or gated (`expert.gated`) W_down (silu(W_gate h) * W_up h).
    Choice and weights: ops.layers.Routing (`router.score`: softmax over the chosen logits, or sigmoid with groups).  `shared`: one more gated
    expert of its own size that every token uses, weighted by a sigmoid gate, whose logit is one more row of the router.
    Up to four rows: three mat-vec launches (router; chosen experts' up and down products, which route for themselves).  More: the rows are
    sorted by expert and each of the two products is one grouped launch."""

    def __init__(self, m: dict, get, device, dtype, width: int):
        r = m["router"]
        self.n, self.top, self.ff, self.gated = r["experts"], r["top"], m["expert"]["ff"], bool(m["expert"].get("gated"))
        if self.n > lops.MAX_EXPERTS or self.top > lops.MAX_TOP:
            raise ValueError(f"feed-forward: {self.top} of {self.n} experts (at most {lops.MAX_TOP} of {lops.MAX_EXPERTS})")
        n, F, E = self.n, pad_to(self.ff, 8), width
        self.F, self.E = F, E
        self.act = lops.OUT_SWIGLU if self.gated else lops.OUT_RELU2
        rows = self.rows = 2 * F if self.gated else F
        up, down = torch.zeros(n, rows, pad_to(E, 8), dtype=dtype, device=device), torch.zeros(n, E, F, dtype=dtype, device=device)
        for e in range(n):
            u, d = get(f"e{e}.up"), get(f"e{e}.down")
            g = get(f"e{e}.gate") if self.gated else u
            if u.shape != (self.ff, E) or g.shape != u.shape or d.shape != (E, self.ff):
                raise ValueError(f"feed-forward: expert {e} does not fit width and ff")
            up[e, :(rows // F) * self.ff, :E] = interleave(g, u).to(device) if self.gated else u.to(device)
            down[e, :, :self.ff] = d.to(device)
        self.up, self.down = Dense(up.view(n * rows, -1), E), Dense(down.view(n * E, F), F)
        router = get("router")
        sigmoid = r.get("score") == "sigmoid"
        bias = get("correction" if sigmoid else "router.b").to(device=device, dtype=torch.float32).contiguous()
        if router.shape != (n, E) or bias.numel() != n:
            raise ValueError("feed-forward: the router does not fit experts and width")
        groups = r.get("groups") or {"count": 1, "keep": 1}
        self.rule = lops.Routing(bias, n, self.top, sigmoid, groups["count"], groups["keep"], float(r.get("scale", 1.0)))
        self.shared = None
        if m.get("shared"):
            ff, sg = m["shared"]["ff"], get("shared.sg")
            g, u, d = get("shared.gate"), get("shared.up"), get("shared.down")
            if g.shape != (ff, E) or u.shape != (ff, E) or d.shape != (E, ff) or sg.shape != (1, E):
                raise ValueError("feed-forward: the shared expert does not fit width and ff")
            Fs = pad_to(ff, 8)
            gu, dn = torch.zeros(2 * Fs, pad_to(E, 8), dtype=dtype, device=device), torch.zeros(E, Fs, dtype=dtype, device=device)
            gu[:2 * ff, :E] = interleave(g, u).to(device)
            dn[:, :ff] = d.to(device)
            self.shared = Dense(gu, E), Dense(dn, Fs)
            router = torch.cat([router, sg.to(router.dtype)], 0)
        self.router = Dense.make(router, device, dtype)

    def weights(self):
        return [self.router, self.up, self.down, *(self.shared or ())]

    def buffers(self, rows: int) -> dict[str, int]:
        a = rows * self.top
        extra = {"act_s": rows * self.shared[1].Kp, "ys": rows * self.E} if self.shared else {}
        return {"router": rows * self.router.N, "act": a * self.F, "ids": a, "gate_w": a, "xs": a * self.up.Kp, "ey": a * self.E, **extra}

    def apply(self, eng, r: Rows, T: int):
        n, k, F, E, A = self.n, self.top, self.F, self.E, T * self.top
        logits = eng.buf("router", T, self.router.N)
        act = eng.buf("act", A, F)
        gu, dn = self.shared or (None, None)
        act_s = eng.buf("act_s", T, dn.Kp) if self.shared else None
        if eng.matvec_rows(T, self.router) and lops.matvec_fits(T, self.up.t) and lops.expert_matvec_fits(T, k, self.down.t, dn.t if dn else None):
            eng.product(r, self.router, logits, T)                # also settles the residual rows (h_out), which the up product reads again
            h = Rows(r.x if r.h_out is None else r.h_out, E, w2=r.w2, b2=r.b2)
            lops.expert_matvec(eng.stage(h, self.up.Kp), logits, self.rule, self.up.t, self.rows, act, T, False, self.act, (gu.t, act_s) if gu else None)
            lops.expert_matvec(eng.stage(Rows(act, F), F), logits, self.rule, self.down.t, E, eng.y[:T], T, True, self.act, (dn.t, act_s) if dn else None)
            return
        x = eng.staged(r, self.up.Kp, T)
        lops.linear(x, self.router.t, logits)
        ids, w = eng.buf("ids", A, 1).view(-1), eng.buf("gate_w", A, 1).view(-1)
        lops.route(logits, self.rule, ids, w, T)
        plan, per = eng.expert_plans[n], A // n
        tile = 64 if eng.dtype == torch.float32 else 16 if per <= 16 else 32 if per <= 32 else 64 if per <= 96 else 128
        lops.expert_plan(ids, n, tile, plan)
        xs = lops.expert_gather(x, plan, k, A, eng.buf("xs", A, self.up.Kp))
        lops.linear_grouped(xs, self.up.t, self.rows, n, tile, plan, act, self.act)
        ey = lops.linear_grouped(act, self.down.t, E, n, tile, plan, eng.buf("ey", A, E))
        shared = None
        if self.shared:
            lops.linear(x, gu.t, act_s, lops.OUT_SWIGLU)
            shared = lops.linear(act_s, dn.t, eng.buf("ys", T, E)), logits[:, n:]
        lops.expert_combine(ey, plan, w, T, k, eng.y[:T], shared)


def interleave(gate: torch.Tensor, up: torch.Tensor) -> torch.Tensor:
    """Rows gate_0, up_0, gate_1, ...: one output of a gated product is one pair of neighbouring rows."""
    return torch.stack([gate, up], 1).reshape(2 * gate.shape[0], gate.shape[1])


MIXERS = {"hgrn2": Hgrn2, "lightning": Lightning, "mamba2": Mamba2, "delta": Delta, "latent_attention": LatentAttention, "attention": Attention}
MLPS = {"dense": GatedMlp, "relu2": Relu2Mlp, "xielu": XieluMlp, "moe": RoutedExperts}
