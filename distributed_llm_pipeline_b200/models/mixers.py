"""Token mixers and feed-forwards of layer-list models: their weights, what they keep per sequence, and their launches.

A mixer multiplies the layer input by one stacked matrix (`w_in`), mixes over the tokens of every request in the batch (`mix`), and
hands the rows of its output product (`w_out`) back.  What it keeps between steps is declared, not allocated: `planes` are per-token
rows of the paged cache, `state` is a recurrent state per sequence (models/engine.py PagedKVCache, RecurrentState).  A layer that runs
several times in one forward keeps them once per run (`run` below).

A feed-forward takes the rows in front of it and leaves its output in the engine's `y` (`apply`).
"""
from __future__ import annotations

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


class Hgrn2:
    """Gated linear recurrence with state expansion: the forget gate decides what is written; fp32 state [heads, dim, vdim]."""
    planes: dict = {}

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
        self.state = (self.H, self.D, self.V)
        self.chunked = self.D <= 128          # the chunk kernels keep a head's channels in one block

    def weights(self):
        return [self.w_in, self.w_out]

    def buffers(self, rows: int) -> dict[str, int]:
        return {"o": rows * self.H * self.V}

    def mix(self, eng, run: int, proj: torch.Tensor, b) -> Rows:
        o = eng.buf("o", b.T, self.H * self.V)
        state = eng.rstate.layers[run]
        for s in (b.short, b.long):
            if s is not None:
                chunks = (s.chunk, s.first, *eng.chunk_ws) if s is b.long and self.chunked else None
                lops.hgrn2(proj, self.fbias, self.lower, state, s.range, s.slot, s.n, b.pos, o, chunks)
        return Rows(o, self.H * self.V, w2=self.norm, groups2=self.H)


class LatentAttention:
    """Softmax attention over one cached latent row per token, shared by all heads and without positions.  Queries are multiplied into
    the latent space (key matrix absorbed), the attended latent is expanded per head and gated."""
    state = None

    def __init__(self, m: dict, get, device, dtype, eps: float):
        self.H, self.D, self.V, self.R, self.scale = m["heads"], m["dim"], m["vdim"], m["kv_rank"], float(m["scale"])
        H, D, V, R = self.H, self.D, self.V, self.R
        self.Rc = pad_to(R, 32)                       # row length of the latent cache
        self.planes = {"c": (1, self.Rc)}
        wq, wd, wg = get("q"), get("dkv"), get("g")
        if wq.shape[0] != H * D or wd.shape[0] != R or wg.shape[0] != H:
            raise ValueError("latent attention: a projection does not fit heads, dim and kv_rank")
        self.w_in = Dense.make(torch.cat([wq, wd, wg], 0), device, dtype)
        self.w_out = Dense.make(get("o"), device, dtype)
        self.c_norm = get("dkv.norm").to(device=device, dtype=torch.float32).contiguous()
        uk, uv = get("uk").to(device).view(H, D, R), get("uv").to(device).view(H, V, R)
        self.uk = torch.zeros(H, self.Rc, pad_to(D, 32), dtype=dtype, device=device)      # per head [latent, dim]
        self.uk[:, :R, :D] = uk.transpose(1, 2)
        self.uv = torch.zeros(H, V, self.Rc, dtype=dtype, device=device)                  # per head [vdim, latent]
        self.uv[:, :, :R] = uv
        # long prompt portions expand keys and values per head instead (tensor-core flash kernel; heads padded to 64 or 128)
        self.expand = dtype == torch.bfloat16 and D <= 128 and V <= 128
        self.Dp, self.Vp = pad_to(D, 64), pad_to(V, 64)
        if self.expand:
            ukv = torch.zeros(H * (self.Dp + self.Vp), self.Rc, dtype=dtype, device=device)
            ukv[:H * self.Dp].view(H, self.Dp, self.Rc)[:, :D, :R] = uk
            ukv[H * self.Dp:].view(H, self.Vp, self.Rc)[:, :V, :R] = uv
            self.ukv = Dense(ukv, R)

    def weights(self):
        return [self.w_in, self.w_out, Dense(self.uk.view(-1, self.uk.shape[2]), self.D), Dense(self.uv.view(-1, self.Rc), self.R)] + ([self.ukv] if self.expand else [])

    def buffers(self, rows: int) -> dict[str, int]:
        return {"q": rows * self.H * self.Rc, "ctx": rows * self.H * self.Rc, "att": rows * self.w_out.Kp}

    def mix(self, eng, run: int, proj: torch.Tensor, b) -> Rows:
        H, D, R, Rc, V = self.H, self.D, self.R, self.Rc, self.V
        cache = eng.kv.planes["c"][run]
        lops.latent_write(proj[:, H * D:H * D + R], self.c_norm, eng.cfg.rms_eps, R, b.slot, cache, b.T)
        gate = proj[:, H * D + R:]
        att = eng.buf("att", b.T, self.w_out.Kp, eng.dtype)
        long = b.long if self.expand else None
        T = b.T_short if long is not None else b.T           # short segments come first
        if T:
            q = eng.buf("q", T, H * Rc, eng.dtype)
            lops.head_matmul(proj, D, D, self.uk, Rc, q, Rc, T)
            ctx = eng.buf("ctx", T, H * Rc, eng.dtype)
            t = b.tiles[H, long is not None]
            lops.latent_attention(q, cache, eng.kv.block_table, b.tok_slot, b.pos, t.row0, t.rows, t.n, t.bm, H, T, self.scale, ctx, n_splits=t.n_splits,
                                  workspace=eng.latent_ws)
            lops.head_matmul(ctx, Rc, Rc, self.uv, V, att, V, T, gate=gate)
        for sid, lo, hi, S in (long.host if long is not None else ()):
            c = eng.grow("c_rows", S, Rc)
            lops.latent_gather(cache, eng.kv.block_table[sid], S, c)
            kv = lops.linear(c, self.ukv.t, eng.grow("kv_rows", S, self.ukv.N))
            q = lops.head_rows(proj[lo:hi], H, D, self.Dp, eng.grow("q_rows", hi - lo, H * self.Dp))
            lops.rows_attention(q, kv, S, S - (hi - lo), H, self.Dp, self.Vp, V, self.scale, att[lo:hi], gate=gate[lo:hi])
        return Rows(att, H * V)


class Attention:
    """Grouped-query softmax attention over cached keys and values: RMS norm of queries and keys over their whole projection, rotation of the
    first `rot` dimensions of a head, a sliding window with kept first tokens."""
    state = None

    def __init__(self, m: dict, get, device, dtype, eps: float):
        self.H, self.G, self.D, self.V, self.scale = m["heads"], m["kv_heads"], m["dim"], m["vdim"], float(m["scale"])
        self.R = self.H // self.G                     # query heads per key / value head
        self.rot, self.window, self.keep, self.eps = m["rot"]["dims"], m["mask"]["size"], m["mask"]["keep_first"], eps
        self.Dc, self.Vc = pad_to(self.D, 16), pad_to(self.V, 16)        # cached rows
        self.planes = {"k": (self.G, self.Dc), "v": (self.G, self.Vc)}
        parts = [get("q"), get("k"), get("v")]
        if [p.shape[0] for p in parts] != [self.H * self.D, self.G * self.D, self.G * self.V]:
            raise ValueError("attention: a projection does not fit heads, kv_heads, dim and vdim")
        self.w_in = Dense.make(torch.cat(parts, 0), device, dtype)
        self.w_out = Dense.make(get("o"), device, dtype)
        if self.w_out.K != self.H * self.V:
            raise ValueError("attention: the output matrix does not fit heads and vdim")
        self.q_norm, self.k_norm = (get(n).to(device=device, dtype=torch.float32).contiguous() for n in ("q.norm", "k.norm"))
        if self.q_norm.numel() != self.H * self.D or self.k_norm.numel() != self.G * self.D:
            raise ValueError("attention: a norm does not span its projection")
        self.base = float(m["rot"]["base"])
        self.inv_freq = (self.base ** (-2.0 * torch.arange(self.rot // 2, dtype=torch.float64) / self.rot)).to(device=device, dtype=torch.float32)
        # tensor-core tiles; prompt portions from 128 tokens on take the tcgen05 flash kernel (bf16 storage, heads up to 128 wide)
        self.mma = dtype == torch.bfloat16 and max(self.Dc, self.Vc) <= lops.GQA_MMA_DIM
        self.flash = dtype == torch.bfloat16 and max(self.Dc, self.Vc) <= lops.GQA_FLASH_DIM

    def weights(self):
        return [self.w_in, self.w_out]

    def buffers(self, rows: int) -> dict[str, int]:
        return {"q": rows * self.H * self.Dc, "att": rows * self.w_out.Kp}

    def visible(self, length: int) -> int:
        """Most keys a token sees in a sequence of this length."""
        return min(length, self.window + self.keep)

    def mix(self, eng, run: int, proj: torch.Tensor, b) -> Rows:
        kc, vc = eng.kv.planes["k"][run], eng.kv.planes["v"][run]
        bt, T = eng.kv.block_table, b.T
        att = eng.buf("att", T, self.w_out.Kp, eng.dtype)
        if b.decode and self.mma:
            t = b.tiles["tokens", self.R, False]
            lops.gqa_decode(self, proj, kc, vc, bt, b.tok_slot, b.pos, t.table, b.key_ranges(self, t), att, T)
            return Rows(att, self.H * self.V)
        q = eng.buf("q", T, self.H * self.Dc, eng.dtype)
        lops.gqa_prepare(self, proj, kc, vc, bt, b.tok_slot, b.pos, b.slot, q, T)
        flash = b.long is not None and self.flash
        if not flash or b.short is not None:
            t = b.tiles["tokens", self.R, flash]
            lops.gqa_attention(self, q, kc, vc, bt, b.tok_slot, b.pos, t.table, t.bm, b.key_ranges(self, t) if self.mma else 1, att, T)
        if flash:
            lops.gqa_flash(self, q, kc, vc, bt, b.tok_slot, b.pos, b.tiles["flash"].table, att, T)
        return Rows(att, self.H * self.V)


class GatedMlp:
    """W_down (act(W_gate h) * W_up h); gate and up rows are interleaved so that one output pair is one pair of neighbouring rows."""

    def __init__(self, m: dict, get, device, dtype, width: int):
        gate, up = get("gate"), get("up")
        if gate.shape != up.shape or gate.shape[0] != m["ff"]:
            raise ValueError("feed-forward: gate / up do not fit ff")
        self.w_gu = Dense.make(torch.stack([gate, up], 1).reshape(2 * gate.shape[0], gate.shape[1]), device, dtype)
        self.w_down = Dense.make(get("down"), device, dtype)

    def weights(self):
        return [self.w_gu, self.w_down]

    def buffers(self, rows: int) -> dict[str, int]:
        return {"act": rows * self.w_down.Kp}

    def apply(self, eng, r: Rows, T: int):
        act = eng.product(r, self.w_gu, eng.buf("act", T, self.w_down.Kp), T, geglu=True)
        eng.product(Rows(act, self.w_down.K), self.w_down, eng.y[:T], T)


class RoutedExperts:
    """Each token uses the `top` of `experts` small feed-forwards W_down relu(W_up h)^2 with the largest router logits (with bias), weighted by
    the softmax over those logits.  Up to four rows: three mat-vec launches (router; chosen experts' up and down products, which route for
    themselves).  More: the rows are sorted by expert and each of the two products is one grouped launch."""

    def __init__(self, m: dict, get, device, dtype, width: int):
        self.n, self.top, self.ff = m["router"]["experts"], m["router"]["top"], m["expert"]["ff"]
        if self.n > lops.MAX_EXPERTS or self.top > lops.MAX_TOP:
            raise ValueError(f"feed-forward: {self.top} of {self.n} experts (at most {lops.MAX_TOP} of {lops.MAX_EXPERTS})")
        n, F, E = self.n, pad_to(self.ff, 8), width
        self.F, self.E = F, E
        up, down = torch.zeros(n, F, pad_to(E, 8), dtype=dtype, device=device), torch.zeros(n, E, F, dtype=dtype, device=device)
        for e in range(n):
            u, d = get(f"e{e}.up"), get(f"e{e}.down")
            if u.shape != (self.ff, E) or d.shape != (E, self.ff):
                raise ValueError(f"feed-forward: expert {e} does not fit width and ff")
            up[e, :self.ff, :E] = u.to(device)
            down[e, :, :self.ff] = d.to(device)
        self.up, self.down = Dense(up.view(n * F, -1), E), Dense(down.view(n * E, F), F)
        self.router = Dense.make(get("router"), device, dtype)
        self.bias = get("router.b").to(device=device, dtype=torch.float32).contiguous()
        if self.router.N != n or self.router.K != E or self.bias.numel() != n:
            raise ValueError("feed-forward: the router does not fit experts and width")

    def weights(self):
        return [self.router, self.up, self.down]

    def buffers(self, rows: int) -> dict[str, int]:
        a = rows * self.top
        return {"router": rows * self.n, "act": a * self.F, "ids": a, "gate_w": a, "xs": a * self.up.Kp, "ey": a * self.E}

    def apply(self, eng, r: Rows, T: int):
        n, k, F, E, A = self.n, self.top, self.F, self.E, T * self.top
        logits = eng.buf("router", T, n)
        act = eng.buf("act", A, F)
        if eng.matvec_rows(T, self.router) and lops.matvec_fits(T, self.up.t) and lops.expert_matvec_fits(T, k, self.down.t):
            eng.product(r, self.router, logits, T)                # also settles the residual rows (h_out), which the up product reads again
            h = Rows(r.x if r.h_out is None else r.h_out, E, w2=r.w2, b2=r.b2)
            lops.expert_matvec(eng.stage(h, self.up.Kp), logits, self.bias, n, k, self.up.t, F, act, T, down=False)
            lops.expert_matvec(eng.stage(Rows(act, F), F), logits, self.bias, n, k, self.down.t, E, eng.y[:T], T, down=True)
            return
        x = eng.staged(r, self.up.Kp, T)
        lops.linear(x, self.router.t, logits)
        ids, w = eng.buf("ids", A, 1).view(-1), eng.buf("gate_w", A, 1).view(-1)
        lops.route(logits, self.bias, n, k, ids, w, T)
        plan, per = eng.expert_plans[n], A // n
        tile = 64 if eng.dtype == torch.float32 else 16 if per <= 16 else 32 if per <= 32 else 64 if per <= 96 else 128
        lops.expert_plan(ids, n, tile, plan)
        xs = lops.expert_gather(x, plan, k, A, eng.buf("xs", A, self.up.Kp))
        lops.linear_grouped(xs, self.up.t, F, n, tile, plan, act, relu2=True)
        ey = lops.linear_grouped(act, self.down.t, E, n, tile, plan, eng.buf("ey", A, E))
        lops.expert_combine(ey, plan, w, T, k, eng.y[:T])


MIXERS = {"hgrn2": Hgrn2, "latent_attention": LatentAttention, "attention": Attention}
MLPS = {"dense": GatedMlp, "moe": RoutedExperts}
