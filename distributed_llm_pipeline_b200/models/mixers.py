"""Token mixers and feed-forwards of layer-list models: their weights, what they keep per sequence, and their launches.

A mixer multiplies the layer input by one stacked matrix (`w_in`), mixes over the tokens of every request in the batch (`mix`), and
hands the rows of its output product (`w_out`) back.  What it keeps between steps is declared, not allocated: `planes` are per-token
rows of the paged cache, `state` is a recurrent state per sequence (models/engine.py PagedKVCache, RecurrentState).
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


class Hgrn2:
    """Gated linear recurrence with state expansion: the forget gate decides what is written; fp32 state [heads, dim, vdim]."""
    planes: dict = {}

    def __init__(self, m: dict, get, device, dtype):
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

    def mix(self, eng, il: int, proj: torch.Tensor, b) -> Rows:
        o = eng.buf("o", b.T, self.H * self.V)
        state = eng.rstate.layers[il]
        for s in (b.short, b.long):
            if s is not None:
                chunks = (s.chunk, s.first, *eng.chunk_ws) if s is b.long and self.chunked else None
                lops.hgrn2(proj, self.fbias, self.lower, state, s.range, s.slot, s.n, b.pos, o, chunks)
        return Rows(o, self.H * self.V, w2=self.norm, groups2=self.H)


class LatentAttention:
    """Softmax attention over one cached latent row per token, shared by all heads and without positions.  Queries are multiplied into
    the latent space (key matrix absorbed), the attended latent is expanded per head and gated."""
    state = None

    def __init__(self, m: dict, get, device, dtype):
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

    def mix(self, eng, il: int, proj: torch.Tensor, b) -> Rows:
        H, D, R, Rc, V = self.H, self.D, self.R, self.Rc, self.V
        cache = eng.kv.planes["c"][il]
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


class GatedMlp:
    """W_down (act(W_gate h) * W_up h); gate and up rows are interleaved so that one output pair is one pair of neighbouring rows."""

    def __init__(self, m: dict, get, device, dtype):
        gate, up = get("gate"), get("up")
        if gate.shape != up.shape or gate.shape[0] != m["ff"]:
            raise ValueError("feed-forward: gate / up do not fit ff")
        self.w_gu = Dense.make(torch.stack([gate, up], 1).reshape(2 * gate.shape[0], gate.shape[1]), device, dtype)
        self.w_down = Dense.make(get("down"), device, dtype)

    def weights(self):
        return [self.w_gu, self.w_down]


MIXERS = {"hgrn2": Hgrn2, "latent_attention": LatentAttention}
MLPS = {"dense": GatedMlp}
