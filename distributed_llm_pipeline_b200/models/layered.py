"""Step of layer-list models on the engine core: mixers of different kinds in one model, norms in front of or behind the sublayers.

The residual stream is fp32.  A sublayer's output `y` is not added at once: it stays pending, and the next matrix product forms
`h + y` (or `h + norm(y)`), and the norm in front of it, while it prepares its input rows (in the mat-vec prologue for up to four rows, in
one row kernel in front of the GEMM for more).  A mixer and a feed-forward that read the same norm share their products (mixers.Joined).  A range of layers may run several times: every run has its own cache and state, and the
embedding output may join at the start of every pass but the first.  One forward takes any mix of prompt portions and single tokens of
different sequences: projections run over all rows, mixers over the segments.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

from ..ops import api as ops
from ..ops import layers as lops
from ..ops.weights import DeviceWeight
from ..gguf.constants import GGMLType
from .engine import EngineCore, PagedKVCache, RecurrentState
from .mixers import MIXERS, MLPS, Attention, Delta, Dense, Joined, LatentAttention, RoutedExperts, Rows, XieluMlp, pad_to
from .modeldir import ModelDir, open_model_dir
from .weights import ModelWeights

DTYPES = {"bf16": torch.bfloat16, "bfloat16": torch.bfloat16, "f32": torch.float32, "float32": torch.float32}
MATVEC_ROWS = 4


@dataclass
class Norm:
    """Weight (fp32) of a norm; with a bias it is a layer norm."""
    w: torch.Tensor
    b: torch.Tensor | None = None


@dataclass
class Pending:
    """What the next product adds to the residual stream first: the sublayer output in the engine's `y` (normalised with w1, or as it is),
    and at the start of a loop pass the embedding output."""
    w1: torch.Tensor | None = None
    y: bool = True
    emb: bool = False


@dataclass
class LayeredLayer:
    mixer: object
    norm1: Norm
    mlp: object | None = None
    norm2: Norm | None = None
    joined: Joined | None = None        # mixer and feed-forward on the same norm (mlp and norm2 are None)

    @property
    def proj_cols(self) -> int:
        return self.mixer.w_in.N if self.joined is None else self.joined.n

    def join(self):
        """Run mixer and feed-forward side by side, behind norm1."""
        if not isinstance(self.mlp, XieluMlp):
            raise NotImplementedError(f"parallel sublayers with a feed-forward of {type(self.mlp).__name__}")
        self.joined, self.mlp = Joined(self.mixer, self.mlp), None

    def weights(self):
        return self.mixer.weights() + (self.mlp.weights() if self.mlp is not None else [])


class LayeredWeights(ModelWeights):
    def nbytes(self) -> int:
        return sum(w.nbytes for lw in self.layers.values() for w in lw.weights()) + self.tok_embd.nbytes + self.lm_head.nbytes


def load_layered_weights(src: str | ModelDir, device, dtype="bf16", progress=None) -> LayeredWeights:
    """Weights of a model folder on the device, in the storage type `dtype` (bf16 | f32); norms, biases and gate bounds are fp32."""
    from .weights import LoadCancelled
    d = open_model_dir(src) if isinstance(src, str) else src
    dt = DTYPES[dtype] if isinstance(dtype, str) else dtype
    cfg, f, dev = d.cfg, d.tensors, torch.device(device)

    def f32(name, n):
        t = f.tensor(name).to(device=dev, dtype=torch.float32).contiguous()
        if t.shape != (n,):
            raise ValueError(f"{name} has the shape {tuple(t.shape)}, expected ({n},)")
        return t

    def norm(name):
        return Norm(f32(name, cfg.n_embd) + cfg.norm_offset, f32(name + ".b", cfg.n_embd) if cfg.norm_type == "layer" else None)
    layers = {}
    for il, spec in enumerate(cfg.layers):
        if progress is not None and progress(il / cfg.n_layer) is False:
            raise LoadCancelled("load cancelled")
        p = f"l{il}."
        lw = LayeredLayer(MIXERS[spec.type](spec.mixer, lambda n: f.tensor(p + "mix." + n), dev, dt, cfg.rms_eps), norm(p + "norm1"))
        if lw.mixer.w_in.K != cfg.n_embd or lw.mixer.w_out.N != cfg.n_embd:
            raise ValueError(f"layer {il}: a mixer projection does not fit the width")
        if spec.mlp is not None:
            lw.mlp = MLPS[spec.mlp["kind"]](spec.mlp, lambda n: f.tensor(p + "mlp." + n), dev, dt, cfg.n_embd)
            if cfg.parallel_residual:
                lw.join()
            else:
                lw.norm2 = norm(p + "norm2")
        layers[il] = lw

    def table(name):
        w = Dense.make(f.tensor(name), dev, dt)
        if w.N != cfg.vocab_size or w.K != cfg.n_embd:
            raise ValueError(f"{name} is [{w.N}, {w.K}], expected [{cfg.vocab_size}, {cfg.n_embd}]")
        return DeviceWeight(GGMLType.F32 if dt == torch.float32 else GGMLType.BF16, w.N, w.K, [w.t])
    emb, head = table("embed"), table("head")
    out_norm = norm("final.norm")
    if progress is not None and progress(1.0) is False:
        raise LoadCancelled("load cancelled")
    return LayeredWeights(cfg, layers, range(cfg.n_layer), 0, 1, emb, out_norm.w, head, (0, cfg.vocab_size), None, out_norm_b=out_norm.b)


@dataclass
class TileTable:
    """Row tiles of one attention shape: (token, head) rows for latent attention, tokens for the others."""
    row0: torch.Tensor
    rows: torch.Tensor
    n: int
    bm: int
    n_splits: int = 1

    @property
    def table(self):
        return self.row0, self.rows, self.n


@dataclass
class Segments:
    """Row ranges of some of a batch's sequences."""
    n: int
    range: torch.Tensor         # [n, 2] first row, row behind the last
    slot: torch.Tensor          # [n] sequence slot
    longest: int = 1            # tokens of the longest one
    chunks: dict | None = None  # long segments, by chunk size: ([chunks, 2] first row and length, [n + 1] first chunk of every segment)
    host: tuple = ()            # long segments: (sequence slot, first row, row behind the last, cached tokens with them)


@dataclass
class Batch:
    """Device-side description of one forward: T rows, grouped into segments (one per sequence), short segments first.  Recurrent mixers
    scan the short ones token by token and take the long ones in chunks; latent attention expands keys and values for the long ones."""
    T: int
    T_short: int
    short: Segments | None
    long: Segments | None
    tok_slot: torch.Tensor      # [T] sequence slot of every row
    pos: torch.Tensor           # [T]
    slot: torch.Tensor          # [T] cache row
    # latent attention: (its kind, short only); windowed attention: ("tokens", query heads per key / value head, short only), "flash"
    tiles: dict[object, TileTable]
    decode: bool = False        # one token of every sequence
    longest: int = 0            # tokens of the longest sequence, these included
    ranges: dict[tuple, int] | None = None      # key ranges of the windowed attentions of a decode step (None: chosen by `longest`)

    def key_ranges(self, m: Attention, t: TileTable) -> int:
        return self.ranges[key_range_kind(m)] if self.ranges is not None else key_ranges(m, t.n, t.bm, self.longest)


def key_range_kind(m: Attention) -> tuple:
    return m.G, m.R, m.window, m.keep, m.chunk


def key_ranges(m: Attention, n_tiles: int, bm: int, longest: int) -> int:
    """Parts the visible keys are split into: about two blocks per SM, at least 64 keys each, at most a cluster of 16 blocks."""
    want, n = min(2 * 148 // (n_tiles * lops.gqa_blocks(m.G, m.R, bm)), (m.visible(longest) + 63) // 64, 16), 1
    while n * 2 <= want:
        n *= 2
    return n


class LayeredEngine(EngineCore):
    mixed_batches = True
    can_shift = False           # a recurrent state has no positions to slide, and cached keys are rotated

    def __init__(self, weights: LayeredWeights, n_ctx: int = 4096, max_seqs: int = 8, page_size: int = 64, max_batch_tokens: int = 2048,
                 n_pages: int | None = None, comm=None, first_stage: bool = True, last_stage: bool = True):
        cfg = weights.cfg
        if comm is not None and comm.tp_size > 1 or not (first_stage and last_stage):
            raise NotImplementedError(f"{cfg.arch}: layer-list models run on one GPU (no tensor-parallel or pipeline split)")
        dev = weights.tok_embd.device
        self._init_core(weights, n_ctx, max_seqs, page_size, max_batch_tokens, comm, True, True, dev)
        if dev.type == "cuda":
            lops.load_library()
        self.dtype = weights.tok_embd.planes[0].dtype
        self.E = cfg.n_embd
        self.runs = cfg.layer_runs()
        mixers = {r: weights.layers[il].mixer for r, (il, _) in enumerate(self.runs)}      # by run: what a run keeps is its own
        mlps = [lw.mlp for lw in weights.layers.values() if lw.mlp is not None]
        max_pages = (n_ctx + page_size - 1) // page_size
        planes: dict[str, dict] = {}
        for r, m in mixers.items():
            for name, shape in m.planes.items():
                planes.setdefault(name, {})[r] = shape
        self.kv = PagedKVCache(planes, max_pages * max_seqs if n_pages is None else n_pages, page_size, max_seqs, max_pages, dev, dtype=self.dtype)
        states: dict[str, dict] = {}
        for r, m in mixers.items():
            for name, shape in m.states.items():
                states.setdefault(name, {})[r] = shape
        self.rstate = RecurrentState(states, max_seqs, dev)
        self.head_norm = weights.out_norm / cfg.logit_scale          # the logit scale is part of the last norm
        M, f32 = self.max_rows, torch.float32
        self.hb = [torch.zeros(M, self.E, dtype=f32, device=dev) for _ in range(2)]      # residual stream; the mat-vec path alternates
        self.h = self.hb[0]
        self.cur = 0                                                 # which of them holds it (-1: still the embedding output)
        self.emb = torch.zeros(M, self.E, dtype=f32, device=dev) if any(again for _, again in self.runs) else None
        self.y = torch.zeros(M, self.E, dtype=f32, device=dev)
        joined = [lw.joined for lw in weights.layers.values() if lw.joined is not None]
        sizes = {"proj": M * max(lw.proj_cols for lw in weights.layers.values()), "xb": M * max([pad_to(self.E, 8)] + [w.Kp for lw in weights.layers.values() for w in lw.weights()])}
        for part in [*mixers.values(), *mlps, *joined]:
            for name, n in part.buffers(M).items():
                sizes[name] = max(sizes.get(name, 0), n)
        types = {"proj": f32, "o": f32, "router": f32, "gate_w": f32, "ey": f32, "ys": f32, "q_up": f32, "v_first": f32, **{n: f32 for n in Delta.WORKSPACES}, "ids": torch.int32}
        self._flat = {n: torch.zeros(sz, dtype=types.get(n, self.dtype), device=dev) for n, sz in sizes.items()}
        experts = [m for m in mlps if isinstance(m, RoutedExperts)]
        self.expert_plans = {n: ops.MoePlan(M * max(m.top for m in experts), n, dev) for n in {m.n for m in experts}}
        self.logits = torch.zeros(max_seqs, cfg.vocab_size, dtype=f32, device=dev)
        lat = [m for m in mixers.values() if isinstance(m, LatentAttention)]
        self._latent_kinds = sorted({m.kind for m in lat})
        att = [m for m in mixers.values() if isinstance(m, Attention)]
        self._att_kinds = {key_range_kind(m): m for m in att}
        self._att_groups = sorted({m.R for m in att})
        self._att_flash = any(m.flash for m in att)
        self._att_all_flash = all(m.flash for m in att)
        self._split_ctas = 148                                       # one CTA per SM: the key range is split until they are there
        self.latent_ws = None
        if lat:
            rows = self._split_ctas * 64
            self.latent_ws = (torch.zeros(rows * max(m.Vc for m in lat), dtype=f32, device=dev), torch.zeros(rows * 2, dtype=f32, device=dev))
        # segments from this length on take the chunked recurrence and the expanded / flash attention (bf16 storage; fp32 always takes the others)
        self.long_from = lops.LONG_FROM if self.dtype == torch.bfloat16 else 1 << 60
        self._expanding_kinds = {m.kind for m in lat if m.expand} - {m.kind for m in lat if not m.expand}
        chunked = [m for m in mixers.values() if m.states and m.chunk]
        self._chunk_sizes = sorted({m.chunk for m in chunked})
        self.chunk_ws = None
        own = [m for m in chunked if not isinstance(m, Delta)]       # (the delta rule's workspaces are buffers)
        if own and self.long_from <= M:
            n = lops.most_chunks(M, self._chunk_sizes[0])
            self.chunk_ws = tuple(torch.zeros(n * max(m.H * m.D * w(m) for m in own), dtype=f32, device=dev) for w in (lambda m: m.V, lambda m: 1))
        self._variant = (1,) * (len(self._latent_kinds) + len(self._att_kinds))      # key ranges per decode query: every kind of latent, then of windowed attention
        self._decode_batches: dict[tuple, Batch] = {}

    def buf(self, name: str, rows: int, cols: int, dtype=None) -> torch.Tensor:
        return self._flat[name][:rows * cols].view(rows, cols)

    def flat(self, name: str) -> torch.Tensor:
        return self._flat[name]

    def grow(self, name: str, rows: int, cols: int) -> torch.Tensor:
        """A buffer in the storage type that grows with the longest context it was asked for (by half again, so that it settles)."""
        n = rows * cols
        if name not in self._flat or self._flat[name].numel() < n:
            self._flat[name] = torch.zeros(n + n // 2, dtype=self.dtype, device=self.device)
        return self.buf(name, rows, cols)

    # ---- matrix products -------------------------------------------------------------------------------
    def stage(self, r: Rows, Kp: int):
        """The row preparation of `r` as the kernels take it."""
        return lops.row_stage(r.x, r.K, Kp, self.cfg.rms_eps, r.y, r.w1, self.cfg.norm_groups if r.w1 is not None else 1, r.h_out, r.w2, r.groups2, r.b2, r.e, r.pair, r.lam, r.g, r.gate,
                              r.tail)

    def staged(self, r: Rows, Kp: int, T: int) -> torch.Tensor:
        """Rows of `r` in the storage type, prepared by one launch if they are not there as they are."""
        if r.y is None and r.w2 is None and r.e is None and r.g is None and not r.pair and r.x.dtype == self.dtype and r.x.shape[1] == Kp:
            return r.x[:T]
        return lops.stage_rows(self.stage(r, Kp), self.buf("xb", T, Kp), T)

    def matvec_rows(self, T: int, w: Dense) -> bool:
        return T <= MATVEC_ROWS and lops.matvec_fits(T, w.t)

    def product(self, r: Rows, w: Dense, out: torch.Tensor, T: int, act: int = lops.OUT_F32, tail=None) -> torch.Tensor:
        """tail: what follows the sums (ops.layers.out_tail)."""
        if self.matvec_rows(T, w):
            return lops.matvec(self.stage(r, w.Kp - (r.tail.shape[1] if r.tail is not None else 0)), w.t, out, T, act, tail)
        return lops.linear(self.staged(r, w.Kp, T), w.t, out, act, tail)

    def _residual(self, T: int, pending: Pending | None, pre: Norm | None = None) -> Rows:
        """Rows of the residual stream with what is pending folded in on the way, and the norm `pre` in front of a sublayer."""
        src = (self.hb[self.cur] if self.cur >= 0 else self.emb)[:T]
        r = Rows(src, self.E)
        if pending is not None:
            # every block of a mat-vec reads the old rows: the new ones go to the other buffer (and the embedding output stays as it is)
            self.cur = max(0, self.cur ^ 1 if T <= MATVEC_ROWS else self.cur)
            r = Rows(src, self.E, y=self.y[:T] if pending.y else None, w1=pending.w1, h_out=self.hb[self.cur][:T], e=self.emb[:T] if pending.emb else None)
        if pre is not None:
            r.w2, r.b2 = pre.w, pre.b
        return r

    def _settle(self, T: int, pending: Pending | None):
        """Fold what is pending into the residual stream now; returns the rows [T, E] fp32."""
        if pending is not None:
            src = (self.hb[self.cur] if self.cur >= 0 else self.emb)[:T]
            self.cur = max(0, self.cur)
            h = self.hb[self.cur][:T]
            r = Rows(src, self.E, y=self.y[:T] if pending.y else None, w1=pending.w1, h_out=h, e=self.emb[:T] if pending.emb else None)
            lops.stage_rows(self.stage(r, self.E), self.buf("xb", T, self.E), T)
        return self.hb[self.cur][:T]

    # ---- one forward over a batch ------------------------------------------------------------------------
    def _forward(self, ids: torch.Tensor, b: Batch) -> Pending | None:
        """Embedding and all layers; returns what is still to be added to the residual stream (None: nothing)."""
        T, pre = b.T, self.cfg.pre_norm
        self.cur = 0 if self.emb is None else -1
        lops.embed(self.w.tok_embd.planes[0], ids, self.hb[0] if self.emb is None else self.emb, T, self.cfg.embedding_scale)
        pending = None
        for run, (il, again) in enumerate(self.runs):
            lw = self.w.layers[il]
            m = lw.mixer
            if again:
                pending = Pending(pending.w1, True, True) if pending is not None else Pending(None, False, True)
            rows = self._residual(T, pending, lw.norm1 if pre else None)
            if lw.joined is not None:
                lw.joined.apply(self, run, rows, b)
            else:
                proj = self.product(rows, m.w_in, self.buf("proj", T, m.w_in.N), T, tail=lops.out_tail(m.bias) if m.bias is not None else None)
                self.product(m.mix(self, run, proj, b), m.w_out, self.y[:T], T)
            pending = Pending(None if pre else lw.norm1.w)
            if lw.mlp is not None:
                lw.mlp.apply(self, self._residual(T, pending, lw.norm2 if pre else None), T)
                pending = Pending(None if pre else lw.norm2.w)
            if self.eval_callback is not None or il in self.cvec:
                h = self._settle(T, pending)
                pending = None
                if il in self.cvec:
                    h.add_(self.cvec[il])
                if self.eval_callback is not None:
                    self.eval_callback("l_out", run, h)
        return pending

    def _head_rows(self, r: Rows, n: int, out: torch.Tensor) -> torch.Tensor:
        r.w2, r.b2, r.groups2 = self.head_norm, self.w.out_norm_b, self.cfg.norm_groups
        head = self.w.lm_head
        return self.product(r, Dense(head.planes[0], head.K), out, n)

    # ---- batch descriptions ---------------------------------------------------------------------------------
    def _n_splits(self, n_tiles: int, max_len: int) -> int:
        want, n = min(self._split_ctas // max(1, n_tiles), (max_len + 63) // 64, 32), 1
        while n * 2 <= want:
            n *= 2
        return n

    @staticmethod
    def _token_tiles(segs: list[tuple[int, int]], n: int) -> tuple[list[int], list[int]]:
        """First row and length of every tile of up to n rows, for row ranges."""
        tiles = [(t, min(n, hi - t)) for lo, hi in segs for t in range(lo, hi, n)]
        return [t for t, _ in tiles], [c for _, c in tiles]

    def _tile_lists(self, H: int, lens: list[int], bm: int):
        row0, rows, base = [], [], 0
        for n in lens:
            for i in range(0, n * H, bm):
                row0.append(base + i)
                rows.append(min(bm, n * H - i))
            base += n * H
        return row0, rows

    def _decode_batch(self, B: int) -> Batch:
        b = self._decode_batches.get((B, self._variant))
        if b is None:
            dev, i32 = self.device, torch.int32
            tiles = {}
            for kind, splits in zip(self._latent_kinds, self._variant):
                H, _, Rc = kind
                bm = lops.latent_tile_rows(H, B, Rc)
                row0, rows = self._tile_lists(H, [1] * B, bm)
                tiles[kind, False] = TileTable(torch.tensor(row0, dtype=i32, device=dev), torch.tensor(rows, dtype=i32, device=dev), len(row0), bm, min(splits, max(1, self._split_ctas // len(row0))))
            rng = torch.tensor([[i, i + 1] for i in range(B)], dtype=i32, device=dev)
            rows = torch.arange(B, dtype=i32, device=dev), torch.ones(B, dtype=i32, device=dev)
            tiles |= {("tokens", R, False): TileTable(*rows, B, lops.gqa_tile(R, 1)[0]) for R in self._att_groups}
            b = Batch(B, B, Segments(B, rng, self.active), None, self.active, self.pos, self.slot, tiles, decode=True,
                      ranges=dict(zip(self._att_kinds, self._variant[len(self._latent_kinds):])))
            self._decode_batches[(B, self._variant)] = b
        return b

    def _mixed_batch(self, parts: list[tuple[int, list[int]]]) -> tuple[torch.Tensor, Batch]:
        """Grow every sequence by its tokens (short parts first) and upload the description in one copy."""
        lens = [len(t) for _, t in parts]
        T = sum(lens)
        pos, slot = zip(*(self._advance_inputs(sid, len(t)) for sid, t in parts))
        cols: list[torch.Tensor] = [torch.cat([torch.as_tensor(t, dtype=torch.int32) for _, t in parts]), torch.cat(pos), torch.cat(slot),
                                    torch.cat([torch.full((len(t),), sid, dtype=torch.int32) for sid, t in parts])]
        ends = torch.tensor(lens).cumsum(0).tolist()
        segs = [(sid, hi - n, hi) for (sid, _), n, hi in zip(parts, lens, ends)]
        groups = [[g for g in segs if (g[2] - g[1] >= self.long_from) == is_long] for is_long in (False, True)]
        assert [g for grp in groups for g in grp] == segs
        T_short = groups[0][-1][2] if groups[0] else 0
        for is_long, grp in zip((False, True), groups):
            lists = [[x for g in grp for x in g[1:]], [g[0] for g in grp]]
            for size in self._chunk_sizes if is_long else ():
                lists += lops.scan_chunk_table([g[1:] for g in grp], size)
            cols += [torch.tensor(x, dtype=torch.int32) for x in lists]
        shapes = []
        for kind in self._latent_kinds:
            H, _, Rc = kind
            for only_short, n in ((False, len(lens)), (True, len(groups[0]))):
                if only_short and (not groups[1] or not n) or not only_short and groups[1] and kind in self._expanding_kinds:
                    continue
                bm = lops.latent_tile_rows(H, sum(lens[:n]), Rc)
                row0, rows = self._tile_lists(H, lens[:n], bm)
                cols += [torch.tensor(row0, dtype=torch.int32), torch.tensor(rows, dtype=torch.int32)]
                shapes.append(((kind, only_short), bm, len(row0)))
        for R in self._att_groups:
            for only_short in (False, True):
                part = groups[0] if only_short else segs
                if only_short and (not groups[1] or not part) or not only_short and groups[1] and self._att_all_flash:
                    continue
                bm, n = lops.gqa_tile(R, max(g[2] - g[1] for g in part))
                row0, rows = self._token_tiles([g[1:] for g in part], n)
                cols += [torch.tensor(row0, dtype=torch.int32), torch.tensor(rows, dtype=torch.int32)]
                shapes.append((("tokens", R, only_short), bm, len(row0)))
        if groups[1] and self._att_flash:       # the tiles with the longest context first
            order = sorted(((self.seqs[sid].length + t - lo, t, n) for sid, lo, hi in groups[1] for t, n in zip(*self._token_tiles([(lo, hi)], lops.FLASH_TILE))), reverse=True)
            row0, rows = [t for _, t, _ in order], [n for _, _, n in order]
            cols += [torch.tensor(row0, dtype=torch.int32), torch.tensor(rows, dtype=torch.int32)]
            shapes.append(("flash", lops.FLASH_TILE, len(row0)))
        dev = iter(torch.cat(cols).to(self.device).split([c.numel() for c in cols]))
        ids, pos_d, slot_d, tok_slot = (next(dev) for _ in range(4))
        most = [max((hi - lo for _, lo, hi in grp), default=0) for grp in groups]
        short = Segments(len(groups[0]), next(dev), next(dev), longest=most[0])
        long = Segments(len(groups[1]), next(dev), next(dev), most[1], {size: (next(dev).view(-1, 2), next(dev)) for size in self._chunk_sizes},
                        tuple((sid, lo, hi, self.seqs[sid].length + hi - lo) for sid, lo, hi in groups[1]))
        longest = max(self.seqs[sid].length + len(t) for sid, t in parts)
        # (latent attention: a tile sees its rows' windows)
        tiles = {key: TileTable(next(dev), next(dev), nt, bm, self._n_splits(nt, min(longest, key[0][1] + bm)) if key[0] in self._latent_kinds else 1) for key, bm, nt in shapes}
        return ids, Batch(T, T_short, short if short.n else None, long if long.n else None, tok_slot, pos_d, slot_d, tiles, longest=longest)

    def _run_mixed(self, parts: list[tuple[int, list[int]]]):
        """Forward over one mixed batch; updates the sequence lengths.  Returns what is pending (see _forward)."""
        ids, b = self._mixed_batch(parts)
        pending = self._forward(ids, b)
        for sid, t in parts:
            self.seqs[sid].length += len(t)
        lens = torch.tensor([[sid, self.seqs[sid].length] for sid, _ in parts], dtype=torch.int32).to(self.device)
        self.seq_len_dev[lens[:, 0].long()] = lens[:, 1]
        return pending

    # ---- public ---------------------------------------------------------------------------------------------
    @torch.no_grad()
    def step(self, entries, want=None) -> torch.Tensor:
        """Append tokens to several sequences in one batch.  entries: [(sid, tokens)], every sequence at most once, portions of any length
        beside single tokens; want: for every entry the places among its tokens whose logits are returned (default: the last one).
        Returns fp32 logits [wanted, vocab] in the order of the entries.  A batch of single tokens is a decode step and runs as one
        (captured graph); more tokens than the engine's batch holds run as several forwards."""
        entries = [(sid, toks.tolist() if isinstance(toks, torch.Tensor) else list(toks)) for sid, toks in entries]
        if want is None:
            want = [[len(t) - 1] for _, t in entries]
        if len({sid for sid, _ in entries}) != len(entries) or any(not t for _, t in entries):
            raise ValueError("step: every sequence may appear once, with at least one token")
        if any(not 0 <= p < len(t) for (_, t), w in zip(entries, want) for p in w):
            raise ValueError("step: a wanted place outside its tokens")
        self._reserve([(sid, len(t)) for sid, t in entries])
        if all(len(t) == 1 for _, t in entries):
            lg = self.decode([sid for sid, _ in entries], [t[0] for _, t in entries], sample=False)
            rows = [i for i, w in enumerate(want) for _ in w]
            return lg[torch.tensor(rows, dtype=torch.long, device=self.device)].clone()
        out = torch.empty(sum(len(w) for w in want), self.cfg.vocab_size, dtype=torch.float32, device=self.device)
        offs = [0]
        for w in want:
            offs.append(offs[-1] + len(w))
        done = [0] * len(entries)
        while any(d < len(t) for d, (_, t) in zip(done, entries)):
            room, cut = self.max_tokens, []
            for i, (_, toks) in enumerate(entries):
                n = min(room, len(toks) - done[i])
                if n > 0:
                    cut.append((i, n))
                    room -= n
            parts, rows, dst, base = [], [], [], 0
            for i, n in sorted(cut, key=lambda c: c[1] >= self.long_from):      # short parts first
                sid, toks = entries[i]
                for j, p in enumerate(want[i]):
                    if done[i] <= p < done[i] + n:
                        rows.append(base + p - done[i])
                        dst.append(offs[i] + j)
                parts.append((sid, toks[done[i]:done[i] + n]))
                done[i] += n
                base += n
            pending = self._run_mixed(parts)
            if rows:
                h = self._settle(sum(len(t) for _, t in parts), pending)
                for k in range(0, len(rows), self.max_rows):
                    idx = torch.tensor(rows[k:k + self.max_rows], dtype=torch.long, device=self.device)
                    lg = self._head_rows(Rows(h[idx], self.E), len(idx), torch.empty(len(idx), self.cfg.vocab_size, dtype=torch.float32, device=self.device))
                    out[torch.tensor(dst[k:k + self.max_rows], dtype=torch.long, device=self.device)] = lg
        if self.device.type == "cuda":
            lops.check_waits()
        return out

    def _reserve(self, grow):
        """Refuse a batch that the pool cannot hold before anything of it is appended."""
        need = 0
        for sid, n in grow:
            seq = self.seqs[sid]
            if seq.length + n > self.n_ctx:
                raise RuntimeError(f"sequence {sid}: context {seq.length + n} exceeds n_ctx")
            need += self.pages_needed(sid, n)
        if need > len(self.kv.free):
            raise RuntimeError("KV cache exhausted (no free pages)")

    @torch.no_grad()
    def prefill(self, sid: int, tokens, hidden_in=None, chunk: int | None = None, all_logits: bool = False):
        """Append `tokens` to one sequence; logits [vocab] of the last token, or [T, vocab] of all of them."""
        toks = tokens.tolist() if isinstance(tokens, torch.Tensor) else list(tokens)
        chunk = min(chunk or len(toks), len(toks))
        outs = []
        for c0 in range(0, len(toks), chunk):
            part = toks[c0:c0 + chunk]
            outs.append(self.step([(sid, part)], [list(range(len(part))) if all_logits else [len(part) - 1]]))
        return torch.cat(outs) if all_logits else outs[-1][-1]

    @torch.no_grad()
    def embed(self, tokens, pooling: str = "mean", normalize: bool = True) -> torch.Tensor:
        """Pooled final-norm hidden states of `tokens` (`mean` | `last` | `cls` | `none`), in a scratch sequence slot."""
        if pooling not in ("mean", "last", "cls", "none"):
            raise ValueError(f"unknown pooling {pooling!r}")
        tokens = list(tokens)
        if len(tokens) > self.max_tokens:
            raise ValueError(f"{len(tokens)} tokens exceed the batch limit {self.max_tokens}")
        sid = self.alloc_seq()
        try:
            h = self._settle(len(tokens), self._run_mixed([(sid, tokens)]))
            st = self.stage(Rows(h, self.E, w2=self.w.out_norm, groups2=self.cfg.norm_groups, b2=self.w.out_norm_b), self.E)
            xn = lops.stage_rows(st, self.buf("xb", len(tokens), self.E), len(tokens)).float()
        finally:
            self.free_seq(sid)
        e = {"mean": lambda: xn.mean(0), "last": lambda: xn[-1], "cls": lambda: xn[0], "none": lambda: xn}[pooling]()
        return torch.nn.functional.normalize(e, dim=-1) if normalize else e.clone()

    def _choose_variant(self, B: int, max_len: int):
        lat = []
        for H, window, Rc in self._latent_kinds:
            bm = lops.latent_tile_rows(H, B, Rc)
            lat.append(self._n_splits(B * ((H + bm - 1) // bm), min(max_len, window)))
        self._variant = (*lat, *(key_ranges(m, B, lops.gqa_tile(m.R, 1)[0], max_len) if m.mma else 1 for m in self._att_kinds.values()))

    def _decode_body(self, B: int, sample: bool):
        ops.advance(self.seq_len_dev, self.active, self.pos, self.slot, self.kv_len, self.kv.block_table, self.page_size, B)
        pending = self._forward(self.next_tok, self._decode_batch(B))
        lg = self._head_rows(self._residual(B, pending), B, self.logits[:B])
        self.logits_full = lg
        if sample:
            ops.sample_dev(lg, self.samp, self.active[:B], self.next_tok[:B])

    def set_control_vector(self, src, scale: float = 1.0, layer_range: tuple[int, int] | None = None):
        """{layer: vector [width]} added to the residual stream behind that layer; None clears."""
        self.cvec = {}
        self._graphs.clear()
        lo, hi = layer_range or (0, self.cfg.n_layer)
        for il, v in (src or {}).items():
            if lo <= il < hi:
                if v.numel() != self.E:
                    raise ValueError(f"control vector for layer {il} has {v.numel()} elements, the model is {self.E} wide")
                self.cvec[il] = (v.float() * scale).to(self.device)

    def memory_breakdown(self) -> dict:
        act = sum(t.numel() * t.element_size() for t in [*self.hb, *([self.emb] if self.emb is not None else []), self.y, self.logits, *self._flat.values(), *(self.latent_ws or ())])
        return {"model": self.w.nbytes(), "kv_cache": self.kv.bytes(), "recurrent_state": self.rstate.bytes(), "compute": act, "graphs": len(self._graphs),
                "device": str(self.device)}
