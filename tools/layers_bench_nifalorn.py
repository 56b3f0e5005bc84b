"""Nifalorn's part of tools/layers_bench.py: a model of every mixer with routed and shared experts beside a Vozinex of equal weight bytes, and its
kernels beside the like ones of Vozinex and Talizen on the same sizes."""
from __future__ import annotations

from types import SimpleNamespace

import torch

DEV = "cuda:0"
VOCAB = 32000
# name: (width, recurrent heads of 128 x 128, Mamba-2 heads of 64 with a state of 128 in 8 groups, attention heads of 2 x 64 keys and 128 values, key / value heads,
#        experts, experts per token, ff of an expert, ff of the shared one, layers, chunk)
HYBRID_SIZES = {
    "hybrid-2048": (2048, 16, 64, 16, 4, 64, 8, 768, 768, 4, 2048),
    "hybrid-4096": (4096, 32, 128, 32, 8, 16, 2, 4096, 4096, 4, 2048),
}


def mat(r, c):
    return (torch.randn(r, c, device=DEV) * c ** -0.5).to(torch.bfloat16)


def weights(cfg, norm_b, vec, shapes):
    """Random weights of a layer list on the device; `shapes` / `vec` name the matrices and vectors of a layer by its type."""
    from distributed_llm_pipeline_b200.gguf.constants import GGMLType
    from distributed_llm_pipeline_b200.models.layered import LayeredLayer, LayeredWeights, Norm
    from distributed_llm_pipeline_b200.models.mixers import MIXERS, MLPS
    from distributed_llm_pipeline_b200.ops.weights import DeviceWeight
    E = cfg.n_embd

    def get(kind):
        def g(name):
            key = name.split(".")[-1] if name[0] == "e" and name[1:2].isdigit() else name
            return mat(*shapes[kind][key]) if key in shapes[kind] else vec[kind][key]
        return g
    norm = Norm(torch.ones(E, device=DEV), torch.zeros(E, device=DEV) if norm_b else None)
    layers = {i: LayeredLayer(MIXERS[s.type](s.mixer, get(s.type), DEV, torch.bfloat16, 1e-5), norm, MLPS[s.mlp["kind"]](s.mlp, get("mlp"), DEV, torch.bfloat16, E), norm)
              for i, s in enumerate(cfg.layers)}
    if cfg.parallel_residual:
        for lw in layers.values():
            lw.join()
    tab = [DeviceWeight(GGMLType.BF16, VOCAB, E, [mat(VOCAB, E)]) for _ in range(2)]
    return LayeredWeights(cfg, layers, range(len(layers)), 0, 1, tab[0], norm.w, tab[1], (0, VOCAB), None, out_norm_b=norm.b)


def nifalorn(size: str):
    """Lightning, Mamba-2, lightning, attention; experts in every layer."""
    from distributed_llm_pipeline_b200.models.modeldir import nifalorn_config
    E, H, M, A, G, NE, k, F, Fs, n, chunk = HYBRID_SIZES[size]
    mlp = {"kind": "moe", "expert": {"ff": F}, "router": {"experts": NE, "top": k, "groups": {"count": 4, "keep": 2}, "scale": 2.5}, "shared": {"ff": Fs}}
    li = {"type": "lightning", "mixer": {"heads": H, "dim": 128, "vdim": 128, "decay": [0.99] * H}, "mlp": mlp}
    ma = {"type": "mamba2", "mixer": {"heads": M, "vdim": 64, "state": 128, "groups": 8, "conv": 4, "norm_groups": 8}, "mlp": mlp}
    at = {"type": "attention", "mlp": mlp, "mixer": {"heads": A, "kv_heads": G, "dim": 64, "vdim": 128, "scale": 0.125, "diff": 0.5, "mask": {"size": chunk},
                                                      "rot": {"dims": 64, "base": 5e5, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}}}
    cfg = nifalorn_config({"width": E, "vocab": VOCAB, "norm": {"eps": 1e-5}, "layers": ([li, ma, li, at] * n)[:n], "embedding": {"scale": 1.0}, "logit_scale": 1.0})
    inner, ch = 64 * M, 64 * M + 2 * 8 * 128
    shapes = {"lightning": {x: (128 * H, E) for x in "qkvg"} | {"o": (E, 128 * H)}, "mamba2": {"in": (inner + ch + M, E), "o": (E, inner), "conv": (ch, 4)},
              "attention": {"q": (128 * A, E), "k": (128 * G, E), "v": (128 * G, E), "o": (E, 128 * A)},
              "mlp": {"gate": (F, E), "up": (F, E), "down": (E, F), "router": (NE, E), "shared.gate": (Fs, E), "shared.up": (Fs, E), "shared.down": (E, Fs), "shared.sg": (1, E)}}
    vec = {"lightning": {"norm": torch.ones(128 * H)}, "attention": {x: torch.full((64,), 0.1) for x in ("lq1", "lk1", "lq2", "lk2")}, "mlp": {"correction": torch.zeros(NE)},
           "mamba2": {"conv.b": torch.zeros(ch), "dt_bias": torch.full((M,), -2.0), "A_log": torch.zeros(M), "D": torch.ones(M), "norm": torch.ones(inner)}}
    return weights(cfg, False, vec, shapes)


def vozinex(size: str):
    """Attention of the same heads and cache bytes, and two matrices per expert instead of three: one and a half times their width, with one expert
    more per token in the place of the shared one (and the recurrent layers' bytes left out)."""
    from distributed_llm_pipeline_b200.models.modeldir import vozinex_config
    E, _, _, A, G, NE, k, F, _, n, chunk = HYBRID_SIZES[size]
    F = F * 3 // 2
    spec = {"type": "attention", "mixer": {"heads": A, "kv_heads": G, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "rot": {"dims": 128, "base": 1e6}, "mask": {"size": chunk, "keep_first": 0}},
            "mlp": {"kind": "moe", "expert": {"ff": F}, "router": {"experts": NE, "top": k + 1}}}
    cfg = vozinex_config({"width": E, "vocab": VOCAB, "norm": {"eps": 1e-5}, "layers": [spec] * n})
    shapes = {"attention": {"q": (128 * A, E), "k": (128 * G, E), "v": (128 * G, E), "o": (E, 128 * A)}, "mlp": {"up": (F, E), "down": (E, F), "router": (NE, E)}}
    vec = {"attention": {"q.norm": torch.ones(128 * A), "k.norm": torch.ones(128 * G)}, "mlp": {"router.b": torch.zeros(NE)}}
    return weights(cfg, True, vec, shapes)


def kernel_numbers(size: str, graph_us, copies, peaks, T: int = 2048):
    """Rows (model, kind, kernel, us, roofline) of Nifalorn's kernels and of the like ones."""
    from distributed_llm_pipeline_b200.models.layered import key_ranges
    from distributed_llm_pipeline_b200.ops import api as ops
    from distributed_llm_pipeline_b200.ops import layers as L
    L.load_library()
    E, H, M, A, G, NE, k, F, Fs, _, chunk = HYBRID_SIZES[size]
    D, N, inner = 128, 128, 64 * M
    ch = inner + 16 * N
    bf, f32, i32 = torch.bfloat16, torch.float32, torch.int32
    bw, fl, src = peaks()
    rows = []

    def rnd(*s, dt=bf):
        return (torch.randn(*s, device=DEV) * 0.1).to(dt)

    def ints(x):
        return torch.tensor(x, device=DEV, dtype=i32)

    def add(model, kind, name, us, nbytes, flops):
        roof = max(nbytes / bw, flops / fl) * 1e6
        rows.append({"model": model, "kind": kind, "kernel": name, "us": round(us, 2), "roofline_us": round(roof, 2), "of_roofline": round(roof / us, 3)})
    ones, zero = torch.ones(max(E, inner), device=DEV), torch.zeros(E, device=DEV)
    HD, AD = H * D, A * D

    def mixer_rows(kind, B):
        """Staged rows of an output product, as the mixers hand them on; their width; the tensors they point to, to be kept."""
        if kind == "lightning":
            x, g, w2 = rnd(B, HD, dt=f32), rnd(B, 4 * HD, dt=f32), torch.ones(HD, device=DEV)
            return L.row_stage(x, HD, HD, 1e-5, w2=w2, g=g[:, 3 * HD:], gate=L.GATE_SIGMOID_AFTER), HD, (x, g, w2)
        if kind == "mamba2":
            x, g, w2 = rnd(B, inner, dt=f32), rnd(B, inner + ch + M, dt=f32), torch.ones(inner, device=DEV)
            return L.row_stage(x, inner, inner, 1e-5, w2=w2, groups2=8, g=g, gate=L.GATE_SILU_BEFORE), inner, (x, g, w2)
        x, w2 = rnd(B, 2 * AD, dt=f32), torch.ones(D, device=DEV)
        return L.row_stage(x, AD, AD, 1e-5, w2=w2, groups2=A, pair=D, lam=0.5), AD, (x, w2)
    for B in (1, 4):
        for kind, n, K in (("in, lightning", 4 * HD, E), ("in, mamba2", inner + ch + M, E), ("in, attention", AD + 2 * G * D, E), ("router", NE + 1, E), ("dense up", 4 * E, E)):
            nb, c = n * K * 2, copies(n * K * 2)
            ws = [rnd(n, K) for _ in range(c)]
            h, y, ho, out = rnd(B, K, dt=f32), rnd(B, K, dt=f32), rnd(B, K, dt=f32), torch.zeros(B, n, device=DEV)
            act = torch.zeros(B, n, device=DEV, dtype=bf)
            w2 = ones[:K].contiguous()
            st = L.row_stage(h, K, K, 1e-5, y, None, 1, ho, w2)
            dense = kind == "dense up"
            add("nifalorn", f"matvec {kind} B={B}", "matvec_kernel", graph_us(lambda i: L.matvec(st, ws[i], act if dense else out, B, L.OUT_RELU2 if dense else L.OUT_F32), c), nb, 2 * B * n * K)
            st = L.row_stage(h, K, K, 1e-5, y, None, 1, ho, w2, 1, zero)
            add("vozinex", f"matvec {kind} B={B}", "matvec_kernel", graph_us(lambda i: L.matvec(st, ws[i], out, B), c), nb, 2 * B * n * K)
        for kind in ("lightning", "mamba2", "attention"):
            st, K, alive = mixer_rows(kind, B)
            c = copies(E * K * 2)
            ws, out, x16 = [rnd(E, K) for _ in range(c)], torch.zeros(B, E, device=DEV), rnd(B, K)
            add("nifalorn", f"matvec out, {kind} B={B}", "matvec_kernel", graph_us(lambda i: L.matvec(st, ws[i], out, B), c), E * K * 2, 2 * B * E * K)
            x, w2 = rnd(B, K, dt=f32), ones[:D].contiguous()
            like, st = ("vozinex", L.row_stage(x16, K, K, 1e-5)) if kind == "attention" else ("talizen", L.row_stage(x, K, K, 1e-5, w2=w2, groups2=K // D))
            add(like, f"matvec out, {kind} B={B}", "matvec_kernel", graph_us(lambda i: L.matvec(st, ws[i], out, B), c), E * K * 2, 2 * B * E * K)
            del ws, alive
        # chosen experts and the shared one; beside them Vozinex' with one and a half times the width and one more per token
        for model, FF, kk, gated in (("nifalorn", F, k, True), ("vozinex", F * 3 // 2, k + 1, False)):
            At, sets, per = B * kk, max(1, NE // (B * kk)), (2 if gated else 1) * FF
            stacks = copies(NE * FF * E * 2)
            n = sets * stacks
            logits = []
            for s in range(sets):
                lg = torch.full((B, NE + 1), -20.0, device=DEV)
                for a in range(At):
                    lg[a // kk, (s * At + a) % NE] = 5.0 + 0.01 * a
                logits.append(lg)
            hot = min(At, NE)
            up, down = ([rnd(NE * per, E) for _ in range(stacks)], [rnd(NE * E, FF) for _ in range(stacks)])
            ups, downs = ([rnd(2 * Fs, E) for _ in range(n)], [rnd(E, Fs) for _ in range(n)]) if gated else (None, None)
            h, act, act_s, y = rnd(B, E, dt=f32), rnd(At, FF), rnd(B, Fs), torch.zeros(B, E, device=DEV)
            w2, extra = ones[:E].contiguous(), Fs * E * 2 if gated else 0
            rule = L.Routing(torch.zeros(NE, device=DEV), NE, kk, gated, 4 if gated else 1, 4 if gated else 1, 2.5)
            st, st2 = L.row_stage(h, E, E, 1e-5, w2=w2, b2=None if gated else zero), L.row_stage(act, FF, FF, 1e-5)
            mode = L.OUT_SWIGLU if gated else L.OUT_RELU2
            us = graph_us(lambda i: L.expert_matvec(st, logits[i % sets], rule, up[i // sets], per, act, B, False, mode, (ups[i], act_s) if gated else None), n)
            add(model, f"experts up B={B}", "expert_matvec_kernel", us, hot * per * E * 2 + 2 * extra, 2 * B * kk * per * E)
            us = graph_us(lambda i: L.expert_matvec(st2, logits[i % sets], rule, down[i // sets], E, y, B, True, mode, (downs[i], act_s) if gated else None), n)
            add(model, f"experts down B={B}", "expert_matvec_kernel", us, hot * FF * E * 2 + extra, 2 * B * kk * FF * E)
            del up, down, ups, downs
    # recurrences, one token per sequence: the state is read and written once
    for B in (1, 4, 16):
        seg, slot, pos = ints([[b, b + 1] for b in range(B)]), torch.arange(B, device=DEV, dtype=i32), torch.full((B,), 100, device=DEV, dtype=i32)
        nb = 2 * B * H * D * D * 4
        st = [torch.zeros(B, H, D, D, device=DEV) for _ in range(copies(nb / 2))]
        proj, o, dec = rnd(B, 4 * HD, dt=f32), torch.zeros(B, HD, device=DEV), torch.full((H,), 0.99, device=DEV)
        us = graph_us(lambda i: L.ssd((proj, proj[:, HD:], proj[:, 2 * HD:]), 1, st[i], dec, dec, seg, slot, B, pos, o, act=True, single=True), len(st))
        add("nifalorn", f"recurrence decode, lightning B={B}", "ssd_decode_kernel", us, nb, 6 * B * H * D * D)
        fb, lo = rnd(HD, dt=f32), torch.full((HD,), 0.3, device=DEV)
        us = graph_us(lambda i: L.hgrn2(proj, fb, lo, st[i], seg, slot, B, pos, o), len(st))
        add("talizen", f"recurrence decode, lightning B={B}", "recurrence_scan_kernel (hgrn2)", us, nb, 6 * B * H * D * D)
        nb = 2 * B * M * N * 64 * 4
        st = [torch.zeros(B, M, N, 64, device=DEV) for _ in range(copies(nb / 2))]
        p, o = rnd(B, inner + ch + M, dt=f32), torch.zeros(B, inner, device=DEV)
        x, ring, w, b, one = p[:, inner:inner + ch], torch.zeros(B, 4, ch, device=DEV), rnd(4, ch, dt=f32), rnd(ch, dt=f32), torch.ones(M, device=DEV)
        minus = -one
        cv = L.conv_args(x, w, b, ring)
        us = graph_us(lambda i: L.ssd((x[:, inner + 8 * N:], x[:, inner:], x), M // 8, st[i], None, minus, seg, slot, B, pos, o, steps=(p[:, inner + ch:], one), skip=one, conv=cv, single=True), len(st))
        add("nifalorn", f"recurrence decode, mamba2 B={B}", "ssd_decode_kernel (with the convolution)", us, nb, 6 * B * M * N * 64)
    # decode attention over one chunk
    rot = (5e5 ** (-torch.arange(0, 64, 2, dtype=torch.float64) / 64)).float().to(DEV)
    two = SimpleNamespace(H=2 * A, G=G, R=2 * A // G, D=64, V=D, Dc=64, Vc=D, rot=64, window=1 << 30, keep=0, chunk=chunk, maps=2, adjacent=True, rot_scale=1.0, eps=1e-5, scale=0.125, q_norm=None, k_norm=None,
                          inv_freq=rot, visible=lambda n: min(n, chunk))
    one = SimpleNamespace(H=A, G=G, R=A // G, D=D, V=D, Dc=D, Vc=D, rot=D, window=chunk, keep=0, chunk=0, maps=1, adjacent=False, rot_scale=1.0, eps=1e-5, scale=D ** -0.5, visible=lambda n: min(n, chunk),
                          q_norm=torch.ones(AD, device=DEV), k_norm=torch.ones(G * D, device=DEV), inv_freq=(1e6 ** (-torch.arange(0, D, 2, dtype=torch.float64) / D)).float().to(DEV))
    NI, ctx = AD + 2 * G * D, 4 * chunk
    for B in (1, 4, 16):
        c, mp = copies(B * chunk * G * D * 4), ctx // 64
        slot, pos = torch.arange(B, device=DEV, dtype=i32), torch.full((B,), ctx - 1, device=DEV, dtype=i32)
        bt, proj, tiles = torch.arange(B * mp, device=DEV, dtype=i32).view(B, mp), rnd(B, NI, dt=f32), (slot, torch.ones_like(slot), B)
        for name, m in (("nifalorn", two), ("vozinex", one)):
            kc, vc = [rnd(B * mp, G * m.maps, 64, m.D) for _ in range(c)], [rnd(B * mp, G, 64, D) for _ in range(c)]
            out = torch.zeros(B, m.H * D, device=DEV, dtype=f32 if m.maps == 2 else bf)
            ns = key_ranges(m, B, L.gqa_tile(m.R, 1)[0], ctx)
            us = graph_us(lambda i: L.gqa_decode(m, proj, kc[i], vc[i], bt, slot, pos, tiles, ns, out, B), c)
            add(name, f"attention decode B={B}", f"gqa_attn_mma_kernel (fused, {ns} key ranges)", us, B * chunk * G * D * 4, B * A * chunk * (4 * D + 2 * D * (m.maps - 1)))
            del kc, vc
    # prompts
    for kind, n, K, mode in (("in, lightning", 4 * HD, E, L.OUT_F32), ("in, mamba2", inner + ch + M, E, L.OUT_F32), ("out, mamba2", E, inner, L.OUT_F32), ("router", NE + 1, E, L.OUT_F32),
                             ("dense up", 4 * E, E, L.OUT_RELU2), ("shared up", 2 * Fs, E, L.OUT_SWIGLU)):
        w, xi = rnd(n, K), rnd(T, K)
        out = torch.zeros(T, n, device=DEV, dtype=f32) if mode == L.OUT_F32 else torch.zeros(T, n // 2 if mode == L.OUT_SWIGLU else n, device=DEV, dtype=bf)
        nb = (n * K + T * K + out.numel() * (2 if mode == L.OUT_F32 else 1)) * 2
        add("nifalorn", f"gemm {kind} T={T}", "gemm_tcgen05_kernel", graph_us(lambda i: L.linear(xi, w, out, mode), 1), nb, 2 * T * n * K)
        if mode != L.OUT_F32:
            out = out if mode == L.OUT_SWIGLU else torch.zeros(T, n, device=DEV, dtype=bf)
            like = ("talizen", L.OUT_GEGLU) if mode == L.OUT_SWIGLU else ("vozinex", L.OUT_F32)
            add(like[0], f"gemm {kind} T={T}", "gemm_tcgen05_kernel", graph_us(lambda i: L.linear(xi, w, out, like[1]), 1), nb, 2 * T * n * K)
    hs, y, xb = [rnd(T, E, dt=f32) for _ in range(4)], rnd(T, E, dt=f32), torch.zeros(T, E, device=DEV, dtype=bf)
    w2 = ones[:E].contiguous()
    add("nifalorn", f"norm T={T}", "stage_reg_kernel", graph_us(lambda i: L.stage_rows(L.row_stage(hs[i], E, E, 1e-5, y, None, 1, hs[i], w2), xb, T), 4), T * E * 14, 0)
    add("vozinex", f"norm T={T}", "stage_reg_kernel", graph_us(lambda i: L.stage_rows(L.row_stage(hs[i], E, E, 1e-5, y, None, 1, hs[i], w2, 1, zero), xb, T), 4), T * E * 14, 0)
    for kind in ("lightning", "mamba2", "attention"):
        sts = [mixer_rows(kind, T) for _ in range(3)]
        K = sts[0][1]
        xk = torch.zeros(T, K, device=DEV, dtype=bf)
        add("nifalorn", f"rows behind {kind} T={T}", "stage_rows_kernel", graph_us(lambda i: L.stage_rows(sts[i][0], xk, T), 3), T * K * 10, 0)
        x = [rnd(T, K, dt=f32) for _ in range(4)]
        w2 = torch.ones(D, device=DEV)
        add("talizen", f"rows behind {kind} T={T}", "stage_rows_kernel", graph_us(lambda i: L.stage_rows(L.row_stage(x[i], K, K, 1e-5, w2=w2, groups2=K // D), xk, T), 4), T * K * 6, 0)
        del sts, x
    At = T * k
    logits, rule = torch.randn(T, NE + 1, device=DEV), L.Routing(torch.zeros(NE, device=DEV), NE, k, True, 4, 2, 2.5)
    ids, w = torch.zeros(At, dtype=i32, device=DEV), torch.zeros(At, device=DEV)
    add("nifalorn", f"route T={T}", "route_kernel", graph_us(lambda i: L.route(logits, rule, ids, w, T), 1), T * NE * 4 + At * 8, 0)
    add("vozinex", f"route T={T}", "route_kernel", graph_us(lambda i: L.route(logits, L.Routing(None, NE, k), ids, w, T), 1), T * NE * 4 + At * 8, 0)
    plan, per = ops.MoePlan(At, NE, DEV), At // NE
    tile = 16 if per <= 16 else 32 if per <= 32 else 64 if per <= 96 else 128
    ops.moe_plan(ids, NE, tile, plan)
    xs, ey, act = rnd(At, E), torch.zeros(At, E, device=DEV), rnd(At, F)
    up, down = rnd(NE * 2 * F, E), rnd(NE * E, F)
    us = graph_us(lambda i: L.linear_grouped(xs, up, 2 * F, NE, tile, plan, act, L.OUT_SWIGLU), 1)
    add("nifalorn", f"experts up T={T}", "gemm_tcgen05_kernel (grouped)", us, (2 * NE * F * E + At * E + At * F) * 2, 4 * At * F * E)
    wide = torch.zeros(At, 2 * F, device=DEV, dtype=bf)
    us = graph_us(lambda i: L.linear_grouped(xs, up, 2 * F, NE, tile, plan, wide, L.OUT_RELU2), 1)
    add("vozinex", f"experts up T={T}", "gemm_tcgen05_kernel (grouped)", us, (2 * NE * F * E + At * E + 2 * At * F) * 2, 4 * At * F * E)
    us = graph_us(lambda i: L.linear_grouped(act, down, E, NE, tile, plan, ey), 1)
    add("both", f"experts down T={T}", "gemm_tcgen05_kernel (grouped)", us, (NE * F * E + At * F + At * E * 2) * 2, 2 * At * F * E)
    ys = rnd(T, E, dt=f32)
    add("nifalorn", f"combine T={T}", "moe_combine_kernel", graph_us(lambda i: L.expert_combine(ey, plan, w, T, k, y, (ys, logits[:, NE:])), 1), (At + 2 * T) * E * 4, 0)
    add("vozinex", f"combine T={T}", "moe_combine_kernel", graph_us(lambda i: L.expert_combine(ey, plan, w, T, k, y), 1), (At + T) * E * 4, 0)
    del up, down, xs, ey, act, wide
    # token mixing of a whole prompt
    pos, cu, z = torch.arange(T, device=DEV, dtype=i32), ints([[0, T]]), ints([0])
    ws = (torch.zeros(T // 64 * max(H * D * D, M * N * 64), device=DEV), torch.zeros(T // 64 * max(H, M) * D, device=DEV))

    def chunks(size):
        table, first = L.scan_chunk_table([(0, T)], size)
        return (ints(table).view(-1, 2), ints(first), *ws)
    c64, c128 = chunks(L.HGRN2_CHUNK), chunks(L.SSD_CHUNK)
    proj, o, st, dec = rnd(T, 4 * HD, dt=f32), torch.zeros(T, HD, device=DEV), torch.zeros(1, H, D, D, device=DEV), torch.full((H,), 0.99, device=DEV)
    minus = -dec
    us = graph_us(lambda i: L.ssd((proj, proj[:, HD:], proj[:, 2 * HD:]), 1, st, dec, minus, cu, z, 1, pos, o, act=True, chunks=c128), 1)
    add("nifalorn", f"token mixing, lightning T={T}", "ssd_chunk_* (3 kernels)", us, T * HD * 16, 6 * T * H * D * D)
    fb, lo = rnd(HD, dt=f32), torch.full((HD,), 0.3, device=DEV)
    us = graph_us(lambda i: L.hgrn2(proj, fb, lo, st, cu, z, 1, pos, o, c64), 1)
    add("talizen", f"token mixing, lightning T={T}", "hgrn2_chunk_* (3 kernels)", us, T * HD * 16, 6 * T * H * D * D)
    p, o, st = rnd(T, inner + ch + M, dt=f32), torch.zeros(T, inner, device=DEV), torch.zeros(1, M, N, 64, device=DEV)
    x, ring, cw, b, one_m, xbc = p[:, inner:inner + ch], torch.zeros(1, 4, ch, device=DEV), rnd(4, ch, dt=f32), rnd(ch, dt=f32), torch.ones(M, device=DEV), torch.zeros(T, ch, device=DEV, dtype=bf)
    minus = -one_m
    us = graph_us(lambda i: L.conv_rows(x, cw, b, ring, cu, z, 1, T, pos, xbc), 1)
    add("nifalorn", f"convolution T={T}", "conv_rows_kernel", us, T * ch * 6, 0)
    us = graph_us(lambda i: L.ssd((xbc[:, inner + 8 * N:], xbc[:, inner:], xbc), M // 8, st, None, minus, cu, z, 1, pos, o, steps=(p[:, inner + ch:], one_m), skip=one_m, chunks=c128), 1)
    add("nifalorn", f"token mixing, mamba2 T={T}", "ssd_chunk_* (3 kernels)", us, T * (ch * 2 + inner * 4), 6 * T * M * N * 64)
    mp = 4 * T // 64
    bt, slot0 = torch.arange(mp, device=DEV, dtype=i32).view(1, -1), torch.zeros(T, device=DEV, dtype=i32)
    proj = rnd(T, NI, dt=f32)
    for name, m in (("nifalorn", two), ("vozinex", one)):
        kc, vc = rnd(mp, G * m.maps, 64, m.D), rnd(mp, G, 64, D)
        q, out = torch.zeros(T, AD, device=DEV, dtype=bf), torch.zeros(T, m.H * D, device=DEV, dtype=f32 if m.maps == 2 else bf)
        us = graph_us(lambda i: L.gqa_prepare(m, proj, kc, vc, bt, slot0, pos, pos, q, T), 1)
        add(name, f"rotation, cache rows T={T}", "gqa_prepare_kernel", us, T * NI * 6, 0)
        row0 = torch.arange(T - 128, -1, -128, device=DEV, dtype=i32)
        tiles = (row0, torch.full_like(row0, 128), row0.numel())
        us = graph_us(lambda i: L.gqa_flash(m, q, kc, vc, bt, slot0, pos, tiles, out, T), 1)
        pairs = T * (T + 1) // 2
        add(name, f"attention prefill T={T}", "attn_prefill_tc_kernel<FA_TILES>", us, (AD + 2 * G * D) * T * 2 + out.numel() * out.element_size(), pairs * A * (4 * D + 2 * D * (m.maps - 1)))
    return rows, src
