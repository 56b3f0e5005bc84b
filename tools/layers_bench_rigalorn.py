"""Rigalorn's part of tools/layers_bench.py: a model of every mixer with dense feed-forwards beside a Nifalorn of equal size, and its kernels beside the
like ones of Nifalorn, Vozinex and Talizen on the same sizes."""
from __future__ import annotations

from types import SimpleNamespace

import torch

from layers_bench_nifalorn import VOCAB, weights as layer_weights

DEV = "cuda:0"
# name: (width, heads, key / value heads of the attention, query / key heads of the delta rule, rotated part and latents of latent attention (queries, keys),
#        ff, layers, window); heads are 128 wide
PARALLEL_SIZES = {
    "parallel-2048": (2048, 16, 4, 8, 64, 768, 512, 8192, 8, 2048),
    "parallel-4096": (4096, 32, 8, 16, 64, 1536, 512, 14336, 4, 2048),
}
D = 128
YARN = {"factor": 8.0, "original": 8192, "fast": 32.0, "slow": 1.0}


def rigalorn(size: str):
    """Latent attention, attention, two delta rules, and again."""
    from distributed_llm_pipeline_b200.models.modeldir import rigalorn_config
    E, H, G, K, P, QR, R, F, n, window = PARALLEL_SIZES[size]
    mlp = {"kind": "dense", "ff": F}
    la = {"type": "latent_attention", "mlp": mlp, "mixer": {"heads": H, "dim": D, "rot_dim": P, "vdim": D, "q_rank": QR, "kv_rank": R, "scale": (D + P) ** -0.5, "mask": {"size": window},
                                                            "rot": {"dims": P, "base": 5e5}}}
    at = {"type": "attention", "mlp": mlp, "mixer": {"heads": H, "kv_heads": G, "dim": D, "vdim": D, "scale": D ** -0.5, "mask": {"size": window}, "v_mix": True,
                                                     "rot": {"dims": D, "base": 1e6, "scaling": YARN}}}
    de = {"type": "delta", "mlp": mlp, "mixer": {"heads": H, "kv_heads": K, "dim": D, "vdim": D, "conv": 4}}
    cfg = rigalorn_config({"width": E, "vocab": VOCAB, "norm": {"eps": 1e-5}, "layers": ([la, at, de, de] * n)[:n], "embedding": {"scale": 1.0}})
    shapes = {"latent_attention": {"dq": (QR, E), "uq": (H * (D + P), QR), "dkv": (R + P, E), "uk": (H * D, R), "uv": (H * D, R), "o": (E, H * D)},
              "attention": {"q": (H * D, E), "k": (G * D, E), "v": (G * D, E), "o": (E, H * D)},
              "delta": {"q": (K * D, E), "k": (K * D, E), "v": (H * D, E), "g": (H * D, E), "a": (H, E), "b": (H, E), "o": (E, H * D), "q.conv": (K * D, 4), "k.conv": (K * D, 4), "v.conv": (H * D, 4)},
              "mlp": {"up": (F, E), "down": (E, F)}}
    vec = {"latent_attention": {"dq.norm": torch.ones(QR), "dkv.norm": torch.ones(R)}, "mlp": {"act": torch.zeros(2)},
           "attention": {"q.b": torch.zeros(H * D), "k.b": torch.zeros(G * D), "v.b": torch.zeros(G * D), "vmix": torch.tensor(0.5)},
           "delta": {"A_log": torch.zeros(H), "dt_bias": torch.full((H,), -3.0), "norm": torch.ones(D)}}
    return layer_weights(cfg, False, vec, shapes)


def nifalorn(size: str):
    """The same width, heads, feed-forward and depth: differential attention twice, Mamba-2, lightning, and again."""
    from distributed_llm_pipeline_b200.models.modeldir import nifalorn_config
    E, H, G, _, _, _, _, F, n, window = PARALLEL_SIZES[size]
    M = 2 * H
    mlp = {"kind": "dense", "ff": F}
    li = {"type": "lightning", "mixer": {"heads": H, "dim": D, "vdim": D, "decay": [0.99] * H}, "mlp": mlp}
    ma = {"type": "mamba2", "mixer": {"heads": M, "vdim": 64, "state": D, "groups": 8, "conv": 4, "norm_groups": 8}, "mlp": mlp}
    at = {"type": "attention", "mlp": mlp, "mixer": {"heads": H, "kv_heads": G, "dim": 64, "vdim": D, "scale": 0.125, "diff": 0.5, "mask": {"size": window},
                                                      "rot": {"dims": 64, "base": 5e5, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}}}
    cfg = nifalorn_config({"width": E, "vocab": VOCAB, "norm": {"eps": 1e-5}, "layers": ([at, at, ma, li] * n)[:n], "embedding": {"scale": 1.0}, "logit_scale": 1.0})
    inner, ch = 64 * M, 64 * M + 2 * 8 * D
    shapes = {"lightning": {x: (D * H, E) for x in "qkvg"} | {"o": (E, D * H)}, "mamba2": {"in": (inner + ch + M, E), "o": (E, inner), "conv": (ch, 4)},
              "attention": {"q": (D * H, E), "k": (D * G, E), "v": (D * G, E), "o": (E, D * H)}, "mlp": {"up": (F, E), "down": (E, F)}}
    vec = {"lightning": {"norm": torch.ones(D * H)}, "attention": {x: torch.full((64,), 0.1) for x in ("lq1", "lk1", "lq2", "lk2")}, "mlp": {},
           "mamba2": {"conv.b": torch.zeros(ch), "dt_bias": torch.full((M,), -2.0), "A_log": torch.zeros(M), "D": torch.ones(M), "norm": torch.ones(inner)}}
    return layer_weights(cfg, False, vec, shapes)


def kernel_numbers(size: str, graph_us, copies, peaks, T: int = 2048):
    """Rows (model, kind, kernel, us, roofline) of Rigalorn's kernels and of the like ones."""
    from distributed_llm_pipeline_b200.models.layered import key_ranges
    from distributed_llm_pipeline_b200.models.mixers import rotation
    from distributed_llm_pipeline_b200.ops import layers as L
    L.load_library()
    E, H, G, KH, P, QR, R, F, _, window = PARALLEL_SIZES[size]
    bf, f32, i32 = torch.bfloat16, torch.float32, torch.int32
    bw, fl, src = peaks()
    rows = []

    def rnd(*s, dt=bf):
        return (torch.randn(*s, device=DEV) * 0.1).to(dt)

    def ints(x):
        return torch.tensor(x, device=DEV, dtype=i32)

    def add(model, kind, name, us, nbytes, flops):
        roof = max(nbytes / bw, flops / fl) * 1e6
        rows.append({"model": model, "kind": kind, "kernel": name, "us": round(us, 2), "roofline_us": round(roof, 2), "of_roofline": round(roof / us, 4)})
    HD, Dq, ch = H * D, D + P, 2 * KH * D + H * D
    pad = lambda n: (n + 31) // 32 * 32
    ones = torch.ones(max(E, F, QR, HD), device=DEV)
    n_in = {"latent": pad(QR + R + P), "attention": pad((H + 2 * G) * D), "delta": pad(ch + HD + 2 * H)}

    # products: the stacked input of mixer and feed-forward, the output over both halves; beside them a norm in front of the same matrix with squared
    # ReLU behind it, and plain rows in front of the other
    for B in (1, 4):
        for kind, n1 in n_in.items():
            n = n1 + F
            c = copies(n * E * 2)
            ws = [rnd(n, E) for _ in range(c)]
            h, y, ho, out, act, w2 = rnd(B, E, dt=f32), rnd(B, E, dt=f32), rnd(B, E, dt=f32), torch.zeros(B, n1, device=DEV), torch.zeros(B, n, device=DEV, dtype=bf), ones[:E].contiguous()
            bias = torch.zeros(n, device=DEV)
            st, tail = L.row_stage(h, E, E, 1e-5, y, None, 1, ho, w2), L.out_tail(bias if kind == "attention" else None, n1, act, (0.7, 1.2))
            add("rigalorn", f"matvec in, {kind} B={B}", "matvec_kernel", graph_us(lambda i: L.matvec(st, ws[i], out, B, tail=tail), c), n * E * 2, 2 * B * n * E)
            add("nifalorn", f"matvec in, {kind} B={B}", "matvec_kernel", graph_us(lambda i: L.matvec(st, ws[i], act, B, L.OUT_RELU2), c), n * E * 2, 2 * B * n * E)
            del ws
        K = HD + F
        c = copies(E * K * 2)
        ws, out, both, x, g, w2 = [rnd(E, K) for _ in range(c)], torch.zeros(B, E, device=DEV), rnd(B, K), rnd(B, HD, dt=f32), rnd(B, HD, dt=f32), ones[:D].contiguous()
        st = L.row_stage(x, HD, HD, 1e-5, w2=w2, groups2=H, g=g, gate=L.GATE_SILU_AFTER, tail=both[:, HD:])
        plain = L.row_stage(both, K, K, 1e-5)
        like = graph_us(lambda i: L.matvec(plain, ws[i], out, B), c)
        for kind, us in (("attention", like), ("delta", graph_us(lambda i: L.matvec(st, ws[i], out, B), c))):
            add("rigalorn", f"matvec out, {kind} B={B}", "matvec_kernel", us, E * K * 2, 2 * B * E * K)
            add("nifalorn", f"matvec out, {kind} B={B}", "matvec_kernel", like, E * K * 2, 2 * B * E * K)
        del ws
        # queries of latent attention out of their latent; beside them a norm behind a sublayer in front of the same matrix
        n = H * Dq
        c = copies(n * QR * 2)
        ws, x, w2, out = [rnd(n, QR) for _ in range(c)], rnd(B, n_in["latent"], dt=f32), ones[:QR].contiguous(), torch.zeros(B, n, device=DEV)
        st = L.row_stage(x, QR, QR, 1e-5, w2=w2)
        add("rigalorn", f"matvec latent queries B={B}", "matvec_kernel", graph_us(lambda i: L.matvec(st, ws[i], out, B), c), n * QR * 2, 2 * B * n * QR)
        y, ho, xq = rnd(B, QR, dt=f32), rnd(B, QR, dt=f32), rnd(B, QR, dt=f32)
        st = L.row_stage(xq, QR, QR, 1e-5, y, w2, 1, ho)
        add("talizen", f"matvec latent queries B={B}", "matvec_kernel", graph_us(lambda i: L.matvec(st, ws[i], out, B), c), n * QR * 2, 2 * B * n * QR)
        del ws
    # one token per sequence
    page, ctx = 64, 4 * window
    rot = rotation({"dims": P, "base": 5e5})[0].float().to(DEV)
    rot_a, amp = rotation({"dims": D, "base": 1e6, "scaling": YARN})
    rot_a = rot_a.float().to(DEV)
    Rc, M = pad(R + P), 2 * H
    ch2 = 64 * M + 16 * D
    for B in (1, 4, 16):
        seg, slot, pos = ints([[b, b + 1] for b in range(B)]), torch.arange(B, device=DEV, dtype=i32), torch.full((B,), ctx - 1, device=DEV, dtype=i32)
        nb = 2 * B * H * D * D * 4
        st = [torch.zeros(B, H, D, D, device=DEV) for _ in range(copies(nb / 2))]
        p, o, w = rnd(B, n_in["delta"], dt=f32), torch.zeros(B, HD, device=DEV), rnd(4, ch, dt=f32)
        ring, minus, one = torch.zeros(B, 4, ch, device=DEV), -torch.ones(H, device=DEV), torch.ones(H, device=DEV)
        x = p[:, :ch]
        cv = L.conv_args(x, w, None, ring)
        us = graph_us(lambda i: L.delta((x, x[:, KH * D:], x[:, 2 * KH * D:]), H // KH, st[i], p[:, ch + HD + H:], p[:, ch + HD:], minus, one, seg, slot, B, pos, o, 1e-6, conv=cv, single=True), len(st))
        add("rigalorn", f"recurrence decode B={B}", "delta_decode_kernel (with the convolution)", us, nb, 8 * B * H * D * D)
        st = [s.view(B, M, D, 64) for s in st]
        p2, o2 = rnd(B, 64 * M + ch2 + M, dt=f32), torch.zeros(B, 64 * M, device=DEV)
        x2, ring2, w_2, b2, one2 = p2[:, 64 * M:64 * M + ch2], torch.zeros(B, 4, ch2, device=DEV), rnd(4, ch2, dt=f32), rnd(ch2, dt=f32), torch.ones(M, device=DEV)
        minus2, cv2 = -one2, L.conv_args(x2, w_2, b2, ring2)
        us = graph_us(lambda i: L.ssd((x2[:, 64 * M + 8 * D:], x2[:, 64 * M:], x2), M // 8, st[i], None, minus2, seg, slot, B, pos, o2, steps=(p2[:, 64 * M + ch2:], one2), skip=one2, conv=cv2, single=True), len(st))
        add("nifalorn", f"recurrence decode B={B}", "ssd_decode_kernel (with the convolution)", us, nb, 6 * B * H * D * D)
        del st
        # latent attention: rows, absorption, attention over the window, expansion; beside it Talizen's over a context of that many tokens
        c, mp = copies(B * window * Rc * 2), ctx // page
        proj, q, w_c = rnd(B, n_in["latent"], dt=f32), rnd(B, H * Dq, dt=f32), ones[:R].contiguous()
        place, cache1, cache0 = slot * mp * page + 5, rnd(B * mp, 1, page, Rc), rnd(B * mp, 1, page, R)
        add("rigalorn", f"latent rows B={B}", "latent_write_kernel (with rotations)",
            graph_us(lambda i: L.latent_write(proj[:, QR:], w_c, 1e-5, R, place, cache1, B, rot=(pos, rot, 1.0), q=q, heads=H), 1), B * (R + P) * 6 + B * H * P * 8, 0)
        add("talizen", f"latent rows B={B}", "latent_write_kernel", graph_us(lambda i: L.latent_write(proj[:, QR:], w_c, 1e-5, R, place, cache0, B), 1), B * R * 6, 0)
        del cache1, cache0
        for name, rc, vc, dq, win, ln in (("rigalorn", Rc, R, Dq, window, ctx), ("talizen", R, R, D, L.NO_WINDOW, window)):
            mp = ln // page
            bt = torch.arange(B * mp, device=DEV, dtype=i32).view(B, mp)
            pos_l = torch.full((B,), ln - 1, device=DEV, dtype=i32)
            cache = [rnd(B * mp, 1, page, rc) for _ in range(min(c, 8 * window // ln * 4))]
            bm = L.latent_tile_rows(H, B, rc)
            per = (H + bm - 1) // bm
            row0, nr = ints([b * H + i * bm for b in range(B) for i in range(per)]), ints([min(bm, H - i * bm) for b in range(B) for i in range(per)])
            ns = 1
            while ns * 2 <= min(148 // (B * per), (window + 63) // 64, 32):
                ns *= 2
            qa, out = rnd(B, H * rc), torch.zeros(B, H * vc, device=DEV, dtype=bf)
            ws = (torch.zeros(ns * B * H * vc, device=DEV), torch.zeros(ns * B * H * 2, device=DEV))
            us = graph_us(lambda i: L.latent_attention(qa, cache[i], bt, slot, pos_l, row0, nr, B * per, bm, H, B, Dq ** -0.5, out, n_splits=ns, workspace=ws, window=win), len(cache))
            add(name, f"latent attention decode B={B}", f"latent_attn_mma_kernel ({ns} key ranges, + combine)", us, B * window * rc * 2, 2 * B * H * window * (rc + vc))
            del cache
            k = copies(H * rc * dq * 2)
            uk = [rnd(H, rc, dq) for _ in range(k)]
            qx = rnd(B, H * dq, dt=f32)
            us = graph_us(lambda i: L.head_matmul(qx, dq, dq, uk[i], rc, qa, rc, B), k)
            add(name, f"key absorption B={B}", "head_matmul_kernel", us, H * rc * dq * 2, 2 * B * H * rc * dq)
            uv, at = [rnd(H, D, vc) for _ in range(k)], torch.zeros(B, HD + F, device=DEV, dtype=bf)
            us = graph_us(lambda i: L.head_matmul(out, vc, vc, uv[i], D, at, D, B), k)
            add(name, f"value expansion B={B}", "head_matmul_kernel", us, H * vc * D * 2, 2 * B * H * vc * D)
            del uk, uv
        # attention over the window, values mixed; beside it Vozinex'
        mp = ctx // page
        bt = torch.arange(B * mp, device=DEV, dtype=i32).view(B, mp)
        base = dict(H=H, G=G, R=H // G, D=D, V=D, Dc=D, Vc=D, rot=D, window=window, keep=0, chunk=0, maps=1, adjacent=False, eps=1e-5, scale=D ** -0.5, visible=lambda n: min(n, window))
        mine = SimpleNamespace(**base, rot_scale=amp, q_norm=None, k_norm=None, inv_freq=rot_a)
        theirs = SimpleNamespace(**base, rot_scale=1.0, q_norm=ones[:HD], k_norm=ones[:G * D], inv_freq=rot_a)
        c = copies(B * window * G * D * 4)
        kc, vc = ([rnd(B * mp, G, page, D) for _ in range(min(c, 8))] for _ in range(2))
        p, out, first, tiles = rnd(B, n_in["attention"], dt=f32), torch.zeros(B, HD + F, device=DEV, dtype=bf), torch.zeros(B, G * D, device=DEV), (slot, torch.ones_like(slot), B)
        ns = key_ranges(mine, B, L.gqa_tile(mine.R, 1)[0], ctx)
        for name, m, mix in (("rigalorn", mine, (first, 0.5)), ("vozinex", theirs, None)):
            us = graph_us(lambda i: L.gqa_decode(m, p, kc[i], vc[i], bt, slot, pos, tiles, ns, out, B, mix=mix), len(kc))
            add(name, f"attention decode B={B}", f"gqa_attn_mma_kernel (fused, {ns} key ranges)", us, B * window * G * D * 4, 4 * B * H * window * D)
        del kc, vc
    # prompts
    for kind, n1 in n_in.items():
        n = n1 + F
        w, xi, out, act, bias = rnd(n, E), rnd(T, E), torch.zeros(T, n1, device=DEV), torch.zeros(T, n, device=DEV, dtype=bf), torch.zeros(n, device=DEV)
        tail = L.out_tail(bias if kind == "attention" else None, n1, act, (0.7, 1.2))
        nb = (n * E + T * E + T * F + 2 * T * n1) * 2
        add("rigalorn", f"gemm in, {kind} T={T}", "gemm_tcgen05_kernel", graph_us(lambda i: L.linear(xi, w, out, tail=tail), 1), nb, 2 * T * n * E)
        add("nifalorn", f"gemm in, {kind} T={T}", "gemm_tcgen05_kernel", graph_us(lambda i: L.linear(xi, w, act, L.OUT_RELU2), 1), (n * E + T * E + T * n) * 2, 2 * T * n * E)
    for kind, n, K in (("out", E, HD + F), ("latent queries", H * Dq, QR)):
        w, xi, out = rnd(n, K), rnd(T, K), torch.zeros(T, n, device=DEV)
        us = graph_us(lambda i: L.linear(xi, w, out), 1)
        for name in ("rigalorn", "nifalorn"):
            add(name, f"gemm {kind} T={T}", "gemm_tcgen05_kernel", us, (n * K + T * K + T * n * 2) * 2, 2 * T * n * K)
    hs, y, xb, w2 = [rnd(T, E, dt=f32) for _ in range(4)], rnd(T, E, dt=f32), torch.zeros(T, E, device=DEV, dtype=bf), ones[:E].contiguous()
    us = graph_us(lambda i: L.stage_rows(L.row_stage(hs[i], E, E, 1e-5, y, None, 1, hs[i], w2), xb, T), 4)
    for name in ("rigalorn", "nifalorn"):
        add(name, f"norm T={T}", "stage_reg_kernel", us, T * E * 14, 0)
    pl = [rnd(T, n_in["latent"], dt=f32) for _ in range(4)]
    xq, wq = torch.zeros(T, QR, device=DEV, dtype=bf), ones[:QR].contiguous()
    add("rigalorn", f"norm of the latent queries T={T}", "stage_reg_kernel", graph_us(lambda i: L.stage_rows(L.row_stage(pl[i], QR, QR, 1e-5, w2=wq), xq, T), 4), T * QR * 6, 0)
    xs = [rnd(T, QR, dt=f32) for _ in range(4)]
    add("nifalorn", f"norm of the latent queries T={T}", "stage_reg_kernel", graph_us(lambda i: L.stage_rows(L.row_stage(xs[i], QR, QR, 1e-5, w2=wq), xq, T), 4), T * QR * 6, 0)
    both = torch.zeros(T, HD + F, device=DEV, dtype=bf)
    x, g, w2, wl = [rnd(T, HD, dt=f32) for _ in range(3)], [rnd(T, n_in["delta"], dt=f32) for _ in range(3)], ones[:D].contiguous(), ones[:HD].contiguous()
    xk = torch.zeros(T, HD, device=DEV, dtype=bf)
    us = graph_us(lambda i: L.stage_rows(L.row_stage(x[i], HD, HD, 1e-5, w2=w2, groups2=H, g=g[i][:, ch:], gate=L.GATE_SILU_AFTER), both[:, :HD], T), 3)
    add("rigalorn", f"rows behind the recurrence T={T}", "stage_rows_kernel", us, T * HD * 10, 0)
    us = graph_us(lambda i: L.stage_rows(L.row_stage(x[i], HD, HD, 1e-5, w2=wl, g=g[i][:, ch:], gate=L.GATE_SIGMOID_AFTER), xk, T), 3)
    add("nifalorn", f"rows behind the recurrence T={T}", "stage_rows_kernel", us, T * HD * 10, 0)
    # token mixing of a whole prompt
    pos, cu, z = torch.arange(T, device=DEV, dtype=i32), ints([[0, T]]), ints([0])
    p, ring, cw, xbc, cb = g[0], torch.zeros(1, 4, ch, device=DEV), rnd(4, ch, dt=f32), torch.zeros(T, ch, device=DEV, dtype=bf), rnd(ch, dt=f32)
    add("rigalorn", f"convolution T={T}", "conv_rows_kernel", graph_us(lambda i: L.conv_rows(g[i][:, :ch], cw, None, ring, cu, z, 1, T, pos, xbc), 3), T * ch * 6, 0)
    add("nifalorn", f"convolution T={T}", "conv_rows_kernel", graph_us(lambda i: L.conv_rows(g[i][:, :ch], cw, cb, ring, cu, z, 1, T, pos, xbc), 3), T * ch * 6, 0)
    table, first = L.scan_chunk_table([(0, T)], L.DELTA_CHUNK)
    n = len(table) // 2
    chunks = (ints(table).view(-1, 2), ints(first), *(torch.zeros(b // 4, device=DEV) for b in L.delta_workspace(n, H, KH, D, D)))
    o, st, minus, one = torch.zeros(T, HD, device=DEV), torch.zeros(1, H, D, D, device=DEV), -torch.ones(H, device=DEV), torch.ones(H, device=DEV)
    us = graph_us(lambda i: L.delta((xbc, xbc[:, KH * D:], xbc[:, 2 * KH * D:]), H // KH, st, p[:, ch + HD + H:], p[:, ch + HD:], minus, one, cu, z, 1, pos, o, 1e-6, chunks=chunks), 1)
    add("rigalorn", f"token mixing, recurrence T={T}", "delta_chunk_* (3 kernels)", us, T * (ch * 2 + HD * 4), 8 * T * H * D * D)
    p2, xbc2, o2, st2 = rnd(T, 64 * M + ch2 + M, dt=f32), rnd(T, ch2), torch.zeros(T, 64 * M, device=DEV), torch.zeros(1, M, D, 64, device=DEV)
    table, first = L.scan_chunk_table([(0, T)], L.SSD_CHUNK)
    n = len(table) // 2
    chunks, minus2, one2 = (ints(table).view(-1, 2), ints(first), torch.zeros(n * M * D * 64, device=DEV), torch.zeros(n * M, device=DEV)), -torch.ones(M, device=DEV), torch.ones(M, device=DEV)
    us = graph_us(lambda i: L.ssd((xbc2[:, 64 * M + 8 * D:], xbc2[:, 64 * M:], xbc2), M // 8, st2, None, minus2, cu, z, 1, pos, o2, steps=(p2[:, 64 * M + ch2:], one2), skip=one2, chunks=chunks), 1)
    add("nifalorn", f"token mixing, recurrence T={T}", "ssd_chunk_* (3 kernels)", us, T * (ch2 * 2 + 64 * M * 4), 6 * T * M * D * 64)
    mp = 4 * T // page
    bt, slot0 = torch.arange(mp, device=DEV, dtype=i32).view(1, -1), torch.zeros(T, device=DEV, dtype=i32)
    kc, vc = rnd(mp, G, page, D), rnd(mp, G, page, D)
    proj, q, out, vf = rnd(T, n_in["attention"], dt=f32), torch.zeros(T, HD, device=DEV, dtype=bf), torch.zeros(T, HD, device=DEV, dtype=bf), torch.zeros(T, G * D, device=DEV)
    for name, m, mix, o_ in (("rigalorn", mine, (vf, 0.5), both), ("vozinex", theirs, None, out)):
        us = graph_us(lambda i: L.gqa_prepare(m, proj, kc, vc, bt, slot0, pos, pos, q, T, mix=mix), 1)
        add(name, f"rotation, cache rows T={T}", "gqa_prepare_kernel", us, T * (HD + 2 * G * D) * 6 + (T * G * D * 4 if mix else 0), 0)
        for p0 in (0, 3 * T):
            at = pos + p0
            row0 = torch.arange(T - 128, -1, -128, device=DEV, dtype=i32)
            tiles = (row0, torch.full_like(row0, 128), row0.numel())
            seen = sum(min(i + 1, window) for i in range(p0, p0 + T))
            us = graph_us(lambda i: L.gqa_flash(m, q, kc, vc, bt, slot0, at, tiles, o_, T), 1)
            add(name, f"attention prefill T={T} at {p0}", "attn_prefill_tc_kernel<FA_TILES>", us, (2 * HD + 2 * G * D) * T * 2, 4 * seen * HD)
    del kc, vc
    # latent attention of a whole prompt: keys and values expanded
    q, cache1, cache0 = rnd(T, H * Dq, dt=f32), rnd(mp, 1, page, Rc), rnd(mp, 1, page, R)
    wc = ones[:R].contiguous()
    us = graph_us(lambda i: L.latent_write(pl[i][:, QR:], wc, 1e-5, R, pos, cache1, T, rot=(pos, rot, 1.0), q=q, heads=H), 4)
    add("rigalorn", f"latent rows T={T}", "latent_write_kernel (with rotations)", us, T * ((R + P) * 6 + H * P * 8), 0)
    add("talizen", f"latent rows T={T}", "latent_write_kernel", graph_us(lambda i: L.latent_write(pl[i][:, QR:], wc, 1e-5, R, pos, cache0, T), 4), T * R * 6, 0)
    for name, rc, dp, dq, win, cache in (("rigalorn", Rc, (Dq + 63) // 64 * 64, Dq, window, cache1), ("talizen", R, D, D, L.NO_WINDOW, cache0)):
        n = H * (dp + D)
        ukv, cx, kv, qx, qf = rnd(n, rc), rnd(T, rc), torch.zeros(T, n, device=DEV, dtype=bf), torch.zeros(T, H * dp, device=DEV, dtype=bf), rnd(T, H * dq, dt=f32)
        add(name, f"latent gather T={T}", "latent_gather_kernel", graph_us(lambda i: L.latent_gather(cache, bt[0], T, cx), 1), T * rc * 4, 0)
        add(name, f"key / value expansion T={T}", "gemm_tcgen05_kernel", graph_us(lambda i: L.linear(cx, ukv, kv), 1), (T * rc + T * n + n * rc) * 2, 2 * T * n * rc)
        add(name, f"query rows T={T}", "head_rows_kernel", graph_us(lambda i: L.head_rows(qf, H, dq, dp, qx), 1), T * H * (dq * 4 + dp * 2), 0)
        us = graph_us(lambda i: L.rows_attention(qx, kv, T, 0, H, dp, D, D, dq ** -0.5, both, window=win), 1)
        add(name, f"latent attention prefill T={T}", "attn_prefill_tc_kernel<FA_ROWS>", us, T * H * (2 * dp + 2 * D) * 2, T * (T + 1) * H * (dq + D))
    return rows, src
