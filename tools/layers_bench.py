#!/usr/bin/env python
"""Throughput of layer-list models beside the closest GGUF model of equal size, and every kernel of both against its roofline
(`bench.py --layers`): Talizen beside a Llama, Vozinex beside a Qwen3-MoE, Nifalorn beside a Vozinex (tools/layers_bench_nifalorn.py),
Rigalorn beside a Nifalorn (tools/layers_bench_rigalorn.py).

Random weights at sizes of real models' layers.  Model numbers are device-timed with CUDA events around whole forwards (prefill) and
blocks of graph replays (decode); a step streams weights larger than L2.  Kernel numbers: a captured graph of launches that rotate
through enough copies of their operands to exceed L2.  roofline = the slower of bytes / measured copy rate and FLOPs / measured GEMM rate.
"""
from __future__ import annotations

import argparse
import json
import os
import statistics
import sys
import tempfile

REPO = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path[:0] = [REPO, os.path.join(REPO, "tools")]

import torch  # noqa: E402

import layers_bench_nifalorn as hybrid  # noqa: E402
import layers_bench_rigalorn as parallel  # noqa: E402

DEV = "cuda:0"
SIZES = {   # name: (width, heads, head size, latent rank, ff, layers)
    "2048": (2048, 16, 128, 512, 5632, 8),
    "4096": (4096, 32, 128, 512, 14336, 4),
}
MOE_SIZES = {   # name: (width, heads, key / value heads, head size, experts, experts per token, ff of an expert, layers, window, kept first tokens)
    "moe-2048": (2048, 32, 4, 128, 64, 8, 768, 4, 1984, 64),
    "moe-4096": (4096, 32, 8, 128, 16, 2, 4096, 4, 1984, 64),
}
VOCAB = 32000


def peaks():
    try:
        p = json.load(open(os.path.join(REPO, "MEASURED_PEAKS.json")))
        return p["hbm_gbs"] * 1e9, p["bf16_tflops"] * 1e12, "measured"
    except (OSError, KeyError):
        return 6.65e12, 1.59e15, "fallback"


def talizen(size: str):
    """Three recurrent layers to one of latent attention, a feed-forward in each, as weights in device memory."""
    from distributed_llm_pipeline_b200.gguf.constants import GGMLType
    from distributed_llm_pipeline_b200.models.layered import LayeredLayer, LayeredWeights, Norm
    from distributed_llm_pipeline_b200.models.mixers import MIXERS, MLPS
    from distributed_llm_pipeline_b200.models.modeldir import talizen_config
    from distributed_llm_pipeline_b200.ops.weights import DeviceWeight
    E, H, D, R, F, n = SIZES[size]
    hg = {"type": "hgrn2", "mixer": {"heads": H, "dim": D, "vdim": D}, "mlp": {"kind": "dense", "ff": F}}
    la = {"type": "latent_attention", "mixer": {"heads": H, "dim": D, "vdim": D, "kv_rank": R, "scale": D ** -0.5}, "mlp": {"kind": "dense", "ff": F}}
    cfg = talizen_config({"width": E, "vocab": VOCAB, "norm": {"groups": 4, "eps": 1e-5}, "layers": [la if i % 4 == 3 else hg for i in range(n)]})

    def mat(r, c):
        return (torch.randn(r, c, device=DEV) * c ** -0.5).to(torch.bfloat16)
    shapes = {"hgrn2": {"q": (H * D, E), "f": (H * D, E), "v": (H * D, E), "o": (E, H * D)},
              "latent_attention": {"q": (H * D, E), "dkv": (R, E), "g": (H, E), "uk": (H * D, R), "uv": (H * D, R), "o": (E, H * D)}}

    def get(kind):
        def g(name):
            if name in shapes[kind]:
                return mat(*shapes[kind][name])
            return {"f.b": torch.full((H * D,), 3.0), "lower": torch.rand(H * D) * 0.9, "norm": torch.ones(D), "dkv.norm": torch.ones(R)}[name]
        return g
    mlp_shapes = {"gate": (F, E), "up": (F, E), "down": (E, F)}
    one = Norm(torch.ones(E, device=DEV))
    layers = {i: LayeredLayer(MIXERS[s.type](s.mixer, get(s.type), DEV, torch.bfloat16, 1e-5), one, MLPS["dense"](s.mlp, lambda k: mat(*mlp_shapes[k]), DEV, torch.bfloat16, E), one)
              for i, s in enumerate(cfg.layers)}
    tab = [DeviceWeight(GGMLType.BF16, VOCAB, E, [mat(VOCAB, E)]) for _ in range(2)]
    return LayeredWeights(cfg, layers, range(n), 0, 1, tab[0], one.w, tab[1], (0, VOCAB), None)


def vozinex(size: str):
    """Windowed attention and routed experts in every layer, each layer once."""
    from distributed_llm_pipeline_b200.gguf.constants import GGMLType
    from distributed_llm_pipeline_b200.models.layered import LayeredLayer, LayeredWeights, Norm
    from distributed_llm_pipeline_b200.models.mixers import MIXERS, MLPS
    from distributed_llm_pipeline_b200.models.modeldir import vozinex_config
    from distributed_llm_pipeline_b200.ops.weights import DeviceWeight
    E, H, G, D, NE, k, F, n, window, keep = MOE_SIZES[size]
    spec = {"type": "attention", "mixer": {"heads": H, "kv_heads": G, "dim": D, "vdim": D, "scale": D ** -0.5, "rot": {"dims": D, "base": 1e6}, "mask": {"size": window, "keep_first": keep}},
            "mlp": {"kind": "moe", "expert": {"ff": F}, "router": {"experts": NE, "top": k}}}
    cfg = vozinex_config({"width": E, "vocab": VOCAB, "norm": {"eps": 1e-5}, "layers": [spec] * n})

    def mat(r, c):
        return (torch.randn(r, c, device=DEV) * c ** -0.5).to(torch.bfloat16)
    shapes = {"q": (H * D, E), "k": (G * D, E), "v": (G * D, E), "o": (E, H * D), "up": (F, E), "down": (E, F), "router": (NE, E)}
    vecs = {"q.norm": H * D, "k.norm": G * D, "router.b": NE}

    def get(name):
        kind = name.split(".")[-1] if name.startswith("e") else name
        return mat(*shapes[kind]) if kind in shapes else torch.ones(vecs[name])
    norm = Norm(torch.ones(E, device=DEV), torch.zeros(E, device=DEV))
    layers = {i: LayeredLayer(MIXERS[s.type](s.mixer, get, DEV, torch.bfloat16, 1e-5), norm, MLPS["moe"](s.mlp, get, DEV, torch.bfloat16, E), norm) for i, s in enumerate(cfg.layers)}
    tab = [DeviceWeight(GGMLType.BF16, VOCAB, E, [mat(VOCAB, E)]) for _ in range(2)]
    return LayeredWeights(cfg, layers, range(n), 0, 1, tab[0], norm.w, tab[1], (0, VOCAB), None, out_norm_b=norm.b)


def qwen3moe(size: str):
    from distributed_llm_pipeline_b200.gguf import write_synthetic_gguf
    from distributed_llm_pipeline_b200.models.config import preset
    from distributed_llm_pipeline_b200.models.weights import load_weights
    E, H, G, D, NE, k, F, n, _, _ = MOE_SIZES[size]
    cfg = preset("qwen3-30b-a3b", vocab_size=VOCAB, n_embd=E, n_layer=n, n_head=H, n_head_kv=G, head_dim=D, n_ff=F, rope_dim=D, n_expert=NE, n_expert_used=k)
    with tempfile.TemporaryDirectory() as d:
        return load_weights(write_synthetic_gguf(os.path.join(d, "m.gguf"), cfg, "F16", seed=0), DEV)


def llama(size: str):
    from distributed_llm_pipeline_b200.gguf import write_synthetic_gguf
    from distributed_llm_pipeline_b200.models.config import preset
    from distributed_llm_pipeline_b200.models.weights import load_weights
    E, H, D, _, F, n = SIZES[size]
    cfg = preset("llama-3-8b", vocab_size=VOCAB, n_embd=E, n_layer=n, n_head=H, n_head_kv=H, head_dim=D, n_ff=F, rope_dim=D)
    with tempfile.TemporaryDirectory() as d:
        return load_weights(write_synthetic_gguf(os.path.join(d, "m.gguf"), cfg, "F16", seed=0), DEV)


def event_ms(fn, reps=1):
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    torch.cuda.synchronize()
    e0.record()
    for _ in range(reps):
        fn()
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) / reps


def model_numbers(weights, prompt_lens=(512, 2048, 8192), batches=(1, 4, 16), ctx=2048, steps=32):
    from distributed_llm_pipeline_b200.models.modeldir import make_engine
    eng = make_engine(weights, n_ctx=max(max(prompt_lens), ctx + 4 * steps + 64), max_seqs=max(batches), page_size=64, max_batch_tokens=max(prompt_lens))
    g = torch.Generator().manual_seed(1)
    out = {"prefill_tok_s": {}, "decode_tok_s": {}}
    for n in prompt_lens:
        ids = torch.randint(3, VOCAB, (n,), generator=g, dtype=torch.int32)
        ms = []
        for _ in range(5):
            sid = eng.alloc_seq()
            ms.append(event_ms(lambda: eng.prefill(sid, ids)))
            eng.free_seq(sid)
        out["prefill_tok_s"][n] = round(n / statistics.median(ms[2:]) * 1e3)
    ids = torch.randint(3, VOCAB, (ctx,), generator=g, dtype=torch.int32)
    for B in batches:
        sids = [eng.alloc_seq() for _ in range(B)]
        for s in sids:
            eng.prefill(s, ids)
        eng.next_tok[:B].fill_(5)
        for _ in range(8):
            eng.decode(sids)
        ms = [event_ms(lambda: eng.decode(sids), steps) for _ in range(3)]
        out["decode_tok_s"][B] = round(B / statistics.median(ms) * 1e3, 1)
        for s in sids:
            eng.free_seq(s)
    return out


def graph_us(fn, n_copies: int, reps: int = 20) -> float:
    """Device time of one launch: `fn(i)` launches on operand copy i; a graph of launches over all copies, replayed."""
    n = max(n_copies, 8)
    s = torch.cuda.Stream()
    s.wait_stream(torch.cuda.current_stream())
    with torch.cuda.stream(s):
        fn(0)
    torch.cuda.current_stream().wait_stream(s)
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g):
        for i in range(n):
            fn(i % n_copies)
    for _ in range(3):
        g.replay()
    return statistics.median(event_ms(g.replay) for _ in range(reps)) / n * 1e3


def copies(nbytes: float) -> int:
    return max(1, min(48, int(300e6 // max(1, nbytes)) + 1))


def kernel_numbers(size: str, ctx: int = 2048, T: int = 2048):
    """(name, like-kernel pair, us, bytes, flops) rows of both models' kernels at this size."""
    from distributed_llm_pipeline_b200.gguf.constants import GGMLType
    from distributed_llm_pipeline_b200.ops import api as ops
    from distributed_llm_pipeline_b200.ops import layers as L
    from distributed_llm_pipeline_b200.ops.weights import DeviceWeight
    L.load_library()
    ops.need_full_library()
    E, H, D, R, F, _ = SIZES[size]
    bf, f16, f32, i32 = torch.bfloat16, torch.float16, torch.float32, torch.int32
    bw, fl, src = peaks()
    rows = []

    def rnd(*s, dt=bf):
        return (torch.randn(*s, device=DEV) * 0.1).to(dt)

    def add(model, kind, name, us, nbytes, flops):
        roof = max(nbytes / bw, flops / fl) * 1e6
        rows.append({"model": model, "kind": kind, "kernel": name, "us": round(us, 2), "roofline_us": round(roof, 2), "of_roofline": round(roof / us, 3)})

    # decode products: the stacked input projection and gate/up, one token
    for B in (1, 4):
        for kind, N, K in (("matvec in", 3 * H * D, E), ("matvec gate/up", 2 * F, E), ("matvec down", E, F), ("matvec out", E, H * D)):
            nb, c = N * K * 2, copies(N * K * 2)
            ws = [rnd(N, K) for _ in range(c)]
            h, y, w1, ho = rnd(B, K, dt=f32), rnd(B, K, dt=f32), rnd(K, dt=f32), rnd(B, K, dt=f32)
            x16 = rnd(B, K)
            if kind in ("matvec in", "matvec gate/up"):
                st = L.row_stage(h, K, K, 1e-5, y, w1, 4, ho)
            elif kind == "matvec out":
                st = L.row_stage(h, K, K, 1e-5, w2=w1[:D].contiguous(), groups2=H)
            else:
                st = L.row_stage(x16, K, K, 1e-5)
            out = torch.zeros(B, N, device=DEV, dtype=f32)
            act = torch.zeros(B, N // 2, device=DEV, dtype=bf)
            gl = kind == "matvec gate/up"
            add("talizen", f"{kind} B={B}", "matvec_kernel", graph_us(lambda i: L.matvec(st, ws[i], act if gl else out, B, L.OUT_GEGLU if gl else L.OUT_F32), c), nb, 2 * B * N * K)
            del ws
            dw = [DeviceWeight(GGMLType.F16, N // 2 if gl else N, K, [rnd(N // 2 if gl else N, K, dt=f16)]) for _ in range(c)]
            up = [DeviceWeight(GGMLType.F16, N // 2, K, [rnd(N // 2, K, dt=f16)]) for _ in range(c)] if gl else None
            o16, hx, xh = torch.zeros(B, N // 2, device=DEV, dtype=f16), rnd(B, K, dt=f32), rnd(B, K, dt=f16)
            if gl:
                us = graph_us(lambda i: ops.linear(dw[i], hx, "swiglu", w_up=up[i], norm_w=w1, eps=1e-5, out=o16), c)
            elif kind == "matvec in":
                us = graph_us(lambda i: ops.linear(dw[i], hx, "f32", norm_w=w1, eps=1e-5, out=out), c)
            else:
                us = graph_us(lambda i: ops.linear(dw[i], xh, "add", out=out), c)
            add("llama", f"{kind} B={B}", "gemv_dense_v3_kernel", us, nb, 2 * B * N * K)
            del dw, up
    # decode attention over ctx cached tokens
    for B in (1, 16):
        pages, mp = B * ctx // 64, ctx // 64
        c = copies(B * ctx * R * 2)
        cache = [rnd(pages, 1, 64, R) for _ in range(c)]
        bt = torch.arange(pages, device=DEV, dtype=i32).view(B, mp)
        slot, pos = torch.arange(B, device=DEV, dtype=i32), torch.full((B,), ctx - 1, device=DEV, dtype=i32)
        bm = L.latent_tile_rows(H, B)
        per = (H + bm - 1) // bm
        row0 = torch.tensor([b * H + i * bm for b in range(B) for i in range(per)], device=DEV, dtype=i32)
        nr = torch.tensor([min(bm, H - i * bm) for b in range(B) for i in range(per)], device=DEV, dtype=i32)
        ns = 1
        while ns * 2 <= min(148 // (B * per), (ctx + 63) // 64, 32):
            ns *= 2
        q, out = rnd(B, H * R), torch.zeros(B, H * R, device=DEV, dtype=bf)
        ws = (torch.zeros(ns * B * H * R, device=DEV), torch.zeros(ns * B * H * 2, device=DEV))
        us = graph_us(lambda i: L.latent_attention(q, cache[i], bt, slot, pos, row0, nr, B * per, bm, H, B, D ** -0.5, out, n_splits=ns, workspace=ws), c)
        add("talizen", f"attention decode B={B}", "latent_attn_mma_kernel (+ combine)", us, B * ctx * R * 2, 4 * B * H * ctx * R)
        del cache
        c = copies(B * ctx * H * D * 4)
        kc, vc = ([rnd(pages, H, 64, D, dt=f16) for _ in range(c)] for _ in range(2))
        ql, ol, kl = rnd(B, H * D, dt=f16), torch.zeros(B, H * D, device=DEV, dtype=f16), torch.full((B,), ctx, device=DEV, dtype=i32)
        wsl = (torch.zeros(B * H * 16 * D, device=DEV), torch.zeros(B * H * 16 * 2, device=DEV), torch.zeros(B * H, device=DEV, dtype=i32))
        us = graph_us(lambda i: ops.attn_paged(ql, kc[i], vc[i], bt, kl, H, H, D, bt_row=slot, n_splits=16, workspace=wsl, out=ol), c)
        add("llama", f"attention decode B={B}", "attn_decode_kernel", us, B * ctx * H * D * 4, 4 * B * H * ctx * D)
        del kc, vc
        # the recurrent step: the state is read and written once
        c = copies(B * H * D * D * 4)
        st = [torch.zeros(B, H, D, D, device=DEV) for _ in range(c)]
        proj, fb, lo, o = rnd(B, 3 * H * D, dt=f32), rnd(H * D, dt=f32), torch.full((H * D,), 0.3, device=DEV), torch.zeros(B, H * D, device=DEV)
        seg = torch.tensor([[b, b + 1] for b in range(B)], device=DEV, dtype=i32)
        us = graph_us(lambda i: L.hgrn2(proj, fb, lo, st[i], seg, slot, B, pos, o), c)
        add("talizen", f"recurrence decode B={B}", "recurrence_scan_kernel (hgrn2)", us, 2 * B * H * D * D * 4, 6 * B * H * D * D)
        # per-head products of latent attention
        c = copies(H * D * R * 2)
        uk = [rnd(H, R, D) for _ in range(c)]
        qr, qa = rnd(B, H * D, dt=f32), torch.zeros(B, H * R, device=DEV, dtype=bf)
        add("talizen", f"key absorption B={B}", "head_matmul_kernel", graph_us(lambda i: L.head_matmul(qr, D, D, uk[i], R, qa, R, B), c), H * D * R * 2, 2 * B * H * D * R)
        uv = [u.view(H, D, R) for u in uk]
        at = torch.zeros(B, H * D, device=DEV, dtype=bf)
        add("talizen", f"value expansion B={B}", "head_matmul_kernel", graph_us(lambda i: L.head_matmul(qa, R, R, uv[i], D, at, D, B, gate=qr[:, :H]), c), H * D * R * 2,
            2 * B * H * D * R)
        del uk, uv, st
    # prefill
    x, xh = rnd(T, E), rnd(T, E, dt=f16)
    for kind, N, K, gl in (("gemm in", 3 * H * D, E, False), ("gemm gate/up", 2 * F, E, True), ("gemm down", E, F, False)):
        w, xi = rnd(N, K), rnd(T, K)
        out = torch.zeros(T, N // 2 if gl else N, device=DEV, dtype=bf if gl else f32)
        add("talizen", f"{kind} T={T}", "gemm_tcgen05_kernel", graph_us(lambda i: L.linear(xi, w, out, L.OUT_GEGLU if gl else L.OUT_F32), 1), (N * K + T * K + T * N) * 2, 2 * T * N * K)
        xq = rnd(T, K, dt=f16)
        dw = DeviceWeight(GGMLType.F16, N // 2 if gl else N, K, [rnd(N // 2 if gl else N, K, dt=f16)])
        if gl:
            up, o16 = DeviceWeight(GGMLType.F16, N // 2, K, [rnd(N // 2, K, dt=f16)]), torch.zeros(T, N // 2, device=DEV, dtype=f16)
            us = graph_us(lambda i: ops.linear(dw, xq, "swiglu", w_up=up, out=o16), 1)
        elif kind == "gemm in":
            o16 = torch.zeros(T, N, device=DEV, dtype=f16)
            us = graph_us(lambda i: ops.linear(dw, xq, "f16", out=o16), 1)
        else:
            us = graph_us(lambda i: ops.linear(dw, xq, "add", out=out), 1)
        add("llama", f"{kind} T={T}", "gemm_tcgen05_kernel", us, (N * K + T * K + T * N) * 2, 2 * T * N * K)
    c = 4
    h, y, w1, xb = [rnd(T, E, dt=f32) for _ in range(c)], rnd(T, E, dt=f32), rnd(E, dt=f32), torch.zeros(T, E, device=DEV, dtype=bf)
    add("talizen", f"norm T={T}", "stage_rows_kernel", graph_us(lambda i: L.stage_rows(L.row_stage(h[i], E, E, 1e-5, y, w1, 4, h[i]), xb, T), c), T * E * 14, 0)
    o16 = torch.zeros(T, E, device=DEV, dtype=f16)
    add("llama", f"norm T={T}", "rmsnorm_kernel", graph_us(lambda i: ops.rmsnorm(h[i], w1, 1e-5, delta=y, out=o16), c), T * E * 14, 0)
    proj, fb, lo = rnd(T, 3 * H * D, dt=f32), rnd(H * D, dt=f32), torch.full((H * D,), 0.3, device=DEV)
    st, o = torch.zeros(1, H, D, D, device=DEV), torch.zeros(T, H * D, device=DEV)
    cu, z = torch.tensor([[0, T]], device=DEV, dtype=i32), torch.zeros(1, device=DEV, dtype=i32)
    pos = torch.arange(T, device=DEV, dtype=i32)
    table, first = L.scan_chunk_table([(0, T)], L.HGRN2_CHUNK)
    n = len(table) // 2
    chunks = (torch.tensor(table, device=DEV, dtype=i32).view(-1, 2), torch.tensor(first, device=DEV, dtype=i32), torch.zeros(n * H * D * D, device=DEV),
              torch.zeros(n * H * D, device=DEV))
    for name, ch in (("recurrence_scan_kernel (hgrn2)", None), ("hgrn2_chunk_* (3 kernels)", chunks)):
        us = graph_us(lambda i: L.hgrn2(proj, fb, lo, st, cu, z, 1, pos, o, ch), 1)
        add("talizen", f"token mixing T={T}", name, us, T * H * D * 16, 6 * T * H * D * D)
    q, k, v = (rnd(T // 64, H, 64, D, dt=f16) for _ in range(3))
    qh, oh = rnd(T, H * D, dt=f16), torch.zeros(T, H * D, device=DEV, dtype=f16)
    bt1 = torch.arange(T // 64, device=DEV, dtype=i32)
    add("llama", f"token mixing T={T}", "attn_prefill_tc_kernel", graph_us(lambda i: ops.attn_prefill(qh, k, v, bt1, 0, H, H, D, out=oh), 1), T * H * D * 8, 2 * T * T * H * D)
    cache = rnd(T // 64, 1, 64, R)
    bm = L.latent_tile_rows(H, T)
    row0 = torch.arange(0, T * H, bm, device=DEV, dtype=i32)
    nr = torch.full_like(row0, bm)
    qa, ctxo = rnd(T, H * R), torch.zeros(T, H * R, device=DEV, dtype=bf)
    at2 = torch.zeros(T, H * D, device=DEV, dtype=bf)
    row, z_t = bt1.view(1, -1), torch.zeros(T, device=DEV, dtype=i32)
    us = graph_us(lambda i: L.latent_attention(qa, cache, row, z_t, pos, row0, nr, row0.numel(), bm, H, T, D ** -0.5, ctxo), 1)
    add("talizen", f"attention prefill T={T} (absorbed)", "latent_attn_mma_kernel", us, T * H * D * 8, 2 * T * T * H * D)
    ukv, cx, kvr, qx = rnd(2 * H * D, R), rnd(T, R), torch.zeros(T, 2 * H * D, device=DEV, dtype=bf), torch.zeros(T, H * D, device=DEV, dtype=bf)
    us = graph_us(lambda i: L.latent_gather(cache, bt1, T, cx), 1)
    add("talizen", f"latent gather T={T}", "latent_gather_kernel", us, T * R * 4, 0)
    us = graph_us(lambda i: L.linear(cx, ukv, kvr), 1)
    add("talizen", f"key / value expansion T={T}", "gemm_tcgen05_kernel", us, (T * R + 2 * T * H * D + 2 * H * D * R) * 2, 4 * T * H * D * R)
    us = graph_us(lambda i: L.rows_attention(qx, kvr, T, 0, H, D, D, D, D ** -0.5, at2, gate=proj[:, :H]), 1)
    add("talizen", f"attention prefill T={T} (expanded)", "attn_prefill_tc_kernel<FA_ROWS>", us, T * H * D * 8, 2 * T * T * H * D)
    return rows, src


def moe_kernel_numbers(size: str, T: int = 2048):
    """The same for windowed attention and routed experts beside Qwen3-MoE.  Decode attention reads what the window shows; expert weights
    are streamed from other experts at every launch."""
    from types import SimpleNamespace

    from distributed_llm_pipeline_b200.gguf.constants import GGMLType
    from distributed_llm_pipeline_b200.ops import api as ops
    from distributed_llm_pipeline_b200.ops import layers as L
    from distributed_llm_pipeline_b200.ops.weights import DeviceWeight
    from distributed_llm_pipeline_b200.models.layered import key_ranges
    L.load_library()
    ops.need_full_library()
    E, H, G, D, NE, k, F, _, window, keep = MOE_SIZES[size]
    bf, f16, f32, i32 = torch.bfloat16, torch.float16, torch.float32, torch.int32
    bw, fl, src = peaks()
    rows = []

    def rnd(*s, dt=bf):
        return (torch.randn(*s, device=DEV) * 0.1).to(dt)

    def add(model, kind, name, us, nbytes, flops):
        roof = max(nbytes / bw, flops / fl) * 1e6
        rows.append({"model": model, "kind": kind, "kernel": name, "us": round(us, 2), "roofline_us": round(roof, 2), "of_roofline": round(roof / us, 3)})
    NI = (H + 2 * G) * D
    ones, zero = torch.ones(E, device=DEV), torch.zeros(E, device=DEV)
    for B in (1, 4):
        for kind, N, K in (("matvec in", NI, E), ("matvec out", E, H * D), ("router", NE, E)):
            nb, c = N * K * 2, copies(N * K * 2)
            ws = [rnd(N, K) for _ in range(c)]
            h, y, ho, x16, out = rnd(B, K, dt=f32), rnd(B, K, dt=f32), rnd(B, K, dt=f32), rnd(B, K), torch.zeros(B, N, device=DEV)
            st = L.row_stage(x16, K, K, 1e-5) if kind == "matvec out" else L.row_stage(h, K, K, 1e-5, y, None, 1, ho, ones, 1, zero)
            add("vozinex", f"{kind} B={B}", "matvec_kernel", graph_us(lambda i: L.matvec(st, ws[i], out, B), c), nb, 2 * B * N * K)
            del ws
            dw = [DeviceWeight(GGMLType.F16, N, K, [rnd(N, K, dt=f16)]) for _ in range(c)]
            xh = rnd(B, K, dt=f16)
            if kind == "matvec out":
                us = graph_us(lambda i: ops.linear(dw[i], xh, "add", out=out), c)
            elif kind == "matvec in":
                us = graph_us(lambda i: ops.linear(dw[i], h, "f32", norm_w=ones, eps=1e-5, out=out), c)
            else:
                us = graph_us(lambda i: [ops.linear(dw[i], h[t:t + 1], "f32", norm_w=ones, eps=1e-5, out=out[t:t + 1]) for t in range(B)], c)
            add("qwen3moe", f"{kind} B={B}", "gemv_dense_v3_kernel", us, nb, 2 * B * N * K)
            del dw
        # the chosen experts: k per token, other ones in every launch
        A, sets = B * k, max(1, NE // (B * k))
        stacks = copies(NE * F * E * 2)
        n = sets * stacks
        picks = [[(s * A + a) % NE for a in range(A)] for s in range(sets)]
        hot = min(A, NE)
        logits = []
        for p in picks:
            lg = torch.zeros(B, NE, device=DEV)
            for a, e in enumerate(p):
                lg[a // k, e] = 20.0 + a
            logits.append(lg)
        up, down = ([rnd(NE * F, E) for _ in range(stacks)], [rnd(NE * E, F) for _ in range(stacks)])
        h, act, y = rnd(B, E, dt=f32), rnd(A, F), torch.zeros(B, E, device=DEV)
        st, st2 = L.row_stage(h, E, E, 1e-5, w2=ones, b2=zero), L.row_stage(act, F, F, 1e-5)
        us = graph_us(lambda i: L.expert_matvec(st, logits[i % sets], L.Routing(None, NE, k), up[i // sets], F, act, B, down=False), n)
        add("vozinex", f"experts up B={B}", "expert_matvec_kernel", us, hot * F * E * 2, 2 * A * F * E)
        us = graph_us(lambda i: L.expert_matvec(st2, logits[i % sets], L.Routing(None, NE, k), down[i // sets], E, y, B, down=True), n)
        add("vozinex", f"experts down B={B}", "expert_matvec_kernel", us, hot * F * E * 2, 2 * A * F * E)
        del up, down
        gate, up, down = ([DeviceWeight(GGMLType.F16, NE * r, c, [rnd(NE * r, c, dt=f16)]) for _ in range(stacks)] for r, c in ((F, E), (F, E), (E, F)))
        ids = [torch.tensor(p, device=DEV, dtype=i32) for p in picks]
        acth, wt = rnd(A, F, dt=f16), torch.ones(A, device=DEV)
        if NE <= 32:          # up to four rows: a mat-vec per (token, expert)
            us = graph_us(lambda i: [ops.gemv_moe(gate[i // sets], h[a // k:a // k + 1], acth[a:a + 1], "swiglu", ids[i % sets][a:a + 1], F, w_up=up[i // sets], norm_w=ones, eps=1e-5)
                                     for a in range(A)], n)
            add("qwen3moe", f"experts up B={B}", "gemv (expert rows)", us, hot * 2 * F * E * 2, 4 * A * F * E)
            us = graph_us(lambda i: [ops.gemv_moe(down[i // sets], acth[a:a + 1], y[a // k:a // k + 1], "add", ids[i % sets][a:a + 1], E, out_scale=wt[a:a + 1]) for a in range(A)], n)
            add("qwen3moe", f"experts down B={B}", "gemv (expert rows)", us, hot * F * E * 2, 2 * A * F * E)
        else:
            plans = [ops.MoePlan(A, NE, DEV) for _ in ids]
            for q, p in zip(ids, plans):
                ops.moe_plan(q, NE, 16, p)
            xs, yh = rnd(A, E, dt=f16), torch.zeros(A, E, device=DEV)
            us = graph_us(lambda i: ops.linear_grouped(gate[i // sets], xs, acth, "swiglu", NE, F, 16, plans[i % sets], w_up=up[i // sets]), n)
            add("qwen3moe", f"experts up B={B}", "gemm_tcgen05_kernel (grouped)", us, hot * 2 * F * E * 2, 4 * A * F * E)
            us = graph_us(lambda i: ops.linear_grouped(down[i // sets], acth, yh, "f32", NE, E, 16, plans[i % sets]), n)
            add("qwen3moe", f"experts down B={B}", "gemm_tcgen05_kernel (grouped)", us, hot * F * E * 2, 2 * A * F * E)
        del gate, up, down
    # decode attention: what the window shows of a long sequence, beside a plain cache of that many keys
    m = SimpleNamespace(H=H, G=G, R=H // G, D=D, V=D, Dc=D, Vc=D, rot=D, window=window, keep=keep, chunk=0, maps=1, adjacent=False, rot_scale=1.0, eps=1e-5, scale=D ** -0.5, visible=lambda n: min(n, window + keep),
                        q_norm=torch.ones(H * D, device=DEV), k_norm=torch.ones(G * D, device=DEV),
                        inv_freq=(1e6 ** (-torch.arange(0, D, 2, dtype=torch.float64) / D)).float().to(DEV))
    seen, ctx = window + keep, 8192
    for B in (1, 4, 16):
        c, mp = copies(B * seen * G * D * 4), ctx // 64
        slot, pos = torch.arange(B, device=DEV, dtype=i32), torch.full((B,), ctx - 1, device=DEV, dtype=i32)
        kc, vc = ([rnd(B * mp, G, 64, D) for _ in range(c)] for _ in range(2))
        bt = torch.arange(B * mp, device=DEV, dtype=i32).view(B, mp)
        proj, out = rnd(B, NI, dt=f32), torch.zeros(B, H * D, device=DEV, dtype=bf)
        tiles = (slot, torch.ones_like(slot), B)
        ns = key_ranges(m, B, L.gqa_tile(m.R, 1)[0], ctx)
        us = graph_us(lambda i: L.gqa_decode(m, proj, kc[i], vc[i], bt, slot, pos, tiles, ns, out, B), c)
        add("vozinex", f"attention decode B={B}", f"gqa_attn_mma_kernel (fused, {ns} key ranges)", us, B * seen * G * D * 4, 4 * B * H * seen * D)
        del kc, vc
        mp = (seen + 63) // 64
        kc, vc = ([rnd(B * mp, G, 64, D, dt=f16) for _ in range(c)] for _ in range(2))
        bt = torch.arange(B * mp, device=DEV, dtype=i32).view(B, mp)
        kl, oh = torch.full((B,), seen, device=DEV, dtype=i32), torch.zeros(B, H * D, device=DEV, dtype=f16)
        us = graph_us(lambda i: ops.attn_decode_rope(proj, m.inv_freq, kc[i], vc[i], bt, kl, H, G, D, bt_row=slot, n_splits=16, neox=True, out=oh), c)
        add("qwen3moe", f"attention decode B={B}", "attn_decode_rope_kernel", us, B * seen * G * D * 4, 4 * B * H * seen * D)
        qh = rnd(B, H * D, dt=f16)
        ns = max(1, min(16, 2 * 148 // (B * G)))
        wsl = (torch.zeros(B * H * ns * D, device=DEV), torch.zeros(B * H * ns * 2, device=DEV), torch.zeros(B * H, device=DEV, dtype=i32))
        us = graph_us(lambda i: ops.attn_paged(qh, kc[i], vc[i], bt, kl, H, G, D, bt_row=slot, n_splits=ns, workspace=wsl, out=oh), c)
        add("qwen3moe", f"attention decode B={B}", "attn_decode_kernel (without norm and rotation)", us, B * seen * G * D * 4, 4 * B * H * seen * D)
        del kc, vc
    # prompts
    for kind, N, K in (("gemm in", NI, E), ("gemm out", E, H * D), ("router", NE, E)):
        w, xi, out = rnd(N, K), rnd(T, K), torch.zeros(T, N, device=DEV)
        add("vozinex", f"{kind} T={T}", "gemm_tcgen05_kernel", graph_us(lambda i: L.linear(xi, w, out), 1), (N * K + T * K + T * N * 2) * 2, 2 * T * N * K)
        dw, xq = DeviceWeight(GGMLType.F16, N, K, [rnd(N, K, dt=f16)]), rnd(T, K, dt=f16)
        o16 = torch.zeros(T, N, device=DEV, dtype=f16)
        us = graph_us(lambda i: ops.linear(dw, xq, "f16", out=o16) if kind == "gemm in" else ops.linear(dw, xq, "add" if kind == "gemm out" else "f32", out=out), 1)
        add("qwen3moe", f"{kind} T={T}", "gemm_tcgen05_kernel", us, (N * K + T * K + T * N * 2) * 2, 2 * T * N * K)
    hs, y, xb, o16 = [rnd(T, E, dt=f32) for _ in range(4)], rnd(T, E, dt=f32), torch.zeros(T, E, device=DEV, dtype=bf), torch.zeros(T, E, device=DEV, dtype=f16)
    us = graph_us(lambda i: L.stage_rows(L.row_stage(hs[i], E, E, 1e-5, y, None, 1, hs[i], ones, 1, zero), xb, T), 4)
    add("vozinex", f"norm T={T}", "stage_reg_kernel", us, T * E * 14, 0)
    add("qwen3moe", f"norm T={T}", "rmsnorm_kernel", graph_us(lambda i: ops.rmsnorm(hs[i], ones, 1e-5, delta=y, out=o16), 4), T * E * 14, 0)
    A = T * k
    logits = torch.randn(T, NE, device=DEV)
    ids, w = torch.zeros(A, dtype=i32, device=DEV), torch.zeros(A, device=DEV)
    add("vozinex", f"route T={T}", "route_kernel", graph_us(lambda i: L.route(logits, L.Routing(None, NE, k), ids, w, T), 1), T * NE * 4 + A * 8, 0)
    add("qwen3moe", f"route T={T}", "moe_route_ex_kernel", graph_us(lambda i: ops.moe_route_ex(logits, NE, k, True, ids, w), 1), T * NE * 4 + A * 8, 0)
    plan, per = ops.MoePlan(A, NE, DEV), A // NE
    tile = 16 if per <= 16 else 32 if per <= 32 else 64 if per <= 96 else 128
    add("both", f"plan T={T}", "moe_plan_kernel", graph_us(lambda i: ops.moe_plan(ids, NE, tile, plan), 1), A * 16, 0)
    xs = rnd(A, E)
    add("both", f"gather T={T}", "moe_gather_kernel", graph_us(lambda i: L.expert_gather(xb, plan, k, A, xs), 1), (T + A) * E * 2, 0)
    up, down, act, ey = rnd(NE * F, E), rnd(NE * E, F), rnd(A, F), torch.zeros(A, E, device=DEV)
    us = graph_us(lambda i: L.linear_grouped(xs, up, F, NE, tile, plan, act, L.OUT_RELU2), 1)
    add("vozinex", f"experts up T={T}", "gemm_tcgen05_kernel (grouped)", us, (NE * F * E + A * E + A * F) * 2, 2 * A * F * E)
    us = graph_us(lambda i: L.linear_grouped(act, down, E, NE, tile, plan, ey), 1)
    add("vozinex", f"experts down T={T}", "gemm_tcgen05_kernel (grouped)", us, (NE * F * E + A * F + A * E * 2) * 2, 2 * A * F * E)
    us = graph_us(lambda i: L.expert_combine(ey, plan, w, T, k, y), 1)
    add("vozinex", f"combine T={T}", "moe_combine_kernel", us, (A + T) * E * 4, 0)
    add("qwen3moe", f"combine T={T}", "moe_combine_kernel", graph_us(lambda i: ops.moe_combine(ey, plan, w, T, k, y), 1), (A + 2 * T) * E * 4, 0)
    del up, down
    gate, up, down = (DeviceWeight(GGMLType.F16, NE * r, c, [rnd(NE * r, c, dt=f16)]) for r, c in ((F, E), (F, E), (E, F)))
    xh, acth = rnd(A, E, dt=f16), rnd(A, F, dt=f16)
    us = graph_us(lambda i: ops.linear_grouped(gate, xh, acth, "swiglu", NE, F, tile, plan, w_up=up), 1)
    add("qwen3moe", f"experts up T={T}", "gemm_tcgen05_kernel (grouped)", us, (2 * NE * F * E + A * E + A * F) * 2, 4 * A * F * E)
    us = graph_us(lambda i: ops.linear_grouped(down, acth, ey, "f32", NE, E, tile, plan), 1)
    add("qwen3moe", f"experts down T={T}", "gemm_tcgen05_kernel (grouped)", us, (NE * F * E + A * F + A * E * 2) * 2, 2 * A * F * E)
    proj, q = rnd(T, NI, dt=f32), torch.zeros(T, H * D, device=DEV, dtype=bf)
    kc, vc = (rnd(4 * T // 64, G, 64, D) for _ in range(2))
    bt = torch.arange(4 * T // 64, device=DEV, dtype=i32).view(1, -1)
    slot0 = torch.zeros(T, device=DEV, dtype=i32)
    out = torch.zeros(T, H * D, device=DEV, dtype=bf)
    q16, k16, v16, o16 = rnd(T, H * D, dt=f16), rnd(4 * T // 64, G, 64, D, dt=f16), rnd(4 * T // 64, G, 64, D, dt=f16), torch.zeros(T, H * D, device=DEV, dtype=f16)
    p16, ar = proj.to(f16), torch.arange(T, device=DEV, dtype=i32)
    us = graph_us(lambda i: L.gqa_prepare(m, proj, kc, vc, bt, slot0, ar, ar, q, T), 1)
    add("vozinex", f"norm, rotation, cache rows T={T}", "gqa_prepare_kernel", us, T * NI * 6, 0)
    us = graph_us(lambda i: ops.rope_kv(p16, ar, ar, m.inv_freq, k16, v16, H, G, D, True), 1)
    add("qwen3moe", f"norm, rotation, cache rows T={T}", "rope_kv_kernel", us, T * NI * 4, 0)
    for p0 in (0, 3 * T):          # the whole prompt; a portion far behind the window
        pos = torch.arange(p0, p0 + T, device=DEV, dtype=i32)
        row0 = torch.arange(T - 128, -1, -128, device=DEV, dtype=i32)
        tiles = (row0, torch.full_like(row0, 128), row0.numel())
        mask = sum(min(p + 1, window + min(keep, max(0, p + 1 - window))) for p in range(p0, p0 + T))
        us = graph_us(lambda i: L.gqa_flash(m, q, kc, vc, bt, slot0, pos, tiles, out, T), 1)
        add("vozinex", f"attention prefill T={T} at {p0}", "attn_prefill_tc_kernel<FA_TILES>", us, (2 * H + 2 * G) * D * T * 2, 4 * mask * H * D)
        us = graph_us(lambda i: ops.attn_prefill(q16, k16, v16, bt[0], p0, H, G, D, out=o16), 1)
        add("qwen3moe", f"attention prefill T={T} at {p0}", "attn_prefill_tc_kernel", us, (2 * H + 2 * G) * D * T * 2, 4 * sum(range(p0 + 1, p0 + T + 1)) * H * D)
    return rows, src


def main(argv=None) -> dict:
    ap = argparse.ArgumentParser(description=__doc__.split("\n")[0])
    ap.add_argument("--sizes", default=",".join([*SIZES, *MOE_SIZES, *hybrid.HYBRID_SIZES, *parallel.PARALLEL_SIZES]))
    ap.add_argument("--no-models", action="store_true", help="kernels only")
    ap.add_argument("--no-kernels", action="store_true", help="whole models only")
    a = ap.parse_args(argv)
    res = {"metric": "layers_bench", "unit": "tok/s", "data": "synthetic (random weights and token ids)", "dtype": "bf16 (talizen, vozinex, nifalorn, rigalorn) / fp16 (llama, qwen3moe)", "sizes": {}}
    for size in a.sizes.split(","):
        moe = size in MOE_SIZES
        if size in hybrid.HYBRID_SIZES or size in parallel.PARALLEL_SIZES:
            if size in hybrid.HYBRID_SIZES:
                names = ("width", "lightning_heads", "mamba2_heads", "heads", "kv_heads", "experts", "experts_per_token", "ff", "shared_ff", "layers", "chunk")
                values, models, kernels = hybrid.HYBRID_SIZES[size], (("nifalorn", hybrid.nifalorn), ("vozinex", hybrid.vozinex)), hybrid.kernel_numbers
            else:
                names = ("width", "heads", "kv_heads", "delta_kv_heads", "rot_dim", "q_rank", "kv_rank", "ff", "layers", "window")
                values, models, kernels = parallel.PARALLEL_SIZES[size], (("rigalorn", parallel.rigalorn), ("nifalorn", parallel.nifalorn)), parallel.kernel_numbers
            r = {"config": {**dict(zip(names, values)), "vocab": VOCAB}}
            if not a.no_models:
                for name, make in models:
                    w = make(size)
                    r[name] = {"weights_gb": round(w.nbytes() / 1e9, 3), **model_numbers(w)}
                    del w
                    torch.cuda.empty_cache()
            if not a.no_kernels:
                r["kernels"], res["peaks"] = kernels(size, graph_us, copies, peaks)
            res["sizes"][size] = r
            continue
        names = ("width", "heads", "kv_heads", "head_dim", "experts", "experts_per_token", "ff", "layers", "window", "keep_first") if moe else \
            ("width", "heads", "head_dim", "kv_rank", "ff", "layers")
        r = {"config": {**dict(zip(names, MOE_SIZES[size] if moe else SIZES[size])), "vocab": VOCAB}}
        if not a.no_models:
            for name, make in (("vozinex", vozinex), ("qwen3moe", qwen3moe)) if moe else (("talizen", talizen), ("llama", llama)):
                w = make(size)
                r[name] = {"weights_gb": round(w.nbytes() / 1e9, 3), **model_numbers(w)}
                del w
                torch.cuda.empty_cache()
        if not a.no_kernels:
            r["kernels"], res["peaks"] = (moe_kernel_numbers if moe else kernel_numbers)(size)
        res["sizes"][size] = r
    return res


if __name__ == "__main__":
    print(json.dumps(main(), indent=1))
