"""Layer-list models on the GPU: every kernel alone, and whole models through the engine and scheduler, against plain float64 code."""
import math

import pytest
import torch

import layer_models as lm
import plain_layers as plain

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F64 = torch.float64
BF16, F32 = torch.bfloat16, torch.float32
TYPES = [pytest.param(BF16, id="bf16"), pytest.param(F32, id="f32")]


def ops():
    from distributed_llm_pipeline_b200.ops import layers
    layers.load_library()
    return layers


def rel(got, want):
    want = want.to(F64).cpu()
    return float((got.to(F64).cpu() - want).abs().max() / want.abs().max().clamp_min(1e-30))


def gen(seed):
    g = torch.Generator().manual_seed(seed)
    return lambda *s, scale=1.0: torch.randn(*s, generator=g) * scale


# ---- matrix products and row preparation -----------------------------------------------------------------------------------
def stage_plain(h, y, w1, g1, w2, g2, eps):
    v = h.to(F64)
    if y is not None:
        v = v + plain.grouped_norm(y.to(F64), w1.to(F64), g1, eps)
    kept = v
    if w2 is not None:
        v = plain.grouped_norm(v, w2.to(F64).repeat(v.shape[-1] // w2.numel()), g2, eps)
    return kept, v


@pytest.mark.parametrize("dt", TYPES)
@pytest.mark.parametrize("T,K,N,g1,g2", [(1, 72, 101, 3, 0), (2, 4096, 512, 4, 0), (3, 200, 33, 0, 0), (4, 1040, 258, 1, 2), (1, 2048, 4, 0, 16), (4, 96, 7, 0, 4),
                                         (9, 72, 101, 3, 0), (70, 1040, 258, 2, 5), (17, 136, 300, 0, 0), (300, 96, 40, 0, 8)])
def test_products_with_staging(dt, T, K, N, g1, g2):
    L, r = ops(), gen(K + N)
    Kp = (K + 7) // 8 * 8
    eps = 1e-4
    h, y, w1 = r(T, K).to(DEV), (r(T, K, scale=0.05) if g1 else None), (r(K) if g1 else None)
    w2 = (r(K // g2 if N in (4, 7, 40) else K) if g2 else None)             # one weight for the whole row, or one shared by all groups
    w = torch.zeros(N, Kp, dtype=dt)
    w[:, :K] = r(N, K, scale=K ** -0.5).to(dt)
    w = w.to(DEV)
    y, w1, w2 = (t.to(DEV) if t is not None else None for t in (y, w1, w2))
    kept, v = stage_plain(*(t.cpu() if isinstance(t, torch.Tensor) else t for t in (h, y, w1, max(g1, 1), w2, max(g2, 1), eps)))
    h_out = torch.zeros(T, K, device=DEV) if g1 else None
    out = torch.full((T, N), float("nan"), device=DEV)
    st = L.row_stage(h, K, Kp, eps, y, w1, max(g1, 1), h_out, w2, max(g2, 1))
    if T <= 4:
        L.matvec(st, w, out, T)
    else:
        xb = torch.full((T, Kp), float("nan"), device=DEV).to(dt)
        L.stage_rows(st, xb, T)
        assert rel(xb[:, :K], v) < (5e-3 if dt == BF16 else 2e-6) and bool((xb[:, K:] == 0).all())
        L.linear(xb, w, out)
    if g1:
        assert rel(h_out, kept) < 1e-6
    want = v.to(dt).to(F64) @ w[:, :K].cpu().to(F64).T
    assert rel(out, want) < (6e-3 if dt == BF16 else 3e-6)


@pytest.mark.parametrize("dt", TYPES)
@pytest.mark.parametrize("T", [1, 2, 4, 5, 40, 200])
@pytest.mark.parametrize("K,F", [(72, 36), (256, 300)])
def test_geglu(dt, T, K, F):
    L, r = ops(), gen(F)
    x, gate, up = r(T, K).to(dt), r(F, K, scale=2 * K ** -0.5).to(dt), r(F, K, scale=K ** -0.5).to(dt)
    w = torch.stack([gate, up], 1).reshape(2 * F, K).to(DEV)
    out = torch.zeros(T, F, dtype=dt, device=DEV)
    xd = x.to(DEV)
    if T <= 4:
        L.matvec(L.row_stage(xd, K, K, 0.0), w, out, T, geglu=True)
    else:
        L.linear(xd, w, out, geglu=True)
    want = plain.gelu_tanh(x.to(F64) @ gate.to(F64).T) * (x.to(F64) @ up.to(F64).T)
    assert rel(out, want) < (6e-3 if dt == BF16 else 3e-6)


@pytest.mark.parametrize("dt", TYPES)
@pytest.mark.parametrize("T,H,kx,N,gated", [(1, 5, 12, 40, False), (4, 2, 64, 160, True), (16, 3, 40, 20, True), (17, 1, 96, 64, False), (130, 4, 32, 70, True)])
def test_head_matmul(dt, T, H, kx, N, gated):
    L, r = ops(), gen(T)
    Kp = (kx + 31) // 32 * 32
    x, gate = r(T, H * kx + 3), r(T, H + 2)
    w = torch.zeros(H, N, Kp)
    w[:, :, :kx] = r(H, N, kx, scale=kx ** -0.5)
    w = w.to(dt)
    out = torch.zeros(T, H * N + 1, dtype=dt, device=DEV)
    L.head_matmul(x.to(DEV), kx, kx, w.to(DEV), N, out, N, T, gate=gate.to(DEV) if gated else None)
    want = torch.einsum("thk,hnk->thn", x[:, :H * kx].reshape(T, H, kx).to(dt).to(F64), w[:, :, :kx].to(F64))
    if gated:
        want = want / (1 + torch.exp(-gate[:, :H, None].to(F64)))
    assert rel(out[:, :H * N], want.reshape(T, -1)) < (6e-3 if dt == BF16 else 3e-6)


# ---- recurrence ----------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("form,H,D,V", [("scan", 3, 20, 12), ("scan", 2, 64, 64), ("scan", 2, 128, 128), ("scan", 1, 160, 48), ("scan", 2, 300, 20), ("scan", 1, 8, 130),
                                        ("chunks", 3, 20, 12), ("chunks", 2, 64, 64), ("chunks", 2, 128, 128), ("chunks", 1, 48, 150), ("chunks", 4, 100, 33), ("chunks", 1, 8, 64)])
def test_hgrn2_segments_and_carried_state(form, H, D, V):
    """Ragged segments, some continuing a state; strong and weak forgetting; every portion length against the whole."""
    L, r = ops(), gen(D)
    lens, n = [297, 1, 2, 140, 64], 5
    q, z, v = [r(t, H * D) for t in lens], [r(t, H * D, scale=3.0) + 1 for t in lens], [r(t, H * V) for t in lens]
    for i in (0, 3):
        z[i][::7] = -40.0        # forgets everything ...
        z[i][1::7] = 25.0        # ... or nothing
    fb, lower = r(H * D), (torch.rand(H * D, generator=torch.Generator().manual_seed(1)) * 0.9)
    lower[::3] = 0
    want, state = [], torch.full((7, H, D, V), float("nan"), device=DEV)      # a new sequence must not read what its slot held
    slots, at = [4, 0, 6, 2, 3], [0] * n
    for i in range(n):
        f = plain.hgrn2_gates((z[i] + fb).to(F64), lower.to(F64)).reshape(-1, H, D)
        want.append(plain.hgrn2_scan((q[i] * torch.sigmoid(q[i])).to(F64).reshape(-1, H, D), f, v[i].to(F64).reshape(-1, H, V)))
    got = [[] for _ in range(n)]
    for portion in (33, 2, 1, 3, 17, 64, 5, 130, 100):
        act = [i for i in range(n) if at[i] < lens[i]]
        if not act:
            break
        cut = {i: min(portion + i, lens[i] - at[i]) for i in act}
        proj = torch.cat([torch.cat([q[i], z[i], v[i]], 1)[at[i]:at[i] + cut[i]] for i in act]).to(DEV)
        ends = torch.tensor([cut[i] for i in act]).cumsum(0).tolist()
        segs = [(hi - cut[i], hi) for i, hi in zip(act, ends)]
        i32 = dict(dtype=torch.int32, device=DEV)
        pos = torch.cat([torch.arange(at[i], at[i] + cut[i]) for i in act]).to(torch.int32).to(DEV)
        out = torch.zeros(proj.shape[0], H * V, device=DEV)
        chunks = None
        if form == "chunks":
            table, first = L.hgrn2_chunk_table(segs)
            k = len(table) // 2
            chunks = (torch.tensor(table, **i32).view(-1, 2), torch.tensor(first, **i32), torch.full((k * H * D * V,), float("nan"), device=DEV),
                      torch.full((k * H * D,), float("nan"), device=DEV))
        L.hgrn2(proj, fb.to(DEV), lower.to(DEV), state, torch.tensor(segs, **i32), torch.tensor([slots[i] for i in act], **i32), len(act), pos, out, chunks)
        for i, o in zip(act, out.split([cut[i] for i in act])):
            got[i].append(o)
            at[i] += cut[i]
    for i in range(n):
        tol = 1e-5 if form == "scan" else 4e-3         # the chunk form rounds v to bf16
        assert rel(torch.cat(got[i]), want[i][0][:at[i]].reshape(at[i], -1)) < tol
        if at[i] == lens[i]:
            assert rel(state[slots[i]], want[i][1]) < tol


# ---- latent attention ------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dt", TYPES)
@pytest.mark.parametrize("H,R,page,splits", [(1, 32, 16, 1), (5, 40, 16, 4), (20, 160, 64, 1), (3, 544, 64, 2), (50, 96, 16, 8), (16, 512, 64, 1)])
def test_latent_attention(dt, H, R, page, splits):
    """Portions of several requests over scattered pages; one key per query stands out: far back, on both sides of every page border,
    the first token, the query's own position."""
    L, r = ops(), gen(R)
    Rc = (R + 31) // 32 * 32
    spans = [(0, 3), (4 * page - 2, 5), (page - 1, 1), (9 * page + 3, 2), (0, 70)]      # (cached before, new) of every request
    max_pages, perm = 12, torch.randperm(60, generator=torch.Generator().manual_seed(2))
    cache, bt = torch.zeros(60, 1, page, Rc), perm.view(5, 12).to(torch.int32)
    cache.view(-1, Rc)[:] = 1e4                      # rows nobody wrote
    scale, rows_q, want, tok_slot, pos, row0, rows = 0.25, [], [], [], [], [], []
    bm, base = L.latent_tile_rows(H, sum(n for _, n in spans)), 0
    for s, (p0, n) in enumerate(spans):
        k = torch.arange(p0 + n)
        c = torch.zeros(p0 + n, Rc)
        c[:, :R] = r(p0 + n, R)
        c = c.to(dt)
        cache.view(-1, Rc)[bt[s, k // page].long() * page + k % page] = c.float()
        q = torch.zeros(n, H, Rc)
        q[:, :, :R] = r(n, H, R, scale=R ** -0.5)
        marks = sorted({0, p0, *[b + d for b in range(page, p0 + n, page) for d in (-1, 0)]})
        for t in range(n):
            for h in range(H):
                j = ([m for m in marks if m <= p0 + t] + [p0 + t])[(t + h) % (len([m for m in marks if m <= p0 + t]) + 1)]
                q[t, h, :R] += c[j, :R].float() * (12 / scale / R)
        q = q.to(dt)
        rows_q.append(q)
        sc = torch.einsum("thr,jr->thj", q.to(F64), c.to(F64)) * scale
        sc = sc.masked_fill(k[None, None] > (p0 + torch.arange(n))[:, None, None], -math.inf)
        want.append(torch.softmax(sc, -1) @ c.to(F64))
        tok_slot += [s] * n
        pos += list(range(p0, p0 + n))
        for i in range(0, n * H, bm):
            row0.append(base + i)
            rows.append(min(bm, n * H - i))
        base += n * H
    q, T = torch.cat(rows_q).reshape(len(pos), H * Rc).to(DEV), len(pos)
    i32 = dict(dtype=torch.int32, device=DEV)
    out = torch.zeros(T, H * Rc, dtype=dt, device=DEV)
    ws = (torch.empty(splits * T * H * Rc, device=DEV), torch.empty(splits * T * H * 2, device=DEV))
    L.latent_attention(q, cache.to(dt).to(DEV), bt.to(DEV), torch.tensor(tok_slot, **i32), torch.tensor(pos, **i32), torch.tensor(row0, **i32),
                       torch.tensor(rows, **i32), len(row0), bm, H, T, scale, out, n_splits=splits, workspace=ws)
    assert rel(out, torch.cat(want).reshape(T, -1)) < (6e-3 if dt == BF16 else 5e-6)


@pytest.mark.parametrize("H,D,V,pos0,T", [(2, 64, 64, 0, 128), (3, 32, 48, 0, 300), (2, 128, 64, 77, 131), (1, 20, 128, 512, 130), (4, 128, 128, 1, 257)])
def test_expanded_attention(H, D, V, pos0, T):
    """The flash kernel on expanded rows: a key that stands out at tile edges, at the start, and at the query itself; later keys unseen."""
    L, r = ops(), gen(T)
    Dp, Vp, S, scale = (D + 63) // 64 * 64, (V + 63) // 64 * 64, pos0 + T, 0.17
    k, v, q, gate = r(S, H, D).to(BF16), r(S, H, V).to(BF16), r(T, H, D, scale=D ** -0.5), r(T, H)
    marks = [m for m in (0, 1, 63, 64, 127, 128, 255, 256, S - 1) if m < S]
    for t in range(T):
        for h in range(H):
            j = marks[(t + h) % len(marks)]                  # also keys the query must not see
            q[t, h] += k[j, h].float() * (12 / scale / D)
    kv = torch.zeros(S, H * (Dp + Vp), dtype=BF16)
    kv[:, :H * Dp].view(S, H, Dp)[:, :, :D] = k
    kv[:, H * Dp:].view(S, H, Vp)[:, :, :V] = v
    qp = torch.empty(T, H * Dp, dtype=BF16, device=DEV)
    L.head_rows(q.reshape(T, H * D).to(DEV), H, D, Dp, qp)
    out = torch.zeros(T, H * V + 3, dtype=BF16, device=DEV)
    L.rows_attention(qp, kv.to(DEV), S, pos0, H, Dp, Vp, V, scale, out, gate=gate.to(DEV))
    L.check_waits()
    s = torch.einsum("thd,jhd->htj", q.to(BF16).to(F64), k.to(F64)) * scale
    s = s.masked_fill(torch.arange(S)[None, None] > (pos0 + torch.arange(T))[None, :, None], -math.inf)
    want = torch.einsum("htj,jhv->thv", torch.softmax(s, -1), v.to(F64)) / (1 + torch.exp(-gate.to(F64)))[:, :, None]
    assert rel(out[:, :H * V], want.reshape(T, -1)) < 6e-3 and not out[:, H * V:].any()


def test_latent_gather():
    L = ops()
    cache = torch.randn(9, 1, 16, 96, device=DEV).to(BF16)
    bt = torch.tensor([7, 0, 3, 8], dtype=torch.int32, device=DEV)
    out = torch.zeros(50, 96, dtype=BF16, device=DEV)
    L.latent_gather(cache, bt, 50, out)
    assert torch.equal(out, cache[[7, 0, 3, 8]].reshape(-1, 96)[:50])


@pytest.mark.parametrize("dt", TYPES)
def test_latent_write_and_embed(dt):
    L, r = ops(), gen(3)
    proj, w = r(7, 50), r(40)
    cache = torch.full((4, 1, 16, 64), 7.0, device=DEV).to(dt)
    slot = torch.tensor([0, 15, 16, 63, -1, 31, 40], dtype=torch.int32, device=DEV)
    L.latent_write(proj.to(DEV)[:, 10:50], w.to(DEV), 1e-4, 40, slot, cache, 7)
    want = plain.rms(proj[:, 10:].to(F64), 1e-4) * w.to(F64)
    rows = cache.view(-1, 64)
    for i, s in enumerate(slot.tolist()):
        if s >= 0:
            assert rel(rows[s, :40], want[i]) < (5e-3 if dt == BF16 else 1e-6) and not rows[s, 40:].any()
    assert int((rows == 7).all(1).sum()) == 64 - 6
    table, h = r(11, 24).to(dt).to(DEV), torch.zeros(5, 20, device=DEV)
    L.embed(table, torch.tensor([0, 10, 3, 3, 9], dtype=torch.int32, device=DEV), h, 5)
    assert torch.equal(h, table[[0, 10, 3, 3, 9], :20].float())


# ---- whole models ------------------------------------------------------------------------------------------------------------------
LIMIT = {"bf16": 0.08, "f32": 6e-5}     # worst row of hundreds; the fp32 runs are the sharp ones


def engine(path, dtype, **kw):
    from distributed_llm_pipeline_b200.models.modeldir import make_engine
    from distributed_llm_pipeline_b200.models.weights import load_weights
    return make_engine(load_weights(path, DEV, dtype=dtype), **{"n_ctx": 768, "max_seqs": 4, "page_size": 16, "max_batch_tokens": 256, **kw})


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    root, out = tmp_path_factory.mktemp("layered"), {}
    for name, cfg in lm.CONFIGS.items():
        w = lm.weights(cfg, seed=len(name))
        out[name] = (cfg, w, lm.write(str(root / name), cfg, w))
    return out


@pytest.mark.parametrize("dtype", ["bf16", "f32"])
@pytest.mark.parametrize("name", list(lm.CONFIGS))
def test_cuts_of_a_prompt(models, name, dtype):
    cfg, w, path = models[name]
    eng = engine(path, dtype)
    ids = lm.tokens(cfg, 150)
    want, _ = plain.forward(cfg, w, ids)
    first = None
    for cut in ([150], [1] * 20 + [130], [2] * 10 + [3] * 10 + [100], [15, 1, 1, 15, 64, 2, 52], [118] + [1] * 32):
        sid, got, at = eng.alloc_seq(), [], 0
        for n in cut:
            got.append(eng.step([(sid, ids[at:at + n])], [list(range(n))]))
            at += n
        got = torch.cat(got)
        first = got if first is None else first
        assert lm.error(got, want) < LIMIT[dtype], cut
        assert lm.error(got, first.double().cpu()) < LIMIT[dtype], cut
        eng.free_seq(sid)
    assert len(eng.kv.free) == eng.kv.n_pages


@pytest.mark.parametrize("dtype", ["bf16", "f32"])
@pytest.mark.parametrize("name", ["odd", "wide", "single"])
def test_mixed_batches_and_reused_slots(models, name, dtype):
    """Eleven unequal requests through four slots and a pool that holds about two of the long ones, in random portions beside single tokens."""
    from distributed_llm_pipeline_b200.serving.trace_runner import TraceRunner
    cfg, w, path = models[name]
    eng = engine(path, dtype, n_pages=40, max_batch_tokens=200)
    run, g = TraceRunner(eng), torch.Generator().manual_seed(5)
    ids = {f"r{i}": lm.tokens(cfg, n, seed=i) for i, n in enumerate((200, 3, 120, 1, 64, 65, 180, 17, 16, 90, 31))}
    want = {k: plain.forward(cfg, w, v)[0] for k, v in ids.items()}
    queue, live, at = list(ids), [], {k: 0 for k in ids}

    def pages(k):
        return (len(ids[k]) + 15) // 16
    while queue or live:
        while queue and len(live) < 4 and sum(map(pages, live)) + pages(queue[0]) <= 40:
            live.append(queue.pop(0))
        entries, rows = [], []
        for k in live:
            n = [1, 1, 1, 2, 3, 16, 33, 70, 150][int(torch.randint(0, 9, (1,), generator=g))]
            n = min(n, len(ids[k]) - at[k])
            entries.append({"id": k, "tokens": ids[k][at[k]:at[k] + n], "want": list(range(n))})
            rows.append(want[k][at[k]:at[k] + n])
            at[k] += n
        end = [k for k in live if at[k] == len(ids[k])]
        assert lm.error(run.step(entries, end), torch.cat(rows)) < LIMIT[dtype]
        live = [k for k in live if k not in end]
    assert len(eng.kv.free) == 40 and not run.sids


@pytest.mark.parametrize("dtype", ["bf16", "f32"])
def test_long_decoding(models, dtype):
    """Hundreds of decoded tokens through captured graphs (several key-range splits), two sequences of different length together."""
    cfg, w, path = models["odd"]
    eng = engine(path, dtype, page_size=64)
    ids = {s: lm.tokens(cfg, 640, seed=s) for s in (0, 1)}
    want = {s: plain.forward(cfg, w, v)[0] for s, v in ids.items()}
    sids = {s: eng.alloc_seq() for s in ids}
    eng.step([(sids[0], ids[0][:200]), (sids[1], ids[1][:7])])
    got = {0: [], 1: []}
    for t in range(330):
        lg = eng.step([(sids[0], [ids[0][200 + t]]), (sids[1], [ids[1][7 + t]])])
        got[0].append(lg[0])
        got[1].append(lg[1])
    assert len(eng._graphs) >= 2
    assert lm.error(torch.stack(got[0]), want[0][200:530]) < LIMIT[dtype]
    assert lm.error(torch.stack(got[1]), want[1][7:337]) < LIMIT[dtype]


@pytest.mark.parametrize("name", ["odd", "attention"])
def test_far_token_decides(models, name):
    """The head reads what one far token left: changing it must move the logits as in the plain model, from prompts and from decoding."""
    cfg, w, path = models[name]
    eng = engine(path, "f32")
    base = lm.tokens(cfg, 300)
    for place in (0, 1, 15, 16, 63, 64, 250):
        ids = list(base)
        ids[place] = (ids[place] + 1) % cfg["vocab"]
        want = plain.forward(cfg, w, ids)[0][-3:] - plain.forward(cfg, w, base)[0][-3:]
        got = []
        for seq in (ids, base):
            sid = eng.alloc_seq()
            rows = [eng.step([(sid, seq[:-2])])] + [eng.step([(sid, [t])]) for t in seq[-2:]]
            got.append(torch.cat(rows))
            eng.free_seq(sid)
        d = (got[0] - got[1]).double().cpu()
        assert (d - want).abs().max() < 2e-3 * max(1e-1, float(want.abs().max())), place


@pytest.mark.parametrize("name", ["odd", "wide", "recurrent"])
@pytest.mark.parametrize("dtype", ["bf16", "f32"])
def test_greedy_generation_through_the_scheduler(models, name, dtype):
    from distributed_llm_pipeline_b200.serving.orchestrator import build_service
    from distributed_llm_pipeline_b200.serving.sampler import SamplingParams
    from distributed_llm_pipeline_b200.serving.scheduler import Request
    cfg, w, path = models[name]
    sched, info, _ = build_service(path, "cuda:0", n_ctx=256, n_slots=3, n_batch=48, page_size=16, dtype=dtype)
    assert info["arch"] == "talizen"
    sched.warmup()
    greedy = SamplingParams(temperature=0.0)
    prompts = [lm.tokens(cfg, n, seed=n) for n in (60, 4, 100, 17, 1)]
    reqs = [sched.submit(Request(prompt=p, n_predict=24, sampling=greedy)) for p in prompts]
    while not all(r.done.is_set() for r in reqs):
        assert sched.step()
    for p, r in zip(prompts, reqs):
        assert len(r.output_ids) == 24
        lg = plain.forward(cfg, w, p + r.output_ids)[0]
        scale = float(lg.std())
        for i, t in enumerate(r.output_ids):
            row = lg[len(p) - 1 + i]
            assert row.max() - row[t] < (0.15 if dtype == "bf16" else 1e-3) * scale
    alone = sched.generate(prompts[0], n_predict=24, sampling=greedy)
    if dtype == "f32":
        assert alone.output_ids == reqs[0].output_ids


def test_seeded_sampling_does_not_depend_on_the_batch(models):
    from distributed_llm_pipeline_b200.serving.orchestrator import build_service
    from distributed_llm_pipeline_b200.serving.sampler import SamplingParams
    from distributed_llm_pipeline_b200.serving.scheduler import Request
    cfg, _, path = models["odd"]
    sched, _, _ = build_service(path, "cuda:0", n_ctx=256, n_slots=3, n_batch=32, page_size=16, dtype="f32")
    p = SamplingParams(temperature=0.9, top_k=20, seed=11)
    a = sched.generate(lm.tokens(cfg, 20), n_predict=16, sampling=p)
    reqs = [sched.submit(Request(prompt=lm.tokens(cfg, 20), n_predict=16, sampling=p, cache_prompt=False))]
    reqs += [sched.submit(Request(prompt=lm.tokens(cfg, n, seed=n), n_predict=9, sampling=SamplingParams(temperature=0.0))) for n in (90, 70)]
    while not all(r.done.is_set() for r in reqs):
        sched.step()
    assert reqs[0].output_ids == a.output_ids


def test_state_copy_session_and_rollback(models, tmp_path):
    from distributed_llm_pipeline_b200.utils.session import load_sequence, save_sequence
    cfg, w, path = models["odd"]
    eng = engine(path, "f32")
    ids = lm.tokens(cfg, 90)
    want, _ = plain.forward(cfg, w, ids)
    a, b = eng.alloc_seq(), eng.alloc_seq()
    eng.prefill(a, ids[:80])
    eng.copy_seq(a, b)
    assert lm.error(eng.prefill(b, ids[80:], all_logits=True), want[80:]) < LIMIT["f32"]
    save_sequence(eng, a, str(tmp_path / "s"))
    eng.truncate_seq(a, 0)
    eng.prefill(a, lm.tokens(cfg, 30, seed=7))
    load_sequence(eng, a, str(tmp_path / "s"))
    assert lm.error(torch.stack([eng.decode([a], [t], sample=False)[0].clone() for t in ids[80:]]), want[80:]) < LIMIT["f32"]
    assert eng.memory_breakdown()["recurrent_state"] > 0


def test_residual_after_every_layer(models):
    cfg, w, path = models["wide"]
    ids = lm.tokens(cfg, 50)
    _, after = plain.forward(cfg, w, ids)
    for dtype, tol in (("f32", 2e-5), ("bf16", 3e-2)):
        eng, got = engine(path, dtype), {}
        eng.eval_callback = lambda n, il, h: got.__setitem__(il, h.double().cpu())
        eng.prefill(eng.alloc_seq(), ids)
        assert all(rel(got[i], after[i]) < tol for i in range(len(after)))


def test_trace_run_program(models, tmp_path):
    import json
    import os
    import subprocess
    import sys
    cfg, w, path = models["odd"]
    ids, exe = lm.tokens(cfg, 70), os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "bin", "trace_run")
    want = plain.forward(cfg, w, ids)[0]
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": ids[:40], "want": [0, 39]}, {"id": "b", "tokens": ids[:3], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": ids[3:4], "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "c", "tokens": ids[:1], "want": [0]}, {"id": "a", "tokens": ids[40:], "want": [29]}], "end": ["a", "c"]}]
    for dtype, lim in (("bfloat16", LIMIT["bf16"]), ("float32", LIMIT["f32"])):
        r = subprocess.run([sys.executable, exe, "--model", path, "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "192"],
                           input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
        assert r.returncode == 0 and [x for x in r.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"], r.stderr
        for n, rows in ((0, [0, 39]), (2, [0, 69])):
            got = torch.frombuffer(bytearray((tmp_path / f"{n}.f32").read_bytes()), dtype=torch.float32).view(2, -1)
            assert lm.error(got, want[rows]) < lim
        assert not (tmp_path / "1.f32").exists()


def test_command_line(models):
    import os
    import subprocess
    import sys
    cfg, w, path = models["odd"]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    ids = lm.tokens(cfg, 12)
    r = subprocess.run([sys.executable, os.path.join(root, "tools", "dlp_cli.py"), "-m", path, "--dtype", "f32", "-p", " ".join(map(str, ids)), "-n", "6", "--temp", "0",
                        "-c", "128", "-no-cnv"], capture_output=True, text=True, timeout=300, stdin=subprocess.DEVNULL)
    out = [int(x) for x in r.stdout.split()]
    assert r.returncode == 0, r.stderr
    out = out[-6:]
    lg = plain.forward(cfg, w, ids + out)[0]
    assert all(lg[len(ids) - 1 + i].max() - lg[len(ids) - 1 + i][t] < 1e-3 for i, t in enumerate(out))
