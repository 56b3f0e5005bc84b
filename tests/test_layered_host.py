"""Layer-list models without a GPU: configuration and weight reading, page and state-slot bookkeeping, batching, scheduler, command line.

The kernels are replaced by plain host code (tests/layer_models.py); what is tested is everything around them."""
import json
import os
import subprocess
import sys

import pytest
import torch

import layer_models as lm
import plain_layers as plain
from distributed_llm_pipeline_b200.models.modeldir import SafetensorsFile, is_model_dir, make_engine, open_model, open_model_dir, write_safetensors
from distributed_llm_pipeline_b200.models.weights import LoadCancelled, load_weights
from distributed_llm_pipeline_b200.serving.sampler import SamplingParams
from distributed_llm_pipeline_b200.serving.scheduler import Request, Scheduler
from distributed_llm_pipeline_b200.serving.trace_runner import TraceRunner
from distributed_llm_pipeline_b200.utils.tokenizer import IdTokenizer, tokenizer_for

TOL = 2e-5


@pytest.fixture(autouse=True)
def few_threads():
    """The tensors are tiny: more threads only wait for one another."""
    n = torch.get_num_threads()
    torch.set_num_threads(min(n, 2))
    yield
    torch.set_num_threads(n)


@pytest.fixture
def model(tmp_path, monkeypatch):
    lm.install_host_ops(monkeypatch)

    def make(name="odd", n_seqs=4, **kw):
        cfg = lm.CONFIGS[name]
        w = lm.weights(cfg, seed=len(name))
        path = lm.write(str(tmp_path / name), cfg, w)
        kw = {"n_ctx": 128, "max_seqs": n_seqs, "page_size": 16, "max_batch_tokens": 64, **kw}
        return cfg, w, make_engine(load_weights(path, "cpu", dtype="f32"), **kw), path
    return make


def test_safetensors_round_trip_and_damage(tmp_path):
    t = {"a": torch.arange(6, dtype=torch.float32).view(2, 3), "b": torch.randn(5).to(torch.bfloat16), "e": torch.zeros(0, 4), "i": torch.tensor([7], dtype=torch.int32)}
    p = write_safetensors(str(tmp_path / "x.safetensors"), t)
    f = SafetensorsFile(p)
    for k, v in t.items():
        assert f.tensor(k).dtype == v.dtype and torch.equal(f.tensor(k), v)
    with pytest.raises(KeyError):
        f.tensor("nope")
    raw = open(p, "rb").read()
    open(p, "wb").write(raw[:-4])
    with pytest.raises(ValueError):
        SafetensorsFile(p)


def test_config_is_checked(tmp_path):
    cfg = lm.CONFIGS["odd"]
    p = lm.write(str(tmp_path / "m"), cfg, lm.weights(cfg))
    assert is_model_dir(p) and open_model(p).cfg.n_layer == 4
    d = open_model_dir(p).cfg
    assert (d.n_embd, d.vocab_size, d.norm_groups, d.rms_eps) == (72, 101, 3, 3e-4)
    assert d.n_params() == sum(t.numel() for t in lm.weights(cfg).values())
    for change in ({"architecture": "Other"}, {"layers": [{"type": "mamba", "mixer": {}, "mlp": None}]}, {"norm": {"groups": 5, "eps": 1e-5}},
                   {"layers": [lm.hgrn2(1, 8, 8) | {"mlp": {"kind": "moe", "ff": 3}}]}, {"layers": [{"type": "hgrn2", "mixer": {"heads": 1, "dim": 8}, "mlp": None}]}):
        json.dump({**cfg, **change}, open(os.path.join(p, "config.json"), "w"))
        with pytest.raises(ValueError):
            open_model_dir(p)


def test_windowed_config_is_checked(tmp_path):
    cfg = lm.CONFIGS["experts"]
    p = lm.write(str(tmp_path / "m"), cfg, lm.weights(cfg))
    d = open_model_dir(p).cfg
    assert (d.n_layer, d.norm_type, d.loop, d.rms_eps) == (4, "layer", (1, 3, 2), 3e-4)
    assert d.layer_runs() == [(0, False), (1, False), (2, False), (1, True), (2, False), (3, False)] == plain.layer_runs(cfg)
    assert d.n_params() == sum(t.numel() for t in lm.weights(cfg).values())
    no_loop = {k: v for k, v in cfg.items() if k != "loop"}
    for c, want in (({**cfg, "loop": {"start": 0, "stop": 4, "times": 3}}, [(i, r > 0 and i == 0) for r in range(3) for i in range(4)]), (no_loop, [(i, False) for i in range(4)]),
                    ({**cfg, "loop": {"start": 3, "stop": 4, "times": 1}}, [(i, False) for i in range(4)])):
        json.dump(c, open(os.path.join(p, "config.json"), "w"))
        assert open_model_dir(p).cfg.layer_runs() == want == plain.layer_runs(c)
    a = lm.attention
    for bad in (a(6, 4, 8, 8, 0.3, 8, 4, 0), a(2, 2, 8, 8, 0.3, 10, 4, 0), a(2, 2, 8, 8, 0.3, 3, 4, 0), a(2, 2, 8, 8, 0.3, 8, 0, 0), a(2, 2, 8, 8, 0.3, 8, 4, -1), a(2, 2, 8, 8, "1", 8, 4, 0),
                a(2, 2, 8, 8, 0.3, 8, 4, 0, 3, 4, 8), a(2, 2, 8, 8, 0.3, 8, 4, 0, 3, 2, 0)):
        json.dump({**no_loop, "layers": [bad]}, open(os.path.join(p, "config.json"), "w"))
        with pytest.raises(ValueError):
            open_model_dir(p)
    for loop in ((2, 2, 1), (0, 5, 2), (0, 2, 0), (-1, 2, 2), (0, 2, None)):
        json.dump({**cfg, "loop": dict(zip(("start", "stop", "times"), loop))}, open(os.path.join(p, "config.json"), "w"))
        with pytest.raises(ValueError):
            open_model_dir(p)


def test_hybrid_config_is_checked(tmp_path):
    cfg = lm.CONFIGS["hybrid"]
    p = lm.write(str(tmp_path / "m"), cfg, lm.weights(cfg))
    d = open_model_dir(p).cfg
    assert (d.n_layer, d.norm_type, d.loop, d.rms_eps, d.norm_offset, d.embedding_scale, d.logit_scale) == (4, "rms", (1, 3, 2), 3e-4, 1.0, 3.0, 2.0)
    assert d.layer_runs() == [(0, False), (1, False), (2, False), (1, False), (2, False), (3, False)] == plain.layer_runs(cfg)
    for name in ("hybrid", "scalar", "maps", "states"):
        c = lm.CONFIGS[name]
        assert open_model_dir(lm.write(str(tmp_path / name), c, lm.weights(c))).cfg.n_params() == sum(t.numel() for t in lm.weights(c).values())
    li, ma, di, moe = lm.lightning, lm.mamba2, lm.differential, lm.shared_moe
    for bad in (li(2, 8, 8, [0.5]), li(2, 8, 8, [0.5, 1.5]), li(2, 8, 0), ma(4, 8, 8, 3, 4, 2), ma(4, 8, 8, 2, 4, 5), ma(4, 8, 8, 2, 33, 2), ma(4, 8, 8, 2, 0, 2), di(6, 4, 8, 8, 0.3, 8, 4, 0.5),
                di(2, 2, 8, 8, 0.3, 10, 4, 0.5), di(2, 2, 8, 8, 0.3, 8, 0, 0.5), di(2, 2, 8, 8, 0.3, 8, 4, None), di(2, 2, 8, 8, 0.3, 8, 4, 0.5, scaling=(8.0, 4.0, 4.0, 64)),
                di(2, 2, 8, 8, 0.3, 8, 4, 0.5, scaling=(8.0, 1.0, 4.0)), li(2, 8, 8, mlp=moe(8, 2, 8, 8, 3, 1)), li(2, 8, 8, mlp=moe(8, 2, 8, 8, 4, 5)), li(2, 8, 8, mlp=moe(8, 5, 8, 8, 4, 2)),
                li(2, 8, 8, mlp=moe(8, 2, 8, 0)), li(2, 8, 8, mlp=lm.dense(0)), {**li(2, 8, 8), "type": "hgrn2"}):
        json.dump({**cfg, "loop": None, "layers": [bad]}, open(os.path.join(p, "config.json"), "w"))
        with pytest.raises(ValueError):
            open_model_dir(p)
    for change in ({"logit_scale": 0}, {"embedding": {"scale": "1"}}, {"loop": {"start": 2, "stop": 2, "times": 1}}):
        json.dump({**cfg, **change}, open(os.path.join(p, "config.json"), "w"))
        with pytest.raises(ValueError):
            open_model_dir(p)
    w = lm.weights(cfg)
    for name in ("l0.mix.g", "l0.mix.norm", "l0.mix.o", "l0.mlp.down", "l1.mix.in", "l1.mix.conv", "l1.mix.dt_bias", "l1.mix.D", "l1.mlp.shared.down", "l1.mlp.correction", "l1.mlp.e3.gate", "l2.mix.lq2", "l2.mix.k",
                 "l2.mlp.shared.gate", "l2.mlp.router", "final.norm"):
        lm.write(p, cfg, {**w, name: w[name][:-1]})
        with pytest.raises(ValueError):
            load_weights(p, "cpu")


def test_parallel_config_is_checked(tmp_path):
    cfg = lm.CONFIGS["parallel"]
    p = lm.write(str(tmp_path / "m"), cfg, lm.weights(cfg))
    d = open_model_dir(p).cfg
    assert (d.n_layer, d.norm_type, d.rms_eps, d.embedding_scale, d.logit_scale, d.parallel_residual) == (7, "rms", 3e-4, 3.0, 1.0, True)
    assert [s.mixer.get("v_mix") for s in d.layers if s.type == "attention"] == [False, "first", "later"]
    for name in ("parallel", "deltas", "windows"):
        c = lm.CONFIGS[name]
        assert open_model_dir(lm.write(str(tmp_path / name), c, lm.weights(c))).cfg.n_params() == sum(t.numel() for t in lm.weights(c).values())
    de, at, la = lm.delta, lm.biased_attention, lm.low_rank_latent
    for bad in ([de(4, 3, 8, 8, 3)], [de(4, 2, 8, 8, 33)], [de(4, 2, 8, 8, 0)], [at(6, 4, 8, 8, 0.3, 8, 4)], [at(2, 2, 8, 8, 0.3, 10, 4)], [at(2, 2, 8, 8, 0.3, 3, 4)], [at(2, 2, 8, 8, 0.3, 8, 0)], [at(2, 2, 8, 8, "1", 8, 4)],
                [at(2, 2, 8, 8, 0.3, 8, 4, yarn=(8.0, 64, 32.0))], [at(2, 2, 8, 8, 0.3, 8, 4, yarn=(0.0, 64, 32.0, 1.0))], [at(2, 2, 8, 8, 0.3, 8, 4), at(2, 1, 8, 8, 0.3, 8, 4)], [la(2, 8, 3, 8, 8, 8, 0.3, 4)],
                [la(2, 8, 4, 8, 0, 8, 0.3, 4)], [{**la(2, 8, 4, 8, 8, 8, 0.3, 4), "type": "mamba2"}], [de(2, 2, 8, 8, 3, ff=0)], [{**de(2, 2, 8, 8, 3), "mlp": lm.shared_moe(4, 2, 8, 8)}]):
        json.dump({**cfg, "layers": bad}, open(os.path.join(p, "config.json"), "w"))
        with pytest.raises(ValueError):
            open_model_dir(p)
    bad = la(2, 8, 4, 8, 8, 8, 0.3, 4)
    bad["mixer"]["rot"]["dims"] = 2
    json.dump({**cfg, "layers": [bad]}, open(os.path.join(p, "config.json"), "w"))
    with pytest.raises(ValueError):
        open_model_dir(p)
    w = lm.weights(cfg)
    for name in ("l0.mix.q.b", "l0.mix.o", "l0.mlp.act", "l0.mlp.down", "l1.mix.dq", "l1.mix.dq.norm", "l1.mix.uq", "l1.mix.dkv", "l1.mix.dkv.norm", "l1.mlp.up", "l2.mix.g", "l2.mix.k.conv", "l2.mix.a", "l2.mix.dt_bias",
                 "l2.mix.A_log", "l2.mix.norm", "l2.norm1", "l5.mix.v.b", "final.norm"):
        lm.write(p, cfg, {**w, name: w[name][:-1]})
        with pytest.raises(ValueError):
            load_weights(p, "cpu")


def test_joined_products_are_stacked_once(tmp_path):
    """Mixer and feed-forward share their matrices' memory; a layer without a feed-forward keeps its own."""
    cfg = lm.CONFIGS["parallel"]
    w = load_weights(lm.write(str(tmp_path / "m"), cfg, lm.weights(cfg)), "cpu", dtype="f32")
    for i, s in enumerate(cfg["layers"]):
        lw = w.layers[i]
        assert (lw.joined is not None) == (s["mlp"] is not None) and lw.mlp is None and lw.norm2 is None
        if lw.joined is not None:
            assert lw.joined.w_in is lw.mixer.w_in and lw.joined.w_out is lw.mixer.w_out and lw.proj_cols % 32 == 0
            assert lw.mixer.w_in.N == lw.proj_cols + s["mlp"]["ff"] and lw.mixer.w_out.K >= s["mlp"]["ff"] + s["mixer"]["heads"] * s["mixer"]["vdim"]


def test_loading_checks_shapes_and_can_be_cancelled(tmp_path):
    cfg = lm.CONFIGS["odd"]
    w = lm.weights(cfg)
    p = lm.write(str(tmp_path / "m"), cfg, w)
    with pytest.raises(LoadCancelled):
        load_weights(p, "cpu", progress=lambda f: f < 0.5)
    with pytest.raises(NotImplementedError):
        load_weights(p, "cpu", tp_size=2)
    lm.write(p, cfg, {**w, "l1.mix.lower": w["l1.mix.lower"][:-1]})
    with pytest.raises(ValueError):
        load_weights(p, "cpu")
    cfg = lm.CONFIGS["experts"]
    w = lm.weights(cfg)
    for name in ("l0.mix.k", "l0.mix.q.norm", "l0.mix.o", "l0.norm1.b", "l2.mlp.e4.down", "l2.mlp.router", "l2.mlp.router.b", "final.norm.b"):
        lm.write(p, cfg, {**w, name: w[name][:-1]})
        with pytest.raises(ValueError):
            load_weights(p, "cpu")


@pytest.mark.parametrize("name", list(lm.CONFIGS))
def test_prompt_portions_and_single_tokens(model, name):
    cfg, w, eng, _ = model(name)
    ids = lm.tokens(cfg, 41)
    want, _ = plain.forward(cfg, w, ids)
    for cut in ([41], [1] * 41, [2, 3, 16, 1, 1, 18], [15, 1, 1, 15, 9]):
        sid, got, at = eng.alloc_seq(), [], 0
        for n in cut:
            got.append(eng.step([(sid, ids[at:at + n])], [list(range(n))]))
            at += n
        assert lm.error(torch.cat(got), want) < TOL, cut
        eng.free_seq(sid)
    assert len(eng.kv.free) == eng.kv.n_pages


@pytest.mark.parametrize("name", ["odd", "experts", "hybrid", "scalar", "parallel"])
def test_batches_larger_than_the_buffers_and_reuse(model, name):
    cfg, w, eng, _ = model(name, max_batch_tokens=24, n_pages=12)
    run = TraceRunner(eng)
    ids = {k: lm.tokens(cfg, n, seed=n) for k, n in dict(a=70, b=33, c=50, d=5, e=61).items()}
    want = {k: plain.forward(cfg, w, v)[0] for k, v in ids.items()}

    def step(end=(), **parts):
        lg = run.step([{"id": k, "tokens": ids[k][lo:hi], "want": list(range(hi - lo))} for k, (lo, hi) in parts.items()], list(end))
        assert lm.error(lg, torch.cat([want[k][lo:hi] for k, (lo, hi) in parts.items()])) < TOL
    step(a=(0, 40), b=(0, 3))
    step(b=(3, 33), a=(40, 41), d=(0, 5), end=["d"])
    step(a=(41, 42), c=(0, 2))
    step(c=(2, 50), a=(42, 70), end=["a", "b"])
    step(e=(0, 60))
    step(e=(60, 61), end=["c", "e"])
    assert len(eng.kv.free) == 12 and not run.sids


def test_step_refuses_bad_batches(model):
    cfg, w, eng, _ = model("odd", n_pages=3)
    a, b = eng.alloc_seq(), eng.alloc_seq()
    for bad in ([(a, [1]), (a, [2])], [(a, [])]):
        with pytest.raises(ValueError):
            eng.step(bad)
    with pytest.raises(ValueError):
        eng.step([(a, [1, 2])], [[2]])
    with pytest.raises(RuntimeError, match="exhausted"):
        eng.step([(a, [1] * 30), (b, [1] * 30)])
    assert eng.seq_len(a) == 0 and len(eng.kv.free) == 3
    with pytest.raises(RuntimeError, match="n_ctx"):
        eng.step([(a, [1] * 129)])


def test_recurrent_state_is_kept_whole(model):
    cfg, w, eng, _ = model("odd")
    ids = lm.tokens(cfg, 30)
    want, _ = plain.forward(cfg, w, ids)
    a, b = eng.alloc_seq(), eng.alloc_seq()
    eng.prefill(a, ids[:20])
    assert eng.reusable(a, 20) == 20 and eng.reusable(a, 19) == 0 and not eng.can_rollback
    with pytest.raises(RuntimeError, match="recurrent"):
        eng.truncate_seq(a, 10)
    with pytest.raises(NotImplementedError):
        eng.copy_seq(a, b, 10)
    eng.copy_seq(a, b)
    assert lm.error(eng.prefill(b, ids[20:], all_logits=True), want[20:]) < TOL
    assert lm.error(eng.step([(a, ids[20:21])]), want[20:21]) < TOL
    eng.truncate_seq(a, 0)
    assert lm.error(eng.prefill(a, ids, all_logits=True), want) < TOL


@pytest.mark.parametrize("name", ["attention", "experts"])
def test_attention_only_models_can_roll_back(model, name):
    cfg, w, eng, _ = model(name)
    ids = lm.tokens(cfg, 30)
    sid = eng.alloc_seq()
    eng.prefill(sid, ids[:12] + [0, 0, 0])
    assert eng.can_rollback
    eng.truncate_seq(sid, 12)
    assert lm.error(eng.prefill(sid, ids[12:], all_logits=True), plain.forward(cfg, w, ids)[0][12:]) < TOL


@pytest.mark.parametrize("name", ["odd", "experts", "hybrid", "parallel"])
def test_session_file(model, name, tmp_path):
    from distributed_llm_pipeline_b200.utils.session import load_sequence, save_sequence
    cfg, w, eng, _ = model(name)
    ids = lm.tokens(cfg, 40)
    a = eng.alloc_seq()
    eng.prefill(a, ids[:37])
    save_sequence(eng, a, str(tmp_path / "s"), ids[:37])
    eng.free_seq(a)
    x, b = eng.alloc_seq(), eng.alloc_seq()
    eng.prefill(x, lm.tokens(cfg, 20, seed=9))
    assert load_sequence(eng, b, str(tmp_path / "s"))["n_tokens"] == 37
    assert lm.error(eng.prefill(b, ids[37:], all_logits=True), plain.forward(cfg, w, ids)[0][37:]) < TOL
    other = model("recurrent")[2]
    with pytest.raises(ValueError, match="different model"):
        load_sequence(other, other.alloc_seq(), str(tmp_path / "s"))


def test_hooks(model):
    cfg, w, eng, _ = model("odd")
    ids = lm.tokens(cfg, 9)
    want, after = plain.forward(cfg, w, ids)
    got = {}
    eng.eval_callback = lambda name, il, h: got.__setitem__(il, h.clone())
    sid = eng.alloc_seq()
    eng.prefill(sid, ids)
    assert all((got[i].double() - after[i]).abs().max() < 1e-4 for i in range(len(after)))
    eng.eval_callback = None
    v = torch.randn(cfg["width"])
    eng.set_control_vector({3: v}, scale=0.5)
    sid = eng.alloc_seq()
    lg = eng.prefill(sid, ids)
    fin = plain.grouped_norm(after[-1][-1] + 0.5 * v.double(), w["final.norm"].double(), 3, 3e-4) @ w["head"].double().T
    assert lm.error(lg[None], fin[None]) < TOL
    eng.set_control_vector(None)
    e = eng.embed(ids, "none", normalize=False)
    assert torch.allclose(e.double(), plain.grouped_norm(after[-1], w["final.norm"].double(), 3, 3e-4), atol=1e-4)


def test_hooks_between_looped_layers(model):
    """The callback sees every run, and what it settles in front of a new pass does not lose the embedding output."""
    cfg, w, eng, _ = model("experts")
    ids = lm.tokens(cfg, 9)
    want, after = plain.forward(cfg, w, ids)
    for cut in ([9], [5, 1, 3]):
        got, at, sid = {}, 0, eng.alloc_seq()
        eng.eval_callback = lambda name, run, h: got.setdefault(run, []).append(h.clone())
        for n in cut:
            lg = eng.step([(sid, ids[at:at + n])])
            at += n
        assert sorted(got) == list(range(len(after))) and lm.error(lg, want[-1:]) < TOL
        assert all((torch.cat(got[i]).double() - after[i]).abs().max() < 1e-4 for i in got)
    eng.eval_callback = None
    e = eng.embed(ids, "last", normalize=False)
    assert torch.allclose(e.double(), plain.layer_norm(after[-1][-1], w["final.norm"].double(), w["final.norm.b"].double(), 3e-4), atol=1e-4)


def check_greedy(cfg, w, prompt, out, min_gap):
    """Every generated token is the plain model's best one given what was generated before it (near ties aside)."""
    ids = list(prompt) + list(out)
    lg = plain.forward(cfg, w, ids)[0]
    for i, t in enumerate(out):
        row = lg[len(prompt) - 1 + i]
        assert row.max() - row[t] < min_gap, i


@pytest.mark.parametrize("name", ["odd", "recurrent", "experts", "hybrid", "parallel"])
def test_scheduler_mixes_prompts_and_decoding(model, name):
    cfg, w, eng, _ = model(name, n_seqs=3)
    sched = Scheduler(eng, IdTokenizer(cfg["vocab"]), n_batch=16, n_slots=3)
    seen = []
    step = eng.step
    eng.step = lambda entries, want=None: (seen.append([len(t) for _, t in entries]), step(entries, want))[1]
    greedy = SamplingParams(temperature=0.0)
    prompts = [lm.tokens(cfg, n, seed=n) for n in (21, 4, 37, 9, 1)]
    reqs = [sched.submit(Request(prompt=p, n_predict=12, sampling=greedy)) for p in prompts]
    while not all(r.done.is_set() for r in reqs):
        assert sched.step()
    for p, r in zip(prompts, reqs):
        assert r.finish_reason == "length" and len(r.output_ids) == 12
        check_greedy(cfg, w, p, r.output_ids, 1e-3)
    assert any(1 in s and max(s) > 1 for s in seen) and max(sum(s) for s in seen) <= 16
    # a continued conversation keeps the cached prefix, an edited one starts over
    ids = prompts[1] + reqs[1].output_ids
    more = sched.generate(ids + [3, 4], n_predict=2, sampling=greedy)
    assert more.n_prompt_cached in (0, len(ids) - 1)
    check_greedy(cfg, w, ids + [3, 4], more.output_ids, 1e-3)
    edited = sched.generate(ids[:-3] + [5], n_predict=2, sampling=greedy)
    assert edited.n_prompt_cached == 0 or not eng.rstate
    check_greedy(cfg, w, ids[:-3] + [5], edited.output_ids, 1e-3)


def test_scheduler_fails_only_the_request_that_does_not_fit(model):
    cfg, w, eng, _ = model("odd", n_seqs=2, n_pages=4)
    sched = Scheduler(eng, IdTokenizer(cfg["vocab"]), n_batch=64, n_slots=2)
    greedy = SamplingParams(temperature=0.0)
    a = sched.submit(Request(prompt=lm.tokens(cfg, 20), n_predict=8, sampling=greedy))
    b = sched.submit(Request(prompt=lm.tokens(cfg, 60), n_predict=8, sampling=greedy))
    while not (a.done.is_set() and b.done.is_set()):
        sched.step()
    assert a.finish_reason == "length" and b.finish_reason == "error"
    check_greedy(cfg, w, lm.tokens(cfg, 20), a.output_ids, 1e-3)


def test_id_tokenizer(model):
    cfg, _, _, path = model("odd")
    tok = tokenizer_for(open_model(path))
    assert tok.encode("3, 17 100") == [3, 17, 100] and tok.decode([3, 17]) == "3 17 "
    with pytest.raises(ValueError):
        tok.encode("101")


def test_trace_runner_needs_a_gpu(tmp_path):
    if torch.cuda.is_available():
        pytest.skip("CUDA device present")
    cfg = lm.CONFIGS["single"]
    p = lm.write(str(tmp_path / "m"), cfg, lm.weights(cfg))
    exe = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "bin", "trace_run")
    r = subprocess.run([sys.executable, exe, "--model", p, "--out", str(tmp_path), "--max-tokens", "64"], input="", capture_output=True, text=True)
    assert r.returncode == 2 and "CUDA" in r.stderr
