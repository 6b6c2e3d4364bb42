"""Mubutar on a machine without a GPU: configuration, plan, loader, cache entries and the engine's host side (step
function, pages, scheduler) over the plain kernel statements of tests/kernel_refs.py, against the plain implementation of
tests/plain_mubutar.py.  The CUDA kernels themselves are the business of test_mubutar_gpu.py."""
import copy

import pytest
import torch

import plain_mubutar as P
import tiny
import tiny_mubutar as TM
from kernel_refs import ReferenceKernels
from infurnace_b200.cache import CacheLayout
from infurnace_b200.config.specs import (
    DenseMLPSpec, GatedMLPSpec, KVCacheNeed, LayerCall, ParallelBlockSpec, PreNormBlockSpec, RMSNormSpec, RotaryValueAttentionSpec,
    RoutedExpertsSpec,
)
from infurnace_b200.engine import Engine, EngineOptions, SamplingParams
from infurnace_b200.errors import ModelConfigError, WeightError
from infurnace_b200.models import config_from_dict, plan_for

TOL = 2e-5      # float32 stream and buffers against the float64 oracle


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    root = str(tmp_path_factory.mktemp("mubutar"))
    return {n: TM.make_model_dir(n, root) for n in ("M1", "M2")}


def engine(model_dir, page_size, pool=320, kernels=None, **kw):
    opts = dict(dtype="float32", device="cpu", page_size=page_size, num_pages=pool // page_size, max_num_seqs=4,
                max_num_batched_tokens=pool)
    opts.update(kw)
    return Engine.from_model_dir(model_dir, EngineOptions(**opts), kernels=kernels or ReferenceKernels(torch.float64))


def tolerance(ref):
    return TOL * max(1.0, float(ref.abs().max()))


# ------------------------------------------------------------------------------ each mechanism of the oracle alone
def test_the_oracles_mechanisms_alone():
    f64 = torch.float64
    # the sink stands beside the keys: n equal scores of 0 get 1 / (n + 1) each; far below 0 nothing is left for the keys
    assert torch.allclose(P.attention_weights(torch.zeros(3, dtype=f64)), torch.full((3,), 0.25, dtype=f64))
    assert float(P.attention_weights(torch.full((3,), -40.0, dtype=f64)).sum()) < 1e-15
    assert torch.allclose(P.attention_weights(torch.tensor([500.0, 0.0], dtype=f64)), torch.tensor([1.0, 0.0], dtype=f64))
    # the cap bounds a score and leaves small ones alone
    assert float(P.capped(torch.tensor(1000.0, dtype=f64), 5.0)) == pytest.approx(5.0)
    assert float(P.capped(torch.tensor(0.01, dtype=f64), 5.0)) == pytest.approx(0.01, rel=1e-5)
    assert float(P.capped(torch.tensor(7.0, dtype=f64), None)) == 7.0
    # causal, two query heads per key head, values of their own width
    q, k = torch.zeros(3, 4, 2, dtype=f64), torch.zeros(3, 2, 2, dtype=f64)
    v = torch.arange(6, dtype=f64).view(3, 2, 1)
    out = P.sink_attention(q, k, v, 1.0, None)
    assert torch.allclose(out[:, 0, 0], torch.tensor([0.0, 2.0 / 3, 6.0 / 4], dtype=f64)) and torch.equal(out[:, 0], out[:, 1])
    assert torch.allclose(out[:, 3, 0], torch.tensor([0.5, 4.0 / 3, 9.0 / 4], dtype=f64))
    # the squares
    assert P.squared_relu(torch.tensor([-2.0, 3.0], dtype=f64)).tolist() == [0.0, 9.0]
    # the router: the correction chooses and does not weigh; the weights sum to one
    z = torch.tensor([[2.0, 1.0, 0.0, -1.0]], dtype=f64)
    s = torch.sigmoid(z[0])
    idx, w = P.route(z, torch.tensor([-1.0, 0.0, 0.0, 0.5], dtype=f64), 2, None)
    assert idx.tolist() == [[3, 1]] and torch.allclose(w[0], torch.stack((s[3], s[1])) / (s[3] + s[1]))
    # a group counts by the sum of its two best: the group of the single best expert loses
    z = torch.tensor([[4.0, -4.0, -4.0, 1.0, 1.0, -4.0]], dtype=f64)
    assert P.route(z, torch.zeros(6, dtype=f64), 2, (2, 1))[0].tolist() == [[3, 4]]
    # nothing of the other groups is ever chosen, also where every score left is below zero
    assert set(P.route(z, torch.full((6,), -3.0, dtype=f64), 3, (2, 1))[0][0].tolist()) == {3, 4, 5}
    # a group of one expert counts by it; the lower index wins among equals
    assert P.route(torch.zeros(1, 4, dtype=f64), torch.zeros(4, dtype=f64), 2, (4, 2))[0].tolist() == [[0, 1]]


# ------------------------------------------------------------------------------ configuration, plan, weights
def test_configuration_round_trip_and_plan():
    for name, spec in TM.TINY.items():
        conf = spec["config"]
        cfg = config_from_dict(conf)
        assert cfg.to_dict() == conf, name
        plan = plan_for(cfg)
        made = TM.make_weights(conf, 0)
        assert set(plan.tensors()) == set(made), name
        for tname, t in made.items():
            assert tuple(plan.tensors()[tname].shape) == tuple(t.shape), tname
        assert not plan.lm_head.tied and plan.lm_head.scale == conf.get("logit_scale", 1.0)
        assert plan.embedding.scale == conf.get("embedding", {}).get("scale", 1.0)
        for i, (block, call, entry) in enumerate(zip(plan.layers, plan.resolved_schedule(), conf["layers"])):
            assert isinstance(block, ParallelBlockSpec) and isinstance(block.mixer, RotaryValueAttentionSpec)
            m, a = entry["mixer"], block.mixer
            assert (a.num_heads, a.num_kv_heads, a.head_dim, a.value_head_dim, a.scale, a.softcap, a.sink_score) == \
                (m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"], m.get("softcap"), 0.0)
            own = "kv_from" not in m
            assert call.layer == i and call.store == own and call.cache == (i if own else m["kv_from"]) and a.reads_cache == (not own)
            assert (a.k_proj is None) == (a.v_bias is None) == (not own)
            mlp = entry["mlp"]
            if mlp is None:
                assert block.ffn is None
            elif mlp["kind"] == "dense":
                assert isinstance(block.ffn, GatedMLPSpec) and block.ffn.intermediate_size == mlp["ff"]
            else:
                f, r = block.ffn, mlp["router"]
                assert isinstance(f, RoutedExpertsSpec) and not f.gated and f.normalise and f.group_best == 2 and f.scoring == "sigmoid"
                assert f.top == r["top"] and len(f.experts) == r["experts"] and f.activation == "relu2"
                assert f.groups == ((r["groups"]["count"], r["groups"]["keep"]) if "groups" in r else None)
                assert isinstance(f.shared, DenseMLPSpec) == ("shared" in mlp)


def test_layers_that_read_another_keep_no_pages():
    conf = TM.TINY["M1"]["config"]
    layout = CacheLayout(plan_for(config_from_dict(conf)))
    assert not layout.state
    ids = sorted(i for need, entries in layout.kv.values() for i in entries)
    assert ids == [0, 2, 5] and all(isinstance(need, KVCacheNeed) and need.window is None for need, _ in layout.kv.values())


def test_configuration_faults_are_named():
    base = TM.TINY["M1"]["config"]

    def broken(edit):
        c = copy.deepcopy(base)
        edit(c)
        with pytest.raises(ModelConfigError) as e:
            config_from_dict(c)
        return str(e.value)

    def mixer(i):
        return lambda c: c["layers"][i]["mixer"]

    assert "type" in broken(lambda c: c["layers"][0].update(type="rglru"))
    assert "vdim" in broken(lambda c: mixer(0)(c).pop("vdim"))
    assert "kv_heads" in broken(lambda c: mixer(0)(c).update(heads=5))
    assert "softcap" in broken(lambda c: mixer(0)(c).update(softcap=0))
    assert "kv_from" in broken(lambda c: mixer(1)(c).update(kv_from=1))
    assert "kv_from" in broken(lambda c: mixer(0)(c).update(kv_from=-1))
    assert "of its own" in broken(lambda c: mixer(3)(c).update(kv_from=1))
    assert "dim" in broken(lambda c: mixer(1)(c).update(dim=16))
    assert "kv_heads" in broken(lambda c: mixer(1)(c).update(kv_heads=3))
    assert "mlp.kind" in broken(lambda c: c["layers"][0]["mlp"].update(kind="conv"))
    assert "mlp.ff" in broken(lambda c: c["layers"][0]["mlp"].pop("ff"))
    assert "groups" in broken(lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=5))
    assert "groups" in broken(lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=5))
    assert "top" in broken(lambda c: c["layers"][1]["mlp"]["router"].update(top=7))
    assert "shared.ff" in broken(lambda c: c["layers"][1]["mlp"].update(shared={}))
    assert "embedding.scale" in broken(lambda c: c.update(embedding={"scale": "3"}))
    assert "logit_scale" in broken(lambda c: c.update(logit_scale="3"))
    assert "layers" in broken(lambda c: c.update(layers=[]))


def test_loader_lists_what_is_wrong(models, tmp_path):
    import os
    import shutil
    from safetensors.torch import load_file, save_file
    d = str(tmp_path / "bad")
    shutil.copytree(models["M1"], d)
    t = load_file(os.path.join(d, "model.safetensors"))
    del t["l0.mix.k.b"]
    t["l1.mix.k"] = torch.zeros(24, 40)              # layer 1 reads layer 0's keys
    t["l1.mlp.e0.gate"] = torch.zeros(20, 40)        # experts have no gate
    t["l2.mlp.up"] = torch.zeros(4, 40)              # layer 2 has no feed-forward
    t["l1.mlp.correction"] = torch.zeros(11)
    save_file(t, os.path.join(d, "model.safetensors"))
    with pytest.raises(WeightError) as e:
        engine(d, 16)
    assert all(name in str(e.value) for name in ("l0.mix.k.b", "l1.mix.k", "l1.mlp.e0.gate", "l2.mlp.up", "l1.mlp.correction"))


# ------------------------------------------------------------------------------ the engine's host side
LENS = [37, 100, 64, 19, 85, 50, 1, 2, 3]


def _requests(vocab, seed=0):
    return {f"r{i}": tiny.random_tokens(vocab, n, seed + i) for i, n in enumerate(LENS)}


@pytest.mark.parametrize("name", ["M1", "M2"])
@pytest.mark.parametrize("mode", ["whole", "bulk_tail", "portions", "mixed"])
def test_cutting_modes_on_the_host_path(models, name, mode):
    cfg, w = TM.load_model_dir(models[name])
    reqs = _requests(cfg["vocab"])
    steps = {"whole": tiny.schedule_whole, "bulk_tail": lambda r: tiny.schedule_bulk_tail(r, tail=40),
             "portions": lambda r: tiny.schedule_portions(r, seed=3),
             "mixed": lambda r: tiny.schedule_mixed(r, max_tokens=320, seed=4)}[mode](reqs)
    eng = engine(models[name], TM.TINY[name]["page_size"])
    out = tiny.collect(steps, tiny.run_inprocess(eng.runner, steps), cfg["vocab"])
    for rid, toks in reqs.items():
        ref = P.forward(cfg, w, toks)
        assert (out[rid] - ref).abs().max() < tolerance(ref), (rid, mode)
    eng.runner.cache.check()
    assert eng.runner.cache.num_free_slots == 4
    assert eng.runner.cache.free_pages() == [g.pool.num_pages for g in eng.runner.cache.kv_groups]


@pytest.mark.parametrize("name", ["M1", "M2"])
def test_the_stream_after_every_layer(models, name):
    """The residual stream after each block is the plain implementation's: what a block hands on (a delta, two deltas side by
    side, a half-done norm over an updated stream) is added up here, nothing is lost or added twice."""
    cfg, w = TM.load_model_dir(models[name])
    toks = tiny.random_tokens(cfg["vocab"], 30, 5)
    _, layers = P.forward(cfg, w, toks, return_layers=True)
    for fold in (True, False):
        eng = engine(models[name], TM.TINY[name]["page_size"], kernels=ReferenceKernels(torch.float64, fold=fold))
        seen = []
        for layer in eng.runner.model.layers:
            inner = layer.forward

            def spy(x, pending, ctx, call, next_layer=None, inner=inner):
                out = inner(x, pending, ctx, call, next_layer=next_layer)
                now = x[:len(toks)].clone()
                if torch.is_tensor(out):
                    now += out if out.dim() == 2 else out.sum(0)
                seen.append(now)
                return out
            layer.forward = spy
        tiny.run_inprocess(eng.runner, tiny.schedule_whole({"a": toks}))
        assert len(seen) == len(cfg["layers"])
        for i, got in enumerate(seen):
            assert (got.double() - layers[i]).abs().max() < tolerance(layers[i]), (fold, i)


def test_the_oracle_would_show_a_lost_mechanism(models):
    """The tiny model is made so that these faults move the logits by far more than the tolerance."""
    cfg, w = TM.load_model_dir(models["M1"])
    toks = tiny.random_tokens(cfg["vocab"], 60, 9)
    ref = P.forward(cfg, w, toks)

    def moved(cfg2=None, **tensors):
        w2 = dict(w)
        w2.update(tensors)
        return float((P.forward(cfg2 or cfg, w2, toks) - ref).abs().max()) > 1000 * tolerance(ref)

    def edited(edit):
        other = copy.deepcopy(cfg)
        edit(other)
        return other

    def swapped(name, function):
        inner = getattr(P, name)
        setattr(P, name, function)
        try:
            return float((P.forward(cfg, w, toks) - ref).abs().max()) > 1000 * tolerance(ref)
        finally:
            setattr(P, name, inner)

    for i in range(6):
        assert moved(edited(lambda c: c["layers"][i]["mixer"].update(softcap=c["layers"][i]["mixer"]["softcap"] * 2.0))), i
        assert moved(edited(lambda c: c["layers"][i]["mixer"].update(scale=c["layers"][i]["mixer"]["scale"] * 1.5))), i
        assert moved(**{f"l{i}.mix.q.b": torch.zeros_like(w[f"l{i}.mix.q.b"])}), i
    for i in (0, 2, 5):
        assert moved(**{f"l{i}.mix.k.b": torch.zeros_like(w[f"l{i}.mix.k.b"])}), i
        assert moved(**{f"l{i}.mix.v.b": torch.zeros_like(w[f"l{i}.mix.v.b"])}), i
    assert moved(edited(lambda c: c["norm"].update(eps=1e-2)))
    assert moved(edited(lambda c: c.update(logit_scale=1.0)))
    assert moved(edited(lambda c: c["embedding"].update(scale=2.9)))
    assert moved(edited(lambda c: c["layers"][1]["mlp"]["router"].update(top=2)))
    assert moved(edited(lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=3)))
    assert moved(edited(lambda c: c["layers"][5]["mlp"]["router"]["groups"].update(keep=2)))
    assert moved(edited(lambda c: c["layers"][1]["mlp"].pop("shared")))
    for i in (1, 3, 4, 5):
        assert moved(**{f"l{i}.mlp.correction": torch.zeros_like(w[f"l{i}.mlp.correction"])}), i
    assert swapped("attention_weights", lambda s: torch.softmax(s, dim=-1))                          # the sink left out
    assert swapped("squared_relu", lambda z: z.clamp(min=0.0))
    assert swapped("silu", lambda z: z.clamp(min=0.0))
    route = P.route

    def weighs_with_correction(z, correction, top, groups):
        chosen, _ = route(z, correction, top, groups)
        s = torch.gather(torch.sigmoid(z) + correction, 1, chosen)
        return chosen, s / (s.sum(-1, keepdim=True) + 1e-20)
    assert swapped("route", weighs_with_correction)
    assert swapped("route", lambda z, c, top, groups: (route(z, c, top, groups)[0], torch.gather(torch.sigmoid(z), 1, route(z, c, top, groups)[0])))

    def masked_with_zero(z, correction, top, groups):
        if groups is None:
            return route(z, correction, top, groups)
        c = torch.sigmoid(z) + correction
        per = c.view(c.shape[0], groups[0], -1)
        score = per.sort(dim=-1, descending=True).values[..., :2].sum(-1)
        kept = score.sort(dim=-1, descending=True, stable=True).indices[:, :groups[1]]
        mask = torch.zeros(score.shape, dtype=torch.bool).scatter_(1, kept, True)
        c = torch.where(mask[:, :, None].expand_as(per).reshape(c.shape), c, torch.zeros_like(c))
        chosen = c.sort(dim=-1, descending=True, stable=True).indices[:, :top]
        s = torch.gather(torch.sigmoid(z), 1, chosen)
        return chosen, s / s.sum(-1, keepdim=True)
    assert swapped("route", masked_with_zero)
    # keys and values: each reading layer takes the layer it names
    inner_kv = P.keys_and_values
    held = {}

    def other_layers(h, weights, p, m):
        held[p] = inner_kv(h, weights, p, m)
        return tuple(t.flip(0) for t in held[p]) if p == "l2.mix." else held[p]
    assert swapped("keys_and_values", other_layers)


def test_prefill_equals_token_by_token_decoding(models):
    for name in ("M1", "M2"):
        cfg, w = TM.load_model_dir(models[name])
        toks = tiny.random_tokens(cfg["vocab"], 75, 21)
        ref = P.forward(cfg, w, toks)
        steps = [{"step": i, "entries": [{"id": "x", "tokens": [t], "want": [0]}], "end": []} for i, t in enumerate(toks)]
        eng = engine(models[name], TM.TINY[name]["page_size"])
        out = tiny.collect(steps, tiny.run_inprocess(eng.runner, steps), cfg["vocab"])["x"]
        assert (out - ref).abs().max() < tolerance(ref), name


@pytest.mark.parametrize("pattern", [[2] * 40, [3, 2, 5, 2, 2, 7, 1, 1, 2, 30, 2, 23], [1, 79], [78, 2], [6] * 13 + [2]])
def test_portions_down_to_two_tokens(models, pattern):
    cfg, w = TM.load_model_dir(models["M1"])
    toks = tiny.random_tokens(cfg["vocab"], sum(pattern), 31)
    ref = P.forward(cfg, w, toks)
    steps, at = [], 0
    for i, n in enumerate(pattern):
        steps.append({"step": i, "entries": [{"id": "x", "tokens": toks[at:at + n], "want": list(range(n))}], "end": []})
        at += n
    eng = engine(models["M1"], 16)
    out = tiny.collect(steps, tiny.run_inprocess(eng.runner, steps), cfg["vocab"])["x"]
    assert (out - ref).abs().max() < tolerance(ref)


VARIANTS = {
    # one layer; one head; an expert that every token takes
    "attention_only": TM.config(30, 16, 1e-5, [TM.layer(1, 1, 5, 3, 0.7, 1.5, None)], logit=4.0),
    "one_expert": TM.config(41, 24, 1e-6, [TM.layer(2, 1, 7, 9, 0.5, 2.0, TM.moe(1, 1, 8, groups=(1, 1), shared=4))], emb=0.5),
    # every layer after the first reads it; dense feed-forwards throughout
    "one_cache": TM.config(33, 16, 1e-5, [TM.layer(4, 2, 6, 4, 0.5, 2.0, TM.dense(20))] + [
        TM.layer(4, 2, 6, 4, 0.4 + 0.1 * i, 2.0 + i, TM.dense(12 + 4 * i), kv_from=0) for i in range(3)], emb=2.0),
    # mixtures one after the other, then a layer without feed-forward, then a dense one
    "order": TM.config(64, 40, 1e-5, [
        TM.layer(5, 5, 8, 4, 0.4, 3.0, TM.moe(16, 5, 8, groups=(8, 4), shared=12)),
        TM.layer(5, 1, 4, 8, 0.6, 2.0, TM.moe(9, 3, 12, groups=(3, 1))), TM.layer(5, 1, 4, 8, 0.5, 3.0, None, kv_from=1),
        TM.layer(10, 5, 8, 4, 0.5, 4.0, TM.dense(30), kv_from=0), TM.layer(2, 2, 3, 5, 0.8, None, TM.moe(2, 1, 6))], logit=0.3),
}


@pytest.mark.parametrize("name", list(VARIANTS))
def test_other_arrangements_of_the_layers(tmp_path, name):
    """Values that make mechanisms coincide or vanish, other sizes and orders, in a mixed schedule over a small pool, and
    greedy generation through the scheduler."""
    conf = VARIANTS[name]
    d = TM.make_model_dir("_" + name, str(tmp_path), config=conf, seed=3, store="float32")
    cfg, w = TM.load_model_dir(d)
    V = conf["vocab"]
    reqs = {f"r{i}": tiny.random_tokens(V, n, i) for i, n in enumerate([20, 1, 33, 7, 2, 15, 70])}
    steps = tiny.schedule_mixed(reqs, max_tokens=192, seed=1)
    eng = engine(d, 4, pool=192)
    out = tiny.collect(steps, tiny.run_inprocess(eng.runner, steps), V)
    for rid, toks in reqs.items():
        ref = P.forward(cfg, w, toks)
        assert (out[rid] - ref).abs().max() < tolerance(ref), rid
    prompt = tiny.random_tokens(V, 5, 9)
    assert eng.generate([prompt], SamplingParams(max_tokens=6)) == [P.greedy(cfg, w, prompt, 6)]


def test_a_parallel_block_beside_blocks_of_other_kinds(models, tmp_path):
    """The block's two deltas side by side go to a block of another kind as well (here: a pre-norm block after it), and a design
    of blocks of both kinds runs; a final norm that cannot take the logits' scale leaves it to the head."""
    from infurnace_b200.config.specs import EmbeddingSpec, GroupRMSNormSpec, LMHeadSpec, ModelPlan
    from infurnace_b200.parts import DecoderModel, Runtime
    from infurnace_b200.cache import CacheManager
    from infurnace_b200.engine.runner import ModelRunner
    W, V, eps = 24, 50, 1e-5
    g = torch.Generator().manual_seed(4)

    def att(p, **kw):
        return RotaryValueAttentionSpec(W, 2, 1, 6, 4, 0.5, eps, p + "q", p + "k", p + "v", p + "o", **kw)

    def mlp(p):
        return GatedMLPSpec(W, 20, "silu", p + "g", p + "u", p + "d")
    layers = (ParallelBlockSpec(RMSNormSpec(W, eps, "n0"), att("a0", softcap=2.0, sink_score=0.7), mlp("m0")),
              PreNormBlockSpec(RMSNormSpec(W, eps, "n1"), att("a1"), RMSNormSpec(W, eps, "n1b"), mlp("m1")),
              ParallelBlockSpec(RMSNormSpec(W, eps, "n2"), att("a2", q_bias="a2b"), mlp("m2")))
    plan = ModelPlan("both", V, W, 64, EmbeddingSpec(V, W, "e", scale=2.0), layers, tuple(LayerCall(i) for i in range(3)),
                     GroupRMSNormSpec(W, eps, 2, "fn"), LMHeadSpec(V, W, "h", tied=False, scale=3.0))
    w = {n: torch.randn(t.shape, generator=g) * (0.3 if len(t.shape) > 1 else 0.1) + (1.0 if n[0] in "nf" else 0.0)
         for n, t in plan.tensors().items()}
    ids = tiny.random_tokens(V, 12, 2)

    def norm(v, name, groups=1):
        p = v.view(v.shape[0], groups, -1)
        return (p / torch.sqrt(p.pow(2).mean(-1, keepdim=True) + eps)).reshape(v.shape) * w[name].double()

    def attend(h, p, bias=None, cap=None, sink=None):
        q, k, v = (h @ w[p + c].double().T for c in "qkv")
        q = q + (w[bias].double() if bias else 0.0)
        T = h.shape[0]
        out = torch.zeros(T, 2, 4, dtype=torch.float64)
        for i in range(T):
            s = P.capped(torch.einsum("hd,jd->hj", q[i].view(2, 6), k[:i + 1]) * 0.5, cap)
            e = torch.exp(s)
            out[i] = (e / (e.sum(-1, keepdim=True) + (torch.exp(torch.tensor(sink)) if sink is not None else 0.0))) @ v[:i + 1]
        return out.reshape(T, 8) @ w[p + "o"].double().T

    def ff(h, p):
        return (P.silu(h @ w[p + "g"].double().T) * (h @ w[p + "u"].double().T)) @ w[p + "d"].double().T
    x = w["e"].double()[torch.tensor(ids)] * 2.0
    h = norm(x, "n0")
    x = x + attend(h, "a0", cap=2.0, sink=0.7) + ff(h, "m0")
    x = x + attend(norm(x, "n1"), "a1")
    x = x + ff(norm(x, "n1b"), "m1")
    h = norm(x, "n2")
    x = x + attend(h, "a2", bias="a2b") + ff(h, "m2")
    want = 3.0 * norm(x, "fn", groups=2) @ w["h"].double().T
    for fold in (True, False):
        rt = Runtime(torch.device("cpu"), torch.float32, ReferenceKernels(torch.float64, fold=fold))
        cache = CacheManager(plan, page_size=4, num_pages=8, max_requests=2, dtype=torch.float32, device="cpu")
        runner = ModelRunner(DecoderModel(plan, w, rt), cache, rt, 32, 32)
        steps = tiny.schedule_portions({"a": ids}, seed=1)
        out = tiny.collect(steps, tiny.run_inprocess(runner, steps), V)["a"]
        assert (out - want).abs().max() < tolerance(want), fold


def test_greedy_generation_through_the_scheduler(models):
    cfg, w = TM.load_model_dir(models["M1"])
    eng = engine(models["M1"], 16, max_num_batched_tokens=24)          # prompts go in as portions beside decoded tokens
    prompts = [tiny.random_tokens(cfg["vocab"], n, 40 + n) for n in (1, 9, 33, 70, 5, 18)]      # six requests, four slots
    outs = eng.generate(prompts, SamplingParams(max_tokens=12))
    for p, o in zip(prompts, outs):
        assert o == P.greedy(cfg, w, p, 12)
    eng.runner.cache.check()
    assert eng.runner.cache.num_free_slots == 4
