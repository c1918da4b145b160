"""Gated layer-list decoders (Sefalorn) on the CPU: configuration, run-time weights, state slots of the backend, registry, and
the plain implementation's own mechanisms (tests/test_gpu_gated*.py compare the engine with it)."""
import json

import pytest
import torch

from conftest import pkg
from gated_cases import CASES, all_chosen, config, light, moe, par, prompt, row_error, weights
from oracle import sefalorn_ref as ref


def test_config_reads_every_size_and_refuses_what_it_does_not_know():
    lay, g = pkg("layered"), pkg("gated")
    cfg = lay.LayeredConfig.from_json(CASES["odd"])
    assert (cfg.vocab_size, cfg.width, cfg.layers, cfg.norm_eps, cfg.logit_scale, cfg.gated) == (211, 204, 4, 1e-5, -1.3, True)
    assert cfg.layer_list[0].mixer == g.LightningSpec(3, 24, 40, (0.5, 0.93, 0.998))
    assert cfg.layer_list[0].mlp == g.MoeSpec(7, 3, 100, 0.6) and cfg.layer_list[1].mlp is None
    assert cfg.layer_list[2].mixer == g.ParallelSpec(g.WindowAttentionSpec(5, 5, 72, 100, 0.09, 16), g.DeltaSpec(4, 2, 48, 24, 3), 1.7, 0.4)
    s = cfg.tensor_shapes()
    assert s["l1.mix.left.k"] == (120, 204) and s["l1.mix.left.v.b"] == (72,) and s["l1.mix.right.v.conv"] == (216, 2)
    assert s["l2.mix.right.q"] == (96, 204) and s["l2.mlp.e4.down"] == (204, 72) and "l2.mlp.e5.down" not in s
    assert "l1.norm2" not in s and "l1.rg2" not in s and s["l0.rg2.b"] == (204,)
    for breakage in (lambda c: c["layers"][0].update(type="other"), lambda c: c["layers"][0]["mlp"].update(kind="dense"),
                     lambda c: c["layers"][0]["mixer"]["decay"].pop(), lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=4),
                     lambda c: c["layers"][1]["mixer"]["right"].update(kv_heads=5), lambda c: c["layers"][0]["mlp"]["router"].update(top=8)):
        bad = json.loads(json.dumps(CASES["odd"]))
        breakage(bad)
        with pytest.raises(ValueError):
            lay.LayeredConfig.from_json(bad)


@pytest.mark.parametrize("name", sorted(CASES))
def test_run_time_weights_compute_the_same_layer(name):
    """The padded, joined form on plain matrix products equals the layer's equations."""
    lay, g = pkg("layered"), pkg("gated")
    raw = CASES[name]
    cfg, t = lay.LayeredConfig.from_json(raw), weights(raw, seed=3)
    gen = torch.Generator().manual_seed(1)
    W = lay.pad_width(cfg.width)
    for i, spec in enumerate(cfg.layer_list):
        f = {k[len(f"l{i}."):]: v for k, v in t.items() if k.startswith(f"l{i}.")}
        w = g.GatedWeights(spec, f, cfg.width, W, 400, "cpu", torch.float32)
        f, m = {k: v.float() for k, v in f.items()}, spec.mixer
        h = torch.randn(5, cfg.width, generator=gen)
        hp = torch.zeros(5, W)
        hp[:, : cfg.width] = h
        y = hp @ w.wproj.T + w.proj_bias
        at = 0

        def take(heads, size, to):
            nonlocal at
            part = y[:, at:at + heads * to].view(5, heads, to)
            at += heads * to
            assert not part[..., size:].any()
            return part[..., :size]

        def same(got, want):
            assert torch.allclose(got.reshape(5, -1), want.reshape(5, -1), atol=1e-4)

        if isinstance(m, g.ParallelSpec):
            a, r = m.left, m.right
            q = take(a.heads, a.dim, w.Dk)
            same(q, h @ f["mix.left.q"].T + f["mix.left.q.b"])
            k = take(a.kv_heads, a.dim, w.Dk)
            same(k, h @ f["mix.left.k"].T + f["mix.left.k.b"])
            same(take(a.kv_heads, a.vdim, w.Dv), h @ f["mix.left.v"].T + f["mix.left.v.b"])
            for n, heads, size, to in (("q", r.kv_heads, r.dim, w.d), ("k", r.kv_heads, r.dim, w.d), ("v", r.heads, r.vdim, w.dv),
                                       ("g", r.heads, r.vdim, w.dv)):
                same(take(heads, size, to), h @ f["mix.right." + n].T)
            same(take(1, cfg.width, W), h @ f["rg1"].T + f["rg1.b"])
            same(take(2, r.heads, r.heads), torch.cat([h @ f["mix.right.b"].T, h @ f["mix.right.a"].T], 1))
            # scores mixed over the heads = mixed queries against the keys of all kv heads, less the table
            per = a.heads // a.kv_heads
            mixed = torch.stack([torch.einsum("hg,mgd->mhd", w.mix[:, c * per:(c + 1) * per], q[:, c * per:(c + 1) * per])
                                 for c in range(a.kv_heads)], 2)
            s = torch.einsum("mhcd,ncd->hmn", mixed, k)
            n = min(a.window, 400)
            bias = w.bias[:, 256:256 + n] / 1.4426950408889634  # kept in log2 units, +inf around it
            assert w.bias.shape[1] % 4 == 0 and bool(w.bias[:, :256].isinf().all()) and bool(w.bias[:, 256 + n:].isinf().all())
            dist = (torch.arange(5)[:, None] - torch.arange(5)[None]).clamp(0, n - 1)
            want = ref.talking_scores(q, k, a.scale, f["mix.left.r1"], f["mix.left.r2"], f["mix.left.talk"])
            seen = ref.window_mask(5, a.window)
            assert torch.allclose((s - bias[:, dist])[:, seen], want[:, seen], atol=2e-4)
            oa, orr = torch.randn(5, a.heads, a.vdim, generator=gen), torch.randn(5, r.heads, r.vdim, generator=gen)
            out = torch.zeros(5, w.out_ld)
            out[:, : a.heads * w.Dv].view(5, a.heads, w.Dv)[..., : a.vdim] = oa * m.left_scale
            out[:, a.heads * w.Dv:w.out_cols].view(5, r.heads, w.dv)[..., : r.vdim] = orr * m.right_scale
            want = m.left_scale * (oa.reshape(5, -1) @ f["mix.left.o"].T + f["mix.left.o.b"]) + m.right_scale * (orr.reshape(5, -1) @ f["mix.right.o"].T)
            got = out @ w.wo.T + w.o_bias
        else:
            for n, size, to in (("q", m.dim, w.d), ("k", m.dim, w.d), ("v", m.vdim, w.dv), ("g", m.vdim, w.dv)):
                same(take(m.heads, size, to), h @ f["mix." + n].T)
            same(take(1, cfg.width, W), h @ f["rg1"].T + f["rg1.b"])
            o = torch.randn(5, m.heads, m.vdim, generator=gen)
            out = torch.zeros(5, w.out_ld)
            out[:, : w.out_cols].view(5, m.heads, w.dv)[..., : m.vdim] = o
            want, got = o.reshape(5, -1) @ f["mix.o"].T, out @ w.wo.T
            assert torch.equal(w.head_norm.view(m.heads, w.dv)[:, : m.vdim].reshape(-1), f["mix.norm"])
        assert at == y.shape[1] and w.out_ld % 64 == 0
        assert torch.allclose(got[:, : cfg.width], want, atol=2e-4) and not got[:, cfg.width:].any()
        if spec.mlp is not None:
            z = hp @ w.w_route.T + w.route_bias
            same(z[:, : cfg.width], h @ f["rg2"].T + f["rg2.b"])
            same(z[:, W:], h @ f["mlp.router"].T)
            for e in (0, spec.mlp.experts - 1):
                gu = (hp @ w.w_gate_up[e].T).view(5, -1, 2, 128)
                a = ref.silu(gu[:, :, 0].reshape(5, -1)) * gu[:, :, 1].reshape(5, -1)
                want = (ref.silu(h @ f[f"mlp.e{e}.gate"].T) * (h @ f[f"mlp.e{e}.up"].T)) @ f[f"mlp.e{e}.down"].T
                out = a @ w.w_down[e].T
                assert torch.allclose(out[:, : cfg.width], want, atol=2e-4) and not out[:, cfg.width:].any()


def test_loading_and_registry(tmp_path, monkeypatch):
    ck, reg, lay = pkg("checkpoint"), pkg("registry"), pkg("layered")
    raw = CASES["plain"]
    t = weights(raw)
    ck.write_safetensors(str(tmp_path / "model.safetensors"), t)
    (tmp_path / "config.json").write_text(json.dumps(dict(raw, eos_token_id=4)))
    assert reg.folder_family(str(tmp_path))[0] is reg.GATED
    assert reg.shape_family("sefalorn-2048")[0] is reg.GATED and reg.shape_family("sulepel-2048")[0] is reg.LAYERED
    assert reg.GATED.kernels in pkg("build").SUBSETS
    seen = {}

    class Recorder:
        takes_reference_pools, num_slots = False, 5

        def __init__(self, cfg, num_blocks, max_batch, max_pages_per_seq, tensors=None, **kw):
            seen.update(cfg=cfg, tensors=tensors)
            self.cfg, self.num_blocks, self.max_batch, self.max_pages = cfg, num_blocks, max_batch, max_pages_per_seq

    monkeypatch.setattr(lay, "LayeredEngine", Recorder)
    be = pkg("backend").B200Backend(max_new_tokens=4)
    be.load_model(str(tmp_path), num_blocks=24, max_batch=2, max_pages_per_seq=8)
    assert seen["cfg"] == lay.LayeredConfig.from_json(raw) and torch.equal(seen["tensors"]["head"], t["head"]) and be.is_eos(4)
    assert len(be._slots.free) == 5


def test_engine_refuses_tensors_that_do_not_fit():
    lay = pkg("layered")

    class Bare:
        cfg = lay.LayeredConfig.from_json(CASES["plain"])
        check = pkg("layered").LayeredEngine._check_tensors

    t = weights(CASES["plain"])
    Bare().check(t)
    for bad in ({k: v for k, v in t.items() if k != "l0.mix.left.talk"}, dict(t, extra=t["head"]),
                dict(t, **{"l1.mix.norm": t["l1.mix.norm"][:-1]})):
        with pytest.raises(ValueError):
            Bare().check(bad)


class FakeEngine:
    """Engine stand-in that records which slot every pass is given."""

    num_blocks, max_batch, max_pages, vocab_size, takes_reference_pools = 40, 4, 8, 50, False
    device = "cpu"

    def __init__(self, num_slots):
        self.num_slots = num_slots
        self.tokens, self.ctx_lens = torch.zeros(4, dtype=torch.int64), torch.zeros(4, dtype=torch.int32)
        self.block_table, self.state_slots = torch.zeros(4, 8, dtype=torch.int32), torch.zeros(4, dtype=torch.int32)
        self.calls, self.fail = [], False

    def prefill(self, token_ids, block_ids, cached_tokens=0, slot=None, want=None):
        self.calls.append(("prefill", slot, cached_tokens))
        if self.fail:
            raise RuntimeError("no")
        return 7, None

    def step(self, B):
        self.calls.append(("step", self.state_slots[:B].tolist()))
        return torch.arange(B)

    def mixed_step(self, B, chunk, block_ids, first_pos, slot=None):
        self.calls.append(("mixed", self.state_slots[:B].tolist(), slot, first_pos))
        if self.fail:
            raise RuntimeError("no")
        return torch.arange(B), 3, None


def test_backend_hands_out_state_slots_and_takes_them_back():
    eng = FakeEngine(3)
    be = pkg("backend").B200Backend(eng, max_new_tokens=4)
    a, _, n = be.prefill([1, 2, 3])
    batch = be.splice_into_batched(None, a, n)
    b, _, _ = be.prefill_chunk([1, 2], None)
    b, _, n = be.prefill_chunk([3], b)  # the same slot for the next portion
    assert eng.calls[-2:] == [("prefill", b.slot, 0), ("prefill", b.slot, 2)] and a.slot != b.slot
    batch = be.splice_into_batched(batch, b, n)
    be.decode_step_batched(torch.tensor([[1], [2]]), batch)
    assert eng.calls[-1] == ("step", [a.slot, b.slot])
    _, batch, c, _, _ = be.decode_step_with_prefill_chunk(torch.tensor([[1], [2]]), batch, [5, 6], None)
    assert eng.calls[-1] == ("mixed", [a.slot, b.slot], c.slot, 0) and len({a.slot, b.slot, c.slot}) == 3
    pages = len(be._alloc.free)
    for call in (lambda: be.prefill([1]), lambda: be.prefill_chunk([1], None),
                 lambda: be.decode_step_with_prefill_chunk(torch.tensor([[1], [2]]), batch, [5], None)):
        with pytest.raises(MemoryError):
            call()  # no slot left: the pages taken for the request go back
        assert len(be._alloc.free) == pages
    gone = a.slot
    be.remove_row_from_cache(batch, 0)
    assert a.slot is None
    eng.fail = True
    for call in (lambda: be.prefill([1]), lambda: be.prefill_chunk([1], None),
                 lambda: be.decode_step_with_prefill_chunk(torch.tensor([[1]]), batch, [5], None)):
        with pytest.raises(RuntimeError):
            call()
        assert be._slots.free == [gone]
    with pytest.raises(RuntimeError):
        be.prefill_chunk([1], c)  # a portion that fails leaves the sequence its slot
    assert c.slot is not None and be._slots.free == [gone]
    eng.fail = False
    be.decode_step_batched(torch.tensor([[1]]), batch)
    assert eng.calls[-1] == ("step", [b.slot])
    del batch  # a dropped batch gives its rows' slots back
    assert sorted(be._slots.free) == sorted([gone, 0, 1, 2][:1] + [s for s in (0, 1, 2) if s not in (gone, c.slot)])


def test_models_without_recurrent_layers_have_no_slots():
    eng = FakeEngine(0)
    be = pkg("backend").B200Backend(eng, max_new_tokens=4)
    kv, _, _ = be.prefill([1, 2])
    assert kv.slot is None and eng.calls == [("prefill", None, 0)]


def test_plain_mechanisms():
    """The oracle's mechanisms on inputs whose results are known by hand."""
    f64 = torch.float64
    # a window of 3 tokens
    see = ref.window_mask(6, 3)
    assert see[4].tolist() == [False, False, True, True, True, False] and see[0].tolist() == [True] + [False] * 5
    # distance penalty and mixing: two heads, the second one's score is the first's with its penalty
    q, k = torch.ones(3, 2, 1, dtype=f64), torch.ones(3, 1, 1, dtype=f64)
    s = ref.talking_scores(q, k, 2.0, torch.tensor([1.0, 0.0], dtype=f64), torch.tensor([1.0, 5.0], dtype=f64), torch.tensor([[0.0, 1.0], [1.0, 0.0]], dtype=f64))
    assert torch.allclose(s[1, 2], 2.0 - torch.log(torch.tensor([3.0, 2.0, 1.0], dtype=f64))) and torch.allclose(s[0], torch.full((3, 3), 2.0, dtype=f64))
    # convolution: an impulse comes out as the taps, latest tap first
    x = torch.zeros(5, 1, dtype=f64)
    x[1] = 1.0
    assert ref.causal_conv(x, torch.tensor([[5.0, 7.0, 11.0]], dtype=f64)).flatten().tolist() == [0, 11, 7, 5, 0]
    # delta rule with beta 1 and no decay stores the last value of a key and reads it in the same step
    e = torch.eye(2, dtype=f64)
    keys, vals = torch.stack([e[0], e[1], e[0]]), torch.tensor([[3.0], [4.0], [5.0]], dtype=f64)
    one = torch.ones(3, dtype=f64)
    assert ref.delta_rule(torch.stack([e[0], e[0], e[0] + e[1]]), keys, vals, one, one).flatten().tolist() == [3.0, 3.0, 9.0]
    # ... with decay 1/2 what was stored has halved before the error is taken
    assert ref.delta_rule(keys, keys, vals, 0.5 * one, 0.5 * one)[2, 0] == 0.375 + 0.5 * (5 - 0.375)
    # lightning: geometric weights
    assert ref.decay_attention(torch.ones(3, 1, dtype=f64), torch.ones(3, 1, dtype=f64), vals, 0.5)[2, 0] == 0.75 + 2 + 5
    # routing: weights of the chosen are normalised by their scores' sum
    ids, w = ref.route(torch.tensor([[0.0, 5.0, -5.0, 5.0]], dtype=f64), 2, 3.0)
    assert sorted(ids[0].tolist()) == [1, 3] and torch.allclose(w, torch.full((1, 2), 1.5, dtype=f64))


@pytest.mark.parametrize("mistake", ["window longer", "window shorter", "penalty", "talk", "head map", "bias", "conv history", "conv tap",
                                     "state lost", "read before write", "decay", "beta", "head norm", "residual gate", "router scale",
                                     "left scale", "logit scale", "mean", "far token"])
def test_the_comparison_would_show_a_mistake(mistake):
    """Weights like the engine tests': every single mistake, planted in the plain implementation, moves the logits by far more
    than the engine tests allow (1e-4 in fp32)."""
    cfg = CASES["plain"]
    t = weights(cfg, seed=1)
    toks = prompt(cfg, 110)
    want, _ = ref.forward(cfg, t, toks)
    bad, tb, ids = json.loads(json.dumps(cfg)), dict(t), list(toks)
    left = bad["layers"][0]["mixer"]["left"]
    patched = {}
    keep = {n: getattr(ref, n) for n in ("window_attention", "causal_conv", "delta_rule", "rms_unit", "residual_gate", "layer_norm", "talking_scores")}
    if mistake == "window longer":
        left["mask"]["size"] += 1
    elif mistake == "window shorter":
        left["mask"]["size"] -= 1
    elif mistake == "penalty":
        tb["l0.mix.left.r2"] = t["l0.mix.left.r2"] * 1.2
    elif mistake == "talk":
        tb["l0.mix.left.talk"] = t["l0.mix.left.talk"].T
    elif mistake == "head map":
        left["kv_heads"] = 1
        for n in ("k", "v"):
            tb["l0.mix.left." + n] = t["l0.mix.left." + n][:64]
            tb[f"l0.mix.left.{n}.b"] = t[f"l0.mix.left.{n}.b"][:64]
    elif mistake == "bias":
        tb["l0.mix.left.q.b"] = torch.zeros_like(t["l0.mix.left.q.b"])
    elif mistake == "conv history":
        patched["causal_conv"] = lambda x, w: torch.cat([keep["causal_conv"](x[:60], w), keep["causal_conv"](x[60:], w)])
    elif mistake == "conv tap":
        tb["l0.mix.right.k.conv"] = t["l0.mix.right.k.conv"].flip(1)
    elif mistake == "state lost":
        patched["delta_rule"] = lambda *a: torch.cat([keep["delta_rule"](*(x[:60] for x in a)), keep["delta_rule"](*(x[60:] for x in a))])
    elif mistake == "read before write":
        patched["delta_rule"] = lambda q, k, v, b, g: keep["delta_rule"](torch.cat([q[1:], q[:1]]), k, v, b, g)
    elif mistake == "decay":
        bad["layers"][1]["mixer"]["decay"][2] = 0.985
    elif mistake == "beta":
        tb["l0.mix.right.b"] = torch.zeros_like(t["l0.mix.right.b"])
    elif mistake == "head norm":
        patched["rms_unit"] = lambda x, eps: x if x.dim() == 3 else keep["rms_unit"](x, eps)
    elif mistake == "residual gate":
        patched["residual_gate"] = lambda h, w, b: torch.sigmoid(h @ w.T)
    elif mistake == "router scale":
        bad["layers"][0]["mlp"]["router"]["scale"] *= 1.05
    elif mistake == "left scale":
        bad["layers"][0]["mixer"]["left_scale"] = 1.0
    elif mistake == "logit scale":
        bad["logit_scale"] = 0.72
    elif mistake == "mean":
        patched["layer_norm"] = lambda x, w, eps: keep["rms_unit"](x, eps) * w
    elif mistake == "far token":
        ids[2] = (ids[2] + 1) % cfg["vocab"]
    with pytest.MonkeyPatch.context() as mp:
        for n, f in patched.items():
            mp.setattr(ref, n, f)
        got, _ = ref.forward(bad, tb, ids)
    assert row_error(got[-40:], want[-40:]) > 20e-4


def test_no_expert_is_left_out_where_all_are_chosen():
    cfg = all_chosen(CASES["generic"])
    assert [(e["mlp"]["router"]["experts"], e["mlp"]["router"]["top"]) for e in cfg["layers"] if e["mlp"]] == [(12, 12)]
    small = config([par((2, 1, 8, 8, 0.3, 4), (2, 1, 8, 8, 2), moe(2, 1, 8)), light(2, 8, 8, (0.5, 0.9))], vocab=23, width=32)
    t = weights(small)
    a, after = ref.forward(small, t, list(range(20)))
    b, _ = ref.forward(small, t, list(range(12)))
    assert torch.allclose(a[:12], b) and after.shape == (2, 20, 32)  # no token sees what follows
