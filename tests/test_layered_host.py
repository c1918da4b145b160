"""Layer-list decoders on the CPU: configuration, padded run-time weights, checkpoint reading, registry, position tables,
and the plain implementation's own mechanisms (tests/test_gpu_layered*.py compare the engine with it)."""
import json

import pytest
import torch

from conftest import pkg
from layered_cases import CASES, att, config, lat, weights
from oracle import layered_ref as ref


def test_config_reads_every_size_and_refuses_what_it_does_not_know():
    lay = pkg("layered")
    cfg = lay.LayeredConfig.from_json(CASES["odd"])
    assert (cfg.vocab_size, cfg.width, cfg.norm_groups, cfg.taps, cfg.layers, cfg.norm_eps) == (211, 204, 6, 2, 4, 1e-5)
    assert cfg.layer_list[1].mixer == lay.AttentionSpec(6, 3, 40, 24, 0.21, 37) and cfg.layer_list[1].mlp is None
    assert cfg.layer_list[0].mixer == lay.LatentSpec(3, 24, 40, 72, 0.3) and cfg.layer_list[0].mlp == lay.GluSpec(100, 0.8)
    shapes = cfg.tensor_shapes()
    assert shapes["l1.mix.k"] == (120, 204) and shapes["l1.mix.v"] == (72, 204) and shapes["l0.mix.uv"] == (120, 72)
    assert "l1.norm2" not in shapes and "l3.mlp.gate" not in shapes and shapes["l2.norm2"] == (204,)
    for breakage in (lambda c: c["layers"][0].update(type="other"), lambda c: c["layers"][0]["mlp"].update(kind="sparse"),
                     lambda c: c["norm"].update(groups=5), lambda c: c["layers"][1]["mixer"].update(kv_heads=4)):
        bad = json.loads(json.dumps(CASES["odd"]))
        breakage(bad)
        with pytest.raises(ValueError):
            lay.LayeredConfig.from_json(bad)


@pytest.mark.parametrize("name", sorted(CASES))
def test_padded_weights_compute_the_same_layer(name):
    """The run-time form on plain matrix products equals the layer's equations: padding changes nothing."""
    lay = pkg("layered")
    raw = CASES[name]
    cfg, t = lay.LayeredConfig.from_json(raw), weights(raw, seed=3)
    g = torch.Generator().manual_seed(1)
    for i, spec in enumerate(cfg.layer_list):
        p = f"l{i}."
        w = lay.LayeredWeights(spec, {k[len(p):]: v for k, v in t.items() if k.startswith(p)}, cfg, "cpu", torch.float32)
        m, D, W = spec.mixer, w.D, lay.pad_width(cfg.width)
        assert W % 64 == 0 and D % 64 == 0
        h = torch.randn(5, cfg.width, generator=g)
        hp = torch.zeros(5, W)
        hp[:, : cfg.width] = h
        y = hp @ w.wproj.T
        if w.col_scale is not None:
            y = y * w.col_scale
        f = {k[len(p) + 4:]: v.float() for k, v in t.items() if k.startswith(p + "mix.")}
        q = (h @ f["q"].T).view(5, m.heads, m.dim) * (-1 if m.scale < 0 else 1)
        if "temp" in f:
            q = q * f["temp"][:, None]
        got = y[:, : m.heads * D].view(5, m.heads, D)
        assert torch.allclose(got[..., : m.dim], q, atol=1e-4) and not got[..., m.dim:].any()
        assert torch.allclose(y[:, -m.heads:], h @ f["g"].T, atol=1e-4)
        o = torch.randn(5, m.heads, m.vdim, generator=g)
        op = torch.zeros(5, m.heads, D)
        op[..., : m.vdim] = o
        out = op.view(5, -1) @ w.wo.T
        assert torch.allclose(out[:, : cfg.width], o.reshape(5, -1) @ f["o"].T, atol=1e-4) and not out[:, cfg.width:].any()
        if isinstance(m, lay.LatentSpec):
            c = torch.randn(5, m.rank, generator=g)
            cp = torch.zeros(5, w.R)
            cp[:, : m.rank] = c
            k, v = (c @ f["uk"].T).view(5, m.heads, m.dim), (c @ f["uv"].T).view(5, m.heads, m.vdim)
            direct = torch.einsum("thd,shd->hts", q, k)
            absorbed = torch.einsum("hrd,thd,sr->hts", w.wuk_t, got, cp)
            assert torch.allclose(direct, absorbed, atol=1e-3)
            vals = torch.einsum("hdr,sr->shd", w.wuv, cp)
            assert torch.allclose(vals[..., : m.vdim], v, atol=1e-4)
        if spec.mlp is not None:
            gu = (hp @ w.wgu.T).view(5, -1, 2, 128)
            gate, up = gu[:, :, 0].reshape(5, -1), gu[:, :, 1].reshape(5, -1)
            a = ref.clamped_glu(gate, up, spec.mlp.limit)
            full = ref.clamped_glu(h @ t[p + "mlp.gate"].float().T, h @ t[p + "mlp.up"].float().T, spec.mlp.limit)
            assert torch.allclose(a[:, : spec.mlp.inner], full, atol=1e-4)
            out = a @ w.wdown.T
            assert torch.allclose(out[:, : cfg.width], full @ t[p + "mlp.down"].float().T, atol=1e-4)
            assert not out[:, cfg.width:].any()


@pytest.mark.parametrize("width,ld", [(204, 256), (64, 64), (7, 64)])
def test_sinusoid_tables_give_every_position_by_the_addition_theorem(width, ld):
    lo, hi = pkg("layered").sinusoid_tables(width, ld, 5000, "cpu")
    assert lo.shape == (64, ld) and hi.shape == (79, ld) and lo.dtype == torch.float32
    p = torch.tensor([0, 1, 63, 64, 65, 127, 1000, 4999])
    a, b = hi[p // 64].double(), lo[p % 64].double()
    s = a[:, 0::2] * b[:, 1::2] + a[:, 1::2] * b[:, 0::2]
    c = a[:, 1::2] * b[:, 1::2] - a[:, 0::2] * b[:, 0::2]
    got = torch.stack([s, c], -1).view(len(p), ld)[:, :width]
    assert float((got - ref.sinusoid(p, width)).abs().max()) < 3e-7


def test_checkpoint_round_trip_registry_and_loading(tmp_path, monkeypatch):
    ck, reg, lay = pkg("checkpoint"), pkg("registry"), pkg("layered")
    raw = CASES["plain"]
    t = weights(raw)
    t["table"] = torch.arange(7, dtype=torch.int32)
    ck.write_safetensors(str(tmp_path / "model.safetensors"), t)
    back = ck.read_safetensors(str(tmp_path / "model.safetensors"))
    assert sorted(back) == sorted(t) and all(torch.equal(back[k], t[k]) and back[k].dtype == t[k].dtype for k in t)
    with open(tmp_path / "cut.safetensors", "wb") as f:
        f.write(open(tmp_path / "model.safetensors", "rb").read()[:-10])
    with pytest.raises(ValueError):
        ck.read_safetensors(str(tmp_path / "cut.safetensors"))
    assert reg.folder_family(str(tmp_path)) is None  # no config.json
    (tmp_path / "config.json").write_text(json.dumps(dict(raw, eos_token_id=[4, 9])))
    family, config_json = reg.folder_family(str(tmp_path))
    assert family is reg.LAYERED and config_json["width"] == raw["width"]
    assert reg.shape_family("sulepel-2048")[0] is reg.LAYERED and reg.shape_family("tiny")[0] is reg.QWEN3_MOE
    assert reg.shape_family("no such shape") is None
    # B200Backend.load_model goes through the registry (the engine itself needs a GPU, so its constructor records instead)
    seen = {}

    class Recorder:
        takes_reference_pools = False

        def __init__(self, cfg, num_blocks, max_batch, max_pages_per_seq, tensors=None, **kw):
            seen.update(cfg=cfg, tensors=tensors, kw=kw)
            self.cfg, self.num_blocks, self.max_batch, self.max_pages = cfg, num_blocks, max_batch, max_pages_per_seq

    monkeypatch.setattr(lay, "LayeredEngine", Recorder)
    be = pkg("backend").B200Backend(max_new_tokens=4)
    be.load_model(str(tmp_path), num_blocks=24, max_batch=2, max_pages_per_seq=8, dtype=torch.float32)
    assert seen["cfg"] == lay.LayeredConfig.from_json(raw) and seen["kw"] == {"dtype": torch.float32}
    assert torch.equal(seen["tensors"]["head"], t["head"]) and be.is_eos(9) and not be.is_eos(5)
    assert len(be._alloc.free) == 24

    class Manager:
        class block_manager:
            k_pools = [torch.zeros(1)]

    with pytest.raises(ValueError, match="does not fit"):
        be.set_cache_adapter(Manager())
    with pytest.raises(ValueError):
        be.kv_shape_per_layer()
    be.load_model("sulepel-2048", num_blocks=24, max_batch=2, max_pages_per_seq=8)
    assert seen["cfg"] is lay.CONFIGS["sulepel-2048"] and seen["tensors"] is None
    (tmp_path / "config.json").write_text(json.dumps(dict(raw, architecture="Other")))
    with pytest.raises(ValueError, match="Other"):
        reg.folder_family(str(tmp_path))


def test_engine_refuses_tensors_that_do_not_fit():
    lay = pkg("layered")
    eng = lay.LayeredEngine.__new__(lay.LayeredEngine)
    eng.cfg = lay.LayeredConfig.from_json(CASES["plain"])
    t = weights(CASES["plain"])
    eng._check_tensors(t)
    with pytest.raises(ValueError, match="missing"):
        eng._check_tensors({k: v for k, v in t.items() if k != "l0.mix.temp"})
    with pytest.raises(ValueError, match="not known"):
        eng._check_tensors(dict(t, extra=t["head"]))
    with pytest.raises(ValueError, match="l1.mix.dkv"):
        eng._check_tensors(dict(t, **{"l1.mix.dkv": t["l1.mix.dkv"][:-1]}))


def test_plain_mechanisms():
    """The oracle's mechanisms on inputs whose results are known by hand."""
    # grouped norm: each part has unit mean square
    x = torch.randn(4, 12, dtype=torch.float64, generator=torch.Generator().manual_seed(0)) * 3
    y = ref.group_rmsnorm(x, torch.ones(12, dtype=torch.float64), 0.0, 3).view(4, 3, 4)
    assert torch.allclose(y.pow(2).mean(-1), torch.ones(4, 3, dtype=torch.float64))
    # convolution: an impulse comes out as itself plus the taps, latest tap first
    h = torch.zeros(6, 1, dtype=torch.float64)
    h[1] = 1.0
    w = torch.tensor([[5.0, 7.0, 11.0]], dtype=torch.float64)
    assert ref.short_conv(h, w).flatten().tolist() == [0, 12, 7, 5, 0, 0]
    # chunks of 3 positions
    see = ref.visible(7, 3)
    assert see[5].tolist() == [False, False, False, True, True, True, False]
    assert see[6].tolist() == [False] * 6 + [True] and int(ref.visible(7, 0).sum()) == 28
    # gated unit: the gate is capped above only, the other side on both sides
    g, u = torch.tensor([9.0, -9.0]), torch.tensor([9.0, -9.0])
    assert torch.allclose(ref.clamped_glu(g, u, 2.0), torch.tensor([2 * torch.sigmoid(torch.tensor(3.404)) * 3,
                                                                    -9 * torch.sigmoid(torch.tensor(-15.318)) * -1]))
    # a request's logits do not depend on what follows, and do on what a latent layer sees far back
    cfg = config([att(2, 1, 8, 8, 0.3, 4), lat(2, 8, 8, 16, 0.3, 16)], vocab=23, width=32, groups=2, taps=3)
    t = weights(cfg)
    a, _ = ref.layered_forward(cfg, t, list(range(20)))
    b, _ = ref.layered_forward(cfg, t, list(range(12)))
    assert torch.allclose(a[:12], b)
    c, _ = ref.layered_forward(cfg, t, [7] + list(range(1, 20)))
    assert float((c[19] - a[19]).abs().max()) > 1e-6


@pytest.mark.parametrize("mistake", ["chunk end", "chunk start", "no chunk", "conv history", "conv tap", "gate", "temp", "limit", "groups",
                                     "far key", "position", "latent norm"])
def test_the_comparison_would_show_a_mistake(mistake):
    """Weights like the engine tests': every single mistake, planted in the plain implementation, moves the logits by far
    more than the engine tests allow (1e-4 in fp32)."""
    from layered_cases import prompt, row_error
    cfg = CASES["plain"]
    t = weights(cfg, seed=1)
    toks = prompt(cfg, 110)
    want, _ = ref.layered_forward(cfg, t, toks)
    bad, tb, ids = json.loads(json.dumps(cfg)), dict(t), list(toks)
    names = [n for n in t]
    patched = {}
    if mistake == "chunk end":
        bad["layers"][0]["mixer"]["mask"]["size"] = 49
    elif mistake == "chunk start":
        patched["visible"] = lambda T, chunk: ref_visible(T, 0) if not chunk else (
            ref_visible(T, chunk) | (torch.arange(T)[None] == torch.arange(T)[:, None] // chunk * chunk - 1))
    elif mistake == "no chunk":
        bad["layers"][0]["mixer"]["mask"]["size"] = 0
    elif mistake == "conv history":
        patched["short_conv"] = lambda h, w: torch.cat([ref_conv(h[:60], w), ref_conv(h[60:], w)])
    elif mistake == "conv tap":
        for n in names:
            if n.endswith("canon1"):
                tb[n] = t[n].flip(1)
    elif mistake == "gate":
        patched["head_gate"] = lambda o, h, wg: o
    elif mistake == "temp":
        tb["l0.mix.temp"] = torch.ones_like(t["l0.mix.temp"])
    elif mistake == "limit":
        patched["clamped_glu"] = lambda g, u, limit: ref_glu(g, u, 1e9)
    elif mistake == "groups":
        bad["norm"]["groups"] = 2
    elif mistake == "far key":
        ids[2] = (ids[2] + 1) % cfg["vocab"]
    elif mistake == "position":
        patched["sinusoid"] = lambda p, width, dtype=torch.float64: ref_sin(p + (p >= 64), width, dtype)
    elif mistake == "latent norm":
        tb["l1.mix.dkv.norm"] = torch.ones_like(t["l1.mix.dkv.norm"])
    ref_visible, ref_conv, ref_glu, ref_sin = ref.visible, ref.short_conv, ref.clamped_glu, ref.sinusoid
    with pytest.MonkeyPatch.context() as mp:
        for k, v in patched.items():
            mp.setattr(ref, k, v)
        got, _ = ref.layered_forward(bad, tb, ids)
    assert row_error(got[-50:], want[-50:]) > 20e-4
