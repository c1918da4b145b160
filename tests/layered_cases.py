"""Small layer-list configurations and random weights for the tests (sizes of no particular model)."""
import torch

from conftest import pkg


def att(heads, kv_heads, dim, vdim, scale, chunk, ff=None, limit=1.5):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                                           "mask": {"size": chunk}},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}


def lat(heads, dim, vdim, rank, scale, ff=None, limit=1.5):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": rank, "scale": scale},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}


def config(layers, vocab=300, width=192, groups=3, taps=4, eps=1e-5):
    return {"architecture": "Sulepel", "vocab": vocab, "width": width, "canon": {"taps": taps},
            "norm": {"eps": eps, "groups": groups}, "layers": layers}


CASES = {
    # sizes that the kernels take as they are
    "plain": config([att(8, 2, 64, 64, 0.13, 48, 256), lat(4, 64, 64, 128, 0.11, 128)], width=256, groups=1, taps=3),
    # odd sizes: everything is padded; a layer without feed-forward; different sizes per layer; query/key size != value size
    "odd": config([lat(3, 24, 40, 72, 0.3, 100, 0.8), att(6, 3, 40, 24, 0.21, 37), att(5, 5, 72, 100, 0.09, 16, 200, 3.0),
                   lat(5, 100, 20, 136, 0.17)], vocab=211, width=204, groups=6, taps=2),
    # one kv head for many query heads, a chunk of 1 position, long convolution, one norm group per 256 columns
    "wide": config([att(24, 1, 16, 64, 0.25, 1, 300), att(16, 1, 128, 128, 0.08, 130, 640), lat(20, 32, 32, 500, 0.2, 384)],
                   vocab=517, width=512, groups=2, taps=18),
    # no convolution history (one tap), more than 16 query heads per kv head, sizes only the generic kernels take
    "generic": config([att(34, 2, 32, 32, -0.2, 50, 128), att(2, 1, 160, 136, 0.07, 64, 64), lat(2, 200, 48, 600, 0.1)],
                      vocab=129, width=128, groups=4, taps=1),
}


def weights(cfg, seed=0, gain=2.0, temp=True):
    """Random tensors, bf16 values; `gain` on the query maps makes attention pick out few keys."""
    g = torch.Generator().manual_seed(seed)
    shapes = pkg("layered").LayeredConfig.from_json(cfg).tensor_shapes()
    out = {}
    for name, shape in shapes.items():
        if "norm" in name:
            t = 1.0 + 0.3 * torch.randn(shape, generator=g)
        elif name.endswith("temp"):
            t = 1.0 + 0.5 * torch.randn(shape, generator=g) if temp else torch.ones(shape)
        elif name.endswith("canon1"):
            t = torch.randn(shape, generator=g) * 0.4
        elif name == "embed":
            t = torch.randn(shape, generator=g)
        else:
            t = torch.randn(shape, generator=g) * shape[-1] ** -0.5 * (gain if name.endswith(("mix.q", "mix.g")) else 1.0)
        out[name] = t.bfloat16()
    return out


def prompt(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(100 + seed)).tolist()


def engine(cfg, tensors, dtype=torch.float32, num_blocks=64, max_batch=8, max_pages=24, **kw):
    lay = pkg("layered")
    return lay.LayeredEngine(lay.LayeredConfig.from_json(cfg), num_blocks, max_batch, max_pages, tensors=tensors, dtype=dtype,
                             keep_logits=True, **kw)


def row_error(got, want):
    """Worst row of |got - want| (mean over the vocabulary taken off), relative to the spread of `want`'s rows."""
    got, want = got.double().cpu(), want.double().cpu()
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    spread = (want - want.mean(-1, keepdim=True)).pow(2).mean().sqrt()
    return float((d.pow(2).mean(-1).sqrt() / spread).max())
