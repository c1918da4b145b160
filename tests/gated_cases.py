"""Small gated layer-list configurations and random weights for the tests (sizes of no particular model)."""
import json

import torch

from conftest import pkg
from layered_cases import engine, prompt, row_error  # noqa: F401  (used by the tests of both designs)


def moe(experts, top, ff, scale=1.5):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}}


def par(left, right, mlp=None, scales=(0.8, 1.3)):
    """left: heads, kv_heads, dim, vdim, scale, window; right: heads, kv_heads, dim, vdim, taps."""
    h, g, d, dv, s, w = left
    rh, rg, rd, rdv, taps = right
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": {"heads": h, "kv_heads": g, "dim": d, "vdim": dv, "scale": s, "mask": {"size": w}},
                      "right": {"heads": rh, "kv_heads": rg, "dim": rd, "vdim": rdv, "conv": taps},
                      "left_scale": scales[0], "right_scale": scales[1]}}


def light(heads, dim, vdim, decay, mlp=None):
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}, "mlp": mlp}


def config(layers, vocab=300, width=192, eps=1e-5, logit_scale=0.7):
    return {"architecture": "Sefalorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale,
            "layers": layers}


CASES = {
    # sizes that the kernels take as they are
    "plain": config([par((8, 2, 64, 64, 0.13, 48), (4, 4, 64, 64, 4), moe(8, 2, 128)), light(4, 64, 64, (0.6, 0.9, 0.99, 0.999), moe(8, 2, 128))],
                    width=256),
    # odd sizes: everything is padded; a layer without experts; different sizes per layer; one value for every size that
    # could be taken for another
    "odd": config([light(3, 24, 40, (0.5, 0.93, 0.998), moe(7, 3, 100, 0.6)), par((6, 3, 40, 24, 0.21, 37), (6, 2, 20, 36, 2)),
                   par((5, 5, 72, 100, 0.09, 16), (4, 2, 48, 24, 3), moe(5, 1, 72, 2.5), (1.7, 0.4)), light(5, 72, 20, (0.2, 0.7, 0.9, 0.97, 1.0))],
                  vocab=211, width=204, logit_scale=-1.3),
    # one kv head for many query heads, a window of one token, a long convolution, every expert chosen
    "wide": config([par((24, 1, 16, 64, 0.25, 1), (2, 1, 128, 128, 18), moe(3, 3, 300, 1.0), (1.0, 1.0)),
                    par((16, 2, 128, 128, 0.08, 130), (8, 4, 64, 128, 4), moe(16, 4, 128))], vocab=517, width=512, logit_scale=1.0),
    # no convolution history (one tap), sizes only the generic kernels take, a window longer than any sequence, a negative scale
    "generic": config([par((34, 2, 32, 32, -0.2, 1000), (2, 2, 144, 136, 1), moe(40, 5, 64)), light(2, 200, 48, (0.9, 0.99)),
                       par((2, 1, 160, 296, 0.07, 64), (3, 1, 16, 264, 5))], vocab=129, width=128, logit_scale=0.25),
}


def all_chosen(cfg, most=12):
    """The configuration with every expert of a layer chosen, at most `most` of them: no choice between two experts of nearly the
    same score is left for bf16 rounding to make."""
    cfg = json.loads(json.dumps(cfg))
    for layer in cfg["layers"]:
        if layer["mlp"] is not None:
            r = layer["mlp"]["router"]
            r["experts"] = r["top"] = min(r["experts"], most)
    return cfg


def weights(cfg, seed=0, gain=2.0):
    """Random tensors, bf16 values; `gain` on the query maps makes attention pick out few keys."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in pkg("layered").LayeredConfig.from_json(cfg).tensor_shapes().items():
        r = torch.randn(shape, generator=g)
        if "norm" in name:
            t = 1.0 + 0.3 * r
        elif name.endswith("talk"):
            t = torch.eye(shape[0]) + 0.3 * r
        elif name.endswith("r1"):
            t = 0.6 * r.abs()
        elif name.endswith("r2"):
            t = 0.3 * r.abs()
        elif name.endswith("A_log"):
            t = -1.5 + 1.5 * r
        elif name.endswith("dt_bias"):
            t = -1.0 + r
        elif name.endswith(".conv"):
            t = r * 0.5
        elif name.endswith(".b") and len(shape) == 1:
            t = 0.3 * r
        elif name == "embed":
            t = r
        else:
            t = r * shape[-1] ** -0.5 * (gain if name.endswith(("left.q", "left.k")) else 1.0)
        out[name] = t.bfloat16()
    return out


def run_cuts(eng, tokens, cuts, block_ids, slot=0):
    """Logits of every position, the sequence fed in portions of the given sizes; size 1 is a decode step (row 0) once the
    sequence has begun."""
    out, at = [], 0
    for n in cuts:
        if n == 1 and at:
            eng.block_table[0].zero_()
            eng.block_table[0, : len(block_ids)] = torch.tensor(block_ids, dtype=torch.int32)
            eng.state_slots[0] = slot
            eng.ctx_lens[0] = at
            eng.tokens[0] = tokens[at]
            eng.step(1)
            out.append(eng.last_logits[:1].float().cpu())
        else:
            _, lg = eng.prefill(tokens[: at + n], block_ids, cached_tokens=at, want=list(range(at, at + n)), slot=slot)
            out.append(lg.float().cpu())
        at += n
    eng.check_status("test")
    return torch.cat(out)
