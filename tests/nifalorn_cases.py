"""Small Nifalorn configurations for the tests, and the plain implementation's logits for them.

The configurations differ from one another in every size and option: loops over inner layers, over the first layers, over
all layers, of one pass, and none; decays of 0 and 1 beside ordinary ones; Mamba-2 layers whose heads share groups, have
one each, and all share one, with convolutions of 1, 2, 3, 4 and 7 taps and norms in 1 to 6 parts; states below and above
what one block of the recurrence kernels holds; chunks of one position, of 17, of one page, and none; rotations of part
of a head, of the whole head, with and without stretched frequencies, and none; experts in groups (also of a single
expert, and one group), all of them chosen, with and without a shared expert; layers without feed-forward; widths that
are no multiples of 8 or of 4, and odd head sizes.
"""

from __future__ import annotations

import copy

import torch

from plain import nifalorn_plain as plain
from starter_b200.config import config_from_dict
from starter_b200.weights import write_model_folder


def _lightning(decay, dim, vdim):
    return {"type": "lightning", "mixer": {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay)}}


def _mamba(heads, vdim, state, groups, conv, norm_groups):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}}


def _attention(heads, kv_heads, dim, vdim, diff, chunk=None, rot=None, scaling=None, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "diff": diff, "scale": dim ** -0.5 if scale is None else scale}
    if chunk is not None:
        m["mask"] = {"size": chunk}
    if rot is not None:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
        if scaling is not None:
            m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return {"type": "attention", "mixer": m}


def _moe(experts, top, ff, groups=None, scale=None, shared=None):
    router = {"experts": experts, "top": top}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    if scale is not None:
        router["scale"] = scale
    mlp = {"kind": "moe", "router": router, "expert": {"ff": ff}}
    if shared is not None:
        mlp["shared"] = {"ff": shared}
    return mlp


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _with(entry, mlp):
    return dict(copy.deepcopy(entry), mlp=mlp)


def _model(vocab, width, eps, loop, layers, embed=1.0, logit=1.0):
    raw = {"architecture": "Nifalorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers,
           "embedding": {"scale": embed}, "logit_scale": logit}
    if loop is not None:
        raw["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return raw


CASES = {
    # two passes over three inner layers; three groups of B and C; twelve experts in three groups; a chunk of 24
    "A": _model(211, 96, 1e-5, (1, 4, 2), [
        _with(_lightning([0.9, 0.5, 0.99], 16, 24), _moe(12, 3, 40, (3, 2), 1.7, 56)),
        _with(_mamba(6, 16, 24, 3, 3, 2), _dense(136)),
        _with(_attention(6, 2, 16, 24, 0.7, 24, (10000.0, 12), (8.0, 1.0, 4.0, 512), scale=0.4), _moe(10, 2, 24, (5, 2), 0.8, 32)),
        _with(_lightning([0.2, 0.999], 40, 8), None),
        _with(_mamba(4, 24, 16, 1, 2, 4), _moe(6, 2, 32, None, 2.0, 16))], embed=0.7, logit=1.5),
    # sizes the tensor-core kernels take; no loop
    "B": _model(300, 128, 1e-6, None, [
        _with(_mamba(8, 64, 128, 2, 4, 4), _moe(8, 2, 96, (4, 2), 1.5, 128)),
        _with(_attention(4, 1, 64, 128, 0.5, 100, (500000.0, 64), (16.0, 1.0, 4.0, 256)), _dense(256)),
        _with(_lightning([0.7, 0.95, 0.995, 0.9999], 64, 64), _moe(16, 4, 64, (8, 3), 1.0, 64)),
        _with(_attention(8, 4, 32, 64, 0.8, 64, (10000.0, 32), scale=0.2), None)]),
    # single heads, a decay of 0 and one of 1, one tap, no rotation, no chunk, groups of one expert, no shared expert,
    # widths that are no multiples of 8; the loop starts at the first layer
    "C": _model(97, 40, 1e-4, (0, 2, 3), [
        _with(_lightning([0.0, 1.0], 20, 12), _moe(4, 2, 24, (4, 3))),
        _with(_mamba(1, 10, 136, 1, 1, 1), _dense(20)),
        _with(_attention(1, 1, 20, 12, 0.9), _moe(3, 3, 16, (1, 1), 1.3)),
        _with(_mamba(3, 4, 12, 3, 7, 6), None)], embed=2.0, logit=0.25),
    # one pass; a chunk of one position; keys wider than 128 columns and values over several blocks
    "D": _model(64, 32, 1e-5, (1, 2, 1), [
        _with(_lightning([0.9], 200, 130), _dense(16)),
        _with(_attention(2, 2, 8, 8, 0.6, 1, (10000.0, 2)), _moe(9, 1, 8, (3, 1), 3.0, 24)),
        _with(_mamba(2, 72, 80, 2, 4, 3), _dense(48))]),
    # a width that is no multiple of 4, odd head sizes everywhere (rows that no 16-byte read fits), the loop over all
    # layers, every expert chosen, twelve query heads on one key head
    "E": _model(131, 30, 1e-6, (0, 3, 2), [
        _with(_mamba(4, 3, 9, 2, 4, 3), _moe(6, 6, 10, (2, 2), 1.1, 14)),
        _with(_attention(12, 1, 5, 7, 0.35, 17, (50.0, 4), (2.0, 0.5, 2.0, 40)), _dense(22)),
        _with(_lightning([0.6, 0.97, 0.8], 7, 5), None)], embed=5.0, logit=0.6),
}
SEEDS = {"A": 45, "B": 46, "C": 47, "D": 48, "E": 49}


def config(name):
    return config_from_dict(copy.deepcopy(CASES[name]))


def write_folder(name, folder, dtype=torch.bfloat16, shards=1, steady=False):
    """``steady``: corrections so far apart that they alone choose the experts, and no close call that rounding turns."""
    cfg = config(name)
    if steady:
        ordinary = cfg.random_init
        object.__setattr__(cfg, "random_init", lambda tensor, shape: (0.0, 6.0) if tensor.endswith("correction") else ordinary(tensor, shape))
    return write_model_folder(cfg, SEEDS[name], folder, dtype=dtype, shards=shards)


def plain_logits(folder, seqs):
    cfg, tensors = plain.read_folder(folder)
    return [plain.forward(cfg, tensors, s) for s in seqs]
