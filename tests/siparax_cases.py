"""Small Siparax configurations for the tests, and the plain implementation's logits for them.

The configurations differ from one another in every size and option: 1, 2, 3, 5 and 8 taps; as many query/key heads as
value heads, fewer, and one; key and value sizes that differ either way, sizes of two columns, beyond the 128 key
channels and 128 value columns that registers hold, and no multiples of 4 or 8; inner sizes of the decay and of the gate
that differ; latents of widths the tensor-core kernels take and do not; one head; rotations stretched (with ramps inside,
above and below the pairs) and plain; rotated parts of 2 columns and more; layers that read another layer's latents, next
to it, further back, twice from one, and with other head counts and sizes; layers without feed-forward; a cap and none.
"""

from __future__ import annotations

import copy

import torch

from plain import siparax_plain as plain
from starter_b200.config import config_from_dict
from starter_b200.weights import write_model_folder


def _delta(heads, kv_heads, dim, vdim, conv, decay_rank, gate_rank):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv,
                                               "decay_rank": decay_rank, "gate_rank": gate_rank}}


def _latent(kind, heads, dim, rot_dim, vdim, q_rank, kv_rank, base, stretch=None, scale=None, kv_from=None):
    rot = {"base": base, "dims": rot_dim}
    if stretch is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), stretch))
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "rot": rot,
         "scale": (dim + rot_dim) ** -0.5 if scale is None else scale}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": kind, "mixer": m}


def _pairs(*args, **kw):
    return _latent("latent_attention", *args, **kw)


def _halves(*args, **kw):
    return _latent("latent_attention_2", *args, **kw)


def _with(entry, ff):
    entry = copy.deepcopy(entry)
    entry["mlp"] = {"kind": "dense", "ff": ff} if ff else None
    return entry


def _model(vocab, width, eps, cap, layers):
    raw = {"architecture": "Siparax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if cap is not None:
        raw["logit_softcap"] = cap
    return raw


STRETCH = (4.0, 64, 8.0, 0.5)
CASES = {
    # every kind; a layer that reads the latents of a layer further back, another of the same; fewer query/key heads
    "A": _model(211, 96, 1e-5, 12.0, [
        _with(_halves(3, 20, 8, 24, 40, 48, 1000.0, STRETCH, scale=0.3), 72),
        _with(_delta(6, 2, 16, 24, 3, 20, 12), 136),
        _with(_halves(4, 12, 8, 16, 36, 48, 1000.0, STRETCH, kv_from=0), None),
        _with(_pairs(5, 24, 12, 20, 28, 44, 500.0, (2.0, 40, 6.0, 1.0)), 64),
        _with(_halves(2, 32, 8, 40, 24, 48, 1000.0, STRETCH, scale=0.5, kv_from=0), 40)]),
    # sizes the tensor-core kernels take
    "B": _model(300, 128, 1e-6, 50.0, [
        _with(_delta(4, 4, 64, 64, 4, 32, 32), 256),
        _with(_pairs(2, 80, 48, 64, 96, 128, 10000.0, (8.0, 128, 24.0, 1.0)), 192),
        _with(_halves(4, 32, 32, 128, 64, 64, 1000000.0, (16.0, 256, 16.0, 2.0)), 128),
        _with(_halves(16, 48, 32, 64, 64, 64, 1000000.0, (16.0, 256, 16.0, 2.0), kv_from=2), 64)]),
    # no feed-forward anywhere but once, no cap, no stretch, single heads, one tap, widths that are no multiples of 8
    "C": _model(97, 40, 1e-4, None, [
        _with(_delta(1, 1, 20, 12, 1, 5, 7), None),
        _with(_pairs(1, 10, 2, 6, 12, 14, 100.0), None),
        _with(_halves(1, 6, 4, 18, 10, 9, 50.0), 20),
        _with(_delta(2, 1, 136, 130, 5, 3, 1), None)]),
    # a delta layer last; more value columns than registers hold in one turn; two readers in a row
    "D": _model(64, 32, 1e-5, 3.0, [
        _with(_pairs(2, 8, 4, 8, 16, 24, 10000.0, (4.0, 32, 4.0, 0.25)), 16),
        _with(_halves(2, 8, 6, 4, 8, 16, 300.0, (3.0, 100, 10.0, 0.5)), None),
        _with(_halves(3, 4, 6, 8, 20, 16, 300.0, (3.0, 100, 10.0, 0.5), kv_from=1), 48),
        _with(_halves(1, 16, 6, 12, 8, 16, 300.0, (3.0, 100, 10.0, 0.5), kv_from=1), None),
        _with(_delta(8, 4, 8, 136, 2, 8, 16), 48)]),
    # a width that is no multiple of 4, odd sizes everywhere (rows that no 16-byte read fits), an odd vocabulary, eight taps,
    # keys of two columns
    "E": _model(131, 30, 1e-6, 20.0, [
        _with(_delta(3, 1, 7, 5, 8, 3, 9), 14),
        _with(_pairs(7, 5, 6, 3, 11, 13, 700.0, STRETCH), 22),
        _with(_delta(5, 5, 2, 3, 2, 1, 1), None),
        _with(_halves(5, 3, 2, 7, 9, 65, 40.0, (2.0, 20, 2.0, 1.0)), 10)]),
}
SEEDS = {"A": 45, "B": 46, "C": 47, "D": 48, "E": 49}


def config(name):
    return config_from_dict(copy.deepcopy(CASES[name]))


def write_folder(name, folder, dtype=torch.bfloat16, shards=1):
    return write_model_folder(config(name), SEEDS[name], folder, dtype=dtype, shards=shards)


def plain_logits(folder, seqs):
    cfg, tensors = plain.read_folder(folder)
    return [plain.forward(cfg, tensors, s) for s in seqs]
