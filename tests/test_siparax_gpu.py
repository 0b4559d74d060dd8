"""Siparax on the GPU against the plain implementation: every mechanism alone, then whole models in every way of cutting
the work; a key that stands out far back, at page borders and on both sides of the causal edge; decays that forget
everything at once; chunk edges of the delta rule; states of several sequences and of a slot that is used again; long
decoding; and greedy generation through the entry point."""

import pytest
import torch

import siparax_cases as cases
from conftest import random_tokens
from helpers import assert_close, make_session, run_ragged_batches, run_tail_by_one, run_whole
from plain import siparax_plain as plain
from starter_b200.cache import Cache
from starter_b200.config import ChannelDeltaSpec, GatedMLPSpec, LatentAttentionSpec, LayerNormSpec, PairRopeSpec, ScaledHalfRopeSpec
from starter_b200.engine import Engine
from starter_b200.engine.context import Runtime, StepContext
from starter_b200.parts import build_part

pytestmark = pytest.mark.gpu
MODES = ["float32", "bfloat16"]
REL = {"float32": 3e-5, "bfloat16": 2.5e-2}
EPS = 1e-5


def runtime(mode):
    from starter_b200.csrc.ops import get_ops
    return Runtime(dtype=getattr(torch, mode), device=torch.device("cuda"), ops=get_ops(verbose=False))


def rand(shape, seed, scale=1.0, mean=0.0):
    g = torch.Generator().manual_seed(seed)
    return (mean + torch.randn(shape, generator=g) * scale).to(torch.bfloat16).float()   # bfloat16 numbers, so both modes read the same


def close(got, want, mode, what, rel=None):
    rel = rel or REL[mode]
    want = want.float()
    assert got.shape == want.shape, f"{what}: {tuple(got.shape)} against {tuple(want.shape)}"
    scale = float(want.abs().max())
    err = float((got.float().cpu() - want).abs().max())
    assert err <= rel * scale, f"{what}: {err:.3g} > {rel * scale:.3g}"


def mostly_close(got, want, mode, what, share=0.97, worst=0.15):
    """32-bit runs: every row within the tolerance.  bfloat16 runs where a unit norm brings a rounded output to full size
    (and layer after layer of it): most rows stay within the tolerance and none strays far.  What a wrong key, state or page
    does shows in the 32-bit run of the same cutting."""
    if mode == "float32":
        return close(got, want, mode, what)
    want = want.float()
    errs = (got.float().cpu() - want).abs().max(dim=1).values / float(want.abs().max())
    within = float((errs <= REL[mode]).float().mean())
    assert within >= share and float(errs.max()) < worst, f"{what}: {within:.3f} of the rows within the tolerance, worst {float(errs.max()):.3g}"


def model_close(got, ref, mode, what):
    if mode == "float32":
        return assert_close(got, ref, mode, what)
    for g, r in zip(got, ref):
        assert g.shape == r.shape
    mostly_close(torch.cat(list(got)), torch.cat(list(ref)), mode, what, share=0.9)


def context(rt, cache, slots, q_lens):
    for s, n in zip(slots, q_lens):
        cache.reserve(s, cache.lengths_host[s] + n)
    cache.flush()
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    cu = [0]
    for n in q_lens:
        cu.append(cu[-1] + n)
    row_seq = [b for b, n in enumerate(q_lens) for _ in range(n)]
    return StepContext(runtime=rt, cache=cache, n_seqs=len(slots), n_rows=cu[-1], max_q_len=max(q_lens),
                       kv_bound=max(cache.lengths_host[s] + n for s, n in zip(slots, q_lens)), seq_slot=i32(slots), cu_q=i32(cu),
                       row_seq=i32(row_seq), lengths=cache.lengths, status=torch.zeros(1, dtype=torch.int32, device="cuda"))


def run_step(rt, parts, cache, slots, pieces):
    """One step of the parts (each a layer of its own) over the sequences' pieces; a list of outputs per part."""
    ctx = context(rt, cache, slots, [len(p) for p in pieces])
    rows = torch.cat(pieces).to(rt.dtype).cuda().contiguous()
    outs = [part.forward(ctx, rows, cache.layers[i]) for i, part in enumerate(parts)]
    rt.ops.advance_lengths(ctx)
    for s, p in zip(slots, pieces):
        cache.advance_host(s, len(p))
    assert int(ctx.status.item()) == 0
    return [o.float().cpu() for o in outs]


def run_parts(rt, parts, h, cuts, pages=16):
    """Mixers, each a layer of its own, over one sequence whose rows h come in pieces of the given sizes; per mixer the
    outputs of all pieces in order."""
    cache = Cache([p.cache_request() for p in parts], n_slots=2, max_tokens=64 * pages, dtype=rt.dtype, device="cuda")
    cache.alloc()                      # the sequence under test sits in the second slot
    slot = cache.alloc()
    outs, at = [], 0
    for n in cuts:
        outs.append(run_step(rt, parts, cache, [slot], [h[at:at + n]]))
        at += n
    return [torch.cat(pieces) for pieces in zip(*outs)]


def run_part(rt, part, h, cuts, pages=16):
    return run_parts(rt, [part], h, cuts, pages)[0]


def cuttings(n):
    """Whole; a tail token by token; portions of two; two unequal portions; around sixteen; every token alone."""
    around = [15, 16, 17, 12, 11, 1, 2]
    return [[n], [n - 9] + [1] * 9, [2] * (n // 2) + [1] * (n % 2), [n // 3, n - n // 3], around + [n - sum(around)], [1] * n]


ROLES = {"q.conv": "q_conv", "k.conv": "k_conv", "v.conv": "v_conv", "dq.norm": "dq_norm", "dkv.norm": "dkv_norm"}


def part_of(rt, spec, w):
    return build_part("mixer", spec, {ROLES.get(k, k): v.to(rt.dtype).cuda() for k, v in w.items()}, rt)


def wide(w):
    return {k: v.double() for k, v in w.items()}


# ---- layer norms, the feed-forward, the capped head ---------------------------------------------------------------

@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("width, rows", [(30, 7), (96, 40), (1024, 33), (1030, 5), (2048, 300), (5000, 3), (16400, 2)])
def test_layer_norm_with_the_residual_sum_in_front(mode, width, rows):
    rt = runtime(mode)
    norm = build_part("norm", LayerNormSpec(size=width, eps=1e-3), {"weight": rand((width,), 1, 0.3, 1.0).cuda(), "bias": rand((width,), 2, 0.5).cuda()}, rt)
    x, delta = rand((rows, width), 3, 2.0, 5.0), rand((rows, width), 4)     # a mean well away from zero
    w, b = norm.weight.double().cpu(), norm.bias.double().cpu()
    rel = 1e-5 if mode == "float32" else 5e-3
    close(norm.forward(x.cuda()), plain.layer_norm(x.double(), w, b, 1e-3), mode, "alone", rel)
    on = x.cuda()
    got = norm.add_forward(on, delta.to(rt.dtype).cuda())
    close(got, plain.layer_norm((x + delta).double(), w, b, 1e-3), mode, "after the sum", rel)
    assert got.dtype == rt.dtype and on.dtype == torch.float32 and torch.equal(on.cpu(), x + delta)


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("width", [30, 96, 1024])
def test_normed_embedding_rows(mode, width):
    rt = runtime(mode)
    norm = build_part("norm", LayerNormSpec(size=width, eps=1e-6), {"weight": rand((width,), 1, 0.3, 1.0).cuda(), "bias": rand((width,), 2).cuda()}, rt)
    table = rand((50, width), 5, 0.02)                                       # rows so small that eps has its share
    tokens = torch.tensor([3, 49, 0, 3], dtype=torch.int32)

    class Step:
        status = torch.zeros(1, dtype=torch.int32, device="cuda")
    got = norm.embed(Step, tokens.cuda(), table.to(rt.dtype).cuda())
    assert got.dtype == torch.float32 and int(Step.status) == 0
    close(got, plain.layer_norm(table[tokens.long()].double(), norm.weight.double().cpu(), norm.bias.double().cpu(), 1e-6), "float32", "rows", 1e-5)
    norm.embed(Step, torch.tensor([50], dtype=torch.int32).cuda(), table.to(rt.dtype).cuda())
    assert int(Step.status) == 1                                             # a token outside the table raises its bit


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("width, ff, rows", [(96, 136, 5), (40, 52, 70), (30, 14, 3), (1024, 2048, 16), (1024, 2048, 1), (1024, 2048, 300)])
def test_gated_gelu_feed_forward_alone(mode, width, ff, rows):
    rt = runtime(mode)
    gate, up, down = rand((ff, width), 3, 2 * width ** -0.5), rand((ff, width), 4, width ** -0.5), rand((width, ff), 5, ff ** -0.5)
    part = build_part("ff", GatedMLPSpec(hidden_size=width, intermediate_size=ff, activation="gelu_tanh"),
                      {"gate": gate.to(rt.dtype).cuda(), "up": up.to(rt.dtype).cuda(), "down": down.to(rt.dtype).cuda()}, rt)
    h = rand((rows, width), 6)
    close(part.forward(None, h.to(rt.dtype).cuda()), plain.feed_forward(h.double(), gate.double(), up.double(), down.double()), mode, "gate, up, down")


def test_gelu_over_its_whole_range():
    ops = runtime("float32").ops
    g = torch.linspace(-12.0, 12.0, 4001)
    got = ops.gated_gelu(torch.stack([g, torch.full_like(g, 1.5)], dim=1).cuda()).cpu()[:, 0]
    want = 1.5 * plain.gelu_tanh(g.double())
    assert float((got.double() - want).abs().max()) < 2e-6


def test_capped_logits():
    ops = runtime("float32").ops
    x = rand((5, 333), 1, 40.0)
    want = 12.0 * torch.tanh(x.double() / 12.0)
    y = x.cuda()
    got = ops.softcap(y, 12.0)
    assert got is y and float((got.cpu().double() - want).abs().max()) < 1e-5


# ---- the delta rule with a decay per key channel -------------------------------------------------------------------

def delta_spec(H, G, D, V, taps, ra=9, rg=6, width=80):
    return ChannelDeltaSpec(hidden_size=width, num_heads=H, num_kv_heads=G, head_dim=D, v_dim=V, taps=taps, decay_rank=ra, gate_rank=rg,
                            norm_eps=EPS)


def delta_weights(s, seed, rate=0.7, bias=-2.0, spread=1.5):
    H, G, D, V, h = s.num_heads, s.num_kv_heads, s.head_dim, s.v_dim, s.hidden_size
    shapes = {"q": (G * D, h), "k": (G * D, h), "v": (H * V, h), "b": (H, h), "a1": (s.decay_rank, h), "a2": (H * D, s.decay_rank),
              "g1": (s.gate_rank, h), "g2": (H * V, s.gate_rank), "o": (h, H * V)}
    w = {n: rand(shape, seed + i, shape[1] ** -0.5) for i, (n, shape) in enumerate(shapes.items())}
    w.update({"q.conv": rand((G * D, s.taps), seed + 20, 0.5, 0.3), "k.conv": rand((G * D, s.taps), seed + 21, 0.5, 0.3),
              "v.conv": rand((H * V, s.taps), seed + 22, 0.5, 0.3), "A_log": rand((H,), seed + 23, rate),
              "dt_bias": rand((H * D,), seed + 24, spread, bias), "norm": rand((V,), seed + 25, 0.2, 1.0)})
    return w


def delta_entry(s):
    return {"heads": s.num_heads, "kv_heads": s.num_kv_heads, "dim": s.head_dim, "vdim": s.v_dim, "conv": s.taps}


def plain_delta(h, w, s):
    return plain.channel_delta(h.double(), wide(w), delta_entry(s), EPS)


DELTA_SIZES = [
    dict(H=6, G=2, D=16, V=24, taps=3),
    dict(H=4, G=4, D=64, V=64, taps=4),
    dict(H=2, G=1, D=128, V=128, taps=4, ra=32, rg=16),
    dict(H=8, G=4, D=64, V=128, taps=2),
    dict(H=1, G=1, D=136, V=12, taps=5),        # more key channels than registers hold
    dict(H=2, G=2, D=10, V=130, taps=8),        # more value columns than one turn covers, a width no 16-byte read fits
    dict(H=3, G=1, D=7, V=5, taps=1),           # one tap keeps no record
    dict(H=2, G=2, D=140, V=150, taps=2),
    dict(H=5, G=5, D=1, V=1, taps=2),           # a scalar state
    dict(H=2, G=1, D=36, V=40, taps=6, ra=8, rg=8),
]


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("sizes", DELTA_SIZES)
def test_delta_rule_alone(mode, sizes):
    rt = runtime(mode)
    spec = delta_spec(**sizes)
    w = delta_weights(spec, 30)
    part = part_of(rt, spec, w)
    n = 100
    h = rand((n, spec.hidden_size), 3)
    want = plain_delta(h, w, spec)
    for cuts in cuttings(n):
        got = run_part(rt, part, h, cuts)
        if spec.v_dim == 1:     # the unit norm of a single value is its sign unless the value is tiny: a rounded input shows in full
            close(got, want, mode, f"cut {cuts[:3]}..", rel=1e-3 if mode == "float32" else 0.3)
        else:
            mostly_close(got, want, mode, f"cut {cuts[:3]}..")


@pytest.mark.parametrize("bias, rate", [(-9.0, 0.1), (6.0, 1.5), (0.0, 2.5)])
def test_decays_from_none_to_all(bias, rate):
    """Channels that keep everything, channels that forget everything at every token, and both side by side; long enough
    for what a summed logarithm would lose to show."""
    rt = runtime("float32")
    spec = delta_spec(H=2, G=2, D=32, V=48, taps=3)
    w = delta_weights(spec, 50, rate=rate, bias=bias, spread=4.0)
    part = part_of(rt, spec, w)
    h = rand((330, 80), 4)
    want = plain_delta(h, w, spec)
    for cuts in ([330], [330 - 120] + [1] * 120, [33] * 10):
        close(run_part(rt, part, h, cuts), want, "float32", f"bias {bias}, cut {cuts[:3]}..")


@pytest.mark.parametrize("at", [0, 3, 14, 15, 16, 17, 31, 40])
def test_a_token_that_wipes_the_state(at):
    """One token's decay is all but zero in every channel (its logarithm in the hundreds), the others' near one: what comes
    after must be as exact as if the sequence had started there, wherever in a chunk that token stands."""
    rt = runtime("float32")
    spec = delta_spec(H=2, G=1, D=24, V=20, taps=2, ra=4, width=48)
    w = delta_weights(spec, 60, rate=0.1, bias=-6.0, spread=0.2)
    w["a1"] = torch.zeros_like(w["a1"])
    w["a1"][0, 0] = 1.0                       # the first input column alone moves the decay
    w["a2"] = torch.zeros_like(w["a2"])
    w["a2"][:, 0] = 1.0
    h = rand((64, 48), 5)
    h[:, 0] = 0.0
    h[at, 0] = 400.0
    want = plain_delta(h, w, spec)
    part = part_of(rt, spec, w)
    for cuts in ([64], [20, 44], [at + 1, 63 - at], [1] * 64):
        close(run_part(rt, part, h, [c for c in cuts if c]), want, "float32", f"wiped at {at}, cut {cuts[:3]}..")


def test_a_write_that_is_read_far_later():
    """The state is a memory: a value written along a key of its own is read back hundreds of tokens later, at every
    distance from the chunk that wrote it; a token's write is read by the same token."""
    rt = runtime("float32")
    D = 16
    spec = delta_spec(H=1, G=1, D=D, V=16, taps=1, ra=2, rg=2, width=40)
    w = delta_weights(spec, 70)
    w = {k: torch.zeros_like(v) for k, v in w.items()}
    w["k"][:, :D], w["q"][:, :D] = torch.eye(D), torch.eye(D)
    w["v"][:, D:2 * D] = torch.eye(16)
    w["b"][0, 2 * D] = 1.0
    w["dt_bias"][:] = -20.0                   # nothing is forgotten
    w["norm"][:], w["o"][:16, :16] = 1.0, torch.eye(16)
    for n in ("q.conv", "k.conv", "v.conv"):
        w[n][:] = 1.0
    n = 300
    h = torch.zeros(n, 40)
    h[:, 2 * D] = -60.0                       # most tokens write nothing ...
    h[5, 0], h[5, D + 3], h[5, 2 * D] = 4.0, 3.0, 60.0       # ... token 5 writes along the first key channel
    h[6:, 0] = 4.0                            # and every later token asks there
    got = run_part(rt, part_of(rt, spec, w), h, [7, 9, 16, 17, 100, 151])
    want = plain_delta(h, w, spec)
    close(got, want, "float32", "far reads")
    assert float(got[:5].abs().max()) < 1e-6 and float(got[5:, 3].min()) > 0.5 * float(got[5, 3]) > 0


@pytest.mark.parametrize("mode", MODES)
def test_long_delta_sequences_keep_their_state(mode):
    rt = runtime(mode)
    spec = delta_spec(H=4, G=2, D=64, V=64, taps=4)
    w = delta_weights(spec, 80, bias=-5.0)
    part = part_of(rt, spec, w)
    n = 900
    h = rand((n, 80), 6)
    want = plain_delta(h, w, spec)
    for cuts in ([n], [n - 300] + [1] * 300, [100] * 9, [13] * 69 + [3]):
        mostly_close(run_part(rt, part, h, cuts, pages=20), want, mode, f"cut {cuts[:3]}..")


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("lengths", [[1, 5, 15, 16, 17, 33, 48, 100], [301, 2, 250, 1, 7, 3, 65, 18]])
def test_unequal_sequences_in_one_step(mode, lengths):
    """Sequences of lengths around sixteen and its multiples (and a step of many rows) in one step, then one token each, then
    unequal pieces again."""
    rt = runtime(mode)
    spec = delta_spec(H=3, G=1, D=32, V=36, taps=4)
    w = delta_weights(spec, 90)
    part = part_of(rt, spec, w)
    seqs = [rand((n + 1 + 19 - i, 80), 100 + i) for i, n in enumerate(lengths)]
    cache = Cache([part.cache_request()], n_slots=8, max_tokens=64 * 24, dtype=rt.dtype, device="cuda")
    slots = [cache.alloc() for _ in seqs]
    got = [[] for _ in seqs]
    at = [0] * len(seqs)
    for take in (lengths, [1] * 8, [len(s) - n - 1 for s, n in zip(seqs, lengths)]):
        out = run_step(rt, [part], cache, slots, [s[a:a + k] for s, a, k in zip(seqs, at, take)])[0]
        for i, piece in enumerate(torch.split(out, take)):
            got[i].append(piece)
        at = [a + k for a, k in zip(at, take)]
    for i, s in enumerate(seqs):
        mostly_close(torch.cat(got[i]), plain_delta(s, w, spec), mode, f"sequence {i}", share=0.9)


def test_delta_records_of_two_sequences_and_a_slot_used_again():
    rt = runtime("float32")
    spec = delta_spec(H=2, G=1, D=16, V=24, taps=4, width=32)
    w = delta_weights(spec, 120)
    part = part_of(rt, spec, w)
    cache = Cache([part.cache_request()], n_slots=2, max_tokens=64 * 8, dtype=rt.dtype, device="cuda")
    a, b, c = rand((41, 32), 1), rand((9, 32), 2), rand((32, 32), 3)
    sa, sb = cache.alloc(), cache.alloc()
    first = run_step(rt, [part], cache, [sa, sb], [a[:20], b[:2]])[0]
    second = run_step(rt, [part], cache, [sb, sa], [b[2:], a[20:]])[0]
    close(torch.cat([first[:20], second[7:]]), plain_delta(a, w, spec), "float32", "first sequence")
    close(torch.cat([first[20:], second[:7]]), plain_delta(b, w, spec), "float32", "second sequence")
    for again in ([32], [1] * 32):
        cache.free(sa)
        assert cache.alloc() == sa
        outs, at = [], 0
        for n in again:
            outs.append(run_step(rt, [part], cache, [sa], [c[at:at + n]])[0])
            at += n
        close(torch.cat(outs), plain_delta(c, w, spec), "float32", "a new sequence in the freed slot")


# ---- attention through latents -------------------------------------------------------------------------------------

STRETCH = dict(factor=4.0, original=64.0, fast=8.0, slow=0.5)


def latent_spec(H, D, R, V, rq, rk, second=False, base=1000.0, stretch=STRETCH, scale=None, kv_from=None, width=80):
    position = (ScaledHalfRopeSpec if second else PairRopeSpec)(theta=base, rotary_dim=R, **(stretch or {}))
    return LatentAttentionSpec(hidden_size=width, num_heads=H, head_dim=D, rot_dim=R, v_dim=V, q_rank=rq, kv_rank=rk,
                               scale=(D + R) ** -0.5 if scale is None else scale, norm_eps=EPS, position=position, head_gate=second,
                               kv_from=kv_from)


def latent_weights(s, seed):
    h, H, D, R, V = s.hidden_size, s.num_heads, s.head_dim, s.rot_dim, s.v_dim
    shapes = {"dq": (s.q_rank, h), "uq": (H * (D + R), s.q_rank), "uk": (H * D, s.kv_rank), "uv": (H * V, s.kv_rank), "o": (h, H * V)}
    if s.kv_from is None:
        shapes["dkv"] = (s.kv_rank + R, h)
    if s.head_gate:
        shapes["g"] = (H, h)
    w = {n: rand(shape, seed + i, shape[1] ** -0.5) for i, (n, shape) in enumerate(shapes.items())}
    w["dq.norm"] = rand((s.q_rank,), seed + 20, 0.2, 1.2)
    if s.kv_from is None:
        w["dkv.norm"] = rand((s.kv_rank,), seed + 21, 0.2, 0.9)
    return w


def latent_entry(s):
    rot = {"base": s.position.theta, "dims": s.position.rotary_dim}
    if s.position.factor is not None:
        rot["scaling"] = {k: getattr(s.position, k) for k in ("factor", "original", "fast", "slow")}
    return {"heads": s.num_heads, "dim": s.head_dim, "rot_dim": s.rot_dim, "vdim": s.v_dim, "kv_rank": s.kv_rank, "scale": s.scale, "rot": rot}


def plain_latent(h, w, s, rows=None):
    """(output, the rows that were read)"""
    return plain.latent_attention(h.double(), wide(w), latent_entry(s), EPS, halves=s.head_gate, gated=s.head_gate, rows=rows)


LATENT_SIZES = [
    dict(H=5, D=24, R=12, V=20, rq=28, rk=44),                                    # the general kernel
    dict(H=2, D=80, R=48, V=64, rq=96, rk=128, base=10000.0),                     # sizes the tensor-core kernels take
    dict(H=16, D=128, R=64, V=128, rq=64, rk=256, stretch=None),
    dict(H=1, D=10, R=2, V=6, rq=12, rk=14, base=100.0, stretch=None),
    dict(H=6, D=40, R=8, V=56, rq=72, rk=64, base=300000.0, stretch=dict(factor=16.0, original=128.0, fast=24.0, slow=2.0), scale=0.3),
    dict(H=3, D=5, R=6, V=7, rq=11, rk=13),
]


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("second", [False, True])
@pytest.mark.parametrize("sizes", LATENT_SIZES)
def test_latent_attention_alone(mode, second, sizes):
    rt = runtime(mode)
    spec = latent_spec(second=second, **sizes)
    w = latent_weights(spec, 20)
    part = part_of(rt, spec, w)
    n = 150
    h = rand((n, spec.hidden_size), 3)
    want, _ = plain_latent(h, w, spec)
    for cuts in cuttings(n):
        close(run_part(rt, part, h, cuts), want, mode, f"cut {cuts[:3]}..")


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("sizes", [dict(rk=48, R=8), dict(rk=128, R=32), dict(rk=15, R=6)])
def test_layers_that_read_another_layers_latents(mode, sizes):
    """A layer with latents of its own and two that read them, with other head counts and sizes; the readers' cache entry is
    the owner's, and its rows are the owner's as they stand in the cache."""
    rt = runtime(mode)
    rk, R = sizes["rk"], sizes["R"]
    own = latent_spec(H=4, D=32, R=R, V=64, rq=40, rk=rk, second=True)
    first = latent_spec(H=8, D=16, R=R, V=24, rq=24, rk=rk, second=True, scale=0.4, kv_from=0)
    second = latent_spec(H=3, D=20, R=R, V=10, rq=56, rk=rk, second=True, kv_from=0)
    specs = [own, first, second]
    weights = [latent_weights(s, 40 + 30 * i) for i, s in enumerate(specs)]
    parts = [part_of(rt, s, w) for s, w in zip(specs, weights)]
    n = 140
    h = rand((n, 80), 5)
    want, rows = plain_latent(h, weights[0], own)
    wants = [want] + [plain_latent(h, w, s, rows)[0] for s, w in zip(specs[1:], weights[1:])]
    for cuts in cuttings(n):
        for i, (got, ref) in enumerate(zip(run_parts(rt, parts, h, cuts), wants)):
            close(got, ref, mode, f"layer {i}, cut {cuts[:3]}..")


@pytest.mark.parametrize("mode", MODES)
def test_a_batch_of_readers_beside_each_request_alone(mode):
    rt = runtime(mode)
    own, reader = latent_spec(H=4, D=32, R=16, V=64, rq=40, rk=64, second=True), latent_spec(H=2, D=48, R=16, V=32, rq=24, rk=64, second=True, kv_from=0)
    weights = [latent_weights(own, 140), latent_weights(reader, 170)]
    parts = [part_of(rt, own, weights[0]), part_of(rt, reader, weights[1])]
    seqs = [rand((n, 80), 150 + n) for n in (70, 3, 131)]
    cache = Cache([p.cache_request() for p in parts], n_slots=3, max_tokens=64 * 8, dtype=rt.dtype, device="cuda")
    slots = [cache.alloc() for _ in seqs]
    steps = [run_step(rt, parts, cache, slots, [s[:len(s) - 2] for s in seqs])] + [run_step(rt, parts, cache, slots, [s[len(s) - k:len(s) - k + 1] for s in seqs])
                                                                                  for k in (2, 1)]
    for i, s in enumerate(seqs):
        want, rows = plain_latent(s, weights[0], own)
        for layer, ref in enumerate((want, plain_latent(s, weights[1], reader, rows)[0])):
            got = torch.cat([torch.split(steps[0][layer], [len(x) - 2 for x in seqs])[i]] + [steps[k][layer][i:i + 1] for k in (1, 2)])
            close(got, ref, mode, f"request {i}, layer {layer}")


def standout(spec, n, at, seed, strength=5.0):
    """Rows and weights in which the key at position ``at`` stands out for every later query of head 0: ordinary rows share
    a direction u, the row at ``at`` is a multiple of another direction z; the first head's key matrix maps the latent of z
    onto the query that u makes.  Seeing or not seeing that key moves the output."""
    h, D, rank = spec.hidden_size, spec.head_dim, spec.kv_rank
    w = latent_weights(spec, seed)
    rows = rand((n, h), seed + 20, 0.05)
    rows[:, 1] = 0.0
    rows[:, 0] += 2.0
    rows[at] = 0.0
    rows[at, 1] = strength
    query = (plain.unit_rms(w["dq"][:, 0].double() * 2.0, EPS) * w["dq.norm"].double()) @ w["uq"][:D].double().T
    latent = plain.unit_rms(w["dkv"][:rank, 1].double() * strength, EPS) * w["dkv.norm"].double()
    w["uk"][:D] += (2.0 * torch.outer(query, latent) / (latent * latent).sum()).float()
    return rows.to(torch.bfloat16).float(), {k: v.to(torch.bfloat16).float() for k, v in w.items()}


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("second", [False, True])
@pytest.mark.parametrize("n, at", [(330, 0), (330, 1), (200, 63), (200, 64), (200, 65), (330, 127), (330, 128), (700, 5), (150, 149)])
def test_a_key_that_stands_out_far_back_and_at_page_borders(mode, second, n, at):
    rt = runtime(mode)
    spec = latent_spec(H=4, D=64, R=16, V=64, rq=96, rk=128, second=second, scale=0.15)
    h, w = standout(spec, n, at, 50)
    want, _ = plain_latent(h, w, spec)
    if 0 < at < n - 1:    # the test can tell: with an ordinary row in the key's place the later outputs move by a good part of their size
        plainer = h.clone()
        plainer[at] = h[at - 1]
        moved = (plain_latent(plainer, w, spec)[0][at + 1:] - want[at + 1:]).abs().mean()
        assert float(moved) > 0.2 * float(want[at + 1:].abs().mean())
    part = part_of(rt, spec, w)
    tail = n - max(at - 1, 1)          # decoding starts one position before the key
    for cuts in ([n], [n - tail] + [1] * tail if tail <= 140 else [n - 40] + [1] * 40, [max(at, 1), n - max(at, 1)]):
        cuts = [c for c in cuts if c > 0]
        close(run_part(rt, part, h, cuts, pages=24), want, mode, f"key at {at}, cut {cuts[:3]}..")


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("rows", [9, 40, 100])
def test_the_gate_shuts_whole_heads(mode, rows):
    """Gates that shut every head but one: what passes is exactly that head's columns, on every path (few rows, a prompt in
    pieces, a whole prompt)."""
    rt = runtime(mode)
    spec = latent_spec(H=4, D=16, R=8, V=24, rq=32, rk=64, second=True, width=96)
    w = latent_weights(spec, 60)
    w["g"] = torch.zeros_like(w["g"])
    w["g"][:, 0] = -60.0
    w["g"][2, 0] = 60.0
    w["o"] = torch.eye(96)                                     # the output shows the heads' columns themselves
    h = rand((rows, 96), 7)
    h[:, 0] = 1.0
    want = plain_latent(h, w, spec)[0]
    for cuts in ([rows], [rows - 5, 5]):
        got = run_part(rt, part_of(rt, spec, w), h, cuts)
        close(got, want, mode, "gated heads")
        assert float(got[:, list(range(48)) + list(range(72, 96))].abs().max()) < 1e-12 and float(got[:, 48:72].abs().max()) > 0.1


def test_gate_heads_alone():
    """Every layout the gate's kernel takes: 16-byte rows and others, a head stride that is not the width."""
    for mode in MODES:
        rt = runtime(mode)
        for rows, H, V in ((70, 3, 8), (5, 7, 24), (33, 2, 5)):
            a, gate = rand((H, rows, V + 8), 1).to(rt.dtype).cuda()[:, :, :V].transpose(0, 1), rand((rows, H + 3), 2).to(rt.dtype).cuda()[:, 1:H + 1]
            want = a.double().cpu() * torch.sigmoid(gate.double().cpu())[:, :, None]
            close(rt.ops.gate_heads(a, gate), want, mode, f"{rows} x {H} x {V}", rel=1e-6 if mode == "float32" else 5e-3)


@pytest.mark.parametrize("second", [False, True])
def test_the_rotation_knows_far_positions(second):
    """Positions in the thousands, with and without stretched frequencies: the kernels' 32-bit angles against 64-bit ones."""
    rt = runtime("float32")
    R, n = 16, 3000
    for stretch in (None, dict(factor=8.0, original=512.0, fast=32.0, slow=1.0)):
        spec = latent_spec(H=1, D=4, R=R, V=4, rq=8, rk=8, second=second, base=10000.0, stretch=stretch)
        part = part_of(rt, spec, latent_weights(spec, 5))
        cache = Cache([part.cache_request()], n_slots=1, max_tokens=64 * 48, dtype=rt.dtype, device="cuda")
        ctx = context(rt, cache, [cache.alloc()], [n])
        x = rand((n, 1, R), 6)
        got = torch.empty((n, 1, R), device="cuda")
        rt.ops.rotate_pairs(ctx, x.cuda(), got, *part.turn)
        close(got, plain.rotate(x.double(), latent_entry(spec)["rot"], second), "float32", "turned rows", rel=2e-4)


# ---- whole models ------------------------------------------------------------------------------------------------

@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    out = {}
    for name in cases.CASES:
        out[name, "bfloat16"] = cases.write_folder(name, tmp_path_factory.mktemp(f"siparax_{name}_bf16"))
        out[name, "float32"] = cases.write_folder(name, tmp_path_factory.mktemp(f"siparax_{name}_f32"), dtype=torch.float32, shards=2)
    return out


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("name", list(cases.CASES))
def test_every_cutting_matches_plain(folders, name, mode):
    folder = folders[name, mode]
    seqs = random_tokens(cases.CASES[name]["vocab"], (5, 90, 41, 1, 64, 65, 2, 130), seed=3)
    ref = cases.plain_logits(folder, seqs)
    sess = make_session(folder, mode, max_tokens=64 * 16, max_seqs=4, max_rows=100)
    model_close(run_whole(sess, seqs), ref, mode, "alone and whole")
    model_close(run_whole(sess, seqs[:4], together=True), ref[:4], mode, "one ragged step")
    model_close(run_tail_by_one(sess, seqs, tail=40), ref, mode, "tail one by one")
    model_close(run_ragged_batches(sess, seqs, batch_size=3, poison=True), ref, mode, "ragged batches, freed pages poisoned")
    assert sess.cache.slots.n_held == 0


@pytest.mark.parametrize("mode", MODES)
def test_portions_down_to_two_tokens(folders, mode):
    seqs = random_tokens(211, (37,), seed=4)
    ref = cases.plain_logits(folders["A", mode], seqs)
    for portion in (2, 3, 7, 16, 21):
        sess = make_session(folders["A", mode], mode, max_tokens=64 * 4, max_seqs=2, max_rows=portion)
        model_close(run_whole(sess, seqs), ref, mode, f"portions of {portion}")


@pytest.mark.parametrize("mode", MODES)
def test_long_decoding_in_a_batch(folders, mode):
    seqs = random_tokens(300, (420, 333), seed=12)
    ref = cases.plain_logits(folders["B", mode], seqs)
    sess = make_session(folders["B", mode], mode, max_tokens=64 * 16, max_seqs=2)
    model_close(run_ragged_batches(sess, seqs, batch_size=2, prefix_fraction=0.2), ref, mode, "hundreds of tokens decoded side by side")


def test_layers_match_plain(folders):
    cfg, tensors = plain.read_folder(folders["A", "float32"])
    tokens = random_tokens(211, (19,), seed=9)[0]
    want = []
    plain.forward(cfg, tensors, tokens, want)
    sess = make_session(folders["A", "float32"], "float32", max_tokens=64 * 4, max_seqs=2)
    seen = []
    for block in sess.model.blocks:
        inner = block.forward

        def spy(ctx, stream, layer_cache, inner=inner):
            inner(ctx, stream, layer_cache)
            seen.append(stream.x + stream.pending)
        block.forward = spy
    run_whole(sess, [tokens])
    assert len(seen) == len(want) == 5
    for i, (got, ref) in enumerate(zip(seen, want)):
        assert float((got.cpu() - ref).abs().max()) <= 2e-5 * float(ref.abs().max()), f"layer {i}"


def test_the_residual_is_32_bit_in_a_bfloat16_run(folders):
    sess = make_session(folders["D", "bfloat16"], "bfloat16", max_tokens=64 * 4, max_seqs=2)
    kinds = []
    for block in sess.model.blocks:
        inner = block.forward

        def spy(ctx, stream, layer_cache, inner=inner):
            inner(ctx, stream, layer_cache)
            kinds.append((stream.x.dtype, stream.pending.dtype))
        block.forward = spy
    run_whole(sess, random_tokens(64, (9,), seed=1))
    assert kinds == [(torch.float32, torch.bfloat16)] * 5


@pytest.mark.parametrize("mode", MODES)
def test_greedy_generation_through_the_entry_point(folders, mode):
    cfg, tensors = plain.read_folder(folders["C", "float32"])
    prompts = random_tokens(97, (3, 11, 1, 30), seed=6)
    want = plain.generate(cfg, tensors, prompts, 12)
    engine = Engine.from_session(make_session(folders["C", "float32"], "float32", max_tokens=64 * 8, max_seqs=4))   # graphs on
    assert engine.generate_all(prompts, 12) == want
    assert engine.session.cache.slots.n_held == 0
    engine = Engine.from_session(make_session(folders["C", "float32"], "float32", max_tokens=64 * 8, max_seqs=4), use_graphs=False)
    assert engine.generate_all(prompts, 12) == want
    if mode == "bfloat16":      # rounding may turn a close call: every request still ends with its tokens
        engine = Engine.from_session(make_session(folders["A", "bfloat16"], "bfloat16", max_tokens=64 * 8, max_seqs=4))
        got = engine.generate_all(prompts, 12)
        assert [len(g) for g in got] == [12] * 4 and engine.session.cache.slots.n_held == 0


def test_the_trace_runner_replays_this_design(folders, tmp_path):
    import json
    import subprocess
    import sys
    from pathlib import Path
    import numpy as np
    root = Path(__file__).resolve().parent.parent
    folder = folders["D", "float32"]
    seqs = random_tokens(64, (20, 9), seed=2)
    ref = cases.plain_logits(folder, seqs)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": seqs[0][:15], "want": [14]}, {"id": "b", "tokens": seqs[1][:8], "want": [0, 7]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": seqs[0][15:16], "want": [0]}, {"id": "b", "tokens": seqs[1][8:9], "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": seqs[0][16:17], "want": []}], "end": []},
             {"step": 3, "entries": [{"id": "a", "tokens": seqs[0][17:20], "want": [2]}], "end": ["a"]}]
    proc = subprocess.run([sys.executable, str(root / "bin" / "trace_run"), "--model", str(folder), "--dtype", "float32", "--out", str(tmp_path),
                           "--max-tokens", "64"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert proc.stdout.split() == ["done", "0", "done", "1", "done", "2", "done", "3"] and not (tmp_path / "2.f32").exists()
    read = lambda i: torch.from_numpy(np.fromfile(tmp_path / f"{i}.f32", dtype="<f4").reshape(-1, 64).copy())
    want = {0: torch.stack([ref[0][14], ref[1][0], ref[1][7]]), 1: torch.stack([ref[0][15], ref[1][8]]), 3: ref[0][19:20]}
    for i, r in want.items():
        assert float((read(i) - r).abs().max()) <= 1e-4 * float(r.abs().max()), f"step {i}"
