"""Nifalorn on the GPU against the plain implementation: every mechanism alone, then whole models in every way of cutting
the work; a token that a slow decay has to carry far, a loud key at chunk and page edges, decays that forget everything
beside decays that forget nothing; states of several sequences and of a slot that is used again; routing inside groups;
long decoding; and greedy generation through the entry point."""

import pytest
import torch

import nifalorn_cases as cases
from conftest import random_tokens
from emulated_ops import EmulatedOps
from helpers import assert_close, make_session, run_ragged_batches, run_tail_by_one, run_whole
from plain import nifalorn_plain as plain
from starter_b200.cache import Cache, StateRequest
from starter_b200.config import DiffAttentionSpec, GatedMLPSpec, LightningSpec, Mamba2Spec, MoESpec, PairRopeSpec
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
    scale = float(want.abs().max())
    err = float((got.float().cpu() - want).abs().max())
    assert err <= rel * scale, f"{what}: {err:.3g} > {rel * scale:.3g}"


def mostly_close(got, want, mode, what, share=0.95, worst=0.15):
    """32-bit runs: every row within the tolerance.  bfloat16 runs of a norm over a few columns, whose sum of squares may
    nearly vanish and bring a rounded gate to full size: most rows within it and none far away."""
    if mode == "float32":
        return close(got, want, mode, what)
    want = want.float()
    errs = (got.float().cpu() - want).abs().max(dim=1).values / float(want.abs().max())
    within = float((errs <= REL[mode]).float().mean())
    assert within >= share and float(errs.max()) < worst, f"{what}: {within:.3f} of the rows within the tolerance, worst {float(errs.max()):.3g}"


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


def run_part(rt, part, h, cuts, pages=16, max_step_tokens=1024):
    """A mixer with its cache entries over one sequence whose rows h come in pieces of the given sizes; the outputs of
    all pieces in order."""
    cache = Cache([part.cache_request()], n_slots=2, max_tokens=64 * pages, dtype=rt.dtype, device="cuda", max_step_tokens=max_step_tokens)
    cache.alloc()                      # the sequence under test sits in the second slot
    slot = cache.alloc()
    outs, at = [], 0
    pieces = [min(cache.step_limit, n - lo) for n in cuts for lo in range(0, n, cache.step_limit)]   # as the step function cuts
    for n in pieces:
        ctx = context(rt, cache, [slot], [n])
        outs.append(part.forward(ctx, h[at:at + n].to(rt.dtype).cuda().contiguous(), cache.layers[0]))
        rt.ops.advance_lengths(ctx)
        cache.advance_host(slot, n)
        assert int(ctx.status.item()) == 0
        at += n
    return torch.cat(outs)


def cuttings(n):
    """Whole; a tail token by token; portions of two; two unequal portions; every token alone."""
    return [[n], [n - 9] + [1] * 9, [2] * (n // 2) + [1] * (n % 2), [n // 3, n - n // 3], [1] * n]


ROLES = {"conv.b": "conv_bias"}


def part_of(rt, spec, w):
    return build_part("mixer", spec, {ROLES.get(k, k): v.to(rt.dtype).cuda() for k, v in w.items()}, rt)


def doubles(w):
    return {k: v.double() for k, v in w.items()}


# ---- the recurrence itself: token by token and 64 tokens at a time ---------------------------------------------

def scan_sizes():
    return [(2, 2, 32, 64, [1]), (2, 1, 32, 48, [5, 20]), (4, 2, 64, 64, [70, 3, 130]), (3, 3, 20, 12, [100]), (4, 1, 128, 64, [200, 64, 65]),
            (1, 1, 136, 10, [90]), (2, 2, 256, 72, [70]), (4, 4, 7, 5, [33]), (2, 2, 300, 40, [40]), (6, 3, 16, 8, [64, 63, 1, 16, 128]), (2, 2, 64, 40, [700, 65, 321])]


@pytest.mark.parametrize("mode, runs", [("float32", None), ("bfloat16", 1), ("bfloat16", 3), ("bfloat16", None)])
@pytest.mark.parametrize("sizes", scan_sizes())
@pytest.mark.parametrize("kind", ["constant", "step"])
def test_the_recurrence_and_its_record(monkeypatch, mode, runs, sizes, kind):
    """Ragged sequences in slots out of order, records that hold something already: outputs and records against the torch
    restatement in 32-bit.  In bfloat16 the inputs are bfloat16 numbers and everything else stays 32-bit, so the two agree
    far beyond bfloat16.  ``runs``: how many shares a sequence's chunks of 64 tokens are dealt out in (None: as the rule
    says)."""
    rt = runtime(mode)
    monkeypatch.setattr(rt.ops, "force_decay_runs", runs)
    H, G, D, V, lens = sizes
    rows = sum(lens)
    cache = Cache([StateRequest((4,))], n_slots=len(lens) + 1, max_tokens=64 * 16, dtype=rt.dtype, device="cuda")
    ctx = context(rt, cache, [cache.alloc() for _ in lens][::-1], lens)
    p = rand((rows, 2 * G * D + 2 * H * V), 1).to(rt.dtype).cuda()
    state = rand((len(lens) + 2, H * D * V), 2).cuda()
    other = state.clone()
    if kind == "constant":
        d = torch.tensor([0.9, 0.0, 1.0, 0.999, 0.5, 0.97][:H])
        options, cols = dict(decay=torch.stack([d, torch.log2(d).clamp(min=-160.0)]).cuda()), (0, G * D, 2 * G * D)
    else:
        options = dict(step=(rand((rows, H), 3, 2.0).cuda(), rand((H,), 4).cuda(), torch.exp(rand((H,), 5)).cuda()), skip=rand((H,), 6).cuda())
        cols = (H * V + G * D, H * V, 0)          # values first, keys, queries
    got = rt.ops.decay_scan(ctx, p, *cols, state, H, G, D, V, **options)
    want = EmulatedOps().decay_scan(ctx, p, *cols, other, H, G, D, V, **options)
    assert got.dtype == torch.float32
    close(got, want.cpu(), mode, "outputs", rel=3e-5)
    close(state, other.cpu(), mode, "records", rel=3e-5)


def test_a_chunk_with_strong_decays_keeps_its_weak_ones_apart():
    """Tokens that forget everything between tokens that forget almost nothing, inside the same 64: the logarithms' sum
    reaches hundreds while the differences between neighbours are thousandths."""
    rt = runtime("bfloat16")
    H, D, V, n = 2, 64, 32, 192
    cache = Cache([StateRequest((4,))], n_slots=2, max_tokens=64 * 8, dtype=rt.dtype, device="cuda")
    ctx = context(rt, cache, [cache.alloc()], [n])
    p = rand((n, 2 * H * D + H * V), 1).to(rt.dtype).cuda()
    dt = torch.full((n, H), -6.0)
    dt[3::11] = 40.0
    state = torch.zeros(3, H * D * V, device="cuda")
    other = state.clone()
    options = dict(step=(dt.cuda(), torch.zeros(H, device="cuda"), torch.tensor([1.0, 0.3], device="cuda")))
    got = rt.ops.decay_scan(ctx, p, 0, H * D, 2 * H * D, state, H, H, D, V, **options)
    want = EmulatedOps().decay_scan(ctx, p, 0, H * D, 2 * H * D, other, H, H, D, V, **options)
    weak = [t for t in range(n) if t % 11 not in (3,)]
    for t0 in range(0, n, 11):                    # each stretch against its own size
        rows = [t for t in weak if t0 <= t < t0 + 11]
        close(got[rows], want[rows].cpu(), "bfloat16", f"rows {rows[0]}..", rel=1e-4)
    close(state, other.cpu(), "bfloat16", "record", rel=1e-4)


# ---- lightning attention ---------------------------------------------------------------------------------------

def light_spec(decay, D, V, width=80):
    return LightningSpec(hidden_size=width, num_heads=len(decay), head_dim=D, v_dim=V, decay=tuple(decay), norm_eps=EPS)


def light_weights(s, seed):
    H, D, V, h = s.num_heads, s.head_dim, s.v_dim, s.hidden_size
    return {"q": rand((H * D, h), seed, h ** -0.5), "k": rand((H * D, h), seed + 1, h ** -0.5), "v": rand((H * V, h), seed + 2, h ** -0.5),
            "g": rand((H * V, h), seed + 3, h ** -0.5), "o": rand((h, H * V), seed + 4, (H * V) ** -0.5), "norm": rand((H * V,), seed + 5, 0.2, 1.0)}


def plain_light(h, w, s):
    m = {"heads": s.num_heads, "dim": s.head_dim, "vdim": s.v_dim, "decay": list(s.decay)}
    return plain.lightning_attention(h.double(), doubles(w), m, EPS)


LIGHT_SIZES = [([0.9, 0.5, 0.99], 16, 24), ([0.7, 0.999], 64, 64), ([0.0, 1.0], 20, 12), ([0.95, 0.2, 0.8, 0.9], 128, 128), ([0.6], 200, 130),
               ([0.6, 0.97, 0.8], 7, 5), ([0.99] * 6, 32, 48)]


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("sizes", LIGHT_SIZES)
def test_lightning_attention_alone(mode, sizes):
    rt = runtime(mode)
    spec = light_spec(*sizes)
    w = light_weights(spec, 10)
    part = part_of(rt, spec, w)
    n = 150
    h = rand((n, spec.hidden_size), 3)
    want = plain_light(h, w, spec)
    for cuts in cuttings(n):
        close(run_part(rt, part, h, cuts), want, mode, f"cut {cuts[:3]}..")


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("at", [0, 1, 63, 64, 127, 128, 190])
def test_a_token_that_a_slow_decay_carries_far(mode, at):
    """One token's input is many times larger than the others': hundreds of positions later a head with a decay near one still
    reads it, whatever chunk or step it stood in."""
    rt = runtime(mode)
    spec = light_spec([0.9995, 0.3], 64, 64)
    w = light_weights(spec, 20)
    n = 460
    h = rand((n, spec.hidden_size), 4)
    quiet = plain_light(h, w, spec)
    h[at] *= 24.0
    want = plain_light(h, w, spec)
    assert float((want[-1] - quiet[-1]).abs().max()) > 0.05 * float(want[-1].abs().max())     # the test can tell
    part = part_of(rt, spec, w)
    for cuts in ([n], [n - 100] + [1] * 100, [at + 1, n - at - 1], [at + 3] + [50] * 5 + [n - at - 253]):
        got = run_part(rt, part, h, cuts)
        for pos in (at, min(at + 1, n - 1), n // 2, n - 1):
            close(got[pos:pos + 1], want[pos:pos + 1], mode, f"token {at}, cut {cuts[:3]}.., position {pos}", rel=REL[mode] if mode == "float32" else 5e-2)


# ---- Mamba-2 ---------------------------------------------------------------------------------------------------

def mamba_spec(H, V, N, G, taps, parts, width=80):
    return Mamba2Spec(hidden_size=width, num_heads=H, v_dim=V, state=N, groups=G, taps=taps, norm_groups=parts, norm_eps=EPS)


def mamba_weights(s, seed, dt_scale=1.0):
    H, V, N, G, h = s.num_heads, s.v_dim, s.state, s.groups, s.hidden_size
    inner, bc = H * V, G * N
    w = {"in": rand((2 * inner + 2 * bc + H, h), seed, h ** -0.5), "conv": rand((inner + 2 * bc, s.taps), seed + 1, 0.5, 0.2),
         "conv.b": rand((inner + 2 * bc,), seed + 2, 0.3), "dt_bias": rand((H,), seed + 3, 1.0, -1.5), "A_log": rand((H,), seed + 4, 0.7),
         "D": rand((H,), seed + 5, 0.2, 1.0), "norm": rand((inner,), seed + 6, 0.2, 1.0), "o": rand((h, inner), seed + 7, inner ** -0.5)}
    w["in"][2 * inner + 2 * bc:] *= dt_scale
    return w


def plain_mamba(h, w, s):
    m = {"heads": s.num_heads, "vdim": s.v_dim, "state": s.state, "groups": s.groups, "conv": s.taps, "norm_groups": s.norm_groups}
    return plain.mamba2(h.double(), doubles(w), m, EPS)


MAMBA_SIZES = [(6, 16, 24, 3, 3, 2), (8, 64, 128, 2, 4, 4), (1, 10, 136, 1, 1, 1), (3, 4, 12, 3, 7, 6), (2, 72, 80, 2, 2, 3), (4, 3, 9, 2, 4, 3),
               (4, 48, 32, 4, 4, 2), (2, 128, 256, 1, 5, 1)]


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("sizes", MAMBA_SIZES)
def test_mamba2_alone(mode, sizes):
    rt = runtime(mode)
    spec = mamba_spec(*sizes)
    w = mamba_weights(spec, 30)
    part = part_of(rt, spec, w)
    n = 150
    h = rand((n, spec.hidden_size), 3)
    want = plain_mamba(h, w, spec)
    small_parts = spec.num_heads * spec.v_dim // spec.norm_groups < 8
    for cuts in cuttings(n):
        (mostly_close if small_parts else close)(run_part(rt, part, h, cuts), want, mode, f"cut {cuts[:3]}..")


@pytest.mark.parametrize("mode", MODES)
def test_step_sizes_that_swing_over_a_long_sequence(mode):
    """Step sizes from nearly none to large, hundreds of tokens: heads forget everything at some tokens and hold on at others."""
    rt = runtime(mode)
    spec = mamba_spec(4, 32, 64, 2, 4, 2)
    w = mamba_weights(spec, 40, dt_scale=5.0)
    part = part_of(rt, spec, w)
    n = 600
    h = rand((n, spec.hidden_size), 5)
    want = plain_mamba(h, w, spec)
    for cuts in ([n], [n - 200] + [1] * 200, [33] * 18 + [6], [300, 17, 283]):
        close(run_part(rt, part, h, cuts), want, mode, f"cut {cuts[:3]}..")


@pytest.mark.parametrize("mode", MODES)
def test_first_tokens_and_records_of_a_convolution(mode):
    """Steps shorter than the convolution reaches back, from the first token on: zeros before the start, then the record."""
    rt = runtime(mode)
    spec = mamba_spec(2, 8, 16, 1, 6, 2, width=32)
    w = mamba_weights(spec, 50)
    h = rand((12, 32), 6, 2.0)
    want = plain_mamba(h, w, spec)
    for cuts in ([1] * 12, [2, 1, 3, 1, 5], [3, 9], [12]):
        close(run_part(rt, part_of(rt, spec, w), h, cuts), want, mode, f"cut {cuts}")


@pytest.mark.parametrize("rows", [5, 40, 300])
@pytest.mark.parametrize("which", ["lightning", "mamba2"])
def test_records_of_two_sequences_and_a_slot_used_again(which, rows):
    """Two sequences side by side in one step, each with its own records; then the first slot is freed and taken by a new
    sequence, which must start from zeros."""
    rt = runtime("float32")
    if which == "mamba2":
        spec = mamba_spec(4, 8, 16, 2, 4, 2, width=32)
        w, oracle = mamba_weights(spec, 60), plain_mamba
    else:
        spec = light_spec([0.9, 0.99], 16, 24, width=32)
        w, oracle = light_weights(spec, 60), plain_light
    part = part_of(rt, spec, w)
    cache = Cache([part.cache_request()], n_slots=2, max_tokens=64 * 16, dtype=rt.dtype, device="cuda")
    a, b, c = rand((rows + 11, 32), 1), rand((9, 32), 2), rand((12, 32), 3)
    sa, sb = cache.alloc(), cache.alloc()

    def step(slots, pieces):
        ctx = context(rt, cache, slots, [len(p) for p in pieces])
        out = part.forward(ctx, torch.cat(pieces).cuda(), cache.layers[0])
        rt.ops.advance_lengths(ctx)
        for s, p in zip(slots, pieces):
            cache.advance_host(s, len(p))
        return out.cpu()

    first = step([sa, sb], [a[:rows], b[:2]])
    second = step([sb, sa], [b[2:], a[rows:]])
    close(torch.cat([first[:rows], second[7:]]), oracle(a, w, spec), "float32", "first sequence")
    close(torch.cat([first[rows:], second[:7]]), oracle(b, w, spec), "float32", "second sequence")
    cache.free(sa)
    assert cache.alloc() == sa
    close(step([sa], [c]), oracle(c, w, spec), "float32", "a new sequence in the freed slot")


# ---- attention with two score maps over the query's chunk --------------------------------------------------------

def diff_spec(H, G, D, V, diff=0.5, chunk=None, rot=None, scaling=None, scale=None, width=80):
    position = None
    if rot is not None:
        stretch = dict(zip(("factor", "low", "high", "original"), scaling)) if scaling else {}
        position = PairRopeSpec(theta=rot[0], rotary_dim=rot[1], **stretch)
    return DiffAttentionSpec(hidden_size=width, num_heads=H, num_kv_heads=G, head_dim=D, v_dim=V, scale=D ** -0.5 if scale is None else scale,
                             diff=diff, norm_eps=EPS, chunk=chunk, position=position)


def diff_weights(s, seed):
    H, G, D, V, h = s.num_heads, s.num_kv_heads, s.head_dim, s.v_dim, s.hidden_size
    w = {"q": rand((H * 2 * D, h), seed, h ** -0.5), "k": rand((G * 2 * D, h), seed + 1, h ** -0.5), "v": rand((G * V, h), seed + 2, h ** -0.5),
         "o": rand((h, H * V), seed + 3, (H * V) ** -0.5)}
    w.update({n: rand((D,), seed + 4 + i, 0.15) for i, n in enumerate(("lq1", "lk1", "lq2", "lk2"))})
    return w


def plain_diff(h, w, s):
    m = {"heads": s.num_heads, "kv_heads": s.num_kv_heads, "dim": s.head_dim, "vdim": s.v_dim, "scale": s.scale, "diff": s.diff}
    if s.chunk:
        m["mask"] = {"size": s.chunk}
    p = s.position
    if p is not None:
        m["rot"] = {"base": p.theta, "dims": p.rotary_dim}
        if p.factor is not None:
            m["rot"]["scaling"] = {"factor": p.factor, "low": p.low, "high": p.high, "original": p.original}
    return plain.diff_attention(h.double(), doubles(w), m, EPS)


DIFF_SIZES = [
    dict(H=6, G=2, D=16, V=24, diff=0.7, chunk=24, rot=(1e4, 12), scaling=(8.0, 1.0, 4.0, 64), scale=0.4),   # the general kernel
    dict(H=8, G=2, D=32, V=64, chunk=64, rot=(5e5, 32), scaling=(16.0, 1.0, 4.0, 256)),                     # the tensor-core kernels, chunks of a page
    dict(H=2, G=1, D=64, V=128, diff=0.8, chunk=100, rot=(1e4, 8)),                                         # part of a head turns
    dict(H=1, G=1, D=20, V=12, diff=0.9),                                                                   # no chunk, nothing turned
    dict(H=4, G=4, D=128, V=128, diff=0.3, chunk=17, rot=(1e4, 128), scaling=(2.0, 0.5, 2.0, 40)),
    dict(H=4, G=2, D=32, V=64, chunk=1, rot=(1e4, 16)),                                                     # a query sees itself only
    dict(H=12, G=1, D=5, V=7, diff=0.35, chunk=130, rot=(50.0, 4)),
    dict(H=3, G=3, D=32, V=64, chunk=33, rot=(1e4, 2)),
]


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("sizes", DIFF_SIZES)
def test_two_map_attention_over_chunks_alone(mode, sizes):
    rt = runtime(mode)
    spec = diff_spec(**sizes)
    w = diff_weights(spec, 70)
    part = part_of(rt, spec, w)
    n = 150
    h = rand((n, spec.hidden_size), 3)
    want = plain_diff(h, w, spec)
    for cuts in cuttings(n):
        close(run_part(rt, part, h, cuts, max_step_tokens=48), want, mode, f"cut {cuts[:3]}..")    # rings of pages wrap


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("chunk, loud", [(48, 95), (48, 96), (64, 63), (64, 64), (64, 127), (64, 190), (7, 62), (100, 99), (100, 100), (128, 3), (1, 64), (None, 2)])
def test_a_loud_key_at_chunk_and_page_edges(mode, chunk, loud):
    """One token's input is many times larger than the others', so its key takes a map's softmax wherever that map's score with
    it is positive: the last query of the chunk still sees it, the first one of the next chunk does not, in a prompt and
    decoded one by one."""
    rt = runtime(mode)
    spec = diff_spec(H=8, G=4, D=32, V=64, chunk=chunk, rot=(1e4, 32))
    w = diff_weights(spec, 80)
    part = part_of(rt, spec, w)
    edge = 420 if chunk is None else (loud // chunk + 1) * chunk        # the first query that no longer sees the loud key
    n = edge + 9
    h = rand((n, 80), 5)
    quiet = plain_diff(h, w, spec)
    h[loud] *= 25.0
    want = plain_diff(h, w, spec)
    if loud < edge - 1:
        assert float((want[edge - 1] - quiet[edge - 1]).abs().max()) > 0.05 * float(want.abs().max())
    if chunk is not None:
        assert float((want[edge:] - quiet[edge:]).abs().max()) < 1e-9
    for cuts in ([n], [loud] + [1] * (n - loud) if n - loud <= 140 else [n - 20] + [1] * 20, [edge, n - edge], [edge - 1, 2, n - edge - 1], [loud + 1, n - loud - 1]):
        got = run_part(rt, part, h, cuts)
        for pos in (loud, edge - 1, edge, n - 1):
            if pos == loud and mode == "bfloat16":      # the loud query's own scores: a rounding of 1/256 of hundreds
                continue
            close(got[pos:pos + 1], want[pos:pos + 1], mode, f"chunk {chunk}, loud {loud}, cut {cuts[:2]}, position {pos}",
                  rel=REL[mode] * float(want.abs().max()) / float(want[pos].abs().max()))


# ---- the mixture of experts ----------------------------------------------------------------------------------------

def moe_spec(width, E, top, ff, groups=(1, 1), scale=1.0, shared=None):
    gated = lambda n: GatedMLPSpec(hidden_size=width, intermediate_size=n)
    return MoESpec(hidden_size=width, n_experts=E, n_identity=0, top=top, route_scale=scale, expert=gated(ff),
                   shared=gated(shared) if shared else None, scores="sigmoid", groups=groups[0], keep_groups=groups[1], shared_gate=bool(shared))


def moe_weights(s, seed):
    h, ff, E = s.hidden_size, s.expert.intermediate_size, s.n_experts
    w = {"router": rand((E, h), seed, 2.0 * h ** -0.5), "correction": rand((E,), seed + 1, 0.3, -0.6)}      # most choice scores are negative
    for e in range(E):
        w.update({f"e{e}.gate": rand((ff, h), seed + 2 + 3 * e, h ** -0.5), f"e{e}.up": rand((ff, h), seed + 3 + 3 * e, h ** -0.5),
                  f"e{e}.down": rand((h, ff), seed + 4 + 3 * e, ff ** -0.5)})
    if s.shared is not None:
        f = s.shared.intermediate_size
        w.update({"shared.gate": rand((f, h), seed + 201, h ** -0.5), "shared.up": rand((f, h), seed + 202, h ** -0.5),
                  "shared.down": rand((h, f), seed + 203, f ** -0.5), "shared.sg": rand((1, h), seed + 204, 2.0 * h ** -0.5)})
    return w


def moe_entry(s):
    m = {"router": {"experts": s.n_experts, "top": s.top, "scale": s.route_scale, "groups": {"count": s.groups, "keep": s.keep_groups}}}
    if s.shared is not None:
        m["shared"] = {"ff": s.shared.intermediate_size}
    return m


MOE_SIZES = [dict(width=72, E=12, top=3, ff=40, groups=(3, 2), scale=1.7, shared=56), dict(width=128, E=8, top=2, ff=96, groups=(4, 2), shared=128),
             dict(width=40, E=4, top=2, ff=24, groups=(4, 3)), dict(width=64, E=3, top=3, ff=16, scale=1.3), dict(width=30, E=6, top=6, ff=10, groups=(2, 2), shared=14),
             dict(width=256, E=64, top=8, ff=64, groups=(8, 3), scale=2.5, shared=96), dict(width=64, E=9, top=1, ff=8, groups=(3, 1), shared=24),
             dict(width=48, E=80, top=5, ff=8, groups=(40, 6), shared=16)]


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("sizes", MOE_SIZES)
@pytest.mark.parametrize("rows", [1, 5, 40, 300])     # a few pairs: every pair streams its expert; many (bfloat16): pairs in the order of their experts
def test_experts_alone(mode, sizes, rows):
    rt = runtime(mode)
    spec = moe_spec(**sizes)
    w = moe_weights(spec, 90)
    roles = {k.replace(".", "_"): v.to(rt.dtype).cuda() for k, v in w.items()}
    part = build_part("ff", spec, roles, rt)
    h = rand((rows, spec.hidden_size), 9)
    chosen, weights = plain.route(h.double(), w["router"].double(), w["correction"].double(), moe_entry(spec)["router"])
    got = rt.ops.moe_route(h.to(rt.dtype).cuda(), part.router, part.correction, spec.top, spec.route_scale, scores="sigmoid",
                           groups=spec.groups, keep_groups=spec.keep_groups, extra=int(spec.shared_gate))
    assert torch.equal(got[0].long().cpu().sort(dim=1).values, chosen.sort(dim=1).values)      # the inputs are bfloat16 numbers: no close call
    order = torch.argsort(got[0].long().cpu(), dim=1), torch.argsort(chosen, dim=1)
    close(torch.gather(got[1].cpu(), 1, order[0]), torch.gather(weights, 1, order[1]), "float32", "weights", rel=1e-5)
    if spec.shared_gate:
        close(got[2], h.double() @ w["shared.sg"].double().T, "float32", "the shared expert's gate, before its sigmoid", rel=1e-5)
    close(part.forward(None, h.to(rt.dtype).cuda()), plain.expert_mixture(h.double(), doubles(w), moe_entry(spec)), mode, f"{rows} rows")


def test_groups_are_ranked_by_their_two_best_and_the_rest_is_out_of_reach():
    """Choice scores below zero: an output of a dropped group must not come in with 0.  Group 1 has the single best output,
    group 0 and 2 the best pairs."""
    rt = runtime("float32")
    s = torch.tensor([0.60, 0.58, 0.10, 0.90, 0.05, 0.02, 0.70, 0.55, 0.20])
    router = torch.zeros(9, 16)
    router[:, 0] = torch.logit(s)
    h = torch.zeros(3, 16)
    h[:, 0] = 1.0
    correction = torch.full((9,), -2.0)
    chosen, weight = rt.ops.moe_route(h.cuda(), router.cuda(), correction.cuda(), 5, 2.0, scores="sigmoid", groups=3, keep_groups=2)
    assert chosen.tolist() == [[6, 0, 1, 7, 8]] * 3
    want = s[[6, 0, 1, 7, 8]] / s[[6, 0, 1, 7, 8]].sum() * 2.0      # the weights use the scores without the correction
    close(weight[0], want, "float32", "weights", rel=1e-6)
    correction[3] = 1.0                                              # the correction moves a group's rank
    chosen, _ = rt.ops.moe_route(h.cuda(), router.cuda(), correction.cuda(), 2, 2.0, scores="sigmoid", groups=3, keep_groups=1)
    assert chosen.tolist() == [[3, 4]] * 3
    equal = torch.zeros(6, 16)
    chosen, _ = rt.ops.moe_route(h.cuda(), equal.cuda(), None, 2, 1.0, scores="sigmoid", groups=3, keep_groups=2)
    assert chosen.tolist() == [[0, 1]] * 3                           # of equals the first


# ---- whole models ------------------------------------------------------------------------------------------------

@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    out = {}
    for name in cases.CASES:
        out[name, "bfloat16"] = cases.write_folder(name, tmp_path_factory.mktemp(f"nifalorn_{name}_bf16"), steady=True)
        out[name, "float32"] = cases.write_folder(name, tmp_path_factory.mktemp(f"nifalorn_{name}_f32"), dtype=torch.float32, shards=2)
    return out


def model_close(got, ref, mode, what, share=0.9, rel=3e-2):
    """bfloat16 (folders whose corrections choose the experts): most rows stay within rounding of the plain result, and no
    row strays far."""
    if mode == "float32":
        return assert_close(got, ref, mode, what)
    scale = max(float(r.abs().max()) for r in ref)
    errs = torch.cat([(g - r).abs().max(dim=1).values for g, r in zip(got, ref)]) / scale
    assert float((errs <= rel).float().mean()) >= share and float(errs.max()) < 0.5, \
        f"{what}: {float((errs <= rel).float().mean()):.2f} of the rows within {rel}, worst {float(errs.max()):.3g}"


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("name", list(cases.CASES))
def test_every_cutting_matches_plain(folders, name, mode):
    folder = folders[name, mode]
    seqs = random_tokens(cases.CASES[name]["vocab"], (5, 150, 41, 1, 64, 65, 2), seed=3)
    ref = cases.plain_logits(folder, seqs)
    sess = make_session(folder, mode, max_tokens=64 * 16, max_seqs=4, max_step_tokens=70, max_rows=100)
    model_close(run_whole(sess, seqs), ref, mode, "alone and whole")
    model_close(run_whole(sess, seqs[:4], together=True), ref[:4], mode, "one ragged step")
    model_close(run_tail_by_one(sess, seqs, tail=40), ref, mode, "tail one by one")
    model_close(run_ragged_batches(sess, seqs, batch_size=3, poison=True), ref, mode, "ragged batches, freed pages poisoned")
    assert sess.cache.slots.n_held == 0


@pytest.mark.parametrize("mode", MODES)
def test_portions_down_to_two_tokens(folders, mode):
    seqs = random_tokens(211, (67,), seed=4)
    ref = cases.plain_logits(folders["A", mode], seqs)
    for portion in (2, 3, 7, 20, 33):
        sess = make_session(folders["A", mode], mode, max_tokens=64 * 4, max_seqs=2, max_step_tokens=portion)
        model_close(run_whole(sess, seqs), ref, mode, f"portions of {portion}", share=0.85)


@pytest.mark.parametrize("mode", MODES)
def test_a_batch_against_each_request_alone_through_long_decoding(folders, mode):
    """Three unequal requests decoded together (chunks end on decoded tokens, rings of pages wrap) against the plain model on
    each alone."""
    seqs = random_tokens(300, (330, 230, 171), seed=7)
    ref = cases.plain_logits(folders["B", mode], seqs)
    sess = make_session(folders["B", mode], mode, max_tokens=64 * 16, max_seqs=3, max_step_tokens=128)
    model_close(run_ragged_batches(sess, seqs, batch_size=3, prefix_fraction=0.3), ref, mode, "batch of three, decoded together")


def test_layer_runs_match_plain(folders):
    cfg, tensors = plain.read_folder(folders["A", "float32"])
    tokens = random_tokens(211, (29,), seed=9)[0]
    want = []
    plain.forward(cfg, tensors, tokens, want)
    sess = make_session(folders["A", "float32"], "float32", max_tokens=64 * 4, max_seqs=2)
    seen = []
    for block in sess.model.blocks:
        inner = block.forward

        def spy(ctx, stream, layer_cache, inner=inner):
            inner(ctx, stream, layer_cache)
            seen.append(stream.x + stream.pending)      # the last branch's output waits for the next norm
        block.forward = spy
    run_whole(sess, [tokens])
    assert len(seen) == len(want) == 8
    for i, (got, ref) in enumerate(zip(seen, want)):
        assert got.dtype == torch.float32
        assert float((got.cpu() - ref).abs().max()) <= 2e-5 * float(ref.abs().max()), f"layer run {i}"


def test_the_residual_is_32_bit_in_a_bfloat16_run(folders):
    sess = make_session(folders["D", "bfloat16"], "bfloat16", max_tokens=64 * 4, max_seqs=2)
    kinds = []
    for block in sess.model.blocks:
        inner = block.forward

        def spy(ctx, stream, layer_cache, inner=inner):
            inner(ctx, stream, layer_cache)
            kinds.append(stream.x.dtype)
        block.forward = spy
    run_whole(sess, random_tokens(64, (9,), seed=1))
    assert kinds == [torch.float32] * 3


@pytest.mark.parametrize("graphs", [False, True])
@pytest.mark.parametrize("name", ["B", "C"])
def test_greedy_generation_through_the_entry_point(folders, name, graphs):
    cfg, tensors = plain.read_folder(folders[name, "float32"])
    prompts = random_tokens(cases.CASES[name]["vocab"], (3, 11, 1, 30), seed=6)
    want = plain.generate(cfg, tensors, prompts, 10)
    engine = Engine(folders[name, "float32"], dtype="float32", max_batch=4, max_context=128, use_graphs=graphs)
    assert engine.generate_all(prompts, 10) == want
    assert engine.session.cache.slots.n_held == 0


def test_captured_decoding_gives_the_tokens_of_eager_decoding_bfloat16(folders):
    prompts = random_tokens(300, (70, 5, 33), seed=8)
    eager = Engine(folders["B", "bfloat16"], dtype="bfloat16", max_batch=4, max_context=256, use_graphs=False).generate_all(prompts, 40)
    captured = Engine(folders["B", "bfloat16"], dtype="bfloat16", max_batch=4, max_context=256, use_graphs=True).generate_all(prompts, 40)
    assert eager == captured


def test_replay_through_the_trace_runner_and_generation_from_the_command_line(folders, tmp_path):
    """bin/trace_run as a user drives it (a prompt in two portions, then two requests decoded in one batch, logits in
    files), and ``python -m starter_b200 generate`` on the same folder."""
    import json
    import subprocess
    import sys
    from pathlib import Path

    import numpy as np
    root = Path(__file__).resolve().parent.parent
    folder, vocab = folders["A", "float32"], 211
    a, b = random_tokens(vocab, (75, 9), seed=12)
    ref = cases.plain_logits(folder, [a, b])
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:40], "want": [0, 39]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[40:70], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[:4], "want": [3]}], "end": []}]
    for t in range(5):
        steps.append({"step": 3 + t, "entries": [{"id": "a", "tokens": [a[70 + t]], "want": [0]}, {"id": "b", "tokens": [b[4 + t]], "want": [0]}],
                      "end": ["a", "b"] if t == 4 else []})
    proc = subprocess.run([sys.executable, str(root / "bin" / "trace_run"), "--model", str(folder), "--dtype", "float32", "--out",
                           str(tmp_path), "--max-tokens", "256"], input="".join(json.dumps(s) + "\n" for s in steps),
                          capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert proc.stdout.split() == [w for s in steps for w in ("done", str(s["step"]))]
    read = lambda n: torch.from_numpy(np.fromfile(tmp_path / f"{n}.f32", dtype="<f4").reshape(-1, vocab).copy())
    tol = 1e-4 * float(ref[0].abs().max())
    assert float((read(0) - ref[0][[0, 39]]).abs().max()) <= tol and not (tmp_path / "1.f32").exists()
    assert float((read(2) - ref[1][[3]]).abs().max()) <= tol
    for t in range(5):
        assert float((read(3 + t) - torch.stack([ref[0][70 + t], ref[1][4 + t]])).abs().max()) <= tol, f"decoded token {t}"
    cfg, tensors = plain.read_folder(folder)
    want = plain.generate(cfg, tensors, [a[:6], b[:3]], 4)
    proc = subprocess.run([sys.executable, "-m", "starter_b200", "generate", "--model", str(folder), "--dtype", "float32", "--input-ids",
                           ",".join(map(str, a[:6])) + ";" + ",".join(map(str, b[:3])), "--max-new-tokens", "4", "--max-batch", "4",
                           "--max-context", "128"],
                          capture_output=True, text=True, timeout=600, cwd=str(root))
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [json.loads(line) for line in proc.stdout.splitlines()] == want
