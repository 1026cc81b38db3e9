"""The engine's Dubazen model against the plain implementation: every mechanism alone, then whole models under every
way of cutting the work (whole prompts, a decoded tail, portions down to two tokens, mixed batches with pages and
slots used again, long decoding, generation through the scheduler), in 32-bit and in bfloat16, on configurations
that differ in every size, constant and in the order of layers."""
import random

import pytest
import torch

import plain_dubazen as pd
import replay_util as ru
from dubazen_configs import CONFIGS, make_folder
from test_balelorn_gpu import floats, inputs, paged
from test_safepel_gpu import CUTS, MixerHarness, load_part, random_tensors, rel, run_in_cuts

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = {"float32": (torch.float32, 5e-5), "bfloat16": (torch.bfloat16, 3e-2)}
# beside the cuts of the other mixers' tests: both requests' whole prompts in one step, and long portions of both
ALL_CUTS = dict(CUTS, **{"together": [(10 ** 6, 10 ** 6)], "large portions": [(70, 30), (78, 7), (2, 0)]})
EPS = 1e-5


def check(part, rt, hidden, want, xs, tol, cuts, **kw):
    """Both requests under a cut, then once more with the slots and pages the other way round."""
    h = MixerHarness(part, rt, hidden, **kw)
    for order in (1, -1):
        got = run_in_cuts(h, xs[::order], [c[::order] for c in cuts])
        for a, b in zip(got, want[::order]):
            assert torch.isfinite(a).all() and rel(a, b) < tol, rel(a, b)
    h.mgr.check_invariants()


# ------------------------------------------------------------------ attention alone
def att_spec(hidden, H, G, D, V, scale, rot, prefix="m.", pairing="halves"):
    from ferrox_b200.parts.specs import AttentionSpec, ScaledRotarySpec

    return AttentionSpec(
        hidden=hidden, n_heads=H, n_kv_heads=G, head_dim=D, value_dim=V, qkv_bias=True, window=None, prefix=prefix,
        position=ScaledRotarySpec(*rot) if rot[0] else None, softmax_scale=scale, output_gate="g", sink="sink",
        tensor_names=(("q", "q"), ("k", "k"), ("v", "v"), ("o", "o"), ("q_bias", "q.b"), ("k_bias", "k.b"),
                      ("v_bias", "v.b"), ("o_bias", "o.b")),
        rotated_norm_eps=EPS, value_turn=(rot[1], pairing), o_bias=True)


def att_mixer(H, G, D, V, scale, rot):
    return dict(heads=H, kv_heads=G, dim=D, vdim=V, scale=scale, rot={"dims": rot[0], "base": rot[1]})


SHAPES = [  # heads, kv heads, dim, vdim, (rot dims, base), page
    (4, 2, 32, 48, (16, 500.0), 8), (3, 3, 20, 10, (6, 1000.0), 4), (6, 1, 12, 36, (0, 33.0), 16),
    (8, 2, 64, 64, (32, 20000.0), 64), (4, 1, 128, 128, (128, 250000.0), 64), (6, 3, 96, 40, (48, 500.0), 64),
    (2, 2, 24, 2, (2, 7.0), 64), (40, 1, 64, 64, (2, 10.0), 64), (4, 2, 128, 80, (64, 10000.0), 128),
    (70, 1, 16, 16, (16, 99.0), 16), (2, 1, 160, 200, (80, 1000.0), 64)]


@pytest.mark.parametrize("cut", list(ALL_CUTS))
@pytest.mark.parametrize("H,G,D,V,rot,page", SHAPES)
@pytest.mark.parametrize("dtype", list(DTYPES))
def test_attention_alone(dtype, H, G, D, V, rot, page, cut):
    dt, tol = DTYPES[dtype]
    hidden, scale = 64, round(3.0 / D, 4)
    spec = att_spec(hidden, H, G, D, V, scale, rot)
    w = random_tensors(spec, seed=H + D, std=0.25)
    w["m.sink"] = (torch.randn(H, generator=torch.Generator().manual_seed(V)) * 1.5 + 1.0).to(torch.bfloat16)
    m, wf = att_mixer(H, G, D, V, scale, rot), floats(w)
    xs = inputs(hidden, (150, 37), 3, dt)
    want = [pd.turned_value_attention(x, wf, "m.", m, EPS) for x in xs]
    part, rt = load_part(spec, w, dt)
    check(part, rt, hidden, want, xs, tol, ALL_CUTS[cut], page_size=page, n_pages=256 // page + 8)


@pytest.mark.parametrize("D,V,page", [(32, 48, 8), (64, 64, 64), (128, 128, 64), (128, 40, 64), (20, 12, 16)])
@pytest.mark.parametrize("dtype", list(DTYPES))
def test_keys_that_stand_out_far_away_and_at_page_borders(dtype, D, V, page):
    """The first keys of the sequence and keys on both sides of page borders are made to share the softmax of every later
    query among them, so that what comes out is their values, turned by the distance; in a prompt, in portions and
    decoded.  A fault of one position in either rotation, or a lost page, shows."""
    dt, tol = DTYPES[dtype]
    hidden, H, G, n, rot = 64, 4, 2, 330, (8, 50.0)
    g = torch.Generator().manual_seed(2)
    spec = att_spec(hidden, H, G, D, V, 25.0 / D, rot)
    w = random_tensors(spec, seed=D, std=0.25)
    # queries are alike; a key is close to them, behind the norm, where the input's first element is large
    for name, heads, noise in (("q", H, 0.02), ("k", G, 0.05)):
        wt = w["m." + name].float() * noise
        w["m." + name] = wt
        w[f"m.{name}.b"] = torch.zeros(heads * D)
    e = torch.zeros(D)
    e[D - 1] = 1.0                                  # (beyond the rotated part)
    w["m.q.b"] = (e * 2.0).repeat(H)
    w["m.k"].view(G, D, hidden)[:, D - 1, 0] = 1.0
    w = {k: v.to(torch.bfloat16) for k, v in w.items()}
    w["m.sink"] = torch.full((H,), -5.0, dtype=torch.bfloat16)
    x = torch.randn(n, hidden, generator=g) * 0.5
    x[:, 0] = 0.0
    loud = [0, 1, 7, 8, 63, 64, 127, 128, 191, 192, 255, 256, 320]
    x[loud, 0] = torch.linspace(2.0, 3.0, len(loud))[torch.randperm(len(loud), generator=g)]
    x = x.to(dt).float()
    m, wf = att_mixer(H, G, D, V, 25.0 / D, rot), floats(w)
    want = pd.turned_value_attention(x, wf, "m.", m, EPS)
    with pd.rounded_to(dt if dt != torch.float32 else None):     # (scores this sharp feel the rounding of queries and keys)
        allowed = max(tol, 2 * rel(pd.turned_value_attention(x, wf, "m.", m, EPS), want))
    assert allowed < 0.08
    for p in loud:         # without one of these keys the result is another one
        y = x.clone()
        y[p, 0] = 0.0
        assert rel(pd.turned_value_attention(y, wf, "m.", m, EPS)[p + 1:], want[p + 1:]) > max(2 * tol, 0.06)
    part, rt = load_part(spec, w, dt)
    for cuts in ([(n,)], [(9,), (2,), (53,), (2,), (62,), (132,), (70,)], [(64,)] + [(1,)] * 266, [(257,)] + [(1,)] * 73):
        got = run_in_cuts(MixerHarness(part, rt, hidden, page_size=page, n_pages=512 // page + 8), [x], cuts)
        assert rel(got[0], want) < allowed


@pytest.mark.parametrize("shift", [0.0, -40.0, 25.0])
def test_sinks_from_nothing_to_everything(shift):
    hidden, H, G, rot = 64, 4, 1, (32, 1000.0)
    for dtype, (dt, tol) in DTYPES.items():
        for D, V in ((64, 64), (64, 48)):
            spec = att_spec(hidden, H, G, D, V, 0.1, rot)
            w = random_tensors(spec, seed=5, std=0.25)
            w["m.sink"] = (w["m.sink"].float() + shift).to(torch.bfloat16)
            part, rt = load_part(spec, w, dt)
            xs = inputs(hidden, (150, 37), 4, dt)
            want = [pd.turned_value_attention(x, floats(w), "m.", att_mixer(H, G, D, V, 0.1, rot), EPS) for x in xs]
            for cut in ("whole", "one by one", "large portions"):
                got = run_in_cuts(MixerHarness(part, rt, hidden, page_size=64, n_pages=16), xs, ALL_CUTS[cut])
                for a, b in zip(got, want):
                    assert torch.isfinite(a).all() and rel(a, b) < tol


def test_values_turned_on_neighbouring_pairs():
    """The other layout of pairs: the plain implementation's with every head's pairs brought together."""
    hidden, H, G, D, V, rot = 64, 4, 2, 32, 24, (16, 500.0)
    dt, tol = DTYPES["float32"]
    spec = att_spec(hidden, H, G, D, V, 0.1, rot, pairing="adjacent")
    w = random_tensors(spec, seed=4, std=0.25)
    halves = dict(w)
    order = torch.arange(V).view(V // 2, 2).T.reshape(-1)                 # element m of the halves layout is order[m] here
    rows = lambda heads: (torch.arange(heads)[:, None] * V + order).reshape(-1)
    halves["m.v"], halves["m.v.b"] = w["m.v"][rows(G)], w["m.v.b"][rows(G)]
    halves["m.g"], halves["m.o"] = w["m.g"][rows(H)], w["m.o"][:, rows(H)]
    xs = inputs(hidden, (60, 20), 3, dt)
    want = [pd.turned_value_attention(x, floats(halves), "m.", att_mixer(H, G, D, V, 0.1, rot), EPS) for x in xs]
    part, rt = load_part(spec, w, dt)
    check(part, rt, hidden, want, xs, tol, CUTS["portions"], page_size=8)


def plain_turned(q, k, v, pos, scale, sinks, gate, turn):
    """One query row [H, D] against keys [n, G, D] and values [n, G, V], the result's neighbouring pairs turned back by
    the angles whose (cos, sin) are ``turn`` [V / 2, 2]; everything 64-bit."""
    H, G = q.shape[0], k.shape[1]
    out = []
    for h in range(H):
        g = h // (H // G)
        s = (k[:pos + 1, g].double() @ q[h].double()) * scale
        e = torch.exp(s - s.max())
        o = (e / (e.sum() + torch.exp(sinks[h].double() - s.max()))) @ v[:pos + 1, g].double()
        c, sn, a, b = turn[:, 0].double(), turn[:, 1].double(), o[0::2], o[1::2]
        out.append(torch.stack([a * c + b * sn, b * c - a * sn], dim=1).reshape(-1))
    return torch.stack(out) * torch.sigmoid(gate.double()).view(H, -1)


def turn_table(n, V, g):
    ang = torch.rand(n, V // 2, generator=g) * 6.28
    return torch.stack([torch.cos(ang), torch.sin(ang)], dim=-1).contiguous()


@pytest.mark.parametrize("run_blocks", [0, 2])
@pytest.mark.parametrize("D,V", [(128, 128), (64, 64), (128, 48), (96, 104), (40, 72)])
def test_prompt_kernel_turns_results_back(D, V, run_blocks):
    """The tcgen05 prompt kernel and its merge behind a long prefix, tiles cut into runs of key blocks or whole."""
    from ferrox_b200.kernels import ops

    g = torch.Generator().manual_seed(D + V)
    H, G, page, start, n = 4, 2, 64, 900, 340
    bf = lambda *s: torch.randn(*s, generator=g).to(torch.bfloat16)
    q, k, v, gates = bf(n, H * D), bf(start + n, G, D), bf(start + n, G, V), bf(n, H * V)
    sinks, turn = torch.randn(H, generator=g) * 2, turn_table(n, V, g)
    kp, vp, table = paged(k.float(), v.float(), page, 3)
    items, merges, parts = ops.prefill_tc_plan([(n, start)], None, H, run_blocks=run_blocks)
    assert (parts > 0) == (run_blocks > 0)
    out = torch.full((n, H * V), float("nan"), dtype=torch.bfloat16, device=DEV)
    part_o = torch.full((max(1, parts), H, 256, ops.prefill_value_width(V)), float("nan"), device=DEV)
    part_ml = torch.full((max(1, parts), H, 256, 2), float("nan"), device=DEV)
    scale = 1.3 / D ** 0.5
    ops.prefill_attention_tc(q.to(DEV), kp.to(DEV).to(torch.bfloat16), vp.to(DEV).to(torch.bfloat16), table.to(DEV), page,
                             torch.from_numpy(items).to(DEV), torch.zeros(1, dtype=torch.int32, device=DEV), out, H, G, D,
                             None, scale, merges=torch.from_numpy(merges).to(DEV) if parts else None, part_o=part_o,
                             part_ml=part_ml, value_dim=V, sinks=sinks.to(DEV), gate=gates.to(DEV), turn=turn.to(DEV))
    assert torch.isfinite(out).all()
    for i in list(range(0, n, 37)) + [n - 1, 255, 256]:
        want = plain_turned(q[i].float().view(H, D), k.float(), v.float(), start + i, scale, sinks, gates[i].float(), turn[i])
        assert rel(out[i].view(H, V), want) < 2e-2, i


@pytest.mark.parametrize("n_splits", [1, 3, 7])
@pytest.mark.parametrize("kernel,D,V", [("tma", 128, 128), ("tma", 64, 64), ("tma, merged inside", 128, 128), ("general", 128, 80),
                                        ("general", 32, 16), ("general", 64, 144)])
def test_decode_kernels_turn_results_back(kernel, D, V, n_splits):
    """One token a request, its keys in one run or in several that a second kernel (or the last block) adds up."""
    from ferrox_b200.kernels import ops

    g = torch.Generator().manual_seed(D + n_splits)
    H, G, page, n = 8, 2, 64, 1000
    bf = lambda *s: torch.randn(*s, generator=g).to(torch.bfloat16)
    k, v = bf(n, G, D), bf(n, G, V)
    positions = [0, 63, 64, 399, 400, 401, 777, 999]
    T = len(positions)
    q, gates, sinks, turn = bf(T, H * D), bf(T, H * V), torch.randn(H, generator=g) * 2, turn_table(T, V, g)
    kp, vp, table = paged(k.float(), v.float(), page, 4)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)
    out = torch.full((T, H * V), float("nan"), dtype=torch.bfloat16, device=DEV)
    acc, ml = torch.empty(T, H, n_splits, V, device=DEV), torch.empty(T, H, n_splits, 2, device=DEV)
    scale, qd, gd, sd, td = 1.3 / D ** 0.5, q.to(DEV), gates.to(DEV), sinks.to(DEV), turn.to(DEV)
    kd, vd, tab = kp.to(DEV).to(torch.bfloat16), vp.to(DEV).to(torch.bfloat16), table.to(DEV)
    if kernel == "general":
        ops.general_attention(qd, H * D, D, kd, vd, D, V, tab, page, i32(positions), i32([0] * T), i32([0]), None, out, H * V, V,
                              H, G, D, V, None, scale, n_splits=n_splits, part_o=acc, part_ml=ml, sinks=sd, gate=gd, turn=td)
    else:
        counters = torch.zeros(1024, dtype=torch.int32, device=DEV) if "inside" in kernel else None
        ops.decode_attention(qd, kd, vd, tab, page, i32(positions), i32([0] * T), i32([0]), out, H, G, D, None, scale, 0, n_splits,
                             acc, ml, counters=counters, extras=ops.DecodeExtras.of(None, sd, gd, turn=td))
    torch.cuda.synchronize()
    for i, p in enumerate(positions):
        want = plain_turned(q[i].float().view(H, D), k.float(), v.float(), p, scale, sinks, gates[i].float(), turn[i])
        assert rel(out[i].view(H, V), want) < 2e-2, p


# ------------------------------------------------------------------ the mixers with a state, and mixers side by side
def gla_tensors(H, D, V, rank, hidden, tau):
    from ferrox_b200.parts.specs import GatedLinearAttentionSpec

    spec = GatedLinearAttentionSpec(hidden=hidden, n_heads=H, head_dim=D, value_dim=V, decay_rank=rank, tau=tau, norm_eps=EPS,
                                    prefix="m.")
    w = random_tensors(spec, seed=D + V, std=0.2)
    # decays from fast to nearly none, channel by channel
    w["m.a2.b"] = torch.linspace(-2.0, 6.0, H * D)[torch.randperm(H * D, generator=torch.Generator().manual_seed(1))].to(torch.bfloat16)
    return spec, w, {"heads": H, "dim": D, "vdim": V, "tau": tau}


@pytest.mark.parametrize("cut", list(ALL_CUTS))
@pytest.mark.parametrize("H,D,V,rank,tau", [(2, 16, 32, 8, 16.0), (1, 20, 12, 5, 1.0), (3, 48, 20, 16, 4.0), (2, 128, 64, 16, 16.0),
                                            (1, 256, 40, 150, 8.0), (2, 1, 1, 1, 2.0), (4, 64, 7, 3, 0.5), (1, 190, 16, 16, 16.0)])
@pytest.mark.parametrize("dtype", list(DTYPES))
def test_gated_linear_attention_alone(dtype, H, D, V, rank, tau, cut):
    dt, tol = DTYPES[dtype]
    hidden = 64
    spec, w, m = gla_tensors(H, D, V, rank, hidden, tau)
    xs = inputs(hidden, (150, 37), 3, dt)
    want = [pd.gated_linear_attention(x, floats(w), "m.", m, EPS) for x in xs]
    part, rt = load_part(spec, w, dt)
    check(part, rt, hidden, want, xs, tol, ALL_CUTS[cut])


def mamba_tensors(inner, state, rank, taps, hidden, step=-3.0):
    from ferrox_b200.parts.specs import SelectiveScanSpec

    spec = SelectiveScanSpec(hidden=hidden, inner=inner, n_state=state, dt_rank=rank, conv_taps=taps, prefix="m.")
    w = random_tensors(spec, seed=inner + state, std=0.2)
    w["m.conv"] = (w["m.conv"].float() * 3).to(torch.bfloat16)
    w["m.dt.b"] = (w["m.dt.b"].float() + 3.0 + step).to(torch.bfloat16)
    w["m.A_log"] = (torch.randn(inner, state, generator=torch.Generator().manual_seed(2)) * 1.5).to(torch.bfloat16)
    return spec, w, {"inner": inner, "state": state, "dt_rank": rank, "conv": taps}


@pytest.mark.parametrize("cut", list(ALL_CUTS))
@pytest.mark.parametrize("inner,state,rank,taps", [(96, 16, 8, 4), (50, 1, 3, 2), (36, 6, 5, 3), (256, 16, 16, 4), (130, 32, 12, 4),
                                                   (40, 33, 1, 1), (24, 100, 20, 5), (17, 200, 7, 16), (64, 8, 40, 3), (31, 4, 9, 4)])
@pytest.mark.parametrize("dtype", list(DTYPES))
def test_selective_scan_alone(dtype, inner, state, rank, taps, cut):
    dt, tol = DTYPES[dtype]
    hidden = 64
    spec, w, m = mamba_tensors(inner, state, rank, taps, hidden)
    xs = inputs(hidden, (150, 37), 3, dt)
    want = [pd.selective_scan(x, floats(w), "m.", m, EPS) for x in xs]
    part, rt = load_part(spec, w, dt)
    check(part, rt, hidden, want, xs, tol, ALL_CUTS[cut])


@pytest.mark.parametrize("kind", ["gla", "mamba"])
def test_what_a_state_remembers_over_a_thousand_tokens(kind):
    """Slow decays, one loud token at the start that every later output carries, in portions of odd sizes: in 32-bit the
    engine stays as close to a 64-bit computation as a few roundings, at the end as at the start."""
    hidden, n = 32, 1200
    dt = torch.float32
    if kind == "gla":
        spec, w, m = gla_tensors(2, 32, 24, 4, hidden, 16.0)
        w["m.a2.b"] = torch.full((64,), 5.0, dtype=torch.bfloat16)
        w["m.norm"] = torch.ones(24, dtype=torch.bfloat16)
        plain = pd.gated_linear_attention
    else:
        spec, w, m = mamba_tensors(48, 16, 4, 4, hidden, step=-5.0)
        w["m.A_log"] = torch.full((48, 16), -2.0, dtype=torch.bfloat16)
        plain = pd.selective_scan
    x = torch.randn(n, hidden, generator=torch.Generator().manual_seed(1)) * 0.1
    x[0] *= 50.0
    wd = {k: v.double() for k, v in w.items()}
    want = plain(x.double(), wd, "m.", m, EPS)
    quiet = x.clone()
    quiet[0] *= 0.02
    assert rel(plain(quiet.double(), wd, "m.", m, EPS)[-100:], want[-100:]) > 1e-2        # the first token still shows
    part, rt = load_part(spec, w, dt)
    for cuts in ([(n,)], [(257,), (2,), (130,), (3,)] * 4, [(1100,)] + [(1,)] * 100):
        got = run_in_cuts(MixerHarness(part, rt, hidden, max_positions=2048), [x], cuts)[0]
        assert rel(got, want) < 2e-5 and rel(got[-100:], want[-100:]) < 2e-5, (rel(got, want), rel(got[-100:], want[-100:]))


def test_sizes_the_recurrences_do_not_hold_are_refused():
    from ferrox_b200.parts.base import build_part
    from ferrox_b200.parts.specs import GatedLinearAttentionSpec, SelectiveScanSpec

    for bad in (GatedLinearAttentionSpec(8, 1, 257, 8, 4, 1.0, EPS, "m."), GatedLinearAttentionSpec(8, 1, 8, 8, 0, 1.0, EPS, "m."),
                GatedLinearAttentionSpec(8, 1, 8, 8, 4, 0.0, EPS, "m."), SelectiveScanSpec(8, 8, 257, 2, 4, "m."),
                SelectiveScanSpec(8, 8, 8, 0, 4, "m."), SelectiveScanSpec(8, 8, 8, 2, 17, "m.")):
        with pytest.raises(ValueError):
            build_part(bad)


@pytest.mark.parametrize("cut", list(ALL_CUTS))
@pytest.mark.parametrize("dtype", list(DTYPES))
def test_two_mixers_side_by_side(dtype, cut):
    from ferrox_b200.parts.specs import DecayedLinearAttentionSpec, MixerSumSpec

    dt, tol = DTYPES[dtype]
    hidden, decay = 64, (0.5, 0.97, 0.999)
    left = att_spec(hidden, 4, 2, 32, 48, 0.1, (16, 500.0), prefix="m.left.")
    right = DecayedLinearAttentionSpec(hidden=hidden, n_heads=3, head_dim=20, value_dim=32, decay=decay, norm_eps=EPS, prefix="m.right.")
    spec = MixerSumSpec((left, right), (0.7, 1.6))
    w = random_tensors(spec, seed=8, std=0.25)
    m = {"left": att_mixer(4, 2, 32, 48, 0.1, (16, 500.0)), "right": {"heads": 3, "dim": 20, "vdim": 32, "decay": decay},
         "left_scale": 0.7, "right_scale": 1.6}
    xs = inputs(hidden, (150, 37), 6, dt)
    want = [pd.parallel(x, floats(w), "m.", m, EPS) for x in xs]
    part, rt = load_part(spec, w, dt)

    class Summed:      # (the harness asks for one output: the parts with their weights)
        def forward_into(self, x, out, batch, cache, accumulate=False):
            out.copy_(sum(s * y for y, s in part.forward_parts(x, batch, cache)))
    h = MixerHarness(part, rt, hidden, page_size=8)
    h.part = Summed()
    got = run_in_cuts(h, xs, ALL_CUTS[cut])
    for a, b in zip(got, want):
        assert rel(a, b) < tol


# ------------------------------------------------------------------ streams, experts, small kernels
@pytest.mark.parametrize("S", range(1, 9))
@pytest.mark.parametrize("dtype", list(DTYPES))
def test_streams_updated_and_read(dtype, S):
    """One pass that updates the streams with results of every kind and reads the new ones; one that reads alone; rows
    picked out."""
    from ferrox_b200.kernels import ops

    dt = DTYPES[dtype][0]
    g = torch.Generator().manual_seed(S)
    R = lambda *s: torch.randn(*s, generator=g)
    tol_x = 1e-5 if dt == torch.float32 else 1e-2
    for T, W, n_terms, K in ((1, 64, 1, 0), (5, 72, 2, 2), (300, 130, 3, 3), (3, 2048, 1, 4), (270, 4096, 2, 1), (2, 51, 0, 2), (2, 5000, 1, 0), (6, 64, 1, 9)):
        X, ys = R(S, T, W), [R(T, W) for _ in range(n_terms)]
        mix, coef, coef_e, reads = R(S, S), [R(S) for _ in ys], R(S), R(S)
        w = 1 + 0.2 * R(W)
        e = torch.zeros(T, W)
        experts = None
        if K:
            rows, shared = R(T * K, W).to(dt), (R(T, W).to(dt) if K != 3 else None)
            place = torch.randperm(T * K, generator=g).to(torch.int32).view(T, K)
            wts = torch.rand(T, K, generator=g)
            e = (rows.float()[place.long()] * wts[:, :, None]).sum(1) + (shared.float() if shared is not None else 0)
            experts = (rows.to(DEV), place.to(DEV), wts.to(DEV), shared.to(DEV) if shared is not None else None, None)
        tied = X.permute(1, 0, 2).reshape(T, S * W).contiguous()
        out = lambda n: torch.full((n, W), float("nan"), dtype=dt, device=DEV)
        # updated and read
        new = torch.einsum("snw,st->tnw", X, mix) + coef_e[:, None, None] * e
        for y, c in zip(ys, coef):
            new = new + c[:, None, None] * y
        h = tied.to(DEV)
        x = ops.stream_step(h, S, terms=[(y.to(DEV), c.tolist()) for y, c in zip(ys, coef)],
                            experts=(experts, coef_e.tolist()) if K else None, mix=mix.tolist(),
                            read=(reads.tolist(), w.to(DEV), EPS, out(T)))
        got = h.cpu().view(T, S, W).permute(1, 0, 2)
        assert rel(got, new) < 3e-6
        assert rel(x, pd.rms(pd.read_streams(new, reads), EPS) * w) < tol_x
        # updated alone
        h = tied.to(DEV)
        assert ops.stream_step(h, S, terms=[(y.to(DEV), c.tolist()) for y, c in zip(ys, coef)],
                               experts=(experts, coef_e.tolist()) if K else None, mix=mix.tolist()) is None
        assert rel(h.cpu().view(T, S, W).permute(1, 0, 2), new) < 3e-6
        # read with results beside, streams as they are
        u = pd.read_streams(X, reads) + sum(float(c[0]) * y for y, c in zip(ys, coef)) + (float(coef_e[0]) * e if K else 0)
        h = tied.to(DEV)
        x = ops.stream_step(h, S, terms=[(y.to(DEV), [float(c[0])]) for y, c in zip(ys, coef)],
                            experts=(experts, [float(coef_e[0])]) if K else None, read=(reads.tolist(), w.to(DEV), EPS, out(T)))
        assert rel(x, pd.rms(u, EPS) * w) < tol_x and torch.equal(h.cpu(), tied)
        # some rows
        rows = torch.tensor([T - 1, 0], dtype=torch.int32, device=DEV)
        x = ops.stream_step(h, S, read=(reads.tolist(), w.to(DEV), EPS, out(2)), rows=rows)
        assert rel(x, (pd.rms(pd.read_streams(X, reads), EPS) * w)[[T - 1, 0]]) < tol_x


def test_embedding_into_every_stream_and_rows_in_two_halves():
    from ferrox_b200.kernels import ops

    g = torch.Generator().manual_seed(0)
    table = torch.randn(50, 72, generator=g).to(torch.bfloat16)
    ids = torch.tensor([0, 49, 7, 50], dtype=torch.int32, device=DEV)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    out = torch.empty(4, 3 * 72, device=DEV)
    ops.embed_streams(table.to(DEV), ids[:3], out[:3], 3, status=status, scale=2.5)
    assert torch.equal(out[:3].cpu().view(3, 3, 72), (table.float()[[0, 49, 7]] * 2.5)[:, None].expand(3, 3, 72)) and int(status) == 0
    ops.embed_streams(table.to(DEV), ids, out, 3, status=status, scale=2.5)
    assert int(status) == 1 and float(out[3].abs().max()) == 0.0          # an id outside the vocabulary raises the status
    x = torch.randn(33, 20, generator=g, dtype=torch.float32).to(DEV)
    halves = torch.full((33, 32), float("nan"), dtype=torch.bfloat16, device=DEV)
    ops.split_rows(x[:, 3:16], halves)
    hi, lo = halves[:, :16].float(), halves[:, 16:].float()
    assert float(((hi + lo)[:, :13] - x[:, 3:16]).abs().max() / x.abs().max()) < 2.0 ** -16 and float((hi + lo)[:, 13:].abs().max()) == 0


def test_a_layer_of_other_parts_on_streams():
    """The block of streams around a mixer without parts of its own and a dense feed-forward: nothing in it knows the design."""
    from ferrox_b200.parts.specs import GatedLinearAttentionSpec, HyperBlockSpec, NormSpec, PlainMlpSpec, StreamNormSpec

    S, W, T = 3, 64, 40
    for ffn in (PlainMlpSpec(W, 96, "f."), None):
        norm = lambda q: StreamNormSpec(NormSpec(W, EPS, "", name=f"n{q}", scalar=q == 1), S, f"in{q}")
        spec = HyperBlockSpec(norm1=norm(1), mixer=GatedLinearAttentionSpec(W, 2, 16, 24, 4, 8.0, EPS, "m."), norm2=norm(2) if ffn else None,
                              ffn=ffn, streams=S, connections=(("mix1", "out1"), ("mix2", "out2"))[:2 if ffn else 1])
        w = random_tensors(spec, seed=3, std=0.2)
        block, rt = load_part(spec, w, torch.float32)
        wf = floats(w)
        X = torch.randn(S, T, W, generator=torch.Generator().manual_seed(4))
        m = {"heads": 2, "dim": 16, "vdim": 24, "tau": 8.0}
        y = pd.gated_linear_attention(pd.rms(pd.read_streams(X, wf["in1"]), EPS) * wf["n1"], wf, "m.", m, EPS)
        A = pd.mix_streams(X, y, wf["mix1"], wf["out1"])
        if ffn:
            u = pd.rms(pd.read_streams(A, wf["in2"]), EPS) * wf["n2"]
            A = pd.mix_streams(A, torch.relu(u @ wf["f.up"].T) ** 2 @ wf["f.down"].T, wf["mix2"], wf["out2"])
        h = X.permute(1, 0, 2).reshape(T, S * W).contiguous().to(DEV)

        class Whole:
            spec = block.mixer.spec
            cache_spec = staticmethod(block.mixer.cache_spec)

            def forward_into(self, x, out, batch, cache, accumulate=False):
                assert block.forward(h, batch, cache) is None
                out.zero_()
        run_in_cuts(MixerHarness(Whole(), rt, W), [torch.zeros(T, W)], [(T,)])
        assert rel(h.cpu().view(T, S, W).permute(1, 0, 2), A) < 2e-5


def clear_of_a_choice(f, W, p, x):
    """The tokens whose last chosen expert's score lies above the next one's by more than a fiftieth."""
    s = torch.softmax(x @ W[p + "router"].T, dim=-1).sort(dim=-1, descending=True).values
    k = f["router"]["top"]
    return (s[:, k - 1] - s[:, k]) > 0.02 * s[:, k - 1] if k < s.shape[1] else torch.ones(x.shape[0], dtype=torch.bool)


@pytest.mark.parametrize("E,top,I,Is", [(6, 2, 32, 48), (3, 3, 24, 0), (12, 3, 64, 96), (5, 1, 20, 36), (70, 4, 32, 64)])
@pytest.mark.parametrize("tokens", [1, 5, 40, 64, 300])
@pytest.mark.parametrize("dtype", list(DTYPES))
def test_experts_alone(dtype, tokens, E, top, I, Is):
    """Both clamps in play, the shared expert with a limit of its own, weights divided by their sum."""
    from types import SimpleNamespace

    from ferrox_b200.kernels import ops
    from ferrox_b200.parts.specs import MoeSpec

    dt, tol = DTYPES[dtype]
    hidden = 64
    spec = MoeSpec(hidden=hidden, n_experts=E, top_k=top, expert_intermediate=I, shared_intermediate=Is, norm_topk_prob=True,
                   shared_gate=False, prefix="f.", activation=("clamped_swish", 0.7, 1.702),
                   shared_activation=("clamped_swish", 1.9, 1.702) if Is else None,
                   tensor_names=("router", "e{e}.{part}", "shared.{part}"), renorm_eps=1e-20)
    w = random_tensors(spec, seed=tokens + E, std=0.3)
    wf = floats(w)
    part, _ = load_part(spec, w, dt)
    x = inputs(hidden, [tokens], tokens, dt)[0]
    f = {"router": {"experts": E, "top": top}, "expert": {"ff": I, "limit": 0.7}}
    if Is:
        f["shared"] = {"ff": Is, "limit": 1.9}
    want = pd.experts(f, wf, "f.", x)
    out = torch.full((tokens, hidden), float("nan"), device=DEV)
    part.forward_into(x.to(DEV).to(dt), out, SimpleNamespace(status=None, stream=ops.stream_ptr(), shared={}), accumulate=False)
    ok = clear_of_a_choice(f, wf, "f.", x)
    assert bool(ok.any()) and rel(out.cpu()[ok], want[ok]) < tol


# ------------------------------------------------------------------ whole models
def prompts_for(name, n=5, hi=150, seed=0):
    cfg = CONFIGS[name][0]
    rng = random.Random(seed)
    lens = [1, 2, hi] + [rng.randint(3, hi) for _ in range(max(0, n - 3))]
    return {f"r{i}": [rng.randrange(cfg["vocab"]) for _ in range(L)] for i, L in enumerate(lens)}


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    tmp = tmp_path_factory.mktemp("dubazen_models")
    return {name: make_folder(tmp, name) for name in CONFIGS}


def position_errors(got, want):
    return (got - want).abs().amax(dim=-1) / want.abs().max()


def rounding_alone(cfg, w, tokens, want):
    """Per position: how far the plain implementation's logits move when everything that may be computed in bfloat16
    is rounded to it."""
    with pd.rounded_to(torch.bfloat16):
        return position_errors(pd.forward(cfg, w, tokens), want)


@pytest.fixture(scope="module")
def expected(folders):
    out = {}
    for name in CONFIGS:
        cfg, w = CONFIGS[name][0], pd.load_weights(folders[name])
        want = {rid: pd.forward(cfg, w, t) for rid, t in prompts_for(name).items()}
        out[name] = (cfg, w, want, {rid: rounding_alone(cfg, w, t, want[rid]) for rid, t in prompts_for(name).items()})
    return out


def engine(folder, dtype, **kw):
    from ferrox_b200 import Engine

    kw.setdefault("page_size", 64 if folder.endswith("_C") else 8)     # C: the page size of serving
    kw.setdefault("n_pages", 64)
    kw.setdefault("max_slots", 4)
    return Engine.from_folder(folder, dtype=dtype, **kw)


def compare(got, want, tol, what, noise=None):
    """32-bit: every position within ``tol``.  bfloat16 (``noise``: what rounding alone does to the plain
    implementation at every position): the median and the ninth decile of the engine's distances over all positions
    lie within three times those of rounding alone, plus a hundredth and two (a choice of experts may turn either way)."""
    errs = []
    for rid in want:
        assert got[rid].shape == want[rid].shape, (what, rid)
        assert torch.isfinite(got[rid]).all(), (what, rid)
        e = position_errors(got[rid], want[rid])
        if noise is None:
            assert float(e.max()) < tol, (what, rid, float(e.max()), int(e.argmax()))
        errs.append(e)
    if noise is not None:
        e, n = torch.cat(errs), torch.cat([noise[rid] for rid in want])
        for q, slack in ((0.5, 1e-2), (0.9, 2e-2)):
            assert float(e.quantile(q)) <= 3 * float(n.quantile(q)) + slack, (what, q, float(e.quantile(q)), float(n.quantile(q)))


RUNS = {
    "whole": lambda eng, p: ru.run_whole(eng, p),
    "decoded tail": lambda eng, p: ru.run_tail_decode(eng, p, tail=50),
    "portions": lambda eng, p: ru.run_portions(eng, p),
    "decoding together": lambda eng, p: ru.run_decode_together(eng, p, tail=9),
    "mixed": lambda eng, p: ru.run_mixed(eng, p, seed=3, max_live=3),
    "mixed, large portions": lambda eng, p: ru.run_mixed(eng, p, seed=6, max_live=4, max_portion=60),
}


@pytest.mark.parametrize("run", list(RUNS))
@pytest.mark.parametrize("name", sorted(CONFIGS))
@pytest.mark.parametrize("dtype", list(DTYPES))
def test_model_under_every_cut(folders, expected, dtype, name, run):
    _, tol = DTYPES[dtype]
    eng = engine(folders[name], dtype)
    got = RUNS[run](eng, prompts_for(name))
    compare(got, expected[name][2], tol, f"{name} {dtype} {run}", expected[name][3] if dtype == "bfloat16" else None)
    eng.cache.check_invariants()
    assert all(n == eng.cache.groups[k].pool.n_pages for k, n in eng.cache.free_pages().items())   # all given back


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_cuts_agree_with_each_other_to_rounding(folders, name):
    eng = engine(folders[name], "float32")
    p = prompts_for(name)
    whole, mixed = ru.run_whole(eng, p), ru.run_mixed(eng, p, seed=5, max_live=4)
    for rid in p:
        assert float((whole[rid] - mixed[rid]).abs().max() / whole[rid].abs().max()) < 2e-5


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_sum_of_the_streams_after_every_layer(folders, expected, name):
    from ferrox_b200.engine.batch import StepEntry

    cfg, w = expected[name][:2]
    toks = prompts_for(name)["r3"]
    want_logits, after = pd.forward(cfg, w, toks, return_layers=True)
    eng = engine(folders[name], "float32")
    seen = []
    for i, block in enumerate(eng.model.layers):
        inner = block.forward

        def spy(h, batch, cache, _inner=inner, _i=i, **kw):
            out = _inner(h, batch, cache, **kw)
            seen.append((_i, h.detach().view(h.shape[0], cfg["streams"], -1).sum(1).cpu()))
            return out
        block.forward = spy
    slot = eng.open_request()
    got = eng.step([StepEntry(slot, toks, want=list(range(len(toks))))]).cpu()
    assert [i for i, _ in seen] == list(range(len(cfg["layers"])))
    for n, (_, h) in enumerate(seen):
        assert rel(h, after[n]) < 2e-5, n
    assert rel(got, want_logits) < 5e-5


@pytest.mark.parametrize("name", ["A", "C"])
@pytest.mark.parametrize("dtype", list(DTYPES))
def test_long_decoding(folders, dtype, name):
    """A few tokens of prompt, then hundreds decoded one by one, across many pages."""
    _, tol = DTYPES[dtype]
    cfg, w = CONFIGS[name][0], pd.load_weights(folders[name])
    rng = random.Random(9)
    n = 303 if name == "A" else 420
    toks = [rng.randrange(cfg["vocab"]) for _ in range(n)]
    want = pd.forward(cfg, w, toks)
    eng = engine(folders[name], dtype, n_pages=40, max_slots=2)
    c = ru.Collector(eng)
    c.step({"x": toks[:3]})
    for t in toks[3:]:
        c.step({"x": [t]})
    compare({"x": c.stacked("x")}, {"x": want}, tol, "long decoding",
            {"x": rounding_alone(cfg, w, toks, want)} if dtype == "bfloat16" else None)


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_greedy_generation_through_the_scheduler(folders, name):
    cfg, w = CONFIGS[name][0], pd.load_weights(folders[name])
    rng = random.Random(4)
    prompts = [[rng.randrange(cfg["vocab"]) for _ in range(n)] for n in (5, 1, 23)]
    want = [pd.greedy(cfg, w, p, 12) for p in prompts]
    eng = engine(folders[name], "float32")
    assert eng.graphs is not None            # every part of the model can be captured: decode steps replay graphs
    got = eng.generate(prompts, max_new_tokens=12, max_batch_tokens=16)     # prompts go in portions
    assert got == want
    again = eng.generate(prompts[::-1], max_new_tokens=12)                  # slots and pages used again
    assert again == want[::-1]
    bf = engine(folders[name], "bfloat16").generate(prompts, max_new_tokens=12)
    assert all(len(g) == 12 for g in bf)
    for p, g in zip(prompts, bf):
        logits = pd.forward(cfg, w, (p + g)[:-1])
        close = sum(float(logits[len(p) - 1 + i].max() - logits[len(p) - 1 + i][tok]) <= 2 * 6e-2 * float(logits.abs().max())
                    for i, tok in enumerate(g))
        assert close >= 10      # (a choice of experts within rounding may differ at a position or two)


def test_trace_replay_and_command_line_with_a_dubazen_folder(folders, tmp_path):
    import json
    import os
    import subprocess
    import sys

    import numpy as np

    cfg, w = CONFIGS["B"][0], pd.load_weights(folders["B"])
    toks = [3, 90, 7, 7, 45, 21, 9, 81]
    want = pd.forward(cfg, w, toks)
    steps = [
        {"step": 0, "entries": [{"id": "a", "tokens": toks[:5], "want": [0, 4]}], "end": []},
        {"step": 1, "entries": [{"id": "a", "tokens": toks[5:6], "want": []}], "end": []},
        {"step": 2, "entries": [{"id": "a", "tokens": toks[6:], "want": [1]}, {"id": "b", "tokens": toks[:2], "want": [1]}],
         "end": ["a", "b"]},
    ]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = tmp_path / "out"
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", folders["B"], "--dtype", "float32",
                        "--out", str(out), "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    s0 = torch.from_numpy(np.fromfile(out / "0.f32", dtype="<f4").reshape(2, -1))
    s2 = torch.from_numpy(np.fromfile(out / "2.f32", dtype="<f4").reshape(2, -1))
    assert rel(s0, want[[0, 4]]) < 5e-5 and rel(s2, want[[7, 1]]) < 5e-5
    nxt = pd.greedy(cfg, w, toks[:4], 2)
    r = subprocess.run([sys.executable, os.path.join(root, "bin", "ferrox"), "-m", folders["B"], "--tokens", "3,90,7,7",
                        "-n", "2", "--temp", "0", "--dtype", "float32", "--ignore-eos", "--repeat-penalty", "1.0"],
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [int(t) for t in r.stdout.split()] == nxt


def test_preemption_decoding_ahead_and_sampling(folders):
    """A request that is preempted gives its pages and slot back and is recomputed; greedy decode steps are replayed
    graphs issued one ahead of the host; sampled ones depend on the seed alone."""
    cfg, w = CONFIGS["B"][0], pd.load_weights(folders["B"])
    prompts = [[i + 1, i + 3, i + 7, 90, 4, 8, 15, 16] for i in range(4)]
    want = [pd.greedy(cfg, w, p, 20) for p in prompts]
    small = engine(folders["B"], "float32", page_size=4, n_pages=14, max_slots=4)     # 4 x 28 positions do not fit 56
    outs, stats = small.generate(prompts, max_new_tokens=20, return_stats=True)
    assert stats["preemptions"] >= 1 and outs == want
    small.cache.check_invariants()
    roomy = engine(folders["B"], "float32", n_pages=64)
    outs, stats = roomy.generate(prompts, max_new_tokens=20, return_stats=True)
    assert outs == want and stats["ahead_steps"] >= 8 and stats["preemptions"] == 0
    sampled = [roomy.generate(prompts, max_new_tokens=10, temperature=0.8, top_k=20, seed=s) for s in (1, 1, 2)]
    assert sampled[0] == sampled[1] and sampled[0] != sampled[2]
