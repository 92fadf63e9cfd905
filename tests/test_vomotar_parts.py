"""Each mechanism of the Vomotar decoder alone, its kernels against the plain implementation's function: norms in equal
parts of a row, the sum of two normed results with the next norm written on the way, gates from low-rank maps, the delta
rule with a decay per key channel and the retention (over steps and slots; token by token, and in chunks whose sums are
tensor-core products), strong and vanishing decays, attention in chunks with a distance bias (a key that stands out on the
first position of the query's chunk and on the last one before it), values cached divided by their root mean square."""
import math

import pytest
import torch

import plain_vomotar as P
from helpers import check_error

pytestmark = pytest.mark.gpu
PAGE = 64


def rel(got, ref):
    got, ref = got.double().cpu(), ref.double().cpu()
    assert got.shape == ref.shape, (got.shape, ref.shape)
    assert torch.isfinite(got).all()
    return float((got - ref).abs().max() / ref.abs().max())


def i32(values):
    return torch.tensor(values, dtype=torch.int32, device="cuda")


def scratch(name, shape, dtype):
    return torch.full(shape, float("nan"), dtype=dtype, device="cuda")      # what a kernel reads it must have written


# --------------------------------------------------------------------------- norms
@pytest.mark.parametrize("T,d,parts", [(5, 72, 3), (1, 8, 8), (3, 1000, 4), (9, 52, 13), (2, 5120, 2), (4, 4096, 1), (3, 24000, 3), (7, 96, 96)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_norm_in_equal_parts(T, d, parts, dtype):
    from llmplayer_b200.kernels import ops
    torch.manual_seed(d + parts)
    x = torch.randn(T, d) * torch.linspace(0.1, 4.0, d)             # the parts' sizes differ, so a norm over the row differs
    w = 1 + 0.3 * torch.randn(d)
    junk = torch.full((777,), 3.0, device="cuda")
    out = torch.empty(T, d, dtype=dtype, device="cuda")
    ops.rmsnorm(x.cuda(), w.cuda(), 2e-5, out, clear=junk, parts=parts)
    ref = P.part_norm(x.double(), w.double(), 2e-5, parts)
    check_error(f"norm in parts, {dtype}", f"{T}x{d} in {parts}", rel(out, ref), 2e-6 if dtype == torch.float32 else 5e-3)
    assert float(junk.abs().max()) == 0.0
    rows = list(range(T - 1, -1, -2))
    some = torch.empty(len(rows), d, dtype=dtype, device="cuda")
    ops.rmsnorm(x.cuda(), w.cuda(), 2e-5, some, rows=i32(rows), parts=parts)
    assert torch.equal(some, out[rows])
    if parts > 1:
        assert rel(out, P.part_norm(x.double(), w.double(), 2e-5, 1)) > 1e-2


def test_norm_refuses_parts_that_do_not_divide_the_row():
    from llmplayer_b200.errors import KernelError
    from llmplayer_b200.kernels import ops
    x, w, out = torch.randn(2, 10).cuda(), torch.ones(10).cuda(), torch.empty(2, 10).cuda()
    with pytest.raises(KernelError):
        ops.rmsnorm(x, w, 1e-5, out, parts=3)


@pytest.mark.parametrize("T,d,parts", [(5, 72, 3), (1, 8, 1), (3, 1000, 40), (19, 52, 2), (2, 4100, 4), (3, 12288, 2), (2, 600, 600)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_two_normed_results_summed(T, d, parts, dtype):
    from llmplayer_b200.kernels import ops
    torch.manual_seed(d)
    x, a, b = torch.randn(T, d), 5 * torch.randn(T, d), 0.2 * torch.randn(T, d)
    wa, wb, wn = 1 + 0.3 * torch.randn(d), 1 + 0.3 * torch.randn(d), 1 + 0.3 * torch.randn(d)
    ref = x.double() + 0.5 * (P.unit_rms(a.double(), 1e-5) * wa.double()) + 0.25 * (P.unit_rms(b.double(), 3e-4) * wb.double())
    got = x.cuda()
    ops.pair_norm_add(a.cuda(), wa.cuda(), 0.5, 1e-5, b.cuda(), wb.cuda(), 0.25, 3e-4, got)
    check_error("two normed results summed, float32", f"{T}x{d}", rel(got, ref), 2e-6)
    got, nxt = x.cuda(), torch.empty(T, d, dtype=dtype, device="cuda")
    junk = torch.full((4000,), 3.0, device="cuda")
    ops.pair_norm_add(a.cuda(), wa.cuda(), 0.5, 1e-5, b.cuda(), wb.cuda(), 0.25, 3e-4, got, next_weight=wn.cuda(), next_eps=2e-6,
                      next_parts=parts, next_out=nxt, clear=junk)
    assert rel(got, ref) < 2e-6 and float(junk.abs().max()) == 0.0
    check_error(f"two normed results summed, the next norm in parts, {dtype}", f"{T}x{d} in {parts}",
                rel(nxt, P.part_norm(ref, wn.double(), 2e-6, parts)), 3e-6 if dtype == torch.float32 else 5e-3)


# --------------------------------------------------------------------------- gates from low-rank maps
@pytest.mark.parametrize("T,H,dk,ra,dv,rg", [(1, 2, 16, 3, 24, 5), (70, 4, 20, 24, 12, 24), (130, 3, 64, 40, 48, 1), (5, 1, 6, 100, 10, 33)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_gates_from_low_rank_maps(T, H, dk, ra, dv, rg, dtype):
    from llmplayer_b200.kernels import ops
    torch.manual_seed(T + ra)
    proj = torch.randn(T, 7 + H + ra + rg + 3)
    b_off, a_off = 7, 7 + H
    g_off = a_off + ra
    a_up, g_up = (torch.randn(H * dk, ra) / ra ** 0.5).to(dtype), (torch.randn(H * dv, rg) / rg ** 0.5).to(dtype)
    dt_bias, a_log = 2 * torch.randn(H * dk), torch.randn(H)
    dt_bias[0], dt_bias[1] = 40.0, -40.0                         # beyond where a naive softplus overflows, and nearly no decay
    decay, strength, gate = torch.empty(T, H * dk).cuda(), torch.empty(T, H).cuda(), torch.empty(T, H * dv).cuda()
    ops.low_rank_gates(proj.cuda(), a_off, a_up.cuda(), dt_bias.cuda(), a_log.cuda(), decay, b_off, strength, key_dim=dk, g_off=g_off,
                       g_up=g_up.cuda(), gate=gate)
    p = proj.double()
    z = p[:, a_off:a_off + ra] @ a_up.double().T + dt_bias.double()
    ref = torch.exp(-torch.exp(a_log.double())[None, :, None] * P.softplus(z).reshape(T, H, dk)).reshape(T, H * dk)
    check_error("decays from a low-rank map", f"{T} x {H} x {dk}, rank {ra}", rel(decay, ref), 5e-6)
    assert rel(strength, torch.sigmoid(p[:, b_off:b_off + H])) < 2e-6
    assert rel(gate, p[:, g_off:g_off + rg] @ g_up.double().T) < 3e-6
    again = torch.empty_like(decay)
    ops.low_rank_gates(proj.cuda(), a_off, a_up.cuda(), dt_bias.cuda(), a_log.cuda(), again, b_off, strength, key_dim=dk)
    assert torch.equal(again, decay)


# --------------------------------------------------------------------------- recurrences
def run_steps(data, steps, dims, slots, state, **kw):
    """The recurrence over steps of given lengths per sequence; ``data``: per sequence a dict of its tokens' tensors."""
    from llmplayer_b200.kernels import ops
    H, G, dk, dv = dims
    done, got = [0] * len(data), [[] for _ in data]
    for step in steps:
        def cat(name):
            return torch.cat([d[name][at:at + n].reshape(n, -1) for d, at, n in zip(data, done, step)])
        mixed = torch.cat([cat("q"), cat("k"), cat("v")], dim=1).float().cuda()
        starts = [0]
        for n in step:
            starts.append(starts[-1] + n)
        args = dict(kw)
        if "fixed" in args:
            decay = args.pop("fixed")
            args["decay_fixed"] = True
        else:
            decay = cat("g").float().cuda()
        if "beta" in data[0]:
            args["delta_strength"] = cat("beta").float().cuda()
        if "rotation" in args:
            positions = i32([at + i for at, n in zip(done, step) for i in range(n)])
            angles = torch.empty(sum(step), args["rotation"].rotary_dim // 2, 2, device="cuda")
            ops.rope_angles(positions, args["rotation"], angles)
            args["angles"] = angles
        out = torch.full((sum(step), H * dv), float("nan"), device="cuda")
        ops.gla_scan(mixed, 0, G * dk, 2 * G * dk, decay, state, i32(slots), i32(starts), out, num_heads=H, key_dim=dk, value_dim=dv,
                     max_new=max(step), scratch=scratch, qk_heads=G, **args)
        for i, n in enumerate(step):
            got[i].append(out[starts[i]:starts[i] + n].cpu())
            done[i] += n
    return [torch.cat(g).reshape(-1, H, dv) for g in got]


STEPS = ([1, 1], [2, 31], [117, 2], [32, 33], [300, 300], [1, 1])
LENGTHS = [sum(s[i] for s in STEPS) for i in (0, 1)]


@pytest.mark.parametrize("products", [False, True])
@pytest.mark.parametrize("H,G,dk,dv,low", [(4, 2, 20, 12, 0.5), (2, 1, 16, 24, 0.9), (2, 2, 128, 128, 0.7), (4, 2, 64, 32, 0.0), (1, 1, 6, 10, 0.3),
                                          (3, 3, 256, 40, 0.8), (2, 1, 33, 70, 0.0), (1, 1, 240, 16, 0.95)])
def test_delta_rule_with_a_decay_per_channel(H, G, dk, dv, low, products):
    """Steps of 1 to 300 tokens of two sequences in slots 2 and 3 (prompt portions that start from a state that is not
    zero, chunks cut short, single tokens between them); slots 0 and 1 stay as they were. Decays from ``low`` to one
    differ from channel to channel; some are zero or nearly so (whole channels forget at once)."""
    torch.manual_seed(dk + dv)
    state = torch.zeros(4, H, dv, dk, device="cuda")
    state[0] = -4.0
    data, refs = [], []
    for n in LENGTHS:
        q, k = torch.randn(n, G, dk).double(), torch.randn(n, G, dk).double()
        d = {"q": (P.unit_length(q) * dk ** -0.5).float(), "k": P.unit_length(k).float(), "v": torch.randn(n, H, dv),
             "g": (low + (1 - low) * torch.rand(n, H, dk)), "beta": torch.rand(n, H)}
        d["g"][5::37] = 0.0
        d["g"][11::23, :, ::3] = 1e-30
        d["g"][40:60] **= 8                                       # a stretch of strong decays: their product underflows
        data.append(d)
        refs.append(P.channel_delta_recurrence(d["q"].double().repeat_interleave(H // G, 1), d["k"].double().repeat_interleave(H // G, 1),
                                               d["v"].double(), d["g"].double(), d["beta"].double()))
    got = run_steps(data, STEPS, (H, G, dk, dv), [2, 3], state, q_scale=1.0, tensor_cores=products)
    for i in (0, 1):
        check_error(f"delta rule with a decay per channel, {'products' if products else 'token by token'}",
                    f"{H} heads on {G}, {dk} x {dv}, sequence {i}", rel(got[i], refs[i][0]), 2e-5)
        assert rel(state[[2, 3][i]].transpose(1, 2), refs[i][1]) < 2e-5
    assert float((state[0] + 4.0).abs().max()) == 0.0 and float(state[1].abs().max()) == 0.0


@pytest.mark.parametrize("H,dk,dv", [(2, 64, 64), (3, 24, 40)])
def test_delta_rule_in_chunks_with_one_decay_per_head(H, dk, dv):
    """The form with one decay per head through the same chunks; and full strength without decay under few keys, where
    every write replaces what its key held (the triangular solve is then far from the identity)."""
    torch.manual_seed(dk)
    for hard in (False, True):
        state = torch.zeros(2, H, dv, dk, device="cuda")
        n = 200
        q, k = torch.randn(n, H, dk).double(), torch.randn(n, H, dk).double()
        if hard:
            k = k[:4].repeat(50, 1, 1) + 0.05 * k                 # four directions, over and over
        d = {"q": P.unit_length(q).float(), "k": P.unit_length(k).float(), "v": torch.randn(n, H, dv),
             "g": torch.ones(n, H) if hard else 0.5 + 0.5 * torch.rand(n, H), "beta": torch.ones(n, H) if hard else torch.rand(n, H)}
        ref, S = P.channel_delta_recurrence(d["q"].double(), d["k"].double(), d["v"].double(), d["g"].double()[:, :, None].expand(n, H, dk),
                                            d["beta"].double())
        got = run_steps([d], ([70], [130]), (H, H, dk, dv), [1], state, q_scale=1.0, tensor_cores=True, decay_per_head=True)
        check_error("delta rule in chunks, one decay per head", f"{H} x {dk} x {dv}, {'hard' if hard else 'usual'}", rel(got[0], ref), 5e-5)
        assert rel(state[1].transpose(1, 2), S) < 5e-5 and float(state[0].abs().max()) == 0.0


@pytest.mark.parametrize("products", [False, True])
@pytest.mark.parametrize("H,dk,dv,rd,decay", [(3, 64, 40, 64, [0.97, 0.99, 0.9975]), (2, 20, 40, 8, [0.5, 1.0]), (1, 128, 256, 128, [0.97]),
                                              (3, 16, 10, 0, [0.0, 0.9, 0.3]), (2, 256, 24, 2, [0.99, 1e-20])])
def test_retention_over_steps_and_slots(H, dk, dv, rd, decay, products):
    """Fixed decays per head (one of them zero: only the token itself; one of them one: nothing is forgotten), queries and
    keys rotated on the way by their positions, which go on from step to step."""
    from llmplayer_b200.kernels import ops
    torch.manual_seed(dk + rd)
    base = 10000.0
    freqs = torch.tensor([base ** (-2.0 * i / rd) for i in range(rd // 2)], dtype=torch.float64).float().cuda() if rd else None
    rotation = ops.Rotation(freqs, rd, False) if rd else ops.NO_ROTATION
    state = torch.zeros(5, H, dv, dk, device="cuda")
    data, refs = [], []
    for n in LENGTHS:
        d = {"q": torch.randn(n, H, dk), "k": torch.randn(n, H, dk), "v": torch.randn(n, H, dv)}
        pos = torch.arange(n)
        q, k = P.rotate_half(d["q"].double(), pos, base, rd), P.rotate_half(d["k"].double(), pos, base, rd) * dk ** -0.5
        refs.append(P.retention_recurrence(q, k, d["v"].double(), torch.tensor(decay, dtype=torch.float64)))
        data.append(d)
    got = run_steps(data, STEPS, (H, H, dk, dv), [4, 0], state, q_scale=dk ** -0.5, tensor_cores=products,
                    fixed=torch.tensor(decay).cuda(), **({"rotation": rotation} if rd else {}))
    for i in (0, 1):
        # angles are float32 products: position x frequency is rounded (1e-5 relative at these positions)
        check_error(f"retention, {'products' if products else 'token by token'}", f"{H} x {dk} x {dv}, rotation {rd}, sequence {i}",
                    rel(got[i], refs[i][0]), 3e-5)
        assert rel(state[[4, 0][i]].transpose(1, 2) * dk ** -0.5, refs[i][1]) < 3e-5
    assert float(state[1:4].abs().max()) == 0.0


def test_chunks_in_several_rounds(monkeypatch):
    """Little room for the chunks' records: the same prompt in several rounds, each from the state the one before left."""
    from llmplayer_b200.kernels import ops
    torch.manual_seed(5)
    H, dk, dv, n = 2, 32, 48, 333
    d = {"q": torch.randn(n, H, dk), "k": P.unit_length(torch.randn(n, H, dk).double()).float(), "v": torch.randn(n, H, dv),
         "g": torch.rand(n, H, dk), "beta": torch.rand(n, H)}
    e = {name: t[:100] for name, t in d.items()}
    want = torch.zeros(2, H, dv, dk, device="cuda")
    ref = run_steps([d, e], ([333, 100],), (H, H, dk, dv), [0, 1], want, q_scale=1.0, tensor_cores=True)
    monkeypatch.setattr(ops, "CHUNKED_BUFFER_BYTES", 200 * 1024)
    state = torch.zeros(2, H, dv, dk, device="cuda")
    got = run_steps([d, e], ([333, 100],), (H, H, dk, dv), [0, 1], state, q_scale=1.0, tensor_cores=True)
    assert torch.equal(state, want) and all(torch.equal(a, b) for a, b in zip(got, ref))


@pytest.mark.parametrize("products", [False, True])
def test_an_early_token_comes_through_hundreds_of_steps(products):
    """One token writes under a key of its own; hundreds of later tokens write elsewhere; its channel hardly decays while all
    other channels forget at once. A read-out under that key much later must return its value, times the decays since."""
    torch.manual_seed(9)
    dk, dv, n = 32, 16, 700
    k = torch.zeros(n, 1, dk)
    k[:, 0, 1 + torch.randint(0, dk - 1, (n,))] = 0.0
    k[torch.arange(n), 0, 1 + torch.randint(0, dk - 1, (n,))] = 1.0
    k[3] = 0.0
    k[3, 0, 0] = 1.0
    q = torch.zeros(n, 1, dk)
    q[:, 0, 0] = 1.0
    v = torch.randn(n, 1, dv)
    g = torch.full((n, 1, dk), 0.01)
    g[:, :, 0] = 0.999
    d = {"q": q, "k": k, "v": v, "g": g, "beta": torch.ones(n, 1)}
    got = run_steps([d], ([n],), (1, 1, dk, dv), [0], torch.zeros(1, 1, dv, dk, device="cuda"), q_scale=1.0, tensor_cores=products)[0]
    ref = v[3, 0].double() * 0.999 ** torch.arange(0, n - 3)[:, None].double()
    assert float((got[3:, 0].double() - ref).abs().max()) < 2e-5 * float(v[3].abs().max())
    assert float(got[:3].abs().max()) == 0.0


# --------------------------------------------------------------------------- what leads up to the recurrence; single steps
@pytest.mark.parametrize("G,dk,rest,K", [(2, 20, 30, 4), (1, 128, 256, 4), (3, 64, 50, 2), (1, 6, 10, 1), (2, 130, 7, 8), (5, 33, 200, 3), (1, 512, 64, 4)])
def test_convolutions_with_unit_heads_behind_them(G, dk, rest, K):
    """Steps of 1, 2, 31, 33 and 100 tokens of two sequences: kept inputs carry over (zeros before the start), queries also
    times dk^-1/2, the other channels pass unnormed; other slots stay as they were."""
    from llmplayer_b200.kernels import ops
    torch.manual_seed(dk + K)
    C = 2 * G * dk + rest
    taps = 0.6 * torch.randn(C, K)
    tail = torch.zeros(4, K - 1, C, device="cuda")
    tail[1] = 7.0
    steps = ([1, 2], [33, 1], [2, 100], [100, 31])
    lengths = [sum(s[i] for s in steps) for i in (0, 1)]
    xs = [torch.randn(n, C + 9) for n in lengths]
    refs = []
    for x in xs:
        y = P.silu(P.short_convolution(x.double()[:, 4:4 + C], taps.double()))
        heads = P.unit_length(y[:, :2 * G * dk].reshape(-1, 2 * G, dk))
        heads[:, :G] *= dk ** -0.5
        refs.append(torch.cat([heads.reshape(-1, 2 * G * dk), y[:, 2 * G * dk:]], dim=1))
    done, got = [0, 0], [[], []]
    for step in steps:
        x = torch.cat([x[at:at + n] for x, at, n in zip(xs, done, step)]).cuda()
        out = torch.full((sum(step), C), float("nan"), device="cuda")
        ops.conv_unit_heads(x[:, 4:4 + C], taps.cuda(), tail, i32([3, 0]), i32([0, step[0], sum(step)]), out, max_new=max(step),
                            heads=2 * G, dim=dk, eps=1e-6, scale=dk ** -0.5, scaled_heads=G)
        got[0].append(out[:step[0]].cpu())
        got[1].append(out[step[0]:].cpu())
        done = [at + n for at, n in zip(done, step)]
    for i in (0, 1):
        check_error("convolutions with unit heads, float32", f"{2 * G} heads of {dk} and {rest} channels, {K} taps, sequence {i}",
                    rel(torch.cat(got[i]), refs[i]), 5e-6)
    assert K == 1 or float((tail[1] - 7.0).abs().max()) == 0.0 and float(tail[2].abs().max()) == 0.0


@pytest.mark.parametrize("low_rank", [True, False])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,dk,dv,ra,rg,K", [(3, 3, 64, 48, 40, 16, 4), (2, 1, 20, 12, 8, 5, 3), (2, 2, 128, 128, 128, 128, 4), (6, 2, 6, 70, 3, 16, 1),
                                              (1, 1, 256, 40, 40, 8, 2), (2, 1, 130, 300, 16, 24, 8), (1, 1, 300, 10, 7, 7, 4)])
def test_single_steps_in_one_kernel(H, G, dk, dv, ra, rg, K, dtype, low_rank):
    """60 steps of one token for three sequences (in slots 4, 0 and 2): projection in, gated heads out, against the plain
    mechanisms over the whole sequences; both forms of decays and gates; the slots between stay as they were."""
    from llmplayer_b200.kernels import ops
    torch.manual_seed(dk + dv)
    n, B, off = 60, 3, 3
    C = 2 * G * dk + H * dv
    rows = (ra, rg) if low_rank else (H, H * dv)
    F = off + C + H + rows[0] + rows[1] + 2
    cols = (off, off + C, off + C + H, off + C + H + rows[0])
    x = torch.randn(B, n, F)
    taps, gain = 0.6 * torch.randn(C, K), 1 + 0.3 * torch.randn(dv)
    a_log = torch.randn(H)
    dt_bias = 1.5 * torch.randn(H * dk if low_rank else H)
    a_up = (torch.randn(H * dk, ra) / ra ** 0.5).to(dtype) if low_rank else None
    g_up = (torch.randn(H * dv, rg) / rg ** 0.5).to(dtype) if low_rank else None
    state, tail = torch.zeros(5, H, dv, dk, device="cuda"), torch.zeros(5, K - 1, C, device="cuda")
    state[1], tail[3] = 2.0, 5.0
    slots = i32([4, 0, 2])
    junk = torch.full((5000,), 3.0, device="cuda")
    got = []
    up = {} if not low_rank else {"a_up": a_up.cuda(), "g_up": g_up.cuda()}
    for t in range(n):
        out = torch.full((B, H * dv), float("nan"), device="cuda", dtype=dtype)
        ops.delta_step(x[:, t].contiguous().cuda(), cols, taps.cuda(), tail, state, slots, dt_bias.cuda(), a_log.cuda(), gain.cuda(), 1e-5, out,
                       num_heads=H, qk_heads=G, key_dim=dk, value_dim=dv, unit_eps=1e-6, q_scale=dk ** -0.5, gate_sigmoid=low_rank, clear=junk, **up)
        got.append(out.float().cpu())
    assert float(junk.abs().max()) == 0.0
    got = torch.stack(got, dim=1)
    for b in range(B):
        p = x[b].double()
        y = P.silu(P.short_convolution(p[:, off:off + C], taps.double()))
        q = (P.unit_length(y[:, :G * dk].reshape(n, G, dk)) * dk ** -0.5).repeat_interleave(H // G, 1)
        k = P.unit_length(y[:, G * dk:2 * G * dk].reshape(n, G, dk)).repeat_interleave(H // G, 1)
        v = y[:, 2 * G * dk:].reshape(n, H, dv)
        beta = torch.sigmoid(p[:, cols[1]:cols[1] + H])
        z = p[:, cols[2]:cols[2] + rows[0]]
        z = (z @ a_up.double().T if low_rank else z) + dt_bias.double()
        z = P.softplus(z).reshape(n, H, -1)
        g = torch.exp(-torch.exp(a_log.double())[None, :, None] * z).expand(n, H, dk)
        o, S = P.channel_delta_recurrence(q, k, v, g, beta)
        gate = p[:, cols[3]:cols[3] + rows[1]]
        gate = torch.sigmoid(gate @ g_up.double().T) if low_rank else P.silu(gate)
        ref = (P.unit_rms(o, 1e-5) * gain.double()).reshape(n, H * dv) * gate
        # a head whose output nearly cancels is divided by its small root mean square: rounding is amplified there
        err = ((got[b].double() - ref).abs() / ref.abs().max()).flatten().sort().values
        assert torch.isfinite(got).all()
        lim = 1e-4 if dtype == torch.float32 else 5e-3
        check_error(f"single delta-rule steps, {dtype}", f"{H} heads on {G}, {dk} x {dv}, sequence {b}", float(err[-1]), lim)
        check_error(f"single delta-rule steps, the state, {dtype}", f"{H} heads on {G}, {dk} x {dv}", rel(state[[4, 0, 2][b]].transpose(1, 2), S), 1e-5)
    assert float((state[1] - 2.0).abs().max()) == 0.0 and float(state[3].abs().max()) == 0.0 and (K == 1 or float((tail[3] - 5.0).abs().max()) == 0.0)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,dk,dv,rd,decay", [(3, 64, 40, 64, [0.97, 0.99, 0.9975]), (2, 20, 300, 8, [0.5, 1.0]), (1, 128, 256, 128, [0.97]),
                                              (3, 6, 10, 0, [0.0, 0.9, 0.3]), (2, 256, 24, 2, [0.99, 0.4]), (1, 301, 12, 300, [0.9])])
def test_single_retention_steps_in_one_kernel(H, dk, dv, rd, decay, dtype):
    """60 steps of one token for three sequences in slots 4, 0 and 2 that started at positions of their own."""
    from llmplayer_b200.kernels import ops
    torch.manual_seed(dk + rd)
    n, B, off, base = 60, 3, 2, 5000.0
    freqs = torch.tensor([base ** (-2.0 * i / rd) for i in range(rd // 2)], dtype=torch.float64).float().cuda() if rd else None
    rotation = ops.Rotation(freqs, rd, False) if rd else ops.NO_ROTATION
    cols = (off, off + H * dk, off + 2 * H * dk, off + 2 * H * dk + H * dv)
    x = torch.randn(B, n, cols[3] + H * dv + 3)
    starts = [0, 7, 100]
    state = torch.zeros(5, H, dv, dk, device="cuda")
    state[1] = 2.0
    junk = torch.full((5000,), 3.0, device="cuda")
    got = []
    for t in range(n):
        out = torch.full((B, H * dv), float("nan"), device="cuda", dtype=dtype)
        ops.retention_step(x[:, t].contiguous().cuda(), cols, rotation, i32([s + t for s in starts]), torch.tensor(decay).cuda(), state,
                           i32([4, 0, 2]), 1e-5, out, num_heads=H, key_dim=dk, value_dim=dv, q_scale=dk ** -0.5, clear=junk)
        got.append(out.float().cpu())
    got = torch.stack(got, dim=1)
    assert float(junk.abs().max()) == 0.0 and torch.isfinite(got).all()
    for b in range(B):
        p, pos = x[b].double(), torch.arange(n) + starts[b]
        q = P.rotate_half(p[:, cols[0]:cols[1]].reshape(n, H, dk), pos, base, rd)
        k = P.rotate_half(p[:, cols[1]:cols[2]].reshape(n, H, dk), pos, base, rd) * dk ** -0.5
        o, S = P.retention_recurrence(q, k, p[:, cols[2]:cols[3]].reshape(n, H, dv), torch.tensor(decay, dtype=torch.float64))
        ref = P.unit_rms(o, 1e-5).reshape(n, H * dv) * P.silu(p[:, cols[3]:cols[3] + H * dv])
        err = float((got[b].double() - ref).abs().max() / ref.abs().max())
        check_error(f"single retention steps, {dtype}", f"{H} x {dk} x {dv}, rotation {rd}, sequence {b}", err, 1e-4 if dtype == torch.float32 else 5e-3)
        assert rel(state[[4, 0, 2][b]].transpose(1, 2) * dk ** -0.5, S) < 2e-5
    assert float((state[1] - 2.0).abs().max()) == 0.0 and float(state[3].abs().max()) == 0.0


# --------------------------------------------------------------------------- output gate without a gain
def test_heads_normed_without_a_gain():
    from llmplayer_b200.kernels import ops
    torch.manual_seed(3)
    T, H, dv = 21, 3, 40
    o, gate = torch.randn(T, H * dv), torch.randn(T, H * dv + 5)
    for sigmoid in (False, True):
        out = torch.empty(T, H * dv, device="cuda")
        ops.gla_finish(o.cuda(), None, 1e-5, gate.cuda()[:, 2:2 + H * dv], out, num_heads=H, value_dim=dv, gate_sigmoid=sigmoid)
        z = gate.double()[:, 2:2 + H * dv]
        ref = P.unit_rms(o.double().reshape(T, H, dv), 1e-5).reshape(T, H * dv) * (torch.sigmoid(z) if sigmoid else P.silu(z))
        assert rel(out, ref) < 2e-6


# --------------------------------------------------------------------------- attention in chunks with a distance bias
def fill_pages(k, v, table_rows, num_pages, dtype):
    T, G, hd = k.shape
    pages = torch.zeros(num_pages, 2, G, PAGE, hd, dtype=dtype, device="cuda")
    for t in range(T):
        page = table_rows[t // PAGE]
        pages[page, 0, :, t % PAGE] = k[t].to(dtype)
        pages[page, 1, :, t % PAGE] = v[t].to(dtype)
    return pages


def plain_attention(q, k, v, scale, r1, r2, chunk, first):
    """The last rows of the plain function: q holds the queries from position ``first`` on."""
    H, length = q.shape[1], k.shape[0]
    full = torch.zeros(length, H, q.shape[2], dtype=q.dtype)
    full[first:] = q
    group = H // k.shape[1]
    return P.distance_attention(full, k.repeat_interleave(group, 1), v.repeat_interleave(group, 1), scale, r1, r2,
                                P.chunk_visible(length, chunk))[first:]


def run_attention(kind, qd, pages, table, length, new, chunk, distance, H, G, hd, scale):
    from llmplayer_b200.kernels import ops
    out = torch.full_like(qd, float("nan"))
    kw = dict(num_heads=H, num_kv_heads=G, head_dim=hd, scale=scale, window=None, chunk=chunk or 0, distance=distance)
    if kind == "plain":
        ops.attention_plain(qd, out, pages, table, i32([0] * new), i32(list(range(length - new, length))), **kw)
    elif kind == "prompt":
        ops.attention_prefill(qd, out, pages, table, i32([0, new]), i32([length]), new, exact_weights=True, **kw)
    else:
        ops.attention_decode(qd, out, pages, table, i32([length]), scratch, exact_weights=True, **kw)
    return out


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("bias", [True, False])
@pytest.mark.parametrize("H,G,hd,length,new,chunk", [(4, 2, 48, 200, 200, 9), (8, 1, 64, 321, 321, 64), (2, 2, 128, 400, 57, 128), (6, 2, 96, 700, 700, 200),
                                                     (5, 1, 16, 130, 130, 1), (2, 1, 64, 400, 300, 65), (3, 3, 16, 300, 1, 256), (2, 2, 64, 260, 2, 257),
                                                     (8, 1, 64, 900, 1, 1000), (6, 2, 128, 1000, 1, 300), (4, 4, 32, 961, 1, 60), (2, 2, 192, 300, 300, 100),
                                                     (2, 1, 192, 200, 1, 70), (20, 2, 64, 450, 450, None), (2, 1, 112, 333, 140, 50), (12, 1, 64, 700, 1, None)])
def test_attention_in_chunks_with_a_distance_bias(dtype, H, G, hd, length, new, chunk, bias):
    """The last ``new`` tokens of a sequence of ``length`` see the earlier tokens of their own chunk (pages in a scrambled
    order; pages of finished chunks are not in the table at all): the plain kernel in float32 and bfloat16, the tensor-core
    prompt and decode kernels in bfloat16. One position more or less in a chunk differs."""
    torch.manual_seed(length + hd)
    scale = 0.3
    q = torch.randn(new, H, hd).to(dtype)
    k, v = torch.randn(length, G, hd).to(dtype), torch.randn(length, G, hd).to(dtype)
    rows = torch.randperm(16).tolist()[:-(-length // PAGE)]
    pages = fill_pages(k, v, rows, 16, dtype)
    first = length - new
    needed = first // chunk * chunk if chunk else 0               # what the cache would have given back by now
    table = i32([r if b >= needed // PAGE else -1 for b, r in enumerate(rows)] + [0] * (16 - len(rows))).view(1, -1)
    r1, r2 = torch.rand(H) * 2 + 0.1, torch.rand(H) * 3 + 0.05
    distance = (r1.cuda(), r2.cuda()) if bias else None
    ref = plain_attention(q.double(), k.double(), v.double(), scale, r1.double() if bias else None, r2.double(), chunk, first)
    qd = q.reshape(new, H * hd).cuda()
    kinds = [("plain", 3e-6)] if dtype == torch.float32 else [("plain", 6e-3), ("prompt", 6e-3) if new > 1 else ("decode", 6e-3)]
    full = i32(rows + [0] * (16 - len(rows))).view(1, -1)
    for kind, lim in kinds:
        out = run_attention(kind, qd, pages, table, length, new, chunk, distance, H, G, hd, scale)
        check_error(f"attention in chunks, {kind} kernel, {dtype}", f"{H}/{G} x {hd}, {new} of {length}, chunks of {chunk}, bias {bias}",
                    rel(out.view(new, H, hd), ref), lim)
        if chunk and chunk < 70 and new > 1:
            off = run_attention(kind, qd, pages, full, length, new, chunk + 1, distance, H, G, hd, scale)
            assert rel(off.view(new, H, hd), ref) > 1e-3
        if bias and new > 1 and chunk != 1:
            swapped = (distance[1], distance[0])
            off = run_attention(kind, qd, pages, full, length, new, chunk, swapped, H, G, hd, scale)
            assert rel(off.view(new, H, hd), ref) > 1e-3


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("step", ["prompt", "decode"])
@pytest.mark.parametrize("length,chunk", [(700, 200), (700, 64), (700, 65), (641, 128), (300, 33), (200, 9), (130, 2), (130, 1), (601, 600), (600, 601), (193, 192)])
def test_a_key_at_the_edges_of_a_chunk(dtype, step, length, chunk):
    """Head 1's last query is made to fit ONE key far better than all others. On the first position of the query's chunk its
    value must come through nearly alone, however long ago that was; on the last position of the chunk before it must not
    be seen at all. A prompt step of 40 tokens (which may cross a border itself) and a one-token step."""
    torch.manual_seed(chunk)
    H, G, hd, scale = 4, 2, 64, 0.5
    new = 40 if step == "prompt" else 1
    direction = torch.randn(hd)
    direction /= direction.norm()
    last = length - 1
    start = last // chunk * chunk
    r1, r2 = torch.full((H,), 0.7), torch.full((H,), 0.5)
    for at, seen in ((start, True), (start - 1, False), (last, True), (0, start == 0)):
        if at < 0:
            continue
        k, v = 0.3 * torch.randn(length, G, hd), torch.randn(length, G, hd)
        q = 0.3 * torch.randn(new, H, hd)
        q[-1, 1] = 8.0 * direction
        k[at, 0] = 8.0 * direction                             # score 64 * 0.5 = 32, less a bias of at most 4, against scores near 0
        k, v, q = k.to(dtype), v.to(dtype), q.to(dtype)
        rows = torch.randperm(16).tolist()[:-(-length // PAGE)]
        pages = fill_pages(k, v, rows, 16, dtype)
        table = i32(rows + [0] * (16 - len(rows))).view(1, -1)
        qd = q.reshape(new, H * hd).cuda()
        kind = "plain" if dtype == torch.float32 else step
        out = run_attention(kind, qd, pages, table, length, new, chunk, (r1.cuda(), r2.cuda()), H, G, hd, scale).view(new, H, hd)
        ref = plain_attention(q.double(), k.double(), v.double(), scale, r1.double(), r2.double(), chunk, length - new)
        check_error(f"attention in chunks, a key that stands out, {step}, {dtype}", f"length {length}, chunks of {chunk}, key at {at}",
                    rel(out, ref), 3e-6 if dtype == torch.float32 else 6e-3)
        got = out[-1, 1].double().cpu()
        if seen:
            assert float((got - v[at, 0].double()).abs().max()) < 1e-3 + (0.02 if dtype == torch.bfloat16 else 0.0), at
        else:
            assert float((got - v[at, 0].double()).abs().max()) > 0.5, at


def test_a_distance_bias_falls_with_the_logarithm():
    """Equal scores for all keys: the weights are then (1 + r2 n)^(-r1), known in closed form, near and far."""
    from llmplayer_b200.kernels import ops
    length, hd = 512, 64
    r1, r2 = torch.tensor([1.5, 0.2]), torch.tensor([0.8, 6.0])
    k, q = torch.zeros(length, 1, hd), torch.zeros(1, 2, hd)
    v = torch.zeros(length, 1, hd)
    for j, at in enumerate((511, 510, 448, 447, 300, 1, 0)):
        v[at, 0, j] = 1.0
    for dtype, kind in ((torch.float32, "plain"), (torch.bfloat16, "decode")):
        rows = list(range(8))
        pages = fill_pages(k.to(dtype), v.to(dtype), rows, 8, dtype)
        out = run_attention(kind, q.reshape(1, -1).to(dtype).cuda(), pages, i32(rows).view(1, -1), length, 1, None, (r1.cuda(), r2.cuda()), 2, 1, hd, 0.4)
        n = (length - 1 - torch.arange(length)).double()
        for h in range(2):
            w = (1.0 + r2[h].double() * n) ** (-r1[h].double())
            w = w / w.sum()
            for j, at in enumerate((511, 510, 448, 447, 300, 1, 0)):
                got = float(out.view(2, hd)[h, j])
                assert math.isclose(got, float(w[at]), rel_tol=2e-6 if dtype == torch.float32 else 5e-3), (kind, h, at)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,dk,dv", [(4, 2, 24, 40), (3, 3, 16, 8), (2, 1, 64, 48)])
def test_values_are_cached_divided_by_their_root_mean_square(dtype, H, G, dk, dv):
    """From a column slice of a wider product; queries and keys pass unchanged, heads are padded with zeros."""
    from llmplayer_b200.kernels import ops
    torch.manual_seed(dv)
    T, off = 70, 5
    hdp = -(-max(dk, dv) // 16) * 16
    F = (H + G) * dk + G * dv
    wide = 3 * torch.randn(T, off + F + 9)
    q_out = torch.empty(T, H * hdp, dtype=dtype, device="cuda")
    pages = torch.zeros(3, 2, G, PAGE, hdp, dtype=dtype, device="cuda")
    ops.qkv_prepare(wide.cuda()[:, off:off + F], None, ops.NO_ROTATION, i32(list(range(T))), i32([0] * T), i32([[2, 0]]), q_out, pages,
                    num_heads=H, num_kv_heads=G, key_dim=dk, value_dim=dv, unit_norm_eps=None, value_norm_eps=1e-3)
    x = wide.double()[:, off:off + F]
    lim = 2e-6 if dtype == torch.float32 else 5e-3
    got_q = q_out.view(T, H, hdp)
    assert rel(got_q[..., :dk], x[:, :H * dk].reshape(T, H, dk)) < lim and float(got_q[..., dk:].abs().sum()) == 0.0
    kv = torch.cat([pages[2], pages[0]], dim=2).cpu()                 # [2, G, 128, hdp]
    assert rel(kv[0, :, :T, :dk].transpose(0, 1), x[:, H * dk:(H + G) * dk].reshape(T, G, dk)) < lim
    ref = P.unit_rms(x[:, (H + G) * dk:].reshape(T, G, dv), 1e-3)
    check_error(f"cached values, {dtype}", f"{H}/{G} x {dk} / {dv}", rel(kv[1, :, :T, :dv].transpose(0, 1), ref), lim)
    assert float(kv[1, :, :T, dv:].abs().sum()) == 0.0 and float(pages[1].abs().sum()) == 0.0
