"""Each mechanism of the Zotolix decoder alone, its kernels against the plain implementation's function: what stands
between two sublayers of a bundle of streams, values shown to and blended by later layers, gated heads in the prompt, decode
and plain attention kernels (in chunks, with keys that stand out at a chunk's borders, over shares that are merged), unit-norm
heads behind additive vectors, squared-ReLU experts weighted on their input, and the parts put together."""
import pytest
import torch

import plain_zotolix as P
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


# --------------------------------------------------------------------------- streams
@pytest.mark.parametrize("S,T,d", [(1, 3, 53), (2, 5, 64), (3, 7, 72), (4, 9, 200), (4, 2, 4096), (5, 3, 96), (8, 2, 1024), (7, 4, 30),
                                   (32, 2, 100), (4, 1, 15000), (3, 2, 14001), (6, 300, 8)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_streams_between_two_sublayers(S, T, d, dtype):
    """Every form of the kernel: before the first sublayer (equal streams, nothing to bring in), behind it (equal streams
    become different ones), between later ones (in place), behind the last one (the plain sum, nothing else stored)."""
    from llmplayer_b200.kernels import ops
    torch.manual_seed(S * 100 + d)
    X, x0, y = torch.randn(S, T, d), torch.randn(T, d), torch.randn(T, d)
    M, b, a, w = torch.randn(S, S), torch.randn(S), torch.randn(S), 1 + 0.3 * torch.randn(d)
    dM, db, da, dw, dy = (t.cuda() for t in (M, b, a, w, y))
    m, eps = 0.7, 3e-5
    lim = 3e-6 if dtype == torch.float32 else 5e-3
    X6, M6, b6, a6, w6, y6, x6 = (t.double() for t in (X, M, b, a, w, y, x0))
    equal6 = torch.stack([x6] * S)
    kind = f"{S} streams of {T} x {d}"

    def out():
        return torch.full((T, d), float("nan"), dtype=dtype, device="cuda")
    junk = torch.full((777,), 3.0, device="cuda")
    h = out()
    ops.stream_bundle(x0.cuda(), streams=S, gather=da, weight=dw, eps=eps, normed=h, clear=junk)
    check_error(f"streams, before the first sublayer, {dtype}", kind, rel(h, P.rms_norm(P.gather_streams(equal6, a6), w6, eps)), lim)
    assert float(junk.abs().max()) == 0.0
    for source, X_old in ((x0.cuda(), equal6), (X.transpose(0, 1).contiguous().cuda(), X6)):
        new = P.scatter_streams(X_old, M6, b6, y6, m)
        before = source.clone()
        # the sum alone, behind a last layer
        total = torch.full((T, d), float("nan"), device="cuda")
        ops.stream_bundle(source, streams=S, y=dy, mix=dM, spread=db, scale=m, total=total)
        check_error("streams, their sum behind the last sublayer", kind, rel(total, new.sum(0)), 3e-6)
        assert torch.equal(source, before)
        # the next sublayer's norm and the new streams (in place where the old ones are a bundle already)
        h, junk = out(), torch.full((5001,), 3.0, device="cuda")
        into = source if source.dim() == 3 else torch.full((T, S, d), float("nan"), device="cuda")
        ops.stream_bundle(source, streams=S, y=dy, mix=dM, spread=db, scale=m, into=into, gather=da, weight=dw, eps=eps, normed=h, clear=junk)
        check_error("streams, the new ones", kind, rel(into.transpose(0, 1), new), 3e-6)
        check_error(f"streams, the next norm, {dtype}", kind, rel(h, P.rms_norm(P.gather_streams(new, a6), w6, eps)), lim)
        assert float(junk.abs().max()) == 0.0
    # the sum may take the place of the row that all streams equal
    one = x0.cuda()
    ops.stream_bundle(one, streams=S, y=dy, mix=dM, spread=db, scale=m, total=one)
    assert rel(one, P.scatter_streams(equal6, M6, b6, y6, m).sum(0)) < 3e-6
    if S > 1:
        assert rel(into.transpose(0, 1), P.scatter_streams(X6, M6.T, b6, y6, m)) > 1e-2           # [from, to], not [to, from]


def test_streams_refuse_what_does_not_fit():
    from llmplayer_b200.errors import KernelError
    from llmplayer_b200.kernels import ops
    x, y = torch.randn(2, 3, 8).cuda(), torch.randn(2, 8).cuda()
    M, v, w, h = torch.eye(3).cuda(), torch.ones(3).cuda(), torch.ones(8).cuda(), torch.empty(2, 8).cuda()
    good = dict(streams=3, y=y, mix=M, spread=v, into=x, gather=v, weight=w, eps=1e-5, normed=h)
    ops.stream_bundle(x, **good)
    for bad in (dict(streams=4), dict(mix=None), dict(weight=None), dict(total=h), dict(y=None), dict(gather=torch.ones(2).cuda()),
                dict(y=torch.randn(2, 9).cuda()), dict(into=torch.empty(2, 2, 8).cuda()), dict(mix=M.double())):
        with pytest.raises(KernelError):
            ops.stream_bundle(x, **dict(good, **bad))


# --------------------------------------------------------------------------- queries, keys and values
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,dk,dv,rd,unit", [(4, 2, 24, 40, 8, True), (3, 3, 16, 8, 16, False), (2, 1, 64, 64, 32, True), (6, 2, 10, 12, 0, False)])
def test_values_are_shown_and_blended(dtype, H, G, dk, dv, rd, unit):
    """The layer that shows its values stores them unchanged and leaves them, with their additive vector, in float32; a later
    layer stores the blend of its own and those. Queries and keys: additive vector, rotation, then the root mean square."""
    from llmplayer_b200.kernels import ops
    torch.manual_seed(dk + dv)
    T, off, eps, base, first_pos = 70, 4, 1e-4, 3000.0, 30
    hdp = -(-max(dk, dv) // 16) * 16
    F = (H + G) * dk + G * dv
    wide = 2 * torch.randn(T, off + F + H)                        # behind the values: gates, which are no business of this kernel
    bias = torch.randn(F)
    freqs = torch.tensor([base ** (-2.0 * i / rd) for i in range(rd // 2)], dtype=torch.float64).float().cuda() if rd else None
    rotation = ops.Rotation(freqs, rd, False) if rd else ops.NO_ROTATION
    pos = list(range(first_pos, first_pos + T))
    x = wide.double()[:, off:off + F] + bias.double()
    q, k, v = x[:, :H * dk].reshape(T, H, dk), x[:, H * dk:(H + G) * dk].reshape(T, G, dk), x[:, (H + G) * dk:].reshape(T, G, dv)
    q, k = P.rotate_half(q, torch.tensor(pos), base, rd), P.rotate_half(k, torch.tensor(pos), base, rd)
    if unit:
        q, k = P.unit_rms(q, eps), P.unit_rms(k, eps)
    first = torch.randn(T, G * dv)
    lam = torch.tensor([0.3])
    lim = 2e-5 if dtype == torch.float32 else 5e-3                # float32: angles of up to 100 are float32 products

    def run(**kw):
        q_out = torch.full((T, H * hdp), float("nan"), dtype=dtype, device="cuda")
        pages = torch.zeros(3, 2, G, PAGE, hdp, dtype=dtype, device="cuda")
        ops.qkv_prepare(wide.cuda()[:, off:off + F], bias.cuda(), rotation, i32(pos), i32([0] * T), i32([[2, 0]]), q_out, pages,
                        num_heads=H, num_kv_heads=G, key_dim=dk, value_dim=dv, unit_norm_eps=eps if unit else None, **kw)
        kv = torch.cat([pages[2], pages[0]], dim=2).cpu()[:, :, first_pos:first_pos + T].transpose(1, 2)          # [2, T, G, hdp]
        assert float(q_out.view(T, H, hdp)[..., dk:].abs().sum()) == 0.0 and float(kv[0, ..., dk:].abs().sum()) == 0.0
        assert float(kv[1, ..., dv:].abs().sum()) == 0.0 and float(pages[1].abs().sum()) == 0.0
        return q_out.view(T, H, hdp)[..., :dk], kv[0, ..., :dk], kv[1, ..., :dv]
    shown = torch.full((T, G * dv), float("nan"), device="cuda")
    angles = None                                                  # a step's table of angles must give the same bits
    if rd:
        angles = ops.rope_angles(i32(pos), rotation, torch.empty(T, rd // 2, 2, device="cuda"))
        assert all(torch.equal(a, b) for a, b in zip(run(), run(angles=angles)))
    for kw, ref in ((dict(keep_values=shown, angles=angles), v),
                    (dict(blend=(first.cuda(), lam.cuda())), P.blend_values(v, first.double().reshape(T, G, dv), 0.3))):
        got = run(**kw)
        for name, g, r in zip(("queries", "keys", "values"), got, (q, k, ref)):
            check_error(f"heads prepared, {name}, {dtype}", f"{H}/{G} x {dk} / {dv}, {list(kw)[0]}", rel(g, r), lim)
    assert rel(shown.view(T, G, dv), v) < 2e-6


# --------------------------------------------------------------------------- attention with gated heads
def fill_pages(k, v, table_rows, num_pages, dtype):
    T, G, hd = k.shape
    pages = torch.zeros(num_pages, 2, G, PAGE, hd, dtype=dtype, device="cuda")
    for t in range(T):
        page = table_rows[t // PAGE]
        pages[page, 0, :, t % PAGE] = k[t].to(dtype)
        pages[page, 1, :, t % PAGE] = v[t].to(dtype)
    return pages


def plain_attention(q, k, v, scale, chunk, first, gate):
    """The last rows of the plain function: q and gate hold the queries from position ``first`` on."""
    H, length = q.shape[1], k.shape[0]
    full = torch.zeros(length, H, q.shape[2], dtype=q.dtype)
    full[first:] = q
    group = H // k.shape[1]
    o = P.softmax_attention(full, k.repeat_interleave(group, 1), v.repeat_interleave(group, 1), scale, P.chunk_visible(length, chunk))[first:]
    return o if gate is None else o * torch.sigmoid(gate)[:, :, None]


def run_attention(kind, qd, pages, table, length, new, chunk, gate, H, G, hd, scale):
    from llmplayer_b200.kernels import ops
    out = torch.full_like(qd, float("nan"))
    kw = dict(num_heads=H, num_kv_heads=G, head_dim=hd, scale=scale, window=None, chunk=chunk or 0, gate=gate)
    if kind == "plain":
        ops.attention_plain(qd, out, pages, table, i32([0] * new), i32(list(range(length - new, length))), **kw)
    elif kind == "prompt":
        ops.attention_prefill(qd, out, pages, table, i32([0, new]), i32([length]), new, exact_weights=True, **kw)
    else:
        ops.attention_decode(qd, out, pages, table, i32([length]), scratch, exact_weights=True, **kw)
    return out


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,hd,length,new,chunk", [(4, 2, 48, 200, 200, 9), (8, 1, 64, 321, 321, 64), (2, 2, 128, 400, 57, 128), (6, 2, 96, 700, 700, 200),
                                                     (5, 1, 16, 130, 130, 1), (2, 1, 64, 400, 300, 65), (3, 3, 16, 300, 1, 256), (2, 2, 64, 260, 2, 257),
                                                     (20, 2, 64, 450, 450, None), (2, 1, 192, 300, 300, 100), (2, 2, 256, 333, 140, None),
                                                     (12, 1, 64, 700, 1, None), (2, 1, 128, 1000, 1, None), (2, 1, 64, 3000, 1, None), (4, 2, 128, 1000, 1, 300)])
def test_attention_with_gated_heads(dtype, H, G, hd, length, new, chunk):
    """The gates are columns of a wider product; the last case but one is long enough for shares that are merged."""
    torch.manual_seed(length + hd)
    scale, blocks = 0.3, -(-length // PAGE)
    q = torch.randn(new, H, hd).to(dtype)
    k, v = torch.randn(length, G, hd).to(dtype), torch.randn(length, G, hd).to(dtype)
    rows = torch.randperm(48).tolist()[:blocks]
    pages = fill_pages(k, v, rows, 48, dtype)
    table = i32(rows + [0] * (48 - blocks)).view(1, -1)
    wide = 2 * torch.randn(new, 3 + H + 2)
    gate = wide.cuda()[:, 3:3 + H]
    first = length - new
    ref = plain_attention(q.double(), k.double(), v.double(), scale, chunk, first, wide.double()[:, 3:3 + H])
    qd = q.reshape(new, H * hd).cuda()
    kinds = [("plain", 3e-6)] if dtype == torch.float32 else [("plain", 6e-3), ("prompt", 6e-3) if new > 1 else ("decode", 6e-3)]
    for kind, lim in kinds:
        out = run_attention(kind, qd, pages, table, length, new, chunk, gate, H, G, hd, scale).view(new, H, hd)
        check_error(f"gated heads, {kind} kernel, {dtype}", f"{H}/{G} x {hd}, {new} of {length}, chunks of {chunk}", rel(out, ref), lim)
        bare = run_attention(kind, qd, pages, table, length, new, chunk, None, H, G, hd, scale).view(new, H, hd)
        assert rel(bare, ref) > 0.1
        assert rel(bare, plain_attention(q.double(), k.double(), v.double(), scale, chunk, first, None)) < lim


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("step", ["prompt", "decode"])
@pytest.mark.parametrize("length,chunk", [(700, 200), (700, 64), (700, 65), (641, 128), (300, 33), (200, 9), (130, 2), (130, 1), (601, 600), (600, 601), (193, 192)])
def test_a_key_at_the_edges_of_a_chunk(dtype, step, length, chunk):
    """Head 1's last query fits ONE key far better than all others. On the first position of the query's chunk its value must
    come through nearly alone (times the gate), however long ago that was; on the last position of the chunk before it must
    not be seen at all. A prompt step of 40 tokens (which may cross a border itself) and a one-token step."""
    torch.manual_seed(chunk)
    H, G, hd, scale = 4, 2, 64, 0.5
    new = 40 if step == "prompt" else 1
    direction = torch.randn(hd)
    direction /= direction.norm()
    last = length - 1
    start = last // chunk * chunk
    gate = torch.randn(new, H)
    for at, seen in ((start, True), (start - 1, False), (last, True), (0, start == 0)):
        if at < 0:
            continue
        k, v = 0.3 * torch.randn(length, G, hd), torch.randn(length, G, hd)
        q = 0.3 * torch.randn(new, H, hd)
        q[-1, 1] = 8.0 * direction
        k[at, 0] = 8.0 * direction                             # score 64 * 0.5 = 32 against scores near 0
        k, v, q = k.to(dtype), v.to(dtype), q.to(dtype)
        rows = torch.randperm(16).tolist()[:-(-length // PAGE)]
        pages = fill_pages(k, v, rows, 16, dtype)
        table = i32([r if b >= start // PAGE or new > 1 else -1 for b, r in enumerate(rows)] + [0] * (16 - len(rows))).view(1, -1)
        kind = "plain" if dtype == torch.float32 else step
        out = run_attention(kind, q.reshape(new, H * hd).cuda(), pages, table, length, new, chunk, gate.cuda(), H, G, hd, scale).view(new, H, hd)
        ref = plain_attention(q.double(), k.double(), v.double(), scale, chunk, length - new, gate.double())
        check_error(f"a key that stands out, {step}, {dtype}", f"length {length}, chunks of {chunk}, key at {at}", rel(out, ref),
                    3e-6 if dtype == torch.float32 else 6e-3)
        got, alone = out[-1, 1].double().cpu(), v[at, 0].double() * torch.sigmoid(gate[-1, 1].double())
        if seen:
            assert float((got - alone).abs().max()) < 1e-3 + (0.02 if dtype == torch.bfloat16 else 0.0), at
        else:
            assert float((got - alone).abs().max()) > 0.25, at


def test_gates_belong_to_their_own_token():
    """Two sequences in one step: a prompt step's gates follow the step's rows, a decode step's its sequences."""
    from llmplayer_b200.kernels import ops
    torch.manual_seed(1)
    H, G, hd = 2, 1, 64
    k, v = torch.zeros(40, G, hd), torch.ones(40, G, hd)          # every output is one: what comes out is the gate
    pages = torch.cat([fill_pages(k, v, [0], 1, torch.bfloat16)] * 2)
    table = i32([[0], [1]])
    gate = torch.randn(50, H).cuda()
    q = torch.randn(50, H * hd).bfloat16().cuda()
    out = torch.empty_like(q)
    ops.attention_prefill(q, out, pages, table, i32([0, 11, 50]), i32([40, 39]), 39, num_heads=H, num_kv_heads=G, head_dim=hd, scale=0.1,
                          window=None, exact_weights=True, chunk=7, gate=gate)
    assert rel(out.view(50, H, hd), torch.sigmoid(gate)[:, :, None].expand(50, H, hd)) < 5e-3
    one = torch.empty_like(q[:2])
    ops.attention_decode(q[:2], one, pages, table, i32([40, 17]), scratch, num_heads=H, num_kv_heads=G, head_dim=hd, scale=0.1, window=None,
                         exact_weights=True, chunk=7, gate=gate[:2])
    assert rel(one.view(2, H, hd), torch.sigmoid(gate[:2])[:, :, None].expand(2, H, hd)) < 5e-3


# --------------------------------------------------------------------------- experts
@pytest.mark.parametrize("T,E,ff,top", [(5, 8, 88, 1), (33, 5, 40, 2), (3, 40, 16, 5), (7, 1, 7, 1), (2, 6, 13, 6), (300, 4, 64, 3), (1, 130, 8, 9)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_experts_chosen_weighted_and_squared(T, E, ff, top, dtype):
    """Choice and activation in one kernel, from the sums and logits of one product; the same with weights from a router of
    its own; the weight on an expert's output instead."""
    from llmplayer_b200.kernels import ops
    torch.manual_seed(T + E)
    z = torch.randn(T, E * ff + E)
    logits = z[:, E * ff:]
    w = P.expert_weights(logits.double(), top)
    columns = w.repeat_interleave(ff, 1)
    z6 = z.double()[:, :E * ff]
    on_input = torch.clamp(columns * z6, min=0.0) ** 2
    on_output = columns * torch.clamp(z6, min=0.0) ** 2
    lim = 3e-6 if dtype == torch.float32 else 5e-3
    weights = torch.full((T, E), float("nan"), device="cuda")
    ops.route_top(logits.contiguous().cuda(), None, weights, num_experts=E, top=top, sigmoid=True)
    check_error("weights of the chosen experts", f"{top} of {E}", rel(weights, w), 2e-6)
    for ref, kw in ((on_input, dict(on_input=True)), (on_output, dict(on_input=False))):
        junk, h = torch.full((3000,), 3.0, device="cuda"), torch.full((T, E * ff), float("nan"), dtype=dtype, device="cuda")
        ops.expert_relu2(z.cuda(), h, num_experts=E, expert_size=ff, top=top, sigmoid=True, clear=junk, **kw)
        check_error(f"experts in one kernel, {dtype}", f"{top} of {E} x {ff}, {kw}", rel(h, ref), lim)
        assert float(junk.abs().max()) == 0.0
        assert float(h.float().cpu()[columns == 0].abs().sum()) == 0.0
        h2 = torch.full((T, E * ff), float("nan"), dtype=dtype, device="cuda")
        ops.expert_relu2(z.cuda()[:, :E * ff], h2, num_experts=E, expert_size=ff, weights=weights, **kw)
        assert torch.equal(h, h2)
    assert rel(on_input, on_output) > 1e-2 or top == E == 1


def test_the_lower_index_wins_a_tie_and_negative_logits_are_chosen_too():
    from llmplayer_b200.kernels import ops
    z = torch.tensor([[-3.0, -1.0, -1.0, -40.0], [-200.0, -150.0, -300.0, -150.0]]).cuda()
    w = torch.full((2, 4), float("nan"), device="cuda")
    ops.route_top(z, None, w, num_experts=4, top=2, sigmoid=True)
    s = 1.0 / (1.0 + torch.exp(torch.tensor(1.0)))
    assert torch.allclose(w[0].cpu(), torch.tensor([0.0, s, s, 0.0])) and float(w[1].abs().max()) < 1e-30
    ops.route_top(z, None, w, num_experts=4, top=1, sigmoid=True)
    assert torch.allclose(w[0].cpu(), torch.tensor([0.0, s, 0.0, 0.0]))


class Step:
    """What the parts read of a step, for one prompt of T tokens in its own pages."""

    def __init__(self, T):
        from llmplayer_b200.engine.step import SequenceStep, StepContext, Workspace
        self.workspace = Workspace(torch.device("cuda"))
        blocks = -(-T // PAGE)
        self.ctx = StepContext(self.workspace, [SequenceStep(0, 0, T, 0)], [0] * T, [[list(range(blocks))]], [T - 1])


@pytest.mark.parametrize("scoring", ["sigmoid_top", "softmax_top"])
@pytest.mark.parametrize("weight_on", ["input", "output"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_mixture_part(dtype, weight_on, scoring):
    """The whole feed-forward, stored and added, with the router in the experts' product and with one of its own."""
    from llmplayer_b200.parts import FEED_FORWARDS
    from llmplayer_b200.parts.base import Runtime
    from llmplayer_b200.parts.specs import ExpertRoutingSpec, MixtureSpec
    torch.manual_seed(3)
    T, d, ff, E, top = 50, 64, 40, 6, 2
    spec = MixtureSpec(hidden_size=d, expert_size=ff, activation="relu2", weight_on=weight_on, expert_prefix="f.",
                       routing=ExpertRoutingSpec(num_experts=E, top=top, groups=1, keep_groups=1, router="f.router", scoring=scoring))
    part = FEED_FORWARDS.build(spec)
    store = torch.float32 if dtype == "float32" else torch.bfloat16
    w = {n: (torch.randn(s.shape) * (0.3 if n != "f.router" else 0.6)).to(store) for n, s in part.tensor_specs().items()}
    part.load(w, Runtime(device=torch.device("cuda"), dtype=dtype))
    assert part.stacked_router == (scoring == "sigmoid_top")
    x = torch.randn(T, d).to(store)
    w6, h = {n: t.double() for n, t in w.items()}, x.double()
    z = h @ w6["f.router"].T
    if scoring == "softmax_top":
        kept = torch.zeros_like(z).scatter(-1, z.topk(top, dim=-1).indices, 1.0) > 0
        g = torch.softmax(z.masked_fill(~kept, float("-inf")), dim=-1)
    else:
        g = P.expert_weights(z, top)
    ref = torch.zeros(T, d, dtype=torch.float64)
    for e in range(E):
        y = P.squared_relu_expert(g[:, e, None] * h if weight_on == "input" else h, w6[f"f.e{e}.up"], w6[f"f.e{e}.down"])
        ref += y if weight_on == "input" else g[:, e, None] * y
    step = Step(T)
    out = torch.full((T, d), float("nan"), device="cuda")
    part.forward(step.ctx, x.cuda(), out, overwrite=True)
    lim = 1e-5 if dtype == "float32" else 1.5e-2
    check_error(f"the mixture part, {dtype}", f"{scoring}, weight on the {weight_on}", rel(out, ref), lim)
    added = torch.ones(T, d, device="cuda")
    part.forward(step.ctx, x.cuda(), added)
    assert rel(added - 1.0, ref) < lim


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width,S", [(64, 3), (52, 4)])
def test_the_block_part(dtype, width, S):
    """Two layers of a bundle handed one stream: copies, connections, the bundle handed on and the sum left at the end."""
    from dataclasses import replace
    from llmplayer_b200.parts import BLOCKS
    from llmplayer_b200.parts.base import Runtime
    from llmplayer_b200.config import config_from_dict
    torch.manual_seed(width)
    raw = {"architecture": "Zotolix", "vocab": 10, "width": width, "norm": {"eps": 1e-5}, "embedding": {"scale": 1.0}, "streams": S,
           "residual_mult": 0.7, "layers": [
               {"type": t, "mixer": {"heads": 2, "kv_heads": 1, "dim": 16, "vdim": 16, "scale": 0.3, "v_mix": True, "mask": {"size": 11},
                                     "rot": {"base": 100.0, "dims": 8}},
                "mlp": {"kind": "moe", "expert": {"ff": 24}, "router": {"experts": 2, "top": 2}} if t == "attention" else None}
               for t in ("attention", "attention_2")]}
    layers = config_from_dict(raw).layout().layers
    blocks = [BLOCKS.build(spec) for spec in layers]
    store = torch.float32 if dtype == "float32" else torch.bfloat16
    w = {}
    for b in blocks:
        for n, s in b.tensor_specs().items():
            w[n] = ((0.5 if ".hc" in n else 0.2) * torch.randn(s.shape) + (1.0 if "norm" in n else 0.0)).to(store)
    w["l1.mix.vmix"] = torch.tensor(0.4).to(store)
    rt = Runtime(device=torch.device("cuda"), dtype=dtype)
    for b in blocks:
        b.load(w, rt)
    T = 40
    x = torch.randn(T, width)
    step = Step(T)

    class View:
        group_index = 0

        def __init__(self):
            self.pages = torch.zeros(1, 2, 1, PAGE, 16, dtype=rt.kv_dtype, device="cuda")
    stream = x.cuda().clone()
    step.ctx.begin_walk()
    handed = blocks[0].forward(step.ctx, View(), stream, next_block=blocks[1])
    assert handed and torch.equal(stream.cpu(), x)                # the bundle is live, the stream's buffer is left alone
    assert not blocks[1].forward(step.ctx, View(), stream, normed_ready=True, next_block=None)
    w6 = {n: t.double() for n, t in w.items()}
    X, first = torch.stack([x.double()] * S), {}
    for i, layer in enumerate(raw["layers"]):
        p = f"l{i}."
        y = P.attention(P.rms_norm(P.gather_streams(X, w6[p + "hc1.in"]), w6[p + "norm1"], 1e-5), w6, p + "mix.", layer["mixer"], 1e-5, layer["type"], first)
        X = P.scatter_streams(X, w6[p + "hc1.mix"], w6[p + "hc1.out"], y, 0.7)
        if layer["mlp"]:
            y = P.mixture(P.rms_norm(P.gather_streams(X, w6[p + "hc2.in"]), w6[p + "norm2"], 1e-5), w6, p + "mlp.", layer["mlp"])
            X = P.scatter_streams(X, w6[p + "hc2.mix"], w6[p + "hc2.out"], y, 0.7)
    check_error(f"the block part, {dtype}", f"width {width}, {S} streams", rel(stream, X.sum(0)), 1e-5 if dtype == "float32" else 2e-2)
    # a follower with another number of streams gets the sum
    other = BLOCKS.build(replace(layers[1], streams=S + 1))
    stream2 = x.cuda().clone()
    assert not blocks[0].forward(step.ctx, View(), stream2, next_block=other) and not torch.equal(stream2.cpu(), x)
