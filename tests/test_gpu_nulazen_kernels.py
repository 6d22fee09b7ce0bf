"""Each kernel of the Nulazen design alone, against plain torch in float64: the norm on both sides of a sublayer (K-split
stacks, a row added, gathered rows, odd widths), the squared-relu product, the side input's gate, the delta rule's
preparation (convolution across cuts and slots, unit heads, beta, low-rank rows), the delta rule walked token by token,
eight tokens at a time, in portions, beside single tokens, with padding rows, strong and weak decays, tall heads and
several value heads a key head, the head norm with its output gate, the router with a corrected choice among groups, and
the experts' activation with two clamps."""

import numpy as np
import pytest
import torch

from tests.gpu_common import cuda_ops
from tests.plain import plain_nulazen as pn

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]


def close(got, want, tol, what=""):
    got, want = got.double().cpu(), want.double().cpu()
    assert got.shape == want.shape, what
    assert torch.isfinite(got).all(), what
    err = float((got - want).abs().max()) / max(1.0, float(want.abs().max()))
    assert err <= tol, f"{what}: {err:.3e} > {tol:.1e}"


def tolerance(dtype):
    return 3e-6 if dtype == torch.float32 else 1e-2


def stacked(rows, partials, generator):
    """`rows` as a stack of partial sums that add up to it (to rounding)."""
    if partials == 1:
        return rows.cuda()
    noise = torch.randn(partials - 1, *rows.shape, generator=generator)
    return torch.cat([(rows - noise.sum(0))[None], noise]).cuda().contiguous()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,width,partials,row", [(5, 256, 1, True), (70, 96, 3, False), (3, 50, 2, True), (300, 1000, 1, True),
                                                  (2, 6000, 4, False), (400, 5000, 1, False), (1, 36, 16, True)])
def test_norm_join_adds_a_normed_branch_and_norms_the_sum(dtype, n, width, partials, row):
    ops = cuda_ops(dtype)
    g = torch.Generator().manual_seed(n + width)
    resid, branch = torch.randn(n, width, generator=g), 3.0 * torch.randn(n, width, generator=g)
    add = torch.randn(width, generator=g) if row else None
    first, second = 1 + 0.1 * torch.randn(width, generator=g), 1 + 0.1 * torch.randn(width, generator=g)
    joined = resid.double() + pn.rms_norm(branch.double(), first, 1e-5) + (add.double() if row else 0.0)
    want = pn.rms_norm(joined, second, 1e-6)
    x, y = resid.cuda(), stacked(branch, partials, g)
    out = torch.empty(n, width, dtype=dtype, device="cuda")
    rows = torch.tensor([n - 1, 0], dtype=torch.int32, device="cuda")
    some = torch.empty(2, width, dtype=dtype, device="cuda")
    more = add.cuda() if row else None
    ops.norm_join(x, y, first.cuda(), 1e-5, more, second.cuda(), 1e-6, some, rows=rows)
    assert torch.equal(x.cpu(), resid)                       # gathered rows leave the residual alone
    close(some, want[[n - 1, 0]], max(tolerance(dtype), 2e-5 if partials > 4 else 0), "gathered")
    ops.norm_join(x, y, first.cuda(), 1e-5, more, second.cuda(), 1e-6, out)
    close(x, joined, 2e-5 if partials > 1 else 3e-6, "residual")
    close(out, want, max(tolerance(dtype), 2e-5 if partials > 1 else 0), "normed sum")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,inter,width", [(1, 48, 64), (8, 200, 96), (64, 128, 40), (65, 128, 64), (300, 36, 64)])
def test_squared_relu_inside_and_behind_the_product(dtype, n, inter, width):
    ops = cuda_ops(dtype)
    g = torch.Generator().manual_seed(n)
    x, w = torch.randn(n, width, generator=g).to(dtype), (0.3 * torch.randn(inter, width, generator=g)).to(dtype)
    z = x.double() @ w.double().T
    out = torch.empty(n, inter, dtype=dtype, device="cuda")
    ops.linear_act(x.cuda(), w.cuda(), out, "relu2")
    if dtype == torch.bfloat16:
        z = z.to(torch.bfloat16).double()
    close(out, torch.relu(z).pow(2), 3e-6 if dtype == torch.float32 else 2e-2, "relu2")
    assert float(out[z.cuda() < -0.1].abs().max()) == 0.0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,dim,padded,partials", [(1, 16, 16, 1), (7, 20, 32, 3), (90, 5, 16, 1)])
def test_side_gate_reads_each_tokens_own_row(dtype, n, dim, padded, partials):
    ops = cuda_ops(dtype)
    g = torch.Generator().manual_seed(dim)
    vocab, parts, part = 37, 4, 2
    table = torch.randn(vocab, parts * dim, generator=g).to(dtype)
    gate = torch.randn(n, padded, generator=g)
    ids = torch.randint(0, vocab, (n,), generator=g)
    drawn = torch.randint(0, vocab, (6,), generator=g)
    given = ids.clone()
    given[0] = -1 - 4                                        # what the step before drew in its row 4
    ids[0] = drawn[4]
    out = torch.full((n, padded), 7.0, dtype=dtype, device="cuda")
    ops.side_gate(stacked(gate, partials, g), table.cuda(), given.to(torch.int32).cuda(), drawn.to(torch.int32).cuda(),
                  part * dim, dim, out)
    want = torch.zeros(n, padded, dtype=torch.float64)
    want[:, :dim] = pn.gelu_tanh(gate[:, :dim].double()) * table[ids, part * dim: (part + 1) * dim].double()
    close(out, want, 2e-5 if dtype == torch.float32 else 1e-2, "gate times row")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,partials", [(4, 2, 16, 8, 1), (3, 3, 128, 160, 1), (2, 1, 10, 7, 3), (5, 5, 200, 24, 1)])
def test_delta_prep_across_cuts_and_slots(dtype, taps, heads, kv_heads, dim, vdim, partials):
    ops = cuda_ops(dtype)
    g = torch.Generator().manual_seed(taps * 10 + heads)
    qk, channels = kv_heads * dim, 2 * kv_heads * dim + heads * vdim
    beta_at, low_width = channels, 24
    low_at = beta_at + -(-heads // 4) * 4
    total = -(-(low_at + low_width) // 16) * 16
    lengths = [123, 1, 9, 40]
    whole = [torch.randn(n, total, generator=g) for n in lengths]
    weights = torch.randn(channels, taps, generator=g)

    def plain(u):
        y = pn.silu(pn.short_convolution(u[:, :channels].double(), weights))
        q = pn.unit_heads(y[:, :qk].view(-1, kv_heads, dim)) * dim ** -0.5
        k = pn.unit_heads(y[:, qk: 2 * qk].view(-1, kv_heads, dim))
        return torch.cat([q.reshape(-1, qk), k.reshape(-1, qk), y[:, 2 * qk:]], -1)

    want = [plain(u) for u in whole]
    state = torch.full((6, max(taps - 1, 0), channels), 7.0, device="cuda")
    slots = [3, 0, 4, 5]
    state[slots] = 0.0
    got, fed = [[] for _ in lengths], [0] * 4
    # portions of unequal length, a request left out, single tokens alone, a portion of more than 64 tokens
    for cut in ([2, 1, 4, 1], [1, 0, 5, 1], [1, 0, 0, 1], [20, 0, 0, 3], [99, 0, 0, 34]):
        live = [i for i, c in enumerate(cut) if c]
        rows = torch.cat([whole[i][fed[i]: fed[i] + cut[i]] for i in live])
        starts = np.cumsum([0] + [cut[i] for i in live]).astype(np.int32)
        n = rows.shape[0]
        mixed = torch.empty(n, channels, device="cuda")
        beta = torch.empty(n, heads, device="cuda")
        low = torch.empty(n, low_width, dtype=dtype, device="cuda")
        seq_of = torch.tensor(sum([[k] * cut[i] for k, i in enumerate(live)], []), dtype=torch.int32, device="cuda")
        ops.delta_prep(stacked(rows, partials, g), weights.cuda(), state, torch.tensor(starts, device="cuda"),
                       torch.tensor([slots[i] for i in live], dtype=torch.int32, device="cuda"), seq_of, mixed, beta, low,
                       len(live), heads, kv_heads, dim, vdim, beta_at, low_at, 1e-6, longest=max(cut))
        close(beta, torch.sigmoid(rows[:, beta_at: beta_at + heads].double()), 1e-5, "beta")
        close(low, rows[:, low_at: low_at + low_width], 1e-5 if dtype == torch.float32 else 1e-2, "low-rank rows")
        for k, i in enumerate(live):
            got[i].append(mixed[starts[k]: starts[k + 1]].cpu())
            fed[i] += cut[i]
    for i in range(4):
        # a bfloat16 engine's SiLU may use the hardware exponential
        close(torch.cat(got[i]), want[i][: fed[i]], 5e-5 if partials > 1 or dtype == torch.bfloat16 else 1e-5, f"sequence {i}")
    if taps > 1:
        assert float(state[1].min()) == 7.0 and float(state[2].min()) == 7.0   # the neighbours' slots stay


def delta_inputs(n, heads, kv_heads, dim, vdim, seed, strength=1.0):
    g = torch.Generator().manual_seed(seed)
    q = pn.unit_heads(torch.randn(n, kv_heads, dim, generator=g)) * dim ** -0.5
    k = pn.unit_heads(torch.randn(n, kv_heads, dim, generator=g))
    v = torch.randn(n, heads, vdim, generator=g)
    beta = torch.sigmoid(2.0 * torch.randn(n, heads, generator=g))
    z = 2.0 * torch.randn(n, heads, dim, generator=g)
    a_log = strength * torch.randn(heads, generator=g)
    bias = torch.randn(heads * dim, generator=g) - 2.0
    return q, k, v, beta, z, a_log, bias


SHAPES = [(2, 1, 16, 8), (4, 2, 64, 32), (3, 3, 128, 128), (6, 6, 40, 24), (2, 2, 7, 5), (2, 1, 136, 48), (1, 1, 256, 20), (2, 2, 320, 12),
          (3, 1, 3, 70)]


@pytest.mark.parametrize("heads,kv_heads,dim,vdim", SHAPES)
@pytest.mark.parametrize("strength", [0.5, 3.0])
def test_delta_scan_whole_walked_and_in_portions(heads, kv_heads, dim, vdim, strength):
    """One sequence: eight tokens at a time, token by token, and cut into portions whose borders fall anywhere, against
    the recurrence in float64; decays from nearly one to nearly zero."""
    ops = cuda_ops(torch.float32)
    n, share = 150, heads // kv_heads
    q, k, v, beta, z, a_log, bias = delta_inputs(n, heads, kv_heads, dim, vdim, dim + heads, strength)
    g = pn.channel_decays(z.double(), a_log.double(), bias.double())
    want, last = pn.delta_recurrence(q.double().repeat_interleave(share, 1), k.double().repeat_interleave(share, 1), v.double(), g,
                                     beta.double())
    mixed = torch.cat([q.reshape(n, -1), k.reshape(n, -1), v.reshape(n, -1)], -1).cuda().contiguous()
    gates = torch.cat([z.reshape(n, -1), torch.randn(n, 20)], -1)
    size = -(-dim * vdim // 4) * 4
    for way, cuts in (("blocks", [n]), ("walk", [n]), ("portions", [1, 2, 37, 16, 1, 1, 15, 17, 8, 52]), ("stack", [n]), ("runs", [110, 40])):
        ops.delta_run_blocks = 3 if way == "runs" else 0   # runs of 24 tokens that walk side by side
        gen = torch.Generator().manual_seed(1)
        state = torch.full((3, heads, size), 5.0, device="cuda")
        state[1] = 0.0
        out = torch.empty(n, heads * vdim, device="cuda")
        at = 0
        for cut in cuts:
            piece = gates[at: at + cut]
            ops.delta_scan(mixed[at: at + cut], beta[at: at + cut].cuda(), stacked(piece, 3 if way == "stack" else 1, gen).contiguous(),
                           a_log.exp().cuda(), bias.cuda(), state, torch.tensor([0, cut], dtype=torch.int32, device="cuda"),
                           torch.tensor([1], dtype=torch.int32, device="cuda"), out[at: at + cut], 1, heads, kv_heads, dim, vdim,
                           q_lens=None if way == "walk" else [cut])
            at += cut
        tol = 3e-5 if way == "stack" else 1e-5
        close(out.view(n, heads, vdim), want, tol, way)
        close(state[1][:, : dim * vdim].view(heads, dim, vdim), last, tol, way + " state")
        assert float(state[0].min()) == 5.0 and float(state[2].max()) == 5.0


@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(4, 2, 64, 32), (3, 3, 20, 36), (2, 1, 128, 100)])
def test_delta_scan_of_unequal_sequences_with_padding_rows(heads, kv_heads, dim, vdim):
    """Portions beside single tokens beside rows without a slot, more sequences than a warp has lanes; each as alone."""
    ops = cuda_ops(torch.float32)
    lengths = [1, 40, 1, 16, 15, 9, 200, 1] + [1, 17] * 16
    n, share = sum(lengths), heads // kv_heads
    q, k, v, beta, z, a_log, bias = delta_inputs(n, heads, kv_heads, dim, vdim, 3)
    mixed = torch.cat([q.reshape(n, -1), k.reshape(n, -1), v.reshape(n, -1)], -1).cuda().contiguous()
    gates = z.reshape(n, -1).cuda().contiguous()
    size = -(-dim * vdim // 4) * 4
    count = len(lengths)
    slots = list(range(count))[::-1]
    slots[2], slots[4], slots[3] = -1, -1, -1
    state = torch.randn(count, heads, size).cuda()
    before = state.clone()
    starts = np.cumsum([0] + lengths)
    out = torch.full((n, heads * vdim), 9.0, device="cuda")
    ops.delta_scan(mixed, beta.cuda(), gates, a_log.exp().cuda(), bias.cuda(), state,
                   torch.tensor(starts, dtype=torch.int32, device="cuda"), torch.tensor(slots, dtype=torch.int32, device="cuda"), out,
                   count, heads, kv_heads, dim, vdim, q_lens=lengths)
    decays = pn.channel_decays(z.double(), a_log.double(), bias.double())
    for i, slot in enumerate(slots):
        a, b = starts[i], starts[i + 1]
        if slot < 0:
            assert float(out[a:b].abs().max()) == 0.0
            continue
        held = before[slot][:, : dim * vdim].double().cpu().view(heads, dim, vdim)
        want, last = pn.delta_recurrence(q[a:b].double().repeat_interleave(share, 1), k[a:b].double().repeat_interleave(share, 1),
                                         v[a:b].double(), decays[a:b], beta[a:b].double(), held)
        close(out[a:b].view(-1, heads, vdim), want, 2e-5, f"sequence {i}")
        close(state[slot][:, : dim * vdim].view(heads, dim, vdim), last, 2e-5, f"state {i}")
    for slot in set(range(count)) - set(slots):
        assert torch.equal(state[slot], before[slot])


def test_delta_scan_takes_heads_in_turns_when_the_scratch_is_bounded():
    ops = cuda_ops(torch.float32)
    heads, dim, vdim, n = 5, 24, 12, 100
    q, k, v, beta, z, a_log, bias = delta_inputs(n, heads, heads, dim, vdim, 8)
    mixed = torch.cat([q.reshape(n, -1), k.reshape(n, -1), v.reshape(n, -1)], -1).cuda().contiguous()
    results = []
    for bound in (ops.DELTA_SCRATCH_FLOATS, 2 * 13 * ops.core.shrike_delta_scan_record(dim, 1)):
        ops.DELTA_SCRATCH_FLOATS = bound
        state, out = torch.zeros(1, heads, dim * vdim, device="cuda"), torch.empty(n, heads * vdim, device="cuda")
        ops.delta_scan(mixed, beta.cuda(), z.reshape(n, -1).cuda(), a_log.exp().cuda(), bias.cuda(), state,
                       torch.tensor([0, n], dtype=torch.int32, device="cuda"), torch.zeros(1, dtype=torch.int32, device="cuda"), out, 1,
                       heads, heads, dim, vdim, q_lens=[n])
        results.append((out, state))
    assert torch.equal(results[0][0], results[1][0]) and torch.equal(results[0][1], results[1][1])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,heads,size,partials,gated", [(5, 3, 16, 1, True), (70, 2, 128, 1, True), (3, 5, 7, 3, True), (9, 4, 200, 2, True),
                                                         (4, 3, 40, 1, False)])
def test_head_norm_with_an_output_gate(dtype, n, heads, size, partials, gated):
    ops = cuda_ops(dtype)
    g = torch.Generator().manual_seed(size)
    x, weight = torch.randn(n, heads * size, generator=g), 1 + 0.1 * torch.randn(size, generator=g)
    at = 12
    gates = 2.0 * torch.randn(n, at + heads * size + 4, generator=g)
    want = pn.rms_norm(x.double().view(n, heads, size), weight, 1e-5).reshape(n, -1)
    if gated:
        want = want * torch.sigmoid(gates[:, at: at + heads * size].double())
    out = torch.empty(n, heads * size, dtype=dtype, device="cuda")
    ops.head_rms(x.cuda(), weight.cuda(), 1e-5, out, heads, **({"gate_source": stacked(gates, partials, g), "gate_at": at} if gated else {}))
    close(out, want, 2e-5 if dtype == torch.float32 else 1e-2, "head norm")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("experts,top,groups", [(8, 3, (4, 2)), (12, 4, (3, 1)), (6, 6, (2, 2)), (16, 1, (16, 5)), (64, 9, (8, 3)), (10, 4, None)])
@pytest.mark.parametrize("shared", [True, False])
def test_router_chooses_by_corrected_scores_among_the_best_groups(dtype, experts, top, groups, shared):
    """Corrections large enough to make choice scores negative and to choose against the scores; the weights are the
    scores, not renormalised."""
    ops = cuda_ops(dtype)
    g = torch.Generator().manual_seed(experts + top)
    n, width = 40, 64
    x = torch.randn(n, width, generator=g).to(dtype)
    router = torch.randn(experts, width, generator=g) * 0.2
    correction = 0.3 * torch.randn(experts, generator=g) - 0.2
    gate = torch.randn(width, generator=g) * 0.2
    scores = torch.softmax(x.double() @ router.double().T, -1)
    spec = {"top": top, "experts": experts, **({"groups": {"count": groups[0], "keep": groups[1]}} if groups else {})}
    margins = []
    chosen = pn.choose(scores, correction.double(), spec, margins)
    sure = margins[0] > 1e-5
    assert sure.sum() > n // 2
    want = torch.where(chosen, scores, torch.zeros_like(scores))
    out = torch.full((n, experts + int(shared)), 5.0, device="cuda")
    ops.route_top(x.cuda(), router.cuda(), gate.cuda() if shared else None, out, top, 0.0, renormalise=False,
                  correction=correction.cuda(), groups=groups)
    got = out.double().cpu()
    close(got[sure][:, :experts], want[sure], 1e-5, "weights")
    assert ((got[:, :experts] > 0).sum(-1) == top).all()
    if groups is not None:
        used = (got[:, :experts] > 0).view(n, groups[0], -1).any(-1).sum(-1)
        assert int(used.max()) <= groups[1]
    if shared:
        close(got[:, experts], torch.sigmoid(x.double() @ gate.double()), 1e-5, "shared gate")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("experts,each,rest", [(3, 16, 24), (4, 5, 7), (2, 8, 0)])
def test_experts_activation_with_two_clamps(dtype, experts, each, rest):
    ops = cuda_ops(dtype)
    g = torch.Generator().manual_seed(each)
    n, inter = 33, experts * each + rest
    gate_up = (3.0 * torch.randn(n, 2 * inter, generator=g)).to(dtype)
    weights = torch.rand(n, experts + (1 if rest else 0), generator=g)
    weights[:, 1] = 0.0
    out = torch.empty(n, inter, dtype=dtype, device="cuda")
    ops.act_mul_blocks(gate_up.cuda(), weights.cuda(), out, experts, each, "clamped_swish", limit=1.5, shared_limit=0.5)
    column = torch.arange(inter)
    block = torch.where(column < experts * each, column // each, torch.full_like(column, experts))
    limit = torch.where(block < experts, 1.5, 0.5).double()
    a = torch.minimum(gate_up[:, :inter].double(), limit)
    u = torch.maximum(torch.minimum(gate_up[:, inter:].double(), limit), -limit)
    close(out, a * torch.sigmoid(1.702 * a) * (u + 1.0) * weights.double()[:, block], 1e-5 if dtype == torch.float32 else 1e-2, "experts")
