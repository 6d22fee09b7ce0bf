"""Each kernel of the Radilix design alone, against plain torch in float64: the norm of several pending sums (K-split
stacks, rows with a factor each, in place, gathered rows, odd widths), the attention's gate per element, the erf GELU inside
and behind the product, the router with identity experts, the ungated experts' activation, the low-rank product, the delta
rule with one decay a head and linear attention with decays per key channel (token by token, eight tokens at a time, in
portions, from stacks, beside single tokens, with padding rows, strong and weak decays, tall heads), the preparation
without low-rank rows, and the head norm with a SiLU gate."""

import math

import numpy as np
import pytest
import torch

from tests.gpu_common import cuda_ops
from tests.plain import plain_radilix as pr

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
        return rows.cuda().contiguous()
    noise = torch.randn(partials - 1, *rows.shape, generator=generator)
    return torch.cat([(rows - noise.sum(0))[None], noise]).cuda().contiguous()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,width,stacks,row", [(5, 256, (1,), True), (70, 96, (3, 1, 8), False), (3, 50, (2, 2), True), (300, 1000, (1, 1, 1), True),
                                                (2, 6000, (4, 16, 16, 16), True), (400, 5000, (1, 1), True), (1, 36, (), True), (8, 3584, (8, 8, 7), True)])
def test_sum_norm_adds_pending_sums_and_norms(dtype, n, width, stacks, row):
    ops = cuda_ops(dtype)
    g = torch.Generator().manual_seed(n + width)
    resid, weight = torch.randn(n, width, generator=g), 1 + 0.1 * torch.randn(width, generator=g)
    terms = [(torch.randn(n, width, generator=g), 0.4 + 0.3 * i) for i in range(len(stacks))]
    x = torch.randn(n, width, generator=g).to(dtype)
    columns = torch.rand(n, 7, generator=g)
    columns[::3, 5] = 0.0                                 # rows without a factor are not read
    if n > 1:
        x[0] = float("nan")
    joined = resid.double() + sum(s * t.double() for t, s in terms)
    if row:
        own = torch.where(columns[:, 5:6] != 0, x.double(), torch.zeros(1, dtype=torch.float64))
        joined = joined + 0.7 * columns[:, 5:6].double() * own
    want = pr.over_rms(joined, 1e-6) * weight.double()
    many = any(p > 1 for p in stacks)
    loose = max(tolerance(dtype), 3e-5 if many else 0)
    given = [(stacked(t, p, g), s) for (t, s), p in zip(terms, stacks)]
    device_columns, device_x = columns.cuda(), x.cuda()
    row_term = (device_x, device_columns[:, 5], 0.7) if row else None
    if n == 1:
        columns[:, 5] = 0.0
    at = resid.cuda()
    rows = torch.tensor([n - 1, 0], dtype=torch.int32, device="cuda")
    some = torch.empty(2, width, dtype=dtype, device="cuda")
    ops.sum_norm(at, given, weight.cuda(), 1e-6, some, rows=rows, row_term=row_term)
    assert torch.equal(at.cpu(), resid)                   # gathered rows leave the residual alone
    close(some, want[[n - 1, 0]], loose, "gathered")
    out = device_x if row else torch.empty(n, width, dtype=dtype, device="cuda")   # the output may lie where the rows lay
    ops.sum_norm(at, given, weight.cuda(), 1e-6, out, row_term=row_term)
    close(at, joined, 3e-5 if many else 3e-6, "residual")
    close(out, want, loose, "normed sum")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,heads,vdim,padded,partials", [(1, 3, 16, 16, 1), (9, 4, 24, 32, 3), (70, 2, 128, 128, 1), (5, 3, 5, 16, 2), (300, 6, 40, 48, 1)])
def test_gate_per_element(dtype, n, heads, vdim, padded, partials):
    ops = cuda_ops(dtype)
    g = torch.Generator().manual_seed(vdim)
    at = 20
    x = torch.randn(n, heads, padded, generator=g).to(dtype)
    fused = 3.0 * torch.randn(n, at + heads * vdim + 8, generator=g)
    want = x.double().clone()
    want[..., :vdim] *= torch.sigmoid(fused[:, at: at + heads * vdim].double()).view(n, heads, vdim)
    y = x.cuda().view(n, heads * padded).contiguous()
    ops.element_gate(y, stacked(fused, partials, g), at, heads, vdim)
    close(y.view(n, heads, padded), want, 2e-5 if dtype == torch.float32 else 1e-2, "gate")
    assert torch.equal(y.view(n, heads, padded)[..., vdim:].cpu(), x[..., vdim:])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,inter,width", [(1, 48, 64), (8, 200, 96), (64, 128, 40), (65, 128, 64), (300, 36, 64)])
def test_gelu_inside_and_behind_the_product(dtype, n, inter, width):
    ops = cuda_ops(dtype)
    g = torch.Generator().manual_seed(n)
    x, w = torch.randn(n, width, generator=g).to(dtype), (0.3 * torch.randn(inter, width, generator=g)).to(dtype)
    z = x.double() @ w.double().T
    out = torch.empty(n, inter, dtype=dtype, device="cuda")
    ops.linear_act(x.cuda(), w.cuda(), out, "gelu")
    if dtype == torch.bfloat16:
        z = z.to(torch.bfloat16).double()
    close(out, pr.gelu_erf(z), 3e-6 if dtype == torch.float32 else 1e-2, "gelu")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("experts,each,n,extra", [(9, 328, 300, 1), (3, 16, 33, 1), (4, 5, 7, 0), (16, 8, 70, 1), (1, 200, 2, 0), (7, 4, 5, 2)])
def test_ungated_experts_activation_times_their_weight(dtype, experts, each, n, extra):
    ops = cuda_ops(dtype)
    g = torch.Generator().manual_seed(each)
    x = (2.0 * torch.randn(n, experts * each, generator=g)).to(dtype)
    weights = torch.rand(n, experts + extra, generator=g)
    weights[:, experts - 1] = 0.0
    weights[0] = 1.0
    x[n - 1, (experts - 1) * each:] = float("nan")            # an expert that was not chosen gives exactly nothing
    want = pr.gelu_erf(x.double()) * weights.double()[:, :experts].repeat_interleave(each, 1)
    want[n - 1, (experts - 1) * each:] = 0.0
    y = x.cuda()
    ops.act_blocks(y, weights.cuda(), experts, each, "gelu")
    close(y, want, 1e-5 if dtype == torch.float32 else 1e-2, "experts")
    assert float(y[n - 1, (experts - 1) * each:].abs().max()) == 0.0
    z = torch.randn(n, experts * each, generator=g).to(dtype)
    y = z.cuda()
    ops.act_blocks(y, weights.cuda(), experts, each, "relu2")
    close(y, torch.relu(z.double()).pow(2) * weights.double()[:, :experts].repeat_interleave(each, 1), 1e-5 if dtype == torch.float32 else 1e-2, "relu2")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("experts,identity,top,width", [(8, 4, 3, 64), (12, 1, 1, 96), (5, 0, 2, 50), (3, 3, 6, 64), (1, 7, 2, 36), (60, 20, 9, 128)])
@pytest.mark.parametrize("n", [70, 702])
@pytest.mark.parametrize("correct,renormalise,shared", [(True, False, False), (False, False, True), (False, True, False), (True, True, True)])
def test_router_with_identity_experts(dtype, experts, identity, top, width, n, correct, renormalise, shared):
    """Identity experts take part in scores, choice and weights; what they are given leaves as one sum.  Many tokens go several to
    a block, with the same bits."""
    ops = cuda_ops(dtype)
    g = torch.Generator().manual_seed(experts + top)
    outputs = experts + identity
    x = torch.randn(n, width, generator=g).to(dtype)
    router = torch.randn(outputs, width, generator=g) * 0.2
    correction = 0.2 * torch.randn(outputs, generator=g) if correct else torch.zeros(outputs)
    gate = torch.randn(width, generator=g) * 0.2
    scores = torch.softmax(x.double() @ router.double().T, -1)
    margins = []
    chosen = pr.choose(scores, correction.double(), top, margins)
    sure = margins[0] > 1e-5
    assert sure.sum() > n // 2
    want = torch.where(chosen, scores, torch.zeros_like(scores))
    if renormalise:
        want = want / (want.sum(-1, keepdim=True) + 1e-9)
    out = torch.full((n, experts + int(shared) + int(identity > 0)), 5.0, device="cuda")
    ops.route_top(x.cuda(), router.cuda(), gate.cuda() if shared else None, out, top, 1e-9, renormalise=renormalise,
                  correction=correction.cuda() if correct else None, identity=identity)
    got = out.double().cpu()
    close(got[sure][:, :experts], want[sure][:, :experts], 1e-5, "weights")
    if identity:
        close(got[sure][:, -1], want[sure][:, experts:].sum(-1), 1e-5, "identity experts")
        if experts > 1:
            assert float(want[:, experts:].sum()) > 0
    if shared:
        close(got[:, experts], torch.sigmoid(x.double() @ gate.double()), 1e-5, "shared gate")
    few = torch.empty(9, out.shape[1], device="cuda")
    ops.route_top(x[:9].cuda().contiguous(), router.cuda(), gate.cuda() if shared else None, few, top, 1e-9, renormalise=renormalise,
                  correction=correction.cuda() if correct else None, identity=identity)
    assert torch.equal(few, out[:9])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,columns,rank,partials", [(1, 96, 16, 1), (7, 300, 3, 3), (90, 130, 20, 1), (65, 64, 128, 1), (8, 40, 200, 8)])
def test_low_rank_product(dtype, n, columns, rank, partials):
    ops = cuda_ops(dtype)
    g = torch.Generator().manual_seed(rank)
    at, padded = 12, -(-rank // 8) * 8
    fused = torch.randn(n, at + rank + 5, generator=g)
    matrix = torch.zeros(columns, padded, dtype=dtype)
    matrix[:, :rank] = torch.randn(columns, rank, generator=g).to(dtype)
    out = torch.full((n, columns), 9.0, device="cuda")
    ops.low_rank(stacked(fused, partials, g), at, rank, matrix.cuda(), out)
    close(out, fused[:, at: at + rank].double() @ matrix[:, :rank].double().T, 2e-5 if partials > 1 else 5e-6, "low rank")


# ------------------------------------------------------------------------------------------- recurrences
SHAPES = [(2, 1, 16, 8), (4, 2, 64, 32), (3, 3, 128, 128), (6, 6, 40, 24), (2, 2, 7, 5), (2, 1, 136, 48), (1, 1, 256, 20), (2, 2, 320, 12),
          (3, 1, 3, 70), (2, 2, 1, 9), (2, 1, 512, 8)]


def recurrence(kind, n, heads, kv_heads, dim, vdim, seed, strength):
    """The scan's inputs and what float64 makes of them: (pieces(a, b, partials) -> keyword arguments, step(a, b, state))."""
    g = torch.Generator().manual_seed(seed)
    share = heads // kv_heads
    q, k = torch.randn(n, kv_heads, dim, generator=g), torch.randn(n, kv_heads, dim, generator=g)
    v = torch.randn(n, heads, vdim, generator=g)
    q = q * dim ** -0.5
    at = 8
    if kind == "head":
        q, k = pr.unit_heads(q) * dim ** -0.5, pr.unit_heads(k)
        beta = torch.sigmoid(2.0 * torch.randn(n, heads, generator=g))
        z = 2.0 * torch.randn(n, heads, generator=g)
        rate, bias = (strength * torch.randn(heads, generator=g)).exp(), torch.randn(heads, generator=g) - 2.0
        decays = pr.head_decays(z.double(), rate.double().log(), bias.double())
        gates = torch.cat([torch.randn(n, at, generator=g), z, torch.randn(n, 4, generator=g)], -1)
        mixed, scale, sign = torch.cat([q.reshape(n, -1), k.reshape(n, -1), v.reshape(n, -1)], -1), 1.0, 1.0
    else:
        beta = None
        k = k * dim ** -0.5
        z = 3.0 * torch.randn(n, heads, dim, generator=g)
        tau = 1.0 / strength
        rate, bias = torch.full((heads,), 1.0 / tau), torch.randn(heads * dim, generator=g)
        decays = pr.channel_decays(z.double() + bias.double().view(heads, dim), tau)
        gates = torch.cat([torch.randn(n, at, generator=g), z.reshape(n, -1)], -1)
        scale, sign = 0.37, -1.0
        mixed = torch.cat([q.reshape(n, -1) / scale, k.reshape(n, -1), v.reshape(n, -1), torch.randn(n, 12, generator=g)], -1)

    def arguments(a, b, partials=1, stack_mixed=False):
        return dict(mixed=stacked(mixed[a:b], partials if stack_mixed else 1, g), beta=None if beta is None else beta[a:b].cuda().contiguous(),
                    gates=stacked(gates[a:b], partials, g), rate=rate.cuda(), bias=bias.cuda(), gate_at=at, per_head=kind == "head",
                    sign=sign, q_scale=scale)

    def step(a, b, state=None):
        wide = lambda t: t[a:b].double().repeat_interleave(share, 1)  # noqa: E731
        if kind == "head":
            return pr.delta_recurrence(wide(q), wide(k), v[a:b].double(), decays[a:b], beta[a:b].double(), state)
        return pr.gated_recurrence(wide(q), wide(k), v[a:b].double(), decays[a:b], state)

    return arguments, step


def scan(ops, arguments, state, starts, slots, out, heads, kv_heads, dim, vdim, q_lens):
    held = dict(arguments)
    ops.delta_scan(held.pop("mixed"), held.pop("beta"), held.pop("gates"), held.pop("rate"), held.pop("bias"), state,
                   torch.tensor(starts, dtype=torch.int32, device="cuda"), torch.tensor(slots, dtype=torch.int32, device="cuda"), out,
                   len(slots), heads, kv_heads, dim, vdim, q_lens=q_lens, **held)


@pytest.mark.parametrize("heads,kv_heads,dim,vdim", SHAPES)
@pytest.mark.parametrize("kind,strength", [("head", 0.5), ("head", 3.0), ("channel", 0.06), ("channel", 1.0)])
def test_scan_whole_walked_and_in_portions(heads, kv_heads, dim, vdim, kind, strength):
    """One sequence: eight tokens at a time, token by token, and cut into portions whose borders fall anywhere, against
    the recurrence in float64; decays from nearly one to nearly zero."""
    ops = cuda_ops(torch.float32)
    n = 150
    arguments, step = recurrence(kind, n, heads, kv_heads, dim, vdim, dim + heads, strength)
    want, last = step(0, n)
    size = -(-dim * vdim // 4) * 4
    for way, cuts in (("blocks", [n]), ("walk", [n]), ("portions", [1, 2, 37, 16, 1, 1, 15, 17, 8, 52]), ("stack", [n]), ("walked stack", [n]),
                      ("runs", [n]), ("runs of one block", [40, 110]), ("runs in portions", [70, 1, 79])):
        ops.delta_run_blocks = 1 if "one block" in way else 4 if "runs" in way else 0   # (150 tokens are cut into runs only when asked)
        state = torch.full((3, heads, size), 5.0, device="cuda")
        state[1] = 0.0
        out = torch.empty(n, heads * vdim, device="cuda")
        at = 0
        for cut in cuts:
            scan(ops, arguments(at, at + cut, 3 if "stack" in way else 1, way == "walked stack"), state, [0, cut], [1], out[at: at + cut],
                 heads, kv_heads, dim, vdim, None if "walk" in way else [cut])
            at += cut
        tol = 3e-5 if "stack" in way else 1e-5
        close(out.view(n, heads, vdim), want, tol, way)
        close(state[1][:, : dim * vdim].view(heads, dim, vdim), last, tol, way + " state")
        assert float(state[0].min()) == 5.0 and float(state[2].max()) == 5.0


@pytest.mark.parametrize("kind", ["head", "channel"])
@pytest.mark.parametrize("runs", [0, 3])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(4, 2, 64, 32), (3, 3, 20, 36), (2, 1, 128, 100), (1, 1, 200, 3)])
def test_scan_of_unequal_sequences_with_padding_rows(kind, runs, heads, kv_heads, dim, vdim):
    """Portions beside single tokens beside rows without a slot, more sequences than a warp has lanes; each as alone, also
    where portions are cut into runs that walk side by side."""
    ops = cuda_ops(torch.float32)
    ops.delta_run_blocks = runs
    lengths = [1, 40, 1, 16, 15, 9, 200, 1] + [1, 17] * 16
    n, count = sum(lengths), len(lengths)
    arguments, step = recurrence(kind, n, heads, kv_heads, dim, vdim, 3, 0.4)
    size = -(-dim * vdim // 4) * 4
    slots = list(range(count))[::-1]
    slots[2], slots[4], slots[3] = -1, -1, -1
    state = torch.randn(count, heads, size, generator=torch.Generator().manual_seed(2)).cuda()
    before = state.clone()
    starts = np.cumsum([0] + lengths)
    out = torch.full((n, heads * vdim), 9.0, device="cuda")
    scan(ops, arguments(0, n), state, starts, slots, out, heads, kv_heads, dim, vdim, lengths)
    for i, slot in enumerate(slots):
        a, b = starts[i], starts[i + 1]
        if slot < 0:
            assert float(out[a:b].abs().max()) == 0.0
            continue
        want, last = step(a, b, before[slot][:, : dim * vdim].double().cpu().view(heads, dim, vdim))
        close(out[a:b].view(-1, heads, vdim), want, 2e-5, f"sequence {i}")
        close(state[slot][:, : dim * vdim].view(heads, dim, vdim), last, 2e-5, f"state {i}")
    for slot in set(range(count)) - set(slots):
        assert torch.equal(state[slot], before[slot])


@pytest.mark.parametrize("kind", ["head", "channel"])
def test_scan_takes_heads_in_turns_when_the_scratch_is_bounded(kind):
    ops = cuda_ops(torch.float32)
    heads, dim, vdim, n = 5, 24, 12, 100
    arguments, _ = recurrence(kind, n, heads, heads, dim, vdim, 8, 0.5)
    results = []
    ops.delta_run_blocks = 4
    for bound in (ops.DELTA_SCRATCH_FLOATS, 2 * 13 * ops.core.shrike_delta_scan_record(dim, int(kind == "head"))):
        ops.DELTA_SCRATCH_FLOATS = bound
        state, out = torch.zeros(1, heads, dim * vdim, device="cuda"), torch.empty(n, heads * vdim, device="cuda")
        scan(ops, arguments(0, n), state, [0, n], [0], out, heads, heads, dim, vdim, [n])
        results.append((out, state))
    assert torch.equal(results[0][0], results[1][0]) and torch.equal(results[0][1], results[1][1])


@pytest.mark.parametrize("kind,heads", [("head", 4), ("channel", 4), ("channel", 12)])
def test_a_long_prompt_is_cut_into_runs(kind, heads):
    """By the library's own rule: few heads and 1,500 tokens in runs, many sequences not; the same numbers either way."""
    ops = cuda_ops(torch.float32)
    dim = vdim = 128
    n = 1500
    blocks = -(-n // 8)
    assert ops.core.shrike_delta_scan_run_blocks(blocks, blocks, 1, heads, dim, vdim, int(kind == "head")) >= 16
    assert ops.core.shrike_delta_scan_run_blocks(64 * blocks, blocks, 64, heads, dim, vdim, int(kind == "head")) == 0
    assert ops.core.shrike_delta_scan_run_blocks(8, 8, 1, heads, dim, vdim, int(kind == "head")) == 0
    arguments, step = recurrence(kind, n, heads, heads, dim, vdim, 4, 0.1)
    want, last = step(0, n)
    for runs in (None, 0):
        ops.delta_run_blocks = runs
        state, out = torch.zeros(1, heads, dim * vdim, device="cuda"), torch.empty(n, heads * vdim, device="cuda")
        before = ops.launches
        scan(ops, arguments(0, n), state, [0, n], [0], out, heads, heads, dim, vdim, [n])
        assert ops.launches - before == (4 if runs is None else 2)
        close(out.view(n, heads, vdim), want, 2e-5, f"runs {runs}")
        close(state[0].view(heads, dim, vdim), last, 2e-5, f"state, runs {runs}")


def test_scan_refuses_what_no_kernel_serves():
    from shrike_b200.ops.cuda_ops import KernelError

    ops = cuda_ops(torch.float32)
    arguments, _ = recurrence("channel", 40, 2, 2, 16, 8, 1, 0.5)
    state, out = torch.zeros(1, 2, 128, device="cuda"), torch.empty(40, 16, device="cuda")
    with pytest.raises(KernelError, match="not as a stack"):
        scan(ops, arguments(0, 40, 3, True), state, [0, 40], [0], out, 2, 2, 16, 8, [40])
    with pytest.raises(KernelError, match="decay per head only with beta"):
        scan(ops, dict(arguments(0, 40), per_head=True, bias=torch.zeros(2, device="cuda")), state, [0, 40], [0], out, 2, 2, 16, 8, [40])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps", [1, 3, 4, 6])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,partials", [(4, 2, 16, 8, 1), (3, 3, 128, 64, 1), (2, 1, 10, 7, 3)])
def test_preparation_without_low_rank_rows_across_cuts(dtype, taps, heads, kv_heads, dim, vdim, partials):
    ops = cuda_ops(dtype)
    g = torch.Generator().manual_seed(taps * 10 + heads)
    qk, channels = kv_heads * dim, 2 * kv_heads * dim + heads * vdim
    beta_at = channels + heads * vdim
    total = -(-(beta_at + 2 * heads) // 16) * 16
    whole = torch.randn(123, total, generator=g)
    weights = torch.randn(channels, taps, generator=g)
    y = pr.silu(pr.short_convolution(whole[:, :channels].double(), weights))
    want = torch.cat([pr.unit_heads(y[:, :qk].view(-1, kv_heads, dim)).reshape(-1, qk) * dim ** -0.5,
                      pr.unit_heads(y[:, qk: 2 * qk].view(-1, kv_heads, dim)).reshape(-1, qk), y[:, 2 * qk:]], -1)
    state = torch.full((3, max(taps - 1, 0), channels), 7.0, device="cuda")
    state[1] = 0.0
    got, at = [], 0
    for cut in (2, 1, 1, 20, 99):
        rows = whole[at: at + cut]
        mixed, beta = torch.empty(cut, channels, device="cuda"), torch.empty(cut, heads, device="cuda")
        ops.delta_prep(stacked(rows, partials, g), weights.cuda(), state, torch.tensor([0, cut], dtype=torch.int32, device="cuda"),
                       torch.tensor([1], dtype=torch.int32, device="cuda"), torch.zeros(cut, dtype=torch.int32, device="cuda"), mixed, beta,
                       None, 1, heads, kv_heads, dim, vdim, beta_at, 0, 1e-6, longest=cut)
        close(beta, torch.sigmoid(rows[:, beta_at: beta_at + heads].double()), 1e-5, "beta")
        got.append(mixed.cpu())
        at += cut
    close(torch.cat(got), want, 5e-5 if partials > 1 or dtype == torch.bfloat16 else 1e-5, "q, k and v")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,heads,size,partials", [(5, 3, 16, 1), (70, 2, 128, 1), (3, 5, 7, 3), (9, 4, 200, 2)])
def test_head_norm_with_a_silu_gate(dtype, n, heads, size, partials):
    ops = cuda_ops(dtype)
    g = torch.Generator().manual_seed(size)
    x, weight = torch.randn(n, heads * size, generator=g), 1 + 0.1 * torch.randn(size, generator=g)
    at = 12
    gates = 3.0 * torch.randn(n, at + heads * size + 4, generator=g)
    gates[0, at] = -200.0                                     # far out on either side the gate is 0 or its input
    gates[0, at + 1] = 200.0
    want = pr.head_norm(x.double().view(n, heads, size), weight, 1e-5).reshape(n, -1) * pr.silu(gates[:, at: at + heads * size].double())
    out = torch.empty(n, heads * size, dtype=dtype, device="cuda")
    ops.head_rms(x.cuda(), weight.cuda(), 1e-5, out, heads, gate_source=stacked(gates, partials, g), gate_at=at, gate="silu")
    close(out, want, 2e-5 if dtype == torch.float32 else 1e-2, "head norm")


def test_decay_exponent_is_the_root_of_a_sigmoid():
    """exp(-softplus(-z) / tau) = sigmoid(z)^(1/tau), also where the sigmoid underflows."""
    z = torch.tensor([-300.0, -20.0, -1.0, 0.0, 3.0, 40.0], dtype=torch.float64)
    for tau in (1.0, 16.0, 200.0):
        assert torch.allclose(pr.channel_decays(z, tau)[1:], torch.sigmoid(z[1:]).pow(1.0 / tau), rtol=1e-12)
        assert math.isclose(float(pr.channel_decays(z, tau)[0]), math.exp(-300.0 / tau), rel_tol=1e-9)
