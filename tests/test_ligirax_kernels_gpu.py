"""The kernels of the Ligirax design, each alone, against the plain implementation's functions (float64), in float32 and
bfloat16 storage: the row-wise kernel between the latent mixer's product and its attention with direct queries and
gates, the pair rotation with a factor, attention over shared rows with a gate and inputs built so that a key just
inside or just outside the window decides the result, the norm of a branch and of the stream in one pass, and routed
experts with identity choices."""

import math

import pytest
import torch

import ligirax_util as lu
from plain import ligirax_plain as plain

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]
TOL = {torch.float32: dict(atol=2e-5, rtol=2e-5), torch.bfloat16: dict(atol=2e-2, rtol=2e-2)}
TURNED = {torch.float32: dict(atol=5e-4, rtol=1e-4), torch.bfloat16: dict(atol=4e-2, rtol=2e-2)}   # float32 angles


def _ops():
    from ampere_kv_engine_b200.kernels import ops
    return ops


def _gen(seed):
    return torch.Generator(device="cuda").manual_seed(seed)


def _turn_at(x, positions, rotation):
    """plain.turn for rows at arbitrary positions."""
    freq, factor = plain.turn_frequencies(rotation)
    dims = rotation["dims"]
    angle = positions.double()[:, None] * freq[None, :]
    shape = [x.shape[0]] + [1] * (x.dim() - 2) + [dims // 2]
    cos, sin = factor * angle.cos().view(shape), factor * angle.sin().view(shape)
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2], out[..., 1:dims:2] = u * cos - v * sin, v * cos + u * sin
    return out


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,heads,dim,rot_dim,dims,rank,has_kv,gated,spare", [
    (29, 3, 12, 8, 8, 24, True, True, 1), (1, 5, 7, 8, 6, 33, False, True, 0), (300, 16, 64, 32, 32, 256, True, True, 0),
    (8, 20, 48, 64, 64, 512, True, False, 4), (3, 1, 4, 2, 2, 16, False, False, 0), (5, 40, 16, 128, 128, 64, True, True, 0)])
def test_latent_prep_with_query_heads_and_gates(dtype, n, heads, dim, rot_dim, dims, rank, has_kv, gated, spare):
    ops = _ops()
    page_size, eps, g = 8, 1e-5, _gen(n + heads)
    pages = n // page_size + 3
    rotation = lu.rot(dims, 500.0, (3.0, 200, 8.0, 1.0))
    freq, factor = plain.turn_frequencies(rotation)
    q_cols, kv_cols = heads * (dim + rot_dim), rank + rot_dim if has_kv else 0
    x = (2.0 * torch.randn((n, q_cols + kv_cols + (heads if gated else 0) + spare), generator=g, device="cuda")).to(dtype)
    positions = torch.randint(0, 1000, (n,), generator=g, device="cuda").to(torch.int32)
    weight = 1 + 0.1 * torch.randn(rank, generator=g, device="cuda")
    slots = torch.randperm(pages * page_size, generator=g, device="cuda")[:n].to(torch.int32)
    if n > 2:
        slots[1] = -1                                    # a row that is not to be kept
    cache = torch.full((pages, 1, page_size, rank + rot_dim), 5.0, device="cuda", dtype=dtype)
    q_rows = torch.full((n, heads * (rank + rot_dim)), 7.0, device="cuda", dtype=dtype)
    q_latent, gate = ops.latent_prep(
        x, positions, slots if has_kv else None, None, weight if has_kv else None, freq.float().cuda(),
        cache if has_kv else None, q_rank=0, kv_rank=rank, rot_dim=rot_dim, rotary_dims=dims, eps=eps, factor=factor,
        q_rows=q_rows, heads=heads, head_dim=dim, has_kv=has_kv, gated=gated)
    assert q_latent is None
    xd, pos = x.double().cpu(), positions.cpu().long()
    got = q_rows.double().cpu().view(n, heads, rank + rot_dim)
    want = _turn_at(xd[:, :q_cols].reshape(n, heads, dim + rot_dim)[..., dim:], pos, rotation)
    torch.testing.assert_close(got[..., rank:], want, **TURNED[dtype])
    assert bool((got[..., :rank] == 7.0).all())
    if gated:
        torch.testing.assert_close(gate.double().cpu(), torch.sigmoid(xd[:, q_cols + kv_cols:q_cols + kv_cols + heads]),
                                   atol=1e-6, rtol=1e-5)
    else:
        assert gate is None
    if has_kv:
        down = xd[:, q_cols:q_cols + kv_cols]
        row = torch.cat((plain.rms_norm(down[:, :rank], weight.double().cpu(), eps), _turn_at(down[:, rank:], pos, rotation)), dim=-1)
        s = slots.cpu().long()
        keep = s >= 0
        flat = cache.double().cpu().view(pages * page_size, -1)
        torch.testing.assert_close(flat[s[keep]], row[keep], **TURNED[dtype])
        untouched = torch.ones(pages * page_size, dtype=torch.bool)
        untouched[s[keep]] = False
        assert bool((flat[untouched] == 5.0).all())


@pytest.mark.parametrize("dtype", DTYPES)
def test_latent_prep_with_a_query_latent_and_gates(dtype):
    """The other composition: a query latent in front, gates behind, no key/value side (another layer's rows are read)."""
    ops = _ops()
    n, q_rank, rank, heads, g = 9, 20, 24, 3, _gen(2)
    x = torch.randn((n, q_rank + heads), generator=g, device="cuda").to(dtype)
    positions = torch.arange(n, device="cuda", dtype=torch.int32)
    weight = 1 + 0.1 * torch.randn(q_rank, generator=g, device="cuda")
    q_latent, gate = ops.latent_prep(x, positions, None, weight, None, torch.ones(4, device="cuda"), None, q_rank=q_rank,
                                     kv_rank=rank, rot_dim=8, rotary_dims=8, eps=1e-6, heads=heads, has_kv=False, gated=True)
    torch.testing.assert_close(q_latent.double().cpu(), plain.rms_norm(x.double().cpu()[:, :q_rank], weight.double().cpu(), 1e-6),
                               **TOL[dtype])
    torch.testing.assert_close(gate.double().cpu(), torch.sigmoid(x.double().cpu()[:, q_rank:]), atol=1e-6, rtol=1e-5)


def test_pair_rotation_with_a_factor():
    ops = _ops()
    n, heads, g = 11, 3, _gen(5)
    rotation = lu.rot(6, 50.0, (4.0, 64, 4.0, 1.0))
    freq, factor = plain.turn_frequencies(rotation)
    q = torch.randn((n, heads * 14), generator=g, device="cuda")
    out = torch.zeros((n, heads * 20), device="cuda")
    positions = torch.arange(n, device="cuda", dtype=torch.int32)
    ops.rotate_pairs(q, out, positions, freq.float().cuda(), heads=heads, cols=8, rotary_dims=6, in_offset=6, out_offset=12,
                     factor=factor)
    want = _turn_at(q.double().cpu().view(n, heads, 14)[..., 6:], torch.arange(n), rotation)
    torch.testing.assert_close(out.double().cpu().view(n, heads, 20)[..., 12:], want, atol=1e-5, rtol=1e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,rank,rot_dim", [(5, 24, 8), (20, 128, 32), (3, 64, 16)])
@pytest.mark.parametrize("splits", [1, 4])
def test_a_key_at_the_edge_of_a_window_over_shared_rows(dtype, heads, rank, rot_dim, splits):
    """All rows but one are orthogonal to the queries; the one that is not owns the output while it lies inside the
    window of the query, times the head's gate, and must not show once it is outside.  Prompt tiles (every query of the
    portion looks at the same row: it leaves the window in the middle of the portion) and single tokens; pages behind
    the window are not held and hold NaN; the marked row sits at page borders too."""
    ops = _ops()
    page_size, ctx, row = 16, 300, rank + rot_dim
    dev = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    for window, mark in ((100, 200), (100, 199), (100, 207), (100, 208), (17, 255), (64, 239), (300, 0), (1, 280)):
        for first, n, q_tile in ((260, 40, 32), (299, 1, 1), (min(mark + window - 1, 299), 1, 1), (min(mark + window, 299), 1, 1)):
            length = first + n
            num_pages = (length + page_size - 1) // page_size
            table = torch.arange(num_pages - 1, -1, -1, dtype=torch.int32)
            rows = torch.zeros((length, row))
            rows[:, 1] = 1.0
            rows[mark:mark + 1, :2] = torch.tensor([1.0, -3.0])
            paged = torch.full((num_pages, 1, page_size, row), float("nan"))
            held = max(0, first - window + 1) // page_size
            for j in range(num_pages):
                if j < held:
                    table[j] = -1
                    continue
                part = rows[j * page_size:(j + 1) * page_size]
                paged[table[j], 0] = 0.0
                paged[table[j], 0, :part.shape[0]] = part
            paged = paged.cuda().to(dtype)
            q = torch.zeros((n, heads, row))
            q[:, :, 0] = 30.0
            gate = torch.linspace(0.2, 1.0, heads)[None].repeat(n, 1)
            out = torch.full((n, heads * rank), float("nan"), device="cuda", dtype=dtype)
            tiles = [(t0, min(q_tile, n - t0)) for t0 in range(0, n, q_tile)]
            ops.scored_attention(q.view(n, -1).cuda().to(dtype), paged, paged, table[None].cuda(), dev([0, n]), dev([length]),
                                 dev([0] * len(tiles)), dev([t for t, _ in tiles]), dev([c for _, c in tiles]),
                                 num_tiles=len(tiles), q_tile=q_tile, num_splits=splits, num_heads=heads, num_kv_heads=1,
                                 v_dim=rank, scale=1.0, window=window, gate=gate.cuda(), out=out)
            got = out.float().cpu().view(n, heads, rank)
            for i in range(n):
                seen = 0 <= first + i - mark < window
                want = gate[i] * (-3.0 if seen else 1.0)
                torch.testing.assert_close(got[i, :, 1], want, atol=2e-2, rtol=1e-2, msg=str((window, mark, first + i, seen)))


@pytest.mark.parametrize("width", [40, 63, 512, 2048])
@pytest.mark.parametrize("n", [1, 7, 300])
@pytest.mark.parametrize("dtype", DTYPES)
def test_branch_norm_and_stream_norm_in_one_pass(dtype, n, width):
    """Clusters (few rows, wide), 16-byte accesses and not, whole batches and gathered rows, without a second norm."""
    ops = _ops()
    g = _gen(width + n)
    hidden = torch.randn((n, width), generator=g, device="cuda")
    branch = (0.3 * torch.randn((n, width), generator=g, device="cuda")).to(dtype)
    w1, w2 = (1 + 0.2 * torch.randn(width, generator=g, device="cuda") for _ in range(2))
    pending = ops.NormedBranch(branch, w1, 1e-3)
    new = hidden.double().cpu() + plain.rms_norm(branch.double().cpu(), w1.double().cpu(), 1e-3)
    want = plain.rms_norm(new, w2.double().cpu(), 1e-5)
    rows = torch.randint(0, n, (5,), generator=g, device="cuda").to(torch.int32)
    before = hidden.clone()
    out = ops.branch_rmsnorm(hidden, pending, w2, 1e-5, dtype, rows=rows)
    assert torch.equal(hidden, before)
    torch.testing.assert_close(out.double().cpu(), want[rows.cpu().long()], **TOL[dtype])
    out = ops.branch_rmsnorm(hidden, pending, w2, 1e-5, dtype)
    assert out.dtype == dtype
    torch.testing.assert_close(out.double().cpu(), want, **TOL[dtype])
    torch.testing.assert_close(hidden.double().cpu(), new, atol=1e-5, rtol=1e-5)
    pending.apply(before)
    torch.testing.assert_close(before, hidden, atol=1e-6, rtol=1e-6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,width,top,shared", [(1, 40, 1, False), (9, 63, 3, True), (200, 256, 4, False), (4, 1024, 8, False)])
def test_a_routed_branch_with_identity_choices_is_summed_and_normed(dtype, n, width, top, shared):
    """Rows of identity choices were never written (NaN here): they must not be read."""
    ops = _ops()
    g = _gen(n * top)
    first = 5
    chosen = torch.stack([torch.randperm(9, generator=torch.Generator().manual_seed(i))[:top] for i in range(n)]).to(torch.int32)
    chosen[0, 0] = 7
    if n > 1:
        chosen[1] = torch.arange(top) + (first if top <= 4 else 0)       # a token with nothing but the identity
    weights = torch.rand((n, top), generator=g, device="cuda")
    x = torch.randn((n, width), generator=g, device="cuda").to(dtype)
    parts = torch.randn((n, top, width), generator=g, device="cuda")
    parts[(chosen >= first).cuda()] = float("nan")
    extra = torch.randn((n, width), generator=g, device="cuda").to(dtype) if shared else None
    same = (chosen >= first)[:, :, None]
    total = torch.where(same, weights.double().cpu()[:, :, None] * x.double().cpu()[:, None], parts.double().cpu()).sum(1)
    if shared:
        total = total + extra.double().cpu()
    e = ops.ExpertParts(parts.view(n * top, width), extra, top,
                        ops.IdentityChoices(chosen.cuda(), weights, x, first))
    torch.testing.assert_close(e.materialize().double().cpu(), total, atol=1e-5, rtol=1e-5)
    hidden = torch.randn((n, width), generator=g, device="cuda")
    w1, w2 = (1 + 0.2 * torch.randn(width, generator=g, device="cuda") for _ in range(2))
    new = hidden.double().cpu() + plain.rms_norm(total, w1.double().cpu(), 1e-4)
    last = torch.tensor([n - 1], dtype=torch.int32, device="cuda")
    out = ops.branch_rmsnorm(hidden, ops.NormedBranch(e, w1, 1e-4), w2, 1e-6, dtype, rows=last)
    torch.testing.assert_close(out.double().cpu(), plain.rms_norm(new[-1:], w2.double().cpu(), 1e-6), **TOL[dtype])
    out = ops.branch_rmsnorm(hidden, ops.NormedBranch(e, w1, 1e-4), w2, 1e-6, dtype)
    torch.testing.assert_close(out.double().cpu(), plain.rms_norm(new, w2.double().cpu(), 1e-6), **TOL[dtype])
    torch.testing.assert_close(hidden.double().cpu(), new, atol=1e-5, rtol=1e-5)


def test_a_gathered_row_outside_the_batch_sets_the_status():
    ops = _ops()
    hidden, branch, w = (torch.ones((2, 512), device="cuda") for _ in range(3))
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    rows = torch.tensor([1, 9], dtype=torch.int32, device="cuda")
    ops.branch_rmsnorm(hidden, ops.NormedBranch(branch, w[0].contiguous(), 1e-5), w[1].contiguous(), 1e-5, torch.float32,
                       rows=rows, status=status)
    assert int(status) != 0


@pytest.mark.parametrize("tokens", [1, 3, 70, 257])
@pytest.mark.parametrize("experts,identity,top", [(5, 3, 3), (3, 0, 2), (2, 2, 4), (30, 10, 6), (1, 1, 1)])
def test_routing_without_renormalisation(tokens, experts, identity, top):
    ops = _ops()
    g = _gen(tokens + experts)
    logits = 3 * torch.randn((tokens, experts + identity), generator=g, device="cuda")
    correction = 0.5 * torch.randn(experts + identity, generator=g, device="cuda")
    for scale in (1.0, 0.5):
        chosen, weights = ops.moe_route(logits, correction, top=top, groups=1, keep_groups=1, group_top=1, scale=scale,
                                        weight_eps=0.0, score="softmax", normalize=False)
        eye = torch.eye(experts + identity, dtype=torch.float64)
        want, s, lead = plain.route(logits.double().cpu(), eye, correction.double().cpu(), top)
        clear = lead > 1e-6
        assert torch.equal(chosen.cpu().long()[clear], want[clear])
        torch.testing.assert_close(weights.double().cpu()[clear], scale * s[clear], atol=1e-6, rtol=1e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens", [1, 5, 90, 400])
@pytest.mark.parametrize("width,ff,experts,identity,top", [(72, 24, 5, 3, 3), (63, 15, 3, 1, 2), (256, 128, 6, 2, 4), (48, 16, 2, 4, 6)])
def test_a_mixture_with_identity_choices(dtype, tokens, width, ff, experts, identity, top):
    """The part as a layer uses it, every kernel of it in its place, against the plain mixture."""
    from ampere_kv_engine_b200.config.spec import PartSpec
    from ampere_kv_engine_b200.parts.base import FEED_FORWARDS, build_part
    from ampere_kv_engine_b200.parts import routed_experts  # noqa: F401  (registers the kind)
    g = torch.Generator().manual_seed(tokens + width)
    part = build_part(FEED_FORWARDS, PartSpec("routed_experts", {
        "experts": experts, "identity": identity, "top": top, "score": "softmax", "normalize": False,
        "intermediate_size": ff, "limit": 0.9, "swish_slope": 1.702,
        "names": {"expert": "e{}", "gate": "gate", "up": "up", "down": "down", "router": "router",
                  "correction": "correction"}}, "mlp"), hidden_size=width, dtype=dtype, device=torch.device("cuda"))
    t = {}
    for name, ps in part.param_specs().items():
        v = torch.randn(ps.shape, generator=g) * (0.2 if name == "correction" else 2.0 * ps.shape[-1] ** -0.5)
        t[name] = v.to(torch.bfloat16).float()
    part.load({k: v.cuda().to(torch.float32 if k == "correction" else dtype) for k, v in t.items()})
    w = {k: v.double() for k, v in t.items()}
    x = torch.randn((4 * tokens, width), generator=g).to(torch.bfloat16).float()
    # tokens whose choice is no close call
    _, _, lead = plain.route(x.double(), w["router"], w["correction"], top)
    x = x[lead > 2e-3][:tokens]
    class Ctx:
        status = None
    got = part.forward(x.cuda().to(dtype), Ctx())
    want = plain.mixture(x.double(), w, {"expert": {"limit": 0.9}, "router": {"experts": experts, "top": top}})
    torch.testing.assert_close(got.double().cpu(), want, **TOL[dtype])
    assert math.isfinite(float(got.sum()))
