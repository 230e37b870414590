"""The kernels of the Gosizen design, each alone, against the plain implementation's functions (float64), in float32 and
bfloat16 storage: attention with sinks in every kernel that takes them (inputs built so that a sink, or a key just inside
or just outside a window or a block, decides the result), the short convolutions before the turn and their inputs across
step borders, gates per element, the delta rule with a decay per channel and its step and gate from a product of their
own, experts without a gate, and what acts on the stream itself."""

import math

import pytest
import torch

import gosizen_util as gu
from paged_case import PagedCase
from plain import gosizen_plain as plain

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]
TOL = {torch.float32: dict(atol=2e-5, rtol=2e-5), torch.bfloat16: dict(atol=2e-2, rtol=2e-2)}
TURNED = {torch.float32: dict(atol=5e-4, rtol=1e-4), torch.bfloat16: dict(atol=4e-2, rtol=2e-2)}   # float32 angles


def _ops():
    from ampere_kv_engine_b200.kernels import ops
    return ops


def _gen(seed):
    return torch.Generator(device="cuda").manual_seed(seed)


def _randn(*shape, seed=0, dtype=torch.float32, scale=1.0):
    return (torch.randn(*shape, generator=_gen(seed), device="cuda") * scale).to(dtype)


def _i32(values):
    return torch.tensor(values, dtype=torch.int32, device="cuda")


# ----------------------------------------------------------------------------- attention with sinks


def _attend(ops, case, sink, scale, window=0, chunk=0, splits=1, kernel="auto", shared=False, v_dim=None, gate=None):
    """scored_attention over a PagedCase; ``shared``: one storage whose rows are key and value at once."""
    v_dim = v_dim or case.d
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    k = case.k_cache.cuda()
    out = ops.scored_attention(
        torch.cat([x.reshape(x.shape[0], -1) for x in case.q_seq]).cuda(), k, k if shared else case.v_cache.cuda(),
        case.table.cuda(), case.cu.cuda(), _i32(case.ctx_lens), *(t.cuda() for t in case.tiles), num_tiles=len(case.tiles[0]),
        q_tile=case.tile_rows, num_splits=splits, num_heads=case.nh, num_kv_heads=case.nkv, v_dim=v_dim, scale=scale,
        window=window, chunk=chunk, gate=gate, status=status, sink=sink, kernel=kernel)
    assert int(status.item()) == 0
    return out.double().cpu()


def _attend_plain(case, sink, scale, window=0, chunk=0, shared=False, v_dim=None):
    v_dim, rows = v_dim or case.d, []
    for s, (n, c) in enumerate(zip(case.q_lens, case.ctx_lens)):
        mask = plain.window_mask(c, window) if window else plain.chunk_mask(c, chunk) if chunk else plain.window_mask(c, c)
        heads = []
        for h in range(case.nh):
            g = h // (case.nh // case.nkv)
            k = case.k_seq[s][:, g].double()
            v = k[:, :v_dim] if shared else case.v_seq[s][:, g].double()
            score = torch.zeros(c, c, dtype=torch.float64)
            score[c - n:] = case.q_seq[s][:, h].double() @ k.T * scale
            heads.append((plain.sink_softmax(score, mask, sink[h].double().cpu()) @ v)[c - n:])
        rows.append(torch.cat(heads, dim=-1))
    return torch.cat(rows)


#: (dtype, heads, kv heads, width, page): the general kernel, the tensor-core decode kernel, the tcgen05 prompt kernel
SINK_CASES = [(torch.float32, 6, 2, 20, 8), (torch.bfloat16, 6, 2, 20, 8), (torch.bfloat16, 4, 2, 64, 16),
              (torch.bfloat16, 8, 2, 128, 16), (torch.float32, 3, 3, 128, 16)]


@pytest.mark.parametrize("dtype,nh,nkv,d,page", SINK_CASES)
@pytest.mark.parametrize("sinks", ["mixed", "high", "low"])
@pytest.mark.parametrize("mask", [(0, 0), (33, 0), (0, 40)])
def test_a_sink_takes_its_share(dtype, nh, nkv, d, page, sinks, mask):
    ops = _ops()
    base = _randn(nh, seed=nh)
    # a sink far above every score leaves almost nothing to the keys, one far below leaves a plain softmax
    sink = {"mixed": 2.0 * base, "high": base + 30.0, "low": base - 60.0}[sinks].contiguous()
    window, chunk = mask
    scale = d ** -0.5
    for q_lens, ctx, splits in (([1, 1, 1], [200, 3, 41], (1, 4)), ([70, 2, 33], [170, 2, 73], (1,))):
        case = PagedCase(dtype, nh, nkv, d, page, q_lens, ctx, seed=d + len(splits), q_tile=32)
        want = _attend_plain(case, sink, scale, window, chunk)
        for n in splits:
            for kernel in ("auto", "general"):
                if n > 1 and kernel == "auto" and d == 20:
                    continue
                got = _attend(ops, case, sink, scale, window, chunk, splits=n, kernel=kernel)
                tol = TOL[dtype] if sinks != "high" else dict(atol=1e-9, rtol=2e-2)
                torch.testing.assert_close(got, want, **tol)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("row,v_dim", [(80, 64), (160, 128), (288, 256), (576, 512), (52, 33)])
@pytest.mark.parametrize("window", [0, 33])
def test_a_sink_over_shared_rows(dtype, row, v_dim, window):
    """Rows that are key and value at once, many heads on them, with a gate."""
    ops = _ops()
    nh, scale = 20, row ** -0.5
    sink = 2.0 * _randn(nh, seed=row)
    for q_lens, ctx, splits in (([1, 1, 1], [300, 7, 65], (1, 3)), ([40, 5], [90, 5], (1, 2))):
        case = PagedCase(dtype, nh, 1, row, 16, q_lens, ctx, seed=row, q_tile=32)
        gate = torch.rand(sum(q_lens), nh, generator=_gen(1), device="cuda")
        want = _attend_plain(case, sink, scale, window, shared=True, v_dim=v_dim)
        want = (want.view(-1, nh, v_dim) * gate.double().cpu()[:, :, None]).reshape(want.shape)
        for n in splits:
            got = _attend(ops, case, sink, scale, window, splits=n, shared=True, v_dim=v_dim, gate=gate)
            torch.testing.assert_close(got, want, **TOL[dtype])


@pytest.mark.parametrize("dtype,nh,nkv,d,page", SINK_CASES)
@pytest.mark.parametrize("prompt", [True, False])
@pytest.mark.parametrize("window,chunk", [(48, 0), (0, 48), (0, 50)])
def test_one_key_stands_out_just_inside_and_just_outside(dtype, nh, nkv, d, page, prompt, window, chunk):
    """A key whose score stands far above the sink and every other key: the output is its value where it is seen, and
    almost nothing (the sink's share is all) where it is not.  Pages wholly out of reach are NaN."""
    ops = _ops()
    ctx = 200
    sink = torch.full((nh,), 6.0, device="cuda")
    last = ctx - 1
    inside = last - window + 1 if window else last // chunk * chunk
    for where in (inside, inside - 1):
        case = PagedCase(dtype, nh, nkv, d, page, [4 if prompt else 1], [ctx], seed=3, q_tile=16)
        case.q_seq[0] *= 0.0
        case.q_seq[0][:, :, 0] = 1.0
        case.k_seq[0] *= 0.05
        case.k_seq[0][:, :, 0] = -1.0
        case.k_seq[0][where, :, 0] = 20.0
        case.rewrite_cache()
        first_row = last - 3 if prompt else last
        reach = max(0, first_row - window + 1) if window else first_row // chunk * chunk
        for lp in range(min(reach, where) // page):         # what no row of the step can see
            case.k_cache[int(case.table[0, lp])] = float("nan")
            case.v_cache[int(case.table[0, lp])] = float("nan")
        got = _attend(ops, case, sink, 1.0, window, chunk)[-1].view(nh, d)
        value = case.v_seq[0][where].double().repeat_interleave(nh // nkv, dim=0)
        if where == inside:
            torch.testing.assert_close(got, value, **TOL[dtype])
        else:
            assert float(got.abs().max()) < 0.2


# ----------------------------------------------------------------------------- short convolutions before the turn


def _conv_case(dtype, n, H, G, D, V, taps, gate_cols, x_off, seed):
    channels = (H + G) * D + G * V
    x = _randn(n, x_off + channels + gate_cols, seed=seed, dtype=dtype)
    return x, _randn(channels, seed=seed + 1), _randn(channels, taps, seed=seed + 2, scale=0.6), channels


def _conv_plain(x, bias, conv, x_off, channels):
    u = x[:, x_off:x_off + channels].double().cpu() + bias.double().cpu()
    return plain.short_conv(u, conv.double().cpu())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,V,taps,dims,layout,x_off", [
    (6, 2, 20, 12, 3, 12, "half", 0), (2, 2, 16, 28, 4, 16, "pairs", 5), (8, 2, 128, 128, 2, 64, "half", 16),
    (1, 1, 9, 5, 1, 8, "half", 3), (3, 1, 64, 33, 6, 2, "pairs", 0), (4, 4, 64, 64, 5, 64, "half", 8), (2, 1, 8, 8, 16, 4, "half", 0)])
def test_convolution_turn_and_cache_write_whatever_the_cut(dtype, H, G, D, V, taps, dims, layout, x_off):
    """Whole, token by token, and in portions of one token and more: the same q, keys and values as the plain functions
    on the whole sequence, however the step borders fall; the slot in use is the one the request holds, others keep
    what they had (NaN), a row that is not to be cached is not."""
    ops = _ops()
    T, page = 41, 8
    x, bias, conv, channels = _conv_case(dtype, T, H, G, D, V, taps, 7, x_off, seed=D + taps)
    rotation = gu.rot(dims, 300.0, (4.0, 1.0, 8.0, 64))
    freq = plain.frequencies(rotation).float().cuda()
    y = _conv_plain(x, bias, conv, x_off, channels)
    q = plain.turn(y[:, :H * D].view(T, H, D), rotation, layout)
    k = plain.turn(y[:, H * D:(H + G) * D].view(T, G, D), rotation, layout)
    v = y[:, (H + G) * D:].view(T, G, V)
    tail, floats = 4, 4 + (taps - 1) * channels
    order = torch.randperm(T // page + 3, generator=torch.Generator().manual_seed(1))
    slots = torch.tensor([int(order[t // page]) * page + t % page for t in range(T)], dtype=torch.int32)
    slots[7] = -1
    sizes = dict(num_heads=H, num_kv_heads=G, head_dim=D, v_dim=V, taps=taps, rotary_dims=dims, layout=layout)
    for cuts, slot in (((T,), 2), ((1,) * T, 0), ((7, 2, 1, 13, 2, 1, 1, 12, 2), 1)):
        k_cache, v_cache = (torch.zeros(T // page + 3, G, page, w, dtype=dtype, device="cuda") for w in (D, V))
        state = torch.full((3, floats), float("nan"), device="cuda")
        state[slot] = 0.0
        got, p = [], 0
        status = torch.zeros(1, dtype=torch.int32, device="cuda")
        for n in cuts:
            got.append(ops.conv_rotary_prep(
                x[p:p + n].contiguous(), conv, torch.arange(p, p + n, dtype=torch.int32, device="cuda"), slots[p:p + n].cuda(),
                freq, k_cache, v_cache, state, _i32([0, n]), _i32([slot]), bias=bias, x_off=x_off, tail_off=tail,
                status=status, **sizes))
            p += n
        assert int(status) == 0
        torch.testing.assert_close(torch.cat(got).double().cpu().view(T, H, D), q, **TURNED[dtype])
        for t in range(T):
            at = int(slots[t])
            if at >= 0:
                torch.testing.assert_close(k_cache[at // page, :, at % page].double().cpu(), k[t], **TURNED[dtype])
                torch.testing.assert_close(v_cache[at // page, :, at % page].double().cpu(), v[t], **TOL[dtype])
        used = set(slots.tolist())
        for at in range(k_cache.shape[0] * page):
            if at not in used:
                assert float(k_cache[at // page, :, at % page].abs().max()) == 0.0
        # what the slot holds now: the last inputs, biases included
        if taps > 1:
            u = x[:, x_off:x_off + channels].double().cpu() + bias.double().cpu()
            torch.testing.assert_close(state[slot, tail:].double().cpu().view(taps - 1, channels), u[T - taps + 1:], atol=1e-5, rtol=1e-5)
            assert bool(state[[s for s in range(3) if s != slot]].isnan().all())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("lens", [[1, 19, 2, 6], [1, 1, 1, 1], [300, 3, 2, 40]])
def test_convolution_in_a_batch_of_unequal_sequences_with_padding(dtype, lens):
    """Sequences that begin inside a block's run of tokens, and a padded one: each as if alone, from the inputs its own
    slot held."""
    ops = _ops()
    H, G, D, V, taps, dims = 4, 2, 24, 16, 4, 24
    channels, n = (H + G) * D + G * V, sum(lens)
    x, bias, conv, _ = _conv_case(dtype, n, H, G, D, V, taps, 0, 0, seed=5)
    freq = plain.frequencies(gu.rot(dims, 100.0)).float().cuda()
    slots, before = [3, 0, 2, -1], _randn(5, (taps - 1) * channels, seed=9)
    state, cu = before.clone(), [0]
    for k in lens:
        cu.append(cu[-1] + k)
    page = 16
    k_cache, v_cache = (torch.zeros(n // page + 2, G, page, w, dtype=dtype, device="cuda") for w in (D, V))
    positions = torch.zeros(n, dtype=torch.int32, device="cuda")        # no turn: it was looked at above
    at = torch.arange(n, dtype=torch.int32, device="cuda")
    at[cu[3]:] = -1
    got = ops.conv_rotary_prep(x, conv, positions, at, freq, k_cache, v_cache, state, _i32(cu), _i32(slots), bias=bias,
                               num_heads=H, num_kv_heads=G, head_dim=D, v_dim=V, taps=taps, rotary_dims=dims, layout="half")
    for i in range(3):
        past = before[slots[i]].double().cpu().view(taps - 1, channels)
        u = torch.cat((past, x[cu[i]:cu[i + 1]].double().cpu() + bias.double().cpu()))
        y = plain.short_conv(u, conv.double().cpu())[taps - 1:]
        torch.testing.assert_close(got[cu[i]:cu[i + 1]].double().cpu(), y[:, :H * D], **TOL[dtype])
        rows = k_cache.transpose(1, 2).reshape(-1, G * D)[cu[i]:cu[i + 1]]
        torch.testing.assert_close(rows.double().cpu(), y[:, H * D:(H + G) * D], **TOL[dtype])
        rows = v_cache.transpose(1, 2).reshape(-1, G * V)[cu[i]:cu[i + 1]]
        torch.testing.assert_close(rows.double().cpu(), y[:, (H + G) * D:], **TOL[dtype])
        torch.testing.assert_close(state[slots[i]].double().cpu().view(taps - 1, channels), u[-(taps - 1):], atol=1e-5, rtol=1e-5)
    assert torch.equal(state[1], before[1]) and torch.equal(state[4], before[4])
    assert float(k_cache.transpose(1, 2).reshape(-1, G * D)[cu[3]:].abs().max()) == 0.0


def test_a_cache_slot_outside_the_pool_sets_the_status():
    ops = _ops()
    x, bias, conv, _ = _conv_case(torch.float32, 2, 1, 1, 8, 8, 2, 0, 0, seed=1)
    caches = [torch.zeros(2, 1, 4, 8, device="cuda") for _ in range(2)]
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    ops.conv_rotary_prep(x, conv, _i32([0, 1]), _i32([0, 8]), torch.ones(4, device="cuda"), *caches, torch.zeros(1, 24, device="cuda"),
                         _i32([0, 2]), _i32([0]), num_heads=1, num_kv_heads=1, head_dim=8, v_dim=8, taps=2, rotary_dims=8,
                         layout="half", bias=bias, status=status)
    assert int(status) != 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,width,gate_off,extra,out_off", [(5, 64, 8, 8, 16), (3, 33, 5, 2, 7), (300, 512, 128, 0, 0), (1, 7, 0, 0, 3)])
def test_gates_and_activations_of_columns(dtype, n, width, gate_off, extra, out_off):
    """Written into columns of a wider matrix whose other columns stay as they are; 16-byte accesses and not."""
    ops = _ops()
    values, x = _randn(n, width, seed=1, dtype=dtype), _randn(n, gate_off + width + extra, seed=2, dtype=dtype)
    want = values.double().cpu() * torch.sigmoid(x[:, gate_off:gate_off + width].double().cpu()) * 0.7
    torch.testing.assert_close(ops.gate_columns(values, x, gate_off, factor=0.7).double().cpu(), want, **TOL[dtype])
    out = torch.full((n, out_off + width + 3), 5.0, dtype=dtype, device="cuda")
    ops.gate_columns(values, x, gate_off, factor=0.7, out=out, out_off=out_off)
    torch.testing.assert_close(out[:, out_off:out_off + width].double().cpu(), want, **TOL[dtype])
    assert bool((out[:, :out_off] == 5).all()) and bool((out[:, out_off + width:] == 5).all())
    z = x[:, gate_off:gate_off + width].double().cpu()
    for kind, want in (("gelu_tanh", plain.gelu_tanh(z)), ("gelu", plain.gelu_erf(z)), ("silu", z * torch.sigmoid(z)),
                       ("relu2", torch.relu(z) ** 2)):
        out = torch.full((n, out_off + width + 3), 5.0, dtype=dtype, device="cuda")
        ops.activation_columns(x, gate_off, width, kind, out=out, out_off=out_off)
        torch.testing.assert_close(out[:, out_off:out_off + width].double().cpu(), want, **TOL[dtype])
        assert bool((out[:, :out_off] == 5).all()) and bool((out[:, out_off + width:] == 5).all())
        torch.testing.assert_close(ops.activation(x, kind)[:, gate_off:gate_off + width].double().cpu(), want, **TOL[dtype])


# ----------------------------------------------------------------------------- a decay per channel


def _delta_case(dtype, T, H, G, D, V, taps, x_off, seed):
    channels = 2 * G * D + H * V
    c = dict(x=_randn(T, x_off + channels + H + 3, seed=seed, dtype=dtype), mid=_randn(T, 2 + H * D + H * V, seed=seed + 1),
             conv=_randn(channels, taps, seed=seed + 2, scale=0.7), rate=_randn(H, seed=seed + 3) - 2.0,
             bias=_randn(H * D, seed=seed + 4), norm=1.0 + 0.2 * _randn(V, seed=seed + 5))
    return c, channels


def _delta_plain(c, rows, H, G, D, V, x_off, channels, eps, factor):
    x, mid = c["x"][rows].double().cpu(), c["mid"][rows].double().cpu()
    y = plain.short_conv(x[:, x_off:x_off + channels], c["conv"].double().cpu())
    y = y * torch.sigmoid(y)
    n = y.shape[0]
    unit = lambda z: z / torch.sqrt((z * z).sum(-1, keepdim=True) + 1e-6)      # noqa: E731
    q, k = unit(y[:, :G * D].view(n, G, D)) * D ** -0.5, unit(y[:, G * D:2 * G * D].view(n, G, D))
    v = y[:, 2 * G * D:].view(n, H, V)
    beta = torch.sigmoid(x[:, x_off + channels:x_off + channels + H])
    step = plain.softplus(mid[:, 2:2 + H * D] + c["bias"].double().cpu()).view(n, H, D)
    decay = torch.exp(-torch.exp(c["rate"].double().cpu())[None, :, None] * step)
    gate = torch.sigmoid(mid[:, 2 + H * D:]).view(n, H, V)
    heads = [plain.rms_unit(plain.channel_delta_rule(q[:, h // (H // G)], k[:, h // (H // G)], v[:, h], beta[:, h], decay[:, h]), eps)
             * c["norm"].double().cpu() * gate[:, h] * factor for h in range(H)]
    return torch.cat(heads, dim=-1)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,V,taps,x_off", [(4, 2, 12, 20, 2, 8), (3, 1, 64, 32, 4, 0), (2, 2, 128, 128, 3, 5), (2, 1, 256, 40, 1, 0),
                                                (2, 2, 130, 16, 2, 3), (1, 1, 3, 1, 5, 0), (4, 1, 40, 256, 2, 1), (6, 3, 33, 7, 4, 0)])
def test_delta_rule_with_a_decay_per_channel_whatever_the_cut(dtype, H, G, D, V, taps, x_off):
    """Prompts, token by token and portions against the plain recurrence; the state is a view into wider rows, as beside
    another mixer; the result goes into columns of a wider matrix; the memory after the last token does not depend on
    the cut."""
    ops = _ops()
    T, eps, factor = 45, 1e-5, 0.6
    c, channels = _delta_case(dtype, T, H, G, D, V, taps, x_off, seed=20 + D)
    want = _delta_plain(c, slice(0, T), H, G, D, V, x_off, channels, eps, factor)
    sizes = dict(num_heads=H, num_kv_heads=G, head_dim=D, v_dim=V, taps=taps)
    floats = ops.delta_state_floats(H, G, D, V, taps)[1]
    tol = dict(atol=5e-5, rtol=5e-4) if dtype == torch.float32 else dict(atol=3e-2, rtol=3e-2)
    memories = []
    for cuts, slot in (((T,), 2), ((1,) * T, 0), ((7, 2, 1, 13, 2, 1, 1, 16, 2), 1)):
        whole = torch.full((3, floats + 12), float("nan"), device="cuda")
        state = whole[:, 8:8 + floats]
        state[slot] = 0.0
        got, p = [], 0
        for n in cuts:
            x, mid = c["x"][p:p + n].contiguous(), c["mid"][p:p + n].contiguous()
            more = dict(channel_decay=True, x_off=x_off)
            qkv, coef = ops.delta_prep(x, c["conv"], c["rate"], c["bias"], state, _i32([0, n]), _i32([slot]), unit_eps=1e-6,
                                       steps=mid, step_off=2, beta_off=x_off + channels, **more, **sizes)
            out = torch.full((n, H * V + 9), 5.0, dtype=dtype, device="cuda")
            ops.delta_scan(qkv, coef, x, c["norm"], state, _i32([0, n]), _i32([slot]), norm_eps=eps, gates=mid,
                           gate_off=2 + H * D, gate="sigmoid", factor=factor, out=out, out_off=4, **more, **sizes)
            assert bool((out[:, :4] == 5).all()) and bool((out[:, 4 + H * V:] == 5).all())
            got.append(out[:, 4:4 + H * V])
            p += n
        torch.testing.assert_close(torch.cat(got).double().cpu(), want, **tol)
        memories.append(state[slot].clone())
        assert bool(whole[:, :8].isnan().all()) and bool(whole[:, 8 + floats:].isnan().all())
    for m in memories[1:]:
        torch.testing.assert_close(m, memories[0], atol=3e-5, rtol=1e-4)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("lens", [[1, 19, 6, 4], [1, 5, 1, 1], [1, 1, 1, 1]])
def test_channel_decays_in_a_batch_of_unequal_sequences_with_padding(dtype, lens):
    ops = _ops()
    H, G, D, V, taps, eps = 4, 2, 32, 16, 3, 1e-5
    cu = [0]
    for n in lens:
        cu.append(cu[-1] + n)
    c, channels = _delta_case(dtype, cu[-1], H, G, D, V, taps, 0, seed=30)
    sizes = dict(num_heads=H, num_kv_heads=G, head_dim=D, v_dim=V, taps=taps)
    slots = [3, 0, 2, -1]
    state = torch.zeros(5, ops.delta_state_floats(H, G, D, V, taps)[1], device="cuda")
    state[1], state[4] = 5.0, -3.0
    qkv, coef = ops.delta_prep(c["x"], c["conv"], c["rate"], c["bias"], state, _i32(cu), _i32(slots), unit_eps=1e-6,
                               steps=c["mid"], step_off=2, beta_off=channels, channel_decay=True, **sizes)
    out = ops.delta_scan(qkv, coef, c["x"], c["norm"], state, _i32(cu), _i32(slots), norm_eps=eps, gates=c["mid"],
                         gate_off=2 + H * D, gate="sigmoid", channel_decay=True, **sizes)
    tol = dict(atol=5e-5, rtol=5e-4) if dtype == torch.float32 else dict(atol=3e-2, rtol=3e-2)
    for i in range(3):
        want = _delta_plain(c, slice(cu[i], cu[i + 1]), H, G, D, V, 0, channels, eps, 1.0)
        torch.testing.assert_close(out[cu[i]:cu[i + 1]].double().cpu(), want, **tol)
    assert float(out[cu[3]:].float().abs().max()) == 0.0
    assert bool((state[1] == 5.0).all()) and bool((state[4] == -3.0).all())


def test_channels_fade_by_their_own_decays():
    """Two values written at the start under keys in different channels, 600 tokens of nothing, then a query for each:
    the channel that does not fade returns its value whole, the other returns it faded by exactly its decay's power."""
    ops = _ops()
    H = G = 1
    D, V, T = 64, 32, 604
    sizes = dict(num_heads=H, num_kv_heads=G, head_dim=D, v_dim=V, taps=1)
    q, k, v = torch.zeros(T, D, device="cuda"), torch.zeros(T, D, device="cuda"), _randn(T, V, seed=1)
    k[0, 5], k[1, 40] = 1.0, 1.0
    q[-2, 5], q[-1, 40] = 1.0, 1.0
    k[2:, 63] = 1.0                                   # everything in between goes to a third channel
    decay = torch.full((T, D), 0.9, device="cuda")
    decay[:, 5], decay[:, 40] = 1.0, 0.995
    coef = torch.cat((torch.ones(T, 1, device="cuda"), decay), dim=1).contiguous()
    qkv = torch.cat((q, k, v), dim=1).contiguous()
    x, gates = torch.zeros(T, 2 * D + V, device="cuda"), torch.full((T, V), 40.0, device="cuda")
    for cuts in ((T,), (300, 1, 1, T - 302)):
        state, p = torch.zeros(2, ops.delta_state_floats(H, G, D, V, 1)[1], device="cuda"), 0
        for n in cuts:
            out = ops.delta_scan(qkv[p:p + n].contiguous(), coef[p:p + n].contiguous(), x[p:p + n].contiguous(),
                                 torch.ones(V, device="cuda"), state, _i32([0, n]), _i32([1]), norm_eps=1e-12,
                                 gates=gates[p:p + n].contiguous(), gate="sigmoid", channel_decay=True, **sizes)
            p += n
        for row, raw in ((-2, v[0].double()), (-1, v[1].double() * 0.995 ** (T - 2))):
            torch.testing.assert_close(out[row].double(), plain.rms_unit(raw, 1e-12), atol=2e-4, rtol=2e-4)


@pytest.mark.parametrize("n", [1, 7, 40, 200])
@pytest.mark.parametrize("k,features", [(64, 96), (72, 200), (128, 1024), (24, 40)])
def test_a_product_over_columns_of_a_wider_matrix(n, k, features):
    ops = _ops()
    wide, w = _randn(n, k + 24, seed=n, dtype=torch.bfloat16), _randn(features, k, seed=k, dtype=torch.bfloat16, scale=k ** -0.5)
    for off in (0, 8, 16):
        got = ops.linear(wide[:, off:off + k], w, out_dtype=torch.float32)
        want = wide[:, off:off + k].double() @ w.double().T
        torch.testing.assert_close(got.double(), want, atol=2e-5, rtol=1e-4)


# ----------------------------------------------------------------------------- experts without a gate


@pytest.mark.parametrize("tokens,experts,top", [(1, 5, 2), (7, 3, 3), (300, 12, 1), (64, 40, 6)])
def test_routing_by_the_softmax_over_the_chosen_logits(tokens, experts, top):
    ops = _ops()
    logits, bias = 3.0 * _randn(tokens, experts, seed=tokens), _randn(experts, seed=experts)
    logits[0] -= 300.0                                 # nothing under- or overflows
    chosen, weights = ops.moe_route(logits, None, top=top, groups=1, keep_groups=1, group_top=1, scale=1.0, weight_eps=0.0,
                                    score="softmax", bias=bias)
    lead: list = []
    want, w = plain.route((logits + bias).double().cpu(), top, lead)
    clear = lead[0] > 1e-4
    assert torch.equal(chosen.cpu().long()[clear], want[clear])
    torch.testing.assert_close(weights.double().cpu()[clear], w[clear], atol=1e-6, rtol=1e-4)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("form", ["auto", "plain", "mma", "few"])
@pytest.mark.parametrize("tokens,width,ff,experts,top", [(1, 72, 24, 5, 2), (9, 64, 96, 3, 3), (90, 256, 200, 6, 2), (600, 128, 72, 2, 1),
                                                         (40, 63, 15, 4, 2)])
def test_experts_without_a_gate(dtype, form, tokens, width, ff, experts, top):
    ops = _ops()
    if form in ("mma", "few") and (dtype == torch.float32 or width % 8):
        return
    x = _randn(tokens, width, seed=tokens, dtype=dtype)
    w_up = _randn(experts, ff, width, seed=ff, dtype=dtype, scale=width ** -0.5)
    g = torch.Generator().manual_seed(tokens)
    chosen = torch.stack([torch.randperm(experts, generator=g)[:top] for _ in range(tokens)]).to(torch.int32)
    order, offsets = ops.moe_sort(chosen.cuda(), experts)
    for activation, fn in (("gelu", plain.gelu_erf), ("gelu_tanh", plain.gelu_tanh)):
        act = ops.moe_up(x, w_up, order, offsets, top=top, activation=activation, kernel=form)
        e_of = chosen.reshape(-1)[order.cpu().long()].long()
        want = fn(torch.einsum("rk,rfk->rf", x.double().cpu()[order.cpu().long() // top], w_up.double().cpu()[e_of]))
        torch.testing.assert_close(act.double().cpu(), want, **TOL[dtype])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens", [1, 5, 90, 400])
@pytest.mark.parametrize("width,ff,experts,top", [(72, 24, 5, 2), (63, 15, 3, 1), (256, 128, 6, 4), (48, 16, 4, 4)])
def test_the_mixture_as_a_layer_uses_it(dtype, tokens, width, ff, experts, top):
    from ampere_kv_engine_b200.models.gosizen import _feed_forward
    from ampere_kv_engine_b200.parts import routed_experts  # noqa: F401  (registers the kind)
    from ampere_kv_engine_b200.parts.base import FEED_FORWARDS, build_part
    g = torch.Generator().manual_seed(tokens + width)
    mlp = gu.moe(experts, top, ff)
    part = build_part(FEED_FORWARDS, _feed_forward(mlp, "mlp"), hidden_size=width, dtype=dtype, device=torch.device("cuda"))
    t = {name: (torch.randn(ps.shape, generator=g) * (0.5 if ps.kind == "vector" else 2.0 * ps.shape[-1] ** -0.5))
         .to(torch.bfloat16).float() for name, ps in part.param_specs().items()}
    part.load({k: v.cuda().to(torch.float32 if k == "router.b" else dtype) for k, v in t.items()})
    w = {f"mlp.{k}": v.double() for k, v in t.items()}
    x = torch.randn((6 * tokens, width), generator=g).to(torch.bfloat16).float()
    _, lead = None, []
    plain.route(x.double() @ w["mlp.router"].T + w["mlp.router.b"], top, lead)
    x = x[lead[0] > 3e-2][:tokens]                     # tokens whose choice is no close call

    class Ctx:
        status = None
    want = plain.experts_mixture(x.double(), w, "mlp", mlp)
    got = part.forward(x.cuda().to(dtype), Ctx())
    # up to four experts' activations, each rounded once, in a sum of unit size
    tol = TOL[dtype] if dtype == torch.float32 else dict(atol=4e-2, rtol=2e-2)
    torch.testing.assert_close(got.double().cpu(), want, **tol)
    # summed into the stream by the kernel that adds up a layer's branches
    hidden = torch.randn((x.shape[0], width), generator=g)
    other = torch.randn((x.shape[0], width), generator=g).to(dtype)
    stream = hidden.cuda()
    copy = _ops().stream_sum(stream, [other.cuda(), part.forward(x.cuda().to(dtype), Ctx(), defer_sum=True)], copy_dtype=dtype)
    torch.testing.assert_close(stream.double().cpu(), hidden.double() + other.double() + want, **tol)
    torch.testing.assert_close(copy, stream.to(dtype), atol=0, rtol=0)


# ----------------------------------------------------------------------------- the stream itself


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,width", [(1, 63), (9, 72), (300, 256), (5, 1000)])
def test_updates_of_the_stream(dtype, n, width):
    ops = _ops()
    hidden, start, row = _randn(n, width, seed=1), _randn(n, width, seed=2), _randn(width, seed=3)
    both = ops.stream_concat(hidden, start, dtype)
    torch.testing.assert_close(both, torch.cat((hidden, start), 1).to(dtype), atol=0, rtol=0)
    stream = hidden.clone()
    ops.stream_row_add(stream, row)
    torch.testing.assert_close(stream, hidden + row, atol=0, rtol=0)
    a, b, c = _randn(n, width, seed=4, dtype=dtype), _randn(n, width, seed=5), _randn(n, width, seed=6, dtype=dtype)
    stream = hidden.clone()
    copy = ops.stream_sum(stream, [a, None, b, c], copy_dtype=dtype)
    torch.testing.assert_close(stream, hidden + a.float() + b + c.float(), atol=2e-6, rtol=2e-6)
    torch.testing.assert_close(copy, stream.to(dtype), atol=0, rtol=0)
    assert (copy is stream) == (dtype == torch.float32)
    # a branch that joins through its norm, and nothing else
    weight = 1.0 + 0.2 * _randn(width, seed=7)
    stream = hidden.clone()
    assert ops.stream_sum(stream, [ops.NormedBranch(b, weight, 1e-5)]) is None
    torch.testing.assert_close(stream.double(), hidden.double() + plain.rms_unit(b.double(), 1e-5) * weight.double(), atol=2e-5, rtol=2e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,dim,off,stride", [(1, 5, 3, 11), (70, 64, 128, 512), (6, 300, 300, 900)])
def test_the_tokens_own_gate(dtype, n, dim, off, stride):
    """Ids the host has not read stand for tokens the last step chose; an id outside the table is reported."""
    ops = _ops()
    z, table = 2.0 * _randn(n, dim, seed=1), _randn(37, stride, seed=2, dtype=dtype)
    z = z.to(dtype)
    ids = torch.randint(0, 37, (n,), generator=_gen(3), device="cuda").to(torch.int32)
    sampled = _i32([36, 4])
    given = ids.clone()
    given[0] = -2
    real = ids.clone()
    real[0] = 4
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    got = ops.token_gate(z, given, table, off, sampled=sampled, status=status)
    want = plain.gelu_tanh(z.double()) * table.double()[real.long(), off:off + dim]
    torch.testing.assert_close(got.double(), want, **TOL[dtype])
    assert int(status) == 0
    given[0] = 37
    ops.token_gate(z, given, table, off, status=status)
    assert int(status) != 0


def test_rescaled_frequencies_and_gelu_limits():
    ops = _ops()
    z = torch.tensor([[-40.0, -1.0, 0.0, 1e-3, 3.0, 40.0]], device="cuda")
    torch.testing.assert_close(ops.activation(z, "gelu").double(), plain.gelu_erf(z.double()), atol=1e-6, rtol=1e-6)
    assert math.isfinite(float(ops.activation(z, "gelu_tanh").sum()))
