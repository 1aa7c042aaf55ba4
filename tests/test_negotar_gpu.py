"""The Negotar decoder in the engine against the plain float64 implementation (``plain_negotar``): each mechanism alone (as a kernel
and in a model of nothing else), the stream after every layer, whole prompts against token-by-token decoding, portions down to two
tokens, batches of unequal requests on pages and state slots that are used again, a far past that shows through sharp attention
or a slow memory, the first tokens, long decoding, sizes unlike one another, and greedy generation through the engine's scheduler."""

import copy

import pytest
import torch

import negotar_cases as cases
import plain_negotar as plain
import trace_modes as modes
from helpers import compare_logits, seeded_tokens, write_model_dir

pytestmark = pytest.mark.gpu
STORED = {"float32": torch.float32, "bfloat16": torch.bfloat16}
F64 = torch.float64


@pytest.fixture(scope="module")
def gpu():
    if not torch.cuda.is_available():
        pytest.skip("needs a CUDA device")


def close(got, want, tol):
    got, want = got.double().cpu(), want.double().cpu()
    assert torch.isfinite(got).all()
    scale = float(want.abs().max())
    err = float((got - want).abs().max())
    assert err <= tol * scale, f"max abs error {err:.3e} against scale {scale:.3e}"


BF16_BOUND = (0.998, 0.06)          # cosine floor and largest error of a row relative to its spread


def compare_rows(got, want, dtype):
    """float32: the helpers' bound (cosine and largest difference). bfloat16: what the rounding of activations leaves of a
    row, a few per cent of its spread for these small random models; a wrong key or memory changes a row outright, and the
    float32 runs of the same cuttings hold the tight bound."""
    if dtype == "float32":
        return compare_logits(got, want, dtype)
    a, b = got.double().reshape(-1), want.double().reshape(-1)
    if not torch.isfinite(a).all():
        return False, "non-finite logits"
    cos = float(torch.nn.functional.cosine_similarity(a, b, dim=0))
    rel = float((a - b).norm() / (b - b.mean()).norm())
    return cos >= BF16_BOUND[0] and rel <= BF16_BOUND[1], f"cosine {cos:.6f}, error {rel:.3f} of the row's spread"


def replay(folder, dtype, steps, want, page, slots, label, min_ok=1.0):
    """Runs the steps through a fresh session and compares every wanted row; pages and state slots start as NaN."""
    from stride_b200.engine.trace import TraceSession
    session = TraceSession(folder, dtype, max_tokens=modes.peak_tokens(steps), block_size=page, max_requests=slots)
    for t in list(session.device_cache.pages) + list(session.device_cache.states.values()):
        t.fill_(float("nan"))
    rows = modes.expected_rows(steps)
    bad, total, first = 0, 0, None
    for s in steps:
        out = session.run_step(s)
        for r, (rid, pos) in enumerate(rows[s["step"]]):
            ok, msg = compare_rows(out[r:r + 1], want[rid][pos:pos + 1], dtype)
            total += 1
            if not ok:
                bad += 1
                first = first or f"{label}: step {s['step']}, request {rid!r}, position {pos}: {msg}"
    allowed = 0 if min_ok == 1.0 else max(1, int((1.0 - min_ok) * total))      # a row that blows rounding up may fall into a short run, too
    assert total and bad <= allowed, f"{bad} of {total} rows differ; first: {first}"
    stats = session.cache.stats()
    assert stats["live"] == 0 and session.cache.free_slots == session.cache.slot_capacity
    return session


def write(tmp_models, name, cfg, state, dtype):
    """The model folder and the weights as the engine will see them, in float64."""
    folder = write_model_dir(str(tmp_models / f"negotar_{name}_{dtype}"), cfg, state, STORED[dtype])
    return folder, {k: v.to(STORED[dtype]).double() for k, v in state.items()}


def model_case(tmp_models, name, cfg, state, dtype, seed, lengths):
    folder, state = write(tmp_models, name, cfg, state, dtype)
    requests = {f"r{i}": seeded_tokens(n, cfg["vocab"], 50 * seed + i) for i, n in enumerate(lengths)}
    return folder, requests, {rid: plain.forward(cfg, state, toks) for rid, toks in requests.items()}


def dev(values, dtype=torch.int32):
    return torch.tensor(values, dtype=dtype, device="cuda")


# ------------------------------------------------------------------------------------------------- kernels alone
def state_space(H, G, N, P, taps, g):
    """Weights as the kernels take them, and in float64 for the plain functions."""
    from stride_b200.csrc import ops
    channels = H * P + 2 * G * N
    w = {"conv": torch.randn(channels, taps, generator=g) * 0.6, "bias": torch.randn(channels, generator=g) * 0.4,
         "dt_bias": torch.randn(H, generator=g), "a_log": torch.randn(H, generator=g), "skip": torch.randn(H, generator=g)}
    c = {k: v.cuda() for k, v in w.items()}
    shape = ops.SsmShape(H, G, N, P, taps, c["dt_bias"], c["a_log"], c["skip"], w["conv"].t().contiguous().cuda(), c["bias"])
    return shape, {k: v.double() for k, v in w.items()}


def plain_state_space(u, raw, S, w, H, G, N, P):
    """y [T, H * P] and the memories afterwards, from x, B, C as the kernels read them and memories S [H, N, P] before."""
    T, S = u.shape[0], S.clone()
    x = u[:, :H * P].reshape(T, H, P)
    B, C = u[:, H * P:H * P + G * N].reshape(T, G, N), u[:, H * P + G * N:H * P + 2 * G * N].reshape(T, G, N)
    d = plain.step_size(raw, w["dt_bias"])
    y = torch.zeros(T, H, P, dtype=F64)
    for h in range(H):
        g = h // (H // G)
        keep = torch.exp(-torch.exp(w["a_log"][h]) * d[:, h])
        for t in range(T):
            S[h] = keep[t] * S[h] + d[t, h] * torch.outer(B[t, g], x[t, h])
            y[t, h] = S[h].T @ C[t, g] + w["skip"][h] * x[t, h]
    return y.reshape(T, H * P), S


SIZES = [(6, 3, 12, 20, 3), (1, 1, 16, 8, 1), (4, 2, 128, 64, 4), (2, 1, 40, 96, 5), (3, 3, 10, 6, 7), (2, 2, 256, 136, 2), (3, 1, 6, 10, 4), (2, 1, 64, 32, 16)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("wide_input", [False, True])
@pytest.mark.parametrize("H,G,N,P,taps", SIZES)
def test_convolution_and_its_ring(gpu, dtype, wide_input, H, G, N, P, taps):
    """A start, a portion deep inside a request, one right behind its first token, a single token, and a padded row, against the plain
    convolution over each request's whole past; then the rings. ``wide_input``: float32 inputs in a bfloat16 model."""
    from stride_b200.csrc import ops
    if wide_input and dtype == "float32":
        pytest.skip("float32 models have float32 inputs anyway")
    g = torch.Generator().manual_seed(N + P + taps)
    shape, w = state_space(H, G, N, P, taps, g)
    C, off = shape.channels, 8
    past, new = [0, 29, 1, 5, 3], [21, 6, 2, 1, 40]
    in_type = torch.float32 if wide_input else STORED[dtype]
    histories = [torch.randn(p + n, C, generator=g).to(in_type) for p, n in zip(past, new)]
    rows = sum(new) + 1
    proj = torch.full((rows, off + -(-C // 8) * 8), float("nan"), dtype=in_type)
    slots, wide = [3, 1, 0, 4, 2], torch.full((6, 4 + shape.state_floats() + 4), float("nan"))
    positions, seq_of, q_start, at = [], [], [], 0
    for s, (p, n) in enumerate(zip(past, new)):
        proj[at:at + n, off:off + C] = histories[s][p:]
        q_start.append(at)
        positions += list(range(p, p + n))
        seq_of += [s] * n
        at += n
        if taps > 1:
            ring = wide[slots[s], 4 + shape.ring_off:4 + shape.state_floats()].view(taps, C)
            for back in range(1, min(p, taps - 1) + 1):
                ring[(p - back) % taps] = histories[s][p - back].float()
    state = wide.cuda()[:, 4:4 + shape.state_floats()]
    out = torch.full((rows, -(-C // 8) * 8), float("nan"), dtype=STORED[dtype], device="cuda")
    where = (dev(q_start), dev(positions + [0]), dev(slots))
    ops.ssm_conv(shape, proj.cuda(), off, state, dev(seq_of + [-1]), *where, out)
    for s, (p, n) in enumerate(zip(past, new)):
        want = plain.silu(plain.short_convolution(histories[s].double(), w["conv"], w["bias"]))[p:]
        close(out[q_start[s]:q_start[s] + n, :C], want, 2e-6 if dtype == "float32" else 6e-3)
    ops.ssm_tail(shape, proj.cuda(), off, state, dev(q_start + [0]), dev(new + [0]), where[1], dev(slots + [0]), 6)
    for s, (p, n) in enumerate(zip(past, new)):
        for pos in range(max(0, p + n - taps + 1), p + n):
            ring = state[slots[s], shape.ring_off:].cpu()[:taps * C].view(taps, C)
            assert torch.equal(ring[pos % taps], histories[s][pos].float()), (s, pos)


@pytest.mark.parametrize("form", ["chain", "chunks"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,N,P,taps", SIZES)
def test_the_memory_over_portions(gpu, dtype, form, H, G, N, P, taps):
    """Requests with a past and fresh ones: portions over several chunks, of exactly one, of one token more, short ones; decays that
    forget within a token and ones that hardly forget. Against the recurrence token by token in float64 on the same inputs."""
    from stride_b200.csrc import ops
    if form == "chunks" and dtype == "float32":
        pytest.skip("float32 models keep the chain")
    g = torch.Generator().manual_seed(H * N + P)
    shape, w = state_space(H, G, N, P, taps, g)
    new = [300, 128, 129, 3, 17] if N * P * H < 40000 else [140, 5]
    rows, C, off = sum(new), shape.channels, 8
    u = torch.randn(rows, -(-C // 8) * 8, generator=g).to(STORED[dtype])
    raw = torch.randn(rows, H + 3, generator=g) * 2.0
    raw[:, 2] += 4.0                         # the first head: large steps, nearly all is forgotten at every token
    proj = torch.randn(rows, off + -(-C // 8) * 8, generator=g).to(STORED[dtype])
    wide = torch.full((len(new) + 2, 4 + shape.state_floats() + 4), float("nan"))
    S0 = torch.randn(len(new) + 1, H, N, P, generator=g)
    S0[1] = 0.0
    for s in range(len(new)):
        wide[s + 1, 4:4 + shape.state_floats()] = 0.0
        wide[s + 1, 4:4 + H * N * P] = S0[s + 1].reshape(-1)
    device = wide.cuda()
    state = device[:, 4:4 + shape.state_floats()]
    starts = [sum(new[:s]) for s in range(len(new))]
    positions = [1000 + i for n in new for i in range(n)]
    q_start, q_len, slots, n_seq = dev(starts + [0]), dev(new + [0]), dev(list(range(1, len(new) + 1)) + [0]), len(new) + 1
    y = torch.full((rows, H * P), float("nan"), device="cuda")
    if form == "chain":
        ops.ssm_scan(shape, u.cuda(), raw.cuda(), 2, y, state, q_start, q_len, slots, n_seq)
    else:
        scratch = torch.full((ops.ssm_chunks_scratch_floats(shape, n_seq, max(new)),), float("nan"), device="cuda")
        ops.ssm_chunks(shape, u.cuda(), raw.cuda(), 2, y, state, proj.cuda(), off, q_start, q_len, dev(positions), slots, n_seq, max(new), scratch)
    for s, n in enumerate(new):
        part = slice(starts[s], starts[s] + n)
        want, S = plain_state_space(u[part].double(), raw[part, 2:2 + H].double(), S0[s + 1].double(), w, H, G, N, P)
        close(y[part], want, 1e-5 if form == "chain" else 4e-5)
        close(state[s + 1, :H * N * P], S.reshape(-1), 1e-5 if form == "chain" else 4e-5)
        if form == "chunks" and taps > 1:           # the rings have moved with them
            ring = state[s + 1, shape.ring_off:].cpu()[:taps * C].view(taps, C)
            for i in range(max(0, n - taps + 1), n):
                assert torch.equal(ring[(1000 + i) % taps], proj[starts[s] + i, off:off + C].float())
    assert torch.isnan(device[0]).all() and torch.isnan(device[:, :4]).all() and torch.isnan(device[:, 4 + shape.state_floats():]).all()


@pytest.mark.parametrize("u_type", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,N,P,taps", [s for s in SIZES if s[3] % 4 == 0] + [(6, 2, 200, 44, 3)])
def test_a_single_token_of_every_request(gpu, u_type, H, G, N, P, taps):
    """Convolution, memory and ring in one kernel: a fresh request, two with a past shorter and longer than the taps, a slot without a
    request; twice in a row, so that the second token reads what the first one left."""
    from stride_b200.csrc import ops
    g = torch.Generator().manual_seed(H * N + P)
    shape, w = state_space(H, G, N, P, taps, g)
    C, off, past = shape.channels, 8, [0, 1, 37]
    histories = [torch.randn(p + 2, C, generator=g).to(STORED[u_type]) for p in past]
    state = torch.zeros(4, -(-shape.state_floats() // 4) * 4)
    S = torch.randn(3, H, N, P, generator=g)
    S[0] = 0.0
    order = [2, 3, 1]
    for s, slot in enumerate(order):
        state[slot, :H * N * P] = S[s].reshape(-1)
        if taps > 1:
            ring = state[slot, shape.ring_off:shape.state_floats()].view(taps, C)
            for back in range(1, min(past[s], taps - 1) + 1):
                ring[(past[s] - back) % taps] = histories[s][past[s] - back].float()
    state, S = state.cuda(), S.double()
    untouched = state[0].clone()
    assert ops.ssm_step_supported(shape, state)
    for k in range(2):
        proj, raw = torch.randn(4, off + -(-C // 8) * 8, generator=g).to(STORED[u_type]), torch.randn(4, H + 1, generator=g) * 2
        for s in range(3):
            proj[s, off:off + C] = histories[s][past[s] + k]
        y = torch.full((4, H * P), float("nan"), device="cuda")
        ops.ssm_step(shape, proj.cuda(), off, raw.cuda(), 1, y, state, dev([0, 1, 2, 0]), dev([1, 1, 1, 0]), dev([p + k for p in past] + [0]),
                     dev(order + [0]), 4)
        for s, slot in enumerate(order):
            u = plain.silu(plain.short_convolution(histories[s][:past[s] + k + 1].double(), w["conv"], w["bias"]))[-1:]
            want, S[s] = plain_state_space(u, raw[s:s + 1, 1:].double(), S[s], w, H, G, N, P)
            close(y[s:s + 1], want, 1e-5)
            close(state[slot, :H * N * P], S[s].reshape(-1), 1e-5)
        assert torch.isnan(y[3]).all() and torch.equal(state[0], untouched)


@pytest.mark.parametrize("dtype,z_type,tol", [("float32", "float32", 3e-6), ("bfloat16", "float32", 6e-3), ("bfloat16", "bfloat16", 6e-3)])
@pytest.mark.parametrize("width,parts", [(24, 1), (40, 5), (2048, 2), (4096, 1), (9000, 1), (30, 3), (36, 36), (8200, 2)])
def test_gate_before_a_norm_of_parts(gpu, dtype, z_type, tol, width, parts):
    from stride_b200.csrc import ops
    g = torch.Generator().manual_seed(width)
    y, z = torch.randn(5, width, generator=g) * 3, (torch.randn(5, width + 16, generator=g) * 2).to(STORED[z_type])
    w = 1.0 + 0.3 * torch.randn(width, generator=g)
    out = torch.zeros(5, width, dtype=STORED[dtype], device="cuda")
    ops.gated_group_norm(y.cuda(), z.cuda(), 8, w.cuda(), out, parts, 1e-3)
    close(out, plain.gated_group_norm(y.double(), z[:, 8:8 + width].double(), w.double(), parts, 1e-3), tol)


@pytest.mark.parametrize("dtype,tol", [("float32", 3e-6), ("bfloat16", 6e-3)])
@pytest.mark.parametrize("nq,nkv,hd,vd,qd,vdim,rot", [(4, 2, 64, 64, 64, 64, 64), (3, 1, 128, 128, 96, 40, 32), (2, 2, 20, 24, 20, 24, 12), (6, 3, 10, 6, 10, 6, 6),
                                                      (1, 1, 256, 200, 256, 200, 256), (5, 5, 7, 3, 7, 3, 0), (2, 1, 128, 128, 80, 64, 80), (4, 4, 24, 16, 24, 16, 20)])
def test_rotation_norms_and_value_mixing(gpu, dtype, tol, nq, nkv, hd, vd, qd, vdim, rot):
    """Far and first positions, a padded row, heads wider in memory than they are; values kept aside by a first call and mixed into a
    second one's; keys and values at their places in the pages, all other places untouched."""
    from stride_b200.csrc import ops
    g = torch.Generator().manual_seed(nq * hd + vd)
    at, eps, page = [0, 1, 37, 4000, 9], 1e-3, 4
    r = cases.rotation(rot, base=500.0, original=300)
    f = torch.tensor(plain.rotation_frequencies(r), dtype=F64)
    a = torch.arange(4001, dtype=F64)[:, None] * f
    cos, sin = a.cos().float().cuda(), a.sin().float().cuda()
    slots = dev([3, 17, 0, 9, -1])
    first = torch.full((5, nkv * vdim), float("nan"), device="cuda")
    kept = None
    for share in (None, torch.tensor(0.3)):
        q = torch.randn(5, nq, qd, generator=g).to(STORED[dtype])
        k, v = torch.randn(5, nkv, qd, generator=g).to(STORED[dtype]), torch.randn(5, nkv, vdim, generator=g).to(STORED[dtype])
        bq, bk, bv = torch.randn(nq, qd, generator=g), torch.randn(nkv, qd, generator=g), torch.randn(nkv, vdim, generator=g)
        wide = lambda t, n: torch.nn.functional.pad(t, (0, n - t.shape[-1]))
        row = lambda q, k, v: torch.cat([wide(q, hd).reshape(*q.shape[:-2], -1), wide(k, hd).reshape(*k.shape[:-2], -1), wide(v, vd).reshape(*v.shape[:-2], -1)], -1)
        qkv = row(q, k, v).contiguous().cuda()
        k_pages = torch.full((5, nkv, page, hd), 7.0, dtype=STORED[dtype], device="cuda")
        v_pages = torch.full((5, nkv, page, vd), 7.0, dtype=STORED[dtype], device="cuda")
        ops.qkv_rotate_norm(qkv, row(bq, bk, bv).contiguous().cuda(), dev(at), cos, sin, rot, slots, k_pages, v_pages, nq, nkv, hd, vd, qd, vdim, page, eps, first,
                            None if share is None else share.cuda())
        turned = lambda x: torch.stack([plain.rms_unit(plain.rotate(x[i:i + 1].double(), r, p), eps)[0] for i, p in enumerate(at)])
        want_q, want_k = turned(q.double() + bq.double()), turned(k.double() + bk.double())
        want_v = plain.mixed_values(v.double() + bv.double(), kept, 0.3)
        if share is None:
            kept = want_v
            close(first, kept.reshape(5, -1), 1e-6)
        close(qkv[:, :nq * hd].reshape(5, nq, hd), wide(want_q, hd), tol)
        for i, slot in enumerate([3, 17, 0, 9]):
            close(k_pages[slot // page, :, slot % page], wide(want_k[i], hd), tol)
            close(v_pages[slot // page, :, slot % page], wide(want_v[i], vd), tol)
            k_pages[slot // page, :, slot % page] = 7.0
            v_pages[slot // page, :, slot % page] = 7.0
        assert (k_pages == 7.0).all() and (v_pages == 7.0).all()


@pytest.mark.parametrize("dtype,tol", [("float32", 3e-6), ("bfloat16", 1e-2)])
@pytest.mark.parametrize("rows,width,ff,experts,top", [(1, 64, 24, 5, 2), (9, 56, 50, 3, 3), (40, 72, 28, 16, 1), (700, 128, 64, 6, 2), (3, 33, 7, 2, 1), (70, 64, 96, 200, 30),
                                                       (16, 256, 160, 8, 3)])
def test_the_mixture_alone(gpu, dtype, tol, rows, width, ff, experts, top):
    """Scores far from zero and one, so that a weight on an expert's output (or a normalized one) is something else outright. The choice
    is checked on the router's own float32 logits; 700 rows take the tcgen05 products."""
    from stride_b200.config import FeedForwardSpec
    from stride_b200.parts import Runtime, build_part
    g = torch.Generator().manual_seed(rows + ff)
    rt = Runtime("cuda", STORED[dtype], max(rows, 16), 4)
    part = build_part("feed_forward", FeedForwardSpec("routed_experts", width, ff, "silu", "m.", params=(
        ("experts", experts), ("top", top), ("router", "sigmoid_scores"), ("weigh", "inputs"))), rt)
    w = {"m.router": torch.randn(experts, width, generator=g) * 2.0 / width ** 0.5}
    for e in range(experts):
        w.update({f"m.e{e}.gate": torch.randn(ff, width, generator=g) * 2.0 / width ** 0.5, f"m.e{e}.up": torch.randn(ff, width, generator=g) * 2.0 / width ** 0.5,
                  f"m.e{e}.down": torch.randn(width, ff, generator=g) / ff ** 0.5})
    w = {k: v.to(STORED[dtype]) for k, v in w.items()}
    assert set(part.declare()) == set(w)
    part.bind({k: v.cuda() for k, v in w.items()})
    x = torch.randn(rows, width, generator=g).to(STORED[dtype])

    class Ctx:
        seq_of_token = torch.zeros(rows, dtype=torch.int32, device="cuda")
    got = part.forward(x.cuda(), Ctx)
    wd = {k: v.double() for k, v in w.items()}
    want = plain.mixture(x.double(), wd, "m.", {"router": {"top": top}})
    z = (x.double() @ wd["m.router"].T).sort(dim=1, descending=True).values         # rows whose last choice is not a close call
    clear = torch.ones(rows, dtype=torch.bool) if top == experts else (z[:, top - 1] - z[:, top]) > 1e-4
    assert clear.sum() >= 0.9 * rows
    close(got.cpu()[clear], want[clear], tol)


@pytest.mark.parametrize("act,row_weights", [(3, True), (2, False), (1, True), (0, False)])
@pytest.mark.parametrize("experts,n,k,counts", [(4, 48, 64, [3, 0, 9, 1]), (3, 40, 2056, [1, 17, 33]), (5, 22, 136, [8, 70, 0, 16, 2]), (2, 2, 8, [1, 1]),
                                                (6, 130, 328, [0, 0, 5, 31, 32, 0])])
def test_expert_products_for_a_few_rows(gpu, act, row_weights, experts, n, k, counts):
    """The weight-streaming form against float64: empty experts, more rows than a turn takes, rows found through a map, widths that end
    inside a tile; both output types. Rows behind the last one stay as they are."""
    from stride_b200.csrc import ops
    g = torch.Generator().manual_seed(n + k + act)
    rows = sum(counts)
    offsets = dev([0] + [sum(counts[:e + 1]) for e in range(experts)])
    a, w = torch.randn(rows + 2, k, generator=g).bfloat16(), (torch.randn(experts, n, k, generator=g) * k ** -0.5).bfloat16()
    perm = torch.randperm(rows, generator=g)
    f = torch.rand(rows, generator=g) if row_weights else torch.ones(rows)
    want, at = [], 0
    for e, c in enumerate(counts):
        z = (a[perm[at:at + c]].double() @ w[e].double().T) * f[at:at + c, None].double()
        if act == 1:
            z = torch.relu(z) ** 2
        elif act == 2:
            gate, up = z[:, 0::2].clamp(max=0.9), z[:, 1::2].clamp(-0.9, 0.9)
            z = gate * torch.sigmoid(1.7 * gate) * (up + 1.0)
        elif act == 3:
            z = plain.silu(z[:, 0::2]) * z[:, 1::2]
        want.append(z)
        at += c
    want = torch.cat(want)
    for out_type, tol in ((torch.float32, 2e-5), (torch.bfloat16, 6e-3)):
        out = torch.full((rows + 2, want.shape[1]), 5.0, dtype=out_type, device="cuda")
        assert ops.moe_stream(a.cuda(), perm.to(torch.int32).cuda(), w.cuda(), offsets, out, act, 0.9, 1.7, f.cuda() if row_weights else None)
        close(out[:rows], want, tol)
        assert (out[rows:] == 5.0).all()


@pytest.mark.parametrize("tokens,experts,top", [(3, 4, 2), (16, 32, 32), (64, 8, 8), (1, 1, 1), (20, 7, 3)])
@pytest.mark.parametrize("act", [3, 1])
def test_expert_products_pair_by_pair(gpu, tokens, experts, top, act):
    """The same without a plan: row p of the output is pair p, a padded token's pairs are left alone, up to 512 pairs; experts chosen by
    more tokens than a turn takes."""
    from stride_b200.csrc import ops
    g = torch.Generator().manual_seed(tokens + experts)
    n, k = 40, 72
    x, w = torch.randn(tokens, k, generator=g).bfloat16(), (torch.randn(experts, n, k, generator=g) * k ** -0.5).bfloat16()
    ids = torch.stack([torch.randperm(experts, generator=g)[:top] for _ in range(tokens)]).to(torch.int32)
    if tokens > 2:
        ids[1] = -1
    f = torch.rand(tokens, top, generator=g)
    out = torch.full((tokens * top, n if act == 1 else n // 2), 5.0, device="cuda")
    assert ops.moe_stream(x.cuda(), None, w.cuda(), None, out, act, row_weight=f.cuda(), ids=ids.cuda())
    back = torch.full((tokens * top, n), 5.0, dtype=torch.bfloat16, device="cuda")
    pair_rows = torch.randn(tokens * top, k, generator=g).bfloat16()
    assert ops.moe_stream(pair_rows.cuda(), None, w.cuda(), None, back, ids=ids.cuda(), by_pair=True)
    for t in range(tokens):
        for c in range(top):
            p, e = t * top + c, int(ids[t, c])
            if e < 0:
                assert (out[p] == 5.0).all() and (back[p] == 5.0).all()
                continue
            z = (w[e].double() @ x[t].double()) * f[t, c].double()
            close(out[p], plain.silu(z[0::2]) * z[1::2] if act == 3 else torch.relu(z) ** 2, 3e-5)
            close(back[p], w[e].double() @ pair_rows[p].double(), 6e-3)


@pytest.mark.parametrize("experts,top,extra,hidden,tokens", [(5, 2, 0, 64, 3), (32, 4, 1, 2056, 16), (256, 32, 0, 328, 9), (1, 1, 0, 8, 1), (33, 7, 3, 1024, 16),
                                                             (16, 16, 0, 264, 5), (64, 3, 0, 40, 2)])
@pytest.mark.parametrize("keep_scores", [True, False])
def test_router_and_choice_in_one_launch(gpu, experts, top, extra, hidden, tokens, keep_scores):
    """Logits against float64; choices and weights against the separate launch on the same logits; a padded token chooses nothing."""
    from stride_b200.csrc import ops
    g = torch.Generator().manual_seed(experts + hidden)
    w = (torch.randn(experts + extra, hidden, generator=g) * 2.0 * hidden ** -0.5).bfloat16()
    x, seq = torch.randn(tokens, hidden, generator=g).bfloat16(), [0] * tokens
    if tokens > 1:
        seq[tokens // 2] = -1
    live = [t for t in range(tokens) if seq[t] == 0]
    logits, weights = torch.zeros(tokens, experts + extra, device="cuda"), torch.full((tokens, top), 7.0, device="cuda")
    ids = torch.full((tokens, top), -7, dtype=torch.int32, device="cuda")
    assert ops.moe_route_rule(x.cuda(), w.cuda(), logits, None, dev(seq), ids, weights, experts, 1, 1, 1.3, group_max=True, keep_scores=keep_scores)
    z = x.double() @ w.double().T
    close(logits, z, 1e-5)
    ids2, weights2 = torch.zeros_like(ids), torch.zeros_like(weights)
    ops.moe_select_groups(logits, None, dev(seq), ids2, weights2, experts, 1, 1, 1.3, group_max=True, keep_scores=keep_scores)
    assert torch.equal(ids, ids2) and torch.equal(weights, weights2)
    scores = torch.sigmoid(logits[live][:, :experts].double().cpu())
    assert all(len(set(row)) == top for row in ids[live].tolist())
    close(scores.gather(1, ids[live].long().cpu()).sum(1), scores.sort(dim=1, descending=True).values[:, :top].sum(1), 1e-6)
    if keep_scores:
        close(weights[live], 1.3 * scores.gather(1, ids[live].long().cpu()), 1e-5)


@pytest.mark.parametrize("cap", [4.0, 30.0])
def test_a_cap_on_the_scores_is_exact(gpu, cap):
    """The tensor-core attention kernels against the exact one on the same bfloat16 inputs: scores up to several times the cap, small
    ones, and both signs."""
    from stride_b200.csrc import ops
    g = torch.Generator().manual_seed(int(cap))
    nq, nkv, hd, page, pages, n = 4, 2, 128, 16, 24, 300
    k = torch.randn(pages, nkv, page, hd, generator=g).bfloat16().cuda()
    v = torch.randn(pages, nkv, page, hd, generator=g).bfloat16().cuda()
    q = (torch.randn(n, nq * hd, generator=g) * torch.logspace(-2, 0.7, n)[:, None]).bfloat16().cuda()
    table = torch.randperm(pages, generator=g).to(torch.int32).cuda()[None]
    geometry = (nq, nkv, hd, page, 0.1, 0)
    f32 = torch.zeros(n, nq * hd, device="cuda")
    ops.paged_attention(q.float(), nq * hd, f32, k.float(), v.float(), table, dev([0] * n), dev(list(range(n))), *geometry, softcap=cap)
    for kernel in (ops.paged_attention_prefill_tc, ops.paged_attention_prefill):
        out = torch.zeros(n, nq * hd, dtype=torch.bfloat16, device="cuda")
        assert kernel(q, nq * hd, out, k, v, table, dev([0]), dev([n]), dev([n]), 1, *geometry, softcap=cap, precise_cap=True) is not False
        close(out, f32, 8e-3)
    scratch = torch.zeros(ops.decode_scratch_floats(n, nq, nkv, hd, 512), device="cuda")
    out = torch.zeros(n, nq * hd, dtype=torch.bfloat16, device="cuda")
    ops.paged_attention_decode(q, nq * hd, out, k, v, table, dev([0] * n), dev(list(range(n))), scratch, *geometry, 512, softcap=cap, precise_cap=True)
    close(out, f32, 8e-3)
    ops.check_kernel_status()


# ------------------------------------------------------------------- each mechanism in a model of nothing else
ONLY_MEMORY = cases.config(48, 67, [(cases.mamba(4, 12, 20, groups=2, conv=3, norm_groups=4), None), (cases.mamba(1, 40, 8, conv=2), None)])
ONLY_ATTENTION = cases.config(56, 89, [(cases.attention(3, 1, 12, 8, cases.rotation(8)), None), (cases.attention(2, 1, 20, 8, cases.rotation(20, scaled=False), cap=None), None),
                                       (cases.attention(4, 1, 8, 8, cases.rotation(2), cap=2.0), None)])
ONLY_MIXTURE = cases.config(56, 89, [(cases.attention(1, 1, 4), cases.moe(9, 3, 40)), (cases.attention(1, 1, 4), cases.moe(4, 1, 22))])


@pytest.mark.parametrize("name,cfg", [("memory", ONLY_MEMORY), ("attention", ONLY_ATTENTION), ("mixture", ONLY_MIXTURE)])
def test_each_mechanism_in_a_model_of_its_own(gpu, tmp_models, name, cfg):
    folder, requests, want = model_case(tmp_models, "only_" + name, cfg, cases.seeded_state(cfg, 7), "float32", 7, [45, 19, 3])
    replay(folder, "float32", modes.whole(requests), want, 8, 2, name + " whole")
    replay(folder, "float32", modes.changing_portions(requests), want, 8, 2, name + " portions")
    replay(folder, "float32", modes.tail_one_by_one(requests, tail=15), want, 8, 2, name + " decode")


@pytest.mark.parametrize("case", ["A", "C"])
def test_the_stream_after_every_layer(gpu, tmp_models, case):
    """Layer by layer in float32: the first one that differs names the mechanism."""
    from stride_b200.engine.trace import TraceSession
    cfg = cases.CASES[case]
    folder, state = write(tmp_models, f"layers_{case}", cfg, cases.seeded_state(cfg, 3), "float32")
    tokens = seeded_tokens(29, cfg["vocab"], 4)
    want = []
    plain.forward(cfg, state, tokens, capture=want)
    session = TraceSession(folder, "float32", max_tokens=64, block_size=8, max_requests=1)
    session.model.capture = []
    session.run_step({"step": 0, "entries": [{"id": "a", "tokens": tokens, "want": [0]}], "end": ["a"]})
    assert len(session.model.capture) == len(want) == len(cfg["layers"])
    for i, (got, expected) in enumerate(zip(session.model.capture, want)):
        err = float((got.double().cpu() - expected).abs().max())
        assert err <= 2e-5 * float(expected.abs().max()), f"the stream differs after layer {i}: {err:.3e}"


@pytest.mark.parametrize("case", ["C", "D"])
def test_the_checkpoints_tensors_come_back_as_stored(gpu, tmp_models, case):
    """Also where heads are laid out wider than they are, and with a number that a layer without value mixing does not read."""
    from stride_b200.engine.loading import load_model
    cfg = copy.deepcopy(cases.CASES[case])
    state = cases.seeded_state(cfg, 5)
    cfg["layers"][2]["mixer"]["v_mix"] = False
    folder, _ = write(tmp_models, "stored_" + case, cfg, state, "bfloat16")
    _config, model = load_model(folder, "bfloat16", token_capacity=16, row_capacity=4)
    named = model.named_tensors()
    assert set(state) - set(named) == {"l2.mix.vmix"} and not set(named) - set(state)
    for name, t in named.items():
        assert torch.equal(t.float().cpu(), state[name].bfloat16().float()), name


# ---------------------------------------------------------------------------- whole models, every cutting
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case,page", [("A", 16), ("B", 8), ("C", 16), ("D", 32)])
def test_every_cutting_gives_the_plain_logits(gpu, tmp_models, case, page, dtype):
    """In bfloat16 every expert is chosen, so that no close call of a router is left to rounding."""
    cfg = cases.CASES[case] if dtype == "float32" else cases.with_every_expert(cases.CASES[case])
    lengths = [230, 33, 1, 120, 9, 2] if case == "C" else [90, 33, 1, 52, 9, 2]
    folder, requests, want = model_case(tmp_models, case, cfg, cases.seeded_state(cfg, 11), dtype, 11, lengths)
    share = 1.0 if dtype == "float32" else 0.97
    replay(folder, dtype, modes.whole(requests), want, page, 2, "whole", min_ok=share)
    session = replay(folder, dtype, modes.tail_one_by_one(requests, tail=40), want, page, 2, "decode", min_ok=share)
    assert session.runner.graph_replays > 0, "single-token steps did not go through captured graphs"
    replay(folder, dtype, modes.changing_portions(requests), want, page, 2, "portions", min_ok=share)
    # three live requests, six requests in all: pages and state slots are used again
    replay(folder, dtype, modes.mixed(requests, live_limit=3, seed=5), want, page, 3, "mixed", min_ok=share)
    replay(folder, dtype, modes.decoding_together(dict(list(requests.items())[:4]), decode_steps=6, prompts_per_step=2), want, page, 4,
           "decoding together", min_ok=share)


def test_routers_that_choose_in_bfloat16(gpu, tmp_models):
    """A close call may fall the other way after rounding, and the memories carry that on: most rows hold the bound all the same."""
    cfg = cases.CASE_A
    folder, requests, want = model_case(tmp_models, "choosing", cfg, cases.seeded_state(cfg, 12), "bfloat16", 12, [70, 25, 4])
    replay(folder, "bfloat16", modes.whole(requests), want, 16, 1, "whole", min_ok=0.6)
    replay(folder, "bfloat16", modes.mixed(requests, live_limit=3, seed=1), want, 16, 3, "mixed", min_ok=0.6)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_portions_beside_single_tokens(gpu, tmp_models, dtype):
    """Steps with two portions long enough for the chunked memory, a short portion and decoded tokens of other requests, the
    portions ending inside chunks and pages; then the same requests decoded on. Against each alone."""
    cfg = cases.CASE_C
    folder, requests, want = model_case(tmp_models, "beside", cfg, cases.seeded_state(cfg, 13), dtype, 13, [300, 210, 21, 13])
    cuts = {"r0": [97, 130, 66, 1, 1, 1, 1, 1, 1, 1], "r1": [3, 100, 101, 1, 1, 1, 1, 1, 1], "r2": [1] * 21, "r3": [4, 1, 1, 1, 1, 1, 1, 1, 1, 1]}
    steps, at = [], {r: 0 for r in requests}
    for s in range(21):
        entries, ends = [], []
        for rid in requests:
            if s >= len(cuts[rid]):
                continue
            n = cuts[rid][s]
            entries.append({"id": rid, "tokens": requests[rid][at[rid]:at[rid] + n], "want": sorted({0, n // 2, n - 1})})
            at[rid] += n
            if s == len(cuts[rid]) - 1:
                ends.append(rid)
        steps.append({"step": s, "entries": entries, "end": ends})
    assert all(at[r] == len(requests[r]) for r in requests)
    replay(folder, dtype, steps, want, 16, 4, "beside", min_ok=1.0 if dtype == "float32" else 0.97)


def test_many_requests_decoding_together(gpu, tmp_models):
    """More single tokens in a step than the products for few rows take: the gate, the convolution's inputs and the step sizes then come
    from two products of other element types."""
    cfg = cases.CASE_C
    folder, requests, want = model_case(tmp_models, "many", cfg, cases.seeded_state(cfg, 14), "bfloat16", 14, [14 + (5 * i) % 13 for i in range(22)])
    session = replay(folder, "bfloat16", modes.decoding_together(requests, decode_steps=7, prompts_per_step=5), want, 16, 22, "many", min_ok=0.97)
    assert session.runner.graph_replays > 0


@pytest.mark.parametrize("name", ["A", "wide"])
def test_float32_logits_do_not_depend_on_the_cutting(gpu, tmp_models, name):
    """Bitwise: every sum of the 32-bit path has an order that depends on the token's position only (the wide model's rows take
    several turns of a CTA's threads)."""
    from stride_b200.engine.trace import TraceSession
    wide = cases.config(1100, 50, [(cases.mamba(9, 140, 70, groups=3, norm_groups=1), cases.moe(5, 2, 70)), (cases.attention(12, 3, 64), None)])
    cfg = wide if name == "wide" else cases.CASE_A
    folder, _state = write(tmp_models, "bitwise_" + name, cfg, cases.seeded_state(cfg, 13), "float32")
    requests = {f"r{i}": seeded_tokens(n, cfg["vocab"], 650 + i) for i, n in enumerate([141, 18, 27])}
    results = []
    for steps in (modes.whole(requests), modes.changing_portions(requests), modes.mixed(requests, live_limit=3, seed=2)):
        session = TraceSession(folder, "float32", max_tokens=modes.peak_tokens(steps), block_size=8, max_requests=3)
        got = {}
        rows = modes.expected_rows(steps)
        for s in steps:
            out = session.run_step(s)
            for r, key in enumerate(rows[s["step"]]):
                got[key] = out[r].clone()
        results.append(got)
    for other in results[1:]:
        for key in other:
            assert torch.equal(other[key], results[0][key]), f"request {key[0]} position {key[1]} differs between cuttings"


# --------------------------------------------------------------------------------- far keys, first values, long memories
def weights_on_outputs(_f, h, w, p, mlp):
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        ids, scores = plain.route(h[t], w[p + "router"], mlp["router"]["top"])
        for e, s in zip(ids, scores):
            out[t] += s * plain.expert(h[t], w, f"{p}e{e}.")
    return out


def with_rule(name, replacement, run):
    original = getattr(plain, name)
    try:
        setattr(plain, name, lambda *a: replacement(original, *a))
        return run()
    finally:
        setattr(plain, name, original)


@pytest.mark.parametrize("dtype,dim", [("float32", 12), ("bfloat16", 12), ("bfloat16", 64), ("bfloat16", 80)])
def test_small_departures_from_the_rules_would_show(gpu, tmp_models, dtype, dim):
    """The plain logits with values not mixed, a cap twice as wide, positions counted from one further on for the first layer's queries
    only, the norm in front of the gate, or the scores on the experts' outputs (a smaller change, which the
    float32 bound tells) differ; the engine gives the design's."""
    cfg = cases.config(64, 61, [(cases.attention(4, 2, dim, dim, scale=6.0 / dim ** 0.5, cap=4.0, rot=cases.rotation(dim // 4 * 2, base=50.0)), None),
                                (cases.mamba(4, 16, 16, norm_groups=4), None),
                                (cases.attention(2, 2, dim, dim, scale=6.0 / dim ** 0.5, cap=5.0, rot=cases.rotation(dim // 4 * 2, base=50.0)), cases.moe(3, 3, 32))])
    state = cases.seeded_state(cfg, 21)
    state["l2.mix.vmix"] = torch.tensor(0.75)
    for e in range(3):
        state[f"l2.mlp.e{e}.gate"] *= 2.0
    state["l2.mlp.router"] *= 1.5
    folder, state = write(tmp_models, f"rules_{dim}", cfg, state, dtype)
    tokens = seeded_tokens(90, cfg["vocab"], 8)
    run = lambda: plain.forward(cfg, state, tokens)
    full = run()
    for name, wrong in (("mixed_values", lambda f, v, first, share: v), ("capped_scores", lambda f, q, k, s, c: f(q, k, s, 2 * c)),
                        ("rotate", lambda f, x, rot: f(x, rot, 1 if x.shape[1] == 4 else 0)),
                        ("gated_group_norm", lambda f, y, z, w, n, eps: plain.rms_unit(y.view(y.shape[0], n, -1), eps).reshape(y.shape) * plain.silu(z) * w),
                        ("mixture", weights_on_outputs)):
        moved = (with_rule(name, wrong, run) - full).abs().amax(dim=1) > (0.01 if name == "mixture" else 0.04) * full.abs().max()
        assert moved[30:].sum() >= 30, f"{name} does not show in these logits"
    requests, want = {"w": tokens}, {"w": full}
    share = 1.0 if dtype == "float32" else 0.97
    replay(folder, dtype, modes.whole(requests), want, 16, 1, "rules whole", min_ok=share)
    replay(folder, dtype, modes.tail_one_by_one(requests, tail=50), want, 16, 1, "rules decode", min_ok=share)
    replay(folder, dtype, modes.changing_portions(requests, sizes=(7, 2, 33, 9, 2, 40)), want, 4, 1, "rules portions", min_ok=share)


@pytest.mark.parametrize("dtype,dim", [("float32", 8), ("bfloat16", 8), ("bfloat16", 112)])
def test_a_far_past_shows_through_sharp_attention(gpu, tmp_models, dtype, dim):
    """Scores sharp enough for single keys to decide, hundreds of tokens back: another far past (positions 0 .. 23 only)
    moves the plain logits beyond position 300, and the engine follows the true past, whole, decoded and in portions."""
    cfg = cases.config(64, 61, [(cases.attention(4, 2, dim, 8 if dim == 8 else 40, cases.rotation(4 if dim == 8 else 12), scale=7.0 / dim ** 0.5 if dim == 8 else 0.85, cap=40.0), None)])
    folder, state = write(tmp_models, f"far_{dim}", cfg, cases.seeded_state(cfg, 41), dtype)
    tokens = seeded_tokens(420, cfg["vocab"], 8)
    full = plain.forward(cfg, state, tokens)
    other = list(tokens)
    other[:24] = seeded_tokens(24, cfg["vocab"], 9)
    moved = (plain.forward(cfg, state, other) - full)[300:].abs().amax(dim=1) > 0.03 * full.abs().max()
    assert moved.sum() >= 12, "the far past does not show in these logits"
    requests, want = {"far": tokens}, {"far": full}
    share = 1.0 if dtype == "float32" else 0.97
    keep = {"far": set(range(0, 420, 5)) | set(range(300, 420)) | {0, 1, 2, 3, 7, 8, 9, 15, 16, 17}}
    for page in (8, 16):
        replay(folder, dtype, modes.restrict_wants(modes.whole(requests), keep), want, page, 1, "far whole", min_ok=share)
        replay(folder, dtype, modes.tail_one_by_one(requests, tail=110), want, page, 1, "far decode", min_ok=share)
        replay(folder, dtype, modes.restrict_wants(modes.changing_portions(requests, sizes=(7, 2, 64, 9, 33, 2, 120)), keep), want, page, 1,
               "far portions", min_ok=share)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("state_size,vdim", [(24, 20), (64, 64)])
def test_a_memory_that_carries_its_first_tokens_over_hundreds_of_steps(gpu, tmp_models, state_size, vdim, dtype):
    """Decays so slow that another beginning (positions 0 .. 11 only) moves the plain logits 400 steps later. The engine carries the
    memory through portions (chunked and short) and single tokens, and a second request finds its slot cleared."""
    cfg = cases.config(48, 67, [(cases.mamba(2, vdim, state_size, groups=1, conv=3), cases.moe(2, 2, 40))])
    state = cases.seeded_state(cfg, 19, decay=-9.0)
    # the first seven ids take large steps, the others small ones
    u = torch.randn(48, generator=torch.Generator().manual_seed(2))
    u = u / u.norm()
    state["embed"] -= 3.0 * u
    state["embed"][:7] += 6.0 * u
    state["l0.mix.in"][-2:] = u
    folder, state = write(tmp_models, f"memory_{state_size}", cfg, state, dtype)
    later = [7 + t for t in seeded_tokens(418, 60, 8)]
    tokens, second = seeded_tokens(12, 7, 7) + later, seeded_tokens(60, cfg["vocab"], 10)
    full = plain.forward(cfg, state, tokens)
    other = seeded_tokens(12, 7, 9) + later
    moved = (plain.forward(cfg, state, other) - full)[400:].abs().amax(dim=1)
    assert (moved > 0.02 * full.abs().max()).sum() >= 10, "the first tokens do not show in these logits"
    requests, want = {"long": tokens, "next": second}, {"long": full, "next": plain.forward(cfg, state, second)}
    keep = {"long": set(range(0, 430, 7)) | set(range(395, 430)), "next": set(range(60))}
    share = 1.0 if dtype == "float32" else 0.97
    replay(folder, dtype, modes.restrict_wants(modes.whole(requests), keep), want, 8, 1, "memory whole", min_ok=share)
    replay(folder, dtype, modes.restrict_wants(modes.changing_portions(requests, sizes=(64, 2, 9, 150, 3)), keep), want, 8, 1, "memory portions", min_ok=share)
    replay(folder, dtype, modes.tail_one_by_one(requests, tail=45), want, 8, 1, "memory decode", min_ok=share)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_on_the_tensor_core_sizes(gpu, tmp_models, dtype):
    """140 tokens decoded one by one after a prompt, across many page borders, and a second request from its first token on."""
    cfg = cases.CASE_C
    folder, requests, want = model_case(tmp_models, "long", cfg, cases.seeded_state(cfg, 17, decay=-3.0), dtype, 17, [389, 141])
    share = 1.0 if dtype == "float32" else 0.97
    keep = {"r0": set(range(0, 389, 7)) | set(range(260, 389)) | {0, 1, 2, 3, 15, 16, 17, 31, 32, 33, 63, 64, 65}, "r1": set(range(0, 141, 3))}
    replay(folder, dtype, modes.restrict_wants(modes.whole(requests), keep), want, 16, 2, "whole", min_ok=share)
    replay(folder, dtype, modes.tail_one_by_one(requests, tail=140), want, 16, 2, "long decode", min_ok=share)


# --------------------------------------------------------------------------- generation through the engine
def test_greedy_generation_through_the_engine(gpu, tmp_models):
    from stride_b200 import Engine, SamplingParams
    cfg = cases.CASE_A
    folder, state = write(tmp_models, "generate", cfg, cases.seeded_state(cfg, 29), "float32")
    prompts = [seeded_tokens(n, cfg["vocab"], 300 + n) for n in (37, 5, 18, 1, 26)]
    new = 9
    expected = []
    for prompt in prompts:
        seq = list(prompt)
        for _ in range(new):
            seq.append(int(plain.forward(cfg, state, seq)[-1].argmax()))
        expected.append(seq[len(prompt):])
    # a token budget below the longest prompt: prompts go in portions beside the others' decoded tokens
    engine = Engine(folder, dtype="float32", block_size=8, num_blocks=64, max_batch_tokens=16, max_batch_seqs=3, max_model_len=64,
                    check_invariants=True)
    outs = engine.generate(copy.deepcopy(prompts), SamplingParams(temperature=0.0, max_tokens=new, ignore_eos=True))
    assert [o.tokens for o in outs] == expected
