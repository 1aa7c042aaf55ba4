"""The Dopudra decoder in the engine against the plain float64 implementation (``plain_dopudra``): each mechanism alone (as a
kernel and in a model of nothing else), the stream after every layer, whole prompts against token-by-token decoding,
portions down to two tokens, batches of unequal requests on pages and state slots that are used again, keys on both sides of
every distance bucket's edge in prompts and among decoded tokens, queries on both sides of a step of their factor, a far past that
shows through sharp attention or a slow memory, the first tokens, long decoding, sizes unlike one another, and greedy
generation through the engine's scheduler."""

import copy
import math

import pytest
import torch

import dopudra_cases as cases
import plain_dopudra as plain
import trace_modes as modes
from helpers import compare_logits, seeded_tokens, write_model_dir

pytestmark = pytest.mark.gpu
STORED = {"float32": torch.float32, "bfloat16": torch.bfloat16}


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
    row, a few per cent of its spread for these small random models; a wrong key, bucket or memory changes a row outright,
    and the float32 runs of the same cuttings hold the tight bound."""
    if dtype == "float32":
        return compare_logits(got, want, dtype)
    a, b = got.double().reshape(-1), want.double().reshape(-1)
    if not torch.isfinite(a).all():
        return False, "non-finite logits"
    cos = float(torch.nn.functional.cosine_similarity(a, b, dim=0))
    rel = float((a - b).norm() / (b - b.mean()).norm())
    return cos >= BF16_BOUND[0] and rel <= BF16_BOUND[1], f"cosine {cos:.6f}, error {rel:.3f} of the row's spread"


def rounded(state, dtype):
    return {k: v.to(STORED[dtype]) for k, v in state.items()}


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
    assert total and bad <= (1.0 - min_ok) * total, f"{bad} of {total} rows differ; first: {first}"
    stats = session.cache.stats()
    assert stats["live"] == 0 and session.cache.free_slots == session.cache.slot_capacity
    return session


def write(tmp_models, name, cfg, state, dtype):
    """The model folder and the weights as the engine will see them, in float64."""
    folder = write_model_dir(str(tmp_models / f"dopudra_{name}_{dtype}"), cfg, state, STORED[dtype])
    return folder, {k: v.double() for k, v in rounded(state, dtype).items()}


def model_case(tmp_models, name, cfg, state, dtype, seed, lengths):
    folder, state = write(tmp_models, name, cfg, state, dtype)
    requests = {f"r{i}": seeded_tokens(n, cfg["vocab"], 50 * seed + i) for i, n in enumerate(lengths)}
    return folder, requests, {rid: plain.forward(cfg, state, toks) for rid, toks in requests.items()}


def dev(values, dtype=torch.int32):
    return torch.tensor(values, dtype=dtype, device="cuda")


# ------------------------------------------------------------------------------------------------- kernels alone
@pytest.mark.parametrize("dtype,tol", [("float32", 2e-6), ("bfloat16", 8e-3)])
@pytest.mark.parametrize("n,width", [(1, 64), (2, 54), (3, 1032), (4, 2048), (5, 50), (6, 96), (7, 33), (8, 128), (9, 40), (13, 100), (16, 36)])
def test_write_and_read_of_the_copies(gpu, dtype, tol, n, width):
    """Through the stream as the layers use it: the first read and write from the embedding's output, then from the copies; a read
    for some rows only leaves the write pending; the sum of the copies at the end."""
    from stride_b200.config import NormSpec
    from stride_b200.parts import Runtime, build_part
    from stride_b200.parts.copies import CopiedStream, CopyWeights
    g = torch.Generator().manual_seed(n * width)
    rt, tokens = Runtime("cuda", STORED[dtype], 16, 8), 11
    norm = build_part("norm", NormSpec("rmsnorm", width, 1e-3, "n", (("tensor", "n"),)), rt)
    norm_w = 1.0 + 0.3 * torch.randn(width, generator=g)
    norm.bind({"n": norm_w.cuda()})
    stream = CopiedStream(rt, tokens, width, n)
    x = torch.randn(tokens, width, generator=g)
    stream.residual.copy_(x)
    X = x.double()[None].repeat(n, 1, 1)
    for step in range(4):
        w = {"in": torch.randn(n, generator=g), "out": torch.randn(n, generator=g), "mix": torch.randn(n, n, generator=g) / math.sqrt(n),
             "s": 1.0 + 0.5 * torch.randn(width, generator=g)}
        part = CopyWeights(n, width, "", "s" if step != 2 else None)
        assert set(part.declare()) == ({"in", "out", "mix", "s"} if step != 2 else {"in", "out", "mix"})
        part.bind({k: v.cuda() for k, v in w.items()})
        wd = {k: v.double() for k, v in w.items()}
        close(stream.read(norm, part.read), plain.rms_norm(plain.read_copies(X, wd, ""), norm_w.double(), 1e-3), tol)
        y = (torch.randn(tokens, width, generator=g) * 2).to(STORED[dtype])
        stream.write(y.cuda(), part)
        X = plain.write_copies(X, y.double() * (wd["s"] if step != 2 else 1.0), wd, "")
        rows = torch.tensor([7, 2, 2], dtype=torch.int32)
        close(stream.normed(norm, rows=rows.cuda()), plain.rms_norm(X.sum(0), norm_w.double(), 1e-3)[rows.long()], tol)
        if step == 1:
            close(stream.materialize(), X.sum(0), 2e-6)
        close(stream.normed(norm, rows=rows.cuda()), plain.rms_norm(X.sum(0), norm_w.double(), 1e-3)[rows.long()], tol)
    close(stream.materialize(), X.sum(0), 2e-6)
    copies = stream.rows_of_copies.view(tokens, n, width).double().cpu()
    close(copies, X.transpose(0, 1), 2e-6)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width", [64, 54, 33])
def test_embedding_with_a_factor_and_a_learned_vector_per_position(gpu, dtype, width):
    from stride_b200.config import EmbeddingSpec
    from stride_b200.parts import Runtime, build_part
    g = torch.Generator().manual_seed(width)
    rt = Runtime("cuda", STORED[dtype], 16, 4)
    part = build_part("embedding", EmbeddingSpec("lookup", 30, width, "e", params=(("scale", 0.37), ("positions", ("p", 12)))), rt)
    assert {k: v.shape for k, v in part.declare().items()} == {"e": (30, width), "p": (12, width)}
    table, pos = torch.randn(30, width, generator=g).to(STORED[dtype]), torch.randn(12, width, generator=g).to(STORED[dtype])
    part.bind({"e": table.cuda(), "p": pos.cuda()})
    assert torch.equal(part.named_tensors()["p"].cpu(), pos)

    class Ctx:
        token_ids, positions, seq_of_token = dev([3, 29, 0, 7, 3]), dev([0, 11, 5, 4, 0]), dev([0, 1, 1, 2, -1])
    out = torch.full((5, width), float("nan"), device="cuda")
    part.forward(Ctx, out)
    want = table.double()[[3, 29, 0, 7]] * 0.37 + pos.double()[[0, 11, 5, 4]]
    close(out[:4], want, 1e-6)
    assert float(out[4].abs().max()) == 0.0


def memory_inputs(H, D, DV, new, dtype, g, ld_extra=8):
    tokens = sum(new) + 1
    k_off, v_off = H * D + 2, 2 * H * D + 2
    proj = (torch.randn(tokens, v_off + H * DV + ld_extra, generator=g)).to(STORED[dtype])
    state = torch.zeros(len(new) + 1, H * D * DV + 3)
    state[1:, :H * D * DV] = torch.randn(len(new), H * D * DV, generator=g)
    return proj, k_off, v_off, state


def plain_memory(x, k_off, v_off, S0, decay, H, D, DV, act, q_scale):
    """o [T, H, DV] and the memories afterwards; ``decay(t, head)`` a factor per row of S."""
    S, T = S0.clone(), x.shape[0]
    out = torch.zeros(T, H, DV, dtype=torch.float64)
    for a in range(H):
        for t in range(T):
            q, k = act(x[t, a * D:(a + 1) * D]) * q_scale, act(x[t, k_off + a * D:k_off + (a + 1) * D])
            v = act(x[t, v_off + a * DV:v_off + (a + 1) * DV])
            S[a] = decay(t, a) * S[a] + torch.outer(k, v)
            out[t, a] = S[a].T @ q
    return out, S


MEMORY_SIZES = [(3, 12, 20), (1, 8, 40), (2, 64, 128), (3, 10, 14), (1, 200, 24), (2, 128, 130), (4, 32, 32), (1, 2, 6)]


@pytest.mark.parametrize("form", ["chain", "chunks"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,D,DV", MEMORY_SIZES)
def test_memory_with_a_constant_decay(gpu, dtype, H, D, DV, form):
    """Two requests with a past and a fresh one (a long portion, a short one, one of exactly a chunk and one token), against the
    recurrence token by token in float64 on the same inputs, in both forms of the kernel; then the state rows as the next step
    must find them. The recurrence is float32 in both storage types, so one bound holds. Decays from 0 to 1."""
    from stride_b200.csrc import ops
    g = torch.Generator().manual_seed(H * D + DV)
    new = [149, 7, 65]
    proj, k_off, v_off, state = memory_inputs(H, D, DV, new, dtype, g)
    state[0] = 0.0
    slots, decay = [2, 0, 1], [0.9, 0.0, 1.0, 0.999][:H]
    state_dev = state.cuda()
    o = torch.full((proj.shape[0], H * DV), float("nan"), device="cuda")
    q_start, q_len = dev([0, new[0], new[0] + new[1], 0]), dev(new + [0])
    d64 = torch.tensor(decay, dtype=torch.float64)
    if form == "chain":
        ops.decay_scan(proj.cuda(), 0, k_off, v_off, None, None, (d64 - 1).float().cuda(), 1.0, 1.0, o, state_dev, q_start, q_len,
                       dev(slots + [0]), 4, H, D, DV)
    else:
        powers = (d64[:, None] ** torch.arange(ops.DECAY_CHUNK + 1, dtype=torch.float64)).float().cuda()
        scratch = torch.full((ops.decay_chunks_scratch_floats(4, 149, H, D, DV),), float("nan"), device="cuda")
        ops.decay_chunks(proj.cuda(), 0, k_off, v_off, None, None, powers, 1.0, 1.0, o, state_dev, q_start, q_len, dev(slots + [0]), 4, H, D, DV,
                         149, scratch)
    at = 0
    for n, slot in zip(new, slots):
        S0 = state[slot, :H * D * DV].double().view(H, D, DV)
        want, S = plain_memory(proj[at:at + n].double(), k_off, v_off, S0, lambda t, a: decay[a], H, D, DV, plain.silu, 1.0)
        for a in range(H):
            close(o[at:at + n, a * DV:(a + 1) * DV], want[:, a], 1e-5)
        close(state_dev[slot, :H * D * DV], S.reshape(-1), 1e-5)
        at += n
    assert torch.equal(state_dev[:, H * D * DV:].cpu(), state[:, H * D * DV:]) and torch.equal(state_dev[3].cpu(), state[3])


@pytest.mark.parametrize("form", ["chain", "chunks"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,D,DV", MEMORY_SIZES)
def test_memory_with_channel_decays(gpu, dtype, H, D, DV, form):
    """The same for decays of the token's own per key channel; some channels forget nearly everything at some tokens (decays down
    to e^-40), so that a chunk's running product leaves the range of float32."""
    from stride_b200.csrc import ops
    g = torch.Generator().manual_seed(H + D * DV)
    new = [149, 7, 65]
    proj, k_off, v_off, state = memory_inputs(H, D, DV, new, dtype, g)
    state[0] = 0.0
    slots, tau = [2, 0, 1], 2.5
    logit = torch.randn(proj.shape[0], H * D, generator=g) * 2.0 + 3.0
    logit[20:75:6, ::3] = -100.0            # within the first two chunks of the first request only: both paths are taken
    bias = torch.randn(H * D, generator=g)
    state_dev = state.cuda()
    o = torch.full((proj.shape[0], H * DV), float("nan"), device="cuda")
    q_start, q_len = dev([0, new[0], new[0] + new[1], 0]), dev(new + [0])
    alpha = (torch.sigmoid(logit.double() + bias.double()) ** (1.0 / tau)).view(-1, H, D)
    if form == "chain":
        ops.decay_scan(proj.cuda(), 0, k_off, v_off, logit.cuda(), bias.cuda(), None, D ** -0.5, 1.0 / tau, o, state_dev, q_start, q_len,
                       dev(slots + [0]), 4, H, D, DV)
    else:
        scratch = torch.full((ops.decay_chunks_scratch_floats(4, 149, H, D, DV),), float("nan"), device="cuda")
        ops.decay_chunks(proj.cuda(), 0, k_off, v_off, logit.cuda(), bias.cuda(), None, D ** -0.5, 1.0 / tau, o, state_dev, q_start, q_len,
                         dev(slots + [0]), 4, H, D, DV, 149, scratch)
    at = 0
    for n, slot in zip(new, slots):
        S0 = state[slot, :H * D * DV].double().view(H, D, DV)
        decay = lambda t, a: alpha[at + t, a][:, None]
        want, S = plain_memory(proj[at:at + n].double(), k_off, v_off, S0, decay, H, D, DV, lambda x: x, D ** -0.5)
        close(o[at:at + n], want.reshape(n, -1), 1e-5)
        close(state_dev[slot, :H * D * DV], S.reshape(-1), 1e-5)
        at += n
    assert torch.equal(state_dev[:, H * D * DV:].cpu(), state[:, H * D * DV:]) and torch.equal(state_dev[3].cpu(), state[3])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("constant", [True, False])
@pytest.mark.parametrize("H,D,DV", [(3, 12, 20), (2, 64, 128), (1, 200, 24), (2, 128, 132), (4, 32, 32), (1, 256, 260), (3, 10, 14)])
def test_a_single_token_of_every_request(gpu, dtype, constant, H, D, DV):
    """The one-pass form: three requests with a past, a slot without a request, state rows inside wider ones. (A width that is no
    multiple of four runs the chain.)"""
    from stride_b200.csrc import ops
    g = torch.Generator().manual_seed(H * D + DV)
    new = [1, 1, 1]
    proj, k_off, v_off, state = memory_inputs(H, D, DV, new, dtype, g)
    wide = torch.full((4, 8 + -(-state.shape[1] // 4) * 4 + 4), float("nan"), device="cuda")
    view = wide[:, 8:8 + state.shape[1]]
    view.copy_(state)
    logit, bias = torch.randn(4, H * D, generator=g) * 3.0, torch.randn(H * D, generator=g)
    decay = torch.rand(H, generator=g, dtype=torch.float64)
    o = torch.full((4, H * DV), float("nan"), device="cuda")
    order = [3, 1, 2]
    ops.decay_scan(proj.cuda(), 0, k_off, v_off, None if constant else logit.cuda(), None if constant else bias.cuda(),
                   (decay - 1).float().cuda() if constant else None, D ** -0.5, 0.3, o, view, dev([0, 1, 2, 0]), dev([1, 1, 1, 0]), dev(order + [0]), 4,
                   H, D, DV, single=True)
    alpha = (torch.sigmoid(logit.double() + bias.double()) ** 0.3).view(-1, H, D)
    for t, slot in enumerate(order):
        rate = (lambda _t, a: float(decay[a])) if constant else (lambda _t, a: alpha[t, a][:, None])
        S0 = state[slot, :H * D * DV].double().view(H, D, DV)
        want, S = plain_memory(proj[t:t + 1].double(), k_off, v_off, S0, rate, H, D, DV, plain.silu if constant else (lambda x: x),
                               1.0 if constant else D ** -0.5)
        close(o[t], want.reshape(-1), 1e-5)
        close(view[slot, :H * D * DV], S.reshape(-1), 1e-5)
    assert torch.equal(view[:, H * D * DV:].cpu(), state[:, H * D * DV:]) and torch.equal(view[0].cpu(), state[0])
    assert torch.isnan(wide[:, :8]).all() and torch.isnan(wide[:, 8 + state.shape[1]:]).all()


@pytest.mark.parametrize("dtype,tol", [("float32", 3e-6), ("bfloat16", 8e-3)])
@pytest.mark.parametrize("width,kind", [(20, "sigmoid_compute"), (520, "sigmoid_compute"), (514, "silu"), (2048, "sigmoid_compute"), (700, "sigmoid")])
def test_norm_over_all_heads_with_a_gate(gpu, dtype, tol, width, kind):
    from stride_b200.csrc import ops
    g = torch.Generator().manual_seed(width)
    o, w = torch.randn(9, 2 * width, generator=g) * 3, 1.0 + 0.3 * torch.randn(width, generator=g)
    gate = torch.randn(9, 2 * width + 8, generator=g) * 2
    gate = gate if kind == "sigmoid" else gate.to(STORED[dtype])
    out = torch.zeros(9, 2 * width, dtype=STORED[dtype], device="cuda")
    ops.head_norm_gate(o.cuda(), w.cuda(), False, gate.cuda(), kind, out, 2, width, 1e-3, gate_off=8)
    z = gate[:, 8:].double()
    want = plain.rms_norm(o.double().view(9, 2, width), w.double(), 1e-3).reshape(9, -1) * (plain.silu(z) if kind == "silu" else torch.sigmoid(z))
    close(out, want, tol)


@pytest.mark.parametrize("dtype,tol", [("float32", 3e-6), ("bfloat16", 8e-3)])
@pytest.mark.parametrize("rows,ff", [(1, 24), (5, 50), (40, 128), (3, 7)])
def test_feed_forward_without_a_gate(gpu, dtype, tol, rows, ff):
    from stride_b200.config import FeedForwardSpec
    from stride_b200.parts import Runtime, build_part
    g = torch.Generator().manual_seed(ff)
    rt, width = Runtime("cuda", STORED[dtype], 64, 4), 56
    part = build_part("feed_forward", FeedForwardSpec("mlp", width, ff, "relu2", "m."), rt)
    up, down = (torch.randn(ff, width, generator=g) * 0.2).to(STORED[dtype]), (torch.randn(width, ff, generator=g) * 0.3).to(STORED[dtype])
    part.bind({"m.up": up.cuda(), "m.down": down.cuda()})
    x = torch.randn(rows, width, generator=g).to(STORED[dtype])
    close(part.forward(x.cuda(), None), plain.feed_forward(x.double(), {"up": up.double(), "down": down.double()}, ""), tol)


@pytest.mark.parametrize("dtype,tol", [("float32", 3e-6), ("bfloat16", 1e-2)])
@pytest.mark.parametrize("nq,nkv,hd,vd,taps,every", [(3, 1, 32, 32, 3, 4), (4, 4, 16, 24, 4, 1), (2, 2, 48, 16, 1, 5), (3, 3, 20, 18, 2, 3), (2, 1, 128, 256, 16, 7),
                                                     (5, 5, 2, 6, 5, 2), (2, 1, 8, 8, 0, 0)])
def test_convolution_row_norms_query_factor_and_tails(gpu, dtype, tol, nq, nkv, hd, vd, taps, every):
    """Three requests in one step (a start, a portion deep inside a request, a single token) against the plain convolution over
    each request's whole past, norms over whole projections and the factor at each query's own position; then the tails. The state
    rows are a column block of wider rows, as they are beside another mixer's state."""
    from stride_b200.csrc import ops
    g = torch.Generator().manual_seed(hd + vd + taps)
    q_dim, k_dim = nq * hd, nkv * hd
    C, keep, coef = q_dim + k_dim + nkv * vd, max(taps - 1, 0), 0.6
    past, new = [0, 9, 1], [7, 5, 1]                        # tokens a request held before the step, and brings now
    page, pages = 4, 12
    histories = [(torch.randn(p + n, C, generator=g) * 2).to(STORED[dtype]) for p, n in zip(past, new)]
    raw = torch.cat([h[p:] for h, p in zip(histories, past)] + [torch.zeros(1, C, dtype=STORED[dtype])])       # one padded row
    tokens = raw.shape[0]
    conv_w = torch.randn(C, taps, generator=g) * 0.7 if taps else None
    wq, wk = 1.0 + 0.3 * torch.randn(q_dim, generator=g), 1.0 + 0.3 * torch.randn(k_dim, generator=g)
    slots_of_state = [2, 0, 1]
    wide = torch.full((3, 12 + keep * C + 7), float("nan"), device="cuda")
    state = wide[:, 8:12 + keep * C]                        # the tail from float 4 of this part on
    for h, p, slot in zip(histories, past, slots_of_state):
        tail = torch.zeros(keep, C)
        if keep and p:
            rows = h[max(0, p - keep):p].float()
            tail[keep - rows.shape[0]:] = rows
        state[slot, 4:] = tail.reshape(-1).cuda()
    seq_of = dev([0] * new[0] + [1] * new[1] + [2] * new[2] + [-1])
    positions = dev([p + i for p, n in zip(past, new) for i in range(n)] + [0])
    q_start, q_len, state_slot = dev([0, new[0], new[0] + new[1], 0]), dev(new + [0]), dev(slots_of_state + [0])
    slot_map = torch.randperm(page * pages, generator=g)[:tokens].to(torch.int32)
    slot_map[-1] = -1
    k_pages = torch.full((pages, nkv, page, hd), 7.0, dtype=STORED[dtype], device="cuda")
    v_pages = torch.full((pages, nkv, page, vd), 7.0, dtype=STORED[dtype], device="cuda")
    out = torch.zeros(tokens, C + 8, dtype=STORED[dtype], device="cuda")
    ops.conv_row_norm(raw.cuda(), out, conv_w.t().contiguous().cuda() if taps else None, state if keep else None, 4, seq_of, q_start, q_len, state_slot,
                      positions, wq.cuda(), wk.cuda(), 1e-5, coef, every, slot_map.cuda(), k_pages, v_pages, nq, nkv, hd, vd, page)
    if keep:
        ops.conv_tail(raw.cuda(), state, 4, q_start, q_len, state_slot, 4, C, taps, min_len=2)
    at = 0
    for h, p, n, slot in zip(histories, past, new, slots_of_state):
        y = plain.short_convolution(h.double(), conv_w.double()) if taps else h.double()
        q, k, v = plain.rms_norm(y[:, :q_dim], wq.double(), 1e-5), plain.rms_norm(y[:, q_dim:q_dim + k_dim], wk.double(), 1e-5), y[:, q_dim + k_dim:]
        if every:
            q = q * torch.tensor([plain.query_factor(i, {"coef": coef, "every": every}) for i in range(p + n)], dtype=torch.float64)[:, None]
        close(out[at:at + n, :C], torch.cat([q, k, v], dim=1)[p:], tol)
        for r in range(n):
            s = int(slot_map[at + r])
            close(k_pages[s // page, :, s % page], k[p + r].view(nkv, hd), tol)
            close(v_pages[s // page, :, s % page], v[p + r].view(nkv, vd), tol)
        if keep:
            tail = torch.zeros(keep, C, dtype=torch.float64)
            rows = h[max(0, p + n - keep):].double()
            tail[keep - rows.shape[0]:] = rows
            assert torch.equal(state[slot, 4:].cpu().double(), tail.reshape(-1)), "the tail is the last projected rows, exactly"
        at += n
    assert float(out[-1].abs().max()) == 0.0            # the padded row is not touched
    assert torch.isnan(wide[:, :12]).all() and torch.isnan(wide[:, 12 + keep * C:]).all()      # nor anything beside the tails


@pytest.mark.parametrize("nq,nkv,hd,page,length", [(4, 2, 64, 16, 40), (2, 1, 128, 16, 300), (3, 1, 64, 8, 2), (6, 2, 128, 32, 131), (2, 2, 64, 4, 1)])
def test_distance_table_in_every_attention_kernel(gpu, nq, nkv, hd, page, length):
    """Portions and single tokens with a table of numbers per head and distance: the exact kernel against the formula, the tcgen05,
    mma.sync and split-decode kernels against the same. ``length`` entries a head: contexts shorter and longer than the table, tiles
    wholly beyond it, across its end and inside it."""
    from stride_b200.csrc import ops
    g = torch.Generator().manual_seed(nq * hd + length)
    lens = [(0, 150), (300, 70), (5, 2), (130, 1), (515, 1), (0, 1)]
    total_pages = sum(-(-(c + n) // page) for c, n in lens) + 2
    perm = torch.randperm(total_pages, generator=g).tolist()
    table = torch.zeros(len(lens), max(-(-(c + n) // page) for c, n in lens), dtype=torch.int32)
    q_start, q_len, ctx_len, seq_of, positions, at = [], [], [], [], [], 0
    for s, (c, n) in enumerate(lens):
        held = [perm.pop() for _ in range(-(-(c + n) // page))]
        table[s, :len(held)] = torch.tensor(held)
        q_start.append(at), q_len.append(n), ctx_len.append(c + n)
        seq_of += [s] * n
        positions += list(range(c, c + n))
        at += n
    tokens, portions = at, 3
    k = torch.randn(total_pages, nkv, page, hd, generator=g).bfloat16()
    v = torch.randn(total_pages, nkv, page, hd, generator=g).bfloat16()
    q = torch.randn(tokens, nq * hd, generator=g).bfloat16()
    rel = torch.randn(nq, length, generator=g) * 2.0
    scale = 0.7 * hd ** -0.5
    want = torch.zeros(tokens, nq, hd, dtype=torch.float64)
    for s, (c, n) in enumerate(lens):
        order = [(int(table[s, j // page]), j % page) for j in range(c + n)]
        keys = torch.stack([k[p, :, o] for p, o in order]).double()
        values = torch.stack([v[p, :, o] for p, o in order]).double()
        for i in range(n):
            t, pos = q_start[s] + i, c + i
            dist = torch.arange(pos, -1, -1).clamp(max=length - 1)
            for a in range(nq):
                kh = a // (nq // nkv)
                sc = keys[:pos + 1, kh] @ q[t, a * hd:(a + 1) * hd].double() * scale + rel[a, dist].double()
                want[t, a] = torch.softmax(sc, 0) @ values[:pos + 1, kh]
    want = want.reshape(tokens, nq * hd)
    q, k, v, rel, table = q.cuda(), k.cuda(), v.cuda(), rel.cuda(), table.cuda()
    out = torch.full((tokens, nq * hd), float("nan"), dtype=torch.bfloat16, device="cuda")
    geometry = (nq, nkv, hd, page, scale, 0)
    ops.paged_attention(q, nq * hd, out, k, v, table, dev(seq_of), dev(positions), *geometry, rel=rel)
    close(out, want, 1e-2)
    f32 = torch.full((tokens, nq * hd), float("nan"), device="cuda")
    ops.paged_attention(q.float(), nq * hd, f32, k.float(), v.float(), table, dev(seq_of), dev(positions), *geometry, rel=rel)
    close(f32, want, 3e-6)
    split = q_start[portions]
    for kernel in (ops.paged_attention_prefill_tc, ops.paged_attention_prefill):
        part = torch.full((split, nq * hd), float("nan"), dtype=torch.bfloat16, device="cuda")
        done = kernel(q[:split], nq * hd, part, k, v, table, dev(q_start), dev(q_len), dev(ctx_len), portions, *geometry, rel=rel)
        assert done is not False
        close(part, want[:split], 2e-2)
    bound = 600
    scratch = torch.zeros(ops.decode_scratch_floats(3, nq, nkv, hd, bound), device="cuda")
    tail = torch.full((3, nq * hd), float("nan"), dtype=torch.bfloat16, device="cuda")
    ops.paged_attention_decode(q[split:], nq * hd, tail, k, v, table, dev(seq_of[split:]), dev(positions[split:]), scratch, *geometry, bound, rel=rel)
    close(tail, want[split:], 2e-2)
    ops.check_kernel_status()


# ------------------------------------------------------------------- each mechanism in a model of nothing else
PASSIVE = cases.memory(1, 2)
ONLY_LIGHTNING = cases.config(48, 67, [(cases.lightning(3, 12, 20, decay=(0.3, 0.97, 1.0)), None), (cases.lightning(1, 40, 8), None)], streams=2)
ONLY_ATTENTION = cases.config(56, 89, [(cases.parallel(cases.attention(3, 1, 12, 8, conv=3, bias_max=20, scale=0.5), PASSIVE, 1.0, 0.0), None),
                                       (cases.parallel(cases.attention(2, 2, 8, 12, conv=5, bias_max=33), PASSIVE, 1.5, 0.0), None)], streams=1)
ONLY_MEMORY = cases.config(48, 67, [(cases.parallel(cases.attention(1, 1, 4), cases.memory(2, 12, 20, tau=2.0), 0.0, 1.0), None),
                                    (cases.parallel(cases.attention(1, 1, 4), cases.memory(1, 40, 8, tau=20.0), 0.0, 0.8), None)], streams=2)
ONLY_FF = cases.config(56, 89, [(cases.lightning(1, 4), cases.dense(70)), (cases.lightning(1, 4), cases.dense(9))], streams=6)


@pytest.mark.parametrize("name,cfg", [("lightning", ONLY_LIGHTNING), ("attention", ONLY_ATTENTION), ("memory", ONLY_MEMORY), ("ff", ONLY_FF)])
def test_each_mechanism_in_a_model_of_its_own(gpu, tmp_models, name, cfg):
    folder, requests, want = model_case(tmp_models, "only_" + name, cfg, cases.seeded_state(cfg, 7, (12, 7), (4, 9)), "float32", 7, [45, 19, 3])
    replay(folder, "float32", modes.whole(requests), want, 8, 2, name + " whole")
    replay(folder, "float32", modes.changing_portions(requests), want, 8, 2, name + " portions")
    replay(folder, "float32", modes.tail_one_by_one(requests, tail=15), want, 8, 2, name + " decode")


@pytest.mark.parametrize("case", ["A", "C"])
def test_the_stream_after_every_layer(gpu, tmp_models, case):
    """Layer by layer in float32: the first one that differs names the mechanism."""
    from stride_b200.engine.trace import TraceSession
    cfg = cases.CASES[case]
    folder, state = write(tmp_models, f"layers_{case}", cfg, cases.case_state(case, 3), "float32")
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


def test_the_checkpoints_tensors_come_back_as_stored(gpu, tmp_models):
    from stride_b200.engine.loading import load_model
    cfg = cases.CASE_D
    state = cases.case_state("D", 5)
    folder, _ = write(tmp_models, "stored", cfg, state, "bfloat16")
    _config, model = load_model(folder, "bfloat16", token_capacity=16, row_capacity=4)
    named = model.named_tensors()
    assert set(named) == set(state)
    for name, t in named.items():
        assert torch.equal(t.float().cpu(), state[name].bfloat16().float()), name


# ---------------------------------------------------------------------------- whole models, every cutting
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case,page", [("A", 16), ("B", 8), ("C", 16), ("D", 32)])
def test_every_cutting_gives_the_plain_logits(gpu, tmp_models, case, page, dtype):
    cfg = cases.CASES[case]
    lengths = [230, 33, 1, 120, 9, 2] if case == "C" else [110, 33, 1, 52, 9, 2]
    folder, requests, want = model_case(tmp_models, case, cfg, cases.case_state(case, 11), dtype, 11, lengths)
    share = 1.0 if dtype == "float32" else 0.97
    replay(folder, dtype, modes.whole(requests), want, page, 2, "whole", min_ok=share)
    session = replay(folder, dtype, modes.tail_one_by_one(requests, tail=40), want, page, 2, "decode", min_ok=share)
    assert session.runner.graph_replays > 0, "single-token steps did not go through captured graphs"
    replay(folder, dtype, modes.changing_portions(requests), want, page, 2, "portions", min_ok=share)
    # three live requests, six requests in all: pages and state slots are used again
    replay(folder, dtype, modes.mixed(requests, live_limit=3, seed=5), want, page, 3, "mixed", min_ok=share)
    replay(folder, dtype, modes.decoding_together(dict(list(requests.items())[:4]), decode_steps=6, prompts_per_step=2), want, page, 4,
           "decoding together", min_ok=share)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_portions_beside_single_tokens(gpu, tmp_models, dtype):
    """Steps with two portions long enough for the chunked memories, a short portion and decoded tokens of other requests, the
    portions ending inside chunks and pages; then the same requests decoded on. Against each alone."""
    cfg = cases.CASE_C
    folder, requests, want = model_case(tmp_models, "beside", cfg, cases.case_state("C", 12), dtype, 12, [300, 210, 21, 13])
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


@pytest.mark.parametrize("name", ["A", "wide"])
def test_float32_logits_do_not_depend_on_the_cutting(gpu, tmp_models, name):
    """Bitwise: every sum of the 32-bit path has an order that depends on the token's position only (the wide model's rows take
    several turns of a CTA's threads)."""
    from stride_b200.engine.trace import TraceSession
    wide = cases.config(1100, 50, [(cases.lightning(4, 32, 144), None), (cases.parallel(cases.attention(12, 3, 64), cases.memory(2, 16, 24)), None)])
    cfg, state = (wide, cases.seeded_state(wide, 13)) if name == "wide" else (cases.CASE_A, cases.case_state("A", 13))
    folder, _state = write(tmp_models, "bitwise_" + name, cfg, state, "float32")
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


# ------------------------------------------------------------------------ distances, factors, far keys, long memories
def distance_model(head=8):
    """Two attention layers (the memories beside them are switched off) with tables of strong numbers: a key in the wrong bucket
    changes the logits outright."""
    scale = 1.7 * head ** -0.5
    return cases.config(64, 61, [(cases.parallel(cases.attention(4, 2, head, conv=2, bias_max=48, scale=scale), PASSIVE, 1.0, 0.0), None),
                                 (cases.parallel(cases.attention(2, 1, head, conv=3, bias_max=25, scale=scale, coef=0.5, every=12), PASSIVE, 1.0, 0.0),
                                  cases.dense(32))])


def with_rule(name, replacement, run):
    original = getattr(plain, name)
    try:
        setattr(plain, name, lambda *a: replacement(original, *a))
        return run()
    finally:
        setattr(plain, name, original)


@pytest.mark.parametrize("dtype,head", [("float32", 8), ("bfloat16", 8), ("bfloat16", 64)])
@pytest.mark.parametrize("page", [4, 16])
def test_keys_on_both_sides_of_a_buckets_edge(gpu, tmp_models, dtype, head, page):
    """The plain logits with every bucket begun one key early or one key late, with the table ending one bucket short, and with
    all far keys' numbers left out differ outright at the compared positions, in the prompt and among decoded tokens; the engine
    gives the design's, on the exact and on the tensor-core kernels."""
    cfg = distance_model(head)
    folder, state = write(tmp_models, f"distance_{head}_{page}", cfg, cases.seeded_state(cfg, 41, (12, 8), bias_std=3.0), dtype)
    tokens = seeded_tokens(130, cfg["vocab"], 8)
    run = lambda: plain.forward(cfg, state, tokens)
    full = run()
    for wrong in (lambda f, n, b, d: f(n + 1, b, d), lambda f, n, b, d: f(max(n - 1, 0), b, d), lambda f, n, b, d: min(f(n, b, d), b - 2)):
        moved = (with_rule("distance_bucket", wrong, run) - full).abs().amax(dim=1) > 0.05 * full.abs().max()
        assert moved[60:].sum() >= 40, "the buckets' edges do not show in these logits"
    requests, want = {"w": tokens}, {"w": full}
    share = 1.0 if dtype == "float32" else 0.97
    replay(folder, dtype, modes.whole(requests), want, page, 1, "distance whole", min_ok=share)
    replay(folder, dtype, modes.tail_one_by_one(requests, tail=80), want, page, 1, "distance decode", min_ok=share)
    replay(folder, dtype, modes.changing_portions(requests, sizes=(7, 2, 33, 9, 2, 40)), want, page, 1, "distance portions", min_ok=share)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_queries_on_both_sides_of_a_step_of_their_factor(gpu, tmp_models, dtype):
    """A factor that jumps from 1 to more than 3 at its first step: one token early or late, or left out, moves the logits outright at
    that position."""
    cfg = cases.config(64, 61, [(cases.parallel(cases.attention(4, 2, 8, conv=2, bias_max=48, scale=0.9, coef=3.0, every=20), PASSIVE, 1.0, 0.0), None)])
    folder, state = write(tmp_models, "factor", cfg, cases.seeded_state(cfg, 43, bias_std=0.3), dtype)
    tokens = seeded_tokens(70, cfg["vocab"], 8)
    run = lambda: plain.forward(cfg, state, tokens)
    full = run()
    for wrong, at in ((lambda f, p, t: f(p + 1, t), [18, 38, 58]), (lambda f, p, t: f(max(p - 1, 0), t), [19, 39, 59]), (lambda f, p, t: 1.0, [19, 25, 69])):
        moved = (with_rule("query_factor", wrong, run) - full).abs().amax(dim=1) > 0.02 * full.abs().max()
        assert moved[at].all() and not moved[:18].any(), "the factor does not show in these logits"
    share = 1.0 if dtype == "float32" else 0.97
    replay(folder, dtype, modes.whole({"f": tokens}), {"f": full}, 8, 1, "factor whole", min_ok=share)
    replay(folder, dtype, modes.tail_one_by_one({"f": tokens}, tail=55), {"f": full}, 8, 1, "factor decode", min_ok=share)


@pytest.mark.parametrize("dtype,head", [("float32", 8), ("bfloat16", 8), ("bfloat16", 128)])
def test_a_far_past_shows_through_sharp_attention(gpu, tmp_models, dtype, head):
    """Scores sharp enough for single keys to decide, hundreds of tokens back: another far past (positions 0 .. 23 only)
    moves the plain logits beyond position 300, and the engine follows the true past, whole, decoded and in portions."""
    cfg = cases.config(64, 61, [(cases.parallel(cases.attention(4, 2, head, conv=2, bias_max=60, scale=2.5 if head == 8 else 0.6, coef=0.1, every=64), PASSIVE,
                                                1.0, 0.0), None)])
    state = cases.seeded_state(cfg, 41, bias_std=0.5)
    state["pos"] *= 0.2
    folder, state = write(tmp_models, f"far_{head}", cfg, state, dtype)
    tokens = seeded_tokens(420, cfg["vocab"], 8)
    full = plain.forward(cfg, state, tokens)
    other = list(tokens)
    other[:24] = seeded_tokens(24, cfg["vocab"], 9)
    moved = (plain.forward(cfg, state, other) - full)[300:].abs().amax(dim=1) > 0.03 * full.abs().max()
    assert moved.sum() >= 20, "the far past does not show in these logits"
    requests, want = {"far": tokens}, {"far": full}
    share = 1.0 if dtype == "float32" else 0.97
    keep = {"far": set(range(0, 420, 5)) | set(range(300, 420)) | {0, 1, 2, 3, 7, 8, 9, 15, 16, 17}}
    for page in (8, 16):
        replay(folder, dtype, modes.restrict_wants(modes.whole(requests), keep), want, page, 1, "far whole", min_ok=share)
        replay(folder, dtype, modes.tail_one_by_one(requests, tail=110), want, page, 1, "far decode", min_ok=share)
        replay(folder, dtype, modes.restrict_wants(modes.changing_portions(requests, sizes=(7, 2, 64, 9, 33, 2, 120)), keep), want, page, 1,
               "far portions", min_ok=share)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind", ["lightning", "memory"])
def test_a_memory_that_carries_its_first_tokens_over_hundreds_of_steps(gpu, tmp_models, kind, dtype):
    """Decays of 0.9999 and more: another beginning (positions 0 .. 11 only) moves the plain logits 400 steps later. The engine
    carries the memory through portions (chunked and short) and single tokens, and a second request finds its slot cleared."""
    if kind == "lightning":
        cfg = cases.config(48, 67, [(cases.lightning(2, 16, 24, decay=(0.9999, 1.0)), cases.dense(40))], streams=2)
        state = cases.seeded_state(cfg, 19)
        # keys open for the first tokens and all but close for later ones: both positions' vectors lie along one direction, and so do
        # the rows of the key projection (silu of a large negative number is next to nothing)
        u = torch.randn(48, generator=torch.Generator().manual_seed(2))
        u = u / u.norm()
        state["l0.mix.k"] += 1.5 * u
        state["pos"][:12] += 40.0 * u
        state["pos"][12:] -= 40.0 * u
    else:
        cfg = cases.config(48, 67, [(cases.parallel(cases.attention(1, 1, 4), cases.memory(2, 16, 24, tau=16.0), 0.0, 1.0), cases.dense(40))], streams=2)
        state = cases.seeded_state(cfg, 19, decay_bias=9.0)
        state["l0.mix.right.a2"] *= 0.1
    state["pos"] *= 0.2
    folder, state = write(tmp_models, f"memory_{kind}", cfg, state, dtype)
    tokens, second = seeded_tokens(430, cfg["vocab"], 8), seeded_tokens(60, cfg["vocab"], 10)
    full = plain.forward(cfg, state, tokens)
    other = seeded_tokens(12, cfg["vocab"], 9) + tokens[12:]
    moved = (plain.forward(cfg, state, other) - full)[400:].abs().amax(dim=1)
    assert (moved > 0.03 * full.abs().max()).sum() >= 15, "the first tokens do not show in these logits"
    requests, want = {"long": tokens, "next": second}, {"long": full, "next": plain.forward(cfg, state, second)}
    keep = {"long": set(range(0, 430, 7)) | set(range(395, 430)), "next": set(range(60))}
    share = 1.0 if dtype == "float32" else 0.97
    replay(folder, dtype, modes.restrict_wants(modes.whole(requests), keep), want, 8, 1, "memory whole", min_ok=share)
    replay(folder, dtype, modes.restrict_wants(modes.changing_portions(requests, sizes=(64, 2, 9, 120, 3)), keep), want, 8, 1, "memory portions", min_ok=share)
    replay(folder, dtype, modes.tail_one_by_one(requests, tail=45), want, 8, 1, "memory decode", min_ok=share)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_on_the_tensor_core_sizes(gpu, tmp_models, dtype):
    """Head sizes 64 and 128, memories of 64 x 128 and 128 x 64: 140 tokens decoded one by one after a prompt, past every bucket and across
    many page borders, and a second request from its first token on."""
    cfg = cases.sharpened(cases.CASE_C, 1.5)
    folder, requests, want = model_case(tmp_models, "long", cfg, cases.case_state("C", 17), dtype, 17, [389, 141])
    share = 1.0 if dtype == "float32" else 0.97
    keep = {"r0": set(range(0, 389, 7)) | set(range(260, 389)) | {0, 1, 2, 3, 15, 16, 17, 31, 32, 33, 63, 64, 65}, "r1": set(range(0, 141, 3))}
    replay(folder, dtype, modes.restrict_wants(modes.whole(requests), keep), want, 16, 2, "whole", min_ok=share)
    replay(folder, dtype, modes.tail_one_by_one(requests, tail=140), want, 16, 2, "long decode", min_ok=share)


def test_a_sequence_may_use_every_position_and_no_more(gpu, tmp_models):
    """The table of position vectors ends where it ends: its last row is used, a longer sequence is refused on the host."""
    from stride_b200.engine.trace import TraceError, TraceSession
    cfg = cases.config(40, 53, [(cases.lightning(1, 8), None)], max_positions=24)
    folder, state = write(tmp_models, "positions", cfg, cases.seeded_state(cfg, 3), "float32")
    tokens = seeded_tokens(24, 53, 1)
    replay(folder, "float32", modes.tail_one_by_one({"p": tokens}, tail=9), {"p": plain.forward(cfg, state, tokens)}, 8, 1, "positions")
    session = TraceSession(folder, "float32", max_tokens=64, block_size=8, max_requests=1)
    session.run_step({"step": 0, "entries": [{"id": "a", "tokens": tokens, "want": [23]}], "end": []})
    with pytest.raises(TraceError, match="max_position"):
        session.run_step({"step": 1, "entries": [{"id": "a", "tokens": [1], "want": [0]}], "end": []})


# --------------------------------------------------------------------------- generation through the engine
def test_greedy_generation_through_the_engine(gpu, tmp_models):
    from stride_b200 import Engine, SamplingParams
    cfg = cases.CASE_A
    folder, state = write(tmp_models, "generate", cfg, cases.case_state("A", 29), "float32")
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
