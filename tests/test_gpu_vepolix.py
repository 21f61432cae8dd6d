"""The Vepolix decoder through the framework's own loader, cache, step function and generation loop, against the plain
implementation (tests/plain_vepolix.py), in float32 and bfloat16.

The float32 runs are the sharp ones: they differ from the plain implementation only by the order of sums, so a key that is
missed, a chunk that is one token off, a bucket that starts too early or a maximum that is lost shows at once.  The
configurations are in vepolix_helpers.py.
"""
from __future__ import annotations

import json

import pytest
import torch

import plain_vepolix as P
from vepolix_helpers import CONFIGS, assert_logits, oracle_logits, random_weights, read_folder, tokens, write_folder

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]
FULL = ["mixed", "odd", "wide"]
DEV = "cuda:0"


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    made = {}

    def get(name: str, seed: int = 0, gain: float = 1.0) -> str:
        key = (name, seed, gain)
        if key not in made:
            c = CONFIGS[name]
            made[key] = write_folder(str(tmp_path_factory.mktemp(f"vepolix-{name}")), c, random_weights(c, seed, gain))
        return made[key]

    return get


@pytest.fixture(scope="module")
def models(folders):
    from kuiperllama_b200.engine import load_model
    made = {}

    def get(name: str, dtype: str, **kw):
        key = (name, dtype, tuple(sorted(kw.items())))
        if key not in made:
            folder = folders(name, **kw)
            with torch.inference_mode():
                made[key] = (load_model(folder, dtype=dtype, device=DEV), folder)
        return made[key]

    return get


def _engine(model, max_tokens=64 * 16, use_graphs=False):
    from kuiperllama_b200.engine import Engine
    return Engine(model, model.new_cache(max_tokens=max_tokens), use_graphs=use_graphs)


def _inputs(slot, toks, want=None):
    from kuiperllama_b200.engine import SequenceInput
    return SequenceInput(slot, list(toks), list(range(len(toks))) if want is None else want)


def _run_in_steps(engine, toks, cuts):
    """One sequence fed in steps of the given sizes; logits of every token."""
    rows, at = [], 0
    with torch.inference_mode():
        slot = engine.alloc_slot()
        for n in cuts:
            rows.append(engine.step([_inputs(slot, toks[at:at + n])]).clone())
            at += n
        engine.free_slot(slot)
    assert at == len(toks)
    engine.check_device_errors()
    return torch.cat(rows)


def _step(starts, news, dev=DEV):
    """A ragged step of len(starts) sequences in slots 0, 1, ...: sequence s brings news[s] tokens from position starts[s]."""
    from kuiperllama_b200.parts.base import StepContext
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
    cu = [0]
    for k in news:
        cu.append(cu[-1] + k)
    pos = i32([st + i for st, k in zip(starts, news) for i in range(k)])
    tslot = i32([sl for sl, k in enumerate(news) for _ in range(k)])
    slots = list(range(len(starts)))
    return StepContext(n_tokens=cu[-1], n_seqs=len(starts), token_ids=pos, positions=pos, token_slot=tslot, seq_slots=i32(slots),
                       seq_starts=i32(starts), seq_new=i32(news), cu_tokens=i32(cu), is_decode=max(news) == 1, max_new=max(news),
                       max_context=max(a + b for a, b in zip(starts, news)), host_slots=slots, host_starts=list(starts), host_new=list(news))


# ----------------------------------------------------------------------------- the new kernels alone

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [8, 33, 192, 1024])
def test_the_sinusoid_in_the_embedding_kernel(dtype, width):
    """Positions from 0 to beyond 100,000 (where a product of 32-bit numbers alone would be off by hundredths), odd widths too."""
    from kuiperllama_b200.config.spec import PartSpec
    from kuiperllama_b200.csrc import ops
    from kuiperllama_b200.parts.base import Runtime
    from kuiperllama_b200.parts.position import SinusoidalPosition
    dt = getattr(torch, dtype)
    g = torch.Generator().manual_seed(width)
    table = torch.randn(11, width, generator=g).to(dt)
    pos = torch.tensor([0, 1, 2, 63, 64, 1000, 4097, 65535, 100003, 131071], dtype=torch.int32)
    ids = torch.arange(10, dtype=torch.int32)
    part = SinusoidalPosition(PartSpec("sinusoidal", {"hidden_size": width, "base": 10000.0}), "", {}, Runtime(torch.device(DEV), dt))
    out = torch.empty(10, width, dtype=torch.float32, device=DEV)
    flag = torch.zeros(1, dtype=torch.int32, device=DEV)
    ops.embedding(ids.to(DEV), table.to(DEV), out, flag, scale=1.7, positions=pos.to(DEV), freq=part.embedding_frequencies())
    want = torch.stack([1.7 * table[i].double() + torch.tensor([(torch.sin if c % 2 == 0 else torch.cos)(
        torch.tensor(float(p) * 10000.0 ** (-2.0 * (c // 2) / width), dtype=torch.float64)) for c in range(width)]) for i, p in enumerate(pos.tolist())])
    assert float((out.cpu().double() - want).abs().max()) < 2e-6 and int(flag) == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("source", ["rows", "pieces"])
@pytest.mark.parametrize("H, G, d, dv, mix, norm, aligned", [(6, 3, 16, 20, None, True, False), (4, 2, 12, 12, "keep", True, True), (5, 5, 10, 6, "mix", True, False),
                                                              (8, 2, 64, 32, "mix", True, True), (16, 4, 128, 64, "keep", True, True), (3, 1, 18, 7, "mix", False, False),
                                                              (40, 8, 64, 128, "mix", True, True), (2, 2, 256, 64, None, True, True), (64, 64, 64, 64, "mix", True, True)])
def test_norm_over_the_whole_projection_and_mixed_values(dtype, source, H, G, d, dv, mix, norm, aligned):
    """``ops.qk_row_prepare`` alone on a ragged step over scattered pages: rows of a product or its float32 pieces, columns on and
    off 16-byte boundaries, widths that take one, two and four pieces a thread (or the form through shared memory)."""
    from kuiperllama_b200.csrc import ops
    dt = getattr(torch, dtype)
    g = torch.Generator().manual_seed(H * 7 + d)
    starts, news = [5, 100, 0], [70, 1, 9]
    step = _step(starts, news)
    n = step.n_tokens
    gap = (lambda c: -c % 8) if aligned else (lambda c: 3)
    q_col = 8
    k_col = q_col + H * d + gap(H * d)
    v_col = k_col + G * d + gap(G * d)
    width = v_col + G * dv + 2
    width += -width % 8 if aligned else 0
    rnd = lambda *s: torch.randn(*s, generator=g)
    if source == "rows":
        proj = rnd(n, width).to(dt)
        total = proj.double()
    else:
        proj = rnd(3, n, width)
        total = proj.double().sum(0)
    qw, kw = 1 + 0.3 * rnd(H * d), 1 + 0.3 * rnd(G * d)
    first, lam = rnd(n, G * dv + 8).to(dt), torch.tensor([0.37])
    table = torch.tensor([[5, 2, 9, 0], [1, 7, 3, 11], [4, 6, 8, 10]], dtype=torch.int32, device=DEV)
    kc = torch.zeros(12, G, 64, d, dtype=dt, device=DEV)
    vc = torch.zeros(12, G, 64, dv, dtype=dt, device=DEV)
    q_out = torch.zeros(n, H * d, dtype=dt, device=DEV)
    keep = torch.zeros(n, G * dv, dtype=dt, device=DEV) if mix == "keep" else None
    kw_args = dict(norm=norm, eps=1e-5, q_norm_weight=qw.to(DEV), k_norm_weight=kw.to(DEV), v_keep=keep)
    if mix == "mix":
        kw_args.update(v_first=first.to(DEV)[:, :G * dv], v_lambda=lam.to(DEV))
    ops.qk_row_prepare(proj.to(DEV), q_col, k_col, v_col, q_out, step, table, kc, vc, H, G, d, dv, **kw_args)
    q, k, v = total[:, q_col:q_col + H * d], total[:, k_col:k_col + G * d], total[:, v_col:v_col + G * dv]
    if norm:
        q, k = P.rms_norm(q, qw.double(), 1e-5), P.rms_norm(k, kw.double(), 1e-5)
    else:
        q, k = q * qw.double(), k * kw.double()
    own = v
    if mix == "mix":
        v = 0.63 * v + 0.37 * first[:, :G * dv].double()
    tol = 2e-5 if dtype == "float32" else 2e-2
    assert torch.allclose(q_out.cpu().double(), q, atol=tol, rtol=tol)
    if keep is not None:
        assert torch.allclose(keep.cpu().double(), own, atol=tol, rtol=tol)
    row = 0
    for s, (st, k_new) in enumerate(zip(starts, news)):
        for i in range(k_new):
            p = st + i
            page = int(table[s, p // 64])
            assert torch.allclose(kc[page, :, p % 64].cpu().double(), k[row].view(G, d), atol=tol, rtol=tol), ("k", s, i)
            assert torch.allclose(vc[page, :, p % 64].cpu().double(), v[row].view(G, dv), atol=tol, rtol=tol), ("v", s, i)
            row += 1
    # a layer that only reads another one's cache: the queries alone
    again = torch.zeros_like(q_out)
    ops.qk_row_prepare(proj.to(DEV), q_col, k_col, v_col, again, step, None, None, None, H, G, d, dv, norm=norm, eps=1e-5,
                       q_norm_weight=qw.to(DEV), k_norm_weight=kw.to(DEV))
    assert torch.equal(again, q_out)


@pytest.mark.parametrize("dtype, kernel", [("float32", "plain"), ("bfloat16", "plain"), ("bfloat16", "mma"), ("bfloat16", "mma3")])
@pytest.mark.parametrize("H, G, d, dv, chunk, window, rel_n", [
    (4, 2, 12, 20, 37, 0, 37), (3, 1, 18, 7, 1, 0, 1), (8, 4, 64, 32, 96, 0, 96), (2, 1, 32, 32, 64, 0, 33), (6, 2, 128, 128, 100, 0, 60),
    (5, 1, 64, 64, 0, 0, 129), (16, 1, 64, 128, 2, 0, 2), (8, 2, 128, 64, 130, 0, 5), (4, 4, 32, 128, 200, 50, 40), (2, 2, 64, 64, 127, 0, 0),
    (3, 3, 32, 64, 65, 0, 65), (12, 4, 128, 32, 77, 100, 20)])
def test_chunks_and_distance_bias_on_scattered_pages(dtype, kernel, H, G, d, dv, chunk, window, rel_n):
    """The attention kernels with chunks and a bias by distance (and a window beside the chunks): three sequences on scattered
    pages grow in ragged steps whose portions start and end inside chunks and pages; after every step every new token's result is
    compared with plain arithmetic.  The tensor-core kernel with single tokens' keys in one piece and cut into three."""
    from kuiperllama_b200.csrc import ops
    if kernel != "plain" and not (d in (32, 64, 128) and dv in (32, 64, 128)):
        pytest.skip("the tensor-core kernel takes key and value sizes of 32, 64 and 128")
    dt = getattr(torch, dtype)
    g = torch.Generator().manual_seed(H * 10 + d + chunk)
    T = 256
    table = torch.tensor([[5, 2, 9, 0], [1, 7, 3, 11], [4, 6, 8, 10]], dtype=torch.int32, device=DEV)
    ks = [torch.randn(T, G, d, generator=g).to(dt) for _ in range(3)]
    vs = [torch.randn(T, G, dv, generator=g).to(dt) for _ in range(3)]
    qs = [(torch.randn(T, H, d, generator=g) * 1.5).to(dt) for _ in range(3)]
    rel = torch.randn(H, rel_n, generator=g) if rel_n else None
    kc = torch.full((12, G, 64, d), float("nan"), dtype=dt, device=DEV).nan_to_num(7.0)
    vc = torch.full((12, G, 64, dv), 7.0, dtype=dt, device=DEV)
    scale, rep = 0.2, H // G
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = P.chunk_mask(T, chunk or None) & ((i - j < window) if window else True)
    want = []
    for s in range(3):
        k, v, q = ks[s].double().repeat_interleave(rep, 1), vs[s].double().repeat_interleave(rep, 1), qs[s].double()
        sc = torch.einsum("ihd,jhd->hij", q, k) * scale
        if rel is not None:
            sc = sc + rel.double()[:, (i - j).clamp(0, rel_n - 1)]
        want.append(torch.einsum("hij,jhd->ihd", torch.softmax(sc.masked_fill(~seen[None], float("-inf")), -1), v))
    tol = 3e-5 if dtype == "float32" else 3e-2
    bias = rel.to(DEV) if rel is not None else None
    at = [0, 0, 0]
    for news in ([100, 1, 67], [30, 2, 56], [1, 1, 1], [3, 110, 60], [1, 1, 1], [121, 141, 71]):
        step = _step(at, news)
        for s in range(3):
            for p in range(at[s], at[s] + news[s]):
                kc[int(table[s, p // 64]), :, p % 64] = ks[s][p].to(DEV)
                vc[int(table[s, p // 64]), :, p % 64] = vs[s][p].to(DEV)
        rows = lambda parts: torch.cat([p[a:a + n].reshape(n, -1) for p, a, n in zip(parts, at, news)])
        out = torch.full((step.n_tokens, H * dv), 9.0, dtype=dt, device=DEV)
        q = rows(qs).to(DEV).contiguous()
        if kernel == "plain":
            ops.attention_simt(q, H * d, out, kc, vc, table, step.positions, step.token_slot, step.n_tokens, H, G, d, scale, window, value_dim=dv,
                               chunk=chunk, distance_bias=bias)
        else:
            ops.attention_chunked_mma(q, H * d, out, kc, vc, table, step, H, G, d, dv, scale, window=window, chunk=chunk, distance_bias=bias,
                                      splits=3 if kernel == "mma3" and step.is_decode else 1, few_rows=step.is_decode)
        ref = rows(want)
        assert torch.allclose(out.cpu().double(), ref, atol=tol, rtol=tol), (at, news, float((out.cpu().double() - ref).abs().max()))
        at = [a + n for a, n in zip(at, news)]
    assert at == [T] * 3


def _memory_case(H, d, dv, starts_state, news, dtype, seed, f_bias=2.0, i_bias=0.0, width=64):
    """Operands of one memory layer for a ragged step, and what plain arithmetic gives: (q, k, v, x, W, b, state, want)."""
    dt = getattr(torch, dtype)
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *s: torch.randn(*s, generator=g)
    n = sum(news)
    q, k, v = rnd(n, H * d).to(dt), rnd(n, H * d).to(dt), rnd(n, H * dv).to(dt)
    x, W = rnd(n, width).to(dt), (3 * rnd(2 * H, width) / width ** 0.5).to(dt)
    b = torch.cat([i_bias + rnd(H), f_bias + rnd(H)])
    return q, k, v, x, W, b


def _memory_plain(q, k, v, x, W, b, cap, news, H, d, dv):
    w = {"i": W[:H].double(), "f": W[H:].double(), "i.b": b[:H].double(), "f.b": b[H:].double()}
    num, den, r = [], [], 0
    for n in news:
        sl = slice(r, r + n)
        i, f = P.log_gates(x[sl].double(), w, cap)
        sums = [P.mlstm_sums(q[sl, h * d:(h + 1) * d].double() * d ** -0.5, k[sl, h * d:(h + 1) * d].double(),
                             v[sl, h * dv:(h + 1) * dv].double(), i[:, h], f[:, h]) for h in range(H)]
        num.append(torch.stack([a for a, _ in sums], 1))
        den.append(torch.stack([b for _, b in sums], 1))
        r += n
    return num, den


@pytest.mark.parametrize("form, dtype", [("walk", "float32"), ("walk", "bfloat16"), ("chunked", "bfloat16")])
@pytest.mark.parametrize("H, d, dv, f_bias, i_bias, cap", [(3, 8, 12, 2.0, 0.0, 9.0), (2, 24, 10, 3.0, 1.0, 4.0), (1, 256, 72, 2.0, 0.0, 12.0), (3, 128, 64, 6.0, 0.0, 12.0),
                                                            (4, 64, 96, 2.0, -4.0, 15.0), (2, 40, 8, -8.0, 0.0, 12.0), (2, 200, 24, 9.0, 6.0, 12.0),
                                                            (3, 7, 5, 2.0, 0.0, 9.0), (1, 33, 9, 5.0, 0.0, 6.0), (2, 300, 16, 2.0, 0.0, 8.0), (1, 1000, 6, 2.0, 0.0, 8.0), (2, 6, 512, 2.0, 0.0, 8.0)])
def test_the_memory_over_ragged_portions(form, dtype, H, d, dv, f_bias, i_bias, cap):
    """Gates, running maximum, matrix, normaliser and denominator alone: sequences of several lengths in portions of many sizes
    (single tokens, portions shorter and longer than a chunk, ends at a chunk's border and one off), gates that forget nearly all
    and nearly nothing, maxima that stay at their start and maxima that rise; the state goes from portion to portion."""
    from kuiperllama_b200.csrc import ops
    total = [200, 131, 64]
    q, k, v, x, W, b = _memory_case(H, d, dv, None, total, dtype, seed=H * 100 + d, f_bias=f_bias, i_bias=i_bias)
    if form == "chunked" and not (d % 8 == 0 and dv % 8 == 0 and d <= 256):
        pytest.skip("the chunked form takes sizes in multiples of 8 and keys up to 256")
    want, want_den = _memory_plain(q, k, v, x, W, b, cap, total, H, d, dv)
    z_off, m_off = H * d * dv, H * d * dv + H * d
    size = -(-(m_off + H) // 4) * 4
    state = torch.zeros(3, size, device=DEV)
    first = [0, total[0], total[0] + total[1]]
    at = [0, 0, 0]
    Wd, bd = W.to(DEV), b.to(DEV)
    for news in ([64, 1, 3], [1, 1, 1], [2, 63, 30], [65, 66, 29], [68, 0, 1]):
        live = [s for s in range(3) if news[s]]
        step = _step([at[s] for s in live], [news[s] for s in live])
        step.seq_slots = torch.tensor(live, dtype=torch.int32, device=DEV)
        rows = torch.cat([torch.arange(first[s] + at[s], first[s] + at[s] + news[s]) for s in live])
        pick = lambda t: t[rows].to(DEV).contiguous()
        n = step.n_tokens
        y, den = torch.full((n, H * dv), 9.0, device=DEV), torch.full((n, H), 9.0, device=DEV)
        if form == "chunked":
            logs = ops.mlstm_gates(pick(x), Wd, bd, cap, state[:, m_off:], step, logs=True)
            ops.mlstm_chunked(pick(q), pick(k), pick(v), logs, state, z_off, y, den, step, H, d, dv, d ** -0.5, 1e-6)
        else:
            a, c, floor = ops.mlstm_gates(pick(x), Wd, bd, cap, state[:, m_off:], step)
            ops.outer_recurrence(pick(q), pick(k), pick(v), a, state, y, step, H, H, d, dv, c=c, q_scale=d ** -0.5,
                                 normaliser=(state[:, z_off:], floor, den, 1e-6))
        # sums and denominators apart (a denominator near a zero of z . q magnifies its rounding), each against its row's size, or
        # a part of the largest one so far where a row's terms cancel
        for got, ref, largest in ((y.view(n, H, dv), torch.cat([want[s][at[s]:at[s] + news[s]] for s in live]), max(float(w.abs().max()) for w in want)),
                                  (den[:, :, None], torch.cat([want_den[s][at[s]:at[s] + news[s]] for s in live])[:, :, None],
                                   max(float(w.max()) for w in want_den))):
            err = (got.cpu().double() - ref).abs().amax(-1) / ref.abs().amax(-1).clamp_min(0.05 * largest)
            assert float(err.max()) < 5e-5 and float(err.median()) < 1e-5, (news, float(err.max()), float(err.median()))
        at = [p + m for p, m in zip(at, news)]
    assert at == total


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, dim", [(4, 12), (2, 96), (3, 130), (1, 512), (2, 640), (1, 1031), (2, 7)])
def test_the_head_norm_with_a_divisor_and_a_sigmoid_gate(dtype, heads, dim):
    from kuiperllama_b200.csrc import ops
    dt = getattr(torch, dtype)
    g = torch.Generator().manual_seed(dim)
    n = 37
    x = torch.randn(n, heads * dim, generator=g)
    wide = torch.randn(n, heads * dim + 8, generator=g).to(dt)
    w = 1 + 0.3 * torch.randn(heads * dim, generator=g)
    div = torch.rand(n, heads, generator=g) + 0.2
    for act, f in (("sigmoid", torch.sigmoid), ("silu", P.silu)):
        for first in (False, True):
            out = torch.zeros(n, heads * dim + 16, dtype=dt, device=DEV)[:, 8:8 + heads * dim]
            ops.head_rmsnorm_gate(x.to(DEV), wide.to(DEV)[:, :heads * dim], w.to(DEV), out, heads, dim, 1e-3, gate_first=first, out_scale=0.7,
                                  divisor=div.to(DEV), gate_act=act)
            gate = f(wide[:, :heads * dim].double()).view(n, heads, dim)
            y = x.double().view(n, heads, dim) / div.double()[:, :, None]
            y = P.rms_norm(y * gate, None, 1e-3) if first else P.rms_norm(y, None, 1e-3) * gate
            want = (y.reshape(n, -1) * w.double()) * 0.7
            tol = 1e-5 if dtype == "float32" else 2e-2
            assert torch.allclose(out.cpu().double(), want, atol=tol, rtol=tol), (act, first)


@pytest.mark.parametrize("E, top, count, keep", [(12, 3, 4, 2), (16, 4, 4, 3), (7, 3, 1, 1), (40, 5, 8, 2), (6, 6, 3, 3), (9, 1, 9, 4), (64, 8, 4, 1), (2, 1, 2, 1), (200, 6, 5, 2)])
def test_sigmoid_scores_with_a_correction_and_groups(E, top, count, keep):
    """Choice by score + correction (scores that are negative too), groups by the sum of their two best, weights without the
    correction times a scale; the lower index among equals."""
    from kuiperllama_b200.csrc import ops
    g = torch.Generator().manual_seed(E)
    z = torch.randn(41, E, generator=g) * 2
    corr = torch.randn(E, generator=g) - 0.8
    z[3, :], tie = 0.25, torch.zeros(E)                        # equal scores (for the run without a correction)
    for c in (corr, tie):
        choice, weight = ops.moe_route(z.to(DEV), top, False, count, keep, scores="sigmoid", correction=c.to(DEV), group_top=2, scale=1.7)
        idx, w = P.route(z.double(), torch.eye(E, dtype=torch.float64), c.double(), {"experts": E, "top": top, "scale": 1.7, "groups": {"count": count, "keep": keep}})
        margin = P.route_margin(z.double(), torch.eye(E, dtype=torch.float64), c.double(), {"experts": E, "top": top, "groups": {"count": count, "keep": keep}})
        for t in range(41):
            if float(margin[t]) < 1e-5 and not (t == 3 and c is tie):
                continue
            assert choice[t].tolist() == idx[t].tolist(), (t, c is tie)
            assert torch.allclose(weight[t].cpu().double(), w[t], atol=1e-6, rtol=1e-5)


@pytest.mark.parametrize("n, hidden, inter", [(3, 64, 72), (40, 100, 50), (9, 128, 64), (70, 192, 256), (300, 256, 192), (700, 64, 128), (1100, 128, 320)])
def test_the_gelu_gate_inside_the_product(n, hidden, inter):
    """gelu(W_gate x) * (W_up x): the kernel after the product (both dtypes) and the tensor-core products' epilogues."""
    from kuiperllama_b200.csrc import ops
    g = torch.Generator().manual_seed(n)
    x, gate, up = torch.randn(n, hidden, generator=g), 2 * torch.randn(inter, hidden, generator=g) / hidden ** 0.5, torch.randn(inter, hidden, generator=g) / hidden ** 0.5
    for dt in (torch.float32, torch.bfloat16):
        xd, gd, ud = x.to(dt), gate.to(dt), up.to(dt)
        want = P.gelu_tanh(xd.double() @ gd.double().T) * (xd.double() @ ud.double().T)
        tol = 2e-5 if dt == torch.float32 else 4e-2
        rows = (xd.to(DEV) @ torch.cat([gd, ud]).to(DEV).T) if dt == torch.bfloat16 else (xd.double() @ torch.cat([gd, ud]).double().T).float().to(DEV)
        out = torch.empty(n, inter, dtype=dt, device=DEV)
        ops.swiglu(rows.contiguous(), out, activation="gelu_tanh")
        assert torch.allclose(out.cpu().double(), want, atol=tol, rtol=tol), dt
        if ops.swiglu_fusable(hidden, inter, dt):
            w = ops.interleave_gate_up(gd, ud).to(DEV)
            for fn in ((ops.gemm_skinny, ops.gemm_tcgen05) if n <= 512 else (ops.gemm_tcgen05,)):
                out.zero_()
                fn(xd.to(DEV), w, out, swiglu=True, activation="gelu_tanh")
                ops.check_status(torch.device(DEV))
                assert torch.allclose(out.cpu().double(), want, atol=tol, rtol=tol), fn.__name__


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("hidden", [40, 101, 256, 2048, 2052, 8192])
def test_the_norm_of_two_results_in_both_forms(dtype, hidden):
    """x += d1 + d2 and the norms of the sum, few rows and many, rows and float32 pieces, one output and two."""
    from kuiperllama_b200.csrc import ops
    dt = getattr(torch, dtype)
    g = torch.Generator().manual_seed(hidden)
    for n in (3, 300):
        x = torch.randn(n, hidden, generator=g)
        d1, d2 = torch.randn(n, hidden, generator=g).to(dt), torch.randn(5, n, hidden, generator=g)
        w1, w2 = 1 + 0.2 * torch.randn(hidden, generator=g), 1 + 0.2 * torch.randn(hidden, generator=g)
        xd = x.to(DEV).clone()
        o1, o2 = (torch.empty(n, hidden, dtype=dt, device=DEV) for _ in range(2))
        ops.pair_rmsnorm(xd, (d1.to(DEV), d2.to(DEV)), w1.to(DEV), w2.to(DEV), o1, o2, 1e-5)
        s = x.double() + d1.double() + d2.double().sum(0)
        assert torch.allclose(xd.cpu().double(), s, atol=1e-5, rtol=1e-5)
        tol = 1e-5 if dtype == "float32" else 2e-2
        for o, w in ((o1, w1), (o2, w2)):
            assert torch.allclose(o.cpu().double(), P.rms_norm(s, w.double(), 1e-5), atol=tol, rtol=tol)
        rows = torch.tensor([n - 1, 0], dtype=torch.int32, device=DEV)
        x2 = x.to(DEV).clone()
        o = torch.empty(2, hidden, dtype=dt, device=DEV)
        ops.pair_rmsnorm(x2, (d2.to(DEV), d1.to(DEV)), w1.to(DEV), None, o, None, 1e-5, rows)
        assert torch.equal(x2.cpu(), x) and torch.allclose(o.cpu().double(), P.rms_norm(s, w1.double(), 1e-5)[[n - 1, 0]], atol=tol, rtol=tol)


# ----------------------------------------------------------------------------- each mechanism alone, layer by layer

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["only_attention", "only_mlstm", "only_dense", "only_moe", "only_v_mix"])
def test_one_mechanism_alone(models, name, dtype):
    model, folder = models(name, dtype, seed=3)
    toks = tokens(90, CONFIGS[name]["vocab"], seed=11)
    ref = oracle_logits(folder, toks)
    assert_logits(_run_in_steps(_engine(model), toks, [90]), ref, dtype, f"{name}: whole")
    assert_logits(_run_in_steps(_engine(model), toks, [1] * 90), ref, dtype, f"{name}: token by token")


def test_the_stream_after_every_layer(models):
    """float32: the residual stream after each layer against the plain implementation's, so that a fault is named by its layer."""
    from kuiperllama_b200.csrc import ops
    from kuiperllama_b200.parts.norm import add_to_stream
    for name in FULL:
        model, folder = models(name, "float32", seed=1)
        c, W = read_folder(folder)
        toks = tokens(90, c["vocab"], seed=12)
        _, streams = P.forward(c, W, toks)
        eng = _engine(model)
        with torch.inference_mode():
            slot = eng.alloc_slot()
            ctx, _, _ = eng._pack([_inputs(slot, toks)], 0)
            residual = torch.empty((ctx.n_tokens, c["width"]), dtype=torch.float32, device=DEV)
            ops.embedding(ctx.token_ids[:ctx.n_tokens], model.embedding, residual, model.error_flag, scale=model.spec.embedding_multiplier,
                          positions=ctx.positions, freq=model.blocks[0].position.embedding_frequencies())
            pending = None
            for i, e in enumerate(model.spec.schedule):
                ctx.next_norm = None
                residual, pending = model.blocks[e.layer].forward(residual, pending, ctx, eng.cache.view(i))
                x = residual.clone()
                add_to_stream(x, pending)
                a, b = x[:90].double().cpu(), streams[i]
                assert float((a - b).abs().max()) <= 1e-4 * float(b.abs().max()), f"{name}: the stream after layer {i} differs"
            eng.free_slot(slot)


# ----------------------------------------------------------------------------- cuts, batches, reuse

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", FULL)
def test_whole_prompt_portions_and_single_tokens(models, name, dtype):
    model, folder = models(name, dtype, seed=1)
    toks = tokens(150, CONFIGS[name]["vocab"], seed=21)
    ref = oracle_logits(folder, toks)
    for cuts in ([150], [118] + [1] * 32, [2] * 75, [63, 1, 2, 62, 3, 1, 1, 17], [1, 64, 64, 21], [5, 59, 2, 84], [31, 32, 33, 54]):
        assert sum(cuts) == 150
        assert_logits(_run_in_steps(_engine(model), toks, cuts), ref, dtype, f"{name}: steps of {cuts[:6]}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_long_prompts(models, name, dtype):
    """Prompts of several hundred tokens (chunks left behind), a long portion after a short one and before one, and a long
    prompt beside a short one in one step."""
    model, folder = models(name, dtype, seed=1)
    V = CONFIGS[name]["vocab"]
    toks = tokens(330, V, seed=41)
    ref = oracle_logits(folder, toks)
    for cuts in ([330], [300, 30], [31, 299], [129, 130, 71]):
        assert_logits(_run_in_steps(_engine(model), toks, cuts), ref, dtype, f"{name}: long steps of {cuts}")
    short = tokens(70, V, seed=42)
    eng = _engine(model)
    with torch.inference_mode():
        a, b = eng.alloc_slot(), eng.alloc_slot()
        out = eng.step([_inputs(a, short), _inputs(b, toks)])
    eng.check_device_errors()
    assert_logits(out[:70], oracle_logits(folder, short), dtype, f"{name}: a short prompt beside a long one")
    assert_logits(out[70:], ref, dtype, f"{name}: a long prompt beside a short one")


def test_a_bfloat16_prompt_in_chunks_and_token_by_token(models):
    """The chunked form against the walk over the same weights, so that bfloat16 itself drops out: logits that agree far below
    bfloat16's own rounding of the model where no router changed its mind."""
    from kuiperllama_b200.parts.matrix_recurrent import MLSTMMixer
    model, folder = models("only_mlstm", "bfloat16", seed=1)
    c = CONFIGS["only_mlstm"]
    W = json.loads(json.dumps(c))
    W["layers"][0]["mixer"].update(heads=3, dim=16, vdim=24)                 # sizes the chunked form takes
    import tempfile
    from kuiperllama_b200.engine import load_model
    with tempfile.TemporaryDirectory() as folder:
        write_folder(folder, W, random_weights(W, 4))
        with torch.inference_mode():
            model = load_model(folder, dtype="bfloat16", device=DEV)
        toks = tokens(200, W["vocab"], seed=5)
        try:
            MLSTMMixer.KERNEL = "walk"
            walk = _run_in_steps(_engine(model), toks, [200])
        finally:
            MLSTMMixer.KERNEL = "chunked"
        for cuts in ([200], [100, 100], [33, 167]):
            got = _run_in_steps(_engine(model), toks, cuts)
            err = (got - walk).pow(2).mean(-1).sqrt() / walk.std(-1)
            assert float(err.quantile(0.9)) < 5e-3 and float(err.max()) < 5e-2, (cuts, float(err.max()))


@pytest.mark.parametrize("use_graphs", [False, True])
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", FULL)
def test_unequal_batches_against_each_alone(models, name, dtype, use_graphs):
    """Requests of 1 to 130 tokens in one step, then decoded together, the shorter ones leaving first."""
    model, folder = models(name, dtype, seed=1)
    V = CONFIGS[name]["vocab"]
    lens, more = [1, 3, 70, 130, 64], [2, 9, 5, 9, 7]
    seqs = [tokens(n + m, V, seed=30 + i) for i, (n, m) in enumerate(zip(lens, more))]
    refs = [oracle_logits(folder, s) for s in seqs]
    eng = _engine(model, max_tokens=64 * 12, use_graphs=use_graphs)
    with torch.inference_mode():
        slots = [eng.alloc_slot() for _ in seqs]
        got = [[] for _ in seqs]
        out = eng.step([_inputs(sl, s[:n]) for sl, s, n in zip(slots, seqs, lens)])
        at = 0
        for i, n in enumerate(lens):
            got[i].append(out[at:at + n].clone())
            at += n
        for k in range(max(more)):
            live = [i for i in range(len(seqs)) if k < more[i]]
            if use_graphs:
                out = eng.decode_step([slots[i] for i in live], [seqs[i][lens[i] + k] for i in live]).clone()
            else:
                out = eng.step([_inputs(slots[i], [seqs[i][lens[i] + k]]) for i in live])
            for j, i in enumerate(live):
                got[i].append(out[j:j + 1].clone())
            for i in live:
                if k + 1 == more[i]:
                    eng.free_slot(slots[i])
    eng.check_device_errors()
    for i in range(len(seqs)):
        assert_logits(torch.cat(got[i]), refs[i], dtype, f"{name}: request {i} of the batch")
    assert eng.cache.slots.held() == 0 and all(h == 0 for h in eng.cache.pages_held())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_small_steps_from_graphs_and_padding_rows(models, name, dtype):
    """Short prompts through captured steps (rows padded to 64) one after another, and a decode step with padding rows: rows that
    belong to no sequence change nothing, and nothing of one replay reaches the next."""
    model, folder = models(name, dtype, seed=1)
    V = CONFIGS[name]["vocab"]
    eng = _engine(model, max_tokens=64 * 12, use_graphs=True)
    for k, n in enumerate((40, 17, 64, 33)):
        toks = tokens(n + 6, V, seed=140 + k)
        with torch.inference_mode():
            slot = eng.alloc_slot()
            rows = [eng.step([_inputs(slot, toks[:n], [0, n - 1])]).clone(), eng.step([_inputs(slot, toks[n:n + 3])]).clone()]
            rows += [eng.step([_inputs(slot, [t])], pad_rows=5).clone() for t in toks[n + 3:]]
            eng.free_slot(slot)
        eng.check_device_errors()
        ref = oracle_logits(folder, toks)
        ref = torch.cat([ref[[0, n - 1]], ref[n:]])
        assert_logits(torch.cat(rows), ref, dtype, f"{name}: prompt of {n} from a graph")


@pytest.mark.parametrize("dtype", DTYPES)
def test_slots_and_pages_are_reused(models, dtype):
    """A cache with room for little: four rounds of requests on the same slots, pages and states, whose old contents must not leak
    into the next request."""
    model, folder = models("mixed", dtype, seed=1)
    V = CONFIGS["mixed"]["vocab"]
    eng = _engine(model, max_tokens=64 * 5)
    for rnd in range(4):
        lens = [[100, 70], [3, 129], [64, 65], [1, 2]][rnd]
        seqs = [tokens(n + 3, V, seed=50 + 10 * rnd + i) for i, n in enumerate(lens)]
        with torch.inference_mode():
            slots = [eng.alloc_slot() for _ in seqs]
            first = eng.step([_inputs(sl, s[:n]) for sl, s, n in zip(slots, seqs, lens)])
            rest = [eng.step([_inputs(sl, [s[n + k]]) for sl, s, n in zip(slots, seqs, lens)]).clone() for k in range(3)]
            for sl in slots:
                eng.free_slot(sl)
        at = 0
        for i, (s, n) in enumerate(zip(seqs, lens)):
            got = torch.cat([first[at:at + n]] + [r[i:i + 1] for r in rest])
            at += n
            assert_logits(got, oracle_logits(folder, s), dtype, f"round {rnd}, request {i}")
    eng.check_device_errors()
    assert all(g.held() == 0 for g in eng.cache.groups)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_the_first_tokens_of_a_sequence(models, name, dtype):
    """Prompts of one to five tokens and what follows token by token and in small portions: the maximum that starts at zero, chunks
    of one and two positions, the sinusoid's first entries."""
    model, folder = models(name, dtype, seed=1)
    V = CONFIGS[name]["vocab"]
    for n in (1, 2, 3, 4, 5):
        toks = tokens(n + 8, V, seed=60 + n)
        assert_logits(_run_in_steps(_engine(model), toks, [n] + [1] * 8), oracle_logits(folder, toks), dtype, f"{name}: prompt of {n}")
        assert_logits(_run_in_steps(_engine(model), toks, [n, 2, 2, 4]), oracle_logits(folder, toks), dtype, f"{name}: prompt of {n}, portions")


@pytest.mark.parametrize("dtype", DTYPES)
def test_chunks_pass_over_decoded_tokens(models, dtype):
    """Chunks of 64, 96 and 127 positions: a prompt shorter than every chunk followed by 340 single tokens from captured decode
    steps, so that every chunk's edge falls among decoded tokens, on and off page borders, and pages of chunks left behind go back."""
    model, folder = models("chunks", dtype, seed=1)
    toks = tokens(400, CONFIGS["chunks"]["vocab"], seed=70)
    ref = oracle_logits(folder, toks)
    eng = _engine(model, max_tokens=64 * 8, use_graphs=True)
    with torch.inference_mode():
        slot = eng.alloc_slot()
        rows = [eng.step([_inputs(slot, toks[:60])]).clone()]
        held = []
        for t in toks[60:]:
            rows.append(eng.decode_step([slot], [t]).clone())
            held.append(max(eng.cache.pages_held()))
        eng.free_slot(slot)
    eng.check_device_errors()
    assert_logits(torch.cat(rows), ref, dtype, "chunks: long decoding")
    assert max(held) <= 4, f"pages of chunks left behind were kept: {max(held)}"
    for cuts in ([400], [149, 1, 1, 1, 148, 100], [96, 96, 1, 95, 112], [127, 1, 126, 146], [20, 1, 129, 250], [63, 2, 62, 2, 271]):
        assert_logits(_run_in_steps(_engine(model), toks, cuts), ref, dtype, f"chunks: steps of {cuts}")


# ----------------------------------------------------------------------------- what random weights would hide

def _needle_folder(tmp_path_factory, size, pairs, T, seed=9):
    """One attention layer whose weights are made so that chosen queries read single keys.  Keys read the first d coordinates of
    the normed row; ordinary tokens have next to nothing there (a large eps keeps the norm over k from blowing that up), a needle
    token B has entries of +-2.5, and the query token A's embedding is a rotation R^T of B's while every head's query map is (its
    key map) R: A's query points along B's key, and scores much on it wherever B lies, if the mask lets it.  ``pairs`` lists
    (query position, needle positions); every pair has token ids of its own."""
    d, width, V = 32, 64, 40 + 2 * len(pairs)
    layer = {"type": "attention", "mixer": {"heads": 4, "kv_heads": 2, "dim": d, "vdim": 64, "scale": 0.8, "bias_max": 40, "mask": {"size": size},
                                            "v_mix": False, "rel_rows": 16}, "mlp": None}
    c = {"architecture": "Vepolix", "vocab": V, "width": width, "norm": {"eps": 1.0}, "embedding": {"scale": 30.0}, "layers": [layer]}
    W = {k: v.float() for k, v in random_weights(c, seed).items()}
    g = torch.Generator().manual_seed(12)
    R = torch.linalg.qr(torch.randn(width, width, generator=g, dtype=torch.float64)).Q
    W["l0.norm1"], W["l0.mix.q.norm"], W["l0.mix.k.norm"] = torch.ones(width), torch.ones(4 * d), torch.ones(2 * d)
    W["l0.mix.rel"] = 0.3 * W["l0.mix.rel"]
    W["embed"][:, :d] = 0.0
    eye = torch.zeros(d, width, dtype=torch.float64)
    eye[:, :d] = torch.eye(d, dtype=torch.float64)
    W["l0.mix.k"] = torch.cat([eye] * 2).float()
    W["l0.mix.q"] = torch.cat([eye @ R] * 4).float()
    W["l0.mix.o"] = 4.0 * W["l0.mix.o"]
    toks = tokens(T, V - 2 * len(pairs), seed=80)                        # the last ids of the vocabulary are kept for the pairs
    for i, (query_at, needles_at) in enumerate(pairs):
        a, b = V - 1 - 2 * i, V - 2 - 2 * i
        e = torch.randn(width, generator=g, dtype=torch.float64)
        e[:d] = 2.5 * torch.sign(torch.randn(d, generator=g, dtype=torch.float64))
        W["embed"][b] = e.float()
        W["embed"][a] = (R.T @ e).float()
        toks[query_at] = a
        for p in needles_at:
            toks[p] = b
    # the stream carries 30 times the embedding, the layer adds numbers around one: the head reads what the layer wrote
    W["head"] = 8.0 * W["head"]
    W = {k: v.to(torch.bfloat16) for k, v in W.items()}
    return write_folder(str(tmp_path_factory.mktemp("vepolix-needle")), c, W), toks, V


def _check_needles(folder, toks, V, seen, unseen):
    """The plain implementation proves which needles are read: taking a pair's needle tokens away changes the query's logits by
    much where they are seen, and by nothing at all where they are not."""
    ref = oracle_logits(folder, toks)
    for i, (qa, needles) in enumerate(seen + unseen):
        b = V - 2 - 2 * i
        without = [0 if (t == b) else t for t in toks]
        other = oracle_logits(folder, without)
        diff = float((ref[qa] - other[qa]).abs().max()) / float(ref[qa].std())
        if i < len(seen):
            assert diff > 0.1, f"the query at {qa} does not read its needle at {needles}: {diff:.3e}"
        else:
            assert diff == 0.0, f"the query at {qa} reads its needle at {needles}: {diff:.3e}"
    return ref


@pytest.mark.parametrize("dtype", DTYPES)
def test_keys_at_the_edges_of_a_chunk_show(tmp_path_factory, dtype):
    """Chunks of 150.  Queries whose one key is the chunk's first (seen), the last of the chunk before (not seen), at a page's last
    and first place inside the chunk, right before the query, and far away.  Then prompts, portions that end at the edges, and
    decoding over them."""
    from kuiperllama_b200.engine import load_model
    T = 460
    seen = [(200, [150]), (298, [151]), (340, [319]), (345, [320]), (330, [329]), (447, [300]), (148, [0]), (459, [450])]
    unseen = [(210, [149]), (305, [299]), (400, [100]), (415, [3]), (152, [1]), (455, [449])]
    folder, toks, V = _needle_folder(tmp_path_factory, 150, seen + unseen, T)
    ref = _check_needles(folder, toks, V, seen, unseen)
    rows = [q for q, _ in seen + unseen]
    with torch.inference_mode():
        model = load_model(folder, dtype=dtype, device=DEV)
    for cuts in ([T], [150, 150, 150, 10], [149, 1, 1, 149, 149, 11], [200, 10, 20, 70, 1, 19, 80, 60], [64, 128, 8, 1, 199, 60], [140] + [1] * 320, [2] * 230):
        assert_logits(_run_in_steps(_engine(model), toks, cuts), ref, dtype, f"edges: steps of {cuts[:5]}", rows)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size, bias_max, rows", [(90, 40, 16), (None, 25, 7), (64, 500, 32), (130, 3, 8)])
def test_the_bias_alone_weighs_the_keys(tmp_path_factory, dtype, size, bias_max, rows):
    """Keys of zero: every weight comes from the table alone, whose rows differ by so much that a distance in the wrong bucket
    shows.  ``scale`` must not touch the bias."""
    from kuiperllama_b200.engine import load_model
    c = json.loads(json.dumps(CONFIGS["only_attention"]))
    c["layers"][0]["mixer"].update(dim=32, vdim=64, bias_max=bias_max, rel_rows=rows, scale=0.01, mask=None if size is None else {"size": size})
    W = random_weights(c, 5)
    W["l0.mix.k"] = torch.zeros_like(W["l0.mix.k"])
    g = torch.Generator().manual_seed(3)
    W["l0.mix.rel"] = (2.5 * torch.randn(W["l0.mix.rel"].shape, generator=g)).to(torch.bfloat16)
    folder = write_folder(str(tmp_path_factory.mktemp("vepolix-bias")), c, W)
    toks = tokens(200, c["vocab"], seed=81)
    ref = oracle_logits(folder, toks)
    with torch.inference_mode():
        model = load_model(folder, dtype=dtype, device=DEV)
    for cuts in ([200], [1] * 200, [7, 93, 100]):
        assert_logits(_run_in_steps(_engine(model), toks, cuts), ref, dtype, f"bias {size}, {bias_max}: steps of {cuts[:3]}", rows=range(200))


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_far_token_only_the_memory_can_remember(tmp_path_factory, dtype):
    """A memory whose forget gates stay open and whose input gates open for one token id alone: that token is read hundreds of
    tokens later, across portions, chunks and decoded tokens; the plain implementation proves that it is."""
    from kuiperllama_b200.engine import load_model
    c = json.loads(json.dumps(CONFIGS["only_mlstm"]))
    c["layers"][0]["mixer"].update(heads=2, dim=16, vdim=24, gate_cap=12.0)
    c["embedding"]["scale"] = 20.0
    W = {k: v.float() for k, v in random_weights(c, 6).items()}
    V, T = c["vocab"], 420
    needle = V - 1
    W["l0.norm1"] = torch.ones(64)
    W["embed"][:, 0] = 0.0
    W["embed"][needle] *= 0.3
    W["embed"][needle, 0] = 6.0
    W["l0.mix.i"], W["l0.mix.f"] = torch.zeros(2, 64), torch.zeros(2, 64)
    W["l0.mix.i"][:, 0] = 2.0                                           # ordinary tokens: i = -6; the needle: far above
    W["l0.mix.i.b"], W["l0.mix.f.b"] = torch.full((2,), -6.0), torch.full((2,), 11.0)
    W["l0.mix.o"], W["head"] = 6.0 * W["l0.mix.o"], 4.0 * W["head"]
    folder = write_folder(str(tmp_path_factory.mktemp("vepolix-memory")), c, {k: v.to(torch.bfloat16) for k, v in W.items()})
    toks = tokens(T, V - 1, seed=82)
    plain = list(toks)
    toks[5] = needle
    ref, other = oracle_logits(folder, toks), oracle_logits(folder, plain)
    rows = [100, 200, 300, 400, 419]
    for r in rows:
        assert float((ref[r] - other[r]).pow(2).mean().sqrt()) > 0.1 * float(ref[r].std()), f"the token at {r} does not remember"
    with torch.inference_mode():
        model = load_model(folder, dtype=dtype, device=DEV)
    for cuts in ([T], [4, 2, 300, 114], [64] * 6 + [36], [150] + [1] * 270, [2] * 210):
        assert_logits(_run_in_steps(_engine(model), toks, cuts), ref, dtype, f"memory: steps of {cuts[:4]}", rows)


@pytest.mark.parametrize("dtype", DTYPES)
def test_mixed_values_take_their_share(tmp_path_factory, dtype):
    """Factors of 0, 1 and -0.5 in the later layers, and a factor in the first one that nobody may read."""
    from kuiperllama_b200.engine import load_model
    c = json.loads(json.dumps(CONFIGS["only_v_mix"]))
    toks = tokens(60, c["vocab"], seed=83)
    refs = []
    for lam in (0.0, 1.0, -0.5):
        for unread in (0.0, 0.9):
            W = random_weights(c, 5)
            W["l0.mix.vmix"] = torch.tensor(unread).to(torch.bfloat16)
            W["l1.mix.vmix"], W["l2.mix.vmix"] = torch.tensor(lam).to(torch.bfloat16), torch.tensor(0.5 * lam).to(torch.bfloat16)
            folder = write_folder(str(tmp_path_factory.mktemp("vepolix-vmix")), c, W)
            ref = oracle_logits(folder, toks)
            with torch.inference_mode():
                model = load_model(folder, dtype=dtype, device=DEV)
            for cuts in ([60], [1] * 60, [7, 53]):
                assert_logits(_run_in_steps(_engine(model), toks, cuts), ref, dtype, f"vmix {lam}: steps of {cuts[:3]}", rows=range(60))
        refs.append(ref)
    assert float((refs[0] - refs[1]).abs().max()) > 0.1 * float(refs[1].std()), "the factor changes nothing: the test shows nothing"


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_from_graphs(models, dtype):
    """400 tokens one by one through captured decode steps after a prompt of five: chunks, pages and states of every layer."""
    model, folder = models("mixed", dtype, seed=1)
    toks = tokens(405, CONFIGS["mixed"]["vocab"], seed=70)
    eng = _engine(model, max_tokens=64 * 8, use_graphs=True)
    with torch.inference_mode():
        slot = eng.alloc_slot()
        rows = [eng.step([_inputs(slot, toks[:5])]).clone()]
        for t in toks[5:]:
            rows.append(eng.decode_step([slot], [t]).clone())
        eng.free_slot(slot)
    eng.check_device_errors()
    assert_logits(torch.cat(rows), oracle_logits(folder, toks), dtype, "long decoding")


# ----------------------------------------------------------------------------- the entry points

def _greedy(c, W, prompt, n):
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(P.forward(c, W, seq)[0][-1].argmax()))
    return seq[len(prompt):]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_greedy_generation_through_the_entry_point(folders, name, dtype):
    """``load(...).generate``: scheduler, batches that reuse slots, captured decode steps, sampler.  float32 gives the plain greedy
    tokens (where the plain logits' two best are apart); in bfloat16 a token may differ where they are close, and the run is
    compared up to there."""
    import kuiperllama_b200 as kl
    folder = folders(name, seed=1)
    c, W = read_folder(folder)
    prompts = [tokens(n, c["vocab"], seed=90 + n) for n in (7, 1, 66, 20, 3)]
    m = kl.load(folder, dtype=dtype, device=DEV, max_tokens=64 * 8, max_batch=2)
    got = m.generate(prompts, max_new_tokens=10, stop_ids=[])
    for p, out in zip(prompts, got):
        assert len(out) == 10
        seq = list(p)
        for tok in out:
            logits = P.forward(c, W, seq)[0][-1]
            top = torch.topk(logits, 2).values
            if int(logits.argmax()) != tok:
                close = float(top[0] - top[1]) < (1e-3 if dtype == "float32" else 0.15) * float(logits.std())
                assert close and float(logits[tok]) >= float(top[1]) - 1e-9, f"{name} {dtype}: token {tok} is not the plain greedy token"
                break
            seq.append(tok)


def test_cli_runs_a_vepolix_folder(folders, capsys):
    from kuiperllama_b200.cli import main
    folder = folders("mixed", seed=1)
    assert main([folder, "--prompt-ids", "1,2,3", "--max-new-tokens", "4", "--dtype", "float32", "--stop-ids", ""]) == 0
    out = capsys.readouterr().out
    c, W = read_folder(folder)
    assert " ".join(str(t) for t in _greedy(c, W, [1, 2, 3], 4)) in out


def test_trace_run_replays_a_vepolix_folder(folders, tmp_path):
    """bin/trace_run as a user runs it, in float32: five requests in one step, then two steps of a token each with the
    shortest leaving first.  The folder's config.json does not name the bias tables' rows: they come from the tensors."""
    import os
    import shutil
    import subprocess
    import sys

    import numpy as np
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    source = folders("mixed", seed=1)
    folder = str(tmp_path / "model")
    shutil.copytree(source, folder)
    c, _ = read_folder(source)
    for l in c["layers"]:
        l["mixer"].pop("rel_rows", None)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(c, f)
    V = c["vocab"]
    lens = [1, 3, 65, 2, 66]
    seqs = [tokens(n + 2, V, seed=110 + i) for i, n in enumerate(lens)]
    steps = [{"step": 0, "entries": [{"id": f"r{i}", "tokens": s[:n], "want": [n - 1]} for i, (s, n) in enumerate(zip(seqs, lens))], "end": []},
             {"step": 1, "entries": [{"id": f"r{i}", "tokens": [s[n]], "want": [0]} for i, (s, n) in enumerate(zip(seqs, lens))], "end": ["r0"]},
             {"step": 2, "entries": [{"id": f"r{i}", "tokens": [s[n + 1]], "want": [0]} for i, (s, n) in enumerate(zip(seqs, lens)) if i],
              "end": [f"r{i}" for i in range(1, 5)]}]
    out = str(tmp_path / "out")
    cmd = [sys.executable, os.path.join(root, "bin", "trace_run"), "--model", folder, "--dtype", "float32", "--out", out,
           "--max-tokens", str(sum(lens) + 2 * len(lens))]
    p = subprocess.run(cmd, input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-3000:]
    assert [l for l in p.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    refs = [oracle_logits(source, s) for s in seqs]
    read = lambda k: torch.from_numpy(np.fromfile(os.path.join(out, f"{k}.f32"), dtype="<f4").reshape(-1, V).copy())
    assert_logits(read(0), torch.stack([r[n - 1] for r, n in zip(refs, lens)]), "float32", "replay: prompts")
    assert_logits(read(1), torch.stack([r[n] for r, n in zip(refs, lens)]), "float32", "replay: first tokens")
    assert_logits(read(2), torch.stack([r[n + 1] for r, n in list(zip(refs, lens))[1:]]), "float32", "replay: second tokens")
