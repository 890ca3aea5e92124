"""The kernels that the Gevipel design added or widened, each alone against a float64 restatement of its own operation
written here: the embedding's multiplier, branches joining the stream behind norms of either kind, values read from the
keys' columns, scores that fall with the distance in all four attention kernels (window edges, page borders, far keys,
with and without caps, sinks and windows), sinks in both latent kernels, the square of relu in the experts' products, and
the gated delta rule with one decay per head (whole, in portions around the chunks' borders, token by token, batches of
unequal sequences, key heads shared by value heads, decays of exactly one and of zero, a write that must be read back after
hundreds of tokens)."""
import numpy as np
import pytest
import torch

from test_gpu_lavutar_kernels import BF16_ULP, DEV, Pages, _blocks, _close, _i32, _ops, _rand
from test_gpu_zoporax_kernels import _blocks_for, _paged, _rel

pytestmark = pytest.mark.gpu


def _d(x):
    return x.double().cpu()


def _rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


# ------------------------------------------------------------------ the stream

@pytest.mark.parametrize("table_dtype", [torch.float32, torch.bfloat16])
def test_embedding_rows_are_multiplied(table_dtype):
    ops = _ops()
    table, toks = _rand((50, 44), table_dtype, 1, 3.0), [3, 49, 0, 3]
    _close(ops.embedding(table, _i32(toks), scale=2.75), _d(table)[toks] * 2.75, 1e-6)
    assert torch.equal(ops.embedding(table, _i32(toks)), table[toks].float())


def _norm(x, n):
    w, b, eps, center = n
    if center:
        x = x - x.mean(-1, keepdim=True)
    return _rms(x, eps) * _d(w) + (0.0 if b is None else _d(b))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("D", [1, 44, 190, 192, 1000, 2048, 4100, 9000])
def test_branches_join_the_stream_behind_norms_of_either_kind(D, dtype):
    """Layer norms and RMS norms on either side, a multiplier, rows that join as well, with and without the next norm's rows;
    a branch and a stream whose means are far from zero."""
    ops = _ops()
    T = 5
    y, x0, e = _rand((T, D), torch.float32, 1, 0.5) + 4.0, _rand((T, D), torch.float32, 3) - 3.0, _rand((T, D), torch.float32, 4)
    w1, w2 = _rand((D,), torch.float32, 5) + 1.0, _rand((D,), torch.float32, 6) + 1.0
    b1, b2 = _rand((D,), torch.float32, 7), _rand((D,), torch.float32, 8)
    layer1, layer2, rms1, rms2 = (w1, b1, 1e-5, True), (w2, b2, 1e-4, True), (w1, None, 1e-6, False), (w2, None, 1e-3, False)
    for first, second, m, extra in ((layer1, layer2, 0.3, None), (layer1, layer2, 1.0, e), (rms1, layer2, -0.7, e), (layer1, rms2, 0.3, None),
                                    (rms1, rms2, 2.0, None), (layer1, None, 0.5, e), (rms1, None, 0.5, None)):
        want = _d(x0) + m * _norm(_d(y), first) + (0.0 if extra is None else _d(extra))
        x = x0.clone()
        h = ops.join_branch(x, y, first, m, extra, second, dtype)
        _close(x, want, 1e-5)
        if second is None:
            assert h is None
        elif D > 1:
            assert h.dtype == dtype
            _close(h, _norm(want, second), 2e-5 if dtype == torch.float32 else 1.5 * BF16_ULP, 0.0 if dtype == torch.float32 else BF16_ULP)


# ------------------------------------------------------------------ attention whose values are the keys, at a distance

@pytest.mark.parametrize("in_dtype,out_dtype", [(torch.float32, torch.float32), (torch.float32, torch.bfloat16)])
@pytest.mark.parametrize("H,G,hd", [(4, 2, 32), (3, 1, 26), (2, 2, 64)])
def test_values_are_the_keys_as_projected(in_dtype, out_dtype, H, G, hd):
    """Rows of q and k alone: queries and keys leave normed per head with a weight and (queries) with their temperature, the
    values are the keys' columns as they came -- also where the queries are written back into the rows."""
    ops = _ops()
    T, page, eps, temp = 70, 64, 1e-5, (0.4, 9)
    rows = _rand((T, (H + G) * hd), in_dtype, 1)
    raw = _d(rows)
    w = _rand(((H + G) * hd,), torch.float32, 2) + 1.0
    k_pages = torch.zeros((3, G, page, hd), dtype=out_dtype, device=DEV)
    v_pages = torch.zeros_like(k_pages)
    table = _i32([[2, 0]])
    q = torch.empty((T, H * hd), dtype=out_dtype, device=DEV) if in_dtype != out_dtype else rows
    ops.rope_partial(rows, None, None, None, 0, _i32(list(range(T))), _i32([0] * T), _i32([0]), table, k_pages, v_pages, H + G, H, G, hd, hd,
                     H * hd, page, qout=None if q is rows else q, unit_norm="head", norm_weight=w, norm_eps=eps, q_temp=temp)
    heads = _rms(raw.reshape(T, H + G, hd), eps) * _d(w).reshape(H + G, hd)
    t = 1.0 + temp[0] * torch.log(torch.floor((torch.arange(T, dtype=torch.float64) + 1) / temp[1]) + 1.0)
    tol, rel = (3e-6, 0.0) if out_dtype == torch.float32 else (1.5 * BF16_ULP, BF16_ULP)
    _close(q[:, :H * hd].reshape(T, H, hd), heads[:, :H] * t[:, None, None], tol, rel)
    for p in range(T):
        pg = [2, 0][p // page]
        _close(k_pages[pg, :, p % page], heads[p, H:], tol, rel)
        _close(v_pages[pg, :, p % page], raw[p, H * hd:].reshape(G, hd), tol, rel)


def _far_reference(case, q, tok_seq, tok_pos, H, scale, slope, window=None, cap=None, sink=None):
    """Softmax over the keys j of the window with slope_h (p - j) taken off the (capped) scores."""
    out = torch.empty((q.shape[0], H, case.vd), dtype=torch.float64)
    per = H // case.G
    for r in range(q.shape[0]):
        s, p = tok_seq[r], tok_pos[r]
        lo = max(0, p - window + 1) if window else 0
        k, v = _d(case.k[s][lo:p + 1]), _d(case.v[s][lo:p + 1])
        sc = torch.einsum("jgd,gd->gj", k.repeat_interleave(per, 1).transpose(0, 1).transpose(0, 1), _d(q[r])) * scale
        if cap:
            sc = cap * torch.tanh(sc / cap)
        sc = sc - _d(slope)[:, None] * torch.arange(p - lo, -1, -1, dtype=torch.float64)
        if sink is not None:
            sc = torch.cat([sc, _d(sink)[:, None]], 1)
        w = torch.softmax(sc, 1)
        out[r] = torch.einsum("gj,jgv->gv", w[:, :p + 1 - lo], v.repeat_interleave(per, 1))
    return out


# H, G, hd, window, cap, sink
FAR = [(4, 2, 64, 40, None, False), (2, 2, 64, None, None, True), (8, 2, 128, 100, None, False), (3, 3, 128, None, 5.0, True), (6, 3, 48, 70, None, True),
       (4, 1, 16, None, 3.0, False), (20, 1, 32, 200, None, False), (5, 5, 80, 1, None, False), (2, 1, 112, 64, None, False)]


def _slopes(H):
    """From falling steeply to hardly at all."""
    return torch.tensor([0.7 * 0.3 ** h for h in range(H)], dtype=torch.float32, device=DEV)


@pytest.mark.parametrize("H,G,hd,window,cap,sink", FAR)
def test_scores_fall_with_the_distance_in_prompts(H, G, hd, window, cap, sink):
    """One sequence whole from its first token, one single token, one that goes on after 270 cached tokens: on tcgen05 (one
    and two heads a block), on mma.sync, and on the plain kernel."""
    ops = _ops()
    lens, new, past = [300, 1, 400], [300, 1, 130], [0, 0, 270]
    case = Pages(lens, G, hd, hd, torch.bfloat16, seed=5, poison=0.0)
    tok_seq = [b for b, n in enumerate(new) for _ in range(n)]
    tok_pos = [p + i for n, p in zip(new, past) for i in range(n)]
    q, slope = _rand((sum(new), H * hd), torch.bfloat16, 73), _slopes(H)
    sinks = _rand((H,), torch.float32, 74) if sink else None
    scale = 1.3 * hd ** -0.5
    ref = _far_reference(case, q.reshape(-1, H, hd), tok_seq, tok_pos, H, scale, slope, window, cap, sinks)
    args = (q, case.k_pages, case.v_pages, case.table)
    more = dict(sink=sinks, softcap=cap, slope=slope)
    outs = [ops.attn_prefill(*args, case.slots, _i32(lens), _blocks(new, past, 64), H, G, hd, 64, scale, window, **more),
            ops.attention_plain(*args, _i32(tok_pos), _i32(tok_seq), case.slots, H, G, hd, 64, scale, window, **more)]
    if hd in (64, 128):
        outs.append(ops.attn_prefill_tc(*args, case.slots, _i32(lens), _blocks(new, past, 128), H, G, hd, 64, scale, window, **more))
    for out in outs:
        _close(out.reshape(-1, H, hd), ref, case.tol(ref), BF16_ULP)


@pytest.mark.parametrize("H,G,hd,window,cap,sink", FAR)
def test_scores_fall_with_the_distance_for_single_tokens(H, G, hd, window, cap, sink):
    """One token per sequence at its end, in equal slices and from work lists, up to 1,500 tokens back."""
    ops = _ops()
    from longbow_quarrel_b200.kernels.attention import MAX_SPLITS, cut_decode_work
    lens = [300, 1, 77, 64, 17, 1500, 33, 201, 200]
    tok_pos, tok_seq = [n - 1 for n in lens], list(range(len(lens)))
    case = Pages(lens, G, hd, hd, torch.bfloat16, seed=3)
    q, slope = _rand((len(lens), H * hd), torch.bfloat16, 71), _slopes(H)
    sinks = _rand((H,), torch.float32, 74) if sink else None
    scale = 0.9 * hd ** -0.5
    ref = _far_reference(case, q.reshape(-1, H, hd), tok_seq, tok_pos, H, scale, slope, window, cap, sinks)
    args = (q, case.k_pages, case.v_pages, case.table, _i32(tok_pos), _i32(tok_seq), case.slots, H, G, hd, 64, scale, window)
    more = dict(sink=sinks, softcap=cap, slope=slope)
    for splits in (1, 3):
        _close(ops.attn_decode(*args, splits, **more).reshape(-1, H, hd), ref, case.tol(ref), BF16_ULP)
    for teams in (9, 40):
        work = cut_decode_work(tok_pos, window or 0, teams)
        out = ops.attn_decode(*args, min(MAX_SPLITS, teams), early_loads=True, work=_i32(work.tolist()), teams=teams, **more)
        _close(out.reshape(-1, H, hd), ref, case.tol(ref), BF16_ULP)
    _close(ops.attention_plain(*args, **more).reshape(-1, H, hd), ref, case.tol(ref), BF16_ULP)


@pytest.mark.parametrize("window", [None, 130])
def test_true_32_bit_attention_with_slopes(window):
    ops = _ops()
    lens = [200]
    case = Pages(lens, 2, 20, 20, torch.float32, seed=9)
    pos = [0, 1, 63, 64, 129, 130, 131, 199]
    q, slope = _rand((len(pos), 4 * 20), torch.float32, 1), _slopes(4)
    ref = _far_reference(case, q.reshape(-1, 4, 20), [0] * len(pos), pos, 4, 0.3, slope, window)
    out = ops.attention_plain(q, case.k_pages, case.v_pages, case.table, _i32(pos), _i32([0] * len(pos)), case.slots, 4, 2, 20, 64, 0.3, window, slope=slope)
    _close(out.reshape(-1, 4, 20), ref, 3e-6)


@pytest.mark.parametrize("kernel", ["tc", "mma", "decode", "plain"])
def test_a_key_outweighs_all_others_up_to_where_its_head_s_slope_has_eaten_it(kernel):
    """A key whose score stands 60 above the others at distance 0, in three heads: one that falls by 1 a position (it loses
    its lead after sixty of them), one by 0.5 (after a hundred and twenty) and one by 2^-8 (it still has it at 400)."""
    ops = _ops()
    n, hd, at = 512, 64, 70
    slope = torch.tensor([1.0, 0.5, 2.0 ** -8], device=DEV)
    case = Pages([n], 3, hd, hd, torch.bfloat16, seed=1, poison=0.0)
    for t in (case.k_pages, case.k[0]):
        t.zero_()
    case.plant(0, at, 60.0 / hd)
    q = torch.ones((n, 3 * hd), dtype=torch.bfloat16, device=DEV)
    args = (q, case.k_pages, case.v_pages, case.table)
    pos = list(range(n))
    if kernel == "tc":
        out = ops.attn_prefill_tc(*args, case.slots, _i32([n]), _blocks([n], [0], 128), 3, 3, hd, 64, 1.0, None, slope=slope)
    elif kernel == "mma":
        out = ops.attn_prefill(*args, case.slots, _i32([n]), _blocks([n], [0], 64), 3, 3, hd, 64, 1.0, None, slope=slope)
    elif kernel == "decode":
        out = ops.attn_decode(*args, _i32(pos), _i32([0] * n), case.slots, 3, 3, hd, 64, 1.0, None, 2, slope=slope)
    else:
        out = ops.attention_plain(*args, _i32(pos), _i32([0] * n), case.slots, 3, 3, hd, 64, 1.0, None, slope=slope)
    out = _d(out).reshape(n, 3, hd)
    want = _d(case.v[0][at])
    for h, (near, far) in enumerate(((50, 70), (100, 140), (441, None))):
        for p, same in ((at, True), (at + near, True), (at - 1, False), *(((at + far, False),) if far else ())):
            assert (float((out[p, h] - want[h]).abs().max()) < 3e-2 * float(want[h].abs().max())) == same, (h, p)


# ------------------------------------------------------------------ sinks over latent rows

def _sunk(q, rows, pos, R, scale, sink):
    s = rows[:pos + 1] @ q.T * scale
    p = torch.softmax(torch.cat([s, sink[None, :]], 0), 0)[:-1]
    return p.T @ rows[:pos + 1, :R]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,R,dr", [(3, 24, 8), (9, 40, 16), (2, 300, 20), (70, 16, 8), (4, 512, 64)])
def test_a_sink_in_both_latent_kernels(dtype, H, R, dr):
    """Prompts, portions and single tokens, whole and in slices; a head whose sink outweighs every key, one whose sink
    counts for nothing, and sinks about as large as the scores."""
    ops = _ops()
    g = torch.Generator().manual_seed(H * 100 + R)
    Dk, page_size = R + dr, 64
    lens = {0: 200, 2: 70, 3: 17}
    rows = {s: torch.randn(n, Dk, generator=g) for s, n in lens.items()}
    pages, table = _paged(rows, Dk, page_size, dtype, 9, seed=H)
    stored = {s: r.to(dtype).double() for s, r in rows.items()}
    slots = [2, 0, 3]
    sink = torch.linspace(-3.0, 6.0, H)
    sink[0], sink[-1] = 50.0, -50.0
    new, past = [70, 117, 17], [0, 83, 0]
    pos = [p for n, b in zip(new, past) for p in range(b, b + n)]
    seq = [i for i, n in enumerate(new) for _ in range(n)]
    q = torch.randn(len(pos), H, Dk, generator=g)
    scale, dsink = 0.3 * Dk ** -0.5, sink.to(DEV)
    pos1, seq1 = [199, 69, 16], [1, 0, 2]

    def check(out, qq, pos, seq, tol, what):
        for t in range(0, len(pos), 7 if len(pos) > 20 else 1):
            ref = _sunk(qq[t].double(), stored[slots[seq[t]]], pos[t], R, scale, sink.double())
            assert float(out[t, 0].abs().max()) < 1e-6, what
            assert _rel(out[t, 1:], ref[1:]) < tol, (what, t)
    for splits in (1, 4):
        if R <= 512 and H < 20:
            out = ops.latent_attention(q.to(DEV), pages, table, _i32(pos), _i32(seq), _i32(slots), H, R, page_size, scale, None, splits, sink=dsink)
            check(out, q, pos, seq, 5e-6, ("plain", splits))
    if dtype == torch.bfloat16:
        qr = q.to(torch.bfloat16)
        out = ops.latent_attention_tc(q.to(DEV), pages, table, _i32(slots), H, R, page_size, scale, None, sink=dsink,
                                      blocks=_blocks_for(new, past, ops.latent_tc_tokens(H)))
        check(out, qr, pos, seq, 6e-3, "tc")
        for splits in (1, 3):
            out = ops.latent_attention_tc(q[:3].contiguous().to(DEV), pages, table, _i32(slots), H, R, page_size, scale, None, sink=dsink,
                                          tok_pos=_i32(pos1), tok_seq=_i32(seq1), splits=splits)
            check(out, qr[:3], pos1, seq1, 6e-3, ("tc", splits))


def test_one_matrix_per_head_stored_in_32_bit_hands_on_bfloat16():
    ops = _ops()
    x, w = _rand((11, 3 * 20), torch.float32, 1), _rand((3, 20, 14), torch.float32, 2)
    out = torch.empty((11, 3 * 14), dtype=torch.bfloat16, device=DEV)
    ops.head_matmul(x, 20, 0, w, out, 14, 0)
    _close(out.reshape(11, 3, 14), torch.einsum("thk,hkn->thn", _d(x).reshape(11, 3, 20), _d(w)), 1.5 * BF16_ULP, BF16_ULP)


# ------------------------------------------------------------------ experts with the square of relu

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_square_of_relu_in_the_experts_products(dtype):
    ops = _ops()
    T, E, top, D, F = 9, 5, 2, 48, 40
    h, w = _rand((T, D), dtype, 1), _rand((E, F, D), dtype, 2, 0.3)
    ids = _i32(np.random.default_rng(0).integers(0, E, (T, top)).tolist())
    u = torch.relu(torch.einsum("tjfd,td->tjf", _d(w)[ids.cpu().long()], _d(h))) ** 2
    tol, rel = (1e-5, 0.0) if dtype == torch.float32 else (1.5 * BF16_ULP, BF16_ULP)
    _close(ops.moe_up(h, w, ids, "relu2"), u, tol, rel)
    if dtype == torch.bfloat16:
        out = torch.empty((T * top, F), dtype=dtype, device=DEV)
        ops.grouped_gemm(h, w, out, listed=ops.group_rows(ids.view(-1), E), a_div=top, act="relu2")
        _close(out.reshape(T, top, F), u, tol, rel)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T", [5, 200, 1100])
def test_a_routed_feed_forward_in_all_three_of_its_forms(dtype, T):
    """Few pairs (streamed), hundreds (grouped products) and thousands (padded tiles): a softmax router with a correction for
    the choice, weights as they are."""
    from longbow_quarrel_b200.parts import make_part
    from longbow_quarrel_b200.parts.base import Runtime
    from longbow_quarrel_b200.parts.spec import PartSpec
    D, E, top, F = 64, 6, 2, 40
    part = make_part("ffn", PartSpec("routed_experts", {"hidden_size": D, "n_experts": E, "top": top, "expert_size": F, "activation": "relu2",
                                                        "score": "softmax", "correction": True, "normalize": False}), Runtime(torch.device(DEV), dtype, 64))
    w = {n: _rand(s.shape, torch.bfloat16, 10 + i, 0.3) for i, (n, s) in enumerate(part.weights().items())}
    part.load(w)
    h = _rand((T, D), dtype, 1)
    z = _d(h) @ _d(w["router"]).T
    s = torch.softmax(z, 1)
    choice = s + _d(w["correction"])
    order = choice.argsort(1, descending=True)
    firm = (choice.gather(1, order[:, top - 1:top]) - choice.gather(1, order[:, top:top + 1]))[:, 0] > 1e-4
    ref = torch.zeros(T, D, dtype=torch.float64)
    for j in range(top):
        for e in range(E):
            m = order[:, j] == e
            u = torch.relu(_d(h)[m] @ _d(w[f"e{e}.up"]).T) ** 2
            ref[m] += s[m, e:e + 1] * (u @ _d(w[f"e{e}.down"]).T)
    out = _d(part.forward(h, None, None))
    assert firm.sum() > 0.9 * T
    _close(out[firm], ref[firm], 2e-5 if dtype == torch.float32 else 9 * BF16_ULP, 0.0 if dtype == torch.float32 else 2 * BF16_ULP)


# ------------------------------------------------------------------ the gated delta rule with one decay per head

class Rule:
    """Random rows of sequences, and the rule in float64 with the state and the convolution's past carried by hand."""

    EPS = 1e-5

    def __init__(self, H, G, dk, dv, taps, lens, seed, rate=None, bias=None):
        self.H, self.G, self.dk, self.dv, self.taps = H, G, dk, dv, taps
        self.C = 2 * G * dk + H * dv
        self.b_off, self.a_off = self.C + 3, self.C + 3 + H
        self.g_off = self.a_off + H
        self.rows = [_rand((n, self.g_off + H * dv + 2), torch.float32, seed * 10 + i) for i, n in enumerate(lens)]
        self.taps_w = _rand((taps, self.C), torch.float32, seed + 900, 0.6)
        self.bias = _rand((H,), torch.float32, seed + 903) - 2.0 if bias is None else torch.full((H,), float(bias), device=DEV)
        self.rate = torch.exp(_rand((H,), torch.float32, seed + 904)) if rate is None else torch.full((H,), float(rate), device=DEV)
        self.norm_w = _rand((dv,), torch.float32, seed + 905) + 1.0
        n_slots = len(lens) + 3
        self.slot_of = [int(s) for s in np.random.default_rng(seed).permutation(n_slots)[:len(lens)]]
        self.state = torch.zeros((n_slots, H, dk, dv), dtype=torch.float32, device=DEV)
        self.ring = torch.full((n_slots, taps, self.C), 77.0, dtype=torch.float32, device=DEV)   # rows ahead of a sequence must not be read

    def reference(self, i):
        """(raw outputs [n, H, dv], finished outputs [n, H dv], S) of sequence i."""
        x = _d(self.rows[i])
        n, H, G, dk, dv = x.shape[0], self.H, self.G, self.dk, self.dv
        w = _d(self.taps_w)
        y = torch.zeros(n, self.C, dtype=torch.float64)
        for j in range(self.taps):
            back = self.taps - 1 - j
            if back < n:
                y[back:] += w[j] * x[:n - back, :self.C]
        y = y * torch.sigmoid(y)
        q, k, v = y[:, :G * dk].reshape(n, G, dk), y[:, G * dk:2 * G * dk].reshape(n, G, dk), y[:, 2 * G * dk:].reshape(n, H, dv)
        q = q / torch.sqrt((q * q).sum(-1, keepdim=True) + 1e-6) * dk ** -0.5
        k = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
        q, k = q.repeat_interleave(H // G, 1), k.repeat_interleave(H // G, 1)
        b = torch.sigmoid(x[:, self.b_off:self.b_off + H])
        a = torch.exp(-_d(self.rate) * torch.nn.functional.softplus(x[:, self.a_off:self.a_off + H] + _d(self.bias)))
        S, o = torch.zeros(H, dk, dv, dtype=torch.float64), torch.zeros(n, H, dv, dtype=torch.float64)
        for t in range(n):
            S = a[t][:, None, None] * S
            u = b[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
            S = S + k[t][:, :, None] * u[:, None, :]
            o[t] = torch.einsum("hdv,hd->hv", S, q[t])
        gate = x[:, self.g_off:self.g_off + H * dv]
        return o, (_rms(o, self.EPS) * _d(self.norm_w)).reshape(n, -1) * gate * torch.sigmoid(gate), S

    def _run(self, fn, rows, takes, dtype, *sizes):
        cu = np.cumsum([0] + [n for _, _, n in takes]).tolist()
        pos = [lo + t for _, lo, n in takes for t in range(n)]
        return fn(rows, self.b_off, self.a_off, self.g_off, self.taps_w, self.ring, self.bias, self.rate, self.state, _i32(cu),
                  _i32([self.slot_of[i] for i, _, _ in takes]), _i32(pos), self.norm_w, self.EPS, dtype, len(takes), *sizes, self.H, self.G, self.dk,
                  self.dv, self.dk ** -0.5, 1e-6)

    def step(self, takes, dtype=torch.float32):
        """takes: (sequence, first row, rows) for each of the step's sequences; finished outputs in that order."""
        rows = torch.cat([self.rows[i][lo:lo + n] for i, lo, n in takes]).contiguous()
        return self._run(_ops().head_delta_prompt, rows, takes, dtype, max(n for _, _, n in takes))

    def single(self, takes, dtype=torch.float32):
        """takes: (sequence, row): one token each."""
        rows = torch.cat([self.rows[i][t:t + 1] for i, t in takes]).contiguous()
        return self._run(_ops().head_delta_single, rows, [(i, t, 1) for i, t in takes], dtype)

    def firm(self, o):
        """(n, H dv): heads whose output is not the small rest of a sum that nearly cancels (the norm behind it blows that up)."""
        size = o.pow(2).mean(-1).sqrt()
        return (size > 0.03 * size.median()).reshape(o.shape[0], self.H, 1).expand(-1, -1, self.dv).reshape(o.shape[0], -1)


def _held(got, ref, case, lo, hi, dtype=torch.float32):
    """Finished rows lo .. hi - 1 of a sequence against its reference."""
    o, want, _ = ref
    firm = case.firm(o)[lo:hi]
    assert torch.isfinite(got).all()
    _close(torch.where(firm, _d(got), want[lo:hi]), want[lo:hi], 3e-4 if dtype == torch.float32 else 2 * BF16_ULP, BF16_ULP)


# H, G, dk, dv, taps
RULES = [(4, 2, 16, 24, 4), (2, 2, 64, 64, 4), (3, 1, 20, 37, 5), (6, 2, 8, 5, 1), (1, 1, 200, 33, 7), (2, 1, 96, 176, 4), (2, 2, 128, 128, 3),
         (1, 1, 256, 256, 2), (2, 1, 160, 16, 4), (40, 8, 64, 96, 4), (3, 3, 33, 70, 6), (64, 16, 32, 64, 4)]


@pytest.mark.parametrize("H,G,dk,dv,taps", RULES)
def test_the_rule_whole_in_portions_and_token_by_token(H, G, dk, dv, taps):
    """Three sequences of unequal lengths in one step; the same in portions that start and end around the chunks' borders,
    mixed with single tokens; one by one; and what each leaves as its state."""
    lens = [150, 3, 70]
    ref = None
    for cuts in ([[150], [3], [70]], [[1, 63, 64, 5, 17], [2, 1], [7, 1, 1, 3, 58]], [[65, 2, 64, 19], [1, 1, 1], [64, 2, 4]]):
        case = Rule(H, G, dk, dv, taps, lens, seed=7)
        ref = ref or [case.reference(i) for i in range(3)]
        at, got = [0, 0, 0], [[], [], []]
        for step in range(max(len(c) for c in cuts)):
            takes = [(i, at[i], cuts[i][step]) for i in (2, 0, 1) if step < len(cuts[i])]
            out, row = case.step(takes), 0
            for i, _, n in takes:
                got[i].append(out[row:row + n])
                row += n
                at[i] += n
        for i in range(3):
            _held(torch.cat(got[i]), ref[i], case, 0, lens[i])
            _close(case.state[case.slot_of[i]], ref[i][2], 2e-5)
        others = [s for s in range(case.state.shape[0]) if s not in case.slot_of]
        assert float(case.state[others].abs().max()) == 0.0 and float((case.ring[others] - 77.0).abs().max()) == 0.0
    case = Rule(H, G, dk, dv, taps, lens, seed=7)
    out = case.step([(0, 0, 150), (1, 0, 3), (2, 0, 70)], torch.bfloat16)
    for i, (lo, hi) in enumerate(((0, 150), (150, 153), (153, 223))):
        _held(out[lo:hi].float(), ref[i], case, 0, lens[i], torch.bfloat16)
    for dtype in (torch.float32, torch.bfloat16):
        case = Rule(H, G, dk, dv, taps, lens, seed=7)
        got = [[], [], []]
        for t in range(max(lens)):
            live = [i for i in (2, 0, 1) if t < lens[i]]
            out = case.single([(i, t) for i in live], dtype)
            for r, i in enumerate(live):
                got[i].append(out[r].float())
        for i in range(3):
            _held(torch.stack(got[i]), ref[i], case, 0, lens[i], dtype)
            _close(case.state[case.slot_of[i]], ref[i][2], 2e-5)


@pytest.mark.parametrize("dk,dv", [(64, 64), (96, 40), (16, 24)])
def test_a_prompt_goes_on_token_by_token_and_back(dk, dv):
    """A prompt by chunks, single tokens, a portion: both kernels leave each other the same state and the same past."""
    n = 160
    case = Rule(4, 2, dk, dv, 4, [n, n], seed=21)
    ref = [case.reference(i) for i in range(2)]
    out = case.step([(0, 0, 61), (1, 0, 66)])
    _held(out[:61], ref[0], case, 0, 61)
    _held(out[61:], ref[1], case, 0, 66)
    at = [61, 66]
    for _ in range(9):
        out = case.single([(1, at[1]), (0, at[0])])
        _held(out[:1], ref[1], case, at[1], at[1] + 1)
        _held(out[1:], ref[0], case, at[0], at[0] + 1)
        at = [p + 1 for p in at]
    out = case.step([(0, at[0], n - at[0]), (1, at[1], n - at[1])])
    _held(out[:n - at[0]], ref[0], case, at[0], n)
    _held(out[n - at[0]:], ref[1], case, at[1], n)


@pytest.mark.parametrize("single", [False, True])
def test_a_write_is_read_back_after_hundreds_of_tokens(single):
    """Nothing decays (rate 0) and only the token at 5 writes (every other step size is sigmoid(-80)): the state holds exactly
    its key's and value's product hundreds of tokens later, and nothing stands in it ahead of the write."""
    n, H, dk, dv = 400, 2, 32, 16
    case = Rule(H, 2, dk, dv, 1, [n], seed=3, rate=0.0)
    rows = case.rows[0]
    rows[:, case.b_off:case.b_off + H] = -80.0
    rows[5, case.b_off:case.b_off + H] = 80.0
    o, want, S = case.reference(0)
    assert float(o[:5].abs().max()) < 1e-30 and float(S.abs().max()) > 0.1
    if single:
        out = torch.stack([case.single([(0, t)])[0] for t in range(n)])
    else:
        out = torch.cat([case.step([(0, 0, 129)]), case.step([(0, 129, n - 129)])])
    assert float(out[:5].abs().max()) < 1e-20
    _close(case.state[case.slot_of[0]], S, 2e-6)
    _held(out[5:], (o[5:], want[5:], S), case, 0, n - 5)


@pytest.mark.parametrize("single", [False, True])
def test_decays_of_zero_and_a_slot_that_is_used_again(single):
    """A rate so large that every decay is exactly zero: each position reads its own write alone, in a slot whose ring still
    holds another sequence's rows and whose state starts from zero."""
    case = Rule(3, 1, 24, 40, 4, [90], seed=5, rate=1e6, bias=5.0)
    case.ring.fill_(float("nan"))                                # a former owner's rows: positions below zero are not read
    ref = case.reference(0)
    got = torch.stack([case.single([(0, t)])[0] for t in range(90)]) if single else case.step([(0, 0, 90)])
    _held(got, ref, case, 0, 90)
    _close(case.state[case.slot_of[0]], ref[2], 2e-5)


@pytest.mark.parametrize("forget", [60.0, 1e4])
def test_a_token_that_forgets_everything_leaves_the_decays_behind_it_their_digits(forget):
    """One token in a chunk decays by e^-(rate * softplus) of sixty and of thousands, the others by a few per cent each: what
    is written behind it must decay as finely as if it had not been there."""
    case = Rule(2, 2, 32, 32, 4, [64 + 40], seed=8, rate=1.0, bias=-3.0)
    case.rows[0][20, case.a_off:case.a_off + 2] = forget
    ref = case.reference(0)
    _held(case.step([(0, 0, 104)]), ref, case, 0, 104)
    _close(case.state[case.slot_of[0]], ref[2], 5e-6)


def test_sizes_that_the_rule_does_not_take_are_refused():
    ops = _ops()
    case = Rule(1, 1, 8, 8, 4, [4], seed=1)
    ring = case.ring
    case.ring = ring[:, :2].contiguous()
    with pytest.raises(ops.KernelError):
        case.step([(0, 0, 4)])
    case.ring = ring
    case.dv, case.norm_w = 300, torch.ones(300, device=DEV)
    with pytest.raises(ops.KernelError):
        case.step([(0, 0, 4)])
