"""The Gevipel design through the engine: every mechanism alone and together, every way of cutting and batching requests,
slots and pages used again, long decoding, the edges of windows made visible by one odd token, the first token carried by
the state and by the latent rows, generation through the entry point and the command line -- each against the plain
implementation (tests/plain_gevipel.py)."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_gevipel
from gevipel_models import CONFIGS, bound, firm_rows, load, make_folder, random_config, rewrite, row_errors, tokens, within
from trace_tools import ROOT, Trace, run_trace, split, trace_batches, trace_chunked, trace_last_one_by_one, trace_mixed, trace_whole

pytestmark = pytest.mark.gpu

DTYPES = ["float32", "bfloat16"]


def _engine(folder, dtype, **kw):
    from longbow_quarrel_b200.engine import Engine
    return Engine.from_pretrained(folder, dtype=dtype, **kw)


_memo: dict = {}


def _plain(folder, toks, dtype=None):
    """The plain implementation's logits for a request and, with a dtype, its bound and firm rows (kept: every cut is compared
    with them)."""
    key = (str(folder), tuple(toks))
    if key not in _memo:
        cfg, weights = load(folder)
        margins = plain_gevipel.new_margins()
        _memo[key] = {"ref": plain_gevipel.forward(cfg, weights, toks, margins=margins).numpy(), "margins": margins}
    entry = _memo[key]
    if dtype is not None and dtype not in entry:
        firm = firm_rows(dtype, *load(folder), toks, entry["margins"])
        entry[dtype] = (bound(dtype, *load(folder), toks, entry["ref"], firm), firm)
    return entry["ref"] if dtype is None else (entry["ref"], *entry[dtype])


def _check(got: dict, requests: dict, folder, dtype: str, what: str):
    """Every request's rows within its bound (`within` says how)."""
    for rid, toks in requests.items():
        ref, tol, firm = _plain(folder, toks, dtype)
        pos = np.asarray(sorted(p for r, p in got if r == rid))
        assert len(pos), f"{what}: nothing came back for {rid}"
        err = row_errors(np.stack([got[(rid, int(p))] for p in pos]), ref[pos])
        bad = [(int(p), float(e)) for p, e, f in zip(pos, err, firm[pos]) if f and e >= tol]
        assert within(dtype, err, firm[pos], tol), f"{what}: request {rid} of {len(toks)}: bound {tol:.3g}, over it {bad[:6]}"


def _rows(eng, slot, toks, cut):
    """The logits of every position: the first `cut` tokens in one step, the others one by one."""
    rows = [eng.step([(slot, toks[:cut])], [list(range(cut))]).cpu().numpy()] if cut else []
    rows += [eng.step([(slot, [t])], [[0]]).cpu().numpy() for t in toks[cut:]]
    return np.concatenate(rows)


def _settle(folder):
    """Corrections so far apart that they alone decide which experts run (their weights still come from the token): in
    bfloat16 a whole model's runs otherwise part where a choice is close and every later row sees another row.  Choices that
    the tokens make are held to in float32, and in bfloat16 by the models of one layer."""
    def change(w):
        for name in w:
            if name.endswith("mlp.correction"):
                w[name] = 2.0 * torch.randperm(w[name].numel(), generator=torch.Generator().manual_seed(len(name))).to(w[name].dtype)
    rewrite(folder, change)


# ------------------------------------------------------------------ each mechanism alone

ALONE = [name for name in sorted(CONFIGS) if name.startswith("only_")]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ALONE)
def test_one_layer_of_each_kind_whole_and_token_by_token(tmp_path, name, dtype):
    """A model of one mechanism: the whole prompt in one step (its first tokens included), and the same tokens one by one
    from the first (133 steps: across two page borders, two chunk borders and past every window; replayed from a captured step)."""
    folder = make_folder(tmp_path, name, seed=3)
    toks = tokens(133, CONFIGS[name]["vocab"], 5)
    ref, tol, firm = _plain(folder, toks, dtype)
    assert firm.sum() > 110
    eng = _engine(folder, dtype, max_tokens=512)
    s = eng.new_sequence()
    whole = _rows(eng, s, toks, len(toks))
    eng.end_sequence(s)
    assert within(dtype, row_errors(whole, ref), firm, tol), row_errors(whole, ref)[firm].max()
    s = eng.new_sequence()
    single = _rows(eng, s, toks, 0)
    eng.end_sequence(s)
    assert within(dtype, row_errors(single, ref), firm, tol), row_errors(single, ref)[firm].max()
    assert within(dtype, row_errors(single, whole), firm, tol)
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["only_delta", "only_attention", "only_latent", "only_experts"])
def test_a_checkpoint_stored_in_32_bit(tmp_path, name, dtype):
    """Every tensor float32: the products keep them as they are, in either precision of the model."""
    folder = make_folder(tmp_path, name, seed=6, dtype=torch.float32)
    toks = tokens(70, CONFIGS[name]["vocab"], 9)
    ref, tol, firm = _plain(folder, toks, dtype)
    import warnings
    with warnings.catch_warnings():
        warnings.simplefilter("ignore")                      # (the loader says that such products run on the CUDA cores)
        eng = _engine(folder, dtype, max_tokens=256)
    s = eng.new_sequence()
    assert within(dtype, row_errors(_rows(eng, s, toks, 40), ref), firm, tol)
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim", [64, 48, 12])
def test_a_window_ends_where_it_ends_when_one_token_outweighs_all_others(tmp_path, dtype, dim):
    """A prompt of one odd token among copies of another, in attention whose softmax is flat but for the distance.  With a
    window of 4 an odd token at position 30 changes the logits of 30 .. 33 and none after; with one of 64, at the last
    place of a page and at the first of the next, the rows up to 63 behind it -- in a prompt, with the edge among decoded
    tokens, and with everything after the odd token decoded.  (Eight heads: the slowest falls by 2^-8 a position, so a key at the
    far edge of 64 still counts.)"""
    for size, at_places in ((4, [30, 31]), (64, [63, 64])):
        data = json.loads(json.dumps(CONFIGS["only_attention"]))
        data["layers"][0]["mixer"].update(heads=8, kv_heads=8, dim=dim, vdim=dim, mask={"size": size}, scale=0.01)
        data["layers"][0]["mixer"].pop("q_temp")
        folder = make_folder(tmp_path / str(size), data, seed=9, std=0.5)
        n = 50 if size == 4 else 135
        base = [7] * n
        ref_base = _plain(folder, base)
        eng = _engine(folder, dtype, max_tokens=512)
        for at in at_places:
            inside, outside = at + size - 1, at + size
            odd = list(base)
            odd[at] = 55
            ref_odd, tol, _ = _plain(folder, odd, dtype)
            assert row_errors(ref_odd[inside], ref_base[inside]) > 1e-4
            assert row_errors(ref_odd[outside:], ref_base[outside:]).max() < 1e-12
            for cut in (n, inside - 2, at + 1):
                s = eng.new_sequence()
                got = _rows(eng, s, odd, cut)
                eng.end_sequence(s)
                assert row_errors(got, ref_odd).max() < tol, (size, at, cut)
                # (an odd key at the far edge of sixty-four weighs less than what rounding to bfloat16 does: the float32 run shows it)
                if size == 4 or dtype == "float32":
                    assert row_errors(got[inside], ref_base[inside]) > 2 * tol, (size, at, cut)
                assert row_errors(got[outside:], ref_base[outside:]).max() < tol, (size, at, cut)
        eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["only_delta", "only_delta_even", "only_latent", "only_attention_open"])
def test_the_first_token_lasts(tmp_path, name, dtype):
    """The first of 300 tokens still shows at the last: in the delta rule's state (decays close to one, small step sizes, so
    that later writes leave it standing), in the latent rows, and in attention over all positions whose slopes are small
    (the last head's is 2^-8); whole, with the last 200 decoded, and in portions that end off the chunks of 64 tokens."""
    folder = make_folder(tmp_path, name, seed=4, std=0.1 if name == "only_latent" else 0.5)

    def change(w):
        w["l0.mix.dt_bias"].fill_(-14.0)
        w["l0.mix.a"].mul_(0.01)
        w["l0.mix.b"].mul_(0.1)
    if name.startswith("only_delta"):
        rewrite(folder, change)
    vocab = CONFIGS[name]["vocab"]
    base = tokens(300, vocab, 8)
    odd = [(base[0] + 1) % vocab] + base[1:]
    ref_base, (ref_odd, tol, firm) = _plain(folder, base), _plain(folder, odd, dtype)
    sharp = row_errors(ref_odd[299], ref_base[299]) > 5 * tol
    assert sharp or dtype == "bfloat16"                      # one token among three hundred may be as small as rounding to bfloat16
    eng = _engine(folder, dtype, max_tokens=512)
    for portions in ([300], [100] + [1] * 200, [97, 2, 3, 1, 101, 96]):
        s = eng.new_sequence()
        rows, at = [], 0
        for n in portions:
            rows.append(eng.step([(s, odd[at:at + n])], [list(range(n))]).cpu().numpy())
            at += n
        eng.end_sequence(s)
        got = np.concatenate(rows)
        assert within(dtype, row_errors(got, ref_odd), firm, tol), portions[:3]
        assert not sharp or row_errors(got[299], ref_base[299]) > 3 * tol, portions[:3]
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_sink_and_a_correction_that_decide(tmp_path, dtype):
    """Sinks of 6 take most of the weight of every second of a latent layer's heads, sinks of -6 none of the others'; a correction of 5 makes one expert everyone's first
    choice without changing its weight: both must show, in prompts and in decoding."""
    for name, key, value in (("only_latent", "l0.mix.sink", 6.0), ("only_experts", "l0.mlp.correction", 5.0)):
        folder = make_folder(tmp_path / key, name, seed=4)
        toks = tokens(90, CONFIGS[name]["vocab"], 8)
        low = _plain(folder, toks)

        def change(w):
            if key.endswith("sink"):
                w[key].fill_(value)
                w[key][::2].neg_()
            else:
                w[key].zero_()
                w[key][4] = value
        folder2 = make_folder(tmp_path / (key + "2"), name, seed=4)
        rewrite(folder2, change)
        ref, tol, firm = _plain(folder2, toks, dtype)
        assert row_errors(ref, low).mean() > 2 * tol
        eng = _engine(folder2, dtype, max_tokens=256)
        for cut in (90, 30):
            s = eng.new_sequence()
            assert within(dtype, row_errors(_rows(eng, s, toks, cut), ref), firm, tol), (key, cut)
            eng.end_sequence(s)
        eng.close()


# ------------------------------------------------------------------ whole models, every cut, through the replay program

LENGTHS = {"r0": 70, "r1": 33, "r2": 140, "r3": 65, "r4": 64, "r5": 34, "r6": 129}
PROMPTS = {"r0": 7, "r1": 1, "r2": 100, "r3": 2, "r4": 63, "r5": 20, "r6": 65}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
def test_every_cut_of_every_request_matches_plain(tmp_path, name, dtype):
    """Whole; the last 32 tokens one by one; batches of three unequal requests that go on together, the shorter
    ending earlier, the next batch in the slots and pages given back; portions of 2, 3, 59, 1, 64 and 7 tokens;
    steps that mix portions with single tokens.  One call of the replay program runs them one after the other."""
    folder = make_folder(tmp_path, name, seed=11)
    if dtype == "bfloat16":
        _settle(folder)
    vocab = CONFIGS[name]["vocab"]
    requests = {rid: tokens(n, vocab, 100 + i) for i, (rid, n) in enumerate(LENGTHS.items())}
    tr = Trace()
    tr.extend(trace_whole(requests), "whole:")
    tr.extend(trace_last_one_by_one(requests), "tail:")
    tr.extend(trace_batches(requests, PROMPTS, width=3), "batched:")
    tr.extend(trace_chunked(requests, [2, 3, 59, 1, 64, 7]), "portions:")
    tr.extend(trace_mixed(requests, PROMPTS, [5, 1, 2, 1, 17]), "mixed:")
    got = run_trace(folder, dtype, tr, tmp_path / "out")
    cuts = {p: split(got, p + ":") for p in ("whole", "tail", "batched", "portions", "mixed")}
    for what, rows in cuts.items():
        assert len(rows) == (33 * len(requests) if what == "tail" else sum(LENGTHS.values())), what
        _check(rows, requests, folder, dtype, what)
    if dtype == "float32":
        for rid, toks in requests.items():
            _, tol, firm = _plain(folder, toks, dtype)
            for what in ("tail", "batched", "portions", "mixed"):
                for (r, pos), row in cuts[what].items():
                    if r == rid and firm[pos]:
                        err = float(row_errors(row, cuts["whole"][(r, pos)]))
                        assert err < 2 * tol, f"{what} against whole: {rid} position {pos}: {err:.3g}, bound {2 * tol:.3g}"


@pytest.mark.parametrize("seed", [3, 12, 25])
def test_configurations_drawn_at_random_match_plain(tmp_path, seed):
    """Sizes and options that nobody chose: whole, the last 30 tokens one by one and an unequal batch, in both precisions."""
    import random
    rng = random.Random(seed)
    folder = make_folder(tmp_path, random_config(rng), seed=seed, std=rng.choice([0.1, 0.2]))
    cfg, _ = load(folder)
    requests = {rid: tokens(n, cfg["vocab"], 50 * seed + i) for i, (rid, n) in enumerate({"a": 150, "b": 70, "c": 33}.items())}
    tr = Trace()
    tr.extend(trace_whole(requests), "whole:")
    tr.extend(trace_last_one_by_one(requests, n_last=30), "tail:")
    tr.extend(trace_batches(requests, {"a": 110, "b": 40, "c": 3}, width=3), "batched:")
    for dtype in DTYPES:
        if dtype == "bfloat16":
            _settle(folder)
            _memo.clear()
        got = run_trace(folder, dtype, tr, tmp_path / ("out_" + dtype))
        for what in ("whole", "tail", "batched"):
            _check(split(got, what + ":"), requests, folder, dtype, f"seed {seed} {dtype} {what}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_stream_after_every_layer_matches_plain(tmp_path, dtype):
    """The residual stream after each run of a layer (before the embedding's rows join it ahead of a pass), for a prompt that
    is longer than every window, and for the same in portions; the logits are the same with and without the look inside,
    although without it the joining kernel adds the embedding's rows."""
    folder = make_folder(tmp_path, "mixed", seed=13)
    if dtype == "bfloat16":
        _settle(folder)
    toks = tokens(150, CONFIGS["mixed"]["vocab"], 17)
    cfg, weights = load(folder)
    exact: list = []
    margins = plain_gevipel.new_margins()
    plain_gevipel.forward(cfg, weights, toks, layers_out=exact, margins=margins)
    other: list = []
    kw = {"dtype": torch.float32} if dtype == "float32" else {"storage": torch.bfloat16}
    plain_gevipel.forward(cfg, weights, toks, layers_out=other, **kw)
    firm = firm_rows(dtype, cfg, weights, toks, margins)
    eng = _engine(folder, dtype, max_tokens=512)
    for portions in ([150], [64, 1, 2, 83]):
        seen: dict = {}
        last = []
        for look in (True, False):
            eng.model.probe = (lambda i, x, ctx: seen.setdefault(i, []).append(x.detach().float().cpu().clone())) if look else None
            s = eng.new_sequence()
            at = 0
            for n in portions:
                out = eng.step([(s, toks[at:at + n])], [[n - 1]])
                at += n
            eng.end_sequence(s)
            last.append(out.cpu().numpy().copy())
        eng.model.probe = None
        assert row_errors(last[0], last[1]).max() < (1e-5 if dtype == "float32" else 5e-2)
        runs = sorted(i for i in seen if i >= 0)
        assert len(runs) == len(exact) == 8
        for i, want, near in zip(runs, exact, other):
            got = torch.cat(seen[i]).numpy()
            e = row_errors(near.numpy(), want.numpy())[firm]
            yard = max(1e-5, 3.0 * float(e.max() if dtype == "float32" else np.quantile(e, 0.9)))
            assert within(dtype, row_errors(got, want.numpy()), firm, yard), (portions, i)
    eng.close()


# ------------------------------------------------------------------ slots and pages used again, long decoding

@pytest.mark.parametrize("dtype", DTYPES)
def test_a_slot_that_is_used_again_starts_from_nothing(tmp_path, dtype):
    """One slot and just enough pages: each request runs in what the one before it gave back, so a state, a convolution's
    last inputs or a page that outlived its request would show in the next one's first tokens."""
    folder = make_folder(tmp_path, "mixed", seed=21)
    if dtype == "bfloat16":
        _settle(folder)
    eng = _engine(folder, dtype, max_tokens=192, max_batch=1)
    rows, requests = {}, {}
    for i, n in enumerate([150, 3, 130, 66]):
        toks = requests[i] = tokens(n, CONFIGS["mixed"]["vocab"], 300 + i)
        s = eng.new_sequence()
        assert s == 0
        got = _rows(eng, s, toks, max(1, n - 40))
        eng.end_sequence(s)
        rows.update({(i, p): row for p, row in enumerate(got)})
    _check(rows, requests, folder, dtype, "one slot")
    assert eng.cache.pages_in_use() == 0
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_from_the_first_token(tmp_path, dtype):
    """260 single-token steps of three sequences side by side (captured once, replayed): the windows of 64 and 100 pass wholly
    over decoded tokens, their pages go back and come to other sequences, and the states are carried over hundreds of steps."""
    folder = make_folder(tmp_path, "mixed", seed=31)
    if dtype == "bfloat16":
        _settle(folder)
    vocab = CONFIGS["mixed"]["vocab"]
    seqs = [tokens(260, vocab, 40), tokens(260, vocab, 41), tokens(150, vocab, 42)]
    eng = _engine(folder, dtype, max_tokens=3 * 320)
    slots = [eng.new_sequence() for _ in seqs]
    got = {}
    for t in range(260):
        live = [i for i, q in enumerate(seqs) if t < len(q)]
        out = eng.step([(slots[i], [seqs[i][t]]) for i in live], [[0]] * len(live)).cpu().numpy()
        for row, i in zip(out, live):
            got[(i, t)] = row
            if t == len(seqs[i]) - 1:
                eng.end_sequence(slots[i])
    _check(got, dict(enumerate(seqs)), folder, dtype, "decoded")
    eng.close()


# ------------------------------------------------------------------ generation through the entry point and the command line

def _greedy_matches(folder, prompt, new, dtype):
    """Every generated token is the plain implementation's choice for what stands before it (bfloat16: or a near tie with it)."""
    cfg, weights = load(folder)
    seq = list(prompt) + list(new)
    margins = plain_gevipel.new_margins()
    logits = plain_gevipel.forward(cfg, weights, seq[:-1], margins=margins).numpy()
    firm = firm_rows(dtype, cfg, weights, seq[:-1], margins)
    held = 0
    for p in range(len(prompt) - 1, len(seq) - 1):
        row, tok = logits[p], seq[p + 1]
        best = int(np.argmax(row))
        gap = (row[best] - row[tok]) / np.sqrt((row ** 2).mean())
        # In bfloat16 a row that saw another expert's rows may differ by more than its own rounding: most must hold.
        held += tok == best or (dtype == "bfloat16" and gap < 5e-2) or not firm[p]
    assert held == len(new) or (dtype == "bfloat16" and held >= len(new) - 1), (dtype, held, len(new))


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_the_scheduler(tmp_path, dtype):
    """Engine.generate: unequal prompts in batches of three (the second batch in the first one's slots), greedy."""
    from longbow_quarrel_b200.sampling import SamplingParams
    folder = make_folder(tmp_path, "mixed", seed=41)
    if dtype == "bfloat16":
        _settle(folder)
    vocab = CONFIGS["mixed"]["vocab"]
    prompts = [tokens(n, vocab, 500 + i) for i, n in enumerate([9, 1, 70, 2, 64])]
    eng = _engine(folder, dtype, max_tokens=3 * 128, max_batch=3)
    out = eng.generate(prompts, max_new_tokens=10, sampling=SamplingParams(temperature=0.0), stop_ids=[], batch_size=3)
    assert [len(o) for o in out] == [10] * 5
    for prompt, new in zip(prompts, out):
        _greedy_matches(folder, prompt, new, dtype)
    eng.close()


def test_the_command_line_generates_with_a_gevipel_folder(tmp_path):
    folder = make_folder(tmp_path, "odd", seed=51)
    prompt = tokens(12, CONFIGS["odd"]["vocab"], 7)
    proc = subprocess.run([str(ROOT / "bin" / "quarrel"), "-model", str(folder), "-prompt-ids", ",".join(map(str, prompt)),
                           "-n", "6", "-temp", "0", "-penalty", "1.0", "-dtype", "float32", "-output", "json"],
                          capture_output=True, text=True, timeout=600, env={**os.environ, "LQ_PYTHON": sys.executable})
    assert proc.returncode == 0, proc.stderr[-3000:]
    new = json.loads(proc.stdout.strip().splitlines()[-1])["output"][0]
    assert len(new) == 6
    _greedy_matches(folder, prompt, new, "float32")


def test_random_weights_from_a_configuration_and_the_kernels_that_served_it():
    """Engine.from_config builds the design from a dict with config.json's keys; in bfloat16 a prompt of seven hundred
    tokens and decoded tokens go through the design's kernels: the delta rule's chunks for the prompt and its one kernel for
    single tokens, attention and latent attention on the tensor cores, grouped experts, one kernel per join."""
    from longbow_quarrel_b200.engine import Engine
    from longbow_quarrel_b200.kernels import ops
    from longbow_quarrel_b200.sampling import SamplingParams
    eng = Engine.from_config(CONFIGS["wide"], seed=3, max_tokens=2048, max_batch=2)
    before = ops.launches_by_name()
    out = eng.generate([[t % 300 for t in range(1, 701)], [4]], max_new_tokens=5, sampling=SamplingParams(temperature=0.0), stop_ids=[])
    ran = ops.launches_since(before)
    assert [len(o) for o in out] == [5, 5]
    for kernel in ("embedding", "head_delta_prompt", "head_delta_single", "join_branch", "join_branch:extra", "rope_partial", "attn_prefill_tc",
                   "attn_decode:teams", "latent_attention_tc", "grouped_gemm", "moe_route", "layernorm"):
        assert ran.get(kernel, 0) >= 1, (kernel, ran)
    for kernel in ("attention", "latent_attention", "head_matmul", "add_scaled"):     # no plain kernel served a layer; nothing fused ran apart
        assert ran.get(kernel, 0) == 0, (kernel, ran)
    eng.close()
