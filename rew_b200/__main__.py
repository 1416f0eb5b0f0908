"""Command line: python -m rew_b200 generate --model DIR --ids 1,2,3 [--max-new N] [sampling options]

Token ids in, token ids out (this backend has no tokenizer).  DIR is any folder the registry (rew_b200/models.py)
knows.  Several --ids are served as one batch over paged lanes: prompts join as lanes free up.
"""
import argparse
import sys


def serve(model, prompts, max_new, stop_ids=(), lanes=8, chunk=512, sampling=None, seeds=None, decode_steps=8):
    """Continuous batching: every step feeds portions of at most `chunk` tokens of waiting prompts; once no prompt is
    waiting, the captured decode step runs `decode_steps` tokens at a time.  Returns the new ids of every prompt."""
    need = max(len(p) for p in prompts) + max_new + decode_steps
    lanes = min(lanes, len(prompts))
    pages = -(-need // 64)
    sess = model.paged_session(lanes, pages * 64, lanes * pages + 1)
    if sampling:
        sess.set_sampling(**sampling)
    out = [[] for _ in prompts]
    queue, live, fed = list(range(len(prompts))), {}, {}
    stops = set(stop_ids)

    def done(r):
        return len(out[r]) >= max_new or (out[r] and out[r][-1] in stops)

    def take(r, ids):
        for i in ids:
            if not done(r):
                out[r].append(int(i))

    while queue or live:
        for lane in range(lanes):
            if lane not in live and queue:
                live[lane] = queue.pop(0)
                fed[live[lane]] = 0
        filling = {l: r for l, r in live.items() if fed[r] < len(prompts[r])}
        if filling:
            portions, flags, order = [], [], []
            for lane, r in live.items():
                if lane in filling:
                    ids = prompts[r][fed[r]:fed[r] + chunk]
                    fed[r] += len(ids)
                    portions.append((lane, ids))
                    flags.append(fed[r] == len(prompts[r]))
                else:                                       # decoding lanes go on beside the prompts
                    portions.append((lane, [out[r][-1]]))
                    flags.append(True)
                order.append(r)
            _, nxt = sess.feed(portions, sample=flags, seeds=[(seeds[r] if seeds else 0) for r in order])
            for r, f, n in zip(order, flags, nxt):
                if f:
                    take(r, [n])
        else:
            ids = sess.step(decode_steps)
            for lane, r in live.items():
                take(r, ids[lane])
        for lane in [l for l, r in live.items() if done(r)]:
            sess.release(lane)
            del live[lane]
    sess.free()
    return out


def main(argv=None):
    ap = argparse.ArgumentParser(prog="python -m rew_b200")
    sub = ap.add_subparsers(dest="command", required=True)
    g = sub.add_parser("generate", help="generate token ids from prompt token ids")
    g.add_argument("--model", required=True, help="folder with config.json and *.safetensors")
    g.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    g.add_argument("--ids", action="append", required=True, help="prompt token ids with commas between them (repeatable)")
    g.add_argument("--max-new", type=int, default=32)
    g.add_argument("--stop", type=int, action="append", default=[], help="token id that ends a sequence (repeatable)")
    g.add_argument("--lanes", type=int, default=8)
    g.add_argument("--chunk", type=int, default=512, help="prompt tokens of one request fed in a step")
    g.add_argument("--sample", action="store_true", help="sample instead of taking the largest logit")
    g.add_argument("--temperature", type=float, default=1.0)
    g.add_argument("--top-k", type=int, default=50)
    g.add_argument("--top-p", type=float, default=1.0)
    g.add_argument("--min-p", type=float, default=0.0)
    g.add_argument("--repetition-penalty", type=float, default=1.0)
    g.add_argument("--seed", type=int, default=0)
    args = ap.parse_args(argv)
    from .models import load_model
    prompts = [[int(v) for v in s.split(",")] for s in args.ids]
    need = max(len(p) for p in prompts) + args.max_new
    model = load_model(args.model, dtype=args.dtype, max_seq=-(-(need + 8) // 64) * 64)
    sampling = dict(temperature=args.temperature, top_k=args.top_k, top_p=args.top_p, min_p=args.min_p,
                    repetition_penalty=args.repetition_penalty) if args.sample else None
    for ids in serve(model, prompts, args.max_new, args.stop, args.lanes, args.chunk, sampling, [args.seed + i for i in range(len(prompts))]):
        print(" ".join(map(str, ids)))
    return 0


if __name__ == "__main__":
    sys.exit(main())
