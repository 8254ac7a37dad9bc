"""Batch inference entry point (``gpatch_v4/entry`` infer / eval mains): loads a checkpoint (torch_dist or HF) into
the rollout engine and writes one jsonl line per prompt with the generated token ids and log-probs.

    python -m gcore_b200.entry.lm_infer --config rl.yaml +task.infer.prompts=prompts.jsonl +task.infer.out=out.jsonl

A checkpoint folder whose ``config.json`` names a serving-only architecture (layer-plan decoders such as Nafitar) goes
straight into the engine, without a trainer around it:

    python -m gcore_b200.entry.lm_infer checkpoint.load_ckpt_path=DIR +task.infer.prompts=prompts.jsonl \
        +task.infer.out=out.jsonl

with the sampling fields of ``sampler.infer_engine_configs`` as usual (``+task.infer.greedy=true``: greedy).
"""
import json
import sys

import torch

from ..configs.config import RlConfig
from ..trainer.grpo_trainer import GrpoTrainer
from .common import finalize, init_runtime, load


def _read_prompts(inf):
    return [json.loads(l)["prompt_token_ids"] for l in open(inf["prompts"])] if inf.get("prompts") else \
        [torch.randint(100, 1000, (16,)).tolist() for _ in range(4)]


def serve_checkpoint(cfg, inf):
    """Generation from a serving-only checkpoint through the rollout engine."""
    from ..checkpoint.hf import load_serving_model
    from ..rollout.engine import InferEngine, RolloutWeights, SamplingParams
    if not torch.cuda.is_available():
        raise RuntimeError("serving a checkpoint needs a GPU")
    device = torch.device("cuda", torch.cuda.current_device())
    ie = cfg.sampler.infer_engine_configs[0]
    model_cfg, model = load_serving_model(cfg.checkpoint.load_ckpt_path, device, ie.dtype)
    prompts = _read_prompts(inf)
    longest = max(len(p) for p in prompts) + ie.generate_max_tokens
    eng = InferEngine(model_cfg, RolloutWeights.from_model(model),
                      max_running_requests=ie.max_running_requests or min(64, len(prompts)),
                      max_model_len=ie.max_model_len or longest, kv_block_size=ie.kv_block_size,
                      num_kv_blocks=ie.num_kv_blocks, gpu_memory_utilization=ie.gpu_memory_utilization,
                      max_prefill_tokens=ie.max_prefill_tokens, use_cuda_graph=not ie.disable_cuda_graph, device=device)
    params = SamplingParams(temperature=ie.temperature, top_k=ie.top_k, top_p=ie.top_p, min_p=ie.min_p,
                            repetition_penalty=ie.repetition_penalty, max_new_tokens=ie.generate_max_tokens, seed=ie.seed,
                            stop_token_ids=tuple(ie.generate_params.get("stop_token_ids", ())),
                            greedy=bool(inf.get("greedy", False)))
    return [{"tokens": r.prompt + r.out_tokens, "prompt_length": len(r.prompt)}
            for r in eng.generate(prompts, params)]


def _write(out, inf):
    if inf.get("out"):
        with open(inf["out"], "w") as f:
            for s in out:
                f.write(json.dumps({"tokens": torch.as_tensor(s["tokens"]).tolist(),
                                    "prompt_length": int(s["prompt_length"])}) + "\n")


def main(argv=None):
    cfg = load(RlConfig, argv)
    init_runtime(cfg)
    inf = dict((cfg.task or {}).get("infer", {}) or {})
    if cfg.checkpoint.load_ckpt_path:
        from ..checkpoint.hf import read_model_config
        model_cfg = read_model_config(cfg.checkpoint.load_ckpt_path)
        if model_cfg is not None and model_cfg.layer_plan is not None:
            _write(serve_checkpoint(cfg, inf), inf)
            finalize()
            return 0
    tr = GrpoTrainer(cfg)
    tr.setup()
    if cfg.checkpoint.load_ckpt_path:
        from ..checkpoint.torch_dist import load_checkpoint, read_latest_step
        if read_latest_step(cfg.checkpoint.load_ckpt_path) is not None:
            load_checkpoint(tr.policy, cfg.checkpoint.load_ckpt_path, load_optim=False)
        else:
            from ..checkpoint.hf import load_hf
            load_hf(tr.policy, cfg.checkpoint.load_ckpt_path)
        tr.update_weights()
    _write(tr.rollout(_read_prompts(inf)), inf)
    finalize()
    return 0


if __name__ == "__main__":
    sys.exit(main())
