#!/usr/bin/env python3
"""Text generation with LLMPipeline on the CUDA device.

usage: llm_generate.py <model> "<prompt>" [max_new_tokens]
  <model>   directory with openvino_model.xml, directory with config.json + model.safetensors, or a .gguf file
  <prompt>  text (byte-level tokenizer), or token ids as "ids:1,15043,29892" (the answer is then printed as ids)
"""
import sys

from openvino_b200.genai import ByteTokenizer, GenerationConfig, LLMPipeline


def main() -> int:
    if len(sys.argv) < 3:
        print(__doc__)
        return 1
    prompt = sys.argv[2]
    if prompt.startswith("ids:"):
        prompt = [int(t) for t in prompt[4:].split(",")]
    pipe = LLMPipeline(sys.argv[1], "CUDA", tokenizer=ByteTokenizer())
    cfg = GenerationConfig(max_new_tokens=int(sys.argv[3]) if len(sys.argv) > 3 else 64)
    print(pipe.generate(prompt, cfg))
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
