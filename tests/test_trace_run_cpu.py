"""The trace replay starts in a checkout where nothing is built: what it does before the build may not need built code."""
import json
import os
import subprocess
import sys

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def test_arguments_are_judged_before_anything_is_built(tmp_path):
    code = ("import sys; sys.path.insert(0, sys.argv[1])\n"
            "from dgpp_b200 import build\n"
            "def ensure(family): print('build', family, sorted(m for m in sys.modules if '_dgpp_rt' in m or m == 'dgpp_b200.runtime')); raise SystemExit(7)\n"
            "build.ensure = ensure\n"
            "from dgpp_b200.tools.trace_run import main\n"
            "sys.exit(main(sys.argv[2:]))\n")
    for cfg, dtype, code_want in (({"architecture": "Potivik"}, "float32", 7), ({"architecture": "Vevapel"}, "float32", 7),
                                  ({"architecture": "Tefudra"}, "float32", 7),
                                  ({"architecture": "Sitirax"}, "bfloat16", 7),
                                  ({"architectures": ["Qwen3ForCausalLM"], "model_type": "qwen3"}, "float32", 3)):
        (tmp_path / "config.json").write_text(json.dumps(cfg))
        p = subprocess.run([sys.executable, "-c", code, ROOT, "--model", str(tmp_path), "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "64"],
                           input="", capture_output=True, text=True, timeout=300)
        assert p.returncode == code_want, p.stderr[-2000:]
        if code_want == 7:
            assert p.stdout.strip() == f"build {cfg['architecture'].lower()} []"
