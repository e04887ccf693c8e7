// The architectures this build of the engine can serve, by the name their model files carry. Each family's source file
// registers its own when the library is loaded, so a build holds exactly the families it was asked for.
#include "step_model.h"

namespace qwen38 {

namespace {
std::map<std::string, Architecture>& table() {
  static std::map<std::string, Architecture> t;
  return t;
}
}  // namespace

void register_architecture(const Architecture& a) { table()[a.name] = a; }

std::vector<std::string> architecture_names() {
  std::vector<std::string> names;
  for (const auto& [name, a] : table()) names.push_back(name);
  return names;
}

const Architecture& find_architecture(const std::string& name) {
  const auto it = table().find(name);
  if (it == table().end()) {
    std::string known;
    for (const std::string& n : architecture_names()) known += (known.empty() ? "" : ", ") + n;
    fail("architecture '" + name + "' is not in this build (it has: " + known + ")");
  }
  return it->second;
}

}  // namespace qwen38
